"""Throughput and per-kernel roofline fractions of the latent-attention / routed design beside the closest dense model of
the framework at equal size:  ``python bench.py --workload ruralorn``.

The dense neighbour has the same width, depth, vocabulary, heads and window, fp16 weights, and a SwiGLU feed-forward of as
many active parameters per token.  Both run on random weights through ``ZStreamerEngine`` (prefill passes and decode steps
timed with CUDA events on the device), then every kernel of a layer is timed alone, cold-cache.  A kernel's fraction is
(the larger of bytes / measured copy bandwidth and FLOPs / measured bf16 rate) / its time; bytes and FLOPs are those of the
operation, not of the way it is carried out.
"""
from __future__ import annotations

import os
import random
import sys
import tempfile
import time
import types
from typing import List, Optional

import torch

from ..format import synth
from ..format.config import ModelConfig

SHAPES = ("ruralorn-2k", "ruralorn-4k")


def dense_neighbour(c: ModelConfig) -> ModelConfig:
    """The windowed dense model of the same width, heads and active feed-forward size."""
    s, m = c.latent_spec(0), c.moe_spec(0)
    active = 2 * (m.top * m.ff + m.shared_ff)                  # rows of the two matrices an expert has
    d = synth.shape_config("small-128", quant="fp16")
    d.arch, d.num_layers, d.hidden_size, d.vocab_size = "mistral", c.num_layers, c.hidden_size, c.vocab_size
    d.num_heads = d.num_kv_heads = s.heads
    d.head_dim = 128
    d.intermediate_size = max(128, round(active / 3 / 128) * 128)
    d.sliding_window, d.max_seq_len, d.rope_theta = s.window, 32768, 10000.0
    return d


def _file(name: str, c: ModelConfig) -> str:
    path = os.path.join(tempfile.gettempdir(), f"zse_bench_{name}.zse")
    if not os.path.exists(path):
        t0 = time.time()
        synth.write_random_model(path + ".tmp", c, fast=True)
        os.replace(path + ".tmp", path)
        print(f"[bench] wrote {path} ({os.path.getsize(path) / 2**30:.1f} GiB) in {time.time() - t0:.0f}s", file=sys.stderr)
    return path


def run_engine(path: str, steps: int, warmup: int, seqs: int = 64, prompt: int = 3072) -> dict:
    """Prefill and decode of ``seqs`` random prompts; device time of the passes, and wall time of the decode steps."""
    from ..config import EngineConfig
    from ..engine import ZStreamerEngine
    from ..ops import native
    need = steps + warmup + 16
    eng = ZStreamerEngine(path, config=EngineConfig(max_seq_len=prompt + need + 64, max_batch_seqs=seqs,
                                                    max_batch_tokens=8192, prefill_chunk_size=2048,
                                                    max_prefill_per_step=16, decode_per_prefill=0,
                                                    max_queue_size=4 * seqs, enable_prefix_cache=False))
    rng = random.Random(1)
    v = eng.model_config.vocab_size
    for _ in range(seqs):
        if eng.add_request_tokens([rng.randrange(v) for _ in range(prompt)], max_tokens=need, temperature=0.0,
                                  stop_tokens=[]) is None:
            raise RuntimeError("the queue is full")
    runner = eng.runner

    def step():
        res = eng.step()
        if res.errors:
            raise RuntimeError(f"engine step failed: {res.errors[0]}")
        return res

    # passes of prompts only: later steps also carry the sequences that decode already
    runner.step_events, tokens = [], 0
    passes, counted = 0, []
    while eng.scheduler.num_waiting or eng.scheduler.num_prefilling:
        before = len(runner.step_events)
        res = step()
        if res.num_decode_tokens == 0 and len(runner.step_events) == before + 1:
            passes += 1
            if passes > 1:                                 # the first pass sets kernels up
                tokens += res.num_prefill_tokens
                counted.append(before)
    torch.cuda.synchronize()
    prefill_ms = sum(runner.step_events[i][0].elapsed_time(runner.step_events[i][1]) for i in counted)
    for _ in range(warmup):
        step()
    torch.cuda.synchronize()
    runner.step_events = []
    launches = runner.kernel_launches
    t0 = time.perf_counter()
    for _ in range(steps):
        step()
    torch.cuda.synchronize()
    wall = time.perf_counter() - t0
    ms = [a.elapsed_time(b) for a, b in runner.step_events]
    out = {"prefill_tok_s": round(tokens / prefill_ms * 1e3, 1) if prefill_ms else None,
           "prefill_tokens_timed": tokens, "decode_tok_s": round(seqs * len(ms) / sum(ms) * 1e3, 1),
           "decode_ms_per_step": round(sum(ms) / len(ms), 4), "decode_tok_s_e2e": round(seqs * steps / wall, 1),
           "e2e_ms_per_step": round(wall * 1e3 / steps, 4), "gpu_launches": runner.kernel_launches - launches,
           "weights_gb": round(eng.runner.model.weight_bytes / 2 ** 30, 2), "max_blocks": runner.max_blocks}
    runner.model.ops.check()
    eng.destroy()
    del eng, runner
    torch.cuda.empty_cache()
    return out


class _Table:
    def __init__(self, iters: int):
        from .profiler import KernelProfiler, measured_peaks
        self.prof, self.peaks, self.rows = KernelProfiler(iters=iters), measured_peaks(), []

    def add(self, phase: str, name: str, like: Optional[str], fn, nbytes: float, flops: float = 0.0) -> None:
        ms = self.prof.time(name, fn).ms
        floor = max(nbytes / (self.peaks["hbm_gbs"] * 1e9), flops / (self.peaks["tflops"] * 1e12)) * 1e3
        self.rows.append({"phase": phase, "kernel": name, "like": like, "us": round(ms * 1e3, 1),
                          "roofline_us": round(floor * 1e3, 1), "fraction": round(floor / ms, 3),
                          "bound": "tensor" if flops / self.peaks["tflops"] / 1e12 > nbytes / self.peaks["hbm_gbs"] / 1e9
                          else "memory"})


def kernel_table(shape: str, iters: int = 20, seqs: int = 64, ctx: int = 4096, chunk: int = 2048,
                 chunks: int = 4, only=()) -> List[dict]:
    """Kernels of one layer in a decode step of ``seqs`` sequences of ``ctx`` tokens and in a prefill pass of ``chunks``
    chunks; the dense neighbour's like kernel is named in ``like``."""
    from ..models.latent_moe import ChunkGroup, attention_splits
    from ..ops.backend import CudaOps, LinearWeight
    ops = CudaOps("cuda")
    c = synth.shape_config(shape)
    d = dense_neighbour(c)
    s, m, H = c.latent_spec(0), c.moe_spec(0), c.hidden_size
    bf, f16, f32 = torch.bfloat16, torch.float16, torch.float32
    T = _Table(iters)
    keep = lambda name: not only or any(o in name for o in only)

    def add(phase, name, like, fn, nbytes, flops=0.0):
        if keep(name):
            T.add(phase, name, like, fn, nbytes, flops)
    rnd = lambda *sh, dt=bf: (torch.randn(*sh, device="cuda") * 0.05).to(dt)
    lin = lambda n, k: ops.dense_linear(rnd(n, k))
    flin = lambda n, k, swiglu=False: LinearWeight("f16", n, k, rnd(n, k, dt=f16), None, swiglu, n * k * 2)
    hw, vw = s.heads * s.qk_dim, s.heads * s.vdim
    kr, row = s.kv_rank, s.row
    w_in, o = lin(s.in_width, H), lin(H, vw)
    ukv = rnd(s.heads * (s.dim + s.vdim), kr)
    L = types.SimpleNamespace(uk=ukv[: s.heads * s.dim], uv=ukv[s.heads * s.dim:], ukv=ops.dense_linear(ukv), moe=m,
                              router=lin(m.experts, H), up=rnd(m.experts * m.ff, H), down=rnd(m.experts * H, m.ff),
                              shared_up=rnd(m.shared_ff, H) if m.shared_ff else None,
                              shared_down=rnd(H, m.shared_ff) if m.shared_ff else None)
    nh, hd, I = d.num_heads, d.head_dim, d.intermediate_size
    fqkv, fo, fgu, fdown = flin(3 * nh * hd, H), flin(H, nh * hd), flin(2 * I, H, True), flin(H, I)
    bs, per_seq = 64, (ctx + 63) // 64
    blocks = seqs * per_seq
    rows = rnd(blocks, bs, row)
    tables = torch.arange(blocks, dtype=torch.int32, device="cuda").view(seqs, per_seq)
    fbs = 16
    fkv = rnd(seqs * ctx // fbs, 2, nh, fbs, hd, dt=f16)
    ftab = torch.arange(seqs * ctx // fbs, dtype=torch.int32, device="cuda").view(seqs, ctx // fbs)
    ii = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    freqs = torch.rand(s.rot_dims // 2, device="cuda")
    for phase, M in (("decode", seqs), ("prefill", chunk * chunks)):
        dec = phase == "decode"
        x, fx = rnd(M, H), rnd(M, H, dt=f16)
        inp, finp = rnd(M, s.in_width), rnd(M, 3 * nh * hd, dt=f16)
        planes = torch.zeros((8 if dec else 1) * M * max(s.in_width, 3 * nh * hd), device="cuda")
        pv = lambda n: planes[: (8 if dec else 1) * M * n].view(8 if dec else 1, M, n)
        res, att, fatt = torch.zeros(M, H, device="cuda"), rnd(M, vw), rnd(M, nh * hd, dt=f16)
        positions = ii([ctx - 1] * M) if dec else ii(list(range(chunk)) * chunks)
        slots = torch.arange(M, device="cuda") * (bs if dec else 1) % (blocks * bs)
        mm = lambda n, k: (2.0 * (n * k + M * k + M * n), 2.0 * M * n * k)
        if dec:
            add(phase, "input projection", "qkv projection", lambda: ops.linear_partial(w_in, x, M, pv(s.in_width)),
                *mm(s.in_width, H))
            add(phase, "qkv projection", None, lambda: ops.linear_partial(fqkv, fx, M, pv(3 * nh * hd)), *mm(3 * nh * hd, H))
        else:
            add(phase, "input projection", "qkv projection", lambda: ops.linear(w_in, x, M, inp), *mm(s.in_width, H))
            add(phase, "qkv projection", None, lambda: ops.linear(fqkv, fx, M, finp), *mm(3 * nh * hd, H))
        n_pl = 2 if dec else 0
        nw = rnd(kr)
        inv = torch.rand(hd // 2, device="cuda")
        traffic = M * (s.in_width * (4.0 * n_pl + 2) if dec else 2.0 * 2 * s.heads * s.rot_dim + 4.0 * row)
        add(phase, "latent norm + rotation + cache write", "rotation + cache write",
            lambda: ops.latent_prep(inp, pv(s.in_width), n_pl, rows, positions, slots, freqs, nw, s, 1e-6, M), traffic)
        traffic = M * 3.0 * nh * hd * (4 * n_pl + 2 if dec else 4)
        add(phase, "rotation + cache write", None,
            lambda: ops.rope_kv_write(finp, fkv, positions, slots, inv, M, nh, nh, hd, fbs,
                                      planes=planes if dec else None, n_planes=n_pl), traffic)
        if dec:
            ql, ol = rnd(M * s.heads * row), rnd(M * s.heads * kr)
            scratch = torch.zeros(M * 16 * s.heads * (kr + 2), device="cuda")
            fscratch = torch.zeros(M * nh * 16 * (hd + 2), device="cuda")
            rc = ops.n.row_cache(rows, tables)
            splits = attention_splits(M, (s.heads + 31) // 32, ctx, 16, ops.sm_count)
            add(phase, "queries into the latent", "output projection", lambda: ops.n.latent_absorb(inp, L.uk, ql, M, s),
                2.0 * (s.heads * s.dim * kr + M * hw + M * s.heads * row), 2.0 * M * s.heads * s.dim * kr)
            add(phase, "latent attention (with merge of splits)", "attention (with merge of splits)",
                lambda: ops.n.latent_attn(ql, rc, None, positions, ol, scratch, M, s, splits, 1,
                                          ops.status.ptr),
                2.0 * M * (ctx * row + s.heads * (row + kr)), 2.0 * M * ctx * s.heads * (row + kr))
            lens = ii([ctx] * M)
            add(phase, "attention (with merge of splits)", None,
                lambda: ops.attn_decode(finp, fkv, ftab, lens, fatt, M, nh, nh, hd, fbs, hd ** -0.5, fscratch, 1,
                                        window=d.sliding_window), 2.0 * M * (ctx * 2 * nh * hd + 2 * nh * hd),
                4.0 * M * ctx * nh * hd)
            add(phase, "values out of the latent + gate", "output projection",
                lambda: ops.n.latent_unabsorb(ol, L.uv, ops._gate_ptr(inp, s), inp.stride(0), att, M, s),
                2.0 * (s.heads * s.vdim * kr + M * s.heads * kr + 2 * M * vw), 2.0 * M * s.heads * s.vdim * kr)
        else:
            cu, p0 = ii([i * chunk for i in range(chunks + 1)]), ii([0] * chunks)
            ctab = tables.view(-1)[: chunks * (chunk // bs)].view(chunks, -1).contiguous()
            off = ii([i * chunk for i in range(chunks)])
            cc, kk = rnd(M * kr), rnd(M * s.rot_dim)
            kvx = rnd(M * L.ukv.N)
            rc = ops.n.row_cache(rows, ctab)
            ch = ops.n.Chunks(cu.data_ptr(), p0.data_ptr(), off.data_ptr(), 0, chunks, s.window)
            g = ChunkGroup(0, chunks, M, chunk)
            pairs = chunks * (chunk * (chunk + 1) // 2)
            add(phase, "gather of cached rows", "rotation + cache write", lambda: ops.n.latent_gather(rc, ch, M, s, cc, kk),
                4.0 * M * row)
            add(phase, "expansion of keys and values", "qkv projection",
                lambda: ops.n.gemm_bf16(L.ukv.data, L.ukv.N, cc, M, kvx, M, L.ukv.N, kr, L.ukv.N, 0, 1, ops.status.ptr),
                *mm(L.ukv.N, kr))
            add(phase, "chunk attention", "prefill attention",
                lambda: ops.n.latent_chunk(inp, kvx, L.ukv.N, s.heads * s.dim, kk, rc, ch, chunk, att,
                                           ops._gate_ptr(inp, s), s),
                2.0 * M * (hw + L.ukv.N + 2 * vw), 2.0 * pairs * s.heads * (s.qk_dim + s.vdim))
            ft = ftab.view(-1)[: chunks * chunk // fbs].view(chunks, -1).contiguous()
            add(phase, "prefill attention", None,
                lambda: ops.attn_prefill(finp, fkv, ft, cu, p0, fatt, chunks, M, chunk, nh, nh, hd, fbs, hd ** -0.5,
                                         window=d.sliding_window), 2.0 * M * 4 * nh * hd, 4.0 * pairs * nh * hd)
        add(phase, "output projection (latent)", "output projection", lambda: ops.linear_partial(o, att, M, pv(H)),
            *mm(H, vw))
        add(phase, "output projection", None, lambda: ops.linear_partial(fo, fatt, M, pv(H)), *mm(H, nh * hd))
        w1, fw1 = rnd(H), rnd(H, dt=f16)
        pl = 4 if dec else 1
        add(phase, "residual + norm (latent)", "residual + norm", lambda: ops.add_norm(res, planes, pl, None, w1, x, M, 1e-6),
            M * H * (4.0 * pl + 8 + 2))
        add(phase, "residual + norm", None, lambda: ops.add_rmsnorm(res, planes, pl, None, fw1, fx, M, 1e-6),
            M * H * (4.0 * pl + 8 + 2))
        ws = ops.moe_workspace([m], H, M, bf)
        per = m.top + (m.shared_ff > 0)
        y32 = M <= ws.F32_ROWS
        touched = min(m.experts, M * m.top)
        act = m.top * m.ff + m.shared_ff
        add(phase, "experts' sum + residual + norm", "residual + norm",
            lambda: ops.add_norm(res, planes, 0, ws.y[: M * per * H * (4 if y32 else 2)].view(f32 if y32 else bf).view(
                M, per, H), w1, x, M, 1e-6), M * H * (per * (4.0 if y32 else 2.0) + 8 + 2))
        ops.moe(L, x, M, ws)                               # tables for the single kernels below
        tile = ops.n.moe_tile_rows(M, m.experts, m.top)
        add(phase, "router logits", "output projection",
            lambda: ops.linear_partial(L.router, x, M, ws.router_views[m.experts]), *mm(m.experts, H))
        add(phase, "routing + sorted rows", "rotation + cache write",
            lambda: ops.n.moe_route(ws.router, 1, M, m, tile, x, H, per, ws), 4.0 * M * m.top * H)
        add(phase, "feed-forward (all routed kernels)", "gate/up + down projections", lambda: ops.moe(L, x, M, ws),
            2.0 * (touched * 2 * m.ff * H + 2 * m.shared_ff * H + 2 * M * (act + m.top * H)), 4.0 * M * act * H)
        for name, epi in (("experts up + gelu", 0), ("experts down", 2 if y32 else 1)):
            add(phase, name, "gate/up projection" if epi == 0 else "down projection",
                ops.moe_product_call(L, x, M, ws, epi),
                2.0 * (touched * m.ff * H + m.shared_ff * H + M * act) + (2.0 if epi != 2 else 4.0) * M * per * H,
                2.0 * M * act * H)
        fa = rnd(M, I, dt=f16)
        tmp = torch.empty(M, 2 * I, dtype=f16, device="cuda")
        add(phase, "gate/up projection", None, lambda: ops.linear_swiglu(fgu, fx, M, fa, tmp=tmp),
            2.0 * (2 * I * H + M * H + M * I), 4.0 * M * I * H)
        add(phase, "down projection", None, lambda: ops.linear_partial(fdown, fa, M, pv(H)), *mm(H, I))

        def ff():
            ops.linear_swiglu(fgu, fx, M, fa, tmp=tmp)
            ops.linear_partial(fdown, fa, M, pv(H))
        add(phase, "gate/up + down projections", None, ff, 2.0 * (3 * I * H + 2 * M * (H + I)), 6.0 * M * I * H)
    ops.check()
    by = {(r["phase"], r["kernel"]): r for r in T.rows}
    for r in T.rows:
        like = by.get((r["phase"], r["like"])) if r["like"] else None
        r["like_fraction"] = like["fraction"] if like else None
    return T.rows


def markdown(rows: List[dict], neighbour: str = "dense") -> str:
    out = [f"| phase | kernel | us | roofline us | fraction | bound | like kernel ({neighbour}) | its us | its fraction |",
           "|---|---|---|---|---|---|---|---|---|"]
    by = {(r["phase"], r["kernel"]): r for r in rows}
    for r in rows:
        like = by.get((r["phase"], r["like"]))
        if like:
            out.append(f"| {r['phase']} | {r['kernel']} | {r['us']} | {r['roofline_us']} | {r['fraction']} | {r['bound']} | "
                       f"{r['like']} | {like['us']} | {like['fraction']} |")
    return "\n".join(out)


def run(steps: int, warmup: int, shapes=SHAPES, kernels_file: Optional[str] = None) -> dict:
    """Both models at every shape; ``kernels_file``: also time the kernels one by one and write the table there."""
    out = {}
    for shape in shapes:
        c = synth.shape_config(shape)
        out[shape] = {"ruralorn": run_engine(_file(shape, c), steps, warmup),
                      "dense": run_engine(_file(shape + "-dense", dense_neighbour(c)), steps, warmup)}
    if kernels_file:
        with open(kernels_file, "w") as f:
            for shape in shapes:
                f.write(f"## {shape}\n\n{markdown(kernel_table(shape))}\n\n")
                torch.cuda.empty_cache()
    return out


if __name__ == "__main__":       # one or a few kernels, for a profiler: --only takes parts of their names
    import argparse
    ap = argparse.ArgumentParser()
    ap.add_argument("--shape", default=SHAPES[0], choices=SHAPES)
    ap.add_argument("--only", default="")
    ap.add_argument("--iters", type=int, default=20)
    a = ap.parse_args()
    for row in kernel_table(a.shape, iters=a.iters, only=[x for x in a.only.split(",") if x]):
        print(row)
