"""Throughput and per-kernel roofline fractions of the design that mixes chunked attention and matrix memories (Nimelorn)
beside the closest dense model of the framework at equal size:  ``python bench.py --workload nimelorn``.

Method and table as in ``design_bench``.  The dense neighbour has the same width, depth, vocabulary, query and key/value heads
and a window as long as the design's chunks, fp16 weights, and a SwiGLU feed-forward of as many active parameters per token as
the design's layers have on average.
"""
from __future__ import annotations

import types
from typing import List, Optional

import torch

from ..format import synth
from ..format.config import DenseSpec, HeadsSpec, MatrixMemorySpec, ModelConfig, MoESpec
from . import design_bench as base

SHAPES = ("nimelorn-2k", "nimelorn-4k")


def dense_neighbour(c: ModelConfig) -> ModelConfig:
    a = next(s for s in (c.mixer_spec(i) for i in range(c.num_layers)) if isinstance(s, HeadsSpec))
    active = 0                                         # rows of matrices as wide as the model
    for i in range(c.num_layers):
        f = c.ff_spec(i)
        if isinstance(f, MoESpec):
            active += 3 * (f.top * f.ff + f.shared_ff)
        elif isinstance(f, DenseSpec):
            active += 2 * f.ff
    d = synth.shape_config("small-128", quant="fp16")
    d.arch, d.num_layers, d.hidden_size, d.vocab_size = "mistral", c.num_layers, c.hidden_size, c.vocab_size
    d.num_heads, d.num_kv_heads, d.head_dim = a.heads, a.kv_heads, 128
    d.intermediate_size = max(128, round(active / 3 / c.num_layers / 128) * 128)
    d.sliding_window, d.max_seq_len, d.rope_theta = a.chunk, 32768, 10000.0
    return d


def kernel_table(shape: str, iters: int = 20, seqs: int = 64, ctx: int = 4096, chunk: int = 2048, chunks: int = 4,
                 only=()) -> List[dict]:
    """Kernels of the layers in a decode step of ``seqs`` sequences of ``ctx`` tokens and in a prefill pass of ``chunks``
    prompts; the dense neighbour's like kernel is named in ``like``."""
    from ..models.hybrid import EmbedDesign, PagedHeads
    from ..ops.backend import CudaOps, LinearWeight
    ops = CudaOps("cuda")
    c = synth.shape_config(shape)
    d = dense_neighbour(c)
    specs = [c.mixer_spec(i) for i in range(c.num_layers)]
    ffs = [c.ff_spec(i) for i in range(c.num_layers)]
    s = next(x for x in specs if isinstance(x, HeadsSpec) and x.own_kv)
    r = next(x for x in specs if isinstance(x, MatrixMemorySpec))
    m = next(x for x in ffs if isinstance(x, MoESpec))
    ff = next(x for x in ffs if isinstance(x, DenseSpec)).ff
    H, bf, f16, f32 = c.hidden_size, torch.bfloat16, torch.float16, torch.float32
    T = base._Table(iters)

    def add(phase, name, like, fn, nbytes, flops=0.0):
        if not only or any(o in name for o in only):
            T.add(phase, name, like, fn, nbytes, flops)
    rnd = lambda *sh, dt=bf: (torch.randn(*sh, device="cuda") * 0.05).to(dt)
    lin = lambda n, k: ops.dense_linear(rnd(n, k))
    flin = lambda n, k, swiglu=False: LinearWeight("f16", n, k, rnd(n, k, dt=f16), None, swiglu, n * k * 2)
    ii = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    vw, rw = s.heads * s.vdim, r.heads * r.vdim
    w_in, o = lin(s.in_width, H), lin(H, vw)
    w_mem, o_mem = lin(r.in_width, H), lin(H, rw)
    w_if = ops.dense_linear(w_mem.data[r.if_col: r.if_col + 2 * r.heads])
    up, down = lin(ff, H), lin(H, ff)
    up_rows = lambda n: (n + 63) // 64 * 128
    L = types.SimpleNamespace(q_norm=rnd(s.dim), k_norm=rnd(s.dim), head_norm=rnd(rw), moe=m, router=lin(m.router_rows, H),
                              if_bias=torch.zeros(2 * r.heads, device="cuda"), up=rnd(m.experts * up_rows(m.ff), H),
                              down=rnd(m.experts * H, m.ff), shared_up=rnd(up_rows(m.shared_ff), H),
                              shared_down=rnd(H, m.shared_ff))
    nh, nkv, hd, I = d.num_heads, d.num_kv_heads, d.head_dim, d.intermediate_size
    qkv_w = (nh + 2 * nkv) * hd
    fqkv, fo, fgu, fdown = flin(qkv_w, H), flin(H, nh * hd), flin(2 * I, H, True), flin(H, I)
    bs, per_seq = 64, (ctx + 63) // 64
    blocks = seqs * per_seq
    kv = PagedHeads(rnd(blocks, 1, 1, bs, s.row), s)
    tables = torch.arange(blocks, dtype=torch.int32, device="cuda").view(seqs, per_seq)
    fbs = 16
    fkv = rnd(seqs * ctx // fbs, 2, nkv, fbs, hd, dt=f16)
    ftab = torch.arange(seqs * ctx // fbs, dtype=torch.int32, device="cuda").view(seqs, ctx // fbs)
    state = torch.zeros(2 * seqs, r.state_floats, device="cuda")
    inv = torch.rand(hd // 2, device="cuda")
    emb = EmbedDesign(rnd(c.vocab_size, H), 1.0, 10000.0, rnd(H), rnd(65522, H), 65521, 31337, 1009)
    last = ii([0] * 2 * seqs)
    for phase, M in (("decode", seqs), ("prefill", chunk * chunks)):
        dec = phase == "decode"
        S = seqs if dec else chunks
        x, fx = rnd(M, H), rnd(M, H, dt=f16)
        inp, finp = rnd(M, s.in_width), rnd(M, qkv_w, dt=f16)
        mem = rnd(M, r.in_width)
        planes = torch.zeros((8 if dec else 1) * M * max(s.in_width, r.in_width, qkv_w), device="cuda")
        pv = lambda n: planes[: (8 if dec else 1) * M * n].view(8 if dec else 1, M, n)
        res, att, fatt, mo = torch.zeros(M, H, device="cuda"), rnd(M, vw), rnd(M, nh * hd, dt=f16), rnd(M, rw)
        positions = ii([ctx - 1] * M) if dec else ii(list(range(chunk)) * chunks)
        slots = torch.arange(M, device="cuda") * (bs if dec else 1) % (blocks * bs)
        cu = None if dec else ii([i * chunk for i in range(chunks + 1)])
        row_seq = None if dec else ii([i for i in range(chunks) for _ in range(chunk)])
        p0 = ii([0] * chunks)
        rows = ii([[2 * i for i in range(S)], [2 * i + 1 for i in range(S)]])
        ids = torch.randint(c.vocab_size, (M,), dtype=torch.int32, device="cuda")
        mm = lambda n, k: (2.0 * (n * k + M * k + M * n), 2.0 * M * n * k)
        add(phase, "embedding (bigram, sinusoid, norm)", "residual + norm",
            lambda: ops.embed_design(emb, ids, positions, row_seq, cu, rows, last, res, x, M, S, 1e-6), M * H * 10.0)

        def project(w, dst):
            if dec:
                ops.linear_partial(w, x, M, pv(w.N))
            else:
                ops.linear(w, x, M, dst)
        add(phase, "input projection (attention)", "qkv projection", lambda: project(w_in, inp), *mm(s.in_width, H))
        add(phase, "input projection (memory)", "qkv projection", lambda: project(w_mem, mem), *mm(r.in_width, H))
        if dec:
            add(phase, "qkv projection", None, lambda: ops.linear_partial(fqkv, fx, M, pv(qkv_w)), *mm(qkv_w, H))
        else:
            add(phase, "qkv projection", None, lambda: ops.linear(fqkv, fx, M, finp), *mm(qkv_w, H))
        n_pl = 2 if dec else 0
        gates, gp = torch.zeros(M * 2 * r.heads, device="cuda"), torch.zeros(8, M * 2 * r.heads, device="cuda")
        add(phase, "head norms + cache write", "rotation + cache write",
            lambda: ops.heads_prep(inp, pv(s.in_width), n_pl, kv, slots, L, s, 1e-6, M),
            M * (s.in_width * (4.0 * n_pl + 2) if dec else 4.0 * s.gate_col))
        add(phase, "rotation + cache write", None,
            lambda: ops.rope_kv_write(finp, fkv, positions, slots, inv, M, nh, nkv, hd, fbs, planes=planes if dec else None,
                                      n_planes=n_pl), M * 1.0 * qkv_w * (4 * n_pl + 2 if dec else 4))
        if not dec:
            add(phase, "gates' projection (memory)", "output projection", lambda: ops.linear_partial(w_if, x, M, gp),
                *mm(2 * r.heads, H))
        add(phase, "logarithms of the gates", "rotation + cache write",
            lambda: ops.memory_prep(mem, pv(r.in_width), n_pl, gp, 1, gates, L, r, M),
            M * (r.in_width * (4.0 * n_pl + 2) if dec else 16.0 * r.heads))
        io = 2.0 * M * (r.if_col + rw)
        if dec:
            scratch = torch.zeros(M * 16 * s.heads * (s.vdim + 2), device="cuda")
            fscratch = torch.zeros(M * nh * 16 * (hd + 2), device="cuda")
            stub = types.SimpleNamespace(heads_specs=[s])
            from ..models.hybrid import HybridModel
            splits = HybridModel.attention_splits(stub, M, ctx, 16, ops.sm_count)
            add(phase, "attention over chunks (with merge of splits)", "attention (with merge of splits)",
                lambda: ops.heads_attn(inp, kv, tables, None, positions, att, M, s, scratch, splits),
                2.0 * M * (ctx * s.row + s.heads * (s.dim + s.vdim)), 2.0 * M * ctx * s.heads * (s.dim + s.vdim))
            lens = ii([ctx] * M)
            fsplits = 1 << max(0, ((2 * ops.sm_count + M * nkv - 1) // (M * nkv)).bit_length() - 1)
            add(phase, "attention (with merge of splits)", None,
                lambda: ops.attn_decode(finp, fkv, ftab, lens, fatt, M, nh, nkv, hd, fbs, hd ** -0.5, fscratch, fsplits,
                                        window=d.sliding_window), 2.0 * M * (ctx * 2 * nkv * hd + 2 * nh * hd),
                4.0 * M * ctx * nh * hd)
            add(phase, "memory step (state, read-out, head norm, gate)", "attention (with merge of splits)",
                lambda: ops.memory_tokens(mem, gates, state, 0, rows, None, L, mo, S, M, r, 1e-6),
                8.0 * M * r.state_floats + io, 4.0 * M * r.heads * r.dim * r.vdim)
        else:
            ctab = tables.view(-1)[: chunks * (chunk // bs)].view(chunks, -1).contiguous()
            pairs = chunks * (chunk * (chunk + 1) // 2)
            ft = ftab.view(-1)[: chunks * chunk // fbs].view(chunks, -1).contiguous()
            add(phase, "attention over chunks", "prefill attention",
                lambda: ops.heads_attn_chunks(inp, kv, ctab, cu, p0, positions, 0, chunks, chunk, att, s),
                2.0 * M * (s.in_width + vw), 2.0 * pairs * s.heads * (s.dim + s.vdim))
            add(phase, "prefill attention", None,
                lambda: ops.attn_prefill(finp, fkv, ft, cu, p0, fatt, chunks, M, chunk, nh, nkv, hd, fbs, hd ** -0.5,
                                         window=d.sliding_window), 2.0 * M * (qkv_w + nh * hd), 4.0 * pairs * nh * hd)
            ws = ops.memory_workspace([r], M)
            add(phase, "memory in chunks (with head norm, gate)", "prefill attention",
                lambda: ops.memory_chunks(mem, gates, state, 0, rows, cu, L, mo, 0, chunks, 0, M, r, 1e-6, ws),
                io + 8.0 * S * r.state_floats, 4.0 * M * r.heads * r.dim * r.vdim)
        add(phase, "output projection (attention)", "output projection", lambda: ops.linear_partial(o, att, M, pv(H)),
            *mm(H, vw))
        add(phase, "output projection (memory)", "output projection", lambda: ops.linear_partial(o_mem, mo, M, pv(H)),
            *mm(H, rw))
        add(phase, "output projection", None, lambda: ops.linear_partial(fo, fatt, M, pv(H)), *mm(H, nh * hd))
        w1, fw1 = rnd(H), rnd(H, dt=f16)
        pl = 4 if dec else 1
        add(phase, "norm + residual", "residual + norm",
            lambda: ops.post_norm(res, planes, pl, None, w1, None, x, M, 1e-6), M * H * (4.0 * pl + 8 + 2))
        add(phase, "residual + norm", None, lambda: ops.add_rmsnorm(res, planes, pl, None, fw1, fx, M, 1e-6),
            M * H * (4.0 * pl + 8 + 2))
        act = rnd(M, ff)
        add(phase, "dense up + squared relu", "gate/up projection", lambda: ops.linear_act(up, x, M, act, "relu2"), *mm(ff, H))
        add(phase, "dense down", "down projection", lambda: ops.linear_partial(down, act, M, pv(H)), *mm(H, ff))
        ws = ops.moe_workspace([m], H, M, bf)
        per = m.top + 1
        y32 = M <= ws.F32_ROWS
        touched = min(m.experts, M * m.top)
        act_w = m.top * m.ff + m.shared_ff
        add(phase, "experts' sum + norm + residual", "residual + norm",
            lambda: ops.post_norm(res, planes, 0, ws.y[: M * per * H * (4 if y32 else 2)].view(f32 if y32 else bf).view(
                M, per, H), w1, None, x, M, 1e-6), M * H * (per * (4.0 if y32 else 2.0) + 8 + 2))
        ops.moe(L, x, M, ws)                               # tables for the single kernels below
        tile = ops.n.moe_tile_rows(M, m.experts, m.top)
        add(phase, "router logits", "output projection",
            lambda: ops.linear_partial(L.router, x, M, ws.router_views[m.router_rows]), *mm(m.router_rows, H))
        add(phase, "routing + sorted rows", "rotation + cache write",
            lambda: ops.n.moe_route(ws.router, 1, M, m, tile, x, H, per, ws), 4.0 * M * m.top * H)
        add(phase, "feed-forward (all routed kernels)", "gate/up + down projections", lambda: ops.moe(L, x, M, ws),
            2.0 * (touched * 3 * m.ff * H + 3 * m.shared_ff * H + 2 * M * (act_w + m.top * H)), 6.0 * M * act_w * H)
        add(phase, "experts gate/up + clamped glu", "gate/up projection", ops.moe_product_call(L, x, M, ws, 3),
            2.0 * (2 * touched * m.ff * H + 2 * m.shared_ff * H + M * act_w) + 2.0 * M * per * H, 4.0 * M * act_w * H)
        add(phase, "experts down", "down projection", ops.moe_product_call(L, x, M, ws, 2 if y32 else 1),
            2.0 * (touched * m.ff * H + m.shared_ff * H + M * act_w) + (4.0 if y32 else 2.0) * M * per * H,
            2.0 * M * act_w * H)
        fa = rnd(M, I, dt=f16)
        tmp = torch.empty(M, 2 * I, dtype=f16, device="cuda")
        add(phase, "gate/up projection", None, lambda: ops.linear_swiglu(fgu, fx, M, fa, tmp=tmp),
            2.0 * (2 * I * H + M * H + M * I), 4.0 * M * I * H)
        add(phase, "down projection", None, lambda: ops.linear_partial(fdown, fa, M, pv(H)), *mm(H, I))

        def both():
            ops.linear_swiglu(fgu, fx, M, fa, tmp=tmp)
            ops.linear_partial(fdown, fa, M, pv(H))
        add(phase, "gate/up + down projections", None, both, 2.0 * (3 * I * H + 2 * M * (H + I)), 6.0 * M * I * H)
        del planes, ws
        torch.cuda.empty_cache()
    ops.check()
    by = {(x["phase"], x["kernel"]): x for x in T.rows}
    for x in T.rows:
        like = by.get((x["phase"], x["like"])) if x["like"] else None
        x["like_fraction"] = like["fraction"] if like else None
    return T.rows


def run(steps: int, warmup: int, shapes=SHAPES, kernels_file: Optional[str] = None) -> dict:
    """Both models at every shape; ``kernels_file``: also time the kernels one by one and write the table there."""
    out = {}
    for shape in shapes:
        c = synth.shape_config(shape)
        out[shape] = {"nimelorn": base.run_engine(base._file(shape, c), steps, warmup),
                      "dense": base.run_engine(base._file(shape + "-dense", dense_neighbour(c)), steps, warmup)}
    if kernels_file:
        with open(kernels_file, "w") as f:
            for shape in shapes:
                f.write(f"## {shape}\n\n{base.markdown(kernel_table(shape))}\n\n")
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
