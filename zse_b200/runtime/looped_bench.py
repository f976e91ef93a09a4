"""Throughput and per-kernel roofline fractions of the design of looped layers (Movinex) beside the closest model of the
framework at equal size, a Nimelorn one:  ``python bench.py --workload movinex``.

Method and table as in ``design_bench``.  The neighbour has the same width, vocabulary, heads, experts and number of layer
runs, and matrix memories whose state is as large as the state spaces'; it runs the like kernels, among them many of the same
ones in another variant.
"""
from __future__ import annotations

import types
from typing import List, Optional

import torch

from ..format import synth
from ..format.config import DenseSpec, HeadsSpec, MatrixMemorySpec, ModelConfig, MoESpec, StateSpaceSpec
from . import design_bench as base

NEIGHBOURS = {"movinex-2k": "nimelorn-2k", "movinex-4k": "nimelorn-4k"}
SHAPES = tuple(NEIGHBOURS)


def _first(c: ModelConfig, kind, which=lambda s: True):
    return next(s for i in range(c.num_layers) for s in (c.mixer_spec(i), c.ff_spec(i)) if isinstance(s, kind) and which(s))


def kernel_table(shape: str, iters: int = 20, seqs: int = 64, ctx: int = 4096, chunk: int = 2048, chunks: int = 4,
                 only=()) -> List[dict]:
    """Kernels of the layers in a decode step of ``seqs`` sequences of ``ctx`` tokens and in a prefill pass of ``chunks``
    prompts; the neighbour's like kernel is named in ``like``."""
    from ..models.hybrid import EmbedDesign, HybridModel, PagedHeads
    from ..ops.backend import CudaOps
    ops = CudaOps("cuda")
    c, nb = synth.shape_config(shape), synth.shape_config(NEIGHBOURS[shape])
    H, bf, f32 = c.hidden_size, torch.bfloat16, torch.float32
    full, win = (_first(c, HeadsSpec, lambda s, w=w: bool(s.window) == w) for w in (False, True))
    sp, m, ff = _first(c, StateSpaceSpec), _first(c, MoESpec), _first(c, DenseSpec).ff
    n_at, n_mem, n_m, n_ff = _first(nb, HeadsSpec), _first(nb, MatrixMemorySpec), _first(nb, MoESpec), _first(nb, DenseSpec).ff
    T = base._Table(iters)

    def add(phase, name, like, fn, nbytes, flops=0.0):
        if not only or any(o in name for o in only):
            T.add(phase, name, like, fn, nbytes, flops)
    rnd = lambda *sh, dt=bf: (torch.randn(*sh, device="cuda") * 0.05).to(dt)
    lin = lambda n, k: ops.dense_linear(rnd(n, k))
    ii = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    zeros = lambda *s: torch.zeros(*s, device="cuda")
    up_rows = lambda n: (n + 63) // 64 * 128
    experts = lambda e: types.SimpleNamespace(
        moe=e, router=lin(e.router_rows, H), up=rnd(e.experts * up_rows(e.ff), H), down=rnd(e.experts * H, e.ff),
        shared_up=rnd(up_rows(e.shared_ff), H) if e.shared_ff else None,
        shared_down=rnd(H, e.shared_ff) if e.shared_ff else None)
    ours, theirs = experts(m), experts(n_m)
    heads_layer = lambda s: types.SimpleNamespace(
        q_norm=rnd(s.dim) if s.learned_norm else None, k_norm=rnd(s.dim) if s.learned_norm else None,
        bias=rnd(s.in_width) if s.bias else None, freqs=ops.rotation(s.rot_dims, s.rot_base))
    L_full, L_win, L_at = heads_layer(full), heads_layer(win), heads_layer(n_at)
    L_sp = types.SimpleNamespace(conv_w=rnd(sp.conv, sp.conv_width, dt=f32), conv_b=zeros(sp.conv_width),
                                 dt_bias=zeros(sp.heads), neg_a=-torch.ones(sp.heads, device="cuda"), D=zeros(sp.heads),
                                 w_in=lin(sp.in_width, H), out_norm=rnd(sp.inner))
    L_mem = types.SimpleNamespace(head_norm=rnd(n_mem.heads * n_mem.vdim), if_bias=zeros(2 * n_mem.heads))
    w = {k: lin(s.in_width, H) for k, s in (("full", full), ("win", win), ("at", n_at), ("mem", n_mem))}
    o = {k: lin(H, s.heads * s.vdim) for k, s in (("at", n_at), ("sp", sp), ("mem", n_mem))}
    loop_in = lin(H, 2 * H)
    gate_up = ops.glu_linear(rnd(ff, H), rnd(ff, H), bf)
    down, n_up, n_down = lin(H, ff), lin(n_ff, H), lin(H, n_ff)
    bs, per_seq = 64, (ctx + 63) // 64
    blocks = seqs * per_seq
    pool = rnd(blocks, 1, 1, bs, max(full.row, win.row, n_at.row))
    kv = {k: PagedHeads(pool, s) for k, s in (("full", full), ("win", win), ("at", n_at))}
    tables = torch.arange(blocks, dtype=torch.int32, device="cuda").view(seqs, per_seq)
    state = zeros(2 * seqs, max(sp.state_floats, n_mem.state_floats))
    emb = EmbedDesign(rnd(c.vocab_size, H), 1.0, 10000.0, rnd(H), rnd(65522, H), 65521, 31337, 1009)
    last = ii([0] * 2 * seqs)
    for phase, M in (("decode", seqs), ("prefill", chunk * chunks)):
        dec = phase == "decode"
        S, n_buf = (seqs, 8) if dec else (chunks, 1)
        x, both = rnd(M, H), rnd(M, 2 * H)
        widest = max(s.in_width for s in (full, win, sp, n_at, n_mem))
        planes = zeros(n_buf * M * widest)
        pv = lambda n: planes[: n_buf * M * n].view(n_buf, M, n)
        res = zeros(M, H)
        positions = ii([ctx - 1] * M) if dec else ii(list(range(chunk)) * chunks)
        slots = torch.arange(M, device="cuda") * (bs if dec else 1) % (blocks * bs)
        cu = None if dec else ii([i * chunk for i in range(chunks + 1)])
        row_seq = None if dec else ii([i for i in range(chunks) for _ in range(chunk)])
        p0 = ii([0] * chunks)
        rows = ii([[2 * i for i in range(S)], [2 * i + 1 for i in range(S)]])
        ids = torch.randint(c.vocab_size, (M,), dtype=torch.int32, device="cuda")
        mm = lambda n, k: (2.0 * (n * k + M * k + M * n), 2.0 * M * n * k)
        add(phase, "embedding (two places)", "embedding", lambda: ops.embedding(emb.table, ids, res, M, copy=both[:, H:]),
            M * H * 8.0)
        add(phase, "embedding", None,
            lambda: ops.embed_design(emb, ids, positions, row_seq, cu, rows, last, res, x, M, S, 1e-6), M * H * 10.0)
        add(phase, "product of a loop's pass", "output projection", lambda: ops.linear_partial(loop_in, both, M, pv(H)),
            *mm(H, 2 * H))

        def project(lw, dst, side=None):
            if dec:
                ops.linear_partial(lw, x, M, pv(lw.N))
            else:
                ops.linear(lw, x, M, dst, side=side)
        inp = {k: rnd(M, s.in_width) for k, s in (("full", full), ("win", win), ("sp", sp), ("at", n_at), ("mem", n_mem))}
        side = zeros(M * (sp.in_width - sp.dt_col))
        for name, key, like in (("attention", "full", "attention"), ("windowed attention", "win", "attention")):
            add(phase, f"input projection ({name})", "input projection", lambda k=key: project(w[k], inp[k]),
                *mm(w[key].N, H))
        add(phase, "input projection (state space)", "input projection (memory)",
            lambda: project(L_sp.w_in, inp["sp"], (sp.dt_col, side)), *mm(sp.in_width, H))
        add(phase, "input projection", None, lambda: project(w["at"], inp["at"]), *mm(n_at.in_width, H))
        add(phase, "input projection (memory)", None, lambda: project(w["mem"], inp["mem"]), *mm(n_mem.in_width, H))
        n_pl = 2 if dec else 0
        moved = lambda s: M * (s.in_width * (4.0 * n_pl + 2) if dec else 2.0 * (s.gate_col + (s.heads + s.kv_heads) * s.dim
                                                                               + s.kv_heads * s.vdim))
        for name, key, s, L, like in (("norms, bias, temperature, cache write", "full", full, L_full, "norms, cache write"),
                                      ("norms, rotation, cache write", "win", win, L_win, "norms, cache write"),
                                      ("norms, cache write", "at", n_at, L_at, None)):
            add(phase, name, like,
                lambda k=key, s=s, L=L: ops.heads_prep(inp[k], pv(s.in_width), n_pl, kv[k], slots, L, s, 1e-6, M, positions),
                moved(s))
        xbc, dt = rnd(M, sp.conv_width), zeros(M, sp.heads)
        add(phase, "convolution, step sizes", "norms, cache write",
            lambda: ops.state_space_prep(inp["sp"], pv(sp.in_width), n_pl, side, xbc, dt, state, 0, rows, row_seq, cu, L_sp, sp,
                                         M, S),
            M * (sp.in_width * 4.0 * n_pl + 2.0 * (sp.x_col + sp.conv_width) if dec else 4.0 * sp.conv_width + 8.0 * sp.heads)
            + 8.0 * S * (sp.conv - 1) * sp.conv_width)
        gates, gp = zeros(M * 2 * n_mem.heads), zeros(8, M * 2 * n_mem.heads)
        out = {k: rnd(M, s.heads * s.vdim) for k, s in (("full", full), ("win", win), ("sp", sp), ("at", n_at), ("mem", n_mem))}
        seen = lambda s, p: min(p + 1, s.window + s.keep_first) if s.window else p + 1
        sp_io = 2.0 * M * (sp.conv_width + 2 * sp.inner) + 4.0 * M * sp.heads
        mem_io = 2.0 * M * (n_mem.if_col + n_mem.heads * n_mem.vdim)
        if dec:
            for name, key, s, like in (("attention rows", "full", full, "chunked attention rows"),
                                       ("windowed attention rows", "win", win, "chunked attention rows"),
                                       ("chunked attention rows", "at", n_at, None)):
                splits = HybridModel.attention_splits(types.SimpleNamespace(heads_specs=[s]), M, ctx, 16, ops.sm_count)
                scratch = zeros(M * splits * s.heads * (s.vdim + 2))
                n = seen(s, ctx - 1)
                add(phase, name, like,
                    lambda k=key, s=s, sc=scratch, sp_=splits: ops.heads_attn(inp[k], kv[k], tables, None, positions, out[k],
                                                                              M, s, sc, sp_),
                    2.0 * M * (n * s.row + s.heads * (s.dim + s.vdim) + s.gate_width),
                    2.0 * M * n * s.heads * (s.dim + s.vdim))
            add(phase, "state space step", "memory step",
                lambda: ops.state_space_tokens(inp["sp"], xbc, dt, state, 0, rows, None, L_sp, out["sp"], S, M, sp),
                8.0 * M * sp.heads * sp.state * sp.vdim + sp_io, 4.0 * M * sp.heads * sp.state * sp.vdim)
            add(phase, "memory step", None,
                lambda: ops.memory_tokens(inp["mem"], gates, state, 0, rows, None, L_mem, out["mem"], S, M, n_mem, 1e-6),
                8.0 * M * n_mem.state_floats + mem_io, 4.0 * M * n_mem.heads * n_mem.dim * n_mem.vdim)
        else:
            ctab = tables.view(-1)[: chunks * (chunk // bs)].view(chunks, -1).contiguous()
            for name, key, s, like in (("attention tiles", "full", full, "chunked attention tiles"),
                                       ("windowed attention tiles", "win", win, "chunked attention tiles"),
                                       ("chunked attention tiles", "at", n_at, None)):
                pairs = chunks * sum(seen(s, p) for p in range(chunk))
                add(phase, name, like,
                    lambda k=key, s=s: ops.heads_attn_chunks(inp[k], kv[k], ctab, cu, p0, positions, 0, chunks, chunk, out[k],
                                                             s),
                    2.0 * M * (s.in_width + s.heads * s.vdim), 2.0 * pairs * s.heads * (s.dim + s.vdim))
            ws = ops.memory_workspace([n_mem], M)
            add(phase, "state space in chunks", "memory in chunks",
                lambda: ops.state_space_chunks(inp["sp"], xbc, dt, state, 0, rows, cu, L_sp, out["sp"], 0, chunks, M, sp),
                sp_io + 8.0 * S * sp.heads * sp.state * sp.vdim, 4.0 * M * sp.heads * sp.state * sp.vdim)
            add(phase, "memory in chunks", None,
                lambda: ops.memory_chunks(inp["mem"], gates, state, 0, rows, cu, L_mem, out["mem"], 0, chunks, 0, M, n_mem,
                                          1e-6, ws), mem_io + 8.0 * S * n_mem.state_floats,
                4.0 * M * n_mem.heads * n_mem.dim * n_mem.vdim)
        add(phase, "norm in parts", "norm + residual",
            lambda: ops.group_norm(out["sp"], L_sp.out_norm, sp.norm_groups, M, 1e-6), 4.0 * M * sp.inner)
        add(phase, "output projection (state space)", "output projection",
            lambda: ops.linear_partial(o["sp"], out["sp"], M, pv(H)), *mm(H, sp.inner))
        add(phase, "output projection", None, lambda: ops.linear_partial(o["at"], out["at"], M, pv(H)),
            *mm(H, n_at.heads * n_at.vdim))
        w1, s1 = rnd(H), rnd(H)
        pl = 4 if dec else 1
        add(phase, "scale + residual + norm", "norm + residual",
            lambda: ops.add_norm(res, planes, pl, None, w1, x, M, 1e-6, scale=s1, offset=1.0), M * H * (4.0 * pl + 8 + 2))
        add(phase, "residual beside the embedding", "norm + residual",
            lambda: ops.add_norm(res, planes, pl, None, None, both[:, :H], M, 1e-6, scale=s1), M * H * (4.0 * pl + 8 + 2))
        add(phase, "norm + residual", None, lambda: ops.post_norm(res, planes, pl, None, w1, None, x, M, 1e-6),
            M * H * (4.0 * pl + 8 + 2))
        act, n_act = rnd(M, ff), rnd(M, n_ff)
        add(phase, "dense gate/up + gelu", "dense up + squared relu",
            lambda: ops.linear_glu(gate_up, x, M, act, "gelu_tanh_glu"), 2.0 * (2 * ff * H + M * H + M * ff), 4.0 * M * ff * H)
        add(phase, "dense up + squared relu", None, lambda: ops.linear_act(n_up, x, M, n_act, "relu2"), *mm(n_ff, H))
        add(phase, "dense down (gated)", "dense down", lambda: ops.linear_partial(down, act, M, pv(H)), *mm(H, ff))
        add(phase, "dense down", None, lambda: ops.linear_partial(n_down, n_act, M, pv(H)), *mm(H, n_ff))
        for L, e, sfx in ((ours, m, " (grouped)"), (theirs, n_m, "")):
            like = (lambda n: n) if sfx else (lambda n: None)
            ws = ops.moe_workspace([e], H, M, bf)
            per = e.top + (e.shared_ff > 0)
            y32 = M <= ws.F32_ROWS
            y = ws.y[: M * per * H * (4 if y32 else 2)].view(f32 if y32 else bf).view(M, per, H)
            touched, act_w = min(e.experts, M * e.top), e.top * e.ff + e.shared_ff
            sum_bytes = M * H * (per * (4.0 if y32 else 2.0) + 8 + 2)
            if sfx:
                add(phase, "experts' sum + scale + norm", "experts' sum + norm",
                    lambda y=y: ops.add_norm(res, planes, 0, y, w1, x, M, 1e-6, scale=s1, offset=1.0), sum_bytes)
            else:
                add(phase, "experts' sum + norm", None, lambda y=y: ops.post_norm(res, planes, 0, y, w1, None, x, M, 1e-6),
                    sum_bytes)
            ops.moe(L, x, M, ws)                           # tables for the single kernels below
            tile = ops.n.moe_tile_rows(M, e.experts, e.top)
            add(phase, "router logits" + sfx, like("router logits"),
                lambda L=L, e=e, ws=ws: ops.linear_partial(L.router, x, M, ws.router_views[e.router_rows]),
                *mm(e.router_rows, H))
            add(phase, "routing, sorted rows" + sfx, like("routing, sorted rows"),
                lambda e=e, ws=ws, tile=tile, per=per: ops.n.moe_route(ws.router, 1, M, e, tile, x, H, per, ws),
                4.0 * M * e.top * H)
            # the last routing call left one plane's choice: sort the rows again as the feed-forward does
            ops.moe(L, x, M, ws)
            add(phase, "experts gate/up" + sfx, like("experts gate/up"), ops.moe_product_call(L, x, M, ws, 3),
                2.0 * (2 * touched * e.ff * H + 2 * e.shared_ff * H + M * act_w) + 2.0 * M * per * H, 4.0 * M * act_w * H)
            add(phase, "experts down" + sfx, like("experts down"), ops.moe_product_call(L, x, M, ws, 2 if y32 else 1),
                2.0 * (touched * e.ff * H + e.shared_ff * H + M * act_w) + (4.0 if y32 else 2.0) * M * per * H,
                2.0 * M * act_w * H)
            del ws, y
        del planes, inp, out
        torch.cuda.empty_cache()
    logits = zeros(seqs, c.vocab_size)
    add("decode", "logit scale", "norm + residual", lambda: ops.logits_finish(logits, seqs, 0.5, 0.0),
        8.0 * seqs * c.vocab_size)
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
        out[shape] = {"movinex": base.run_engine(base._file(shape, synth.shape_config(shape)), steps, warmup),
                      "nimelorn": base.run_engine(base._file(NEIGHBOURS[shape], synth.shape_config(NEIGHBOURS[shape])), steps,
                                                  warmup)}
    if kernels_file:
        with open(kernels_file, "w") as f:
            for shape in shapes:
                f.write(f"## {shape}\n\n{base.markdown(kernel_table(shape), 'Nimelorn')}\n\n")
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
