"""Throughput and per-kernel roofline fractions of the design of mixers side by side (Vobisun) beside the closest model of the
framework at equal size, a Movinex one:  ``python bench.py --workload vobisun``.

Method and table as in ``design_bench``.  The neighbour has the same width, vocabulary, heads, window, number of layer runs and
dense feed-forward, and state spaces whose state is as large as the memories'; its other layers' feed-forwards are experts,
whose kernels have no counterpart here and are not in the table.
"""
from __future__ import annotations

import types
from typing import List, Optional

import torch

from ..format import synth
from ..format.config import DenseSpec, HeadsSpec, ModelConfig, StateSpaceSpec
from . import design_bench as base

NEIGHBOURS = {"vobisun-2k": "movinex-2k", "vobisun-4k": "movinex-4k"}
SHAPES = tuple(NEIGHBOURS)


def _first(c: ModelConfig, kind, which=lambda s: True):
    return next(s for i in range(c.num_layers) for s in (c.mixer_spec(i), c.ff_spec(i)) if isinstance(s, kind) and which(s))


def kernel_table(shape: str, iters: int = 20, seqs: int = 64, ctx: int = 4096, chunk: int = 2048, chunks: int = 4,
                 only=()) -> List[dict]:
    """Kernels of a layer in a decode step of ``seqs`` sequences of ``ctx`` tokens and in a prefill pass of ``chunks``
    prompts; the neighbour's like kernel is named in ``like``."""
    from ..models.hybrid import HybridModel, PagedHeads
    from ..ops.backend import CudaOps
    ops = CudaOps("cuda")
    c, nb = synth.shape_config(shape), synth.shape_config(NEIGHBOURS[shape])
    H, bf, f32 = c.hidden_size, torch.bfloat16, torch.float32
    twin, ff, taps = c.mixer_spec(0), c.ff_spec(0).ff, c.input_conv
    a, g = twin.left, twin.right
    win, sp = _first(nb, HeadsSpec, lambda s: s.window > 0), _first(nb, StateSpaceSpec)
    n_ff = _first(nb, DenseSpec).ff
    T = base._Table(iters)

    def add(phase, name, like, fn, nbytes, flops=0.0):
        if not only or any(o in name for o in only):
            T.add(phase, name, like, fn, nbytes, flops)
    rnd = lambda *sh, dt=bf: (torch.randn(*sh, device="cuda") * 0.05).to(dt)
    lin = lambda n, k: ops.dense_linear(rnd(n, k))
    ii = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    zeros = lambda *s: torch.zeros(*s, device="cuda")
    L = types.SimpleNamespace(
        w_in=lin(twin.in_width, H), q_norm=rnd(a.heads * a.dim), k_norm=rnd(a.kv_heads * a.dim), bias=rnd(a.gate_col),
        temp=1 + rnd(a.heads, dt=f32), sink=rnd(a.heads, dt=f32), freqs=ops.rotation(a.rot_dims, a.rot_base, a.rot_factor),
        decay_w=rnd(g.heads * g.dim, g.rank, dt=f32), decay_b=3 + rnd(g.heads * g.dim, dt=f32), head_norm=rnd(g.vdim))
    L_win = types.SimpleNamespace(q_norm=None, k_norm=None, bias=None, freqs=ops.rotation(win.rot_dims, win.rot_base))
    L_sp = types.SimpleNamespace(conv_w=rnd(sp.conv, sp.conv_width, dt=f32), conv_b=zeros(sp.conv_width),
                                 dt_bias=zeros(sp.heads), neg_a=-torch.ones(sp.heads, device="cuda"), D=zeros(sp.heads),
                                 w_in=lin(sp.in_width, H), out_norm=rnd(sp.inner))
    w_win, o_sp = lin(win.in_width, H), lin(H, sp.inner)
    out_w = twin.out_width + ff
    o, gate_up = lin(H, out_w), ops.glu_linear(rnd(ff, H), rnd(ff, H), bf)
    n_gate_up, conv_w = ops.glu_linear(rnd(n_ff, H), rnd(n_ff, H), bf), rnd(taps, H, dt=f32)
    bs, per_seq = 64, (ctx + 63) // 64
    means = (ctx // a.pool + bs - 1) // bs
    blocks = seqs * (per_seq + means)
    pool = rnd(blocks, 1, 1, bs, max(a.row, win.row))
    kv, kv_win = PagedHeads(pool, a, per_seq), PagedHeads(pool, win)
    tables = torch.arange(blocks, dtype=torch.int32, device="cuda").view(seqs, per_seq + means)
    state = zeros(2 * seqs, max(sp.state_floats, g.state_floats + (taps - 1) * H))
    table = rnd(c.vocab_size, H)
    for phase, M in (("decode", seqs), ("prefill", chunk * chunks)):
        dec = phase == "decode"
        S, n_buf = (seqs, 8) if dec else (chunks, 1)
        x, x2, both = rnd(M, H), rnd(M, H), rnd(M, 2 * H)
        planes = zeros(n_buf * M * max(twin.in_width, sp.in_width))
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
        n_pl = 2 if dec else 0
        pl = 4 if dec else 1
        w1, s1 = rnd(H), rnd(H)
        inp, inp_win, inp_sp = rnd(M, twin.in_width), rnd(M, win.in_width), rnd(M, sp.in_width)
        side, side_sp = zeros(M * (g.in_width - g.rank_col)), zeros(M * (sp.in_width - sp.dt_col))

        add(phase, "embedding", "embedding (two places)", lambda: ops.embedding(table, ids, res, M, 45.0), M * H * 6.0)
        add(phase, "embedding (two places)", None, lambda: ops.embedding(table, ids, res, M, copy=both[:, H:]), M * H * 8.0)
        norm_bytes = M * H * (4.0 * pl + 8 + 2)
        add(phase, "residual + norm" + (" + convolution" if dec else ""), "scale + residual + norm",
            lambda: ops.add_norm_conv(res, planes, pl, w1, x, conv_w, x2, state, g.state_floats, rows, row_seq, None, M, S, 1e-6)
            if dec else ops.add_norm(res, planes, pl, None, w1, x, M, 1e-6),
            norm_bytes + (M * H * (2.0 + 8.0 * (taps - 1)) if dec else 0.0))
        add(phase, "scale + residual + norm", None,
            lambda: ops.add_norm(res, planes, pl, None, w1, x, M, 1e-6, scale=s1, offset=1.0), norm_bytes)
        if not dec:
            cv = ops.n.row_conv_args(conv_w, state, g.state_floats, rows)
            add(phase, "convolution of the inputs", "convolution, step sizes",
                lambda: ops.n.row_conv(x, x2, cv, row_seq, cu, M, H), 4.0 * M * H + 8.0 * S * (taps - 1) * H)

        def project(lw, dst, side):
            if dec:
                ops.linear_partial(lw, x, M, pv(lw.N))
            else:
                ops.linear(lw, x, M, dst, side=side)
        add(phase, "input projection (both mixers)", "input projection (state space)",
            lambda: project(L.w_in, inp, (g.rank_col, side)), *mm(twin.in_width, H))
        add(phase, "input projection (state space)", None, lambda: project(L_sp.w_in, inp_sp, (sp.dt_col, side_sp)),
            *mm(sp.in_width, H))
        add(phase, "input projection (windowed attention)", None, lambda: project(w_win, inp_win, None), *mm(win.in_width, H))

        moved = lambda s: M * (s.in_width * (4.0 * n_pl + 2) if dec else 2.0 * (s.gate_col + (s.heads + s.kv_heads) * s.dim
                                                                               + s.kv_heads * s.vdim))
        add(phase, "norm over all heads, rotation, cache write" + (", means" if dec else ""), "norms, rotation, cache write",
            lambda: ops.heads_prep(inp, pv(twin.in_width), n_pl, kv, slots, L, a, 1e-6, M, positions, tables if dec else None),
            moved(a) + (2.0 * M * (a.pool + 1) * a.row if dec else 0.0))
        add(phase, "norms, rotation, cache write", None,
            lambda: ops.heads_prep(inp_win, pv(win.in_width), n_pl, kv_win, slots, L_win, win, 1e-6, M, positions), moved(win))
        ctab = tables if dec else torch.cat([tables[:chunks, : chunk // bs], tables[:chunks, per_seq:]], 1).contiguous()
        kv_c = kv if dec else PagedHeads(pool, a, chunk // bs)
        if not dec:
            add(phase, "means of blocks", "norms, rotation, cache write",
                lambda: ops.heads_pool(kv_c, ctab, row_seq, positions, a, M), 2.0 * a.row * (M + M // a.pool))
            decays = zeros(M * g.heads * g.dim)
            add(phase, "logarithms of the decays", "convolution, step sizes",
                lambda: ops.gated_linear_prep(inp, None, 0, side, decays, L, g, M),
                4.0 * M * (g.heads * g.dim + g.rank) + 4.0 * g.heads * g.dim * g.rank, 2.0 * M * g.heads * g.dim * g.rank)
        xbc, dt = rnd(M, sp.conv_width), zeros(M, sp.heads)
        add(phase, "convolution, step sizes", None,
            lambda: ops.state_space_prep(inp_sp, pv(sp.in_width), n_pl, side_sp, xbc, dt, state, 0, rows, row_seq, cu, L_sp, sp,
                                         M, S),
            M * (sp.in_width * 4.0 * n_pl + 2.0 * (sp.x_col + sp.conv_width) if dec else 4.0 * sp.conv_width + 8.0 * sp.heads)
            + 8.0 * S * (sp.conv - 1) * sp.conv_width)

        out, out_win, out_sp = rnd(M, out_w), rnd(M, win.heads * win.vdim), rnd(M, sp.inner)
        right = out[:, twin.right_at:]
        seen = lambda s, p: (min(p + 1, s.window + s.keep_first) + (s.blocks_seen(p) if s.pool else 0))
        g_io = 2.0 * M * (2 * g.heads * g.dim + 3 * g.heads * g.vdim)
        g_flops = 4.0 * M * g.heads * g.dim * g.vdim
        sp_io = 2.0 * M * (sp.conv_width + 2 * sp.inner) + 4.0 * M * sp.heads
        sp_flops = 4.0 * M * sp.heads * sp.state * sp.vdim
        if dec:
            for name, s, k, i, o_, sink, like in (
                    ("attention rows over tokens and means", a, kv, inp, out, L.sink, "windowed attention rows"),
                    ("windowed attention rows", win, kv_win, inp_win, out_win, None, None)):
                splits = HybridModel.attention_splits(types.SimpleNamespace(heads_specs=[s]), M, ctx, 16, ops.sm_count)
                scratch = zeros(M * splits * s.heads * (s.vdim + 2))
                n = seen(s, ctx - 1)
                add(phase, name, like,
                    lambda s=s, k=k, i=i, o_=o_, sc=scratch, sp_=splits, sink=sink: ops.heads_attn(
                        i, k, tables, None, positions, o_, M, s, sc, sp_, sink),
                    2.0 * M * (n * s.row + s.heads * (s.dim + s.vdim) + s.gate_width),
                    2.0 * M * n * s.heads * (s.dim + s.vdim))
            add(phase, "gated linear step", "state space step",
                lambda: ops.gated_linear_tokens(inp, pv(twin.in_width), n_pl, None, state, 0, rows, None, L, right, S, M, g,
                                                1e-6),
                2 * g_flops + 4.0 * n_pl * M * (g.in_width - g.col) + 2.0 * M * g.heads * g.vdim, g_flops)
            add(phase, "state space step", None,
                lambda: ops.state_space_tokens(inp_sp, xbc, dt, state, 0, rows, None, L_sp, out_sp, S, M, sp),
                2 * sp_flops + sp_io, sp_flops)
        else:
            pairs = lambda s: chunks * sum(seen(s, p) for p in range(chunk))
            for name, s, k, i, o_, sink, like, t in (
                    ("attention tiles over tokens and means", a, kv_c, inp, out, L.sink, "windowed attention tiles", ctab),
                    ("windowed attention tiles", win, kv_win, inp_win, out_win, None, None, ctab)):
                add(phase, name, like,
                    lambda s=s, k=k, i=i, o_=o_, sink=sink, t=t: ops.heads_attn_chunks(i, k, t, cu, p0, positions, 0, chunks,
                                                                                       chunk, o_, s, sink),
                    2.0 * M * (s.in_width + s.heads * s.vdim), 2.0 * pairs(s) * s.heads * (s.dim + s.vdim))
            ws = ops.gated_linear_workspace([g], M)
            add(phase, "gated linear in chunks", "state space in chunks + norm",
                lambda: ops.gated_linear_chunks(inp, decays, state, 0, rows, cu, L, right, 0, chunks, 0, M, g, 1e-6, ws),
                g_io + 4.0 * M * g.heads * g.dim + 8.0 * S * g.state_floats, g_flops)

            def chunks_and_norm():
                ops.state_space_chunks(inp_sp, xbc, dt, state, 0, rows, cu, L_sp, out_sp, 0, chunks, M, sp)
                ops.group_norm(out_sp, L_sp.out_norm, sp.norm_groups, M, 1e-6)
            add(phase, "state space in chunks + norm", None, chunks_and_norm,
                sp_io + 8.0 * S * sp.heads * sp.state * sp.vdim, sp_flops)
        add(phase, "gate/up + silu", "dense gate/up + gelu",
            lambda: ops.linear_glu(gate_up, x, M, out[:, twin.out_width:], "silu_glu"),
            2.0 * (2 * ff * H + M * H + M * ff), 4.0 * M * ff * H)
        act = rnd(M, n_ff)
        add(phase, "dense gate/up + gelu", None, lambda: ops.linear_glu(n_gate_up, x, M, act, "gelu_tanh_glu"),
            2.0 * (2 * n_ff * H + M * H + M * n_ff), 4.0 * M * n_ff * H)
        add(phase, "one output product", "output projection (state space)", lambda: ops.linear_partial(o, out, M, pv(H)),
            *mm(H, out_w))
        add(phase, "output projection (state space)", None, lambda: ops.linear_partial(o_sp, out_sp, M, pv(H)), *mm(H, sp.inner))
        del planes, inp, inp_win, inp_sp, out
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
        out[shape] = {"vobisun": base.run_engine(base._file(shape, synth.shape_config(shape)), steps, warmup),
                      "movinex": base.run_engine(base._file(NEIGHBOURS[shape], synth.shape_config(NEIGHBOURS[shape])), steps,
                                                 warmup)}
    if kernels_file:
        with open(kernels_file, "w") as f:
            for shape in shapes:
                f.write(f"## {shape}\n\n{base.markdown(kernel_table(shape), 'Movinex')}\n\n")
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
