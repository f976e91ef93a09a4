"""Vobisun on the GPU: every kernel against the plain float64 statements of the same mechanism, whole models against the plain
oracle in float32 and bfloat16, generation through the engine."""
import os
import sys
import types

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import vobisun_oracle as oracle                                      # noqa: E402
from helpers.latent_oracle import write_model                                     # noqa: E402
from helpers.ruralorn_cases import (LENGTHS, MAX_TOKENS, SCHEDULES, assert_close, assert_near, replay,  # noqa: E402
                                    schedule)
from helpers.vobisun_cases import CASES, SPECS, Model, PooledAttention, loud_places, make_loud, spec  # noqa: E402

from zse_b200.format.config import GatedLinearSpec                                # noqa: E402
from zse_b200.models.hybrid import PagedHeads                                     # noqa: E402

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64


@pytest.fixture(scope="module")
def ops():
    from zse_b200.ops.backend import CudaOps
    o = CudaOps("cuda")
    yield o
    o.check()


def rel(a, b):
    b = b.to(a.device)
    return ((a.to(F64) - b).abs().max() / b.abs().max()).item()


def tol(dt):
    return 1.5e-2 if dt == BF else 2e-5


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


@pytest.fixture
def form(ops, request):
    """The tensor-core form of attention in tiles of queries that the test runs on."""
    ops.heads_form, old = request.param, ops.heads_form
    yield request.param
    ops.heads_form = old


# ---- attention over tokens and means --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", [n for n in SPECS if SPECS[n].pool])
@pytest.mark.parametrize("bs", [64, 16])
def test_means_of_blocks(ops, name, dt, bs):
    A = PooledAttention(ops, SPECS[name], dt, "cuda", bs=bs)
    for s in range(3):
        for x, y in zip(A.means(s), (A.k[s], A.v[s])):
            assert rel(x, oracle.block_means(y.to(F64), A.spec.pool)) < (5e-3 if dt == BF else 1e-6)
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(SPECS))
@pytest.mark.parametrize("bs", [64, 16])
def test_rows_against_tokens_and_means(ops, name, dt, bs):
    A = PooledAttention(ops, SPECS[name], dt, "cuda", bs=bs)
    s = A.spec
    seqs = [0, 1, 2, 2, 1, 0, 0, 1]
    pos = [0, 1, s.window - 1, s.window, s.window + max(1, s.pool) - 1, s.window + max(1, s.pool) - 2, 699, 300]
    want = torch.stack([A.plain(t, q, max(0, p)) for t, (q, p) in enumerate(zip(seqs, pos))])
    for splits in (1, 2, 8):
        assert rel(A.rows(seqs, [max(0, p) for p in pos], splits), want) < tol(dt), splits
    ops.check()


@pytest.mark.parametrize("name", [n for n in SPECS if n != "general"])
@pytest.mark.parametrize("bs", [64, 32, 48])
@pytest.mark.parametrize("form", [1, 2], indirect=True)
def test_tiles_of_queries_against_tokens_and_means(ops, name, bs, form):
    A = PooledAttention(ops, SPECS[name], BF, "cuda", bs=bs, seqs=5)
    assert ops.heads_expands(A.spec, BF)
    spans = [(3, 5), (0, 150), (300, 17), (470, 130), (63, 64)]    # the first sequence is not part of the call
    out, cu = A.chunks(spans, first=1)
    assert (out[: cu[1]] == 0).all()
    for s in range(1, len(spans)):
        for i in sorted({0, 1, spans[s][1] // 2, 63 % spans[s][1], 64 % spans[s][1], 128 % spans[s][1], spans[s][1] - 1}):
            assert rel(out[cu[s] + i], A.plain(cu[s] + i, s, spans[s][0] + i)) < tol(BF), (s, i)
    ops.check()


@pytest.mark.parametrize("name", ["window", "short-window", "single-tokens"])
def test_blocks_that_left_are_not_read(ops, name):
    A = PooledAttention(ops, SPECS[name], BF, "cuda")
    s, pos = A.spec, 600
    want = torch.stack([A.plain(t, 0, pos - 20 + t) for t in range(21)])
    A.tables[0, : s.first_seen(pos - 20) // 64] = -1
    assert rel(A.chunks([(pos - 20, 21)])[0], want) < tol(BF)
    assert rel(A.rows([0] * 21, list(range(pos - 20, pos + 1)), 4), want) < tol(BF)
    ops.check()


@pytest.mark.parametrize("dt,what,form", [(BF, "rows", 1), (F32, "rows", 1), (BF, "tiles", 1), (BF, "tiles", 2)],
                         indirect=["form"])
@pytest.mark.parametrize("name", ["window", "short-window", "single-tokens", "blocks-of-the-cache"])
def test_one_loud_key_inside_and_outside(ops, name, dt, what, form):
    """A key that takes nearly all the weight, alone or in the mean of its block, at every border of what is seen."""
    s = SPECS[name]
    for pos in (s.window - 1, s.window + s.pool - 1, 447, 640):
        for key in loud_places(s, pos):
            if key >= 700:
                continue
            A = PooledAttention(ops, s, dt, "cuda", seed=pos, seqs=1)
            t = 20                                       # a query in the middle of the portion
            make_loud(A, key, s.heads - 1, t)
            want = A.plain(t, 0, pos)
            if what == "rows":
                A.inp[0] = A.inp[t]
                got = A.rows([0], [pos], 2)[0]
            elif pos < t:
                continue
            else:
                got = A.chunks([(pos - t, 40)])[0][t]
            assert rel(got, want) < (3e-2 if dt == BF else 2e-5), (pos, key)


@pytest.mark.parametrize("sink", [-60.0, 0.0, 25.0])
@pytest.mark.parametrize("form", [1, 2], indirect=True)
def test_sinks_far_below_and_above_the_scores(ops, sink, form):
    A = PooledAttention(ops, SPECS["window"], BF, "cuda")
    A.sink[:] = sink
    want = A.plain(5, 0, 305)
    assert rel(A.chunks([(300, 40)])[0][5], want) < tol(BF)
    for splits in (1, 4):
        assert rel(A.rows([0] * 6, [305] * 6, splits)[5], want) < tol(BF)


PREP = {
    "rotated": spec(6, 2, 64, 64, 50, 4, rot_dims=32, rot_base=5e4, rot_factor=4.0),
    "all-rotated": spec(3, 3, 128, 72, 50, 9, rot_dims=128),
    "pair": spec(5, 1, 24, 24, 50, 2, rot_dims=2),
    "not-by-four": spec(4, 2, 48, 16, 50, 7, rot_dims=38, rot_base=300.0, rot_factor=0.5),
    "still": spec(4, 2, 48, 40, 50, 0, gated=False),
    "many": spec(64, 8, 128, 128, 50, 4, rot_dims=64),
    "long-heads": spec(2, 1, 320, 320, 50, 3, rot_dims=300),
    "general": spec(3, 3, 10, 14, 50, 5, rot_dims=6),
    "odd": spec(3, 1, 7, 5, 50, 2, rot_dims=4),
}


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(PREP))
@pytest.mark.parametrize("planes", [0, 1, 4])
@pytest.mark.parametrize("M", [60, 700])
def test_one_norm_over_all_heads(ops, name, dt, planes, M):
    s, eps = PREP[name], 1e-5
    H, G, d, vd = s.heads, s.kv_heads, s.dim, s.vdim
    g = torch.Generator(device="cuda").manual_seed(3)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", generator=g)
    wide = s.in_width + 24                                   # other columns follow
    inp, pl = rnd(M, wide).to(dt), rnd(max(1, planes), M, wide)
    rest = inp[:, s.in_width:].clone()
    full = (pl.to(F64).sum(0) if planes else inp.to(F64)).cpu()
    L = types.SimpleNamespace(q_norm=rnd(H * d).to(dt), k_norm=rnd(G * d).to(dt), bias=rnd(s.gate_col).to(dt), temp=rnd(H),
                              freqs=ops.rotation(s.rot_dims, s.rot_base, s.rot_factor))
    full[:, : s.gate_col] += L.bias.cpu().to(F64)
    pos = ([0, 1, 2, 63, 64, 100, 5000, 131071] + list(range(300, 992)))[:M]
    pool = torch.zeros(20, 1, 1, 64, s.row + 8, device="cuda", dtype=dt)
    kv = PagedHeads(pool, s)
    slots = torch.randperm(20 * 64, device="cuda", generator=g)[:M]
    slots[5] = -1
    ops.heads_prep(inp, pl, planes, kv, slots, L, s, eps, M, i32(pos))

    def finish(x, n, w):
        x = oracle.norm(x, w.cpu().to(F64), eps).view(M, n, d).clone()
        for i in range(s.rot_dims // 2):
            a = torch.tensor([p * s.rot_base ** (-2 * i / s.rot_dims) / s.rot_factor for p in pos], dtype=F64)[:, None]
            u, v = x[..., 2 * i].clone(), x[..., 2 * i + 1].clone()
            x[..., 2 * i], x[..., 2 * i + 1] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
        return x
    q = finish(full[:, : H * d], H, L.q_norm) * L.temp.cpu().to(F64)[:, None]
    assert rel(inp[:, : H * d], q.reshape(M, -1)) < tol(dt)
    if s.gated and planes:
        assert rel(inp[:, s.gate_col: s.gate_col + H], full[:, s.gate_col: s.gate_col + H]) < tol(dt)
    assert torch.equal(inp[:, s.in_width:], rest)
    ok = (slots >= 0).cpu()
    blk, at = (slots[slots >= 0] // 64), (slots[slots >= 0] % 64)
    k, v = finish(full[:, s.k_col: s.k_col + G * d], G, L.k_norm), full[:, s.v_col: s.v_col + G * vd].view(M, G, vd)
    assert rel(kv.k[blk, :, at, :d], k[ok]) < tol(dt)
    assert rel(kv.v[blk, :, at, :vd], v[ok]) < tol(dt)
    assert (kv.k[..., d:] == 0).all() and (kv.v[..., vd:] == 0).all()
    untouched = torch.ones(20 * 64, dtype=torch.bool, device="cuda")
    untouched[slots[slots >= 0]] = False
    assert (kv.k.transpose(1, 2).reshape(20 * 64, -1)[untouched] == 0).all()
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", ["rotated", "all-rotated", "not-by-four", "general", "odd"])
def test_decoding_rows_leave_means(ops, name, dt):
    """Rows of several sequences: those that complete a block leave its mean, over earlier tokens and their own."""
    s = PREP[name]
    A = PooledAttention(ops, s, dt, "cuda", tokens=300, seqs=4)
    P, M, eps = s.pool, 4, 1e-5
    pos = [P - 1, 20 * P - 1, 20 * P, 10 * P + P - 1]
    before = [tuple(x.clone() for x in A.means(q)) for q in range(4)]
    g = torch.Generator(device="cuda").manual_seed(3)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", generator=g)
    L = types.SimpleNamespace(q_norm=rnd(s.heads * s.dim).to(dt), k_norm=rnd(s.kv_heads * s.dim).to(dt),
                              bias=rnd(s.gate_col).to(dt), temp=rnd(s.heads),
                              freqs=ops.rotation(s.rot_dims, s.rot_base, s.rot_factor))
    pl = rnd(2, M, s.in_width)
    slots = torch.tensor([int(A.tables[q, p // 64]) * 64 + p % 64 for q, p in enumerate(pos)], device="cuda")
    ops.heads_prep(A.inp, pl, 2, A.kv, slots, L, s, eps, M, i32(pos), A.tables)
    for q, p in enumerate(pos):
        got = A.means(q)
        blocks = torch.arange(300 // P, device="cuda")
        at = torch.arange(p // P * P, p // P * P + P, device="cuda")
        for x, old, cache, n in zip(got, before[q], (A.kv.k, A.kv.v), (s.dim, s.vdim)):
            same = blocks != p // P if (p + 1) % P == 0 else blocks >= 0
            assert torch.equal(x[same], old[same])
            if (p + 1) % P == 0:
                rows = cache[A.tables[q, at // 64].long(), :, at % 64, :n].to(F64)
                assert rel(x[p // P], rows.mean(0)) < (5e-3 if dt == BF else 1e-6)
    ops.check()


# ---- gated linear attention -------------------------------------------------------------------------------------------------
MEMORIES = {
    "small": GatedLinearSpec(4, 16, 24, 2.0, 5, 16),
    "usual": GatedLinearSpec(3, 128, 128, 16.0, 16, 8, 0.5),
    "big": GatedLinearSpec(2, 256, 72, 16.0, 16, 0),
    "half-steps": GatedLinearSpec(5, 72, 40, 1.0, 8, 24, -2.0),
    "many-columns": GatedLinearSpec(2, 40, 264, 8.0, 64, 0),
    "between": GatedLinearSpec(2, 200, 64, 4.0, 3, 0),
    "general": GatedLinearSpec(3, 10, 7, 3.0, 6, 8),
    "one": GatedLinearSpec(1, 8, 8, 1.0, 1, 0),
}


class Memory:
    def __init__(self, s, dt, rows=420, slots=7, seed=0, slow=True):
        g = torch.Generator(device="cuda").manual_seed(seed)
        rnd = lambda *sh: torch.randn(*sh, device="cuda", generator=g)
        self.spec, self.dt, self.at, self.eps = s, dt, 12, 1e-5
        self.inp = rnd(rows, s.in_width).to(dt)
        n = s.heads * s.dim
        self.decays = torch.nn.functional.logsigmoid(rnd(rows, n) + (4.0 if slow else -1.0)).contiguous()
        self.L = types.SimpleNamespace(decay_w=rnd(n, s.rank), decay_b=rnd(n), head_norm=rnd(s.vdim).to(dt),
                                       w_in=types.SimpleNamespace(kind="bf16" if dt == BF else "f32", K=64))
        self.states = torch.zeros(2 * slots, self.at + s.state_floats + 4, device="cuda")
        self.size = n * s.vdim
        self.states[:, self.at: self.at + self.size] = rnd(2 * slots, self.size)

    def memory(self, row):
        s = self.spec
        return self.states[row, self.at: self.at + self.size].to(F64).view(s.heads, s.dim, s.vdim).clone()

    def plain(self, a, e, read):
        """Rows [a, e) from the memory in row ``read`` (-1: none): (finished read-outs, memory) in float64."""
        s = self.spec
        H, d, v = s.heads, s.dim, s.vdim
        S = self.memory(read) if read >= 0 else torch.zeros(H, d, v, dtype=F64, device="cuda")
        x = self.inp[a:e].to(F64)
        q, k = x[:, s.col: s.col + H * d].view(-1, H, d) * d ** -0.5, x[:, s.k_col: s.k_col + H * d].view(-1, H, d)
        val, alpha = x[:, s.v_col: s.v_col + H * v].view(-1, H, v), torch.exp(self.decays[a:e].to(F64)).view(-1, H, d)
        out = []
        for t in range(e - a):
            S = alpha[t][:, :, None] * S + k[t][:, :, None] * val[t][:, None, :]
            out.append((S * q[t][:, :, None]).sum(1))
        y = oracle.norm(torch.stack(out), self.L.head_norm.to(F64), self.eps).view(e - a, -1)
        return s.out_scale * y * oracle.silu(x[:, s.gate_col: s.gate_col + H * v]), S

    def run(self, ops, cu, rows, chunkwise, first=0):
        s, M, S = self.spec, cu[-1] if cu is not None else rows.shape[1], rows.shape[1]
        wide = torch.zeros(M, s.out_width + 24, dtype=self.dt, device="cuda")
        out, cu_d = wide[:, 16:], i32(cu) if cu is not None else None
        if chunkwise:
            ops.gated_linear_chunks(self.inp, self.decays, self.states, self.at, rows, cu_d, self.L, out, first, S, cu[first],
                                    M, s, self.eps, ops.gated_linear_workspace([s], M))
        else:
            ops.gated_linear_tokens(self.inp, None, 0, self.decays, self.states, self.at, rows, cu_d, self.L, out, S, M, s,
                                    self.eps)
        assert (wide[:, :16] == 0).all() and (wide[:, 16 + s.out_width:] == 0).all()
        return out[:, : s.out_width]


def check_memory(ops, name, dt, cu, rows, chunkwise, first=0, slow=True, change=None):
    m, limit = Memory(MEMORIES[name], dt, slow=slow), 1e-2 if dt == BF else 2e-5
    if change is not None:
        change(m)
    want = [m.plain(cu[i], cu[i + 1], rows[0][i]) for i in range(len(rows[0]))]
    expect = m.states.clone()
    out = m.run(ops, cu, i32(rows), chunkwise, first)
    for i in range(first, len(rows[0])):
        y, S = want[i]
        a, e, w = cu[i], cu[i + 1], rows[1][i]
        err = (out[a:e].to(F64) - y).pow(2).mean(1).sqrt() / y.pow(2).mean(1).sqrt()
        assert err.max() < limit, (i, err.max().item(), int(err.argmax()))
        if w >= 0:
            assert rel(m.memory(w), S) < (1e-4 if chunkwise else 1e-5)       # 32 bits, also through the tensor cores
            expect[w, m.at: m.at + m.size] = m.states[w, m.at: m.at + m.size]
    assert torch.equal(m.states, expect)                 # other rows, other layers' parts
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(MEMORIES))
def test_memory_token_by_token(ops, name, dt):
    check_memory(ops, name, dt, [0, 1, 2, 3, 4], [[4, -1, 7, -1], [5, 2, 6, -1]], False)      # a row each
    check_memory(ops, name, dt, [0, 2, 18, 19, 150], [[4, -1, 7, 0], [5, 2, 6, 1]], False)


@pytest.mark.parametrize("slow", [True, False])
@pytest.mark.parametrize("name", [n for n in MEMORIES if n != "general"])
def test_memory_in_chunks(ops, name, slow):
    assert ops.gated_linear_expands(MEMORIES[name], BF)
    check_memory(ops, name, BF, [0, 64, 147, 160, 400], [[4, -1, 7, 0], [5, 2, 6, 1]], True, slow=slow)
    check_memory(ops, name, BF, [0, 3, 130, 195], [[4, 2, -1], [5, 3, -1]], True, first=1, slow=slow)


@pytest.mark.parametrize("name", ["usual", "half-steps", "big"])
def test_memory_in_chunks_of_extreme_decays(ops, name):
    """Channels that forget everything at every token, from some token on, beside channels that forget nothing."""
    def change(m):
        m.decays[:, ::3] = -60.0
        m.decays[50:, 1::3] = -9.0
        m.decays[:, 2::3] = 0.0
        m.decays[100, 2::3] = -200.0
    check_memory(ops, name, BF, [0, 64, 147, 160, 400], [[4, -1, 7, 0], [5, 2, 6, 1]], True, change=change)


def test_memory_decodes_without_row_offsets(ops):
    m = Memory(MEMORIES["usual"], BF, seed=4)
    rows = [[0, 2, -1, -1], [1, 3, 4, -1]]
    want = torch.cat([m.plain(i, i + 1, rows[0][i])[0] for i in range(4)])
    assert rel(m.run(ops, None, i32(rows), False), want) < 1e-2
    many = Memory(MEMORIES["usual"], BF, rows=150, slots=120, seed=5)        # enough CTAs: a head each
    rows = [[2 * i for i in range(120)], [2 * i + 1 for i in range(120)]]
    want = torch.cat([many.plain(i, i + 1, 2 * i)[0] for i in range(120)])
    assert rel(many.run(ops, None, i32(rows), False), want) < 1e-2


@pytest.mark.parametrize("chunkwise", [True, False])
def test_memory_keeps_a_token_from_long_ago(ops, chunkwise):
    """No decay to speak of: one loud token at the start is what every later token reads; one that closes, and it is gone."""
    s = GatedLinearSpec(2, 64, 128, 16.0, 4, 0)
    for closed_at in (None, 200):
        m = Memory(s, BF)
        m.decays.fill_(-1e-4)
        m.inp[:, s.k_col: s.v_col] *= 1e-2
        m.inp[3, s.k_col: s.v_col] *= 1e4
        if closed_at is not None:
            m.decays[closed_at] = -80.0
        want = m.plain(0, 400, -1)[0]
        out = m.run(ops, [0, 400], i32([[-1], [1]]), chunkwise)
        err = (out.to(F64) - want).pow(2).mean(1).sqrt() / want.pow(2).mean(1).sqrt()
        assert err.max() < 1.5e-2, (int(err.argmax()), err.max().item())


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(MEMORIES))
@pytest.mark.parametrize("planes,side", [(0, False), (0, True), (1, False), (5, False)])
def test_decays_and_columns_of_the_memory(ops, name, dt, planes, side):
    s, M = MEMORIES[name], 61
    m = Memory(s, dt)
    g = torch.Generator(device="cuda").manual_seed(1)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", generator=g)
    pl, sd, inp = 2 * rnd(max(1, planes), M, s.in_width), 3 * rnd(M, s.in_width - s.rank_col), m.inp[:M].clone()
    old = inp.clone()
    full = (pl.to(F64).sum(0) if planes else inp.to(F64)).cpu()
    decays = torch.zeros(M * s.heads * s.dim, device="cuda")
    ops.gated_linear_prep(inp, pl, planes, sd if side else None, decays, m.L, s, M)
    u = full[:, s.rank_col: s.rank_col + s.rank]
    if side and dt == BF:                                # the general kernel leaves them in the projected row
        u = sd[:, : s.rank].cpu().to(F64)
    z = u @ m.L.decay_w.cpu().to(F64).T + m.L.decay_b.cpu().to(F64)
    want = -torch.nn.functional.softplus(-z) / s.tau
    assert ((decays.view(M, -1).cpu().to(F64) - want).abs() <= 2e-6 * (1 + z.abs())).all()
    assert torch.equal(inp[:, : s.col], old[:, : s.col])
    if planes:
        assert rel(inp[:, s.col: s.rank_col], full[:, s.col: s.rank_col]) < tol(dt)
        # a decode step takes all of it from the planes
        m.inp[:M], m.decays = inp, decays.view(M, -1)
        rows = i32([[0, 2, -1, -1], [1, 3, 4, -1]])
        start = m.states.clone()
        want = m.run(ops, None, rows, False)
        want_states, m.states = m.states, start
        got = torch.zeros(4, s.out_width, dtype=dt, device="cuda")
        ops.gated_linear_tokens(old, pl[:, :4].contiguous(), planes, None, m.states, m.at, rows, None, m.L, got, 4, 4, s, m.eps)
        assert rel(got, want.to(F64)) < (3e-2 if dt == BF else 1e-4)
        assert rel(m.states, want_states.to(F64)) < (2e-2 if dt == BF else 1e-5)
    ops.check()


# ---- rows -------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H", [64, 51, 4096, 10000])
@pytest.mark.parametrize("planes", [0, 1, 4])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_norm_and_convolution_of_decoding_rows(ops, dt, H, planes, taps):
    M, eps, at = 9, 1e-5, 8
    g = torch.Generator(device="cuda").manual_seed(H)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    res, pl, w, cw = rnd(M, H), rnd(max(1, planes), M, H), rnd(H).to(dt), rnd(taps, H)
    states = rnd(20, at + (taps - 1) * H + (-(taps - 1) * H) % 4 + 4)
    read, write = [0, 2, -1, 4, -1, 6, 8, 10, -1], [1, 3, 12, 5, 13, 7, 9, 11, -1]
    out, conv = torch.zeros(M, H, device="cuda", dtype=dt), torch.zeros(M, H, device="cuda", dtype=dt)
    want = res.to(F64) + (pl.to(F64).sum(0) if planes else 0)
    expect = states.clone()
    ops.add_norm_conv(res, pl, planes, w, out, cw, conv, states, at, i32([read, write]), None, None, M, M, eps)
    assert rel(res, want) < 1e-5
    h = oracle.norm(want, w.to(F64), eps)
    assert rel(out, h) < tol(dt)
    for s in range(M):
        before = expect[read[s], at: at + (taps - 1) * H].view(-1, H).to(F64) if read[s] >= 0 else \
            torch.zeros(taps - 1, H, dtype=F64, device="cuda")
        rows = torch.cat([before, out[s: s + 1].to(F64)])
        assert rel(conv[s], out[s].to(F64) + (cw.to(F64) * rows).sum(0)) < tol(dt), s
        if write[s] >= 0:
            expect[write[s], at: at + (taps - 1) * H] = rows[1:].reshape(-1).float()
    assert torch.equal(states, expect)
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,cu", [(96, [0, 1, 3, 6, 9, 30, 61]), (51, [0, 1, 3, 6, 9, 30, 61]), (1032, [0, 500, 509, 510, 1200]),
                                  (64, [0, 3000, 3001, 3004, 4500])])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_convolution_of_portions(ops, dt, H, cu, taps):
    """Portions of one to many tokens, the rows that are carried on, several sequences in a thread's rows."""
    M, S, eps, at = cu[-1], len(cu) - 1, 1e-5, 4
    g = torch.Generator(device="cuda").manual_seed(H)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    res, w, cw = rnd(M, H), rnd(H).to(dt), rnd(taps, H)
    states = rnd(12, at + (taps - 1) * H + (-(taps - 1) * H) % 4 + 4)
    rows = [[0, -1, 2, 4, -1, 6][:S], [1, 8, 3, 5, -1, 7][:S]]
    out, conv = torch.zeros(M, H, device="cuda", dtype=dt), torch.zeros(M, H, device="cuda", dtype=dt)
    expect = states.clone()
    seq = [i for i in range(S) for _ in range(cu[i + 1] - cu[i])]
    ops.add_norm_conv(res, rnd(1, M, H), 0, w, out, cw, conv, states, at, i32(rows), i32(seq), i32(cu), M, S, eps)
    for i in range(S):
        a, e = cu[i], cu[i + 1]
        before = expect[rows[0][i], at: at + (taps - 1) * H].view(-1, H).to(F64) if rows[0][i] >= 0 else \
            torch.zeros(taps - 1, H, dtype=F64, device="cuda")
        x = torch.cat([before, out[a:e].to(F64)])
        y = out[a:e].to(F64) + sum(cw[j].to(F64) * x[j: j + e - a] for j in range(taps))
        assert rel(conv[a:e], y) < tol(dt), i
        if rows[1][i] >= 0:
            expect[rows[1][i], at: at + (taps - 1) * H] = x[len(x) - (taps - 1):].reshape(-1).float()
    assert torch.equal(states, expect)
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("M,ff,K", [(5, 40, 24), (300, 136, 96), (13, 19, 51)])
def test_gated_product_into_a_part_of_a_row(ops, dt, M, ff, K):
    g = torch.Generator(device="cuda").manual_seed(ff)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    x, a, u = (2 * rnd(M, K)).to(dt), (rnd(ff, K) * K ** -0.5).to(dt), (rnd(ff, K) * K ** -0.5).to(dt)
    wide, tmp = torch.zeros(M, 24 + ff + 5, device="cuda", dtype=dt), torch.zeros(M * 2 * ff, device="cuda", dtype=dt)
    ops.linear_glu(ops.glu_linear(a, u, dt), x, M, wide[:, 24: 24 + ff], "silu_glu", tmp)
    want = oracle.silu(x.to(F64) @ a.to(F64).T) * (x.to(F64) @ u.to(F64).T)
    assert rel(wide[:, 24: 24 + ff], want) < tol(dt)
    assert (wide[:, :24] == 0).all() and (wide[:, 24 + ff:] == 0).all()
    ops.check()


# ---- whole models -----------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp("vobisun") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("vobisun-small"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_schedules_match_the_oracle(model, dtype):
    from zse_b200.trace import TraceRunner
    r = TraceRunner(model.path, dtype, MAX_TOKENS)
    try:
        for name in SCHEDULES + ["token-by-token"]:
            got = replay(r, model, schedule(name))
            if dtype == "float32":
                assert_close(model, got, 5e-4)
            else:
                assert_near(model, got)
        cache = r.engine.kv_cache
        assert cache.num_free_blocks == cache.num_total_blocks and cache.states.num_free == 4
    finally:
        r.close()


def test_bfloat16_logits_do_not_depend_on_the_schedule(model):
    from zse_b200.trace import TraceRunner
    r = TraceRunner(model.path, "bfloat16", MAX_TOKENS)
    whole = replay(r, model, schedule("whole"))
    for name in ("portions-2", "mixed", "prompt-then-decode"):
        for rid, rows in replay(r, model, schedule(name)).items():
            d = np.sqrt(((rows - whole[rid.split("#")[0]][: len(rows)]) ** 2).mean(1)) / model.want["a"].std()
            assert np.median(d) < 0.03 and (d < 0.3).mean() > 0.9, (name, rid)
    r.close()


def gpu_engine(path, **kw):
    from zse_b200.config import EngineConfig
    from zse_b200.engine import ZStreamerEngine
    kw = dict(dict(dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=40, max_seq_len=512), **kw)
    return ZStreamerEngine(path, config=EngineConfig(**kw))


@pytest.mark.parametrize("kw", [dict(), dict(pipeline_decode=False), dict(use_cuda_graphs=False, prefill_chunk_size=32),
                                dict(max_batch_seqs=2, prefill_chunk_size=24, decode_per_prefill=0),
                                dict(speculative_k=3)])
def test_greedy_generation_matches_the_oracle(small, kw):
    eng = gpu_engine(small.path, **kw)
    prompts = [small.tokens["a"][:75], small.tokens["b"][:5], small.tokens["c"], small.tokens["d"][:40]]
    rids = [eng.add_request_tokens(p, max_tokens=8, temperature=0.0, stop_tokens=[]) for p in prompts]
    eng.run_until_done()
    for p, rid in zip(prompts, rids):
        assert eng.get_result(rid).output_tokens == oracle.greedy(small.cfg, small.weights, p, 8)
    eng.destroy()


def test_long_decoding(small):
    """A hundred and twenty steps through graphs, over several window and block borders, against the oracle's logits."""
    from zse_b200.trace import TraceRunner
    r = TraceRunner(small.path, "float32", MAX_TOKENS)
    assert_close(small, replay(r, small, [[("a", 30)]] + [[("a", 1)] for _ in range(LENGTHS["a"] - 30)]), 5e-4)
    assert r.engine.runner.timings["graph_replays"] >= 100
    r.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_and_wide_passes(tmp_path, dtype):
    """Passes of more rows than take split-K planes, means in several blocks of the cache, in portions and decoded."""
    from zse_b200.trace import TraceRunner
    cfg, ranks = oracle.config(64, 90, [oracle.layer(oracle.window(4, 2, 32, 24, 200, 4, rot=16), oracle.memory(2, 32, 72),
                                                     oracle.dense(40)),
                                        oracle.layer(oracle.window(4, 1, 64, 64, 30, 90), oracle.memory(4, 64, 32, tau=30.0),
                                                     None)], loop=(0, 2, 2))
    weights = oracle.random_weights(cfg, ranks, 5)
    m = types.SimpleNamespace(cfg=cfg, weights=weights, path=write_model(tmp_path / "long", cfg, weights))
    rng = np.random.default_rng(3)
    m.tokens = {"a": rng.integers(0, 90, 700).tolist(), "b": rng.integers(0, 90, 420).tolist()}
    with torch.no_grad():
        m.want = {k: oracle.forward(cfg, weights, t).numpy() for k, t in m.tokens.items()}
    r = TraceRunner(m.path, dtype, 704 + 448)
    for steps in ([[("a", 700), ("b", 420)]], [[("b", 5)], [("a", 320), ("b", 255)], [("a", 350), ("b", 1)], [("b", 159)]]
                  + [[("a", 1)]] * 30):
        got = replay(r, m, steps)
        assert_close(m, got, 5e-4) if dtype == "float32" else assert_near(m, got)
    r.close()


def test_synthetic_model_generates_in_bfloat16(tmp_path):
    from zse_b200.format import synth
    path = str(tmp_path / "s.zse")
    synth.write_random_model(path, synth.shape_config("tiny-vobisun"), seed=3)
    eng = gpu_engine(path, dtype=None)
    rids = [eng.add_request_tokens(list(range(k, k + 60)), max_tokens=6, temperature=0.0, stop_tokens=[]) for k in range(6)]
    eng.run_until_done()
    assert all(len(eng.get_result(r).output_tokens) == 6 for r in rids)
    eng.destroy()
