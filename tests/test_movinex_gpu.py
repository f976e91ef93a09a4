"""Movinex on the GPU: every kernel against the plain float64 statements of the same mechanism, whole models against the plain
oracle in float32 and bfloat16, generation through the engine."""
import dataclasses
import math
import os
import sys
import types

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import movinex_oracle as oracle                                      # noqa: E402
from helpers.latent_oracle import write_model                                     # noqa: E402
from helpers.movinex_cases import CASES, Model                                    # noqa: E402
from helpers.ruralorn_cases import (LENGTHS, MAX_TOKENS, SCHEDULES, assert_close, assert_near, replay,  # noqa: E402
                                    schedule)

from zse_b200.format.config import HeadsSpec, MoESpec, StateSpaceSpec             # noqa: E402
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


# ---- attention --------------------------------------------------------------------------------------------------------
W = dict(gate_each=True, learned_norm=False, k_as_v=True)
SPECS = {
    "window": HeadsSpec(8, 2, 64, 64, 0.3, window=130, keep_first=20, softcap=9.0, **W),
    "kept-past-a-block": HeadsSpec(6, 3, 128, 128, 0.2, window=100, keep_first=70, softcap=20.0, **W),
    "many-kept": HeadsSpec(4, 4, 40, 40, 0.4, window=33, keep_first=200, softcap=5.0, **W),
    "one-kv-head": HeadsSpec(20, 1, 48, 48, 0.4, window=64, keep_first=1, softcap=12.0, **W),
    "token-and-kept": HeadsSpec(4, 2, 32, 32, 0.5, window=1, keep_first=3, softcap=7.0, **W),
    "no-cap": HeadsSpec(4, 2, 72, 72, 0.3, window=128, keep_first=64, **W),
    "nothing-kept": HeadsSpec(4, 2, 24, 24, 0.4, window=65, softcap=4.0, **W),
    "cap-alone": HeadsSpec(6, 2, 64, 32, 0.3, softcap=6.0, gated=False, learned_norm=False),
    "everything": HeadsSpec(6, 2, 56, 40, 0.4, gated=False, learned_norm=False, bias=True),
    "wide": HeadsSpec(4, 2, 256, 200, 0.1, window=90, keep_first=40, softcap=10.0, gate_each=True),
    "general": HeadsSpec(6, 2, 18, 18, 0.4, window=50, keep_first=7, softcap=6.0, **W),
}


class Attention:
    """Sequences whose keys and values lie in blocks of a pool of wider rows, in random order."""

    def __init__(self, spec, dt, bs=64, seqs=5, tokens=700, seed=0, rows=420):
        g = torch.Generator(device="cuda").manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
        self.spec, self.dt, self.bs = spec, dt, bs
        width = (tokens + bs - 1) // bs
        self.tables = torch.randperm(width * seqs + 3, device="cuda", generator=g)[: width * seqs].view(seqs, width).int()
        pool = torch.zeros(width * seqs + 3, 1, 1, bs, spec.row + 8, device="cuda", dtype=dt)
        self.kv = PagedHeads(pool, spec)
        self.k, self.v = rnd(seqs, tokens, spec.kv_heads, spec.dim).to(dt), rnd(seqs, tokens, spec.kv_heads, spec.vdim).to(dt)
        self.inp = rnd(rows, spec.in_width).to(dt)
        self.store()

    def store(self):
        j = torch.arange(self.k.shape[1], device="cuda")
        for s in range(self.k.shape[0]):
            blk = self.tables[s, j // self.bs].long()
            self.kv.k[blk, :, j % self.bs, : self.spec.dim] = self.k[s]
            self.kv.v[blk, :, j % self.bs, : self.spec.vdim] = self.v[s]

    def plain(self, t, seq, pos):
        s = self.spec
        q = self.inp[t, : s.heads * s.dim].cpu().to(F64).view(s.heads, s.dim)
        k, v = self.k[seq, : pos + 1].cpu().to(F64), self.v[seq, : pos + 1].cpu().to(F64)
        see = oracle.visible(pos + 1, s.window or None, s.keep_first)[pos:]
        per = s.heads // s.kv_heads
        y = torch.cat([oracle.weighted_values(q[n: n + 1], k[:, n // per], v[:, n // per], s.scale, see, s.softcap or None)
                       for n in range(s.heads)], -1)[0]
        if s.gated:
            y = y * oracle.sigmoid(self.inp[t, s.gate_col: s.gate_col + s.gate_width].cpu().to(F64))
        return y

    def rows(self, ops, seqs, positions, splits=1):
        s, M = self.spec, len(seqs)
        out = torch.zeros(M, s.heads * s.vdim, dtype=self.dt, device="cuda")
        ops.heads_attn(self.inp, self.kv, self.tables, i32(seqs), i32(positions), out, M, s,
                       torch.zeros(M * splits * s.heads * (s.vdim + 2), device="cuda"), splits)
        return out

    def chunks(self, ops, spans, first=0):
        cu = np.cumsum([0] + [n for _, n in spans]).tolist()
        pos = i32([a + i for a, n in spans for i in range(n)])
        out = torch.zeros(cu[-1], self.spec.heads * self.spec.vdim, dtype=self.dt, device="cuda")
        ops.heads_attn_chunks(self.inp, self.kv, self.tables, i32(cu), i32([a for a, _ in spans]), pos, first, len(spans),
                              max(n for _, n in spans[first:]), out, self.spec)
        return out, cu


@pytest.fixture
def form(ops, request):
    """The tensor-core form of attention in tiles of queries that the test runs on."""
    ops.heads_form, old = request.param, ops.heads_form
    yield request.param
    ops.heads_form = old


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(SPECS))
@pytest.mark.parametrize("bs", [64, 16])
def test_rows_against_cached_keys(ops, name, dt, bs):
    A = Attention(SPECS[name], dt, bs=bs)
    seqs, pos = [0, 1, 2, 3, 4, 4, 0, 1, 2, 3], [0, 1, 63, 150, 64, 690, 511, 199, 20, 130]
    want = torch.stack([A.plain(t, s, p) for t, (s, p) in enumerate(zip(seqs, pos))])
    for splits in (1, 2, 8):
        assert rel(A.rows(ops, seqs, pos, splits), want) < tol(dt), splits
    ops.check()


@pytest.mark.parametrize("name", [n for n in SPECS if n != "general"])
@pytest.mark.parametrize("bs", [64, 32, 48])
@pytest.mark.parametrize("form", [1, 2], indirect=True)
def test_tiles_of_queries_against_cached_keys(ops, name, bs, form):
    A = Attention(SPECS[name], BF, bs=bs)
    assert ops.heads_expands(A.spec, BF)
    spans = [(3, 5), (0, 150), (300, 17), (470, 130), (63, 64)]    # the first sequence is not part of the call
    out, cu = A.chunks(ops, spans, first=1)
    assert (out[: cu[1]] == 0).all()
    for s in range(1, len(spans)):
        for i in sorted({0, 1, spans[s][1] // 2, 63 % spans[s][1], 64 % spans[s][1], 128 % spans[s][1], spans[s][1] - 1}):
            assert rel(out[cu[s] + i], A.plain(cu[s] + i, s, spans[s][0] + i)) < tol(BF), (s, i)
    ops.check()


@pytest.mark.parametrize("name", ["window", "kept-past-a-block", "many-kept", "no-cap"])
def test_blocks_that_left_are_not_read(ops, name):
    """Between the kept tokens' blocks and the window's there are holes."""
    A = Attention(SPECS[name], BF)
    s, pos = A.spec, 600
    want = torch.stack([A.plain(t, 0, pos - 20 + t) for t in range(21)])
    A.tables[0, (s.keep_first + 63) // 64: s.first_seen(pos - 20) // 64] = -1
    assert rel(A.chunks(ops, [(pos - 20, 21)])[0], want) < tol(BF)
    assert rel(A.rows(ops, [0] * 21, list(range(pos - 20, pos + 1)), 4), want) < tol(BF)
    ops.check()


@pytest.mark.parametrize("dt,what,form", [(BF, "rows", 1), (F32, "rows", 1), (BF, "tiles", 1), (BF, "tiles", 2)],
                         indirect=["form"])
@pytest.mark.parametrize("name", ["window", "kept-past-a-block", "no-cap", "nothing-kept"])
def test_one_loud_key_inside_and_outside(ops, name, dt, what, form):
    """A key that takes nearly all the weight sits on the window's first place, one before it, on the last kept token and the
    next one, far away, on block borders, on the token itself and on the next one."""
    spec = dataclasses.replace(SPECS[name], softcap=SPECS[name].softcap and 14.0)
    size, keep, g = spec.window, spec.keep_first, spec.kv_heads - 1
    for pos in (size - 1, size, size + keep, 447, 640):
        lo = spec.first_seen(pos)
        for key in sorted({pos, pos + 1, lo, lo - 1, (lo + pos) // 2, pos // 64 * 64, pos // 64 * 64 - 1, keep - 1, keep, 0}):
            if not 0 <= key < 700:
                continue
            A = Attention(spec, dt, seed=pos, seqs=1)
            t = 20                                       # a query in the middle of the portion
            q = A.inp[t, (spec.heads - 1) * spec.dim: spec.heads * spec.dim].float()
            A.k[0, key, g] = (q * (40 / spec.scale / q.pow(2).sum())).to(dt)
            A.store()
            want = A.plain(t, 0, pos)
            if what == "rows":
                A.inp[0] = A.inp[t]
                got = A.rows(ops, [0], [pos], 2)[0]
            elif pos < t:
                continue
            else:
                got = A.chunks(ops, [(pos - t, 40)])[0][t]
            assert rel(got, want) < tol(dt), (pos, key)


PREP = {
    "rotated": HeadsSpec(6, 2, 64, 64, 0.3, window=50, keep_first=4, rot_dims=32, rot_base=5e4, **W),
    "all-rotated": HeadsSpec(3, 3, 128, 128, 0.3, window=50, rot_dims=128, rot_base=1e4, **W),
    "pair": HeadsSpec(5, 1, 24, 24, 0.3, window=50, rot_dims=2, rot_base=1e4, **W),
    "not-by-four": HeadsSpec(4, 2, 48, 48, 0.3, window=50, rot_dims=38, rot_base=300.0, **W),
    "bias": HeadsSpec(4, 2, 48, 40, 0.3, gated=False, learned_norm=False, bias=True, temp_coef=0.3, temp_every=64),
    "head-gates": HeadsSpec(4, 2, 16, 24, 0.3, bias=True, temp_coef=-0.2, temp_every=1, rot_dims=8),
    "long-heads": HeadsSpec(2, 1, 320, 320, 0.3, rot_dims=300, rot_base=1e4, **W),
    "general": HeadsSpec(3, 3, 10, 10, 0.3, bias=True, rot_dims=6, temp_coef=0.5, temp_every=7, **W),
}


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(PREP))
@pytest.mark.parametrize("planes", [0, 1, 4])
def test_heads_prep(ops, name, dt, planes):
    s, M, eps = PREP[name], 60, 1e-5
    H, G, d, vd = s.heads, s.kv_heads, s.dim, s.vdim
    g = torch.Generator(device="cuda").manual_seed(3)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", generator=g)
    inp, pl = rnd(M, s.in_width).to(dt), rnd(max(1, planes), M, s.in_width)
    full = (pl.to(F64).sum(0) if planes else inp.to(F64)).cpu()
    L = types.SimpleNamespace(q_norm=rnd(d).to(dt) if s.learned_norm else None, k_norm=rnd(d).to(dt) if s.learned_norm else None,
                              bias=rnd(s.in_width).to(dt) if s.bias else None, freqs=ops.rotation(s.rot_dims, s.rot_base))
    if s.bias:
        L.bias[s.gate_col:] = 0                         # gates have none
        full = full + L.bias.cpu().to(F64)
    pos = [0, 1, 2, 63, 64, 100, 5000, 131071] + list(range(300, 352))
    pool = torch.zeros(20, 1, 1, 64, s.row + 8, device="cuda", dtype=dt)
    kv = PagedHeads(pool, s)
    slots = torch.randperm(20 * 64, device="cuda", generator=g)[:M]
    slots[5] = -1
    ops.heads_prep(inp, pl, planes, kv, slots, L, s, eps, M, i32(pos))

    def finish(x, w):
        """[M, n, d]: rotation at the rows' own positions, then the norm."""
        x = x.clone()
        for i in range(s.rot_dims // 2):
            a = torch.tensor([p * s.rot_base ** (-2 * i / s.rot_dims) for p in pos], dtype=F64)[:, None]
            u, v = x[..., 2 * i].clone(), x[..., 2 * i + 1].clone()
            x[..., 2 * i], x[..., 2 * i + 1] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
        x = x / oracle.rms(x, eps)
        return x if w is None else x * w.cpu().to(F64)
    temp = torch.tensor([1 + s.temp_coef * math.log((p + 1) // s.temp_every + 1) for p in pos], dtype=F64)
    q = finish(full[:, : H * d].view(M, H, d), L.q_norm) * temp[:, None, None]
    assert rel(inp[:, : H * d], q.reshape(M, -1)) < tol(dt)
    if s.gated:
        assert rel(inp[:, s.gate_col: s.gate_col + s.gate_width], full[:, s.gate_col: s.gate_col + s.gate_width]) < tol(dt)
    ok = (slots >= 0).cpu()
    blk, at = (slots[slots >= 0] // 64), (slots[slots >= 0] % 64)
    raw = full[:, s.k_col: s.k_col + G * d].view(M, G, d)
    v = raw if s.k_as_v else full[:, s.v_col: s.v_col + G * vd].view(M, G, vd)
    assert rel(kv.k[blk, :, at, :d], finish(raw, L.k_norm)[ok]) < tol(dt)
    assert rel(kv.v[blk, :, at, :vd], v[ok]) < tol(dt)
    assert (kv.k[..., d:] == 0).all() and (kv.v[..., vd:] == 0).all()
    untouched = torch.ones(20 * 64, dtype=torch.bool, device="cuda")
    untouched[slots[slots >= 0]] = False
    assert (kv.k.transpose(1, 2).reshape(20 * 64, -1)[untouched] == 0).all()
    ops.check()


# ---- state space -------------------------------------------------------------------------------------------------------
SPACES = {
    "small": StateSpaceSpec(4, 24, 16, 2, 3, 1),
    "usual": StateSpaceSpec(6, 64, 128, 1, 4, 1),
    "big": StateSpaceSpec(2, 72, 256, 2, 2, 4),
    "half-steps": StateSpaceSpec(5, 40, 72, 1, 4, 5),
    "many-columns": StateSpaceSpec(3, 136, 40, 3, 1, 2),
    "between": StateSpaceSpec(2, 64, 200, 1, 5, 1),
    "general": StateSpaceSpec(3, 7, 10, 3, 6, 7),
    "one": StateSpaceSpec(1, 8, 8, 1, 3, 1),
}


class Space:
    def __init__(self, spec, dt, rows=420, slots=7, seed=0, slow=True):
        g = torch.Generator(device="cuda").manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
        self.spec, self.dt, self.at = spec, dt, 12
        s = spec
        self.inp, self.xbc = rnd(rows, s.in_width).to(dt), rnd(rows, s.conv_width).to(dt)
        self.dt_ = torch.nn.functional.softplus(rnd(rows, s.heads) - 1.5).contiguous()
        A_log = (-3.0 if slow else 0.5) + 1.2 * rnd(s.heads)
        w = torch.zeros(s.conv, s.conv_width, device="cuda")
        b = torch.zeros(s.conv_width, device="cuda")
        for at, n in self.channels():
            w[:, at: at + n], b[at: at + n] = rnd(s.conv, n), rnd(n)
        self.A_log = A_log
        self.L = types.SimpleNamespace(conv_w=w, conv_b=b, dt_bias=rnd(s.heads), neg_a=-torch.exp(A_log), D=rnd(s.heads),
                                       w_in=types.SimpleNamespace(kind="bf16" if dt == BF else "f32", K=64))
        floats = (s.state_floats + 3) // 4 * 4
        self.states = torch.zeros(2 * slots, self.at + floats + 4, device="cuda")
        self.states[:, self.at: self.at + s.state_floats] = rnd(2 * slots, s.state_floats)

    def channels(self):
        s = self.spec
        return (0, s.inner), (s.b_at, s.groups * s.state), (s.c_at, s.groups * s.state)

    def memory(self, row):
        s = self.spec
        return self.states[row, self.at: self.at + s.heads * s.state * s.vdim].to(F64).view(s.heads, s.state, s.vdim).clone()

    def tail(self, row):
        s = self.spec
        return self.states[row, self.at + s.conv_at: self.at + s.state_floats].view(s.conv - 1, s.conv_width).clone()

    def plain(self, a, e, read):
        """Rows [a, e) from the memory in row ``read`` (-1: none): (gated read-outs, memory) in float64."""
        s = self.spec
        H, v, G, n = s.heads, s.vdim, s.groups, s.state
        S = self.memory(read) if read >= 0 else torch.zeros(H, n, v, dtype=F64, device="cuda")
        x = self.xbc[a:e].to(F64)
        B, C = (x[:, at: at + G * n].view(-1, G, n).repeat_interleave(H // G, 1) for at in (s.b_at, s.c_at))
        X, d = x[:, : H * v].view(-1, H, v), self.dt_[a:e].to(F64)
        out = []
        for t in range(e - a):
            S = torch.exp(-torch.exp(self.A_log.to(F64)) * d[t])[:, None, None] * S \
                + d[t][:, None, None] * B[t][:, :, None] * X[t][:, None, :]
            out.append((S * C[t][:, :, None]).sum(1) + self.L.D.to(F64)[:, None] * X[t])
        return torch.stack(out).view(e - a, -1) * oracle.silu(self.inp[a:e, : H * v].to(F64)), S

    def run(self, ops, cu, rows, chunkwise, first=0):
        s, M, S = self.spec, cu[-1] if cu is not None else rows.shape[1], rows.shape[1]
        out = torch.zeros(M, s.inner, dtype=self.dt, device="cuda")
        cu_d = i32(cu) if cu is not None else None
        if chunkwise:
            ops.state_space_chunks(self.inp, self.xbc, self.dt_, self.states, self.at, rows, cu_d, self.L, out, first, S, M, s)
        else:
            ops.state_space_tokens(self.inp, self.xbc, self.dt_, self.states, self.at, rows, cu_d, self.L, out, S, M, s)
        return out


def check_space(ops, name, dt, cu, rows, chunkwise, first=0, slow=True):
    m, limit = Space(SPACES[name], dt, slow=slow), 8e-3 if dt == BF else 2e-5
    want = [m.plain(cu[i], cu[i + 1], rows[0][i]) for i in range(len(rows[0]))]
    before, s = m.states.clone(), m.spec
    out = m.run(ops, cu, i32(rows), chunkwise, first)
    expect = before.clone()
    for i in range(first, len(rows[0])):
        y, S = want[i]
        a, e, w = cu[i], cu[i + 1], rows[1][i]
        err = (out[a:e].to(F64) - y).pow(2).mean(1).sqrt() / y.pow(2).mean(1).sqrt()
        assert err.max() < limit, (i, err.max().item(), int(err.argmax()))
        if w >= 0:
            assert rel(m.memory(w), S) < (1e-4 if chunkwise else 1e-5)       # 32 bits, also through the tensor cores
            n = s.heads * s.state * s.vdim
            expect[w, m.at: m.at + n] = m.states[w, m.at: m.at + n]
    assert torch.equal(m.states, expect)                 # other rows, other layers' parts, the convolution's inputs
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(SPACES))
def test_state_space_token_by_token(ops, name, dt):
    check_space(ops, name, dt, [0, 1, 2, 3, 4], [[4, -1, 7, -1], [5, 2, 6, -1]], False)      # a row each
    check_space(ops, name, dt, [0, 2, 18, 19, 150], [[4, -1, 7, 0], [5, 2, 6, 1]], False)


@pytest.mark.parametrize("slow", [True, False])
@pytest.mark.parametrize("name", [n for n in SPACES if n != "general"])
def test_state_space_in_chunks(ops, name, slow):
    assert ops.state_space_expands(SPACES[name], BF)
    check_space(ops, name, BF, [0, 64, 147, 160, 400], [[4, -1, 7, 0], [5, 2, 6, 1]], True, slow=slow)
    check_space(ops, name, BF, [0, 3, 130, 195], [[4, 2, -1], [5, 3, -1]], True, first=1, slow=slow)


def test_state_space_decodes_without_row_offsets(ops):
    m = Space(SPACES["usual"], BF, seed=4)
    rows = [[0, 2, -1, -1], [1, 3, 4, -1]]
    want = torch.cat([m.plain(i, i + 1, rows[0][i])[0] for i in range(4)])
    assert rel(m.run(ops, None, i32(rows), False), want) < 1e-2
    many = Space(SPACES["usual"], BF, rows=80, slots=64, seed=5)             # enough CTAs for the widest share of columns
    rows = [[2 * i for i in range(64)], [2 * i + 1 for i in range(64)]]
    want = torch.cat([many.plain(i, i + 1, 2 * i)[0] for i in range(64)])
    assert rel(many.run(ops, None, i32(rows), False), want) < 1e-2


@pytest.mark.parametrize("chunkwise", [True, False])
def test_state_space_keeps_a_token_from_long_ago(ops, chunkwise):
    """Almost no decay: one loud token at the start is what every later token reads; one long step, and it is gone."""
    spec = StateSpaceSpec(2, 64, 32, 1, 4, 1)
    for closed_at in (None, 200):
        m = Space(spec, BF)
        m.A_log = torch.full((2,), -9.0, device="cuda")
        m.L.neg_a, m.L.D = -torch.exp(m.A_log), torch.zeros(2, device="cuda")
        m.dt_.fill_(1e-3)
        m.dt_[3] = 50.0
        if closed_at is not None:
            m.dt_[closed_at] = 2e5
            m.xbc[closed_at, : spec.inner] *= 1e-6       # it forgets, and adds as much as the others
        want = m.plain(0, 400, -1)[0]
        out = m.run(ops, [0, 400], i32([[-1], [1]]), chunkwise)
        err = (out.to(F64) - want).pow(2).mean(1).sqrt() / want.pow(2).mean(1).sqrt()
        assert err.max() < 1.5e-2, (int(err.argmax()), err.max().item())


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(SPACES))
@pytest.mark.parametrize("planes,side", [(0, False), (0, True), (1, False), (5, False)])
def test_state_space_prep(ops, name, dt, planes, side):
    """Convolution over portions of one to many tokens, its inputs that are carried on, step sizes."""
    s = SPACES[name]
    m = Space(s, dt)
    cu, rows = [0, 1, 3, 6, 9, 30, 61], [[0, -1, 2, 4, -1, 6], [1, 8, 3, 5, -1, 7]]
    M, S = cu[-1], len(cu) - 1
    g = torch.Generator(device="cuda").manual_seed(1)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", generator=g)
    pl, sd, inp = 2 * rnd(max(1, planes), M, s.in_width), 3 * rnd(M, s.in_width - s.dt_col), m.inp[:M].clone()
    full = (pl.to(F64).sum(0) if planes else inp.to(F64)).cpu()
    before = [m.tail(r) if r >= 0 else torch.zeros(s.conv - 1, s.conv_width, device="cuda") for r in rows[0]]
    memory = m.states[:, m.at: m.at + s.conv_at].clone()
    xbc, dt_ = torch.zeros(M, s.conv_width, device="cuda", dtype=dt), torch.zeros(M, s.heads, device="cuda")
    seq = [i for i in range(S) for _ in range(cu[i + 1] - cu[i])]
    ops.state_space_prep(inp, pl, planes, sd if side else None, xbc, dt_, m.states, m.at, i32(rows), i32(seq), i32(cu), m.L, s,
                         M, S)
    z = full[:, s.dt_col: s.dt_col + s.heads]
    if side and dt == BF:                                # the general kernel leaves them in the projected row
        z = sd[:, : s.heads].cpu().to(F64)
    want = oracle.softplus(z + m.L.dt_bias.cpu().to(F64))
    assert ((dt_.cpu().to(F64) - want).abs() <= 2e-6 * (1 + want)).all()
    w, b = m.L.conv_w.cpu().to(F64).T, m.L.conv_b.cpu().to(F64)
    for i in range(S):
        x = torch.cat([before[i].cpu().to(F64), full[cu[i]: cu[i + 1], s.x_col: s.dt_col]])
        y = oracle.silu(oracle.causal_conv(x, w, b))[s.conv - 1:]
        for at, n in m.channels():
            assert rel(xbc[cu[i]: cu[i + 1], at: at + n], y[:, at: at + n]) < tol(dt), i
            if rows[1][i] >= 0 and s.conv > 1:
                assert rel(m.tail(rows[1][i])[:, at: at + n], x[-(s.conv - 1):, at: at + n]) < 1e-6, i
    assert torch.equal(m.states[:, m.at: m.at + s.conv_at], memory)
    if planes:
        assert rel(inp[:, : s.inner], full[:, : s.inner]) < tol(dt)
    ops.check()


def test_state_space_prep_of_decoding_rows_and_of_long_passes(ops):
    s = SPACES["usual"]
    m = Space(s, BF, rows=4200, slots=8)
    rows = [[0, 2, -1, -1], [1, 3, 4, -1]]
    before = [m.tail(r) if r >= 0 else torch.zeros(3, s.conv_width, device="cuda") for r in rows[0]]
    xbc, dt_ = torch.zeros(4200, s.conv_width, device="cuda", dtype=BF), torch.zeros(4200, s.heads, device="cuda")
    ops.state_space_prep(m.inp, m.xbc, 0, None, xbc, dt_, m.states, m.at, i32(rows), None, None, m.L, s, 4, 4)
    w, b = m.L.conv_w.to(F64).T, m.L.conv_b.to(F64)
    for i in range(4):
        x = torch.cat([before[i].to(F64), m.inp[i: i + 1, s.x_col: s.dt_col].to(F64)])
        assert rel(xbc[i], oracle.silu((w.T * x).sum(0) + b)) < tol(BF)
        if rows[1][i] >= 0:
            assert rel(m.tail(rows[1][i]), x[1:]) < 1e-6
    # several rows a thread: sequences begin and end inside a thread's rows
    cu = [0, 1000, 1009, 1010, 4100]
    seq = [i for i in range(4) for _ in range(cu[i + 1] - cu[i])]
    before = [m.tail(r) if r >= 0 else torch.zeros(3, s.conv_width, device="cuda") for r in rows[0]]
    ops.state_space_prep(m.inp, m.xbc, 0, None, xbc, dt_, m.states, m.at, i32(rows), i32(seq), i32(cu), m.L, s, 4100, 4)
    for i in range(4):
        x = torch.cat([before[i].to(F64), m.inp[cu[i]: cu[i + 1], s.x_col: s.dt_col].to(F64)])
        y = b + sum(w.T[j] * x[j: j + cu[i + 1] - cu[i]] for j in range(4))
        assert rel(xbc[cu[i]: cu[i + 1]], oracle.silu(y)) < tol(BF)
        if rows[1][i] >= 0:
            assert rel(m.tail(rows[1][i]), x[-3:]) < 1e-6
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("width,parts", [(96, 1), (96, 4), (51, 3), (4096, 1), (20000, 1), (8192, 8)])
def test_norm_in_parts(ops, dt, width, parts):
    g = torch.Generator(device="cuda").manual_seed(width)
    x, w = torch.randn(9, width, device="cuda", generator=g).to(dt), torch.randn(width, device="cuda", generator=g).to(dt)
    x[3] *= 1e-3
    want = (oracle.norm_in_parts(x.cpu().to(F64), parts, 1e-5) * w.cpu().to(F64))
    ops.group_norm(x, w, parts, 8, 1e-5)
    assert rel(x[:8], want[:8]) < tol(dt)
    ops.check()


# ---- rows --------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H", [64, 51, 4096, 10000])
@pytest.mark.parametrize("planes,slots", [(1, 0), (4, 0), (0, 3), (0, 0)])
@pytest.mark.parametrize("scaled,replace,normed", [(True, False, True), (False, True, True), (True, False, False),
                                                   (False, False, False)])
def test_residual_with_layer_scale(ops, dt, H, planes, slots, scaled, replace, normed):
    M, eps = 9, 1e-5
    if replace and not planes:
        return
    g = torch.Generator(device="cuda").manual_seed(H)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    res, pl, w, f = rnd(M, H), rnd(max(1, planes), M, H), 0.3 * rnd(H).to(dt), rnd(H).to(dt)
    sl = rnd(M, slots, H).to(dt) if slots else None
    y = pl.to(F64).sum(0) if planes else torch.zeros(M, H, dtype=F64, device="cuda")
    y = (y if sl is None else y + sl.to(F64).sum(1)) * (f.to(F64) if scaled else 1.0)
    want = y if replace else res.to(F64) + y
    both = torch.zeros(M + 1, 2 * H, device="cuda", dtype=dt)
    ops.add_norm(res, pl, planes, sl, w if normed else None, both[:, :H], M, eps, scale=f if scaled else None, offset=1.0,
                 replace=replace)
    assert rel(res, want) < 1e-5
    assert rel(both[:M, :H], oracle.norm(want, w.to(F64), eps) if normed else want) < tol(dt)
    assert (both[:, H:] == 0).all() and (both[M] == 0).all()
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
def test_embedding_in_two_places(ops, dt):
    table = torch.randn(50, 72, device="cuda").to(dt)
    ids, res, both = i32([3, 49, 0, 3]), torch.zeros(4, 72, device="cuda"), torch.zeros(5, 144, device="cuda", dtype=dt)
    ops.embedding(table, ids, res, 4, copy=both[:, 72:])
    assert torch.equal(res, table[ids.long()].float()) and torch.equal(both[:4, 72:], table[ids.long()])
    assert (both[:, :72] == 0).all() and (both[4] == 0).all()


# ---- feed-forwards -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("M,ff,K", [(1, 40, 24), (70, 264, 96), (300, 520, 200), (13, 19, 51), (64, 64, 64)])
@pytest.mark.parametrize("kind", ["gelu_tanh_glu", "silu_glu"])
def test_gated_dense_products(ops, dt, M, ff, K, kind):
    g = torch.Generator(device="cuda").manual_seed(ff)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    x, a, u = (2 * rnd(M, K)).to(dt), (rnd(ff, K) * K ** -0.5).to(dt), (rnd(ff, K) * K ** -0.5).to(dt)
    out, tmp = torch.zeros(M, ff, device="cuda", dtype=dt), torch.zeros(M * 2 * ff, device="cuda", dtype=dt)
    ops.linear_glu(ops.glu_linear(a, u, dt), x, M, out, kind, tmp)
    act = oracle.gelu_tanh if kind == "gelu_tanh_glu" else oracle.silu
    assert rel(out, act(x.to(F64) @ a.to(F64).T) * (x.to(F64) @ u.to(F64).T)) < tol(dt)
    ops.check()


@pytest.mark.parametrize("M", [5, 300])
def test_columns_of_a_product_in_full_precision(ops, M):
    x, w = torch.randn(M, 96, device="cuda").to(BF), (torch.randn(200, 96, device="cuda") * 0.1).to(BF)
    out, side = torch.zeros(M, 200, device="cuda", dtype=BF), torch.zeros(M * 24, device="cuda")
    ops.linear(ops.dense_linear(w), x, M, out, side=(176, side))
    want = x.to(F64) @ w.to(F64).T
    assert rel(out[:, :176], want[:, :176]) < tol(BF) and (out[:, 176:] == 0).all()
    assert rel(side.view(M, 24), want[:, 176:]) < 1e-5
    ops.check()


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,E,top,ff,groups,keep", [(64, 8, 2, 40, 4, 2), (96, 20, 5, 64, 5, 2), (128, 33, 3, 24, 33, 7),
                                                    (51, 6, 3, 17, 2, 1), (256, 64, 6, 200, 8, 4), (64, 80, 4, 32, 40, 3),
                                                    (64, 12, 2, 24, 1, 1)])
@pytest.mark.parametrize("M", [1, 90, 700])
def test_experts_of_the_best_groups(ops, dt, H, E, top, ff, groups, keep, M):
    m = MoESpec(E, top, ff, activation="silu_glu", weigh="output", groups=groups, keep_groups=keep)
    g = torch.Generator(device="cuda").manual_seed(E * 100 + M)
    rnd = lambda *s, k=1.0: (torch.randn(*s, device="cuda", generator=g) * k).to(dt)
    x = rnd(M, H)
    ups = [(rnd(ff, H, k=H ** -0.5), rnd(ff, H, k=H ** -0.5)) for _ in range(E)]
    down, router = rnd(E * H, ff, k=ff ** -0.5), rnd(E, H, k=2 * H ** -0.5)
    L = types.SimpleNamespace(moe=m, router=ops.dense_linear(router), up=ops.moe_up(ups, dt, m), down=down, shared_up=None,
                              shared_down=None)
    s = oracle.sigmoid(x.to(F64) @ router.to(F64).T).cpu()
    ids = [oracle.choose(s[t], top, groups, keep) for t in range(M)]
    # rows where a slightly different score would choose otherwise may go either way
    noise = torch.randn(2, E, dtype=F64, generator=torch.Generator().manual_seed(7))
    sure = torch.tensor([all(sorted(oracle.choose(s[t] * (1 + 1e-4 * n), top, groups, keep)) == sorted(ids[t]) for n in noise)
                         for t in range(M)])
    weights = torch.zeros(M, E, dtype=F64)
    for t in range(M):
        weights[t, ids[t]] = s[t, ids[t]]
    xs, want = x.to(F64), torch.zeros(M, H, dtype=F64, device="cuda")
    for e in range(E):
        y = (oracle.silu(xs @ ups[e][0].to(F64).T) * (xs @ ups[e][1].to(F64).T)) @ down[e * H: (e + 1) * H].to(F64).T
        want += weights[:, e: e + 1].cuda() * y
    ws = ops.moe_workspace([m], H, max(M, 8), dt)
    for _ in range(2):
        got = ops.moe(L, x, M, ws).to(F64).sum(1)
    assert sure.float().mean() > 0.9 and rel(got[sure.cuda()], want[sure.cuda()]) < (2e-2 if dt == BF else 2e-5)
    ops.check()


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp("movinex") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("movinex-small"))


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
        assert cache.num_free_blocks == cache.num_total_blocks and (cache.states is None or cache.states.num_free == 4)
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
    kw = dict(dict(dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=24, max_seq_len=512), **kw)
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
    """Passes of more rows than take split-K planes, windows and kept tokens many blocks apart, in portions and decoded."""
    from zse_b200.trace import TraceRunner
    cfg = oracle.config(64, 90, [oracle.attention_layer(4, 2, 32, 24, oracle.dense(40), every=100),
                                 oracle.window_layer(4, 2, 32, 300, 70, oracle.moe(6, 2, 16, 3, 2), rot=16),
                                 oracle.mamba_layer(4, 32, 32, None, groups=2)], loop=(0, 3, 2))
    weights = oracle.random_weights(cfg, 5)
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
    synth.write_random_model(path, synth.shape_config("tiny-movinex"), seed=3)
    eng = gpu_engine(path, dtype=None)
    rids = [eng.add_request_tokens(list(range(k, k + 60)), max_tokens=6, temperature=0.0, stop_tokens=[]) for k in range(6)]
    eng.run_until_done()
    assert all(len(eng.get_result(r).output_tokens) == 6 for r in rids)
    eng.destroy()
