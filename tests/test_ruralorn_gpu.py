"""Ruralorn on the GPU: every kernel against float64 statements of the same operation, whole models against the plain
oracle in float32 and bfloat16, generation through the engine."""
import math
import os
import sys
import types

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import latent_oracle as oracle                                       # noqa: E402
from helpers.ruralorn_cases import (CASES, MAX_TOKENS, SCHEDULES, Model, assert_close, assert_near, errors,  # noqa: E402
                                    replay, schedule)

from zse_b200.format.config import LatentSpec, MoESpec                            # noqa: E402

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
F64 = torch.float64


@pytest.fixture(scope="module")
def ops():
    from zse_b200.ops.backend import CudaOps
    o = CudaOps("cuda")
    yield o
    o.check()


def rel(a, b):
    return ((a.to(F64) - b).abs().max() / b.abs().max()).item()


def tol(dt):
    return 1.5e-2 if dt == BF else 2e-5


# ---- kernels ----------------------------------------------------------------------------------------------------------
# spec, with the head counts, ranks and windows that take different kernels: one and two groups of 16 heads, latent up to
# 128 / 256 / 512, and shapes only the general kernels take (in bfloat16: nothing a multiple of 8)
SPECS = {
    "one-group": LatentSpec(5, 24, 8, 40, 72, 77, 0.3, 8, 1e3),
    "two-groups": LatentSpec(18, 64, 32, 64, 192, 300, 0.12, 32, 1e4),
    "wide": LatentSpec(48, 128, 64, 128, 512, 700, 0.072, 64, 1e4),
    "wide-values": LatentSpec(3, 32, 16, 144, 344, 129, 0.14, 8, 1e4),
    "long-row": LatentSpec(20, 32, 128, 32, 512, 200, 0.08, 128, 1e4),       # more than the tcgen05 form's nine panels
    "smallest": LatentSpec(1, 8, 8, 8, 8, 3, 0.3, 8, 1e2),
    "no-window": LatentSpec(4, 16, 16, 24, 128, 0, 0.2, 16, 1e4),
    "general": LatentSpec(3, 10, 6, 7, 22, 50, 0.4, 4, 1e3),
}


class Layer:
    """One layer's projections and cached rows; the plain results come from float64 copies."""

    def __init__(self, ops, spec, dt, blocks=40, bs=64, seqs=6, width=12, seed=0):
        g = torch.Generator(device="cuda").manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
        H, d, vd, kr = spec.heads, spec.dim, spec.vdim, spec.kv_rank
        v0 = (H * d + 7) // 8 * 8
        self.spec, self.dt, self.bs = spec, dt, bs
        self.ukv = torch.zeros(v0 + (H * vd + 7) // 8 * 8, kr, device="cuda", dtype=dt)
        self.ukv[: H * d] = (rnd(H * d, kr) * kr ** -0.5).to(dt)
        self.ukv[v0: v0 + H * vd] = (rnd(H * vd, kr) * kr ** -0.5).to(dt)
        self.w = types.SimpleNamespace(uk=self.ukv[: H * d], uv=self.ukv[v0: v0 + H * vd],
                                       ukv=ops.dense_linear(self.ukv))
        # the pool's blocks are wider than this layer's: strided rows
        pool = torch.zeros(blocks, bs * (spec.row + 16), device="cuda", dtype=dt)
        self.rows = pool.as_strided((blocks, bs, spec.row), (pool.stride(0), spec.row, 1))
        self.rows[..., : kr + spec.rot_dim] = rnd(blocks, bs, kr + spec.rot_dim).to(dt)
        self.tables = torch.stack([torch.randperm(blocks, device="cuda", generator=g)[:width]
                                   for _ in range(seqs)]).int()
        self.inp = torch.zeros(400, spec.in_width, device="cuda", dtype=dt)
        self.inp.copy_(rnd(400, spec.in_width))

    def row_at(self, seq, pos):
        return self.rows[self.tables[seq, pos // self.bs].long(), pos % self.bs]

    def plain(self, t, seq, pos):
        """Row t of ``inp`` as the query at ``pos`` of sequence ``seq``: gated heads, float64."""
        s = self.spec
        H, d, r, kr, vd = s.heads, s.dim, s.rot_dim, s.kv_rank, s.vdim
        lo = max(0, pos + 1 - s.window) if s.window else 0
        j = torch.arange(lo, pos + 1, device="cuda")
        blk = self.tables[seq][j // self.bs].long()
        j, blk = j[blk >= 0], blk[blk >= 0]
        rows = self.rows[blk, j % self.bs].to(F64)
        q = self.inp[t, : H * (d + r)].to(F64).view(H, d + r)
        k = torch.einsum("hdc,nc->hnd", self.w.uk.to(F64).view(H, d, kr), rows[:, :kr])
        v = torch.einsum("hvc,nc->hnv", self.w.uv.to(F64).view(H, vd, kr), rows[:, :kr])
        sc = torch.einsum("hd,hnd->hn", q[:, :d], k) + q[:, d:] @ rows[:, kr: kr + r].T
        y = torch.einsum("hn,hnv->hv", torch.softmax(sc * s.scale, -1), v).reshape(-1)
        return y * torch.sigmoid(self.inp[t, s.gate_col: s.gate_col + H * vd].to(F64))

    def tokens(self, ops, seqs, positions, splits=1):
        s, M = self.spec, len(seqs)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
        z = lambda n, dt: torch.zeros(n, dtype=dt, device="cuda")
        out = z(M * s.heads * s.vdim, self.dt).view(M, -1)
        ops.latent_attn(self.inp, self.w, self.rows, self.tables, i32(seqs), i32(positions), z(M * s.heads * s.row, self.dt),
                        z(M * s.heads * s.kv_rank, self.dt), out, M, s, z(M * splits * s.heads * (s.kv_rank + 2), F32),
                        splits)
        return out

    def chunks(self, ops, spans, first=0):
        """``spans``: (start, tokens) per sequence, packed from row 0 of ``inp``."""
        from zse_b200.models.latent_moe import ChunkGroup
        s = self.spec
        cu, off, total = [0], [], 0
        for start, n in spans:
            off.append(total if len(off) >= first else 0)
            if len(off) > first:
                total += n + (min(start, s.window - 1) if s.window else start)
            cu.append(cu[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
        z = lambda n: torch.zeros(n, dtype=self.dt, device="cuda")
        out = z(cu[-1] * s.heads * s.vdim).view(cu[-1], -1)
        ops.latent_attn_chunks(self.inp, self.w, self.rows, self.tables, i32(cu), i32([a for a, _ in spans]), i32(off),
                               ChunkGroup(first, len(spans), total, max(n for _, n in spans[first:])),
                               (z((total + 3) * s.kv_rank), z((total + 3) * s.rot_dim), z((total + 3) * self.ukv.shape[0])),
                               out, s)
        return out, cu


@pytest.fixture
def form(ops, request):
    """The tensor-core form of decode attention that the test runs on."""
    ops.latent_form, old = request.param, ops.latent_form
    yield request.param
    ops.latent_form = old


@pytest.mark.parametrize("form,dt", [(1, BF), (2, BF), (0, F32)], indirect=["form"])
@pytest.mark.parametrize("name", list(SPECS))
@pytest.mark.parametrize("bs", [64, 16, 128])
def test_tokens_against_cached_rows(ops, name, dt, form, bs):
    L = Layer(ops, SPECS[name], dt, blocks=40 * 64 // bs, bs=bs, width=12 * 64 // bs)
    L.tables[3, 1] = -1                                 # a hole, inside some windows
    seqs, pos = [0, 1, 2, 3, 4, 5, 5, 0], [0, 1, 63, 150, 64, 700, 511, 199]
    want = torch.stack([L.plain(t, s, p) for t, (s, p) in enumerate(zip(seqs, pos))])
    for splits in (1, 2, 8):
        assert rel(L.tokens(ops, seqs, pos, splits), want) < tol(dt), splits
    ops.check()


@pytest.mark.parametrize("name", [n for n in SPECS if n != "general"])
def test_chunks_against_expanded_rows(ops, name):
    L = Layer(ops, SPECS[name], BF)
    assert ops.latent_expands(L.spec, BF)
    L.tables[2, 2] = -1
    spans = [(3, 5), (0, 70), (200, 17), (400, 130), (63, 64)]     # the first sequence is not part of the group
    out, cu = L.chunks(ops, spans, first=1)
    assert (out[: cu[1]] == 0).all()
    for s in range(1, len(spans)):
        for i in sorted({0, 1, spans[s][1] // 2, 63 % spans[s][1], spans[s][1] - 1}):
            t = cu[s] + i
            assert rel(out[t], L.plain(t, s, spans[s][0] + i)) < tol(BF), (s, i)


@pytest.mark.parametrize("form,dt,what", [(1, BF, "tokens"), (2, BF, "tokens"), (0, F32, "tokens"), (1, BF, "chunks")],
                         indirect=["form"])
@pytest.mark.parametrize("name", ["one-group", "two-groups", "wide"])
def test_one_loud_key_inside_and_outside_the_window(ops, name, dt, form, what):
    """A key that takes all the weight sits on the last place that is seen, one before it, far away, on block borders, on
    the token itself and on the next one."""
    spec = SPECS[name]
    H, d, r, kr = spec.heads, spec.dim, spec.rot_dim, spec.kv_rank
    for pos in (spec.window - 1, spec.window, 447, 640):
        for key in sorted({pos, pos + 1, pos - spec.window + 1, pos - spec.window, pos - spec.window // 2,
                           pos // 64 * 64, pos // 64 * 64 - 1, 0}):
            if not 0 <= key < 760:
                continue
            L = Layer(ops, spec, dt, seed=pos)
            t = 20                                       # a query in the middle of the chunk
            q = L.inp[t, : H * (d + r)].float().view(H, d + r)
            lat = torch.einsum("hd,hdc->hc", q[:, :d], L.w.uk.float().view(H, d, kr))
            loud = torch.cat([lat[H - 1], q[H - 1, d:]])
            L.row_at(0, key)[: kr + r] = (loud * (60 / spec.scale / loud.pow(2).sum())).to(dt)
            want = L.plain(t, 0, pos)
            if what == "tokens":
                one = Layer.tokens.__get__(L)
                L.inp[0] = L.inp[t]
                got = one(ops, [0], [pos], 2)[0]
            else:
                if pos < t:
                    continue
                got = L.chunks(ops, [(pos - t, 40)])[0][t]
            assert rel(got, want) < tol(dt), (pos, key)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(SPECS))
@pytest.mark.parametrize("planes", [0, 1, 4])
def test_prep(ops, name, dt, planes):
    L = Layer(ops, SPECS[name], dt)
    s = L.spec
    H, d, r, kr = s.heads, s.dim, s.rot_dim, s.kv_rank
    M = 70
    pl = torch.randn(max(planes, 1), M, s.in_width, device="cuda")
    src = pl.to(F64).sum(0) if planes else L.inp[:M].to(F64)
    pos = torch.randint(0, 3000, (M,), device="cuda", dtype=torch.int32)
    slots = torch.randperm(40 * 64, device="cuda")[:M]
    slots[5] = -1
    freqs = torch.tensor([s.rot_base ** (-2 * i / s.rot_dims) for i in range(s.rot_dims // 2)], device="cuda")
    w = (1 + 0.2 * torch.randn(kr, device="cuda")).to(dt)
    before = L.rows.clone()
    ops.latent_prep(L.inp, pl, planes, L.rows, pos, slots, freqs, w, s, 1e-3, M)

    def turn(v):                                        # [M, R]
        return oracle.rotate(v.cpu(), pos.cpu(), s.rot_dims, s.rot_base).cuda()
    lat = src[:, s.latent_col: s.latent_col + kr + r]
    c = oracle.rms_norm(lat[:, :kr], w.to(F64), 1e-3)
    k = turn(lat[:, kr:])
    limit = 1e-2 if dt == BF else 5e-4                  # fp32 angles of positions in the thousands
    for t in range(M):
        if t != 5:
            row = L.rows[slots[t] // 64, slots[t] % 64]
            assert rel(row[:kr], c[t]) < limit and rel(row[kr: kr + r], k[t]) < limit
            before[slots[t] // 64, slots[t] % 64, : kr + r] = row[: kr + r]
    assert torch.equal(before, L.rows)                  # nothing else was written
    for h in range(H):
        q = src[:, h * (d + r): (h + 1) * (d + r)]
        got = L.inp[:M, h * (d + r): (h + 1) * (d + r)]
        assert rel(got[:, :d], q[:, :d]) < limit and rel(got[:, d:], turn(q[:, d:])) < limit
    g = slice(s.gate_col, s.gate_col + H * s.vdim)
    assert rel(L.inp[:M, g], src[:, g]) < limit


MOES = {"shared": (256, MoESpec(16, 2, 64, 96)), "no-shared": (96, MoESpec(5, 1, 40, 0)), "all": (64, MoESpec(4, 4, 200, 24)),
        "general": (50, MoESpec(7, 3, 30, 21)), "many": (128, MoESpec(300, 8, 16, 136))}


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("name", list(MOES))
@pytest.mark.parametrize("M", [1, 2, 17, 130, 1100])
def test_routed_feed_forward(ops, name, dt, M):
    H, m = MOES[name]
    g = torch.Generator(device="cuda").manual_seed(M)
    mk = lambda *s: (torch.randn(*s, device="cuda", generator=g) * s[-1] ** -0.5).to(dt)
    router, up, down = mk(m.experts, H), mk(m.experts * m.ff, H), mk(m.experts * H, m.ff)
    su, sd = (mk(m.shared_ff, H), mk(H, m.shared_ff)) if m.shared_ff else (None, None)
    x = (2 * torch.randn(M, H, device="cuda", generator=g)).to(dt)
    if name == "shared" and M > 16:
        x[:] = x[:1]                                     # every token takes the same experts
    L = types.SimpleNamespace(moe=m, router=ops.dense_linear(router), up=up, down=down, shared_up=su, shared_down=sd)
    ws = ops.moe_workspace([m, MoESpec(3, 2, 8)], H, 1200, dt)
    xd = x.to(F64)
    score = torch.sigmoid(xd @ router.to(F64).T)
    w, e = score.topk(m.top, -1)
    want = torch.zeros(M, H, dtype=F64, device="cuda")
    ud, dd = up.to(F64).view(m.experts, m.ff, H), down.to(F64).view(m.experts, H, m.ff)
    for k in range(m.top):
        for ex in e[:, k].unique().tolist():
            t = torch.where(e[:, k] == ex)[0]
            want[t] += oracle.gelu((w[t, k, None] * xd[t]) @ ud[ex].T) @ dd[ex].T
    if m.shared_ff:
        want += oracle.gelu(xd @ su.to(F64).T) @ sd.to(F64).T
    for _ in range(2):                                   # the tables are ready for the next layer
        slots = ops.moe(L, x, M, ws)
        assert slots.shape == (M, m.top + (m.shared_ff > 0), H)
        assert rel(slots.to(F64).sum(1), want) < tol(dt)
    assert int(ws.counts.abs().sum()) == 0


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H", [50, 96, 2048, 7168])
@pytest.mark.parametrize("M", [1, 33, 300])
def test_residual_sum_and_norm(ops, dt, H, M):
    for n_planes, n_slots, sd in ((0, 0, F32), (3, 0, F32), (0, 4, F32), (1, 3, dt)):
        res = torch.randn(M, H, device="cuda")
        planes, w = torch.randn(max(n_planes, 1), M, H, device="cuda"), torch.randn(H, device="cuda").to(dt)
        slots = torch.randn(M, n_slots, H, device="cuda").to(sd) if n_slots else None
        want = res.to(F64) + (planes.to(F64).sum(0) if n_planes else 0) + (slots.to(F64).sum(1) if n_slots else 0)
        out = torch.zeros(M, H, device="cuda", dtype=dt)
        ops.add_norm(res, planes, n_planes, slots, w, out, M, 0.5)
        assert rel(res, want) < 1e-6
        assert rel(out, oracle.rms_norm(want, w.to(F64), 0.5)) < (5e-3 if dt == BF else 1e-5)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("M,N,K", [(1, 77, 50), (5, 130, 96), (64, 1000, 320), (300, 513, 136), (33, 64, 2050)])
def test_linear(ops, dt, M, N, K):
    w, x = torch.randn(N, K, device="cuda").to(dt), torch.randn(M + 3, K, device="cuda").to(dt)
    want = x[:M].to(F64) @ w.to(F64).T
    L = ops.dense_linear(w)
    out = torch.zeros(M, N, device="cuda", dtype=dt)
    ops.linear(L, x, M, out)
    assert rel(out, want) < (5e-3 if dt == BF else 1e-5)
    planes = torch.full((8 * M * N,), float("nan"), device="cuda")
    n = ops.linear_partial(L, x, M, planes.view(8, M, N))
    assert rel(planes[: n * M * N].view(n, M, N).sum(0), want) < 1e-5
    f = torch.zeros(M, N, device="cuda")
    ops.linear_f32(L, x, M, f)
    assert rel(f, want) < 1e-5


def test_logits_and_token_choice(ops):
    x = torch.randn(9, 1003, device="cuda") * 30
    got = x.clone()
    ops.logits_finish(got, 9, 0.7, 25.0)
    want = 25 * torch.tanh(x.to(F64) * 0.7 / 25)
    assert rel(got, want) < 1e-6
    x[2, 100] = x[2, 900] = 1e3
    out = torch.zeros(9, dtype=torch.int32, device="cuda")
    ops.argmax(x, out, 9)
    assert out.tolist() == x.argmax(-1).tolist()[:2] + [100] + x.argmax(-1).tolist()[3:]
    pen = torch.tensor([1.0, 2.0] + [1.0] * 7, device="cuda")
    y = x.clone()
    one = lambda v: torch.tensor([v], dtype=torch.int32, device="cuda")
    ops.apply_repetition_penalty(y, one(1), one(5), one(2), 1, pen)
    y[1, 5] = x[1, 5]
    assert torch.equal(x, y)


# ---- whole models -------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp("ruralorn-gpu") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("ruralorn-gpu-small"))


@pytest.mark.parametrize("name", SCHEDULES + ["token-by-token"])
def test_schedules_in_float32(model, name):
    from zse_b200.trace import TraceRunner
    r = TraceRunner(model.path, "float32", MAX_TOKENS)
    try:
        assert_close(model, replay(r, model, schedule(name)), 2e-4)
    finally:
        r.close()


@pytest.mark.parametrize("name", SCHEDULES)
def test_schedules_in_bfloat16(model, name):
    from zse_b200.trace import TraceRunner
    r = TraceRunner(model.path, "bfloat16", MAX_TOKENS)
    try:
        assert_near(model, replay(r, model, schedule(name)))
    finally:
        r.close()


def test_a_request_in_company_gets_its_own_logits(small):
    """Same portions, alone and beside others: nothing of the batch reaches a request's logits (exactly, where its rows
    go through the same kernels with the same split of the work)."""
    from zse_b200.trace import TraceRunner
    alone = TraceRunner(small.path, "float32", MAX_TOKENS)
    a = replay(alone, small, [[("a", 40)], [("a", 2)], [("a", 17)], [("a", 91)]])["a"]
    alone.close()
    many = TraceRunner(small.path, "float32", MAX_TOKENS)
    b = replay(many, small, [[("c", 9), ("a", 40), ("b", 30)], [("a", 2), ("b", 31)], [("d", 64), ("a", 17)],
                             [("d", 33), ("a", 91)]])["a"]
    many.close()
    assert np.abs(a - b).max() < 1e-4


def engine(path, **kw):
    from zse_b200.config import EngineConfig
    from zse_b200.engine import ZStreamerEngine
    kw = dict(dict(dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=24, max_seq_len=512), **kw)
    return ZStreamerEngine(path, config=EngineConfig(**kw))


def test_greedy_generation_matches_the_oracle(small):
    eng = engine(small.path, prefill_chunk_size=32)
    prompts = [small.tokens["a"][:75], small.tokens["b"][:5], small.tokens["c"], small.tokens["d"][:40]]
    rids = [eng.add_request_tokens(p, max_tokens=10, temperature=0.0, stop_tokens=[]) for p in prompts]
    eng.run_until_done()
    for p, rid in zip(prompts, rids):
        assert eng.get_result(rid).output_tokens == oracle.greedy(small.cfg, small.weights, p, 10)
    assert eng.runner.timings["graph_replays"] > 0
    eng.destroy()


def test_long_generation_is_the_same_with_and_without_graphs_and_company(small):
    out = []
    for graphs, company in ((True, False), (False, False), (True, True)):
        eng = engine(small.path, use_cuda_graphs=graphs)
        rid = eng.add_request_tokens(small.tokens["b"], max_tokens=230, temperature=0.0, stop_tokens=[])
        if company:
            for r in "acd":
                eng.add_request_tokens(small.tokens[r][:50], max_tokens=40, temperature=0.0, stop_tokens=[])
        eng.run_until_done()
        out.append(eng.get_result(rid).output_tokens)
        eng.destroy()
    assert out[0] == out[1] == out[2] and len(out[0]) == 230


def test_sampling_in_bfloat16(small):
    got = []
    for _ in range(2):
        eng = engine(small.path, dtype="bfloat16")
        rid = eng.add_request_tokens(small.tokens["c"], max_tokens=12, temperature=0.9, top_k=20, top_p=0.9, seed=7,
                                     repetition_penalty=1.1, stop_tokens=[])
        eng.run_until_done()
        got.append(eng.get_result(rid).output_tokens)
        eng.destroy()
    assert got[0] == got[1] and len(got[0]) == 12 and all(0 <= t < small.cfg["vocab"] for t in got[0])
