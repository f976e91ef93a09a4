"""Vobisun on the CPU path: configuration, loaders, means of blocks in the cache, recurrent state, batching and generation against
the plain oracle."""
import copy
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import vobisun_oracle as oracle                                      # noqa: E402
from helpers.latent_oracle import write_model                                     # noqa: E402
from helpers.ruralorn_cases import (LENGTHS, MAX_TOKENS, SCHEDULES, assert_close, assert_near, replay,  # noqa: E402
                                    schedule)
from helpers.vobisun_cases import CASES, SPECS, Model, PooledAttention, loud_places, make_loud  # noqa: E402

from zse_b200.cache.cache_manager import KVCacheManager                           # noqa: E402
from zse_b200.config import EngineConfig                                          # noqa: E402
from zse_b200.engine import ZStreamerEngine                                       # noqa: E402
from zse_b200.format.config import GatedLinearSpec, HeadsSpec, ModelConfig, TwinSpec  # noqa: E402
from zse_b200.format.directory import open_model                                  # noqa: E402
from zse_b200.ops import reference as ref                                         # noqa: E402
from zse_b200.ops.backend import TorchOps                                         # noqa: E402
from zse_b200.sched.memory_budget import MemoryBudget                             # noqa: E402
from zse_b200.trace import TraceRunner                                            # noqa: E402

F64 = torch.float64


@pytest.fixture(scope="module", autouse=True)
def few_threads():
    """The matrices are small: more threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp("vobisun") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("vobisun-small"))


def cpu_engine(path, **kw):
    kw = dict(dict(device="cpu", dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=40, max_seq_len=512),
              **kw)
    return ZStreamerEngine(path, config=EngineConfig(**kw))


@pytest.mark.parametrize("name", [s for s in SCHEDULES if s != "portions-2"])
def test_schedules_match_the_oracle(model, name):
    r = TraceRunner(model.path, "float32", MAX_TOKENS, device="cpu")
    try:
        assert_close(model, replay(r, model, schedule(name)), 5e-4)
        cache = r.engine.kv_cache
        assert cache.num_free_blocks == cache.num_total_blocks and cache.states.num_free == 4
    finally:
        r.close()


def test_portions_of_two_tokens(small):
    r = TraceRunner(small.path, "float32", MAX_TOKENS, device="cpu")
    assert_close(small, replay(r, small, schedule("portions-2")), 5e-4)
    r.close()


def test_bfloat16_stays_near_the_oracle(small):
    r = TraceRunner(small.path, "bfloat16", MAX_TOKENS, device="cpu")
    assert_near(small, replay(r, small, schedule("mixed")))
    r.close()


def _left(i, *path, value):
    def change(cfg, W):
        at = cfg["layers"][i]["mixer"]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value(at[path[-1]])
    return change


def _weights(suffix, value):
    def change(cfg, W):
        for k in W:
            if k.endswith(suffix):
                W[k] = value(W[k].float())
    return change


MISTAKES = {
    "window one longer": _left(0, "left", "mask", "size", value=lambda v: v + 1),
    "window one shorter": _left(0, "left", "mask", "size", value=lambda v: v - 1),
    "blocks one longer": _left(0, "left", "mask", "pool", value=lambda v: v + 1),
    "no blocks": _left(0, "left", "mask", "pool", value=lambda v: 10 ** 6),
    "rotated dimensions": _left(0, "left", "rot", "dims", value=lambda v: v + 4),
    "factor of the rotation": _left(0, "left", "rot", "scaling", "factor", value=lambda v: 1.0),
    "base of the rotation": _left(1, "left", "rot", "base", value=lambda v: 1e4),
    "scale": _left(2, "left", "scale", value=lambda v: v * 1.2),
    "share of the left mixer": _left(1, "left_scale", value=lambda v: v * 1.1),
    "share of the right mixer": _left(1, "right_scale", value=lambda v: v * 1.1),
    "divisor of the decays": _left(0, "right", "tau", value=lambda v: v * 1.3),
    "passes of the loop": lambda cfg, W: cfg["loop"].update(times=3),
    "embedding's scale": lambda cfg, W: cfg["embedding"].update(scale=1.0),
    "sinks": _weights(".sink", lambda w: w - 40),
    "factors of the heads": _weights(".temp", lambda w: w * 0 + 1),
    "query norm": _weights("q.norm", lambda w: w * 0 + 1),
    "biases of the values": _weights("v.b", lambda w: w * 0),
    "oldest tap": _weights("canon1", lambda w: torch.cat([w[:, :1] * 0, w[:, 1:]], 1)),
    "own tap": _weights("canon1", lambda w: torch.cat([w[:, :-1], w[:, -1:] * 0], 1)),
    "biases of the decays": _weights("a2.b", lambda w: w + 1),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_the_models_of_these_tests_show_a_mistake(small, name):
    """The oracle with one constant changed leaves the limits of the tests above by far, at some positions at least."""
    cfg, W = copy.deepcopy(small.cfg), dict(small.weights)
    MISTAKES[name](cfg, W)
    off = oracle.forward(cfg, W, small.tokens["a"]).numpy()
    d = np.sqrt(((off - small.want["a"]) ** 2).mean(1)) / small.want["a"].std()
    assert np.quantile(d, 0.85) > 3e-3


def test_a_lost_state_shows(small):
    """Without what came before position 84 the logits after it move, also beyond every window."""
    off = oracle.forward(small.cfg, small.weights, small.tokens["a"][84:]).numpy()
    d = np.sqrt(((off - small.want["a"][84:]) ** 2).mean(1)) / small.want["a"].std()
    assert d[:3].min() > 0.05 and d[:60].min() > 1e-2


# ---- configuration and files ----------------------------------------------------------------------------------------------
def test_configuration(small):
    with open_model(small.path) as l:
        c = l.config
    assert (c.arch, c.num_layers, c.hidden_size, c.vocab_size, c.input_conv) == ("vobisun", 4, 96, 131, 4)
    assert c.embed_multiplier == 3.0 and c.norm_weight_offset == 0.0 and c.is_hybrid and c.side_by_side
    assert c.layer_runs == [0, 1, 2, 1, 2, 3] and not any(c.enters_loop(r) for r in range(6))
    s = c.mixer_spec(0)
    assert isinstance(s, TwinSpec) and isinstance(s.left, HeadsSpec) and isinstance(s.right, GatedLinearSpec)
    a, g = s.left, s.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.pool, a.rot_dims, a.rot_base, a.rot_factor) == (
        6, 2, 24, 16, 21, 5, 16, 1e4, 3.0)
    assert a.bias and a.whole_norm and a.sink and a.head_temp and a.gated and not a.gate_each and a.out_scale == 0.9
    assert (g.heads, g.dim, g.vdim, g.tau, g.out_scale, g.col) == (3, 16, 24, 8.0, 0.6, a.in_width)
    assert [c.mixer_spec(i).right.rank for i in range(4)] == [16, 8, 5, 24]        # only the tensors tell
    assert c.ff_spec(1) is None and c.ff_spec(0).activation == "silu_glu" and c.ff_spec(0).ff == 40
    # every pass of the loop has its own keys, values and states; every run the inputs of its convolution
    assert c.cache_layers == {i: i for i in range(6)} and sorted(c.state_offsets) == list(range(6))
    parts = sorted([(at, c.mixer_spec(c.layer_runs[r]).right.state_floats) for r, at in c.state_offsets.items()]
                   + [(at, 3 * 96) for at in c.input_offsets.values()])
    assert all(a + n <= b for (a, n), (b, _) in zip(parts, parts[1:])) and sum(parts[-1]) <= c.state_floats
    assert c.pool_step == 5 and c.mean_rows(64) == 12 and c.cache_blocks(640, 4, 64) == 10 + 128 // 64 + 4
    assert c.first_seen(500) == min(500 + 1 - 70, 500 // 32 * 32, 500 // 17 * 17)
    again = ModelConfig.deserialize(c.serialize())
    assert again.mixer_spec(3) == c.mixer_spec(3) and again.loop == c.loop and again.input_conv == 4


def test_first_position_that_is_needed():
    s = HeadsSpec(1, 1, 8, 8, 1.0, window=9, pool=17)
    assert [s.first_seen(p) for p in (0, 8, 9, 40)] == [0, 0, 1, 32]
    # token 33 completes the second block; until then its tokens stay, though the window has left them
    assert [s.first_needed(p) for p in (33, 34, 50)] == [17, 26, 34]
    assert [s.blocks_seen(p) for p in (16, 24, 25, 41, 42)] == [0, 0, 1, 1, 2]


def test_bad_models_are_refused(small, tmp_path):
    def opened(name, change, drop=()):
        cfg = copy.deepcopy(small.cfg)
        change(cfg)
        write_model(tmp_path / name, cfg, {k: v for k, v in small.weights.items() if k not in drop})
        return open_model(str(tmp_path / name))

    layer = lambda i, **kw: lambda c: c["layers"][i].update(**kw)
    left = lambda i, **kw: lambda c: c["layers"][i]["mixer"]["left"].update(**kw)
    right = lambda i, **kw: lambda c: c["layers"][i]["mixer"]["right"].update(**kw)
    for n, (change, drop, what) in enumerate([
            (layer(0, type="something"), (), "something"),
            (layer(0, mlp={"kind": "sparse", "ff": 8}), (), "sparse"),
            (lambda c: None, ("l0.mix.left.sink",), "l0.mix.left.sink"),
            (lambda c: None, ("l3.canon1",), "l3.canon1"),
            (lambda c: None, ("l1.mix.right.a2.b",), "l1.mix.right.a2.b"),
            (left(0, kv_heads=4), (), "evenly"),
            (left(0, rot={"dims": 26, "base": 1e4}), (), "rotate"),
            (left(0, rot={"dims": 8, "base": 1e4, "scaling": {"factor": 0.0}}), (), "slower"),
            (left(0, mask={"pool": 4}), (), "window of 0"),
            (right(0, tau=0.0), (), "positive divisor"),
            (lambda c: c["canon"].update(taps=0), (), "tap"),
            (lambda c: c["loop"].update(stop=6), (), "cannot run")]):
        with pytest.raises(ValueError, match=what):
            opened(str(n), change, drop)


def test_converted_file_gives_the_same_logits(small, tmp_path):
    from zse_b200.format.convert import convert_hf_to_zse
    from zse_b200.format.loader import ZSELoader
    out = str(tmp_path / "m.zse")
    convert_hf_to_zse(small.path, out)
    with ZSELoader(out) as l:
        assert {e.dtype for e in l.weight_index} == {"bfloat16"} and l.config.mixer_spec(3).right.rank == 24
    r = TraceRunner(out, "float32", MAX_TOKENS, device="cpu")
    assert_close(small, replay(r, small, [[("c", LENGTHS["c"])]]), 1e-4)
    r.close()


def test_synthetic_models_open(tmp_path):
    from zse_b200.format import synth
    path = str(tmp_path / "s.zse")
    synth.write_random_model(path, synth.shape_config("tiny-vobisun"), seed=3)
    eng = cpu_engine(path)
    rid = eng.add_request_tokens(list(range(20)), max_tokens=4, temperature=0.0, stop_tokens=[])
    eng.run_until_done()
    assert len(eng.get_result(rid).output_tokens) == 4
    eng.destroy()


def test_other_dtypes_and_tensor_parallelism_are_refused(small):
    with pytest.raises(ValueError, match="float16"):
        cpu_engine(small.path, dtype="float16")
    with pytest.raises((NotImplementedError, ValueError)):
        cpu_engine(small.path, tp_size=2)


# ---- mechanisms -----------------------------------------------------------------------------------------------------
def test_memory_and_convolution_of_one_sequence_in_pieces():
    g = torch.Generator().manual_seed(5)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    T, H, d, v, taps = 90, 3, 6, 5, 4
    q, k, val, alpha = rnd(T, H, d), rnd(T, H, d), rnd(T, H, v), torch.rand(T, H, d, generator=g, dtype=F64)
    want = torch.stack([oracle.decayed_memory(q[:, h], k[:, h], val[:, h], alpha[:, h]) for h in range(H)], 1)
    S = torch.zeros(H, d, v, dtype=F64)
    cuts = ((0, 1), (1, 3), (3, 64), (64, 65), (65, 90))
    got = torch.cat([ref.gated_linear_tokens(q[a:e], k[a:e], val[a:e], torch.log(alpha[a:e]), S) for a, e in cuts])
    assert (got - want).abs().max() < 1e-12
    y, w = rnd(T, 7), rnd(7, taps)
    want, before, got = oracle.with_history(y, w), torch.zeros(taps - 1, 7, dtype=F64), []
    for a, e in cuts:
        z, before = ref.conv_inputs(y[a:e], before, w.T)
        got.append(z)
    assert (torch.cat(got) - want).abs().max() < 1e-12 and torch.equal(before, y[-3:])


def test_logarithms_of_the_decays():
    g = torch.Generator().manual_seed(1)
    u, w, b = 4 * torch.randn(20, 5, generator=g), torch.randn(12, 5, generator=g), torch.randn(12, generator=g)
    want = torch.log(oracle.sigmoid(u.to(F64) @ w.to(F64).T + b.to(F64)) ** (1 / 7.0))
    assert (ref.log_decays(u, w, b, 7.0).to(F64) - want).abs().max() < 1e-5
    assert torch.isfinite(ref.log_decays(1e4 * u, w, b, 7.0)).all()


@pytest.mark.parametrize("name", list(SPECS))
def test_attention_over_tokens_and_means(name):
    A = PooledAttention(TorchOps(), SPECS[name], torch.float32, "cpu", tokens=300, rows=130)
    s = A.spec
    if s.pool:
        for x, y in zip(A.means(1), (A.k[1], A.v[1])):
            assert (x - oracle.block_means(y, s.pool)).abs().max() < 1e-5
    seqs, pos = [0, 1, 2, 2, 1, 0, 0], [0, 1, s.window - 1, s.window, s.window + max(1, s.pool) - 1, 299, 200]
    want = torch.stack([A.plain(t, q, p) for t, (q, p) in enumerate(zip(seqs, pos))])
    assert (A.rows(seqs, pos) - want).abs().max() < 1e-5
    out, cu = A.chunks([(3, 5), (150, 125)], first=1)
    for i in (0, 1, 60, 124):
        assert (out[cu[1] + i] - A.plain(cu[1] + i, 1, 150 + i)).abs().max() < 1e-5


@pytest.mark.parametrize("name", ["window", "short-window", "single-tokens", "blocks-of-the-cache"])
def test_one_loud_key_inside_and_outside(name):
    s = SPECS[name]
    for pos in (s.window - 1, s.window + s.pool - 1, 447):
        for key in loud_places(s, pos):
            if key >= 500:
                continue
            A = PooledAttention(TorchOps(), s, torch.float32, "cpu", seqs=1, tokens=500, rows=1, seed=pos)
            quiet = A.plain(0, 0, pos)
            make_loud(A, key, s.heads - 1, 0)
            want = A.plain(0, 0, pos)
            assert (A.rows([0], [pos])[0] - want).abs().max() < 1e-4, (pos, key)
            seen = s.first_seen(pos) <= key <= pos or key < s.blocks_seen(pos) * s.pool
            moved = ((want - quiet).view(s.heads, -1)[-1].norm() / quiet.view(s.heads, -1)[-1].norm()).item()
            assert (moved > 0.3) == seen, (pos, key, moved)


# ---- means of blocks in the cache -----------------------------------------------------------------------------------------
def manager(small, blocks=40):
    with open_model(small.path) as l:
        c = l.config
    return KVCacheManager(c, torch.device("cpu"), block_size=64, num_blocks=blocks, dtype=torch.float32, state_slots=4)


def test_blocks_of_means_come_and_go(small):
    m = manager(small)                                       # a mean per 5 tokens: a block of the cache per 320 tokens
    free = m.num_free_blocks
    m.allocate_sequence(0, num_tokens=319)
    assert len(m.mean_block_ids(0)) == 1 and free - m.num_free_blocks == 6
    for n in range(6):                                       # token 325 is the last of the 65th block
        assert m.extend_batch([0]) == [None] and len(m.mean_block_ids(0)) == (2 if 320 + n >= 325 else 1)
    m.truncate_sequence(0, 324)
    assert len(m.mean_block_ids(0)) == 1
    m.extend_sequence(0, 400)
    assert len(m.mean_block_ids(0)) == 3
    ids = m.get_block_ids(0)                                 # tokens left the windows, their means stay
    assert ids[0] == -1 and all(b >= 0 for b in m.mean_block_ids(0))
    m.free_sequence(0)
    assert m.num_free_blocks == free


def test_a_fork_writes_its_own_means(small):
    m = manager(small)
    m.allocate_sequence(0, num_tokens=100)
    m.slab[:, m.mean_block_ids(0)[0]] = 7.0
    m.fork_sequence(0, 1)
    assert m.mean_block_ids(0) == m.mean_block_ids(1)
    m.extend_sequence(1, 4)                                  # no mean is completed: still shared
    assert m.mean_block_ids(0) == m.mean_block_ids(1)
    m.extend_sequence(1, 1)
    assert m.mean_block_ids(0) != m.mean_block_ids(1) and (m.slab[:, m.mean_block_ids(1)[0]] == 7.0).all()
    m.free_sequence(0)
    m.free_sequence(1)
    assert m.num_free_blocks == m.num_total_blocks


def test_the_pool_and_the_budget_count_the_means(small):
    m = manager(small, blocks=11)
    m.allocate_sequence(0, num_tokens=9 * 64)                # nine blocks of tokens, two of means
    assert m.num_free_blocks == 0
    m.free_sequence(0)
    with pytest.raises(RuntimeError, match="12 KV blocks"):
        m.allocate_sequence(1, num_tokens=10 * 64)
    assert MemoryBudget(100, 64, mean_step=5)._tokens_to_blocks(576) == 11
    assert MemoryBudget(100, 64)._tokens_to_blocks(576) == 9


def test_blocks_leave_with_the_window_and_their_means_stay(small):
    eng = cpu_engine(small.path, kv_blocks=12)
    cache, runner = eng.kv_cache, eng.runner
    first = eng.model_config.first_seen
    cache.allocate_sequence(0, num_tokens=40)
    toks = (small.tokens["a"] * 3)[:400]
    runner.prefill([(0, toks[:40], 0)])
    at = 40
    for n in [64, 30] + [1] * 90 + [2, 97, 20]:
        errs = cache.extend_batch([0]) if n == 1 else cache.extend_sequence(0, n)
        assert not errs or errs == [None]
        ids = cache.get_block_ids(0)
        assert [b < 0 for b in ids] == [i < first(at) // 64 for i in range(len(ids))]
        logits = runner.prefill([(0, toks[at: at + n], at)], want=[range(max(0, n - 20), n)], select=False)
        at += n
    want = oracle.forward(small.cfg, small.weights, toks[:at])[-20:].numpy()
    assert np.abs(logits.numpy() - want).max() < 5e-4 * want.std()
    cache.free_sequence(0)
    assert cache.num_free_blocks == cache.num_total_blocks
    eng.destroy()


# ---- through the engine and its scheduler ---------------------------------------------------------------------------
def run(eng, prompts, n=8, **kw):
    rids = [eng.add_request_tokens(p, max_tokens=n, temperature=0.0, stop_tokens=[], **kw) for p in prompts]
    eng.run_until_done()
    return [eng.get_result(r).output_tokens for r in rids]


@pytest.mark.parametrize("pipeline", [False, True])
def test_greedy_generation_matches_the_oracle(small, pipeline):
    eng = cpu_engine(small.path, prefill_chunk_size=32, pipeline_decode=pipeline)
    prompts = [small.tokens["a"][:75], small.tokens["b"][:5], small.tokens["c"], small.tokens["d"][:40]]
    assert run(eng, prompts) == [oracle.greedy(small.cfg, small.weights, p, 8) for p in prompts]
    assert not pipeline or eng._batch_runner.ahead_launches > 0
    eng.destroy()


def test_prompts_and_decoding_share_a_pass_without_changing_the_tokens(small):
    eng = cpu_engine(small.path, prefill_chunk_size=24, decode_per_prefill=0)
    alone = {r: run(eng, [small.tokens[r]], 10)[0] for r in "abd"}
    rids = {"b": eng.add_request_tokens(small.tokens["b"], max_tokens=10, temperature=0.0, stop_tokens=[])}
    for _ in range(5):
        eng.step()
    for r in "ad":
        rids[r] = eng.add_request_tokens(small.tokens[r], max_tokens=10, temperature=0.0, stop_tokens=[])
    eng.run_until_done()
    assert eng._batch_runner.mixed_passes > 0
    assert {r: eng.get_result(i).output_tokens for r, i in rids.items()} == alone
    eng.destroy()


def test_more_requests_than_state_slots_and_equal_prefixes(small):
    p = small.tokens["a"][:100]
    want = oracle.greedy(small.cfg, small.weights, p, 5)
    eng = cpu_engine(small.path, max_batch_seqs=2, enable_prefix_cache=True)
    assert run(eng, [p] * 5, 5) == [want] * 5
    assert eng.kv_cache.states.num_free == eng.kv_cache.states.slots
    eng.destroy()


def test_speculative_decoding_keeps_the_tokens(small):
    """Rejected drafts roll the recurrent state back, the convolution's inputs too; means that held them are written again."""
    loop = (small.tokens["c"] * 9)[:70]
    want = oracle.greedy(small.cfg, small.weights, loop, 10)
    eng = cpu_engine(small.path, speculative_k=3, speculative_mode="ngram")
    assert run(eng, [loop], 10) == [want]
    eng.destroy()


def test_sampling_and_embeddings_run(small):
    eng = cpu_engine(small.path)
    got = []
    for _ in range(2):
        rid = eng.add_request_tokens(small.tokens["c"], max_tokens=6, temperature=0.9, top_k=20, top_p=0.9, seed=7,
                                     repetition_penalty=1.2, stop_tokens=[])
        eng.run_until_done()
        got.append(eng.get_result(rid).output_tokens)
    assert got[0] == got[1] and len(got[0]) == 6
    e = eng.embed_tokens(small.tokens["b"])
    assert e.shape == (96,) and abs(float(e.norm()) - 1) < 1e-5
    logits = eng.last_token_logits(small.tokens["b"])
    assert np.abs(logits.numpy() - small.want["b"][-1]).max() < 1e-3 * np.abs(small.want["b"]).max()
    eng.destroy()
