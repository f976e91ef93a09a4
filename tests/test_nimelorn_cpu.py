"""Nimelorn on the CPU path: configuration, loaders, cache, recurrent state, batching and generation against the plain
oracle."""
import copy
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import nimelorn_oracle as oracle                                     # noqa: E402
from helpers.latent_oracle import write_model                                     # noqa: E402
from helpers.nimelorn_cases import CASES, Model                                   # noqa: E402
from helpers.ruralorn_cases import LENGTHS, MAX_TOKENS, SCHEDULES, assert_close, assert_near, replay, schedule  # noqa: E402

from zse_b200.cache.state_slots import StateSlots                                 # noqa: E402
from zse_b200.config import EngineConfig                                          # noqa: E402
from zse_b200.engine import ZStreamerEngine                                       # noqa: E402
from zse_b200.format.config import HeadsSpec, MatrixMemorySpec                    # noqa: E402
from zse_b200.trace import TraceRunner                                            # noqa: E402


@pytest.fixture(scope="module", autouse=True)
def few_threads():
    """The matrices are small: more threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    return Model(request.param, tmp_path_factory.mktemp("nimelorn") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("nimelorn-small"))


def cpu_engine(path, **kw):
    kw = dict(dict(device="cpu", dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=24, max_seq_len=512),
              **kw)
    return ZStreamerEngine(path, config=EngineConfig(**kw))


@pytest.mark.parametrize("name", SCHEDULES)
def test_schedules_match_the_oracle(model, name):
    r = TraceRunner(model.path, "float32", MAX_TOKENS, device="cpu")
    try:
        assert_close(model, replay(r, model, schedule(name)), 5e-4)
        assert r.engine.kv_cache.num_free_blocks == r.engine.kv_cache.num_total_blocks
        assert r.engine.kv_cache.states.num_free == 4
    finally:
        r.close()


def test_bfloat16_stays_near_the_oracle(small):
    r = TraceRunner(small.path, "bfloat16", MAX_TOKENS, device="cpu")
    assert_near(small, replay(r, small, schedule("mixed")))
    r.close()


def _set(path, value):
    def change(cfg):
        at = cfg
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value(at[path[-1]])
    return change


MISTAKES = {
    "chunk one longer": _set(("layers", 1, "mixer", "mask", "size"), lambda v: v + 1),
    "chunk one shorter": _set(("layers", 4, "mixer", "mask", "size"), lambda v: v - 1),
    "mask of the layer that has the keys": _set(("layers", 2, "mixer", "mask", "size"), lambda v: 21),
    "scale of the layer that has the keys": _set(("layers", 2, "mixer", "scale"), lambda v: 24 ** -0.5),
    "gate cap": _set(("layers", 3, "mixer", "gate_cap"), lambda v: 12.0),
    "hash of the token before": _set(("embedding", "bigram", "mul_prev"), lambda v: v + 1),
    "embedding scale": _set(("embedding", "scale"), lambda v: v * 1.2),
    "limit of the experts": _set(("layers", 1, "mlp", "expert", "limit"), lambda v: 0.8),
    "limit of the shared expert": _set(("layers", 1, "mlp", "shared", "limit"), lambda v: 1.2),
    "router's choice": _set(("layers", 1, "mlp", "router", "top"), lambda v: 1),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_the_models_of_these_tests_show_a_mistake(small, name):
    """The oracle with one constant changed leaves the limits of the tests above by far."""
    wrong = copy.deepcopy(small.cfg)
    MISTAKES[name](wrong)
    off = oracle.forward(wrong, small.weights, small.tokens["a"]).numpy()
    d = np.sqrt(((off - small.want["a"]) ** 2).mean(1)) / small.want["a"].std()
    assert np.quantile(d, 0.8) > 3e-3


def test_a_lost_state_and_a_lost_token_show(small):
    """Dropping what came before position 80 moves the logits after it, in a chunk's first positions too."""
    cut = 84                                  # a multiple of the first attention layer's chunk
    off = oracle.forward(small.cfg, small.weights, small.tokens["a"][cut:]).numpy()
    d = np.sqrt(((off - small.want["a"][cut:]) ** 2).mean(1)) / small.want["a"].std()
    assert d[:3].min() > 0.05 and d[:40].min() > 1e-2


def test_configuration(small):
    from zse_b200.format.config import ModelConfig
    from zse_b200.format.directory import open_model
    with open_model(small.path) as l:
        c = l.config
    assert (c.arch, c.num_layers, c.hidden_size, c.vocab_size) == ("nimelorn", 5, 96, 131)
    a, m = c.mixer_spec(2), c.mixer_spec(3)
    assert isinstance(a, HeadsSpec) and (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.kv_from) == (6, 2, 24, 16, 70, 1)
    assert isinstance(m, MatrixMemorySpec) and (m.heads, m.dim, m.vdim, m.gate_cap) == (2, 32, 40, 5.0)
    assert c.ff_spec(2) is None and c.ff_spec(0).ff == 40 and c.ff_spec(3).shared_ff == 0
    r = c.ff_spec(1)
    assert (r.top, r.scale, r.limit, r.shared_limit, r.normalise, r.weigh, r.router_rows) == (2, 1.7, 1.2, 0.8, True,
                                                                                             "output", 6)
    assert c.cache_layers == {1: 0, 4: 1} and c.num_cache_layers == 2 and c.kv_planes == 1
    assert c.state_offsets == {0: 0, 3: c.mixer_spec(0).state_floats} and c.keeps_state
    assert c.kv_pool_dims() == (1, max(c.mixer_spec(i).row for i in (1, 4)))
    # what some layer still sees: the smallest first position over chunks of 21, 70 and 64
    assert [c.first_seen(p) for p in (0, 20, 63, 64, 69, 70, 127, 128, 140)] == [0, 0, 0, 0, 0, 63, 64, 70, 126]
    again = ModelConfig.deserialize(c.serialize())
    assert again.mixer_spec(3) == m and again.ff_spec(1) == r and again.embed_design == c.embed_design


def test_bad_models_are_refused(small, tmp_path):
    from zse_b200.format.directory import open_model

    def opened(name, change, drop=()):
        cfg = copy.deepcopy(small.cfg)
        change(cfg)
        write_model(tmp_path / name, cfg, {k: v for k, v in small.weights.items() if k not in drop})
        return open_model(str(tmp_path / name))

    with pytest.raises(ValueError, match="something"):
        opened("a", lambda c: c["layers"][0].update(type="something"))
    with pytest.raises(ValueError, match="sparse"):
        opened("b", lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    with pytest.raises(ValueError, match="l3.mix.f.b"):
        opened("c", lambda c: None, drop=("l3.mix.f.b",))
    with pytest.raises(ValueError, match="no keys and values"):
        opened("d", lambda c: c["layers"][2]["mixer"].update(kv_from=0))
    with pytest.raises(ValueError, match="other sizes"):
        opened("e", lambda c: c["layers"][2]["mixer"].update(vdim=24))


def test_converted_file_gives_the_same_logits(small, tmp_path):
    from zse_b200.format.convert import convert_hf_to_zse
    from zse_b200.format.loader import ZSELoader
    out = str(tmp_path / "m.zse")
    convert_hf_to_zse(small.path, out)
    with ZSELoader(out) as l:
        assert {e.dtype for e in l.weight_index} == {"bfloat16"}
    r = TraceRunner(out, "float32", MAX_TOKENS, device="cpu")
    assert_close(small, replay(r, small, [[("c", LENGTHS["c"])]]), 1e-4)
    r.close()


def test_synthetic_models_open(tmp_path):
    from zse_b200.format import synth
    path = str(tmp_path / "s.zse")
    synth.write_random_model(path, synth.shape_config("tiny-nimelorn"), seed=3)
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
def test_memory_of_one_sequence_in_pieces():
    from zse_b200.ops import reference as ref
    g = torch.Generator().manual_seed(5)
    T, H, d, v = 90, 2, 6, 5
    q, k, x = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (d, d, v))
    i = 6 * torch.randn(T, H, generator=g, dtype=torch.float64)
    f = torch.nn.functional.logsigmoid(3 + 3 * torch.randn(T, H, generator=g, dtype=torch.float64))
    i[40:60] -= 12.0                          # the running maximum falls with the forget gates
    want = torch.stack([oracle.mlstm_recurrence(q[:, n], k[:, n], x[:, n], i[:, n], f[:, n]) for n in range(H)], 1)
    S, n, m = torch.zeros(H, d, v).double(), torch.zeros(H, d).double(), torch.zeros(H).double()
    got = torch.cat([ref.memory_tokens(q[a:e], k[a:e], x[a:e], i[a:e], f[a:e], S, n, m)
                     for a, e in ((0, 1), (1, 3), (3, 64), (64, 65), (65, 90))])
    assert (got - want).abs().max() < 1e-9 * want.abs().max()


def test_sinusoid_and_bigram_rows():
    from zse_b200.ops import reference as ref
    pos = torch.tensor([0, 1, 5, 1000, 40000])
    got = ref.sinusoid(pos, 9, 10000.0)
    want = torch.stack([oracle.sinusoid(6, 9)[p] if p < 6 else torch.tensor(
        [getattr(np, "cos" if j % 2 else "sin")(float(p) * 10000.0 ** (-(j - j % 2) / 9)) for j in range(9)])
        for p in pos.tolist()])
    assert (got - want).abs().max() < 1e-6
    ids, last = torch.tensor([4, 5, 6, 7, 8]), torch.tensor([0, 11, 12, 13], dtype=torch.int32)
    prev = ref.previous_tokens(ids, [0, 2, 3, 5], torch.tensor([[3, -1, 1], [0, 0, 0]]), last)
    assert prev.tolist() == [13, 4, -1, 11, 7]


def test_state_slots():
    s = StateSlots(2, 8, "cpu")
    s.allocate(7)
    r0, w0 = s.advance(7, 0, 5)
    assert r0 == -1 and w0 in (0, 1) and s.position(7) == 5
    r1, w1 = s.advance(7, 5, 1)
    assert (r1, w1) == (w0, 1 - w0)
    assert s.advance(7, 5, 3) == (r1, w1) and s.position(7) == 8      # the same pass again, longer
    assert s.advance(7, 8, 1) == (w1, r1)
    with pytest.raises(RuntimeError, match="not held"):
        s.advance(7, 5, 1)
    assert s.advance(7, 0, 2)[0] == -1                               # from the start: nothing is read
    s.allocate(8)
    with pytest.raises(RuntimeError, match="no state slot"):
        s.allocate(9)
    s.free(8)
    s.rows[s.advance(7, 2, 1)[1]] = 3.0
    s.last_token[:] = torch.tensor([1, 2, 3, 4], dtype=torch.int32)
    s.fork(7, 9)
    a, b = s.advance(7, 3, 1), s.advance(9, 3, 1)
    assert a != b and torch.equal(s.rows[a[0]], s.rows[b[0]]) and int(s.last_token[a[0]]) == int(s.last_token[b[0]])
    s.free(7)
    s.free(9)
    assert s.num_free == 2


def test_blocks_leave_with_the_chunk(small):
    """A growing sequence holds the blocks that some layer's chunk reaches, and no others."""
    eng = cpu_engine(small.path)
    cache, runner = eng.kv_cache, eng.runner
    first = eng.model_config.first_seen
    cache.allocate_sequence(0, num_tokens=40)
    runner.prefill([(0, small.tokens["a"][:40], 0)])
    at = 40
    for n in [64, 30] + [1] * 90 + [2, 17]:
        errs = cache.extend_batch([0]) if n == 1 else cache.extend_sequence(0, n)
        assert not errs or errs == [None]
        ids = cache.get_block_ids(0)
        assert all(b >= 0 for b in ids[first(at) // 64:]) and all(b < 0 for b in ids[: first(at) // 64])
        at += n
    cache.free_sequence(0)
    assert cache.num_free_blocks == cache.num_total_blocks and cache.states.num_free == cache.states.slots
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


def test_a_step_launched_ahead_and_dropped_leaves_the_state_alone(small):
    """Requests that arrive while others decode make the engine drop the step it launched ahead and take it again."""
    eng = cpu_engine(small.path, pipeline_decode=True, prefill_chunk_size=16, decode_per_prefill=0)
    first = eng.add_request_tokens(small.tokens["d"][:30], max_tokens=14, temperature=0.0, stop_tokens=[])
    for _ in range(6):
        eng.step()
    late = [eng.add_request_tokens(small.tokens[r][:20], max_tokens=6, temperature=0.0, stop_tokens=[]) for r in "ab"]
    eng.run_until_done()
    assert eng._batch_runner.ahead_dropped > 0
    assert eng.get_result(first).output_tokens == oracle.greedy(small.cfg, small.weights, small.tokens["d"][:30], 14)
    for r, rid in zip("ab", late):
        assert eng.get_result(rid).output_tokens == oracle.greedy(small.cfg, small.weights, small.tokens[r][:20], 6)
    eng.destroy()


def test_prompts_and_decoding_share_a_pass_without_changing_the_tokens(small):
    eng = cpu_engine(small.path, prefill_chunk_size=24, decode_per_prefill=0)
    alone = {r: run(eng, [small.tokens[r]], 12)[0] for r in "abd"}
    rids = {"b": eng.add_request_tokens(small.tokens["b"], max_tokens=12, temperature=0.0, stop_tokens=[])}
    for _ in range(5):
        eng.step()
    for r in "ad":
        rids[r] = eng.add_request_tokens(small.tokens[r], max_tokens=12, temperature=0.0, stop_tokens=[])
    eng.run_until_done()
    assert eng._batch_runner.mixed_passes > 0
    assert {r: eng.get_result(i).output_tokens for r, i in rids.items()} == alone
    eng.destroy()


def test_more_requests_than_state_slots_and_equal_prefixes(small):
    """Slots and blocks are used again; equal prompts share nothing that the recurrent state would need."""
    p = small.tokens["a"][:100]
    want = oracle.greedy(small.cfg, small.weights, p, 6)
    eng = cpu_engine(small.path, max_batch_seqs=2, enable_prefix_cache=True)
    assert run(eng, [p] * 5, 6) == [want] * 5
    assert eng.kv_cache.states.num_free == eng.kv_cache.states.slots
    eng.destroy()


@pytest.mark.parametrize("mode", ["ngram", "self"])
def test_speculative_decoding_keeps_the_tokens(small, mode):
    """Rejected drafts roll the recurrent state back."""
    loop = (small.tokens["c"] * 9)[:70]
    want = oracle.greedy(small.cfg, small.weights, loop, 12)
    eng = cpu_engine(small.path, speculative_k=3, speculative_mode=mode)
    assert run(eng, [loop], 12) == [want]
    eng.destroy()


def test_preempted_requests_start_over(small):
    """A request that loses its blocks and its state slot and runs again gives the same tokens."""
    p = small.tokens["d"][:60]
    want = oracle.greedy(small.cfg, small.weights, p, 10)
    eng = cpu_engine(small.path)
    rid = eng.add_request_tokens(p, max_tokens=10, temperature=0.0, stop_tokens=[])
    for _ in range(4):
        eng.step()
    sched = eng.scheduler
    r = sched.active_requests()[0]
    assert r.num_generated > 0
    eng._batch_runner._drop_inflight()
    eng._batch_runner._release_kv(r)
    r.mark_preempted()
    r.prefill_offset = 0
    sched._budget.release(r.request_id)
    del sched._active[r.request_id]
    sched._queue.add_preempted(r)
    eng.run_until_done()
    assert eng.get_result(rid).output_tokens == want
    eng.destroy()


def test_sampling_and_embeddings_run(small):
    eng = cpu_engine(small.path)
    got = []
    for _ in range(2):
        rid = eng.add_request_tokens(small.tokens["c"], max_tokens=8, temperature=0.9, top_k=20, top_p=0.9, seed=7,
                                     repetition_penalty=1.2, stop_tokens=[])
        eng.run_until_done()
        got.append(eng.get_result(rid).output_tokens)
    assert got[0] == got[1] and len(got[0]) == 8
    e = eng.embed_tokens(small.tokens["b"])
    assert e.shape == (96,) and abs(float(e.norm()) - 1) < 1e-5
    logits = eng.last_token_logits(small.tokens["b"])
    assert np.abs(logits.numpy() - small.want["b"][-1]).max() < 1e-3 * np.abs(small.want["b"]).max()
    eng.destroy()
