"""Movinex on the CPU path: configuration, loaders, cache, recurrent state, loops, batching and generation against the plain
oracle."""
import copy
import math
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import movinex_oracle as oracle                                      # noqa: E402
from helpers.latent_oracle import write_model                                     # noqa: E402
from helpers.movinex_cases import CASES, Model                                    # noqa: E402
from helpers.ruralorn_cases import LENGTHS, MAX_TOKENS, SCHEDULES, assert_close, assert_near, replay, schedule  # noqa: E402

from zse_b200.config import EngineConfig                                          # noqa: E402
from zse_b200.engine import ZStreamerEngine                                       # noqa: E402
from zse_b200.format.config import HeadsSpec, ModelConfig, MoESpec, StateSpaceSpec  # noqa: E402
from zse_b200.format.directory import open_model                                  # noqa: E402
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
    return Model(request.param, tmp_path_factory.mktemp("movinex") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("movinex-small"))


def cpu_engine(path, **kw):
    kw = dict(dict(device="cpu", dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=24, max_seq_len=512),
              **kw)
    return ZStreamerEngine(path, config=EngineConfig(**kw))


@pytest.mark.parametrize("name", [s for s in SCHEDULES if s != "portions-2"])
def test_schedules_match_the_oracle(model, name):
    r = TraceRunner(model.path, "float32", MAX_TOKENS, device="cpu")
    try:
        assert_close(model, replay(r, model, schedule(name)), 5e-4)
        cache = r.engine.kv_cache
        assert cache.num_free_blocks == cache.num_total_blocks and (cache.states is None or cache.states.num_free == 4)
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


def _set(path, value):
    def change(cfg):
        at = cfg
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value(at[path[-1]])
    return change


MISTAKES = {
    "window one longer": _set(("layers", 1, "mixer", "mask", "size"), lambda v: v + 1),
    "window one shorter": _set(("layers", 1, "mixer", "mask", "size"), lambda v: v - 1),
    "one kept token more": _set(("layers", 1, "mixer", "mask", "keep_first"), lambda v: v + 1),
    "one kept token less": _set(("layers", 1, "mixer", "mask", "keep_first"), lambda v: v - 1),
    "soft cap": _set(("layers", 1, "mixer", "softcap"), lambda v: v * 1.3),
    "rotated dimensions": _set(("layers", 1, "mixer", "rot", "dims"), lambda v: v + 4),
    "base of the rotation": _set(("layers", 4, "mixer", "rot", "base"), lambda v: 1e4),
    "step of the temperature": _set(("layers", 3, "mixer", "q_temp", "every"), lambda v: v + 1),
    "temperature": _set(("layers", 3, "mixer", "q_temp", "coef"), lambda v: 0.0),
    "scale": _set(("layers", 3, "mixer", "scale"), lambda v: v * 1.1),
    "passes of the loop": _set(("loop", "times"), lambda v: v + 1),
    "end of the loop": _set(("loop", "stop"), lambda v: v - 1),
    "parts of the norm": _set(("layers", 0, "mixer", "norm_groups"), lambda v: 1),
    "best groups of experts": _set(("layers", 2, "mlp", "router", "groups", "keep"), lambda v: v - 1),
    "experts": _set(("layers", 1, "mlp", "router", "top"), lambda v: v - 1),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_the_models_of_these_tests_show_a_mistake(small, name):
    """The oracle with one constant changed leaves the limits of the tests above by far, at some positions at least."""
    wrong = copy.deepcopy(small.cfg)
    MISTAKES[name](wrong)
    off = oracle.forward(wrong, small.weights, small.tokens["a"]).numpy()
    d = np.sqrt(((off - small.want["a"]) ** 2).mean(1)) / small.want["a"].std()
    assert np.quantile(d, 0.85) > 3e-3


def test_a_lost_state_shows(small):
    """Without what came before position 84 the logits after it move, also beyond every window."""
    off = oracle.forward(small.cfg, small.weights, small.tokens["a"][84:]).numpy()
    d = np.sqrt(((off - small.want["a"][84:]) ** 2).mean(1)) / small.want["a"].std()
    assert d[:3].min() > 0.05 and d[:60].min() > 1e-2


def test_configuration(small):
    with open_model(small.path) as l:
        c = l.config
    assert (c.arch, c.num_layers, c.hidden_size, c.vocab_size, c.logit_scale) == ("movinex", 5, 96, 131, 0.7)
    assert c.norm_weight_offset == 1.0 and not c.norms_outputs and c.is_hybrid
    assert c.layer_runs == [0, 1, 2, 3, 1, 2, 3, 4] and [r for r in range(8) if c.enters_loop(r)] == [1, 4]
    m, w, a = (c.mixer_spec(i) for i in (0, 1, 3))
    assert isinstance(m, StateSpaceSpec) and (m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups) == (6, 16, 24, 2, 3, 3)
    assert isinstance(w, HeadsSpec) and (w.heads, w.kv_heads, w.dim, w.vdim) == (6, 2, 24, 24)
    assert (w.window, w.keep_first, w.softcap, w.rot_dims, w.rot_base, w.k_as_v, w.gate_each, w.bias) == (
        21, 5, 6.0, 16, 1e4, True, True, False)
    assert (a.bias, a.gated, a.k_as_v, a.window, a.rot_dims, a.temp_coef, a.temp_every, a.learned_norm) == (
        True, False, False, 0, 0, 0.4, 7, False)
    assert c.ff_spec(3) is None and c.ff_spec(0).activation == "gelu_tanh_glu" and c.ff_spec(0).gated
    r = c.ff_spec(2)
    assert isinstance(r, MoESpec) and (r.experts, r.top, r.ff, r.groups, r.keep_groups, r.score, r.weigh, r.normalise,
                                       r.activation) == (8, 3, 16, 4, 3, "sigmoid", "output", False, "silu_glu")
    # every pass of the loop has its own keys, values and states
    assert c.cache_layers == {1: 0, 3: 1, 4: 2, 6: 3, 7: 4} and c.num_cache_layers == 5
    assert sorted(c.state_offsets) == [0, 2, 5] and c.state_floats == c.state_offsets[5] + c.mixer_spec(2).state_floats
    assert c.first_seen(500) == 0 and c.kept_first == 70
    again = ModelConfig.deserialize(c.serialize())
    assert again.mixer_spec(1) == w and again.ff_spec(2) == r and again.loop == c.loop and again.layer_runs == c.layer_runs


def test_bad_models_are_refused(small, tmp_path):
    def opened(name, change, drop=()):
        cfg = copy.deepcopy(small.cfg)
        change(cfg)
        write_model(tmp_path / name, cfg, {k: v for k, v in small.weights.items() if k not in drop})
        return open_model(str(tmp_path / name))

    layer = lambda i, **kw: lambda c: c["layers"][i].update(**kw)
    mixer = lambda i, **kw: lambda c: c["layers"][i]["mixer"].update(**kw)
    for n, (change, drop, what) in enumerate([
            (layer(0, type="something"), (), "something"),
            (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), (), "sparse"),
            (lambda c: None, ("l0.mix.dt_bias",), "l0.mix.dt_bias"),
            (lambda c: None, ("l4.ls2",), "l4.ls2"),
            (lambda c: None, ("loop.in",), "loop.in"),
            (mixer(0, groups=4), (), "equal groups"),
            (mixer(0, norm_groups=7), (), "equal parts"),
            (mixer(1, vdim=16), (), "have their width"),
            (mixer(1, kv_heads=4), (), "evenly"),
            (mixer(1, rot={"dims": 26, "base": 1e4}), (), "rotate"),
            (lambda c: c["loop"].update(stop=6), (), "cannot run"),
            (lambda c: c["layers"][2]["mlp"]["router"].update(groups={"count": 3, "keep": 1}), (), "equal groups"),
            (lambda c: c["layers"][2]["mlp"]["router"].update(groups={"count": 4, "keep": 1}), (), "cannot come from")]):
        with pytest.raises(ValueError, match=what):
            opened(str(n), change, drop)


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
    synth.write_random_model(path, synth.shape_config("tiny-movinex"), seed=3)
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
def test_state_space_and_convolution_of_one_sequence_in_pieces():
    from zse_b200.ops import reference as ref
    g = torch.Generator().manual_seed(5)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    T, H, G, n, v, taps = 90, 4, 2, 6, 5, 4
    x, B, C, dt = rnd(T, H, v), rnd(T, G, n), rnd(T, G, n), torch.rand(T, H, generator=g, dtype=F64)
    A_log, D = rnd(H), rnd(H)
    want = torch.stack([oracle.state_space(x[:, h], B[:, h // 2], C[:, h // 2], dt[:, h], A_log[h], D[h]) for h in range(H)], 1)
    S = torch.zeros(H, n, v, dtype=F64)
    cuts = ((0, 1), (1, 3), (3, 64), (64, 65), (65, 90))
    got = torch.cat([ref.state_space_tokens(x[a:e], B[a:e], C[a:e], dt[a:e], -torch.exp(A_log), D, S) for a, e in cuts])
    assert (got - want).abs().max() < 1e-12
    y, w, b = rnd(T, 7), rnd(7, taps), rnd(7)
    want, before, got = oracle.silu(oracle.causal_conv(y, w, b)), torch.zeros(taps - 1, 7, dtype=F64), []
    for a, e in cuts:
        z, before = ref.conv_tokens(y[a:e], before, w.T, b)
        got.append(z)
    assert (torch.cat(got) - want).abs().max() < 1e-12 and torch.equal(before, y[-3:])


def test_temperature_and_rotation():
    from zse_b200.ops import reference as ref
    T = 300
    for coef, every in ((0.4, 11), (-0.3, 1), (1.0, 400)):
        got = ref.query_temperature(torch.arange(T), coef, every).double()
        assert (got - oracle.query_factor(T, coef, every)).abs().max() < 1e-6
    x = torch.randn(T, 3, 12, dtype=F64)
    f = 7e3 ** (-torch.arange(0, 8, 2, dtype=F64) / 8)
    ang = torch.arange(T, dtype=F64)
    assert (ref.rotate_pairs(x.float(), ang, f).double() - oracle.turn_pairs(x, 8, 7e3)).abs().max() < 1e-4


def test_choice_of_experts():
    from zse_b200.ops import reference as ref
    g = torch.Generator().manual_seed(2)
    for experts, top, groups, keep in ((15, 3, 5, 2), (8, 4, 2, 1), (9, 3, 9, 4), (10, 3, 1, 1), (6, 2, 3, 3)):
        m = MoESpec(experts, top, 8, activation="silu_glu", weigh="output", groups=groups, keep_groups=keep)
        z = torch.randn(200, experts, generator=g)
        z[:50] = z[:50].round().abs()                  # ties
        ids, w = ref.route(z, m)
        s = torch.sigmoid(z)
        for t in range(200):
            assert ids[t].tolist() == oracle.choose(s[t], top, groups, keep)
            assert torch.equal(w[t], s[t][ids[t]])


def test_gated_activations():
    from zse_b200.ops import reference as ref
    g, u = torch.randn(50, dtype=F64), torch.randn(50, dtype=F64)
    for kind, act in (("silu_glu", lambda z: z / (1 + math.e ** -z)), ("gelu_tanh_glu", oracle.gelu_tanh)):
        assert (ref.glu(kind, g, u) - act(g) * u).abs().max() < 1e-12


def test_blocks_leave_with_the_window_but_not_those_of_the_kept_tokens(tmp_path):
    m = Model("windows-only", tmp_path / "w")
    eng = cpu_engine(m.path)
    cache, runner = eng.kv_cache, eng.runner
    first, kept = eng.model_config.first_seen, (eng.model_config.kept_first + 63) // 64
    assert eng.model_config.kept_first == 66 and cache.states is None
    cache.allocate_sequence(0, num_tokens=40)
    toks = (m.tokens["a"] * 3)[:400]
    runner.prefill([(0, toks[:40], 0)])
    at = 40
    for n in [64, 30] + [1] * 90 + [2, 97, 20]:
        errs = cache.extend_batch([0]) if n == 1 else cache.extend_sequence(0, n)
        assert not errs or errs == [None]
        ids = cache.get_block_ids(0)
        assert all(b >= 0 for i, b in enumerate(ids) if i < kept or i >= first(at) // 64)
        assert all(b < 0 for b in ids[kept: first(at) // 64])
        logits = runner.prefill([(0, toks[at: at + n], at)], want=[range(max(0, n - 20), n)], select=False)
        at += n
    assert -1 in ids
    want = oracle.forward(m.cfg, m.weights, toks[:at])[-20:].numpy()
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
    """Rejected drafts roll the recurrent state back, the convolution's inputs too."""
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
