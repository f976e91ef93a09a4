"""Ruralorn on the CPU path: configuration, loaders, cache, batching and generation against the plain oracle."""
import json
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from helpers import latent_oracle as oracle                                       # noqa: E402
from helpers.ruralorn_cases import (CASES, LENGTHS, MAX_TOKENS, SCHEDULES, Model, assert_close,  # noqa: E402
                                    assert_near, replay, schedule)

from zse_b200.config import EngineConfig                                          # noqa: E402
from zse_b200.engine import ZStreamerEngine                                       # noqa: E402
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
    return Model(request.param, tmp_path_factory.mktemp("ruralorn") / request.param)


@pytest.fixture(scope="module")
def small(tmp_path_factory):
    return Model("layers-differ", tmp_path_factory.mktemp("ruralorn-small"))


def cpu_engine(path, **kw):
    kw = dict(dict(device="cpu", dtype="float32", max_batch_seqs=4, max_batch_tokens=128, kv_blocks=24, max_seq_len=512),
              **kw)
    return ZStreamerEngine(path, config=EngineConfig(**kw))


@pytest.mark.parametrize("name", SCHEDULES)
def test_schedules_match_the_oracle(model, name):
    r = TraceRunner(model.path, "float32", MAX_TOKENS, device="cpu")
    try:
        assert_close(model, replay(r, model, schedule(name)), 1e-4)
        assert r.engine.kv_cache.num_free_blocks == r.engine.kv_cache.num_total_blocks
    finally:
        r.close()


def test_bfloat16_stays_near_the_oracle(small):
    r = TraceRunner(small.path, "bfloat16", MAX_TOKENS, device="cpu")
    assert_near(small, replay(r, small, schedule("mixed")))
    r.close()


def test_one_key_at_the_windows_edge_moves_the_logits(small):
    """The models of these tests show a window that is one token off: the oracle itself, with a wrong window."""
    wrong = json.loads(json.dumps(small.cfg))
    for L in wrong["layers"]:
        L["mixer"]["mask"]["size"] += 1
    toks = small.tokens["a"]
    off = oracle.forward(wrong, small.weights, toks).numpy()
    d = np.sqrt(((off - small.want["a"]) ** 2).mean(1)) / small.want["a"].std()
    assert np.median(d[30:]) > 1e-2


def test_configuration(small):
    from zse_b200.format.directory import open_model
    with open_model(small.path) as l:
        c = l.config
        assert (c.arch, c.num_layers, c.hidden_size, c.vocab_size) == ("ruralorn", 3, 96, 131)
        s = c.latent_spec(1)
        assert (s.heads, s.dim, s.rot_dim, s.vdim, s.kv_rank, s.window, s.rot_base) == (5, 8, 16, 8, 24, 70, 1e4)
        assert c.moe_spec(1) is None and c.moe_spec(2).shared_ff == 0 and c.moe_spec(0).top == 2
        assert c.cache_window == 70 and c.kv_planes == 1
        assert c.kv_pool_dims() == (1, max(c.latent_spec(i).row for i in range(3)))
        assert s.row % 8 == 0 and s.latent_col % 8 == 0 and s.gate_col % 8 == 0
    # survives the .zse configuration section
    from zse_b200.format.config import ModelConfig
    again = ModelConfig.deserialize(c.serialize())
    assert again.latent_spec(1) == s and again.moe_spec(0) == c.moe_spec(0) and again.logit_scale == c.logit_scale


def test_unknown_mixers_and_missing_tensors_are_refused(small, tmp_path):
    from zse_b200.format.directory import open_model
    cfg = json.loads(json.dumps(small.cfg))
    cfg["layers"][1]["type"] = "something_else"
    oracle.write_model(tmp_path / "a", cfg, small.weights)
    with pytest.raises(ValueError, match="something_else"):
        open_model(str(tmp_path / "a"))
    w = dict(small.weights)
    del w["l2.mix.uv"]
    oracle.write_model(tmp_path / "b", small.cfg, w)
    with pytest.raises(ValueError, match="l2.mix.uv"):
        open_model(str(tmp_path / "b"))


def test_converted_file_gives_the_same_logits(small, tmp_path):
    from zse_b200.format.convert import convert_hf_to_zse
    from zse_b200.format.loader import ZSELoader
    out = str(tmp_path / "m.zse")
    convert_hf_to_zse(small.path, out)
    with ZSELoader(out) as l:
        assert {e.dtype for e in l.weight_index} == {"bfloat16"}
        e = l.weight_index.find("l0.mix.uk")
        assert np.array_equal(l.get_weight_as_float(e), small.weights["l0.mix.uk"].float().numpy())
    r = TraceRunner(out, "float32", MAX_TOKENS, device="cpu")
    assert_close(small, replay(r, small, [[("c", LENGTHS["c"])]]), 1e-4)
    r.close()


def test_other_dtypes_and_tensor_parallelism_are_refused(small):
    with pytest.raises(ValueError, match="float16"):
        cpu_engine(small.path, dtype="float16")
    with pytest.raises((NotImplementedError, ValueError)):
        cpu_engine(small.path, tp_size=2)


# ---- through the engine and its scheduler ---------------------------------------------------------------------------
def test_greedy_generation_matches_the_oracle(small):
    eng = cpu_engine(small.path, prefill_chunk_size=32)
    prompts = [small.tokens["a"][:75], small.tokens["b"][:5], small.tokens["c"], small.tokens["d"][:40]]
    rids = [eng.add_request_tokens(p, max_tokens=8, temperature=0.0, stop_tokens=[]) for p in prompts]
    eng.run_until_done()
    for p, rid in zip(prompts, rids):
        assert eng.get_result(rid).output_tokens == oracle.greedy(small.cfg, small.weights, p, 8)
    eng.destroy()


def test_prompts_and_decoding_share_a_pass_without_changing_the_tokens(small):
    alone = {}
    eng = cpu_engine(small.path, prefill_chunk_size=24, decode_per_prefill=0)
    for r in "abd":
        rid = eng.add_request_tokens(small.tokens[r], max_tokens=12, temperature=0.0, stop_tokens=[])
        eng.run_until_done()
        alone[r] = eng.get_result(rid).output_tokens
    rids = {"b": eng.add_request_tokens(small.tokens["b"], max_tokens=12, temperature=0.0, stop_tokens=[])}
    for _ in range(5):
        eng.step()
    for r in "ad":
        rids[r] = eng.add_request_tokens(small.tokens[r], max_tokens=12, temperature=0.0, stop_tokens=[])
    eng.run_until_done()
    assert eng._batch_runner.mixed_passes > 0
    assert {r: eng.get_result(i).output_tokens for r, i in rids.items()} == alone
    eng.destroy()


def test_prefix_cache_and_speculative_decoding_keep_the_tokens(small):
    p = small.tokens["a"][:100]
    want = oracle.greedy(small.cfg, small.weights, p, 10)
    eng = cpu_engine(small.path)
    for _ in range(2):                     # the second run starts from the first one's blocks, if they are still there
        a = eng.add_request_tokens(p, max_tokens=10, temperature=0.0, stop_tokens=[])
        b = eng.add_request_tokens(p, max_tokens=10, temperature=0.0, stop_tokens=[])
        eng.run_until_done()
        assert eng.get_result(a).output_tokens == want and eng.get_result(b).output_tokens == want
    eng.destroy()
    eng = cpu_engine(small.path, speculative_k=3, speculative_mode="ngram")
    a = eng.add_request_tokens(p, max_tokens=10, temperature=0.0, stop_tokens=[])
    eng.run_until_done()
    assert eng.get_result(a).output_tokens == want
    eng.destroy()


def test_sampling_and_penalties_run(small):
    eng = cpu_engine(small.path)
    got = []
    for _ in range(2):
        rid = eng.add_request_tokens(small.tokens["c"], max_tokens=8, temperature=0.9, top_k=20, top_p=0.9, seed=7,
                                     repetition_penalty=1.2, stop_tokens=[])
        eng.run_until_done()
        got.append(eng.get_result(rid).output_tokens)
    assert got[0] == got[1] and len(got[0]) == 8
    eng.destroy()


def test_blocks_leave_with_the_window(small):
    """While a sequence grows it holds the blocks its widest window reaches, and no others."""
    eng = cpu_engine(small.path)
    cache, runner = eng.kv_cache, eng.runner
    cache.allocate_sequence(0, num_tokens=40)
    runner.prefill([(0, small.tokens["a"][:40], 0)])
    at = 40
    for n in (64, 30, 2, 1, 1, 90, 17):
        cache.extend_sequence(0, n)
        ids = cache.get_block_ids(0)
        first_seen = max(0, at + 1 - 70)
        assert all(b >= 0 for b in ids[first_seen // 64:])
        assert all(b < 0 for b in ids[: first_seen // 64])
        at += n
    cache.free_sequence(0)
    assert cache.num_free_blocks == cache.num_total_blocks
    eng.destroy()


def test_trace_program_and_subcommand(small, tmp_path):
    import subprocess
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    lines = "\n".join(json.dumps(s) for s in (
        {"step": 0, "entries": [{"id": "x", "tokens": small.tokens["c"][:4], "want": [1, 3]}], "end": []},
        {"step": 1, "entries": [{"id": "x", "tokens": small.tokens["c"][4:6], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "x", "tokens": small.tokens["c"][6:], "want": [2, 0]}], "end": ["x"]}))
    for i, cmd in enumerate(([os.path.join(root, "bin", "trace_run")],
                             [sys.executable, os.path.join(root, "zse"), "trace-run"])):
        out = tmp_path / str(i)
        out.mkdir()
        p = subprocess.run(cmd + ["--model", small.path, "--dtype", "float32", "--out", str(out), "--max-tokens", "64",
                                  "--device", "cpu"], input=lines + "\n", text=True, capture_output=True, timeout=300)
        assert p.returncode == 0, p.stderr
        assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
        got = np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1)
        assert np.abs(got - small.want["c"][[8, 6]]).max() < 1e-3
