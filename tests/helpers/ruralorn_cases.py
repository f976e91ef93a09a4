"""Small Ruralorn models and the checks that the CPU and the GPU tests share: schedules of a trace against the oracle."""
import random

import numpy as np
import torch

from . import latent_oracle as oracle
from .latent_oracle import config, mixer, moe

CASES = {
    # layers that differ in everything; one without a feed-forward, one without a shared expert; windows around a block
    "layers-differ": config(96, 131, [(mixer(3, 16, 8, 24, 40, 21), moe(5, 2, 24, 32)),
                                      (mixer(5, 8, 16, 8, 24, 70, base=1e4), None),
                                      (mixer(2, 24, 8, 16, 64, 9), moe(3, 3, 40))]),
    # nothing is a multiple of 8: the general kernels
    "odd-sizes": config(50, 77, [(mixer(3, 10, 6, 7, 18, 13), moe(4, 1, 9, 11)), (mixer(1, 5, 2, 3, 30, 100), moe(2, 1, 6))],
                        embed_scale=1.0, softcap=9.0),
    # more heads than one group of 16, a latent wider than 128, a part of the rotated dimensions that does not turn, a
    # window of the token alone, window sizes of exactly a block and a block and one
    "many-heads": config(128, 200, [(mixer(20, 32, 16, 48, 144, 65), moe(20, 4, 32, 16)),
                                    (mixer(17, 16, 16, 16, 272, 1, rot_dims=8), moe(6, 1, 16)),
                                    (mixer(33, 8, 8, 8, 136, 64), moe(9, 8, 8))], eps=1e-6),
}
LENGTHS = {"a": 150, "b": 61, "c": 9, "d": 97}


class Model:
    """A case on disk with its oracle logits; ``tokens[r]`` / ``want[r]`` per request."""

    def __init__(self, name, folder, seed=1):
        self.cfg = CASES[name]
        self.weights = oracle.random_weights(self.cfg, seed)
        self.path = oracle.write_model(folder, self.cfg, self.weights)
        rng = random.Random(seed)
        self.tokens = {r: [rng.randrange(self.cfg["vocab"]) for _ in range(n)] for r, n in LENGTHS.items()}
        with torch.no_grad():
            self.want = {r: oracle.forward(self.cfg, self.weights, t).numpy() for r, t in self.tokens.items()}


def blocks_of(tokens):
    return (tokens + 63) // 64 * 64


def replay(runner, model, steps):
    """Runs ``steps`` (lists of (request, tokens)) with every logits row asked for; requests end with their last token.
    A request may run several times: ``a#2`` is ``a`` once more.  Returns {request: logits [T, vocab]}."""
    at, got = {}, {}
    for step in steps:
        entries, end = [], []
        for rid, n in step:
            toks = model.tokens[rid.split("#")[0]]
            lo = at.get(rid, 0)
            at[rid] = lo + n
            entries.append({"id": rid, "tokens": toks[lo: lo + n], "want": list(range(n))})
            if lo + n == len(toks):
                end.append(rid)
        rows = runner.step(entries, end)
        k = 0
        for rid, n in step:
            got.setdefault(rid, []).append(rows[k: k + n])
            k += n
    return {r: np.concatenate(v) for r, v in got.items()}


def errors(model, got):
    """Per request: difference of the logits at every position, root mean square over the vocabulary, relative to the
    spread of the logits."""
    out = {}
    for rid, rows in got.items():
        want = model.want[rid.split("#")[0]]
        assert rows.shape == want.shape, (rid, rows.shape, want.shape)
        out[rid] = np.sqrt(((rows - want) ** 2).mean(1)) / want.std()
    return out


def assert_close(model, got, limit):
    for rid, e in errors(model, got).items():
        worst = int(e.argmax())
        assert e.max() <= limit, f"request {rid}: {e.max():.2e} at position {worst}, first over the limit at " \
                                 f"{int(np.argmax(e > limit))}"


def assert_near(model, got, typical=0.05, most=0.3, share=0.85):
    """For 16-bit activations: nearly every position is close.  A few may be far, where rounding decides between two
    experts whose scores are almost equal."""
    e = np.concatenate(list(errors(model, got).values()))
    assert np.median(e) <= typical and (e <= most).mean() >= share, \
        f"median {np.median(e):.3f}, {100 * (e <= most).mean():.0f}% of the positions within {most}"


def cut(total, sizes):
    out, i = [], 0
    while total > 0:
        n = min(total, sizes[i % len(sizes)])
        out.append(n)
        total -= n
        i += 1
    return out


def schedule(name):
    """Named schedules over the requests a, b, c, d."""
    n = LENGTHS
    if name == "whole":
        return [[(r, n[r])] for r in n]
    if name == "token-by-token":
        return [[("a", 1)] for _ in range(n["a"])]
    if name == "prompt-then-decode":
        return [[("a", 70)]] + [[("a", 1)] for _ in range(n["a"] - 70)] + [[("d", 33)]] + [[("d", 1)] for _ in range(64)]
    if name.startswith("portions-"):
        sizes = [int(s) for s in name[9:].split("-")]
        return [[("a", k)] for k in cut(n["a"], sizes)] + [[("b", k)] for k in cut(n["b"], sizes)]
    if name == "mixed":
        # portions beside single tokens, a request that pauses, blocks that are given back and used again
        return ([[("a", 40), ("c", 5)], [("c", 1), ("a", 2), ("b", 20)], [("c", 1), ("b", 1), ("d", 64), ("a", 17)],
                 [("c", 1), ("b", 1), ("d", 1)], [("c", 1), ("a", 60), ("b", 1)]]
                + [[("b", 1), ("d", 1), ("a", 1)] for _ in range(31)] + [[("b", 7), ("d", 1), ("c#2", 9)]]
                + [[("c#3", 2)], [("d#2", 90), ("c#3", 7)], [("d#2", 7)]])
    raise KeyError(name)


SCHEDULES = ["whole", "prompt-then-decode", "portions-2", "portions-3-16-17", "portions-64-1-65", "mixed"]
MAX_TOKENS = sum(blocks_of(v) for v in LENGTHS.values()) - 64
