"""Small Nimelorn models for the CPU and the GPU tests; schedules and comparisons are those of the other listed-layer
design."""
import random

import torch

from . import nimelorn_oracle as oracle
from .latent_oracle import write_model
from .nimelorn_oracle import attention_layer, config, dense, mlstm_layer, moe
from .ruralorn_cases import LENGTHS

CASES = {
    # layers that differ in everything: both mixers, both feed-forwards and none, shared keys and values under another mask,
    # chunks around a block, equal and unequal widths of keys and values
    "layers-differ": config(96, 131, [mlstm_layer(3, 16, 24, dense(40)),
                                      attention_layer(6, 2, 24, 16, 21, moe(5, 2, 24, 1.2, 1.7, 32, 0.8)),
                                      attention_layer(6, 2, 24, 16, 70, None, scale=0.3, kv_from=1),
                                      mlstm_layer(2, 32, 40, moe(3, 3, 40, 0.7), gate_cap=5.0),
                                      attention_layer(4, 4, 16, 32, 64, dense(72))]),
    # nothing is a multiple of 8, the width is odd: the general kernels
    "odd-sizes": config(51, 77, [attention_layer(3, 1, 10, 7, 13, moe(4, 1, 9, 1.0, 0.6, 11, 1.4)),
                                 mlstm_layer(2, 10, 7, dense(15)),
                                 attention_layer(3, 1, 10, 7, 40, moe(2, 1, 6, 2.0), kv_from=0),
                                 mlstm_layer(1, 5, 19, None)], embed_scale=3.0, buckets=13),
    # more query heads on a kv head than one tile of 16, memories wider than one block of columns and one tile of rows, a
    # chunk of the token alone, chunks of a block and of a block and one
    "wide": config(128, 200, [attention_layer(34, 2, 40, 72, 65, moe(20, 4, 32, 1.0, 1.0, 16)),
                              mlstm_layer(2, 136, 200, dense(136)),
                              attention_layer(5, 5, 8, 8, 1, dense(64)),
                              attention_layer(8, 1, 136, 144, 64, None),
                              mlstm_layer(5, 48, 64, moe(9, 8, 16, 0.9, 2.0, 24)),
                              attention_layer(34, 2, 40, 72, 32, None, kv_from=0)], eps=1e-6),
    # one kind of mixer only: no cached keys at all, no recurrent layer at all
    "memories-only": config(64, 90, [mlstm_layer(2, 24, 32, None), mlstm_layer(1, 64, 16, dense(24))]),
    "attention-only": config(64, 90, [attention_layer(4, 2, 16, 24, 30, None),
                                      attention_layer(2, 1, 32, 16, 200, moe(4, 2, 16, 1.0, 1.3, 16))]),
}


class Model:
    """A case on disk with its oracle logits; ``tokens[r]`` / ``want[r]`` per request."""

    def __init__(self, name, folder, seed=1):
        self.cfg = CASES[name]
        self.weights = oracle.random_weights(self.cfg, seed)
        self.path = write_model(folder, self.cfg, self.weights)
        rng = random.Random(seed)
        self.tokens = {r: [rng.randrange(self.cfg["vocab"]) for _ in range(n)] for r, n in LENGTHS.items()}
        with torch.no_grad():
            self.want = {r: oracle.forward(self.cfg, self.weights, t).numpy() for r, t in self.tokens.items()}
