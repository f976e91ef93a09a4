"""Small Movinex models for the CPU and the GPU tests; schedules and comparisons are those of the other listed-layer
designs."""
import random

import torch

from . import movinex_oracle as oracle
from .latent_oracle import write_model
from .movinex_oracle import attention_layer, config, dense, mamba_layer, moe, window_layer
from .ruralorn_cases import LENGTHS

CASES = {
    # all mixers and feed-forwards, layers that differ in everything, a loop in the middle that holds a recurrent layer; windows
    # shorter and longer than a block, kept tokens that end inside a block and past one
    "layers-differ": config(96, 131, [mamba_layer(6, 16, 24, dense(40), groups=2, conv=3, norm_groups=3),
                                      window_layer(6, 2, 24, 21, 5, moe(6, 2, 24, 3, 2), rot=16, softcap=6.0),
                                      mamba_layer(4, 24, 16, moe(8, 3, 16, 4, 3), conv=4),
                                      attention_layer(4, 1, 16, 24, None, every=7),
                                      window_layer(4, 4, 32, 40, 70, dense(72), base=2e5, scale=1.5, softcap=30.0)], loop=(1, 4, 2)),
    # nothing is a multiple of 8, the width is odd: the general kernels
    "odd-sizes": config(51, 77, [attention_layer(3, 1, 10, 7, moe(4, 1, 9, 2, 1), coef=-0.2, every=30),
                                 mamba_layer(2, 7, 10, dense(15), conv=2),
                                 window_layer(3, 3, 6, 13, 3, moe(3, 2, 6), rot=4, base=300.0),
                                 mamba_layer(3, 5, 19, None, groups=3, conv=6, norm_groups=5)], loop=(0, 2, 3),
                        logit_scale=1.9),
    # more query heads on a kv head than one tile of 16, heads wider than a tensor-core tile of columns, states wider than one
    # tile of rows, a window of the token alone beside kept ones, taps of 1 and 5
    "wide": config(128, 200, [window_layer(34, 2, 40, 65, 64, moe(20, 4, 32, 5, 2), rot=0),
                              mamba_layer(2, 72, 136, dense(136), conv=1, norm_groups=2),
                              attention_layer(8, 1, 136, 144, dense(64), every=1),
                              window_layer(5, 1, 8, 1, 9, None),
                              mamba_layer(5, 64, 256, None, groups=5, conv=5)], loop=(2, 5, 2), eps=1e-6),
    # no layer sees everything: blocks leave, those of the kept tokens stay; groups of one expert
    "windows-only": config(64, 90, [window_layer(4, 2, 16, 30, 3, None), window_layer(2, 1, 32, 17, 66, moe(9, 4, 16, 9, 5))],
                           loop=(0, 2, 1)),
    # no cached keys at all, no loop
    "states-only": config(64, 90, [mamba_layer(2, 32, 24, None), mamba_layer(4, 16, 64, dense(24), conv=3, norm_groups=4)]),
    # no recurrent layer, the loop is the last layer
    "attention-only": config(64, 90, [attention_layer(4, 2, 16, 24, dense(40)), window_layer(2, 2, 24, 50, 0, moe(2, 1, 16))],
                             loop=(1, 2, 4)),
}


# of the weights and tokens: one with which no early token's choice of experts is a close call, which rounding would decide
SEEDS = {"wide": 2}


class Model:
    """A case on disk with its oracle logits; ``tokens[r]`` / ``want[r]`` per request."""

    def __init__(self, name, folder, seed=None):
        seed = seed or SEEDS.get(name, 1)
        self.cfg = CASES[name]
        self.weights = oracle.random_weights(self.cfg, seed)
        self.path = write_model(folder, self.cfg, self.weights)
        rng = random.Random(seed)
        self.tokens = {r: [rng.randrange(self.cfg["vocab"]) for _ in range(n)] for r, n in LENGTHS.items()}
        with torch.no_grad():
            self.want = {r: oracle.forward(self.cfg, self.weights, t).numpy() for r, t in self.tokens.items()}
