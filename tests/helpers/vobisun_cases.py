"""Small Vobisun models and attention over a paged pool for the CPU and the GPU tests; schedules and comparisons are those of the
other listed-layer designs."""
import random

import torch

from zse_b200.format.config import HeadsSpec
from zse_b200.models.hybrid import PagedHeads

from . import vobisun_oracle as oracle
from .latent_oracle import write_model
from .ruralorn_cases import LENGTHS
from .vobisun_oracle import config, dense, layer, memory, window

CASES = {
    # layers that differ in everything, a loop in the middle; windows shorter and longer than a block of the cache, blocks of
    # tokens longer than the window, that end on a border of the cache's blocks or across one
    "layers-differ": config(96, 131, [layer(window(6, 2, 24, 16, 21, 5, rot=16, factor=3.0), memory(3, 16, 24), dense(40)),
                                      layer(window(4, 4, 16, 24, 70, 8, base=2e5), memory(2, 24, 16, tau=1.0), None, (0.4, 1.3)),
                                      layer(window(4, 1, 32, 40, 40, 32, scale=0.2), memory(4, 8, 40, tau=20.0), dense(72)),
                                      layer(window(2, 2, 24, 8, 9, 17, rot=2, factor=0.5), memory(1, 40, 48), dense(24))],
                            loop=(1, 3, 2), ranks=[16, 8, 5, 24]),
    # nothing is a multiple of 8, the width is odd: the general kernels
    "odd-sizes": config(51, 77, [layer(window(3, 1, 10, 7, 13, 3, rot=4, base=300.0, factor=1.7), memory(2, 7, 10, tau=2.5),
                                       dense(15)),
                                 layer(window(3, 3, 6, 5, 30, 7, rot=0), memory(1, 5, 3), None)],
                        loop=(0, 2, 3), taps=2, embed_scale=1.0, ranks=[3, 1]),
    # more query heads on a kv head than one tile of 16, heads wider than a tensor-core tile of columns, memories wider than one
    # tile of rows, blocks of one token, a window of the token alone; no convolution to speak of
    "wide": config(128, 200, [layer(window(34, 2, 40, 48, 65, 1), memory(2, 136, 72), dense(136)),
                              layer(window(5, 1, 136, 144, 1, 2, rot=64), memory(1, 256, 64, tau=16.0), dense(8)),
                              layer(window(3, 3, 24, 72, 100, 10), memory(5, 64, 128), None)], taps=1, eps=1e-6),
    # one head of everything, blocks and windows of a cache block each, factors of one, more taps than a portion has tokens
    "ones": config(64, 90, [layer(window(1, 1, 64, 64, 64, 64, rot=32), memory(1, 16, 16, tau=1.0), dense(64), (1.0, 1.0)),
                            layer(window(8, 8, 8, 8, 20, 4), memory(8, 8, 8), None, (-1.0, 0.3))], loop=(1, 2, 4), taps=6,
                   embed_scale=1.0, ranks=[1, 64]),
}


class Model:
    """A case on disk with its oracle logits; ``tokens[r]`` / ``want[r]`` per request."""

    def __init__(self, name, folder, seed=1):
        self.cfg, self.ranks = CASES[name]
        self.weights = oracle.random_weights(self.cfg, self.ranks, seed)
        self.path = write_model(folder, self.cfg, self.weights)
        rng = random.Random(seed)
        self.tokens = {r: [rng.randrange(self.cfg["vocab"]) for _ in range(n)] for r, n in LENGTHS.items()}
        with torch.no_grad():
            self.want = {r: oracle.forward(self.cfg, self.weights, t).numpy() for r, t in self.tokens.items()}


# ---- attention that sees means of blocks ------------------------------------------------------------------------------------
def spec(heads, kv_heads, dim, vdim, size, pool, scale=0.3, **kw):
    return HeadsSpec(heads, kv_heads, dim, vdim, scale, window=size, pool=pool, sink=True, whole_norm=True, bias=True, **kw)


SPECS = {
    "window": spec(8, 2, 64, 64, 130, 8),
    "short-window": spec(6, 3, 128, 128, 20, 50, 0.2, out_scale=0.7),
    "token-alone": spec(4, 2, 32, 48, 1, 3, 0.5),
    "one-kv-head": spec(20, 1, 48, 40, 64, 16, 0.4),
    "single-tokens": spec(4, 4, 40, 24, 33, 1, 0.4, out_scale=-1.5),
    "blocks-of-the-cache": spec(4, 2, 72, 72, 128, 64),
    "long-blocks": spec(4, 2, 24, 24, 65, 100, 0.4, gated=False),
    "no-blocks": spec(4, 2, 64, 32, 100, 0),
    "wide": spec(4, 2, 256, 200, 90, 9, 0.1),
    "general": spec(6, 2, 18, 22, 50, 7, 0.4),
}


class PooledAttention:
    """Sequences whose keys, values and means of blocks lie in blocks of a pool of wider rows, in random order."""

    def __init__(self, ops, s, dt, device, bs=64, seqs=3, tokens=700, seed=0, rows=420):
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *sh: torch.randn(*sh, generator=g).to(device)
        self.ops, self.spec, self.dt, self.bs, self.device = ops, s, dt, bs, device
        width = (tokens + bs - 1) // bs
        means = (tokens // s.pool + bs - 1) // bs if s.pool else 0
        n = (width + means) * seqs
        self.tables = torch.randperm(n + 3, generator=g)[:n].view(seqs, width + means).int().to(device)
        pool = torch.zeros(n + 3, 1, 1, bs, s.row + 8, device=device, dtype=dt)
        self.kv = PagedHeads(pool, s, width)
        self.k, self.v = rnd(seqs, tokens, s.kv_heads, s.dim).to(dt), rnd(seqs, tokens, s.kv_heads, s.vdim).to(dt)
        self.inp = rnd(rows, s.in_width).to(dt)
        self.sink = 2 + rnd(s.heads)
        self.store()

    def i32(self, v):
        return torch.tensor(v, dtype=torch.int32, device=self.device)

    def store(self):
        seqs, tokens = self.k.shape[:2]
        j = torch.arange(tokens, device=self.device)
        for s in range(seqs):
            blk = self.tables[s, j // self.bs].long()
            self.kv.k[blk, :, j % self.bs, : self.spec.dim] = self.k[s]
            self.kv.v[blk, :, j % self.bs, : self.spec.vdim] = self.v[s]
        if self.spec.pool:
            self.ops.heads_pool(self.kv, self.tables, self.i32([s for s in range(seqs) for _ in range(tokens)]),
                                self.i32(list(range(tokens)) * seqs), self.spec, seqs * tokens)

    def means(self, seq):
        """The stored means of a sequence's keys and values."""
        b = torch.arange(self.k.shape[1] // self.spec.pool, device=self.device)
        blk = self.tables[seq, self.kv.means_at + b // self.bs].long()
        return (self.kv.k[blk, :, b % self.bs, : self.spec.dim], self.kv.v[blk, :, b % self.bs, : self.spec.vdim])

    def plain(self, t, seq, pos):
        s = self.spec
        f = lambda x: x.detach().cpu().to(oracle.F)
        q = f(self.inp[t, : s.heads * s.dim]).view(s.heads, s.dim)
        k, v = f(self.k[seq, : pos + 1]), f(self.v[seq, : pos + 1])
        P, per, T = s.pool or pos + 2, s.heads // s.kv_heads, pos + 1
        keys, values = torch.cat([k, oracle.block_means(k, P)]), torch.cat([v, oracle.block_means(v, P)])
        see = torch.cat([oracle.seen_tokens(T, s.window)[pos], oracle.seen_blocks(T, s.window, P)[pos]])
        y = []
        for n in range(s.heads):
            z = torch.cat([(keys[see, n // per] @ q[n]) * s.scale, f(self.sink[n: n + 1])])
            y.append(torch.softmax(z, 0)[:-1] @ values[see, n // per])
        y = torch.stack(y)
        if s.gated:
            y = y * oracle.sigmoid(f(self.inp[t, s.gate_col: s.gate_col + s.heads]))[:, None]
        return s.out_scale * y.reshape(-1)

    def rows(self, seqs, positions, splits=1):
        s, M = self.spec, len(seqs)
        out = torch.zeros(M, s.heads * s.vdim, dtype=self.dt, device=self.device)
        self.ops.heads_attn(self.inp, self.kv, self.tables, self.i32(seqs), self.i32(positions), out, M, s,
                            torch.zeros(M * splits * s.heads * (s.vdim + 2), device=self.device), splits, self.sink)
        return out

    def chunks(self, spans, first=0):
        cu = [0]
        for _, n in spans:
            cu.append(cu[-1] + n)
        pos = self.i32([a + i for a, n in spans for i in range(n)])
        out = torch.zeros(cu[-1], self.spec.heads * self.spec.vdim, dtype=self.dt, device=self.device)
        self.ops.heads_attn_chunks(self.inp, self.kv, self.tables, self.i32(cu), self.i32([a for a, _ in spans]), pos, first,
                                   len(spans), max(n for _, n in spans[first:]), out, self.spec, self.sink)
        return out, cu


def loud_places(s, pos):
    """Keys at the borders of what the token at ``pos`` sees: of the window, of the last mean that is seen and the next one, of
    the cache's blocks, far away, the token itself and the next one."""
    lo, P = s.first_seen(pos), s.pool
    at = {pos, pos + 1, lo, lo - 1, (lo + pos) // 2, pos // 64 * 64, pos // 64 * 64 - 1, 0}
    if P:
        n = s.blocks_seen(pos) * P
        at |= {n - 1, n, n - P, P - 1, P, min(n - 1, 64), 63 // P * P}
    return sorted(k for k in at if 0 <= k)


def make_loud(A, key, head, query_row, strength=40.0):
    """The key at ``key`` of sequence 0 takes nearly all the weight of ``head`` of the query in ``query_row``, alone or in its
    block's mean."""
    s = A.spec
    q = A.inp[query_row, head * s.dim: (head + 1) * s.dim].float()
    size = max(1, s.pool) if s.pool and key // s.pool < s.blocks_seen(10 ** 6) else 1
    A.k[0, key, head // (s.heads // s.kv_heads)] = (q * (strength * size / abs(s.scale) / q.pow(2).sum())).to(A.dt)
    A.store()
