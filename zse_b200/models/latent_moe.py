"""Decoders of latent attention and routed feed-forwards (Ruralorn) over the paged cache.

Same pass contract as ``DecoderModel``.  A token caches ONE row per layer, [normed latent | rotated key part]; the heads'
keys and values are linear images of it.  A layer:

    x     = RMSNorm(h) * w1                                  (fused with the residual sum of the sub-layer before it)
    q|c|g = x W_in           fused projection [queries | latent, rotated key | gate]
    prep                     latent norm, rotation of keys and queries, cache write                        1 kernel
    a     = attention        two forms, below
    h    += (a * sigmoid(g)) W_o ;  x = RMSNorm(h) * w2                                                    1 kernel
    y     = sum over the chosen experts e of  down_e(gelu(score_e * up_e(x)))  +  the shared expert
    h    += y                                                (the next layer's first kernel)

Attention in two forms with the same result.  Rows that decode, and chunks of at most ``SHORT_CHUNK`` tokens, attend to
the cached rows directly: the query is multiplied by W_uk once, all heads then share the row as key and its leading part
as value, and the result is multiplied by W_uv - the cache is read once per token whatever the number of heads.  Longer
chunks expand the cached rows that their windows reach into per-head keys and values (one GEMM), which costs a fraction
of the arithmetic when many queries use the same key.  A packed pass may hold both kinds: short ones are laid out first.

Activations and cache are bfloat16 with fp32 accumulation (residual, norms, scores, softmax, router and gates in fp32),
or fp32 throughout (``dtype="float32"``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..format.config import LatentSpec, MoESpec
from ..format.loader import ZSELoader
from ..ops.backend import LinearWeight
from .decoder import StepBuffers
from .design import PLANE_ROWS, SHORT_CHUNK, DesignModel


def attention_splits(seqs: int, groups: int, span: int, most: int, sms: int) -> int:
    """Key splits of a decode step's attention.  One CTA of it fills an SM, so the time goes with the number of waves; a
    wave costs its tiles of 64 keys and about four tiles' time to start and end, every split its part of the merge.  A
    split holds at least two tiles."""
    best, cost = 1, float("inf")
    for n in (1, 2, 3, 4, 5, 7, 9, 12, 16):
        if n > most or (n > 1 and span < 128 * n):
            break
        waves = (seqs * groups * n + sms - 1) // sms
        c = waves * (span / 64 / n + 4) + 0.5 * n
        if c < cost:
            best, cost = n, c
    return best


@dataclass
class LatentLayer:
    spec: LatentSpec
    moe: Optional[MoESpec]
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor]
    w_in: LinearWeight
    latent_norm: torch.Tensor
    freqs: torch.Tensor
    ukv: LinearWeight                       # [W_uk (padded to 8 rows) ; W_uv]
    uk: torch.Tensor                        # views of it: [heads * dim, kv_rank], [heads * vdim, kv_rank]
    uv: torch.Tensor
    o: LinearWeight
    router: Optional[LinearWeight] = None
    up: Optional[torch.Tensor] = None       # [experts * ff, H]
    down: Optional[torch.Tensor] = None     # [experts * H, ff]
    shared_up: Optional[torch.Tensor] = None
    shared_down: Optional[torch.Tensor] = None


@dataclass
class ChunkGroup:
    """Sequences [first, last) of a packed pass whose expanded keys fit the scratch together."""
    first: int
    last: int
    rows: int                               # expanded rows of the group
    max_q: int


class LatentStepBuffers(StepBuffers):
    def __init__(self, model: "LatentMoEModel", max_tokens: int, max_seqs: int, max_blocks: int, max_planes: int,
                 logits_rows: int, attn_splits: int):
        c, dev, act = model.config, model.device, model.act_dtype
        f32, i32 = torch.float32, torch.int32
        z = lambda *s, dt: torch.zeros(*s, dtype=dt, device=dev)
        H = c.hidden_size
        self._common(dev, H, c.vocab_size, max_tokens, max_seqs, max_blocks, logits_rows, attn_splits, act=act,
                     logits=f32)
        specs = [L.spec for L in model.layers]
        self.plane_rows = min(max_tokens, PLANE_ROWS)
        in_w = max(s.in_width for s in specs)
        self.inp = z(max_tokens * in_w, dt=act)
        self.in_views = {w: self.inp[: max_tokens * w].view(max_tokens, w) for w in {s.in_width for s in specs}}
        self.in_planes = z(max_planes * self.plane_rows * in_w, dt=f32)
        self.in_plane_views = {w: self.in_planes[: max_planes * self.plane_rows * w].view(max_planes, self.plane_rows, w)
                               for w in {s.in_width for s in specs}}
        out_w = max(s.heads * s.vdim for s in specs)
        self.attn_flat = z(max_tokens * out_w, dt=act)
        self.attn_views = {w: self.attn_flat[: max_tokens * w].view(max_tokens, w)
                           for w in {s.heads * s.vdim for s in specs}}
        # split-K planes of decode-sized passes, one plane of any other
        self.partials = z(max(max_planes * self.plane_rows, max_tokens) * H, dt=f32)
        self.partial_views = (self.partials[: max_planes * self.plane_rows * H].view(max_planes, self.plane_rows, H),
                              self.partials[: max_tokens * H].view(1, max_tokens, H))
        short = max_tokens if not model.expands else min(max_tokens, max(256, max_seqs * SHORT_CHUNK))
        self.short_rows = short
        self.q_lat = z(short * max(s.heads * s.row for s in specs), dt=act)
        self.o_lat = z(short * max(s.heads * s.kv_rank for s in specs), dt=act)
        rows_split = min(short, max(256, max_seqs))      # only decode passes split their keys
        self.attn_scratch = z(rows_split * attn_splits * max(s.heads * (s.kv_rank + 2) for s in specs), dt=f32)
        self.row_seq = z(max_tokens, dt=i32)
        # expanded keys and values of one group of chunks
        windows = [s.window for s in specs]
        reach = max_blocks * model.cache_block_size
        if windows and min(windows) > 0:
            reach = min(reach, max(windows))
        self.ctx_cap = max_tokens + reach if model.expands else 0
        cap = max(self.ctx_cap, 1)
        self.ctx_c = z(cap * max(s.kv_rank for s in specs), dt=act)
        self.ctx_kr = z(cap * max((s.rot_dim + 7) // 8 * 8 for s in specs), dt=act)
        self.ctx_kvx = z(cap * max(L.ukv.N for L in model.layers), dt=act)
        self.windows = sorted(set(windows))
        self.ctx_off = z(len(self.windows), max_seqs + 1, dt=i32)
        pin = dev.type == "cuda"
        self.h_ctx_off = torch.zeros(len(self.windows), max_seqs + 1, dtype=i32, pin_memory=pin)
        self.h_row_seq = torch.zeros(max_tokens, dtype=i32, pin_memory=pin)
        self.short: int = 0                       # rows of the staged pass that read the cache directly
        self.groups: List[List[ChunkGroup]] = [[] for _ in self.windows]
        self.moe_ws = model.ops.moe_workspace([L.moe for L in model.layers if L.moe is not None], H, max_tokens, act)


class LatentMoEModel(DesignModel):
    kernel_group = "latent"

    # ---- loading --------------------------------------------------------------------------------------
    def _load(self, loader: ZSELoader, progress=None) -> None:
        c, ops, dev = self.config, self.ops, self.device
        r = self._open(loader)
        tensor, keep, stack = r.tensor, r.keep, r.stack
        H = c.hidden_size
        self.embed = keep(tensor("embed"))
        self.norm = keep(tensor("final.norm"))
        for i in range(c.num_layers):
            p, s, m = f"l{i}.", c.latent_spec(i), c.moe_spec(i)
            parts = [(0, tensor(p + "mix.q")), (s.latent_col, tensor(p + "mix.dkv"))]
            if s.gated:
                parts.append((s.gate_col, tensor(p + "mix.g")))
            w_in = stack(parts, s.in_width, H)
            v0 = (s.heads * s.dim + 7) // 8 * 8
            ukv = stack([(0, tensor(p + "mix.uk")), (v0, tensor(p + "mix.uv"))], v0 + (s.heads * s.vdim + 7) // 8 * 8,
                        s.kv_rank)
            j = torch.arange(s.rot_dims // 2, dtype=torch.float64)
            freqs = (s.rot_base ** (-2.0 * j / s.rot_dims)).to(torch.float32).to(dev)
            L = LatentLayer(s, m, keep(tensor(p + "norm1")), None, ops.dense_linear(w_in),
                            keep(tensor(p + "mix.dkv.norm")), freqs, ops.dense_linear(ukv), ukv[: s.heads * s.dim],
                            ukv[v0: v0 + s.heads * s.vdim], ops.dense_linear(keep(tensor(p + "mix.o"))))
            if m is not None:
                L.norm2 = keep(tensor(p + "norm2"))
                L.router = ops.dense_linear(keep(tensor(p + "mlp.router")))
                L.up = stack([(e * m.ff, tensor(f"{p}mlp.e{e}.up")) for e in range(m.experts)], m.experts * m.ff, H)
                L.down = stack([(e * H, tensor(f"{p}mlp.e{e}.down")) for e in range(m.experts)], m.experts * H, m.ff)
                if m.shared_ff:
                    L.shared_up = keep(tensor(p + "mlp.shared.up"))
                    L.shared_down = keep(tensor(p + "mlp.shared.down"))
            self.layers.append(L)
            if progress:
                progress(i + 1, c.num_layers)
        self.lm_head = ops.dense_linear(keep(tensor("head")))
        r.release()
        self.embed_scale = float(c.embed_multiplier if c.embed_multiplier is not None else 1.0)
        self.logit_scale = float(c.logit_scale if c.logit_scale is not None else 1.0)
        self.logit_cap = float(c.final_logit_softcapping or 0.0)
        self.expands = all(ops.latent_expands(L.spec, self.act_dtype) for L in self.layers)
        self.max_window = c.cache_window
        self._row_views = {}

    # ---- buffers --------------------------------------------------------------------------------------
    def make_buffers(self, max_tokens: int, max_seqs: int, max_blocks: int, logits_rows: Optional[int] = None,
                     max_planes: int = 8, attn_splits: int = 1) -> LatentStepBuffers:
        return LatentStepBuffers(self, max_tokens, max_seqs, max_blocks, max_planes, logits_rows or max_seqs, attn_splits)

    def _rows(self, kv: torch.Tensor, li: int, spec: LatentSpec) -> torch.Tensor:
        """This layer's cached rows [blocks, block_size, row] inside the pool (rows as wide as the widest layer's)."""
        key = (kv.data_ptr(), li)
        v = self._row_views.get(key)
        if v is None:
            layer = kv[li]
            v = layer.as_strided((layer.shape[0], layer.shape[3], spec.row), (layer.stride(0), spec.row, 1),
                                 layer.storage_offset())
            self._row_views[key] = v
        return v

    def attention_splits(self, seqs: int, max_len: int, most: int, sms: int) -> int:
        span = min(max_len, self.max_window) if self.max_window else max_len
        return attention_splits(seqs, max((L.spec.heads + 31) // 32 for L in self.layers), span, most, sms)

    # ---- layout of a packed pass ----------------------------------------------------------------------
    def pass_order(self, items) -> Optional[List[int]]:
        if not self.expands:
            return None
        return sorted(range(len(items)), key=lambda i: len(items[i][1]) > SHORT_CHUNK)

    def stage_prefill(self, b: LatentStepBuffers, spans) -> None:
        at, n_short = 0, 0
        for s, (_, n) in enumerate(spans):
            if self.expands and n > SHORT_CHUNK:
                break
            b.h_row_seq[at: at + n] = s
            at += n
            n_short = s + 1
        b.short = at
        if at:
            b.row_seq[:at].copy_(b.h_row_seq[:at], non_blocking=True)
        for wi, window in enumerate(b.windows):
            groups: List[ChunkGroup] = []
            for s in range(n_short, len(spans)):
                start, n = spans[s]
                rows = n + (min(start, window - 1) if window > 0 else start)
                if not groups or groups[-1].rows + rows > b.ctx_cap:
                    groups.append(ChunkGroup(s, s, 0, 0))
                g = groups[-1]
                b.h_ctx_off[wi, s] = g.rows
                g.last, g.rows, g.max_q = s + 1, g.rows + rows, max(g.max_q, n)
            b.groups[wi] = groups
        if n_short < len(spans):
            b.ctx_off[:, : len(spans)].copy_(b.h_ctx_off[:, : len(spans)], non_blocking=True)

    # ---- forward --------------------------------------------------------------------------------------
    def forward(self, b: LatentStepBuffers, kv: torch.Tensor, M: int, mode: str, num_seqs: int, max_q_len: int = 1,
                n_logit_rows: int = 0, attn_splits: int = 1) -> None:
        c, ops = self.config, self.ops
        eps = c.rms_norm_eps
        decode = mode == "decode"
        short = M if decode else b.short
        planes_ok = M <= b.plane_rows
        partials = b.partial_views[0 if planes_ok else 1]
        ops.embedding(self.embed, b.ids, b.residual, M, self.embed_scale)
        planes, slots = 0, None
        for li, L in enumerate(self.layers):
            s = L.spec
            ops.add_norm(b.residual, partials, planes, slots, L.norm1, b.xnorm, M, eps)
            slots = None
            inp = b.in_views[s.in_width]
            in_planes, n_in = b.in_plane_views[s.in_width], 0
            if planes_ok:
                n_in = ops.linear_partial(L.w_in, b.xnorm, M, in_planes)
            else:
                ops.linear(L.w_in, b.xnorm, M, inp)
            rows = self._rows(kv, li, s)
            ops.latent_prep(inp, in_planes, n_in, rows, b.positions, b.slots, L.freqs, L.latent_norm, s, eps, M)
            out = b.attn_views[s.heads * s.vdim]
            if short:
                ops.latent_attn(inp, L, rows, b.block_tables, None if decode else b.row_seq, b.positions, b.q_lat,
                                b.o_lat, out, short, s, b.attn_scratch, attn_splits)
            if short < M:
                wi = b.windows.index(s.window)
                for g in b.groups[wi]:
                    ops.latent_attn_chunks(inp, L, rows, b.block_tables, b.cu_q, b.q_pos0, b.ctx_off[wi], g,
                                           (b.ctx_c, b.ctx_kr, b.ctx_kvx), out, s)
            planes = ops.linear_partial(L.o, out, M, partials)
            if L.moe is not None:
                ops.add_norm(b.residual, partials, planes, None, L.norm2, b.xnorm, M, eps)
                slots, planes = ops.moe(L, b.xnorm, M, b.moe_ws), 0
        ops.add_norm(b.residual, partials, planes, slots, self.norm, b.xnorm, M, eps)
        if n_logit_rows:
            torch.index_select(b.xnorm, 0, b.logit_rows[:n_logit_rows], out=b.xsel[:n_logit_rows])
            ops.linear_f32(self.lm_head, b.xsel, n_logit_rows, b.logits)
            ops.logits_finish(b.logits, n_logit_rows, self.logit_scale, self.logit_cap)
