"""Decoders whose layers mix attention over heads and recurrent mixers (matrix memories, state spaces), over the paged cache
and the state slots: layer runs, mixers, feed-forwards, and the placement of norms on the sublayers' outputs (Nimelorn).
``looped`` and ``twin`` have the other placements.

Same pass contract as ``DecoderModel``.  The residual x is fp32; sublayers read x itself (rounded to the activations' type):

    x     = norm(embedding + what the design adds to it)                                       1 kernel
    y     = mixer(x);  x += norm(y) * w1                                    (sum of the split-K planes, norm, add: 1 kernel)
    y     = ff(x);     x += norm(y) * w2                                                       (the same kernel)
    after the last sublayer the same kernel also writes norm(x) * w_final for the head

Attention caches normed keys and values as [kv head][token][dim] tiles of a block; a layer that takes another layer's keys
and values projects queries only.  Rows that decode, and chunks of at most ``SHORT_CHUNK`` tokens, run a row at a time with
the keys split over CTAs; longer chunks run in tiles of queries.  A matrix memory does the same: short chunks step through
the state token by token, with read-out, head norm and output gate in the step's kernel; longer ones run chunkwise, with the
decays inside a chunk as a lower-triangular matrix.  A state space passes its inputs through a short convolution first, whose
last inputs are part of its state, and does the same; so does gated linear attention.  Attention that sees older tokens as means
of blocks keeps those in blocks of the cache of their own, behind the tokens' in the block tables; the kernel that writes a
block's last key and value writes the mean in a decode step, one more kernel in any other pass.  A packed pass may hold both kinds: short ones are laid out first.

A sequence's recurrent state and its last token live in ``cache.state_slots``; ``state_rows`` names the rows that a pass's
sequences read and write.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Union

import torch

from ..format.config import (DenseSpec, GatedLinearSpec, HeadsSpec, MatrixMemorySpec, MoESpec, StateSpaceSpec, TwinSpec,
                             attention_of, recurrent_of)
from ..format.loader import ZSELoader
from ..ops.backend import LinearWeight
from .decoder import StepBuffers
from .design import PLANE_ROWS, SHORT_CHUNK, DesignModel


@dataclass
class EmbedDesign:
    table: torch.Tensor
    scale: float
    base: float                             # of the sinusoid
    norm: torch.Tensor
    bigram: Optional[torch.Tensor] = None   # [buckets + 1, H]; the last row is that of a sequence's first token
    buckets: int = 0
    mul_prev: int = 0
    mul_cur: int = 0
    turns: Optional[torch.Tensor] = None    # device form of the sinusoid's frequencies


@dataclass
class HybridLayer:
    spec: Union[HeadsSpec, MatrixMemorySpec, StateSpaceSpec, TwinSpec]
    ff: Union[DenseSpec, MoESpec, None]
    norm1: torch.Tensor
    w_in: LinearWeight
    o: LinearWeight
    norm2: Optional[torch.Tensor] = None
    # attention
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None     # of the columns of w_in before the gates
    freqs: Optional[torch.Tensor] = None    # of the rotation
    temp: Optional[torch.Tensor] = None     # fp32 [heads], factor of a head's scores
    sink: Optional[torch.Tensor] = None     # fp32 [heads], score without a value
    # matrix memory
    w_if: Optional[LinearWeight] = None     # the rows of w_in that make the gates
    if_bias: Optional[torch.Tensor] = None  # fp32 [2 * heads]
    head_norm: Optional[torch.Tensor] = None  # also of gated linear attention: [vdim], shared by the heads
    # gated linear attention
    decay_w: Optional[torch.Tensor] = None  # fp32 [heads * dim, rank]
    decay_b: Optional[torch.Tensor] = None  # fp32 [heads * dim]
    # state space; of what a twin layer's mixers read
    conv_w: Optional[torch.Tensor] = None   # fp32 [taps, channels]
    conv_b: Optional[torch.Tensor] = None
    dt_bias: Optional[torch.Tensor] = None  # fp32 [heads], like the next two
    neg_a: Optional[torch.Tensor] = None    # -exp(A_log)
    D: Optional[torch.Tensor] = None
    out_norm: Optional[torch.Tensor] = None
    # factors of the sublayers' results
    scale1: Optional[torch.Tensor] = None
    scale2: Optional[torch.Tensor] = None
    # feed-forward
    up_w: Optional[LinearWeight] = None
    down_w: Optional[LinearWeight] = None
    router: Optional[LinearWeight] = None
    up: Optional[torch.Tensor] = None
    down: Optional[torch.Tensor] = None
    shared_up: Optional[torch.Tensor] = None
    shared_down: Optional[torch.Tensor] = None

    @property
    def moe(self) -> Optional[MoESpec]:
        return self.ff if isinstance(self.ff, MoESpec) else None

    @property
    def out_width(self) -> int:
        """Columns that the mixer's last product reads; of a twin layer that of the feed-forward reads them too."""
        w = self.spec.out_width
        return w + (self.ff.ff + 7) // 8 * 8 if isinstance(self.spec, TwinSpec) and self.ff is not None else w


@dataclass
class LayerRun:
    """One run of a layer: layers of a loop run several times, each run with its own keys and values or its own state."""
    layer: HybridLayer
    cache_layer: int = -1                   # of the cache pool (attention)
    state_at: int = 0                       # first element of its part of a sequence's state (recurrent mixers)
    inputs_at: int = 0                      # ... of the last inputs of the convolution ahead of its mixer
    enters_loop: bool = False               # first of a pass of the loop


@dataclass
class Pass:
    """What a pass's layers need to know about it."""
    kv: torch.Tensor
    M: int
    num_seqs: int
    max_q_len: int
    row_seq: Optional[torch.Tensor]         # None: every row is a sequence of its own (decode), like the next
    cu_q: Optional[torch.Tensor]
    short: tuple                            # rows and sequences that run token by token
    planes_ok: bool                         # projections come as split-K planes
    partials: torch.Tensor
    splits: int


class PagedHeads:
    """One layer's cached keys [blocks, kv_heads, block_size, dim] and values inside the pool, whose rows are as wide as the
    widest layer's; dims are padded to 8.  ``means_at``: where the blocks of means begin in a row of the block tables."""

    def __init__(self, layer: torch.Tensor, spec: HeadsSpec, means_at: int = 0):
        self.means_at = means_at
        # layer: [blocks, 1, 1, block_size, pool row]
        bs, G = layer.shape[3], spec.kv_heads
        d, v = (spec.dim + 7) // 8 * 8, (spec.vdim + 7) // 8 * 8
        self.block_size, self.block_stride = bs, layer.stride(0)
        self.k = layer.as_strided((layer.shape[0], G, bs, d), (layer.stride(0), bs * d, d, 1), layer.storage_offset())
        self.v = layer.as_strided((layer.shape[0], G, bs, v), (layer.stride(0), bs * v, v, 1),
                                  layer.storage_offset() + G * bs * d)


class HybridStepBuffers(StepBuffers):
    def __init__(self, model: "HybridModel", max_tokens: int, max_seqs: int, max_blocks: int, max_planes: int,
                 logits_rows: int, attn_splits: int):
        c, dev, act = model.config, model.device, model.act_dtype
        f32, i32 = torch.float32, torch.int32
        z = lambda *s, dt: torch.zeros(*s, dtype=dt, device=dev)
        H = c.hidden_size
        self._common(dev, H, c.vocab_size, max_tokens, max_seqs, max_blocks, logits_rows, attn_splits, act=act,
                     logits=f32)
        specs = [L.spec for L in model.layers]
        heads = [a for a in map(attention_of, specs) if a is not None]
        memories = [s for s in specs if isinstance(s, MatrixMemorySpec)]
        self.plane_rows = min(max_tokens, PLANE_ROWS)

        def views(widths, dt):
            flat = z(max_tokens * max(widths), dt=dt)
            return {w: flat[: max_tokens * w].view(max_tokens, w) for w in set(widths)}

        self.in_views = views([s.in_width for s in specs], act)
        self.out_views = views([L.out_width for L in model.layers], act)
        spaces = [s for s in specs if isinstance(s, StateSpaceSpec)]
        self.xbc_views = views([s.conv_width for s in spaces], act) if spaces else {}
        self.dt = z(max_tokens * max([1] + [s.heads for s in spaces]), dt=f32)
        linears = [s for s in map(recurrent_of, specs) if isinstance(s, GatedLinearSpec)]
        self.dt_side = z(max_tokens * max([1] + [s.in_width - s.dt_col for s in spaces]
                                          + [s.in_width - s.rank_col for s in linears]), dt=f32)
        self.decays = z(max_tokens * max([1] + [s.heads * s.dim for s in linears]), dt=f32)
        self.linear_ws = model.ops.gated_linear_workspace(linears, max_tokens) if linears else None
        planes = z(max_planes * self.plane_rows * max(s.in_width for s in specs), dt=f32)
        self.in_plane_views = {w: planes[: max_planes * self.plane_rows * w].view(max_planes, self.plane_rows, w)
                               for w in {s.in_width for s in specs}}
        # split-K planes of decode-sized passes, one plane of any other
        partials = z(max(max_planes * self.plane_rows, max_tokens) * H, dt=f32)
        self.partial_views = (partials[: max_planes * self.plane_rows * H].view(max_planes, self.plane_rows, H),
                              partials[: max_tokens * H].view(1, max_tokens, H))
        dense = [L.ff.ff for L in model.layers if isinstance(L.ff, DenseSpec)]
        self.act_views = views(dense, act) if dense else {}
        wide = [L.ff.ff for L in model.layers if isinstance(L.ff, DenseSpec) and L.ff.gated
                and model.ops.glu_expands(L.ff.ff, H, act)]
        self.glu = z(max_tokens * 2 * max([0] + wide), dt=act)
        rows_split = min(max_tokens, max(256, max_seqs))      # only decode passes split their keys
        self.attn_scratch = z(rows_split * attn_splits * max([1] + [s.heads * (s.vdim + 2) for s in heads]), dt=f32)
        gate_w = max([1] + [2 * s.heads for s in memories])
        self.gates = z(max_tokens * gate_w, dt=f32)
        self.gate_planes = z(max_planes, max_tokens * gate_w, dt=f32)
        self.memory_ws = model.ops.memory_workspace(memories, max_tokens)
        self.row_seq = z(max_tokens, dt=i32)
        self.state_rows = torch.full((2, max_seqs), -1, dtype=i32, device=dev)
        self.h_row_seq = torch.zeros(max_tokens, dtype=i32, pin_memory=dev.type == "cuda")
        self.short_rows = self.short_seqs = 0     # rows and sequences of the staged pass that run token by token
        self.moe_ws = model.ops.moe_workspace([L.moe for L in model.layers if L.moe is not None], H, max_tokens, act)


class HybridModel(DesignModel):
    """Layers whose norms sit on the sublayers' outputs; ``models.looped`` and ``models.twin`` have the other placements."""
    kernel_group = "hybrid"
    means_at = 0                # column of the block tables from which on the blocks of means stand; set by the runner

    # ---- loading --------------------------------------------------------------------------------------
    def _load(self, loader: ZSELoader, progress=None) -> None:
        c, ops, dev = self.config, self.ops, self.device
        r = self._open(loader)
        H, ex = c.hidden_size, c.embed_design
        self.embed = r.get("embed")
        self.embed_design = EmbedDesign(self.embed, float(c.embed_multiplier or 1.0), float(ex["sinusoid_base"]),
                                        r.get("embed.norm"))
        if ex.get("bigram"):
            b, e = ex["bigram"], self.embed_design
            e.bigram, e.buckets, e.mul_prev, e.mul_cur = r.get("bigram"), b["buckets"], b["mul_prev"], b["mul_cur"]
        self.norm = r.get("final.norm")
        for i in range(c.num_layers):
            p, s, m = f"l{i}.", c.mixer_spec(i), c.ff_spec(i)
            t = lambda name: r.tensor(p + name)
            if isinstance(s, MatrixMemorySpec):
                w = r.stack([(0, t("mix.q")), (s.k_col, t("mix.k")), (s.v_col, t("mix.v")), (s.gate_col, t("mix.g")),
                             (s.if_col, t("mix.i")), (s.if_col + s.heads, t("mix.f"))], s.in_width, H)
                L = HybridLayer(s, m, r.get(p + "norm1"), ops.dense_linear(w), r.linear(p + "mix.o"))
                L.w_if = ops.dense_linear(w[s.if_col: s.if_col + 2 * s.heads])
                L.if_bias = torch.cat([t("mix.i.b"), t("mix.f.b")]).float().contiguous()
                L.head_norm = r.get(p + "mix.norm")
            else:
                parts = [(0, t("mix.q")), (s.gate_col, t("mix.g"))]
                if s.own_kv:
                    parts += [(s.k_col, t("mix.k")), (s.v_col, t("mix.v"))]
                L = HybridLayer(s, m, r.get(p + "norm1"), ops.dense_linear(r.stack(parts, s.in_width, H)),
                                r.linear(p + "mix.o"), q_norm=r.get(p + "mix.q.norm"))
                if s.own_kv:
                    L.k_norm = r.get(p + "mix.k.norm")
            if m is not None:
                L.norm2 = r.get(p + "norm2")
            if isinstance(m, DenseSpec):
                L.up_w, L.down_w = r.linear(p + "mlp.up"), r.linear(p + "mlp.down")
            elif m is not None:
                self._load_experts(r, L, p, m, H)
            self.layers.append(L)
            if progress:
                progress(i + 1, c.num_layers)
        self.lm_head = r.linear("head")
        r.release()
        self._plan_runs()

    def _load_experts(self, r, L: HybridLayer, p: str, m: MoESpec, H: int) -> None:
        ops, t = self.ops, lambda name: r.tensor(p + name)
        rows = [(0, t("mlp.router"))] + ([(m.experts, t("mlp.shared.sg"))] if m.shared_gate else [])
        L.router = ops.dense_linear(r.stack(rows, m.router_rows, H))
        L.up = self._count(ops.moe_up([(t(f"mlp.e{e}.gate"), t(f"mlp.e{e}.up")) for e in range(m.experts)],
                                      self.act_dtype, m))
        L.down = r.stack([(e * H, t(f"mlp.e{e}.down")) for e in range(m.experts)], m.experts * H, m.ff)
        if m.shared_ff:
            L.shared_up = self._count(ops.moe_up([(t("mlp.shared.gate"), t("mlp.shared.up"))], self.act_dtype, m))
            L.shared_down = r.get(p + "mlp.shared.down")

    def _plan_runs(self) -> None:
        """The order of the layers' runs, and where each keeps its keys and values or its state."""
        c, caches, states = self.config, self.config.cache_layers, self.config.state_offsets
        inputs = c.input_offsets
        self.runs: List[LayerRun] = []
        for n, i in enumerate(c.layer_runs):
            s = attention_of(self.layers[i].spec)
            own = s is None or s.own_kv
            self.runs.append(LayerRun(self.layers[i], caches.get(n if own else s.kv_from, -1), states.get(n, 0),
                                      inputs.get(n, 0), c.enters_loop(n)))
        self.heads_specs = [a for a in (attention_of(L.spec) for L in self.layers) if a is not None]
        self._views: Dict[tuple, PagedHeads] = {}

    def _count(self, w: torch.Tensor) -> torch.Tensor:
        self.weight_bytes += w.numel() * w.element_size()
        return w

    # ---- buffers --------------------------------------------------------------------------------------
    def make_buffers(self, max_tokens: int, max_seqs: int, max_blocks: int, logits_rows: Optional[int] = None,
                     max_planes: int = 8, attn_splits: int = 1) -> HybridStepBuffers:
        return HybridStepBuffers(self, max_tokens, max_seqs, max_blocks, max_planes, logits_rows or max_seqs, attn_splits)

    def _heads_view(self, kv: torch.Tensor, run: LayerRun) -> PagedHeads:
        key = (kv.data_ptr(), run.cache_layer)
        v = self._views.get(key)
        if v is None:
            v = self._views[key] = PagedHeads(kv[run.cache_layer], attention_of(run.layer.spec), self.means_at)
        return v

    def attention_splits(self, seqs: int, max_len: int, most: int, sms: int) -> int:
        if not self.heads_specs:
            return 1
        span = max(min(max_len, s.chunk or max_len, s.window + s.keep_first if s.window else max_len)
                   + (max_len // s.pool if s.pool else 0) for s in self.heads_specs)
        ctas = seqs * min(s.kv_heads * ((s.heads // s.kv_heads + 15) // 16) for s in self.heads_specs)
        want = (2 * sms + ctas - 1) // ctas
        n = int(max(1, min(want, span // 128, most)))
        return 1 << (n.bit_length() - 1)

    # ---- layout of a packed pass ----------------------------------------------------------------------
    def pass_order(self, items) -> Optional[List[int]]:
        return sorted(range(len(items)), key=lambda i: len(items[i][1]) > SHORT_CHUNK)

    def stage_prefill(self, b: HybridStepBuffers, spans) -> None:
        at = b.short_rows = b.short_seqs = 0
        for s, (_, n) in enumerate(spans):
            b.h_row_seq[at: at + n] = s
            at += n
            if n <= SHORT_CHUNK:
                b.short_rows, b.short_seqs = at, s + 1
        b.row_seq[:at].copy_(b.h_row_seq[:at], non_blocking=True)

    # ---- forward --------------------------------------------------------------------------------------
    def _pass(self, b: HybridStepBuffers, kv, M: int, mode: str, num_seqs: int, max_q_len: int, attn_splits: int) -> Pass:
        decode = mode == "decode"
        planes_ok = M <= b.plane_rows
        return Pass(kv, M, num_seqs, max_q_len, None if decode else b.row_seq, None if decode else b.cu_q,
                    (M, num_seqs) if decode else (b.short_rows, b.short_seqs), planes_ok,
                    b.partial_views[0 if planes_ok else 1], attn_splits)

    def _mix(self, b: HybridStepBuffers, p: Pass, run: LayerRun) -> int:
        """The layer's mixer on ``b.xnorm``; its result is in the returned number of planes of ``p.partials``."""
        ops, L, s, M = self.ops, run.layer, run.layer.spec, p.M
        inp, planes, n_in = b.in_views[s.in_width], b.in_plane_views[s.in_width], 0
        side = b.dt_side if isinstance(s, StateSpaceSpec) else None      # step sizes stay fp32
        if p.planes_ok:
            n_in = ops.linear_partial(L.w_in, b.xnorm, M, planes)
        else:
            ops.linear(L.w_in, b.xnorm, M, inp, side=None if side is None else (s.dt_col, side))
        out = b.out_views[L.out_width]
        mixer = self._attend if isinstance(s, HeadsSpec) else self._space if side is not None else self._remember
        mixer(b, p, run, s, inp, planes, n_in, out)
        return ops.linear_partial(L.o, out, M, p.partials)

    def _attend(self, b, p: Pass, run: LayerRun, s: HeadsSpec, inp, planes, n_in: int, out) -> None:
        ops, L, M = self.ops, run.layer, p.M
        view = self._heads_view(p.kv, run)
        alone = s.pool > 0 and p.row_seq is None           # a decode step's rows leave the means of blocks themselves
        ops.heads_prep(inp, planes, n_in, view, b.slots, L, s, self.config.rms_norm_eps, M, b.positions,
                       b.block_tables if alone else None)
        if s.pool and not alone:
            ops.heads_pool(view, b.block_tables, p.row_seq, b.positions, s, M)
        rows, seqs = p.short if ops.heads_expands(s, self.act_dtype) else (M, p.num_seqs)
        if rows:
            ops.heads_attn(inp, view, b.block_tables, p.row_seq, b.positions, out, rows, s, b.attn_scratch, p.splits,
                           L.sink)
        if seqs < p.num_seqs:
            ops.heads_attn_chunks(inp, view, b.block_tables, b.cu_q, b.q_pos0, b.positions, seqs, p.num_seqs, p.max_q_len,
                                  out, s, L.sink)

    def _remember(self, b, p: Pass, run: LayerRun, s: MatrixMemorySpec, inp, planes, n_in: int, out) -> None:
        ops, L, M, eps = self.ops, run.layer, p.M, self.config.rms_norm_eps
        n_gate = 0 if n_in else ops.linear_partial(L.w_if, b.xnorm, M, b.gate_planes)
        ops.memory_prep(inp, planes, n_in, b.gate_planes, n_gate, b.gates, L, s, M)
        rows, seqs = p.short if ops.memory_expands(s, self.act_dtype) else (M, p.num_seqs)
        states = self.states.rows
        if seqs:
            ops.memory_tokens(inp, b.gates, states, run.state_at, b.state_rows, p.cu_q, L, out, seqs, M, s, eps)
        if seqs < p.num_seqs:
            ops.memory_chunks(inp, b.gates, states, run.state_at, b.state_rows, b.cu_q, L, out, seqs, p.num_seqs, rows, M, s,
                              eps, b.memory_ws)

    def _recall(self, b, p: Pass, run: LayerRun, s: GatedLinearSpec, inp, planes, n_in: int, out) -> None:
        ops, L, M, eps, states = self.ops, run.layer, p.M, self.config.rms_norm_eps, self.states.rows
        rows, seqs = p.short if ops.gated_linear_expands(s, self.act_dtype) else (M, p.num_seqs)
        decays = b.decays
        if n_in and seqs == p.num_seqs:
            decays = None                    # token by token only: the step's kernel reads the planes
        else:
            ops.gated_linear_prep(inp, planes, n_in, b.dt_side, decays, L, s, M)
        if seqs:
            ops.gated_linear_tokens(inp, planes, n_in, decays, states, run.state_at, b.state_rows, p.cu_q, L, out, seqs, M, s,
                                    eps)
        if seqs < p.num_seqs:
            ops.gated_linear_chunks(inp, decays, states, run.state_at, b.state_rows, b.cu_q, L, out, seqs, p.num_seqs,
                                    rows, M, s, eps, b.linear_ws)

    def _space(self, b, p: Pass, run: LayerRun, s: StateSpaceSpec, inp, planes, n_in: int, out) -> None:
        ops, L, M, states = self.ops, run.layer, p.M, self.states.rows
        xbc = b.xbc_views[s.conv_width]
        ops.state_space_prep(inp, planes, n_in, b.dt_side, xbc, b.dt, states, run.state_at, b.state_rows, p.row_seq, p.cu_q,
                             L, s, M, p.num_seqs)
        seqs = p.short[1] if ops.state_space_expands(s, self.act_dtype) else p.num_seqs
        if seqs:
            ops.state_space_tokens(inp, xbc, b.dt, states, run.state_at, b.state_rows, p.cu_q, L, out, seqs, M, s)
        if seqs < p.num_seqs:
            ops.state_space_chunks(inp, xbc, b.dt, states, run.state_at, b.state_rows, b.cu_q, L, out, seqs, p.num_seqs, M, s)
        ops.group_norm(out, L.out_norm, s.norm_groups, M, self.config.rms_norm_eps)

    def _mix_both(self, b: HybridStepBuffers, p: Pass, run: LayerRun, x: torch.Tensor) -> None:
        """Both mixers of a twin layer on ``x``, their results side by side in the layer's output buffer."""
        ops, L, s, M = self.ops, run.layer, run.layer.spec, p.M
        inp, planes, n_in = b.in_views[s.in_width], b.in_plane_views[s.in_width], 0
        if p.planes_ok:
            n_in = ops.linear_partial(L.w_in, x, M, planes)
        else:
            ops.linear(L.w_in, x, M, inp, side=(s.right.rank_col, b.dt_side))
        out = b.out_views[L.out_width]
        self._attend(b, p, run, s.left, inp, planes, n_in, out)
        self._recall(b, p, run, s.right, inp, planes, n_in, out[:, s.right_at:])

    def _feed(self, b: HybridStepBuffers, p: Pass, L: HybridLayer):
        """The layer's feed-forward on ``b.xnorm``: (planes of ``p.partials``, the experts' rows or None)."""
        if L.moe is not None:
            return 0, self.ops.moe(L, b.xnorm, p.M, b.moe_ws)
        act = b.act_views[L.ff.ff]
        if L.ff.gated:
            self.ops.linear_glu(L.up_w, b.xnorm, p.M, act, L.ff.activation, b.glu)
        else:
            self.ops.linear_act(L.up_w, b.xnorm, p.M, act, L.ff.activation)
        return self.ops.linear_partial(L.down_w, act, p.M, p.partials), None

    def _logits(self, b: HybridStepBuffers, rows: int) -> None:
        torch.index_select(b.xnorm, 0, b.logit_rows[:rows], out=b.xsel[:rows])
        self.ops.linear_f32(self.lm_head, b.xsel, rows, b.logits)

    def forward(self, b: HybridStepBuffers, kv: torch.Tensor, M: int, mode: str, num_seqs: int, max_q_len: int = 1,
                n_logit_rows: int = 0, attn_splits: int = 1) -> None:
        ops, eps = self.ops, self.config.rms_norm_eps
        p = self._pass(b, kv, M, mode, num_seqs, max_q_len, attn_splits)
        last_token = self.states.last_token if self.states is not None else None
        ops.embed_design(self.embed_design, b.ids, b.positions, p.row_seq, p.cu_q, b.state_rows, last_token, b.residual,
                         b.xnorm, M, num_seqs, eps)
        for run in self.runs:
            L, last = run.layer, run is self.runs[-1]
            planes = self._mix(b, p, run)
            ops.post_norm(b.residual, p.partials, planes, None, L.norm1, self.norm if last and L.ff is None else None,
                          b.xnorm, M, eps)
            if L.ff is not None:
                planes, slots = self._feed(b, p, L)
                ops.post_norm(b.residual, p.partials, planes, slots, L.norm2, self.norm if last else None, b.xnorm, M, eps)
        if n_logit_rows:
            self._logits(b, n_logit_rows)
