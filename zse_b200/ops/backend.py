"""The op set the decoder is written against, with two implementations.

``CudaOps``  - the hand-written sm_100a kernels in ``libzse_b200.so`` (fails loudly when the library is missing).
``TorchOps`` - ``ops.reference`` on any device; runs the engine on CPU-only machines and serves as the oracle.

Both work in place on caller-owned buffers so that a step allocates nothing and can be captured in a CUDA graph.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Optional

import numpy as np
import torch

from ..format.layer_specs import GLU
from . import reference as ref

EPI_F16, EPI_SWIGLU, EPI_PARTIAL, EPI_RELU2 = 0, 1, 2, 5


@dataclass
class LinearWeight:
    """One (possibly fused / sharded) linear layer ready for the device."""
    kind: str                  # "w4t" tiled INT4 | "w8t" tiled INT8 | "f16" dense fp16 | "ref" fp32 (TorchOps)
    N: int                     # output rows as the kernel sees them (gate+up counted together for swiglu)
    K: int
    data: torch.Tensor
    bias: Optional[torch.Tensor] = None
    swiglu: bool = False       # rows are gate/up interleaved in 64-row halves (w4t) or [gate; up] stacked (f16/ref)
    nbytes: int = 0


def _np_to_dev(a: np.ndarray, device) -> torch.Tensor:
    """Host array -> tensor on ``device``.  Arrays that view a read-only file mapping are copied on the CPU path so
    the tensor never aliases the mapping."""
    if isinstance(a, torch.Tensor):
        return a.to(device)
    a = np.ascontiguousarray(a)
    if torch.device(device).type == "cpu" or not a.flags.writeable:
        a = np.array(a, copy=True)
    return torch.from_numpy(a).to(device, non_blocking=False)


np_to_dev = _np_to_dev


class TorchOps:
    name = "torch"

    def __init__(self, device="cpu"):
        self.device = torch.device(device)
        self.status = None

    # ---- weights --------------------------------------------------------------------------------------
    def make_linear(self, parts, K: int, group_size: int, bias=None, swiglu: bool = False) -> LinearWeight:
        """``parts``: list of dicts {dtype, data(np), scales(np), zeros(np), shape, row_major_group_ok}; rows are
        concatenated in order (q,k,v or gate,up)."""
        ws = []
        for p in parts:
            ws.append(_dense_f32(p, group_size, self.device))
        w = torch.cat(ws, dim=0) if len(ws) > 1 else ws[0]
        b = None if bias is None else _np_to_dev(bias, self.device)
        return LinearWeight("ref", w.shape[0], K, w, b, swiglu, w.numel() * 4)

    def check(self):
        pass

    # ---- ops ------------------------------------------------------------------------------------------
    def linear(self, w: LinearWeight, x, M, out, x_cap=None, gather=None, side=None):
        """``side``: (first column, fp32 buffer): columns from there on go to the buffer [M, N - first] instead."""
        if side is not None:
            y = x[:M].float() @ w.data.T
            out[:M, : side[0]] = y[:, : side[0]]
            side[1].view(-1)[: M * (w.N - side[0])].view(M, -1).copy_(y[:, side[0]:])
        elif out.dtype != torch.float16:
            out[:M, : w.N] = x[:M].float() @ w.data.T
        else:
            out[:M, : w.N] = ref.linear(x[:M], w.data, w.bias)

    def linear_swiglu(self, w: LinearWeight, x, M, out, x_cap=None, gelu=False, gather=None):
        y = x[:M].float() @ w.data.T
        half = w.N // 2
        out[:M, :half] = ref.swiglu(y[:, :half], y[:, half:], gelu)

    def linear_partial(self, w: LinearWeight, x, M, partials, k_split=1, x_cap=None) -> int:
        # planes are laid out [plane][M rows][N] with the *actual* M as the row count, like the CUDA kernels do
        partials.view(-1)[: M * w.N].view(M, w.N).copy_(x[:M].float() @ w.data.T)
        return 1

    def embedding(self, table, ids, out, M, scale=1.0, copy=None):
        """out (fp32) = scaled rows of the table; ``copy``: a second place for them, in the activations' type."""
        out[:M] = table[ids[:M].long()].float() * scale
        if copy is not None:
            copy[:M] = out[:M]

    def add_rmsnorm(self, residual, partials, n_partials, add_f16, weight, out, M, eps):
        H = residual.shape[1]
        if n_partials:
            residual[:M] += partials.view(-1)[: n_partials * M * H].view(n_partials, M, H).sum(0)
        if add_f16 is not None:
            residual[:M] += add_f16[:M].float()
        if out is not None:
            out[:M] = ref.rmsnorm(residual[:M], weight, eps)

    def qkv_rope_fused_ok(self, w: LinearWeight, M: int, hd: int, kv_layer) -> bool:
        """Whether ``qkv_rope_fused`` takes this pass (the torch implementation never does: it has the unfused ops)."""
        return False

    def residual_norm_fused_ok(self, w: LinearWeight, M: int, H: int) -> bool:
        """Whether ``linear_residual_norm`` (projection + residual add + RMSNorm in one kernel) takes this layer."""
        return False

    def rope_kv_write(self, qkv, kv_layer, positions, slots, inv_freq, M, nh, nkv, hd, block_size, planes=None,
                      n_planes=0, bias=None):
        if planes is not None:
            ld = qkv.shape[1]
            full = planes.view(-1)[: n_planes * M * ld].view(n_planes, M, ld).sum(0)
            if bias is not None:
                full = full + bias.float()
            qkv[:M] = full.clamp(-65504, 65504).to(qkv.dtype)
        ref.rope_kv_write(qkv[:M], kv_layer, positions[:M], slots[:M], inv_freq, nh, nkv, hd, block_size)

    def attn_decode(self, qkv, kv_layer, block_tables, seq_lens, out, S, nh, nkv, hd, block_size, scale, scratch=None,
                    num_splits=1, softcap=0.0, window=0):
        out[:S, : nh * hd] = ref.attn_decode(qkv[:S, : nh * hd], kv_layer, block_tables[:S], seq_lens[:S], nh, nkv, hd,
                                             block_size, scale, softcap, window)

    def attn_prefill(self, qkv, kv_layer, block_tables, cu_q, q_pos0, out, num_seqs, total_q, max_q_len, nh, nkv, hd,
                     block_size, scale, softcap=0.0, window=0):
        out[:total_q, : nh * hd] = ref.attn_prefill(qkv[:total_q, : nh * hd], kv_layer, block_tables[:num_seqs],
                                                    cu_q[: num_seqs + 1], q_pos0[:num_seqs], nh, nkv, hd, block_size,
                                                    scale, softcap, window)

    # ---- latent attention and routed feed-forward -----------------------------------------------------
    # (activations and cache at the model's own width: bfloat16 or fp32)
    def dense(self, t: torch.Tensor, dtype) -> torch.Tensor:
        """Weights of the ops below, as this back end keeps them."""
        return t.to(self.device, torch.float32)

    def dense_linear(self, w: torch.Tensor) -> LinearWeight:
        """``w`` [N, K] as ``dense`` returned it."""
        kind = {torch.bfloat16: "bf16", torch.float32: "f32"}[w.dtype] if self.name == "cuda" else "ref"
        return LinearWeight(kind, w.shape[0], w.shape[1], w, None, False, w.numel() * w.element_size())

    def linear_f32(self, w: LinearWeight, x, M, out):
        """out [M, N] fp32, one plane."""
        out[:M, : w.N] = x[:M].float() @ w.data.T

    def add_norm(self, residual, partials, n_partials, slots, weight, out, M, eps, scale=None, offset=0.0, replace=False):
        """residual += scale * (the planes' sum + the sum over a row's ``slots`` [M, n, H]), or the sum alone with
        ``replace``; out = RMSNorm(residual) * (weight + offset), or the residual itself without a weight."""
        H = residual.shape[1]
        y = torch.zeros(M, H, device=residual.device)
        if n_partials:
            y += partials.view(-1)[: n_partials * M * H].view(n_partials, M, H).sum(0)
        if slots is not None:
            y += slots[:M].float().sum(1)
        if scale is not None:
            y *= scale.float()
        residual[:M] = y if replace else residual[:M] + y
        out[:M] = residual[:M] if weight is None else ref.rmsnorm_f32(residual[:M], weight, eps, offset)

    def latent_prep(self, inp, planes, n_planes, rows, positions, slots, freqs, norm_w, spec, eps, M):
        if n_planes:
            ld = inp.shape[1]
            inp[:M] = planes.view(-1)[: n_planes * M * ld].view(n_planes, M, ld).sum(0)
        ref.latent_prep(inp[:M], rows, positions[:M], slots[:M], freqs, norm_w, spec, eps)

    def latent_attn(self, inp, L, rows, block_tables, row_seq, positions, q_lat, o_lat, out, M, spec, scratch, num_splits):
        """Rows [0, M) attend to the cached rows themselves: queries go through W_uk, results through W_uv and the gate.
        Row t belongs to sequence ``row_seq[t]`` (None: t)."""
        H, vd = spec.heads, spec.vdim
        q = ref.latent_absorb(inp[:M], L.uk, spec).to(inp.dtype)
        o = torch.zeros(M, H, spec.kv_rank, dtype=inp.dtype, device=inp.device)
        for t in range(M):
            s = t if row_seq is None else int(row_seq[t])
            o[t] = ref.latent_attn_token(q[t], rows, block_tables[s], int(positions[t]), spec)
        y = torch.einsum("thc,hvc->thv", o.float(), L.uv.view(H, vd, spec.kv_rank)).reshape(M, H * vd)
        self._gate(y, inp[:M], out[:M], spec)

    def latent_attn_chunks(self, inp, L, rows, block_tables, cu_q, q_pos0, ctx_off, group, ctx, out, spec):
        """Rows of the sequences ``group.first .. group.last - 1`` attend to keys and values expanded from the cached rows
        their windows reach; ``ctx``: scratch (c, kr, kvx), ``ctx_off[s]``: sequence s's first row in it."""
        bs = rows.shape[1]
        kr, r = spec.kv_rank, spec.rot_dim
        for s in range(group.first, group.last):
            a, e, p0 = int(cu_q[s]), int(cu_q[s + 1]), int(q_pos0[s])
            lo = max(0, p0 + 1 - spec.window) if spec.window > 0 else 0
            pos = torch.arange(lo, p0 + e - a, device=rows.device)
            blk = block_tables[s][pos // bs].long()
            got = rows[blk.clamp_min(0), pos % bs]
            c = got[:, :kr].contiguous()
            kvx = (c.float() @ L.ukv.data.T).to(inp.dtype)
            y = ref.latent_attn_chunk(inp[a:e], c, got[:, kr: kr + r], blk >= 0, kvx,
                                      torch.arange(p0, p0 + e - a, device=rows.device), pos, spec)
            self._gate(y.reshape(e - a, -1), inp[a:e], out[a:e], spec)

    @staticmethod
    def _gate(y, inp, out, spec):
        w = spec.heads * spec.vdim
        if spec.gated:
            y = y * torch.sigmoid(inp[:, spec.gate_col: spec.gate_col + w].float())
        out[:, :w] = y

    def moe(self, L, x, M, ws):
        """The routed feed-forward of rows [0, M): returns ``slots`` [M, top (+1), H], to be summed."""
        m, H = L.moe, x.shape[1]
        xs = x[:M].float()
        z = xs @ L.router.data.T
        ids, w = ref.route(z[:, : m.experts], m)
        slots = torch.zeros(M, m.top + (m.shared_ff > 0), H, dtype=torch.float32, device=x.device)

        def act(t, up, ff, limit, score=None):
            y = t @ up.T
            if score is not None and m.weigh == "input":
                y = score[:, None] * y
            return (ref.glu(m.activation, y[:, :ff], y[:, ff:], limit) if m.gated else ref.gelu_exact(y)).to(x.dtype).float()

        up, down = L.up.view(m.experts, -1, H), L.down.view(m.experts, H, m.ff)
        for e in torch.unique(ids).tolist():
            t, k = torch.where(ids == e)
            y = act(xs[t], up[e], m.ff, m.limit, w[t, k]) @ down[e].T
            slots[t, k] = w[t, k, None] * y if m.weigh == "output" else y
        if m.shared_ff:
            y = act(xs, L.shared_up, m.shared_ff, m.shared_limit) @ L.shared_down.T
            slots[:, m.top] = torch.sigmoid(z[:, m.experts:]) * y if m.shared_gate else y
        return slots

    def moe_up(self, pairs, dtype, m=None):
        """Up products of gated experts from their (gate, up) matrices [ff, H], all experts in one tensor."""
        return self.dense(torch.cat([t for pair in pairs for t in pair]), dtype)

    def latent_expands(self, spec, dtype) -> bool:
        """Whether long chunks of such a layer take ``latent_attn_chunks``."""
        return True

    def moe_workspace(self, specs, H: int, max_tokens: int, dtype):
        return None

    # ---- designs of attention over heads, matrix memories and post-norms ---------------------------------
    def embed_design(self, E, ids, positions, row_seq, cu_q, state_rows, last_token, residual, out, M, S, eps):
        """residual = norm(scaled embedding + what the design adds to it), in fp32, and ``out`` the same for the products.
        ``cu_q``: first row of every sequence (None: a row each), ``row_seq``: the rows' sequences.  The last token of every
        sequence goes to ``last_token[state_rows[1, s]]``."""
        cu = list(range(S + 1)) if cu_q is None else [int(v) for v in cu_q[: S + 1]]
        t = ids[:M].long()
        x = E.table[t].float() * E.scale
        if E.bigram is not None:
            prev = ref.previous_tokens(t, cu, state_rows, last_token)
            x = x + E.bigram[torch.where(prev < 0, E.buckets, (prev * E.mul_prev + t * E.mul_cur) % E.buckets)].float()
            for s in range(S):
                if int(state_rows[1, s]) >= 0:
                    last_token[int(state_rows[1, s])] = t[cu[s + 1] - 1].to(last_token.dtype)
        x = x + ref.sinusoid(positions[:M], x.shape[1], E.base)
        residual[:M] = ref.rmsnorm_f32(x, E.norm, eps)
        out[:M] = residual[:M]

    def post_norm(self, residual, partials, n_partials, slots, weight, next_weight, out, M, eps):
        """residual += RMSNorm(the planes' sum + the sum over a row's ``slots``) * weight; out = residual, or its RMSNorm
        with ``next_weight``."""
        H = residual.shape[1]
        y = torch.zeros(M, H, device=residual.device)
        if n_partials:
            y += partials.view(-1)[: n_partials * M * H].view(n_partials, M, H).sum(0)
        if slots is not None:
            y += slots[:M].float().sum(1)
        residual[:M] += ref.rmsnorm_f32(y, weight, eps)
        out[:M] = residual[:M] if next_weight is None else ref.rmsnorm_f32(residual[:M], next_weight, eps)

    def linear_act(self, w: LinearWeight, x, M, out, activation: str):
        """out = activation(x W^T) in the activations' type."""
        out[:M, : w.N] = {"relu2": ref.relu2}[activation](x[:M].float() @ w.data.T)

    def glu_linear(self, gate: torch.Tensor, up: torch.Tensor, dtype) -> LinearWeight:
        """The two up products of a gated dense feed-forward as one weight for ``linear_glu``."""
        return self.dense_linear(self.dense(torch.cat([gate, up]), dtype))

    def linear_glu(self, w: LinearWeight, x, M, out, activation: str, tmp=None):
        """out [M, ff] = glu(x W_gate^T, x W_up^T) in the activations' type; ``tmp``: room for both products."""
        y, ff = x[:M].float() @ w.data.T, out.shape[1]
        out[:M] = ref.glu(activation, y[:, :ff], y[:, ff:])

    def glu_expands(self, ff: int, H: int, dtype) -> bool:
        """Whether ``linear_glu`` needs its ``tmp``."""
        return False

    def heads_expands(self, spec, dtype) -> bool:
        """Whether long chunks of such a layer take ``heads_attn_chunks``."""
        return True

    def rotation(self, dims: int, base: float, factor: float = 1.0):
        """Frequencies of the pairs (2i, 2i + 1), base^(-2i / dims) / factor per position, in this back end's form."""
        if not dims:
            return None
        return base ** (-torch.arange(0, dims, 2, dtype=torch.float64, device=self.device) / dims) / factor

    def heads_prep(self, inp, planes, n_planes, kv, slots, L, spec, eps, M, positions=None, block_tables=None):
        if n_planes:
            ld, w = inp.shape[1], spec.in_width
            inp[:M, :w] = planes.view(-1)[: n_planes * M * ld].view(n_planes, M, ld)[..., :w].sum(0)
        ref.heads_prep(inp[:M], kv.k if kv else None, kv.v if kv else None, slots[:M], spec, L.q_norm, L.k_norm, eps,
                       None if positions is None else positions[:M].long(), getattr(L, "bias", None),
                       getattr(L, "freqs", None), getattr(L, "temp", None))
        if spec.pool and block_tables is not None:
            self.heads_pool(kv, block_tables, None, positions, spec, M)

    def heads_pool(self, kv, block_tables, row_seq, positions, spec, M):
        """Means of the blocks of ``spec.pool`` tokens that rows [0, M) complete, from the cached keys and values into the cache.
        Row t belongs to sequence ``row_seq[t]`` (None: t)."""
        for t in range(M):
            p, s = int(positions[t]), t if row_seq is None else int(row_seq[t])
            if (p + 1) % spec.pool == 0:
                for cache in (kv.k, kv.v):
                    ref.pool_rows(cache, block_tables[s], kv.means_at, p // spec.pool, spec.pool)

    def heads_attn(self, inp, kv, block_tables, row_seq, positions, out, M, spec, scratch, num_splits, sink=None):
        """Rows [0, M) against the cached keys and values; row t belongs to sequence ``row_seq[t]`` (None: t)."""
        for t in range(M):
            s = t if row_seq is None else int(row_seq[t])
            self._heads_rows(inp, kv, block_tables[s], positions, out, t, t + 1, spec, sink)

    def heads_attn_chunks(self, inp, kv, block_tables, cu_q, q_pos0, positions, first, last, max_q, out, spec, sink=None):
        """Rows of the sequences ``first .. last - 1``."""
        for s in range(first, last):
            self._heads_rows(inp, kv, block_tables[s], positions, out, int(cu_q[s]), int(cu_q[s + 1]), spec, sink)

    @staticmethod
    def _heads_rows(inp, kv, table, positions, out, a, e, spec, sink=None):
        H, w = spec.heads, spec.heads * spec.vdim
        y = ref.heads_attn(inp[a:e, : H * spec.dim].reshape(e - a, H, spec.dim), positions[a:e].long(), kv.k, kv.v, table,
                           spec, sink, getattr(kv, "means_at", 0))
        if spec.gated:
            y = y * torch.sigmoid(inp[a:e, spec.gate_col: spec.gate_col + spec.gate_width].float()).view(e - a, H, -1)
        out[a:e, :w] = (spec.out_scale * y).reshape(e - a, w)

    def memory_expands(self, spec, dtype) -> bool:
        """Whether long chunks of such a layer take ``memory_chunks``."""
        return False

    def memory_workspace(self, specs, max_tokens: int):
        return None

    def memory_prep(self, inp, planes, n_planes, gate_planes, n_gate_planes, gates, L, spec, M):
        """Sums the split-K planes of the input projection and takes the logarithms of the gates, ``gates`` [M, 2 * heads].
        With ``n_planes`` 0 ``inp`` is complete and the gates' pre-activations are in ``gate_planes`` [n, M, 2 * heads]."""
        g = 2 * spec.heads
        if n_planes:
            ld = inp.shape[1]
            full = planes.view(-1)[: n_planes * M * ld].view(n_planes, M, ld).sum(0)
            inp[:M] = full
            z = full[:, spec.if_col: spec.if_col + g]
        else:
            z = gate_planes.view(-1)[: n_gate_planes * M * g].view(n_gate_planes, M, g).sum(0)
        gates.view(-1)[: M * g].view(M, g).copy_(ref.memory_gates(z, L.if_bias, spec.gate_cap))

    def memory_tokens(self, inp, gates, states, at, state_rows, cu_q, L, out, S, M, spec, eps):
        """Sequences [0, S), token by token: memory, read-out, head norm and output gate.  ``states``: the state pool's rows,
        ``at``: where the layer's part of a row begins; ``cu_q``: first row of every sequence (None: a row each)."""
        H, d, vd = spec.heads, spec.dim, spec.vdim
        g = gates.view(-1)[: M * 2 * H].view(M, 2 * H)
        for s in range(S):
            a, e = (s, s + 1) if cu_q is None else (int(cu_q[s]), int(cu_q[s + 1]))
            read, write = int(state_rows[0, s]), int(state_rows[1, s])
            row = states[read, at: at + spec.state_floats].clone() if read >= 0 else torch.zeros(
                spec.state_floats, device=inp.device)
            x = inp[a:e].float()
            y = ref.memory_tokens(x[:, : H * d].reshape(-1, H, d) * d ** -0.5,
                                  x[:, spec.k_col: spec.k_col + H * d].reshape(-1, H, d),
                                  x[:, spec.v_col: spec.v_col + H * vd].reshape(-1, H, vd), g[a:e, :H], g[a:e, H:],
                                  row[: H * d * vd].view(H, d, vd), row[spec.sum_at: spec.sum_at + H * d].view(H, d),
                                  row[spec.max_at: spec.max_at + H])
            if write >= 0:
                states[write, at: at + spec.state_floats] = row
            y = ref.rmsnorm_f32(y, L.head_norm.view(H, vd), eps).reshape(e - a, H * vd)
            out[a:e, : H * vd] = y * torch.sigmoid(x[:, spec.gate_col: spec.gate_col + H * vd])

    # ---- state space (Mamba-2) --------------------------------------------------------------------------------------------
    def state_space_expands(self, spec, dtype) -> bool:
        """Whether long chunks of such a layer take ``state_space_chunks``."""
        return False

    def state_space_prep(self, inp, planes, n_planes, side, xbc, dt, states, at, state_rows, row_seq, cu_q, L, spec, M, S):
        """Sums the split-K planes of the input projection [z | x | B | C | step sizes], passes x, B and C through the
        convolution and silu into ``xbc`` and takes softplus of the biased step sizes, ``dt`` [M, heads].  Without planes
        ``inp`` is complete; ``side``: the step sizes before bias and softplus in fp32 (None: those of ``inp``)."""
        if n_planes:
            ld = inp.shape[1]
            full = planes.view(-1)[: n_planes * M * ld].view(n_planes, M, ld).sum(0)
            inp[:M] = full
        else:
            full = inp[:M].float()
        H, w = spec.heads, spec.conv_width
        z = full[:, spec.dt_col: spec.dt_col + H]
        if not n_planes and side is not None:
            z = side.view(-1)[: M * (spec.in_width - spec.dt_col)].view(M, -1)[:, :H]
        dt.view(-1)[: M * H].view(M, H).copy_(torch.nn.functional.softplus(z + L.dt_bias, threshold=40))
        tail = slice(at + spec.conv_at, at + spec.conv_at + (spec.conv - 1) * w)
        for s in range(S):
            a, e = (s, s + 1) if cu_q is None else (int(cu_q[s]), int(cu_q[s + 1]))
            read, write = int(state_rows[0, s]), int(state_rows[1, s])
            before = states[read, tail].view(spec.conv - 1, w) if read >= 0 else torch.zeros(spec.conv - 1, w,
                                                                                             device=inp.device)
            y, last = ref.conv_tokens(full[a:e, spec.x_col: spec.dt_col], before, L.conv_w, L.conv_b)
            xbc[a:e] = y
            if write >= 0:
                states[write, tail] = last.reshape(-1)

    def state_space_tokens(self, inp, xbc, dt, states, at, state_rows, cu_q, L, out, S, M, spec):
        """Sequences [0, S), token by token: memory, read-out, and the gate silu(z).  ``states``: the state pool's rows,
        ``at``: where the layer's part of a row begins; ``cu_q``: first row of every sequence (None: a row each)."""
        H, v, G, n = spec.heads, spec.vdim, spec.groups, spec.state
        d = dt.view(-1)[: M * H].view(M, H)
        for s in range(S):
            a, e = (s, s + 1) if cu_q is None else (int(cu_q[s]), int(cu_q[s + 1]))
            read, write = int(state_rows[0, s]), int(state_rows[1, s])
            mem = states[read, at: at + H * n * v].clone() if read >= 0 else torch.zeros(H * n * v, device=inp.device)
            x = xbc[a:e].float()
            y = ref.state_space_tokens(x[:, : H * v].view(-1, H, v), x[:, spec.b_at: spec.b_at + G * n].view(-1, G, n),
                                       x[:, spec.c_at: spec.c_at + G * n].view(-1, G, n), d[a:e], L.neg_a, L.D,
                                       mem.view(H, n, v))
            if write >= 0:
                states[write, at: at + H * n * v] = mem
            out[a:e, : H * v] = y.reshape(e - a, H * v) * torch.nn.functional.silu(inp[a:e, : H * v].float())

    # ---- gated linear attention -------------------------------------------------------------------------------------------
    def gated_linear_expands(self, spec, dtype) -> bool:
        """Whether long chunks of such a layer take ``gated_linear_chunks``."""
        return False

    def gated_linear_workspace(self, specs, max_tokens: int):
        return None

    def gated_linear_prep(self, inp, planes, n_planes, side, decays, L, spec, M):
        """Sums the split-K planes of its part of the input projection and makes the logarithms of the decays, ``decays``
        [M, heads * dim].  Without planes ``inp`` is complete; ``side``: the decays' inner vectors in fp32 (None: those of
        ``inp``)."""
        ld = inp.shape[1]
        if n_planes:
            full = planes.view(-1)[: n_planes * M * ld].view(n_planes, M, ld).sum(0)
            inp[:M, spec.col: spec.in_width] = full[:, spec.col: spec.in_width]
            u = full[:, spec.rank_col: spec.rank_col + spec.rank]
        elif side is not None:
            u = side.view(-1)[: M * (ld - spec.rank_col)].view(M, -1)[:, : spec.rank]
        else:
            u = inp[:M, spec.rank_col: spec.rank_col + spec.rank]
        w = spec.heads * spec.dim
        decays.view(-1)[: M * w].view(M, w).copy_(ref.log_decays(u, L.decay_w, L.decay_b, spec.tau))

    def gated_linear_tokens(self, inp, planes, n_planes, decays, states, at, state_rows, cu_q, L, out, S, M, spec, eps):
        """Sequences [0, S), token by token: memory, read-out, head norm and output gate.  ``states``: the state pool's rows,
        ``at``: where the layer's part of a row begins; ``cu_q``: first row of every sequence (None: a row each).  With
        ``decays`` None the rows of ``inp`` are still in the planes and the decays are made on the way."""
        if decays is None:
            decays = torch.empty(M * spec.heads * spec.dim, device=inp.device)
            self.gated_linear_prep(inp, planes, n_planes, None, decays, L, spec, M)
        H, d, vd = spec.heads, spec.dim, spec.vdim
        g = decays.view(-1)[: M * H * d].view(M, H, d)
        n = H * d * vd
        for s in range(S):
            a, e = (s, s + 1) if cu_q is None else (int(cu_q[s]), int(cu_q[s + 1]))
            read, write = int(state_rows[0, s]), int(state_rows[1, s])
            mem = states[read, at: at + n].clone() if read >= 0 else torch.zeros(n, device=inp.device)
            x = inp[a:e].float()
            y = ref.gated_linear_tokens(x[:, spec.col: spec.col + H * d].reshape(-1, H, d) * d ** -0.5,
                                        x[:, spec.k_col: spec.k_col + H * d].reshape(-1, H, d),
                                        x[:, spec.v_col: spec.v_col + H * vd].reshape(-1, H, vd), g[a:e], mem.view(H, d, vd))
            if write >= 0:
                states[write, at: at + n] = mem
            y = ref.rmsnorm_f32(y, L.head_norm, eps).reshape(e - a, H * vd) * spec.out_scale
            out[a:e, : H * vd] = y * torch.nn.functional.silu(x[:, spec.gate_col: spec.gate_col + H * vd])

    def add_norm_conv(self, residual, partials, n_partials, weight, out, conv_w, conv_out, states, at, state_rows, row_seq,
                      cu_q, M, S, eps):
        """residual += the planes' sum; out = RMSNorm(residual) * weight; conv_out = out plus its causal convolution along the
        sequence, ``conv_w`` [taps, H].  ``states``: the state pool's rows, which hold a sequence's last taps - 1 rows of
        ``out`` from ``at`` on."""
        H, taps = residual.shape[1], conv_w.shape[0]
        self.add_norm(residual, partials, n_partials, None, weight, out, M, eps)
        tail = slice(at, at + (taps - 1) * H)
        for s in range(S):
            a, e = (s, s + 1) if cu_q is None else (int(cu_q[s]), int(cu_q[s + 1]))
            read, write = int(state_rows[0, s]), int(state_rows[1, s])
            before = states[read, tail].view(taps - 1, H) if read >= 0 else torch.zeros(taps - 1, H, device=out.device)
            y, last = ref.conv_inputs(out[a:e].float(), before, conv_w)
            conv_out[a:e] = y
            if write >= 0:
                states[write, tail] = last.reshape(-1)

    def group_norm(self, x, weight, parts: int, M, eps):
        """Rows of ``x`` normed in place in ``parts`` equal parts, times ``weight``."""
        y = x[:M].float().view(M, parts, -1)
        x[:M] = ref.rmsnorm_f32(y, None, eps).view(M, -1) * weight.float()

    def logits_finish(self, logits, M, scale, cap):
        """logits <- cap * tanh(scale * logits / cap) in place (cap 0: only scaled)."""
        z = logits[:M] * scale
        logits[:M] = cap * torch.tanh(z / cap) if cap > 0 else z

    # ---- Gemma-family ops ---------------------------------------------------------------------------
    def headnorm_rope_kv_write(self, qkv, kv_layer, positions, slots, freqs, q_norm_w, k_norm_w, norm_v, k_is_v, eps,
                               M, nh, nkv, hd, block_size):
        ref.headnorm_rope_kv_write(qkv[:M], kv_layer, positions[:M], slots[:M], freqs, q_norm_w, k_norm_w, norm_v,
                                   k_is_v, eps, nh, nkv, hd, block_size)

    def norm_add_rmsnorm(self, x, w_post, residual, scalar, w_next, out, M, eps):
        y = ref.norm_add_rmsnorm(x[:M], w_post, residual[:M], scalar, w_next, eps)
        if out is not None and y is not None:
            out[:M] = y

    def glu(self, gate_up, out, M, I, gelu=False):
        out[:M, :I] = ref.swiglu(gate_up[:M, :I], gate_up[:M, I: 2 * I], gelu)

    def softcap(self, logits, M, cap):
        logits[:M] = ref.softcap(logits[:M], cap)

    def argmax(self, logits, out, M):
        out[:M] = logits[:M].float().argmax(dim=-1).to(out.dtype)

    def sample(self, logits, out, M, temperature, top_k, top_p, seeds, step):
        for r in range(M):
            t = float(temperature[r])
            if t <= 0 or int(top_k[r]) == 1:
                out[r] = int(logits[r].float().argmax())
                continue
            p = ref.filtered_probs(logits[r], t, int(top_k[r]), float(top_p[r]))
            # the row's own seed and nothing about its place in the batch (same rule as the CUDA kernel)
            g = torch.Generator(device="cpu").manual_seed((int(seeds[r]) * 1000003 + int(step) * 7919) % (2 ** 63))
            out[r] = int(torch.multinomial(p.cpu(), 1, generator=g))

    def apply_repetition_penalty(self, logits, rows, tokens, counts, n, penalty):
        for i in range(n):
            r, t, c = int(rows[i]), int(tokens[i]), int(counts[i])
            pen = float(penalty[r])
            if c > 0 and pen != 1.0:
                f = pen ** (1.0 + float(np.log2(c)))
                v = float(logits[r, t])
                logits[r, t] = v / f if v > 0 else v * f

    def lora_apply(self, x, a_table, b_table, ids, scales, y, M, K, N, rank, tmp=None, y_col0=0):
        for t in range(M):
            a = int(ids[t])
            if a >= 0:
                d = ref.lora_delta(x[t: t + 1, :K], a_table[a], b_table[a], float(scales[a]))
                y[t, y_col0: y_col0 + N] = (y[t, y_col0: y_col0 + N].float() + d[0]).clamp(-65504, 65504).to(y.dtype)


def _dense_f32(p: dict, group_size: int, device) -> torch.Tensor:
    shape = tuple(p["shape"])
    if p["dtype"] == "float16":
        return _np_to_dev(p["data"], device).reshape(shape).float()
    if p["dtype"] == "int8":
        return ref.dequant_int8(_np_to_dev(p["data"], device), _np_to_dev(p["scales"], device), shape, group_size)
    if "flat_data" in p:   # a column slice of a tensor whose flat groups straddle rows: dequantise whole, slice
        full = ref.dequant_int4(_np_to_dev(p["flat_data"], device), _np_to_dev(p["flat_scales"], device),
                                _np_to_dev(p["flat_zeros"], device), p["flat_shape"], group_size)
        (r0, r1), (c0, c1) = p["rows"], p["cols"]
        return full[r0:r1, c0:c1].contiguous()
    return ref.dequant_int4(_np_to_dev(p["data"], device), _np_to_dev(p["scales"], device),
                            _np_to_dev(p["zeros"], device), shape, group_size)


def _dp(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def moe_tensor_cores(m, H: int, dtype) -> bool:
    """Whether the experts' products take the grouped tensor-core kernel (rows of whole 16-byte pieces)."""
    return dtype == torch.bfloat16 and H % 8 == 0 and m.ff % 8 == 0 and m.shared_ff % 8 == 0


class MoeWorkspace:
    """Device tables and activations of the routed feed-forward, shared by all layers of a model."""
    F32_ROWS = 1024

    def __init__(self, specs, H: int, max_tokens: int, dtype, device):
        z = lambda n, dt: torch.zeros(max(1, n), dtype=dt, device=device)
        i32, f32 = torch.int32, torch.float32
        E, top = max(s.experts for s in specs), max(s.top for s in specs)
        slots = max_tokens * top
        per = max(s.top + (s.shared_ff > 0) for s in specs)
        self.counts, self.first_row, self.n_tiles = z(E, i32), z(E, i32), z(1, i32)
        self.slot_expert, self.slot_rank, self.slot_score = z(slots, i32), z(slots, i32), z(slots, f32)
        self.row_score, self.out_rows = z(slots, f32), z(slots, i32)
        self.shared_score = z(max_tokens, f32)
        self.tiles = z((E + slots // 16 + 1) * 4, i32)
        self.xs = z(slots * H, dtype)
        self.act = z(max_tokens * max(s.top * s.ff for s in specs), dtype)
        self.act_shared = z(max_tokens * max(s.shared_ff for s in specs), dtype)
        self.y = z(max(min(max_tokens, self.F32_ROWS) * 4, max_tokens * dtype.itemsize) * per * H, torch.uint8)
        # router logits in split-K planes: few columns, so the reduction is what fills the GPU
        widths = {s.router_rows for s in specs}
        self.router = z(8 * max_tokens * max(widths), f32)
        self.router_views = {w: self.router[: 8 * max_tokens * w].view(8, max_tokens * w) for w in widths}
        # gate and up products of gated experts that do not take the tensor-core kernel
        self.glu = z(2 * max_tokens * max([0] + [max(s.top * s.ff, s.shared_ff) for s in specs
                                                 if s.gated and not moe_tensor_cores(s, H, dtype)]), dtype)


class CudaOps(TorchOps):
    name = "cuda"

    def __init__(self, device="cuda", group: Optional[str] = None):
        """``group``: the kernels the model needs (``build.GROUPS``); None = the whole library."""
        from . import native
        if not torch.cuda.is_available():
            raise RuntimeError("CudaOps needs a CUDA device")
        self.n = native
        native.load(build_if_missing=True, group=group, whole=group is None)
        self.device = torch.device(device)
        self.status = native.Status(self.device)
        self.sm_count = torch.cuda.get_device_properties(self.device).multi_processor_count
        # decode-sized passes (<= 64 tokens) of the INT4 layers: bit 0 = gate/up + SwiGLU, bit 1 = fused QKV + bias +
        # RoPE + KV-cache write, bit 2 = every other INT4 linear, through the persistent kernel (csrc/gemm_w4_dec.cu)
        from ..utils import env
        self.dec_mode = env.integer("ZSE_W4_DEC")
        self._dec_ws = None
        # INT8 weights stay INT8 on the device (ZSE_W8_RESIDENT=0: expanded to fp16 at load, twice the memory)
        self.int8_resident = env.flag("ZSE_W8_RESIDENT")
        self._w8_scratch = None
        self._norm_ctx = None
        self._logits16 = None
        self.latent_form = 1           # decode attention over latent rows: 1 tcgen05 (csrc/latent_tc.cu), 2 mma.sync
        self.heads_form = 1            # tiles of queries over cached heads: 1 tcgen05 (csrc/heads_tc.cu), 2 mma.sync
        self._no_tables = torch.zeros(1, 1, dtype=torch.int32, device=self.device)
        self.attn_prefill_tc = env.flag("ZSE_ATTN_PREFILL_TC")

    def _w8_dense(self, w: "LinearWeight") -> torch.Tensor:
        """fp16 [N, K] view of an INT8 weight in the scratch buffer that all layers share (rows: gate then up for a
        fused gate/up tensor).  Valid until the next call."""
        need = w.N * w.K
        if self._w8_scratch is None or self._w8_scratch.numel() < need:
            self._w8_scratch = torch.empty(need, dtype=torch.float16, device=self.device)
        dense = self._w8_scratch[:need].view(w.N, w.K)
        self.n.dequant_w8_tiled(w.data, dense, w.N, w.K, w.N // 2 if w.swiglu else 0)
        return dense

    def norm_ctx(self, H: int) -> int:
        """A one-rank tensor-parallel context: lets a single GPU use the kernel that does a row-parallel projection,
        the residual add and the next RMSNorm in one launch (there is simply no peer to exchange with)."""
        if self._norm_ctx is None or self._norm_ctx[1] != H:
            z = lambda n, dt: torch.zeros(n, dtype=dt, device=self.device)
            keep = [z(8, torch.float16), z(8, torch.int32), z(8, torch.int64), z(8, torch.int32),
                    z(2 * 64 * H, torch.float16), z(2, torch.int32), z(4, torch.int32)]
            p = [t.data_ptr() for t in keep]
            ctx = self.n.tp_ctx_create(1, 0, 64, H, [p[0]], [p[1]], 0, [p[2]], [p[3]])
            self.n.tp_ctx_set_push(ctx, 64, [p[4]], 0, [p[5]], 0, [p[6]])
            self._norm_ctx = (ctx, H, keep)
        return self._norm_ctx[0]

    def residual_norm_fused_ok(self, w, M: int, H: int) -> bool:
        return bool((self.dec_mode & 8) and w.kind in ("w4t", "w8t") and M <= 64 and w.N == H and w.bias is None
                    and self.n.gemm_w4_dec_supported(M, w.N, w.K, 4)
                    and self.n.gemm_w4_dec_plan(w.N, w.K, 4, self.sm_count)[1] > 0)

    def linear_residual_norm(self, w, x, M: int, residual, norm_w, out, eps: float, slot: int) -> None:
        """residual += x W^T; out = RMSNorm(residual) * norm_w, one kernel (decode-sized passes, single GPU)."""
        self.n.tp_gemm_dec_allreduce_norm(self.norm_ctx(w.N), w.data, w.kind == "w8t", x, x.shape[0], M, w.N, w.K,
                                          slot & 1, False, residual, norm_w, out, float(eps), self.dec_ws,
                                          self.status.ptr)

    @property
    def dec_ws(self) -> torch.Tensor:
        if self._dec_ws is None:
            self._dec_ws = self.n.gemm_w4_dec_workspace(self.device, self.sm_count)
        return self._dec_ws

    def check(self):
        self.status.check()

    # ---- weights --------------------------------------------------------------------------------------
    def make_linear(self, parts, K: int, group_size: int, bias=None, swiglu: bool = False) -> LinearWeight:
        n = self.n
        b = None if bias is None else _np_to_dev(bias, self.device)
        tiled_ok = (K % 128 == 0 and group_size == 128
                    and all(p["dtype"] == "int4" and "flat_data" not in p for p in parts))
        if swiglu and tiled_ok:
            tiled_ok = len(parts) == 2 and parts[0]["shape"][0] == parts[1]["shape"][0]
        if tiled_ok:
            packed = torch.cat([_np_to_dev(p["data"], self.device).reshape(p["shape"][0], K // 2) for p in parts])
            scales = torch.cat([_np_to_dev(p["scales"], self.device).reshape(p["shape"][0], K // 128) for p in parts])
            zeros = torch.cat([_np_to_dev(p["zeros"], self.device).reshape(p["shape"][0], K // 128) for p in parts])
            N = packed.shape[0]
            inter = N // 2 if swiglu else 0
            n_tiles = (inter + 63) // 64 if swiglu else (N + 127) // 128
            out = torch.empty(n_tiles * (K // 128) * 8704, dtype=torch.uint8, device=self.device)
            n.repack_w4(packed, scales, zeros, out, N, K, inter)
            return LinearWeight("w4t", N, K, out, b, swiglu, out.numel())
        # INT8 (symmetric groups of 128): kept 8 bits wide, tiled for the decode kernel.  Passes of more than 64 tokens
        # expand the tensor into a scratch buffer that all layers share and run the fp16 GEMM on it.
        w8_ok = (K % 128 == 0 and group_size == 128 and all(p["dtype"] == "int8" and "scales" in p for p in parts)
                 and self.int8_resident)
        if swiglu and w8_ok:
            w8_ok = len(parts) == 2 and parts[0]["shape"][0] == parts[1]["shape"][0]
        if w8_ok:
            q = torch.cat([_np_to_dev(p["data"], self.device).reshape(p["shape"][0], K) for p in parts]).contiguous()
            sc = torch.cat([_np_to_dev(p["scales"], self.device).reshape(p["shape"][0], K // 128)
                            for p in parts]).contiguous()
            N = q.shape[0]
            inter = N // 2 if swiglu else 0
            n_tiles = (inter + 63) // 64 if swiglu else (N + 127) // 128
            out = torch.empty(n_tiles * (K // 128) * 16640, dtype=torch.uint8, device=self.device)
            n.repack_w8(q.view(torch.int8) if q.dtype != torch.int8 else q, sc, out, N, K, inter)
            return LinearWeight("w8t", N, K, out, b, swiglu, out.numel())
        # anything else becomes dense fp16 for the SS-mode kernel
        if all(p["dtype"] == "float16" for p in parts):      # already fp16: one copy, no fp32 round trip
            ws = [_np_to_dev(p["data"], self.device).reshape(tuple(p["shape"])) for p in parts]
            w = torch.cat(ws, dim=0) if len(ws) > 1 else ws[0].clone(memory_format=torch.contiguous_format)
            return LinearWeight("f16", w.shape[0], K, w, b, swiglu, w.numel() * 2)
        ws = [_dense_f32(p, group_size, self.device).to(torch.float16) for p in parts]
        w = torch.cat(ws, dim=0).contiguous() if len(ws) > 1 else ws[0].contiguous()
        return LinearWeight("f16", w.shape[0], K, w, b, swiglu, w.numel() * 2)

    # ---- ops ------------------------------------------------------------------------------------------
    def linear(self, w, x, M, out, x_cap=None, gather=None, side=None):
        """``gather``: a tensor-parallel context whose gathered activation buffer ``x`` is - the GEMM then waits, tile
        by tile, for the rows to arrive from the ranks that own them (INT4 weights, more than 64 rows)."""
        cap = x.shape[0] if x_cap is None else x_cap
        if gather is not None:
            if w.kind != "w4t" or M <= 64:
                raise NotImplementedError("a gathered activation buffer is read by the wide INT4 GEMM only")
            self.n.tp_gemm_w4_gathered(gather, w.data, x, cap, w.bias, out, M, w.N, w.K, out.stride(0), EPI_F16, 0,
                                       self.status.ptr)
        elif w.kind == "w8t":
            if M <= 64 and out.stride(0) % 8 == 0 and self.n.gemm_w4_dec_supported(M, w.N, w.K, EPI_F16):
                self.n.gemm_w8_dec(w.data, x, cap, w.bias, out, M, w.N, w.K, out.stride(0), EPI_F16, self.dec_ws,
                                   self.status.ptr)
            else:
                self.n.gemm_f16(self._w8_dense(w), w.N, x, cap, w.bias, out, M, w.N, w.K, out.stride(0), EPI_F16, 1,
                                self.status.ptr)
        elif (w.kind == "w4t" and (self.dec_mode & 4) and M <= 64 and out.stride(0) % 8 == 0
                and self.n.gemm_w4_dec_supported(M, w.N, w.K, EPI_F16)):
            self.n.gemm_w4_dec(w.data, x, cap, w.bias, out, M, w.N, w.K, out.stride(0), EPI_F16, self.dec_ws,
                               self.status.ptr)
        elif w.kind == "w4t":
            self.n.gemm_w4(w.data, x, cap, w.bias, out, M, w.N, w.K, out.stride(0), EPI_F16, 0, self.status.ptr)
        elif side is not None and self.linear_has_side(w):
            self.n.gemm_bf16_side(w.data, x, cap, out, M, w.N, w.K, out.stride(0), side[1], side[0], self.status.ptr)
        elif w.kind in ("bf16", "f32"):
            self._typed_linear(w, x, M, out, out.stride(0), EPI_F16, 1, cap)
        else:
            self.n.gemm_f16(w.data, w.N, x, cap, w.bias, out, M, w.N, w.K, out.stride(0), EPI_F16, 1, self.status.ptr)

    def linear_swiglu(self, w, x, M, out, x_cap=None, gelu=False, tmp=None, gather=None):
        cap = x.shape[0] if x_cap is None else x_cap
        if gather is not None:
            if w.kind != "w4t" or M <= 64 or gelu:
                raise NotImplementedError("a gathered activation buffer is read by the wide INT4 GEMM only")
            self.n.tp_gemm_w4_gathered(gather, w.data, x, cap, None, out, M, w.N, w.K, out.stride(0), EPI_SWIGLU, 0,
                                       self.status.ptr)
        elif w.kind == "w8t":
            if (not gelu and M <= 64 and out.stride(0) % 8 == 0
                    and self.n.gemm_w4_dec_supported(M, w.N, w.K, EPI_SWIGLU)):
                self.n.gemm_w8_dec(w.data, x, cap, None, out, M, w.N, w.K, out.stride(0), EPI_SWIGLU, self.dec_ws,
                                   self.status.ptr)
            else:
                gu = torch.empty(M, w.N, dtype=torch.float16, device=self.device) if tmp is None else tmp
                self.n.gemm_f16(self._w8_dense(w), w.N, x, cap, None, gu, M, w.N, w.K, gu.stride(0), EPI_F16, 1,
                                self.status.ptr)
                self.n.swiglu(gu, out, M, w.N // 2, gelu)
        elif (w.kind == "w4t" and not gelu and (self.dec_mode & 1) and M <= 64 and out.stride(0) % 8 == 0
                and self.n.gemm_w4_dec_supported(M, w.N, w.K, EPI_SWIGLU)):
            self.n.gemm_w4_dec(w.data, x, cap, None, out, M, w.N, w.K, out.stride(0), EPI_SWIGLU, self.dec_ws,
                               self.status.ptr)
        elif w.kind == "w4t" and not gelu:
            self.n.gemm_w4(w.data, x, cap, None, out, M, w.N, w.K, out.stride(0), EPI_SWIGLU, 0, self.status.ptr)
        else:
            if w.kind == "w4t":
                raise NotImplementedError("GeGLU needs the dense path")
            gu = torch.empty(M, w.N, dtype=torch.float16, device=self.device) if tmp is None else tmp
            self.n.gemm_f16(w.data, w.N, x, cap, None, gu, M, w.N, w.K, gu.stride(0), EPI_F16, 1, self.status.ptr)
            self.n.swiglu(gu, out, M, w.N // 2, gelu)

    def pick_k_split(self, w, M) -> int:
        """fp16 kernel only (the INT4 kernel plans its own on-chip split): planes so that the grid fills the GPU."""
        n_tiles = (w.N + 127) // 128
        nt = 16 if M <= 16 else 32 if M <= 32 else 64 if M <= 64 else 128 if M <= 128 else 256
        ctas = n_tiles * ((M + nt - 1) // nt)
        want = max(1, (self.sm_count * (2 if nt <= 64 else 1)) // max(1, ctas))
        return max(1, min(want, 8, (w.K // 64) // 4 or 1))

    def linear_partial(self, w, x, M, partials, k_split=None, x_cap=None) -> int:
        """fp32 result planes in ``partials`` [planes, M, N] (plane stride M*N); returns how many planes were written.
        The consumer (``add_rmsnorm`` / the tensor-parallel reduce) adds them in plane order."""
        cap = x.shape[0] if x_cap is None else x_cap
        if w.kind == "w8t":
            if M <= 64 and self.n.gemm_w4_dec_supported(M, w.N, w.K, EPI_PARTIAL):
                # one fp32 plane (row stride N): the decode kernel adds its K splits on chip
                self.n.gemm_w8_dec(w.data, x, cap, None, partials, M, w.N, w.K, w.N, EPI_PARTIAL, self.dec_ws,
                                   self.status.ptr)
                return 1
            dense = self._w8_dense(w)
            dw = LinearWeight("f16", w.N, w.K, dense, None, False, 0)
            return self.linear_partial(dw, x, M, partials, k_split, x_cap)
        if w.kind == "w4t":
            ks = 0 if k_split is None else min(k_split, partials.shape[0])
            planes = self.n.gemm_w4_splits(M, w.N, w.K, ks)
            if planes > partials.shape[0]:
                ks = partials.shape[0]
                planes = self.n.gemm_w4_splits(M, w.N, w.K, ks)
            self.n.gemm_w4(w.data, x, cap, None, partials, M, w.N, w.K, partials.stride(1), EPI_PARTIAL, ks,
                           self.status.ptr)
            return planes
        ks = self.pick_k_split(w, M) if k_split is None else k_split
        ks = min(ks, partials.shape[0])
        if w.kind in ("bf16", "f32"):
            return self._typed_linear(w, x, M, partials, w.N, EPI_PARTIAL, ks, cap)
        planes = self.n.gemm_f16_splits(M, w.N, w.K, ks)
        self.n.gemm_f16(w.data, w.N, x, cap, None, partials, M, w.N, w.K, partials.stride(1), EPI_PARTIAL, ks,
                        self.status.ptr)
        return planes

    # ---- bfloat16 / float layers ------------------------------------------------------------------------
    def _typed_linear(self, w, x, M, out, ldo, epilogue, k_split, cap) -> int:
        """Store (EPI_F16: in the activations' type) or fp32 planes; returns how many planes.  The tensor-core kernel
        takes bfloat16 rows of whole 16-byte pieces, everything else the general kernel (one plane)."""
        if w.kind == "bf16" and w.K % 8 == 0:
            planes = self.n.gemm_f16_splits(M, w.N, w.K, k_split) if epilogue == EPI_PARTIAL else 1
            self.n.gemm_bf16(w.data, w.N, x, cap, out, M, w.N, w.K, ldo, epilogue, k_split, self.status.ptr)
            return planes
        self.n.gemm_tile(w.data.dtype, x, x.stride(0), w.data, (w.K, 1), out, ldo, M, w.N, w.K,
                         self.n.TILE_STORE if epilogue == EPI_F16 else self.n.TILE_F32)
        return 1

    @staticmethod
    def linear_has_side(w) -> bool:
        """Whether ``linear`` puts columns into its ``side`` (the general kernel leaves them among the others)."""
        return w.kind == "bf16" and w.K % 8 == 0

    def dense(self, t: torch.Tensor, dtype) -> torch.Tensor:
        return t.to(self.device, dtype)

    def linear_f32(self, w, x, M, out):
        self._typed_linear(w, x, M, out, out.stride(0), EPI_PARTIAL, 1, x.shape[0])

    def add_norm(self, residual, partials, n_partials, slots, weight, out, M, eps, scale=None, offset=0.0, replace=False):
        self.n.add_norm(residual, partials, n_partials, slots, 0 if slots is None else slots.shape[1], weight, out, M,
                        residual.shape[1], float(eps), scale, offset, replace)

    def logits_finish(self, logits, M, scale, cap):
        self.n.logits_finish(logits, M, scale, cap)

    def latent_expands(self, spec, dtype) -> bool:
        return dtype == torch.bfloat16 and self.n.latent_mma_ok(spec)

    def latent_prep(self, inp, planes, n_planes, rows, positions, slots, freqs, norm_w, spec, eps, M):
        rc = self.n.row_cache(rows, self._no_tables)
        self.n.latent_prep(inp, planes, n_planes, M, rc, positions, slots, freqs, norm_w, spec, eps)

    @staticmethod
    def _gate_ptr(inp, spec):
        return inp.data_ptr() + spec.gate_col * inp.element_size() if spec.gated else None

    def latent_attn(self, inp, L, rows, block_tables, row_seq, positions, q_lat, o_lat, out, M, spec, scratch, num_splits):
        n, H, d, r, kr, vd = self.n, spec.heads, spec.dim, spec.rot_dim, spec.kv_rank, spec.vdim
        rc = n.row_cache(rows, block_tables)
        if self.latent_expands(spec, inp.dtype) and (rows.shape[1] in (16, 32) or rows.shape[1] % 64 == 0):
            if num_splits > 1 and scratch.numel() < M * num_splits * H * (kr + 2):
                num_splits = 1
            n.latent_absorb(inp, L.uk, q_lat, M, spec)
            n.latent_attn(q_lat, rc, row_seq, positions, o_lat, scratch, M, spec, num_splits, self.latent_form,
                          self.status.ptr)
            n.latent_unabsorb(o_lat, L.uv, self._gate_ptr(inp, spec), inp.stride(0), out, M, spec)
            return
        ql = q_lat[: M * H * spec.row].view(M, H, spec.row)
        n.gemm_tile(inp.dtype, inp, inp.stride(0), L.uk, (1, kr), ql, H * spec.row, M, kr, d, batch=H, a_batch=d + r,
                    b_batch=d * kr, o_batch=spec.row)
        ql[:, :, kr: kr + r].copy_(inp[:M, : H * (d + r)].view(M, H, d + r)[:, :, d:])
        n.latent_attn(q_lat, rc, row_seq, positions, o_lat, scratch, M, spec, 1, False, self.status.ptr)
        gate = inp[:, spec.gate_col:] if spec.gated else None
        n.gemm_tile(inp.dtype, o_lat, H * kr, L.uv, (kr, 1), out, out.stride(0), M, vd, kr,
                    n.TILE_GATE if spec.gated else n.TILE_STORE, batch=H, a_batch=kr, b_batch=vd * kr, o_batch=vd,
                    gate=gate, ldg=inp.stride(0), gate_batch=vd)

    def latent_attn_chunks(self, inp, L, rows, block_tables, cu_q, q_pos0, ctx_off, group, ctx, out, spec):
        n = self.n
        c, kr, kvx = ctx
        rc = n.row_cache(rows, block_tables)
        ch = n.Chunks(cu_q.data_ptr(), q_pos0.data_ptr(), ctx_off.data_ptr(), group.first, group.last, spec.window)
        n.latent_gather(rc, ch, group.rows, spec, c, kr)
        cap = c.numel() // spec.kv_rank
        n.gemm_bf16(L.ukv.data, L.ukv.N, c, cap, kvx, group.rows, L.ukv.N, L.ukv.K, L.ukv.N, EPI_F16, 1, self.status.ptr)
        v_col = (spec.heads * spec.dim + 7) // 8 * 8
        n.latent_chunk(inp, kvx, L.ukv.N, v_col, kr, rc, ch, group.max_q, out, self._gate_ptr(inp, spec), spec)

    def moe_workspace(self, specs, H: int, max_tokens: int, dtype):
        return MoeWorkspace(specs, H, max_tokens, dtype, self.device) if specs else None

    def moe_up(self, pairs, dtype, m=None):
        """Tensor-core form: tiles of 64 gate rows and their 64 up rows, the experts' rows padded to whole tiles."""
        if not moe_tensor_cores(m, pairs[0][0].shape[1], dtype):
            return super().moe_up(pairs, dtype, m)
        return self._interleaved(pairs, dtype)

    def _interleaved(self, pairs, dtype) -> torch.Tensor:
        ff, H = pairs[0][0].shape
        n = (ff + 63) // 64
        out = torch.zeros(len(pairs), n, 2, 64, H, dtype=dtype, device=self.device)
        pad = torch.zeros(n * 64, H, dtype=dtype, device=self.device)
        for e, pair in enumerate(pairs):
            for j, w in enumerate(pair):
                pad[:ff] = w
                out[e, :, j] = pad.view(n, 64, H)
        return out.view(-1, H)

    def moe(self, L, x, M, ws):
        n, m, H = self.n, L.moe, x.shape[1]
        dt = x.dtype
        per = m.top + (m.shared_ff > 0)
        planes = self.linear_partial(L.router, x, M, ws.router_views[m.router_rows])
        slots = M * m.top
        # result rows in fp32 while they are few, in the activations' type for long passes
        y_dt = torch.float32 if M <= ws.F32_ROWS else dt
        y = ws.y[: M * per * H * y_dt.itemsize].view(y_dt).view(M, per, H)
        if moe_tensor_cores(m, H, dt):
            tile = n.moe_tile_rows(M, m.experts, m.top)
            n.moe_route(ws.router, planes, M, m, tile, x, H, per, ws)
            self.moe_product_call(L, x, M, ws, 3 if m.gated else 0)()
            self.moe_product_call(L, x, M, ws, 2 if y_dt == torch.float32 else 1)()
            return y
        max_tiles = min(slots, m.experts + slots // 64)
        n.moe_route(ws.router, planes, M, m, 64, x, H, per, ws)
        store = n.TILE_F32 if y_dt == torch.float32 else n.TILE_STORE
        group = dict(tiles=ws.tiles, n_tiles=ws.n_tiles, max_tiles=max_tiles)
        before, after = (None, ws.row_score) if m.weigh == "output" else (ws.row_score, None)
        shared_after = ws.shared_score if m.shared_gate else None
        w = 2 if m.gated else 1

        def up(src, weights, act, ff, rows, limit, scale=None, **kw):
            if m.gated:
                n.gemm_tile(dt, src, H, weights, (H, 1), ws.glu, 2 * ff, rows, 2 * ff, H, n.TILE_STORE, **kw)
                n.glu(ws.glu, act, rows, ff, GLU[m.activation], limit)
            else:
                n.gemm_tile(dt, src, H, weights, (H, 1), act, ff, rows, ff, H, n.TILE_GELU, row_scale=scale, **kw)

        up(ws.xs, L.up, ws.act, m.ff, slots, m.limit, before, b_group=w * m.ff * H, **group)
        n.gemm_tile(dt, ws.act, m.ff, L.down, (m.ff, 1), y, H, slots, H, m.ff, store, out_rows=ws.out_rows,
                    row_scale=after, b_group=m.ff * H, **group)
        if m.shared_ff:
            up(x, L.shared_up, ws.act_shared, m.shared_ff, M, m.shared_limit)
            n.gemm_tile(dt, ws.act_shared, m.shared_ff, L.shared_down, (m.shared_ff, 1), y, H, M, H, m.shared_ff, store,
                        row_scale=shared_after, out_row=(per, m.top))
        return y

    def moe_product_call(self, L, x, M, ws, epilogue: int):
        """The tensor-core launch of one half of the experts (0: up + gelu, 3: gate and up + glu; 1, 2: down to
        bfloat16 / fp32 rows), over the tables that ``moe_route`` left in ``ws``."""
        n, m, H = self.n, L.moe, x.shape[1]
        tile = n.moe_tile_rows(M, m.experts, m.top)
        max_tiles = min(M * m.top, m.experts + M * m.top // tile)
        score = ws.row_score.data_ptr()
        if epilogue in (0, 3):
            rows_of = lambda ff: (ff + 63) // 64 * 128 if m.gated else ff
            g = n.MoeGemm(L.up.data_ptr(), ws.xs.data_ptr(), ws.act.data_ptr(), _dp(L.shared_up), x.data_ptr(),
                          ws.act_shared.data_ptr(), score if m.weigh == "input" else None, None, ws.tiles.data_ptr(),
                          ws.n_tiles.data_ptr(), None, rows_of(m.ff), H, m.ff, rows_of(m.shared_ff), H, m.shared_ff, 1, 0,
                          x.shape[0], m.ff, m.shared_ff, m.limit, m.shared_limit, GLU.get(m.activation, 0))
            rows = ws.xs.numel() // H
        else:
            per = m.top + (m.shared_ff > 0)
            g = n.MoeGemm(L.down.data_ptr(), ws.act.data_ptr(), ws.y.data_ptr(), _dp(L.shared_down),
                          ws.act_shared.data_ptr(), ws.y.data_ptr(), score if m.weigh == "output" else None,
                          ws.out_rows.data_ptr(), ws.tiles.data_ptr(), ws.n_tiles.data_ptr(),
                          ws.shared_score.data_ptr() if m.shared_gate else None, H, m.ff, H, H if m.shared_ff else 0,
                          m.shared_ff, H, per, m.top, ws.act_shared.numel() // max(1, m.shared_ff), H, H, 0.0, 0.0, 0)
            rows = ws.act.numel() // m.ff
        return lambda: n.moe_gemm(g, M, m.experts, rows, tile, max_tiles, epilogue, self.status.ptr)

    # ---- designs of attention over heads, matrix memories and post-norms ---------------------------------
    def embed_design(self, E, ids, positions, row_seq, cu_q, state_rows, last_token, residual, out, M, S, eps):
        n, H = self.n, E.table.shape[1]
        if E.turns is None:              # turns per token as two floats: the angle of any position keeps fp32 accuracy
            E.turns = self._turns(E.base ** (-torch.arange(0, H, 2, dtype=torch.float64) / H)).to(self.device)
        a = n.Embed(E.table.data_ptr(), _dp(E.bigram), E.norm.data_ptr(), E.turns.data_ptr(), ids.data_ptr(),
                    positions.data_ptr(), _dp(row_seq), _dp(cu_q), state_rows.data_ptr(), _dp(last_token),
                    residual.data_ptr(), out.data_ptr(), E.buckets, E.mul_prev, E.mul_cur, H, E.table.shape[0],
                    state_rows.stride(0), float(E.scale), float(eps))
        n.embed_design(a, out.dtype, M, self.status.ptr)

    def post_norm(self, residual, partials, n_partials, slots, weight, next_weight, out, M, eps):
        self.n.post_norm(residual, partials, n_partials, slots, 0 if slots is None else slots.shape[1], weight, next_weight,
                         out, M, residual.shape[1], float(eps))

    def linear_act(self, w, x, M, out, activation: str):
        if activation != "relu2":
            raise NotImplementedError(activation)
        if w.kind == "bf16" and w.K % 8 == 0:
            self.n.gemm_bf16(w.data, w.N, x, x.shape[0], out, M, w.N, w.K, out.stride(0), EPI_RELU2, 1, self.status.ptr)
        else:
            self.n.gemm_tile(w.data.dtype, x, x.stride(0), w.data, (w.K, 1), out, out.stride(0), M, w.N, w.K,
                             self.n.TILE_RELU2)

    def glu_expands(self, ff: int, H: int, dtype) -> bool:
        return not (dtype == torch.bfloat16 and H % 8 == 0)

    def glu_linear(self, gate, up, dtype):
        """Tensor-core form: tiles of 64 gate rows and their 64 up rows."""
        if self.glu_expands(gate.shape[0], gate.shape[1], dtype):
            return super().glu_linear(gate, up, dtype)
        return self.dense_linear(self._interleaved([(gate, up)], dtype))

    def linear_glu(self, w, x, M, out, activation: str, tmp=None):
        n, ff = self.n, out.shape[1]
        if not self.glu_expands(ff, w.K, x.dtype):
            n.gemm_bf16_glu(w.data, x, x.shape[0], out, M, w.N, w.K, out.stride(0), ff, GLU[activation], self.status.ptr)
            return
        n.gemm_tile(x.dtype, x, x.stride(0), w.data, (w.K, 1), tmp, 2 * ff, M, 2 * ff, w.K)
        n.glu(tmp, out, M, ff, GLU[activation], 0.0)

    def heads_expands(self, spec, dtype) -> bool:
        return dtype == torch.bfloat16 and self.n.heads_mma_ok(spec, 64)

    @staticmethod
    def _turns(f: torch.Tensor) -> torch.Tensor:
        """Frequencies (radians per token, float64) as turns per token in two floats [n, 2]: the angle of any position keeps
        fp32 accuracy."""
        f = f / (2 * math.pi)
        hi = f.float()
        return torch.stack([hi, (f - hi.double()).float()], 1).contiguous()

    def rotation(self, dims: int, base: float, factor: float = 1.0):
        f = super().rotation(dims, base, factor)
        return None if f is None else self._turns(f)

    def heads_prep(self, inp, planes, n_planes, kv, slots, L, spec, eps, M, positions=None, block_tables=None):
        """``block_tables``: of a pass whose rows are sequences of their own, which leaves the means of blocks as well."""
        tables = self._no_tables if block_tables is None else block_tables
        self.n.heads_prep(inp, planes, n_planes, M, self.n.heads(kv, spec, tables), slots, L.q_norm, L.k_norm,
                          getattr(L, "bias", None), getattr(L, "freqs", None), positions, spec, eps,
                          getattr(L, "temp", None), block_tables is not None)

    def heads_pool(self, kv, block_tables, row_seq, positions, spec, M):
        self.n.heads_pool(self.n.heads(kv, spec, block_tables), kv.k.dtype, row_seq, positions, M)

    @staticmethod
    def _head_gate(inp, spec):
        return inp.data_ptr() + spec.gate_col * inp.element_size() if spec.gated else None

    def heads_attn(self, inp, kv, block_tables, row_seq, positions, out, M, spec, scratch, num_splits, sink=None):
        tc = inp.dtype == torch.bfloat16 and self.n.heads_mma_ok(spec, kv.block_size)
        if not tc or scratch.numel() < M * num_splits * spec.heads * (spec.vdim + 2):
            num_splits = 1
        self.n.heads_attn(inp, self.n.heads(kv, spec, block_tables, sink), row_seq, positions, out,
                          self._head_gate(inp, spec), scratch, M, num_splits, tc)

    def heads_attn_chunks(self, inp, kv, block_tables, cu_q, q_pos0, positions, first, last, max_q, out, spec, sink=None):
        self.n.heads_attn_chunks(inp, self.n.heads(kv, spec, block_tables, sink), cu_q, q_pos0, first, last, max_q, out,
                                 self._head_gate(inp, spec), self.heads_form, self.status.ptr)

    def memory_expands(self, spec, dtype) -> bool:
        return dtype == torch.bfloat16 and self.n.memory_chunk_ok(spec)

    def memory_workspace(self, specs, max_tokens: int):
        w = max([0] + [s.heads * s.vdim for s in specs])
        return torch.zeros(max(1, max_tokens * w), dtype=torch.float32, device=self.device)

    def memory_prep(self, inp, planes, n_planes, gate_planes, n_gate_planes, gates, L, spec, M):
        self.n.memory_prep(inp, planes, n_planes, gate_planes, n_gate_planes, L.if_bias, gates, spec, M)

    def memory_tokens(self, inp, gates, states, at, state_rows, cu_q, L, out, S, M, spec, eps):
        self.n.memory_tokens(inp, gates, self.n.memory(states, at, state_rows, L.head_norm, spec, eps), cu_q, S, out)

    def memory_chunks(self, inp, gates, states, at, state_rows, cu_q, L, out, first, last, row0, M, spec, eps, ws):
        """Sequences ``first .. last - 1`` chunkwise; their rows are [row0, M)."""
        self.n.memory_chunks(inp, gates, self.n.memory(states, at, state_rows, L.head_norm, spec, eps), cu_q, first, last, ws,
                             M, row0, out)

    def state_space_expands(self, spec, dtype) -> bool:
        return dtype == torch.bfloat16 and self.n.space_chunk_ok(spec)

    def state_space_prep(self, inp, planes, n_planes, side, xbc, dt, states, at, state_rows, row_seq, cu_q, L, spec, M, S):
        if not self.linear_has_side(L.w_in):
            side = None
        self.n.space_prep(inp, planes, n_planes, side, spec.in_width - spec.dt_col,
                          self.n.space(states, at, state_rows, L, spec), row_seq, cu_q, xbc, dt, M)

    def state_space_tokens(self, inp, xbc, dt, states, at, state_rows, cu_q, L, out, S, M, spec):
        self.n.space_tokens(inp, xbc, dt, self.n.space(states, at, state_rows, L, spec), cu_q, S, out)

    def state_space_chunks(self, inp, xbc, dt, states, at, state_rows, cu_q, L, out, first, last, M, spec):
        """Sequences ``first .. last - 1`` chunkwise."""
        self.n.space_chunks(inp, xbc, dt, self.n.space(states, at, state_rows, L, spec), cu_q, first, last, out)

    def gated_linear_expands(self, spec, dtype) -> bool:
        return dtype == torch.bfloat16 and self.n.gated_linear_chunk_ok(spec)

    def gated_linear_workspace(self, specs, max_tokens: int):
        return torch.zeros(max_tokens * max(s.heads * s.vdim for s in specs), dtype=torch.float32, device=self.device)

    def gated_linear_prep(self, inp, planes, n_planes, side, decays, L, spec, M):
        if not self.linear_has_side(L.w_in):
            side = None
        self.n.gated_linear_prep(inp, planes, n_planes, side, spec.in_width - spec.rank_col,
                                 self.n.gated_linear(None, 0, None, L, spec, 0.0), decays, M)

    def gated_linear_tokens(self, inp, planes, n_planes, decays, states, at, state_rows, cu_q, L, out, S, M, spec, eps):
        self.n.gated_linear_tokens(inp, planes, n_planes, M, decays,
                                   self.n.gated_linear(states, at, state_rows, L, spec, eps), cu_q, S, out)

    def gated_linear_chunks(self, inp, decays, states, at, state_rows, cu_q, L, out, first, last, row0, M, spec, eps, ws):
        """Sequences ``first .. last - 1`` chunkwise; their rows are [row0, M)."""
        self.n.gated_linear_chunks(inp, decays, self.n.gated_linear(states, at, state_rows, L, spec, eps), cu_q, first, last,
                                   ws, M, row0, out)

    def add_norm_conv(self, residual, partials, n_partials, weight, out, conv_w, conv_out, states, at, state_rows, row_seq,
                      cu_q, M, S, eps):
        n, H = self.n, residual.shape[1]
        cv = n.row_conv_args(conv_w, states, at, state_rows)
        if cu_q is None:                     # every row is a sequence of its own: one kernel
            n.add_norm_conv(residual, partials, n_partials, weight, out, cv, conv_out, M, H, float(eps))
            return
        self.add_norm(residual, partials, n_partials, None, weight, out, M, eps)
        n.row_conv(out, conv_out, cv, row_seq, cu_q, M, H)

    def group_norm(self, x, weight, parts: int, M, eps):
        self.n.group_norm(x, weight, parts, M, eps)

    def embedding(self, table, ids, out, M, scale=1.0, copy=None):
        if table.dtype != torch.float16:
            self.n.embedding_typed(table, ids, out, M, table.shape[1], table.shape[0], float(scale), copy, self.status.ptr)
            return
        self.n.embedding(table, ids, out, M, table.shape[1], table.shape[0], float(scale), self.status.ptr)

    def add_rmsnorm(self, residual, partials, n_partials, add_f16, weight, out, M, eps):
        # partial planes are laid out [plane][M rows][H]: the plane stride the kernel assumes is M*H
        self.n.add_rmsnorm(residual, partials, n_partials, add_f16, weight, out, M, residual.shape[1], float(eps))

    def rope_kv_write(self, qkv, kv_layer, positions, slots, inv_freq, M, nh, nkv, hd, block_size, planes=None,
                      n_planes=0, bias=None):
        self.n.rope_kv_write(qkv, kv_layer, positions, slots, inv_freq, M, nh, nkv, hd, inv_freq.numel() * 2,
                             block_size, planes, n_planes, bias)

    def qkv_rope_fused_ok(self, w, M, hd, kv_layer) -> bool:
        ok_kind = w.kind == "w8t" or (w.kind == "w4t" and (self.dec_mode & 2))
        return bool(ok_kind and M <= 64 and hd == 128 and kv_layer.is_contiguous()
                    and self.n.gemm_w4_dec_supported(M, w.N, w.K, 3))

    def qkv_rope_fused(self, w, x, M, qkv, kv_layer, positions, slots, cos_sin, nh, nkv, block_size, x_cap=None):
        """One kernel: fused QKV projection + bias + rotate-half RoPE + K/V rows into the paged cache; ``qkv`` gets
        the rotated q heads.  head_dim 128, full rotary, ``cos_sin`` [max_position, 64, 2] fp32."""
        cap = x.shape[0] if x_cap is None else x_cap
        fn = self.n.gemm_w8_dec_qkv_rope if w.kind == "w8t" else self.n.gemm_w4_dec_qkv_rope
        fn(w.data, x, cap, w.bias, qkv, qkv.stride(0), M, w.K, nh, nkv, kv_layer, block_size, positions, slots, cos_sin,
           cos_sin.shape[0], self.dec_ws, self.status.ptr)

    @staticmethod
    def _tensor_core_attention(kv_layer, hd, nh, nkv, block_size) -> bool:
        """The tensor-core attention kernels cover head_dim 64/128/256 with up to 16 query heads per kv head; other
        shapes (Gemma-4 global layers with head_dim 512) take the CUDA-core kernel."""
        return (hd in (64, 128, 256) and nh // nkv <= 16 and block_size % 16 == 0 and kv_layer.stride(0) % 8 == 0
                and kv_layer.stride(1) % 8 == 0 and kv_layer.data_ptr() % 16 == 0)

    def attn_decode(self, qkv, kv_layer, block_tables, seq_lens, out, S, nh, nkv, hd, block_size, scale, scratch=None,
                    num_splits=1, softcap=0.0, window=0):
        if not self._tensor_core_attention(kv_layer, hd, nh, nkv, block_size):
            self.n.attn_generic(qkv, qkv.stride(0), kv_layer, block_tables, seq_lens, None, None, S, out,
                                out.stride(0), S, nh, nkv, hd, block_size, scale, softcap, window)
            return
        if scratch is None or scratch.numel() < S * nh * num_splits * (hd + 2):
            num_splits = 1
        self.n.attn_decode_ext(qkv, qkv.stride(0), kv_layer, block_tables, seq_lens, out, out.stride(0), scratch, S,
                               nh, nkv, hd, block_size, num_splits, scale, softcap, window)

    def attn_prefill(self, qkv, kv_layer, block_tables, cu_q, q_pos0, out, num_seqs, total_q, max_q_len, nh, nkv, hd,
                     block_size, scale, softcap=0.0, window=0):
        if not self._tensor_core_attention(kv_layer, hd, nh, nkv, block_size):
            self.n.attn_generic(qkv, qkv.stride(0), kv_layer, block_tables, None, cu_q, q_pos0, num_seqs, out,
                                out.stride(0), total_q, nh, nkv, hd, block_size, scale, softcap, window)
            return
        if (self.attn_prefill_tc and hd == 128 and softcap == 0.0 and window == 0 and kv_layer.is_contiguous()
                and kv_layer.shape[1:] == (2, nkv, block_size, hd)):
            self.n.attn_prefill_tc(qkv, qkv.stride(0), total_q, kv_layer, block_tables, cu_q, q_pos0, out,
                                   out.stride(0), num_seqs, max_q_len, nh, nkv, hd, block_size, scale,
                                   self.status.ptr)
            return
        self.n.attn_prefill_ext(qkv, qkv.stride(0), kv_layer, block_tables, cu_q, q_pos0, out, out.stride(0),
                                num_seqs, max_q_len, nh, nkv, hd, block_size, scale, softcap, window)

    def headnorm_rope_kv_write(self, qkv, kv_layer, positions, slots, freqs, q_norm_w, k_norm_w, norm_v, k_is_v, eps,
                               M, nh, nkv, hd, block_size):
        self.n.headnorm_rope_kv_write(qkv, kv_layer, positions, slots, freqs, q_norm_w, k_norm_w, norm_v, k_is_v, eps,
                                      M, nh, nkv, hd, block_size)

    def norm_add_rmsnorm(self, x, w_post, residual, scalar, w_next, out, M, eps):
        self.n.norm_add_rmsnorm(x, w_post, residual, scalar, w_next, out, M, residual.shape[1], eps)

    def glu(self, gate_up, out, M, I, gelu=False):
        self.n.swiglu(gate_up, out, M, I, gelu)

    def softcap(self, logits, M, cap):
        self.n.softcap(logits, M, logits.shape[1], cap)

    def argmax(self, logits, out, M):
        if logits.dtype == torch.float32:
            self.n.argmax_f32(logits, logits.stride(0), out, M, logits.shape[1])
            return
        self.n.argmax(logits, logits.stride(0), out, M, logits.shape[1])

    def _half_logits(self, logits, M):
        """fp16 copy of fp32 logits for the sampling kernel, whose cut-offs work on 16-bit keys."""
        h = self._logits16
        if h is None or h.shape[0] < logits.shape[0] or h.shape[1] != logits.shape[1]:
            h = self._logits16 = torch.empty(logits.shape, dtype=torch.float16, device=self.device)
        h[:M].copy_(logits[:M])
        return h

    def sample(self, logits, out, M, temperature, top_k, top_p, seeds, step):
        if logits.dtype == torch.float32:
            logits = self._half_logits(logits, M)
        self.n.sample(logits, logits.stride(0), out, M, logits.shape[1], temperature, top_k, top_p, seeds, int(step))

    def apply_repetition_penalty(self, logits, rows, tokens, counts, n, penalty):
        if logits.dtype == torch.float32:
            self.n.apply_repetition_penalty_f32(logits, logits.stride(0), rows, tokens, counts, n, penalty,
                                                logits.shape[1])
            return
        self.n.apply_repetition_penalty(logits, logits.stride(0), rows, tokens, counts, n, penalty, logits.shape[1])

    def lora_apply(self, x, a_table, b_table, ids, scales, y, M, K, N, rank, tmp=None, y_col0=0):
        yv = y[:, y_col0:]
        if rank % 2 == 0 and rank <= 64 and K % 8 == 0 and K * 2 + 256 <= 200 * 1024:
            # one launch: the token's activation row is read once, nothing passes through global memory in between
            self.n.lora_apply(x, x.stride(0), a_table, b_table, ids, scales, yv, y.stride(0), M, K, N, rank)
            return
        if tmp is None:
            tmp = torch.empty(M, rank, dtype=torch.float32, device=self.device)
        self.n.lora_shrink(x, x.stride(0), a_table, ids, tmp, M, K, rank)
        self.n.lora_expand(tmp, b_table, ids, scales, yv, y.stride(0), M, N, rank)


def make_ops(device, group: Optional[str] = None) -> TorchOps:
    device = torch.device(device)
    if device.type == "cuda":
        return CudaOps(device, group)
    return TorchOps(device)
