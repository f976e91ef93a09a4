"""Plain PyTorch restatement of every device op (fp32 math on whatever device the tensors live on).

Two jobs: the execution path on machines without a GPU (the tiny CPU configuration), and the oracle that the
numerics tests compare each CUDA kernel against.  Semantics follow the reference runner's numerics contract
(zse-engine/zse_engine/orchestrator/kernels.py, see the per-function notes); accumulation is fp32 and results are
rounded to fp16 where the CUDA kernels round.
"""
from __future__ import annotations

import math
from typing import Optional

import torch


def dequant_int4(packed: torch.Tensor, scales: torch.Tensor, zeros: torch.Tensor, shape, group_size: int = 128):
    """Flat-group dequantisation: element i belongs to group i // group_size of the flattened tensor."""
    n = int(math.prod(shape))
    groups = (n + group_size - 1) // group_size
    p = packed.reshape(-1)[: groups * group_size // 2]
    q = torch.stack([p & 0xF, p >> 4], dim=-1).reshape(groups, group_size).to(torch.float32)
    w = q * scales.reshape(-1)[:groups].float()[:, None] + zeros.reshape(-1)[:groups].float()[:, None]
    return w.reshape(-1)[:n].reshape(shape)


def dequant_int8(q: torch.Tensor, scales: torch.Tensor, shape, group_size: int = 128):
    n = int(math.prod(shape))
    groups = (n + group_size - 1) // group_size
    v = q.reshape(-1)[: groups * group_size].to(torch.float32).reshape(groups, group_size)
    return (v * scales.reshape(-1)[:groups].float()[:, None]).reshape(-1)[:n].reshape(shape)


def linear(x: torch.Tensor, w_f32: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """fp32 accumulate, clamp to the fp16 range, round to fp16 (kernels.py:1984-1987)."""
    y = x.float() @ w_f32.T
    if bias is not None:
        y = y + bias.float()
    return y.clamp(-65504, 65504).to(torch.float16)


def swiglu(gate: torch.Tensor, up: torch.Tensor, gelu: bool = False) -> torch.Tensor:
    g, u = gate.float(), up.float()
    act = torch.nn.functional.gelu(g, approximate="tanh") if gelu else g / (1 + torch.exp(-g))
    return (act * u).clamp(-65504, 65504).to(torch.float16)


def rmsnorm(x_f32: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    x = x_f32.float()
    return (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight.float()).to(torch.float16)


def inv_freq(rotary_dim: int, theta: float, rope_scaling: Optional[dict] = None) -> torch.Tensor:
    """theta^(-2i/rotary_dim) in float64, rounded to fp32.  ``linear`` and ``llama3`` scaling are applied here so
    the kernels only ever see a frequency table."""
    i = torch.arange(rotary_dim // 2, dtype=torch.float64)
    f = theta ** (-2.0 * i / rotary_dim)
    if rope_scaling:
        kind = rope_scaling.get("rope_type", rope_scaling.get("type"))
        factor = float(rope_scaling.get("factor", 1.0))
        if kind == "linear":
            f = f / factor
        elif kind == "llama3":
            lo, hi = float(rope_scaling.get("low_freq_factor", 1.0)), float(rope_scaling.get("high_freq_factor", 4.0))
            old = float(rope_scaling.get("original_max_position_embeddings", 8192))
            wavelen = 2 * math.pi / f
            smooth = ((old / wavelen) - lo) / (hi - lo)
            mid = (1 - smooth) * f / factor + smooth * f
            f = torch.where(wavelen < old / hi, f, torch.where(wavelen > old / lo, f / factor, mid))
    return f.to(torch.float32)


def rope_(x: torch.Tensor, positions: torch.Tensor, freqs: torch.Tensor) -> torch.Tensor:
    """Rotate-half RoPE on x [T, heads, hd] (pairs (i, i + rot/2) of the first ``2*len(freqs)`` dims)."""
    rot = freqs.numel() * 2
    ang = positions.to(torch.float32)[:, None] * freqs.to(positions.device)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    xf = x.float()
    a, b = xf[..., : rot // 2], xf[..., rot // 2: rot]
    out = xf.clone()
    out[..., : rot // 2] = a * c - b * s
    out[..., rot // 2: rot] = b * c + a * s
    return out.to(x.dtype)


def rope_kv_write(qkv: torch.Tensor, kv_layer: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
                  freqs: torch.Tensor, nh: int, nkv: int, hd: int, block_size: int) -> None:
    """In place: rotates q and k inside ``qkv`` [M, (nh+2nkv)*hd], scatters k/v into ``kv_layer``
    [blocks, 2, nkv, block_size, hd] at ``slots`` (-1 = do not store)."""
    M = qkv.shape[0]
    q = qkv[:, : nh * hd].view(M, nh, hd)
    k = qkv[:, nh * hd: (nh + nkv) * hd].view(M, nkv, hd)
    v = qkv[:, (nh + nkv) * hd:].view(M, nkv, hd)
    q.copy_(rope_(q, positions, freqs))
    k.copy_(rope_(k, positions, freqs))
    ok = slots >= 0
    if ok.any():
        blk, off = slots[ok] // block_size, slots[ok] % block_size
        kv_layer[blk, 0, :, off, :] = k[ok].to(kv_layer.dtype)
        kv_layer[blk, 1, :, off, :] = v[ok].to(kv_layer.dtype)


def headnorm_rope_kv_write(qkv: torch.Tensor, kv_layer: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
                           freqs: torch.Tensor, q_norm_w, k_norm_w, norm_v: bool, k_is_v: bool, eps: float, nh: int,
                           nkv: int, hd: int, block_size: int) -> None:
    """Gemma-family variant of ``rope_kv_write``: per-head RMSNorm of q and k (weights [hd] or None) and of v (no
    weight), RoPE with a full-length frequency table (0 = pair not rotated), V = raw k projection when ``k_is_v``
    (zse-engine/zse_engine/orchestrator/model_runner.py:455-486).  q is rotated in place; k and v only go to the
    cache."""
    M = qkv.shape[0]

    def hnorm(x, w):
        y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)
        return y if w is None else y * w.float()

    q = qkv[:, : nh * hd].view(M, nh, hd)
    k_raw = qkv[:, nh * hd: (nh + nkv) * hd].float().view(M, nkv, hd)
    v = k_raw if k_is_v else qkv[:, (nh + nkv) * hd: (nh + 2 * nkv) * hd].float().view(M, nkv, hd)
    qf = q.float()
    if q_norm_w is not None:
        qf = hnorm(qf, q_norm_w)
    kf = hnorm(k_raw, k_norm_w) if k_norm_w is not None else k_raw
    if norm_v:
        v = hnorm(v, None)
    q.copy_(rope_(qf, positions, freqs).clamp(-65504, 65504).to(q.dtype))
    kf = rope_(kf, positions, freqs)
    ok = slots >= 0
    if ok.any():
        blk, off = slots[ok] // block_size, slots[ok] % block_size
        kv_layer[blk, 0, :, off, :] = kf[ok].clamp(-65504, 65504).to(kv_layer.dtype)
        kv_layer[blk, 1, :, off, :] = v[ok].clamp(-65504, 65504).to(kv_layer.dtype)


def norm_add_rmsnorm(x: torch.Tensor, w_post: torch.Tensor, residual: torch.Tensor, scalar, w_next, eps: float):
    """residual (fp32, in place) = (residual + RMSNorm(x)*w_post) * scalar; returns RMSNorm(residual)*w_next in fp16
    (or None without ``w_next``)."""
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w_post.float()
    residual.add_(y)
    if scalar is not None:
        residual.mul_(float(scalar.reshape(-1)[0]))
    return None if w_next is None else rmsnorm(residual, w_next, eps)


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    return (cap * torch.tanh(x.float() / cap)).to(x.dtype)


def _gather_kv(kv_layer: torch.Tensor, table: torch.Tensor, length: int, block_size: int):
    """K, V [length, nkv, hd] plus a bool mask of positions that sit in holes (block id -1)."""
    nblk = (length + block_size - 1) // block_size
    ids = table[:nblk].long()
    hole = ids < 0
    safe = ids.clamp(min=0)
    k = kv_layer[safe, 0].permute(0, 2, 1, 3).reshape(nblk * block_size, kv_layer.shape[2], kv_layer.shape[4])
    v = kv_layer[safe, 1].permute(0, 2, 1, 3).reshape(nblk * block_size, kv_layer.shape[2], kv_layer.shape[4])
    mask = hole.repeat_interleave(block_size)[:length]
    return k[:length].float(), v[:length].float(), mask


def attn_decode(q: torch.Tensor, kv_layer: torch.Tensor, block_tables: torch.Tensor, seq_lens: torch.Tensor,
                nh: int, nkv: int, hd: int, block_size: int, scale: float, softcap: float = 0.0,
                window: int = 0) -> torch.Tensor:
    """q [S, nh*hd] -> out [S, nh*hd] fp16; sequence s attends to its first seq_lens[s] cached tokens."""
    S = q.shape[0]
    out = torch.zeros(S, nh * hd, dtype=torch.float16, device=q.device)
    rep = nh // nkv
    for s in range(S):
        n = int(seq_lens[s])
        if n == 0:
            continue
        k, v, hole = _gather_kv(kv_layer, block_tables[s], n, block_size)
        qs = q[s].float().view(nh, hd)
        sc = torch.einsum("hd,thd->ht", qs, k.repeat_interleave(rep, dim=1)) * scale
        if softcap:
            sc = softcap * torch.tanh(sc / softcap)
        if window:
            hole = hole | (torch.arange(n, device=q.device) < n - window)
        sc = sc.masked_fill(hole[None, :], float("-inf"))
        p = torch.softmax(sc, dim=-1).nan_to_num(0.0)
        out[s] = torch.einsum("ht,thd->hd", p, v.repeat_interleave(rep, dim=1)).reshape(-1).to(torch.float16)
    return out


def attn_prefill(q: torch.Tensor, kv_layer: torch.Tensor, block_tables: torch.Tensor, cu_q: torch.Tensor,
                 q_pos0: torch.Tensor, nh: int, nkv: int, hd: int, block_size: int, scale: float,
                 softcap: float = 0.0, window: int = 0) -> torch.Tensor:
    """Packed causal attention: query row r of sequence s sits at cache position q_pos0[s] + r and sees every
    cached token at or before it."""
    out = torch.zeros(q.shape[0], nh * hd, dtype=torch.float16, device=q.device)
    rep = nh // nkv
    for s in range(cu_q.numel() - 1):
        a, b = int(cu_q[s]), int(cu_q[s + 1])
        if b <= a:
            continue
        p0 = int(q_pos0[s])
        n = p0 + (b - a)
        k, v, hole = _gather_kv(kv_layer, block_tables[s], n, block_size)
        qs = q[a:b].float().view(b - a, nh, hd)
        sc = torch.einsum("qhd,thd->hqt", qs, k.repeat_interleave(rep, dim=1)) * scale
        if softcap:
            sc = softcap * torch.tanh(sc / softcap)
        pos_q = torch.arange(p0, n, device=q.device)[:, None]
        pos_k = torch.arange(n, device=q.device)[None, :]
        hidden = (pos_k > pos_q) | hole[None, :]
        if window:
            hidden = hidden | (pos_k <= pos_q - window)
        sc = sc.masked_fill(hidden[None], float("-inf"))
        p = torch.softmax(sc, dim=-1).nan_to_num(0.0)
        out[a:b] = torch.einsum("hqt,thd->qhd", p, v.repeat_interleave(rep, dim=1)).reshape(b - a, -1).to(torch.float16)
    return out


def apply_repetition_penalty(logits: torch.Tensor, counts: dict, penalty: float) -> torch.Tensor:
    """``counts``: token -> occurrences.  positive logits are divided, negative multiplied by
    ``penalty^(1+log2(count))`` (zse-engine/zse_engine/orchestrator/sampler.py:64-80)."""
    out = logits.clone().float()
    for tok, c in counts.items():
        if c > 0 and 0 <= tok < out.numel():
            f = penalty ** (1.0 + math.log2(c))
            out[tok] = out[tok] / f if out[tok] > 0 else out[tok] * f
    return out


def filtered_probs(logits: torch.Tensor, temperature: float, top_k: int, top_p: float) -> torch.Tensor:
    """The distribution the sampler draws from: temperature, then keep values >= the k-th largest, then the smallest
    sorted prefix whose softmax mass reaches top_p (ties at the cut are kept), renormalised."""
    x = logits.float() / max(temperature, 1e-6)
    if 0 < top_k < x.numel():
        kth = torch.topk(x, top_k).values[-1]
        x = torch.where(x >= kth, x, torch.full_like(x, float("-inf")))
    p = torch.softmax(x, dim=-1)
    if top_p < 1.0:
        sp, idx = torch.sort(p, descending=True)
        cum = torch.cumsum(sp, dim=-1)
        cut = int((cum < top_p).sum().item())
        thr = sp[min(cut, sp.numel() - 1)]
        p = torch.where(p >= thr, p, torch.zeros_like(p))
        p = p / p.sum()
    return p


def lora_delta(x: torch.Tensor, a: torch.Tensor, b: torch.Tensor, scaling: float) -> torch.Tensor:
    """x [M, K], a [r, K], b [N, r] -> scaling * (x a^T) b^T in fp32."""
    return scaling * ((x.float() @ a.float().T) @ b.float().T)


# ---- latent attention (one cached latent row per token) -------------------------------------------------------------
def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, freqs: torch.Tensor) -> torch.Tensor:
    """Interleaved rotation of the leading ``2 * len(freqs)`` of the last dimension: (2i, 2i+1) turn by
    ``position * freqs[i]``.  ``x`` [T, ..., R] fp32, ``positions`` [T]."""
    n = 2 * freqs.numel()
    ang = positions.float().reshape(-1, *([1] * (x.dim() - 1))) * freqs
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def latent_prep(inp: torch.Tensor, cache_rows: torch.Tensor, positions, slots, freqs, norm_w, spec, eps: float) -> None:
    """Second half of the fused input projection [q | latent, rotated key | gate]: the latent is RMS-normed and joins the
    rotated key part in the cache, the rotated part of every query head is rotated in place.  ``cache_rows``
    [blocks, block_size, row]."""
    H, d, r, kr = spec.heads, spec.dim, spec.rot_dim, spec.kv_rank
    T, bs = inp.shape[0], cache_rows.shape[1]
    q = inp[:, : H * (d + r)].float().reshape(T, H, d + r).clone()
    lat = inp[:, spec.latent_col: spec.latent_col + kr + r].float()
    c = lat[:, :kr] * torch.rsqrt(lat[:, :kr].pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
    row = torch.cat([c, rotate_pairs(lat[:, kr:], positions, freqs)], dim=-1).to(cache_rows.dtype)
    ok = slots >= 0
    s = slots[ok]
    cache_rows[s // bs, s % bs, : kr + r] = row[ok]
    q[..., d:] = rotate_pairs(q[..., d:], positions, freqs)
    inp[:, : H * (d + r)] = q.view(T, -1).to(inp.dtype)


def latent_absorb(inp: torch.Tensor, uk: torch.Tensor, spec) -> torch.Tensor:
    """Queries in the space of the cached rows: [T, H, row], the unrotated part multiplied by W_uk."""
    H, d, r, kr = spec.heads, spec.dim, spec.rot_dim, spec.kv_rank
    T = inp.shape[0]
    q = inp[:, : H * (d + r)].float().view(T, H, d + r)
    out = torch.zeros(T, H, spec.row, device=inp.device)
    out[..., :kr] = torch.einsum("thd,hdc->thc", q[..., :d], uk.float().view(H, d, kr))
    out[..., kr: kr + r] = q[..., d:]
    return out


def latent_attn_token(q_lat: torch.Tensor, cache_rows: torch.Tensor, table: torch.Tensor, pos: int, spec) -> torch.Tensor:
    """One token's heads against the cached rows it sees: [H, kv_rank] fp32.  ``q_lat`` [H, row]."""
    bs = cache_rows.shape[1]
    lo = max(0, pos + 1 - spec.window) if spec.window > 0 else 0
    j = torch.arange(lo, pos + 1, device=cache_rows.device)
    blk = table[j // bs].long()
    j, blk = j[blk >= 0], blk[blk >= 0]
    if j.numel() == 0:
        return torch.zeros(spec.heads, spec.kv_rank, device=cache_rows.device)
    rows = cache_rows[blk, j % bs].float()
    w = torch.softmax(q_lat.float() @ rows.T * spec.scale, dim=-1)
    return w @ rows[:, : spec.kv_rank]


def latent_attn_chunk(inp: torch.Tensor, c_ctx: torch.Tensor, kr_ctx: torch.Tensor, valid: torch.Tensor, kvx: torch.Tensor,
                      q_pos: torch.Tensor, ctx_pos: torch.Tensor, spec) -> torch.Tensor:
    """A chunk's heads against expanded keys and values ``kvx`` [C, H*dim (padded) | H*vdim]: [T, H, vdim] fp32."""
    H, d, r, vd = spec.heads, spec.dim, spec.rot_dim, spec.vdim
    T, C = inp.shape[0], kvx.shape[0]
    q = inp[:, : H * (d + r)].float().view(T, H, d + r)
    v0 = (H * d + 7) // 8 * 8
    k = kvx[:, : H * d].float().view(C, H, d)
    v = kvx[:, v0: v0 + H * vd].float().view(C, H, vd)
    s = torch.einsum("thd,chd->htc", q[..., :d], k) + torch.einsum("thr,cr->htc", q[..., d:], kr_ctx[:, :r].float())
    dist = q_pos[:, None] - ctx_pos[None, :]
    see = (dist >= 0) & valid[None, :]
    if spec.window > 0:
        see &= dist < spec.window
    s = (s * spec.scale).masked_fill(~see, float("-inf"))
    return torch.einsum("htc,chv->thv", torch.softmax(s, dim=-1).nan_to_num(0.0), v)


def gelu_exact(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.erf(x * math.sqrt(0.5)))


def rmsnorm_f32(x: torch.Tensor, w: Optional[torch.Tensor], eps: float, offset: float = 0.0) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * (w + offset), fp32 in and out; without ``w`` the factor is 1."""
    y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return y if w is None else y * (w.float() + offset)


# ---- embedding with what a design adds to it ------------------------------------------------------------------------
def previous_tokens(ids: torch.Tensor, cu_q, state_rows, last_token: torch.Tensor) -> torch.Tensor:
    """The token before each of the packed ``ids``; -1 for the first of a sequence.  ``cu_q[s]``: first row of sequence s
    (and the end); the token before it is ``last_token[state_rows[0, s]]``."""
    prev = torch.cat([ids.new_zeros(1), ids[:-1]])
    for s in range(len(cu_q) - 1):
        read = int(state_rows[0, s])
        prev[int(cu_q[s])] = int(last_token[read]) if read >= 0 else -1
    return prev


def sinusoid(positions: torch.Tensor, width: int, base: float) -> torch.Tensor:
    """[T, width]: entry 2i is sin(p * base^(-2i/width)), entry 2i + 1 the cosine of the same angle."""
    j = torch.arange(width, dtype=torch.float64, device=positions.device)
    even = j - j % 2
    ang = positions.double()[:, None] * base ** (-even / width)
    return torch.where(j % 2 == 0, torch.sin(ang), torch.cos(ang)).float()


# ---- attention over heads whose keys and values have their own widths ------------------------------------------------
def heads_prep(inp: torch.Tensor, k_cache, v_cache, slots, spec, q_norm, k_norm, eps: float, positions=None, bias=None,
               freqs=None, temp=None) -> None:
    """Second half of the fused input projection [q | k | v | gate]: bias, query and key norm (over a head's dimensions after
    the rotation, or over all heads' before it), rotation, factors of the queries (by position, or ``temp`` [heads]), keys and
    values into the cache (``k_cache`` [blocks, kv_heads, block_size, dim..]); queries are finished in place.  ``freqs``:
    radians per position of every pair that rotates."""
    T, H, G, d, vd = inp.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
    full = inp.float()
    if bias is not None:
        full = full.clone()
        full[:, : bias.numel()] += bias.float()
    turn = (lambda x: rotate_pairs(x.double(), positions.double(), freqs).float()) if spec.rot_dims else lambda x: x

    def normed(x, n, w):
        if spec.whole_norm:
            return turn(rmsnorm_f32(x, w, eps).reshape(T, n, d))
        return rmsnorm_f32(turn(x.reshape(T, n, d)), w, eps)

    q = normed(full[:, : H * d], H, q_norm)
    if spec.temp_coef:
        q = q * query_temperature(positions, spec.temp_coef, spec.temp_every)[:, None, None]
    if temp is not None:
        q = q * temp.float()[:, None]
    inp[:, : H * d] = q.reshape(T, -1).to(inp.dtype)
    if not spec.own_kv:
        return
    bs = k_cache.shape[2]
    raw = full[:, spec.k_col: spec.k_col + G * d]
    k = normed(raw, G, k_norm)
    v = (raw.reshape(T, G, d) if spec.k_as_v else full[:, spec.v_col: spec.v_col + G * vd].reshape(T, G, vd)).to(v_cache.dtype)
    ok = slots >= 0
    s = slots[ok]
    k_cache[s // bs, :, s % bs, :d] = k[ok].to(k_cache.dtype)
    v_cache[s // bs, :, s % bs, :vd] = v[ok]


def pool_rows(cache: torch.Tensor, table: torch.Tensor, means_at: int, block: int, size: int) -> None:
    """Writes the mean of the cached rows of block ``block`` of ``size`` tokens (``cache`` [blocks, kv_heads, block_size, d]) to
    its place behind ``means_at`` in the sequence's block table."""
    bs = cache.shape[2]
    pos = torch.arange(block * size, block * size + size, device=cache.device)
    blk = table[pos // bs].long()
    rows = cache[blk.clamp_min(0), :, pos % bs].float() * (blk >= 0)[:, None, None]
    to = int(table[means_at + block // bs])
    if to >= 0:
        cache[to, :, block % bs] = (rows.sum(0) / size).to(cache.dtype)


def heads_attn(q: torch.Tensor, positions, k_cache, v_cache, table, spec, sink=None, means_at: int = 0) -> torch.Tensor:
    """Queries [T, heads, dim] of one sequence at ``positions`` against its cached keys: [T, heads, vdim] fp32.  ``sink``
    [heads]: one more score of every row, without a value; ``means_at``: where the blocks of means begin in ``table``."""
    bs, rep = k_cache.shape[2], spec.heads // spec.kv_heads
    first = torch.tensor([spec.first_seen(int(p)) for p in positions], device=q.device)
    pos = torch.arange(int(first.min()), int(positions.max()) + 1, device=q.device)
    if spec.keep_first:
        pos = torch.cat([torch.arange(min(spec.keep_first, int(first.min())), device=q.device), pos])
    blk, at = table[pos // bs].long(), pos % bs
    see = (pos[None] <= positions[:, None]) & ((pos[None] >= first[:, None]) | (pos[None] < spec.keep_first))
    if spec.pool:
        seen = torch.tensor([spec.blocks_seen(int(p)) for p in positions], device=q.device)
        b = torch.arange(int(seen.max()), device=q.device)
        blk, at = torch.cat([table[means_at + b // bs].long(), blk]), torch.cat([b % bs, at])
        see = torch.cat([b[None] < seen[:, None], see], 1)
    k = k_cache[blk.clamp_min(0), :, at, : spec.dim].float().repeat_interleave(rep, 1)
    v = v_cache[blk.clamp_min(0), :, at, : spec.vdim].float().repeat_interleave(rep, 1)
    see = see & (blk >= 0)[None]
    s = torch.einsum("thd,nhd->htn", q.float(), k) * spec.scale
    if spec.softcap:
        s = spec.softcap * torch.tanh(s / spec.softcap)
    s = s.masked_fill(~see, float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.float()[:, None, None].expand(-1, s.shape[1], 1)], -1)
    w = torch.softmax(s, -1).nan_to_num(0.0)[..., : k.shape[0]]
    return torch.einsum("htn,nhv->thv", w, v)


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    """Factor of the queries at ``positions``, fp32."""
    return 1.0 + coef * torch.log((torch.div(positions + 1, every, rounding_mode="floor") + 1).float())


# ---- matrix memory (mLSTM) --------------------------------------------------------------------------------------------
def memory_gates(z: torch.Tensor, bias: torch.Tensor, cap: float) -> torch.Tensor:
    """Pre-activations [T, 2 * heads] of the input and forget gates -> their logarithms, fp32."""
    H = z.shape[1] // 2
    g = cap * torch.tanh((z.float() + bias) / cap)
    return torch.cat([g[:, :H], torch.nn.functional.logsigmoid(g[:, H:])], 1)


def memory_tokens(q, k, v, log_i, log_f, S, n, m):
    """Tokens of one sequence through one layer's memory.  q, k [T, H, d] and v [T, H, vd] fp32, gates [T, H]; S [H, d, vd],
    n [H, d], m [H] are updated in place.  Returns the read-outs [T, H, vd]."""
    out = torch.empty_like(v)
    for t in range(q.shape[0]):
        new = torch.maximum(log_f[t] + m, log_i[t])
        keep, add = torch.exp(log_f[t] + m - new), torch.exp(log_i[t] - new)
        S.mul_(keep[:, None, None]).add_((add[:, None] * k[t])[:, :, None] * v[t][:, None, :])
        n.mul_(keep[:, None]).add_(add[:, None] * k[t])
        m.copy_(new)
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out


# ---- state space (Mamba-2) ---------------------------------------------------------------------------------------------
def conv_tokens(x: torch.Tensor, before: torch.Tensor, w: torch.Tensor, bias: torch.Tensor):
    """Causal convolution per channel and silu of one sequence's rows ``x`` [T, C] after its inputs ``before`` [taps - 1, C];
    ``w`` [taps, C] with the row's own tap last.  Returns the result and the last taps - 1 inputs."""
    taps, T = w.shape[0], x.shape[0]
    full = torch.cat([before, x])
    y = bias + sum(w[j] * full[j: j + T] for j in range(taps))
    return torch.nn.functional.silu(y), full[T:]


def state_space_tokens(x, B, C, dt, neg_a, D, S):
    """Tokens of one sequence through one layer's memory.  x [T, H, v], B and C [T, G, n], dt [T, H], neg_a [H] = -exp(A_log);
    S [H, n, v] is updated in place.  Returns the read-outs [T, H, v]."""
    H, G = x.shape[1], B.shape[1]
    out = torch.empty_like(x)
    for t in range(x.shape[0]):
        b, c = (z[t].repeat_interleave(H // G, 0) for z in (B, C))
        S.mul_(torch.exp(neg_a * dt[t])[:, None, None]).add_((dt[t][:, None] * b)[:, :, None] * x[t][:, None, :])
        out[t] = torch.einsum("hnv,hn->hv", S, c) + D[:, None] * x[t]
    return out


# ---- gated linear attention -------------------------------------------------------------------------------------------
def log_decays(u: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, tau: float) -> torch.Tensor:
    """Logarithms of the decays [T, heads * dim] from their inner vectors ``u`` [T, rank], fp32."""
    return torch.nn.functional.logsigmoid(u.float() @ w.float().T + bias) / tau


def gated_linear_tokens(q, k, v, log_alpha, S):
    """Tokens of one sequence through one layer's memory.  q, k, log_alpha [T, H, d] and v [T, H, vd] fp32; S [H, d, vd] is
    updated in place.  Returns the read-outs [T, H, vd]."""
    out = torch.empty_like(v)
    for t in range(q.shape[0]):
        S.mul_(torch.exp(log_alpha[t])[:, :, None]).add_(k[t][:, :, None] * v[t][:, None, :])
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def conv_inputs(h: torch.Tensor, before: torch.Tensor, w: torch.Tensor):
    """One sequence's rows ``h`` [T, C] plus their causal convolution per channel, after the inputs ``before`` [taps - 1, C];
    ``w`` [taps, C] with the row's own tap last.  Returns the result and the last taps - 1 inputs."""
    taps, T = w.shape[0], h.shape[0]
    full = torch.cat([before, h])
    return h + sum(w[j] * full[j: j + T] for j in range(taps)), full[T:]


# ---- feed-forwards ----------------------------------------------------------------------------------------------------
def relu2(x: torch.Tensor) -> torch.Tensor:
    return torch.relu(x).square()


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def glu(kind: str, g: torch.Tensor, u: torch.Tensor, limit: float = 0.0) -> torch.Tensor:
    """Gated activations: "silu_glu" silu(g) u, "gelu_tanh_glu" gelu(g) u, "clamped_glu" g sigmoid(1.702 g) (u + 1) with g
    clamped from above and u from both sides."""
    if kind == "clamped_glu":
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        return g * torch.sigmoid(1.702 * g) * (u + 1.0)
    return {"silu_glu": torch.nn.functional.silu, "gelu_tanh_glu": gelu_tanh}[kind](g) * u


def best_groups(scores: torch.Tensor, groups: int, keep: int) -> torch.Tensor:
    """[T, experts] bool: experts of the ``keep`` groups whose two largest scores have the largest sum (the lower group on a
    tie)."""
    per = scores.view(scores.shape[0], groups, -1)
    total = torch.topk(per, min(2, per.shape[-1]), dim=-1).values.sum(-1)
    best = torch.sort(total, dim=-1, descending=True, stable=True).indices[:, :keep]
    return torch.zeros_like(total, dtype=torch.bool).scatter_(1, best, True)[:, :, None].expand_as(per).reshape(scores.shape)


def route(logits: torch.Tensor, moe):
    """(expert ids [T, top], their weights): largest scores first, the lower id on a tie."""
    s = torch.sigmoid(logits.float()) if moe.score == "sigmoid" else torch.softmax(logits.float(), -1)
    if moe.keep_groups < moe.groups:
        s = s.masked_fill(~best_groups(s, moe.groups, moe.keep_groups), -1.0)
    w, e = torch.sort(s, dim=-1, descending=True, stable=True)
    e, w = e[:, : moe.top], w[:, : moe.top]
    if moe.normalise:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return e, w * moe.scale
