"""ctypes binding of ``libzse_b200.so`` (see ``csrc/api.h``) on torch tensors.

Every call launches on ``torch.cuda.current_stream()``, so the kernels order with torch ops and are captured by
``torch.cuda.graph``.  A negative return code raises ``NativeError``; device-side failures are read with
``check_status``.  On a machine with a GPU a missing library is an error, never a silent fallback.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import c_char_p, c_float, c_int, c_int32, c_int64, c_uint64, c_void_p, POINTER, Structure, byref, c_uint32
from typing import Optional

import torch

from . import build as _build

_ERRORS = {-1: "unsupported shape", -2: "misaligned pointer or stride", -3: "CUDA driver call failed",
           -4: "kernel launch failed", -5: "size beyond a built-in limit"}


class NativeError(RuntimeError):
    pass


class DeviceStatusError(RuntimeError):
    """A kernel reported a failure through the status word (bounded wait ran out, bad index, ...)."""


# mirrors of the structs in csrc/api.h
class TileGemm(Structure):
    _fields_ = [("a", c_void_p), ("lda", c_int64), ("a_batch", c_int64), ("b", c_void_p), ("ldb_n", c_int64),
                ("ldb_k", c_int64), ("b_batch", c_int64), ("b_group", c_int64), ("out", c_void_p), ("ldo", c_int64),
                ("o_batch", c_int64), ("M", c_int32), ("N", c_int32), ("K", c_int32), ("epilogue", c_int32),
                ("row_scale", c_void_p), ("out_rows", c_void_p), ("out_row_mul", c_int32), ("out_row_add", c_int32),
                ("gate", c_void_p), ("ldg", c_int64), ("gate_batch", c_int64), ("tiles", c_void_p),
                ("n_tiles", c_void_p)]


class RowCache(Structure):
    _fields_ = [("rows", c_void_p), ("block_stride", c_int64), ("block_size", c_int32), ("row", c_int32),
                ("tables", c_void_p), ("max_blocks", c_int32), ("num_blocks", c_int32)]


class Chunks(Structure):
    _fields_ = [("cu_q", c_void_p), ("q_pos0", c_void_p), ("ctx_off", c_void_p), ("first", c_int32), ("last", c_int32),
                ("window", c_int32)]


class Router(Structure):
    _fields_ = [("planes", c_void_p)] + [(n, c_int32) for n in ("n_planes", "experts", "cols", "top", "softmax",
                                                                "normalise")] + [("scale", c_float), ("groups", c_int32),
                                                                                 ("keep", c_int32)]


class MoeGemm(Structure):
    _fields_ = [(n, c_void_p) for n in ("routed_w", "routed_x", "routed_out", "shared_w", "shared_x", "shared_out",
                                        "row_score", "out_rows", "tiles", "n_tiles", "shared_score")] + \
               [(n, c_int32) for n in ("routed_n", "routed_k", "routed_ldo", "shared_n", "shared_k", "shared_ldo",
                                       "shared_mul", "shared_add", "shared_x_rows", "routed_cols", "shared_cols")] + \
               [("routed_limit", c_float), ("shared_limit", c_float), ("glu", c_int32)]


class Embed(Structure):
    _fields_ = [(n, c_void_p) for n in ("table", "bigram", "norm", "turns", "ids", "positions", "row_seq", "cu_q",
                                        "state_rows", "last_token", "residual", "out")] + \
               [(n, c_int64) for n in ("buckets", "mul_prev", "mul_cur")] + \
               [("H", c_int32), ("vocab", c_int32), ("state_ld", c_int32), ("scale", c_float), ("eps", c_float)]


class Heads(Structure):
    _fields_ = [("k", c_void_p), ("v", c_void_p), ("block_stride", c_int64)] + \
               [(n, c_int32) for n in ("block_size", "dim_pad", "vdim_pad", "max_blocks")] + [("tables", c_void_p)] + \
               [(n, c_int32) for n in ("heads", "kv_heads", "dim", "vdim", "chunk", "window")] + [("scale", c_float),
                   ("num_blocks", c_int32), ("keep_first", c_int32), ("softcap", c_float), ("gate_each", c_int32),
                   ("pool", c_int32), ("means_at", c_int32), ("sink", c_void_p), ("out_scale", c_float)]


class HeadsPrep(Structure):
    _fields_ = [(n, c_void_p) for n in ("q_norm", "k_norm", "bias", "turns", "positions")] + \
               [(n, c_int32) for n in ("k_col", "v_col", "gate_col", "gate_w", "own_kv", "rot_dims")] + \
               [("temp_coef", c_float), ("temp_every", c_int32), ("eps", c_float), ("whole", c_int32),
                ("head_temp", c_void_p), ("pool_rows", c_int32)]


class RowConv(Structure):
    _fields_ = [("w", c_void_p), ("taps", c_int32), ("states", c_void_p), ("row_floats", c_int64), ("state_rows", c_void_p),
                ("state_ld", c_int32)]


class GatedLinear(Structure):
    _fields_ = [(n, c_int32) for n in ("heads", "dim", "vdim", "rank", "q_col", "k_col", "v_col", "gate_col", "rank_col")] + \
               [("states", c_void_p), ("row_floats", c_int64), ("state_rows", c_void_p), ("state_ld", c_int32),
                ("tau", c_float), ("eps", c_float), ("out_scale", c_float)] + \
               [(n, c_void_p) for n in ("head_norm", "decay_w", "decay_b")]


class Memory(Structure):
    _fields_ = [(n, c_int32) for n in ("heads", "dim", "vdim", "k_col", "v_col", "gate_col", "if_col")] + \
               [("states", c_void_p), ("row_floats", c_int64), ("sum_at", c_int32), ("max_at", c_int32),
                ("state_rows", c_void_p), ("state_ld", c_int32), ("gate_cap", c_float), ("eps", c_float),
                ("head_norm", c_void_p)]


class Space(Structure):
    _fields_ = [(n, c_int32) for n in ("heads", "vdim", "state", "groups", "taps", "x_col", "b_at", "c_at", "conv_width",
                                       "dt_col")] + \
               [("states", c_void_p), ("row_floats", c_int64), ("conv_at", c_int32), ("state_rows", c_void_p),
                ("state_ld", c_int32)] + [(n, c_void_p) for n in ("conv_w", "conv_b", "dt_bias", "neg_a", "skip")]


_lib: Optional[ctypes.CDLL] = None

_SIGS = {
    "zse_gemm_w4": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
                            c_void_p, c_void_p]),
    "zse_gemm_w4_splits": (c_int, [c_int, c_int, c_int, c_int]),
    "zse_gemm_w4_dec": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                c_void_p, c_void_p, c_void_p]),
    "zse_gemm_w4_dec_qkv_rope": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                         c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p,
                                         c_void_p, c_void_p]),
    "zse_gemm_w8_dec": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                c_void_p, c_void_p, c_void_p]),
    "zse_gemm_w8_dec_qkv_rope": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                         c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p,
                                         c_void_p, c_void_p]),
    "zse_w8_tiled_bytes": (c_int64, [c_int, c_int]),
    "zse_repack_w8": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "zse_dequant_w8_tiled": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "zse_gemm_w4_dec_workspace_bytes": (c_int64, [c_int]),
    "zse_gemm_w4_dec_supported": (c_int, [c_int, c_int, c_int, c_int]),
    "zse_gemm_w4_dec_plan": (None, [c_int, c_int, c_int, c_int, POINTER(c_int)]),
    "zse_gemm_w4_dec_set_tuning": (None, [c_int, c_int]),
    "zse_gemm_f16": (c_int, [c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                             c_int, c_void_p, c_void_p]),
    "zse_gemm_f16_splits": (c_int, [c_int, c_int, c_int, c_int]),
    "zse_w4_tiled_bytes": (c_int64, [c_int, c_int]),
    "zse_repack_w4": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "zse_dequant_w4": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int64, c_int, c_void_p]),
    "zse_dequant_w8": (c_int, [c_void_p, c_void_p, c_void_p, c_int64, c_int, c_void_p]),
    "zse_quantize_w4": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int64, c_void_p]),
    "zse_embedding": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_void_p, c_void_p]),
    "zse_add_rmsnorm": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float,
                                c_void_p]),
    "zse_rmsnorm_f16": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p]),
    "zse_rope_kv_write": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                  c_int, c_void_p, c_int, c_void_p, c_void_p]),
    "zse_swiglu": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "zse_headnorm_rope_kv_write": (c_int, [c_void_p, c_int, c_void_p, c_int64, c_int64, c_void_p, c_void_p, c_void_p,
                                           c_void_p, c_void_p, c_int, c_int, c_float, c_int, c_int, c_int, c_int,
                                           c_int, c_void_p]),
    "zse_attn_generic": (c_int, [c_void_p, c_int, c_void_p, c_int64, c_int64, c_void_p, c_int, c_void_p, c_void_p,
                                 c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_float,
                                 c_int, c_void_p]),
    "zse_norm_add_rmsnorm": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                     c_float, c_void_p]),
    "zse_softcap_f16": (c_int, [c_void_p, c_int, c_int, c_int, c_float, c_void_p]),
    "zse_bias_add": (c_int, [c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "zse_attn_decode_scratch_floats": (c_int64, [c_int, c_int, c_int, c_int]),
    "zse_attn_decode": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                c_int, c_int, c_int, c_int, c_int, c_float, c_void_p]),
    "zse_attn_prefill": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int,
                                 c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_void_p]),
    "zse_attn_decode_ext": (c_int, [c_void_p, c_int, c_void_p, c_int64, c_int64, c_void_p, c_int, c_void_p, c_void_p,
                                    c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_float, c_int,
                                    c_void_p]),
    "zse_attn_prefill_ext": (c_int, [c_void_p, c_int, c_void_p, c_int64, c_int64, c_void_p, c_int, c_void_p, c_void_p,
                                     c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_float,
                                     c_int, c_void_p]),
    "zse_argmax": (c_int, [c_void_p, c_int, c_void_p, c_int, c_int, c_void_p]),
    "zse_sample": (c_int, [c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_uint64,
                           c_void_p]),
    "zse_apply_repetition_penalty": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                             c_void_p]),
    "zse_apply_repetition_penalty_f32": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                                 c_void_p]),
    "zse_lora_shrink": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p]),
    "zse_attn_prefill_tc": (c_int, [c_void_p, c_int, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
                                    c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_void_p, c_void_p]),
    "zse_lora_apply": (c_int, [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
                               c_int, c_int, c_void_p]),
    "zse_lora_expand": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                c_void_p]),
    "zse_tp_ctx_create": (c_void_p, [c_int, c_int, c_int, c_int, POINTER(c_uint64), POINTER(c_uint64), c_uint64,
                                     POINTER(c_uint64), POINTER(c_uint64)]),
    "zse_tp_ctx_destroy": (None, [c_void_p]),
    "zse_tp_reduce_add_rmsnorm": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_float,
                                          c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_reduce_add_rmsnorm_emulated": (c_int, [c_void_p, POINTER(c_uint64), POINTER(c_uint64), c_int, c_void_p,
                                                   POINTER(c_uint64), c_int, c_float, c_int, c_void_p, c_void_p]),
    "zse_tp_reduce_scatter_add_rmsnorm": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_float,
                                          c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_reduce_scatter_add_rmsnorm_emulated": (c_int, [c_void_p, POINTER(c_uint64), POINTER(c_uint64), c_int, c_void_p,
                                                   POINTER(c_uint64), c_int, c_float, c_int, c_void_p, c_void_p]),
    "zse_tp_ctx_set_push": (c_int, [c_void_p, c_int, POINTER(c_uint64), c_uint64, POINTER(c_uint64), c_uint64,
                                    POINTER(c_uint64)]),
    "zse_tp_gemm_w4_push": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                    c_void_p, c_void_p]),
    "zse_tp_gemm_dec_allreduce_norm": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                               c_int, c_int, c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_void_p,
                                               c_void_p]),
    "zse_tp_sum_add_rmsnorm": (c_int, [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_float, c_int, c_int, c_void_p,
                                       c_void_p]),
    "zse_tp_ctx_set_sp": (c_int, [c_void_p, c_int, c_int, POINTER(c_uint64), POINTER(c_uint64), POINTER(c_uint64),
                                  c_uint64, POINTER(c_uint64), POINTER(c_uint64)]),
    "zse_tp_gemm_w4_scatter": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p,
                                       c_void_p]),
    "zse_tp_gemm_w4_gathered": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int,
                                        c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_sp_sum_norm_gather": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_float, c_int, c_int, c_void_p,
                                          c_void_p]),
    "zse_tp_sp_sum_norm_gather_emulated": (c_int, [c_void_p, POINTER(c_uint64), c_void_p, c_int, c_float, c_int,
                                                   c_void_p, c_void_p]),
    "zse_tp_sp_wait": (c_int, [c_void_p, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_sum_add_rmsnorm_emulated": (c_int, [c_void_p, POINTER(c_uint64), c_void_p, POINTER(c_uint64), c_int,
                                                c_float, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_ctx_set_gather": (c_int, [c_void_p, c_int, c_int, POINTER(c_uint64), POINTER(c_uint64)]),
    "zse_gemm_bf16": (c_int, [c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
                              c_void_p, c_void_p]),
    "zse_gemm_bf16_glu": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p,
                                  c_void_p]),
    "zse_gemm_bf16_side": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_int, c_void_p,
                                   c_void_p]),
    "zse_gemm_tile": (c_int, [c_int, POINTER(TileGemm), c_int, c_int, c_void_p]),
    "zse_embedding_typed": (c_int, [c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_void_p, c_int,
                                    c_void_p, c_void_p]),
    "zse_add_norm": (c_int, [c_int, c_int, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_float,
                             c_void_p, c_int, c_int, c_int, c_float, c_void_p]),
    "zse_add_norm_conv": (c_int, [c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, POINTER(RowConv), c_void_p, c_int,
                                  c_int, c_float, c_void_p]),
    "zse_row_conv": (c_int, [c_int, c_void_p, c_void_p, POINTER(RowConv), c_void_p, c_void_p, c_int, c_int, c_void_p]),
    "zse_logits_finish": (c_int, [c_void_p, c_int, c_int, c_int, c_float, c_float, c_void_p]),
    "zse_argmax_f32": (c_int, [c_void_p, c_int, c_void_p, c_int, c_int, c_void_p]),
    "zse_latent_mma_ok": (c_int, [c_int] * 6),
    "zse_latent_prep": (c_int, [c_int, c_void_p, c_int, c_void_p, c_int, c_int, POINTER(RowCache), c_void_p, c_void_p,
                                c_void_p, c_void_p] + [c_int] * 8 + [c_float, c_void_p]),
    "zse_latent_attn": (c_int, [c_int, c_void_p, POINTER(RowCache), c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                c_int, c_int, c_int, c_float, c_int, c_int, c_void_p, c_void_p]),
    "zse_latent_absorb": (c_int, [c_void_p, c_int, c_void_p, c_void_p] + [c_int] * 6 + [c_void_p]),
    "zse_latent_unabsorb": (c_int, [c_void_p, c_void_p, c_void_p, c_int, c_void_p] + [c_int] * 5 + [c_void_p]),
    "zse_latent_gather": (c_int, [POINTER(RowCache), POINTER(Chunks), c_int, c_int, c_int, c_void_p, c_void_p, c_void_p]),
    "zse_latent_chunk": (c_int, [c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, POINTER(RowCache), POINTER(Chunks),
                                 c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_float, c_void_p]),
    "zse_moe_tile_rows": (c_int, [c_int, c_int, c_int]),
    "zse_moe_route": (c_int, [c_int, POINTER(Router), c_int, c_int, c_void_p, c_int, c_int] + [c_void_p] * 12),
    "zse_post_norm": (c_int, [c_int, c_int, c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int,
                              c_int, c_float, c_void_p]),
    "zse_embed_design": (c_int, [c_int, POINTER(Embed), c_int, c_void_p, c_void_p]),
    "zse_glu": (c_int, [c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_float, c_void_p]),
    "zse_heads_mma_ok": (c_int, [c_int] * 3),
    "zse_heads_prep": (c_int, [c_int, c_void_p, c_int, c_void_p, c_int, c_int, POINTER(Heads), c_void_p, POINTER(HeadsPrep),
                               c_void_p]),
    "zse_heads_pool": (c_int, [c_int, POINTER(Heads), c_void_p, c_void_p, c_int, c_void_p]),
    "zse_heads_attn": (c_int, [c_int, c_void_p, c_int, POINTER(Heads), c_void_p, c_void_p, c_void_p, c_int, c_void_p,
                               c_void_p, c_int, c_int, c_int, c_void_p]),
    "zse_heads_attn_chunks": (c_int, [c_void_p, c_int, c_int, POINTER(Heads), c_void_p, c_void_p, c_int, c_int, c_int,
                                      c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p]),
    "zse_memory_chunk_ok": (c_int, [c_int] * 2),
    "zse_memory_prep": (c_int, [c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p,
                                POINTER(Memory), c_int, c_void_p]),
    "zse_memory_tokens": (c_int, [c_int, c_void_p, c_int, c_void_p, POINTER(Memory), c_void_p, c_int, c_void_p, c_int,
                                  c_void_p]),
    "zse_memory_chunks": (c_int, [c_void_p, c_int, c_void_p, POINTER(Memory), c_void_p, c_int, c_int, c_void_p, c_int, c_int,
                                  c_void_p, c_int, c_void_p]),
    "zse_space_chunk_ok": (c_int, [c_int] * 2),
    "zse_space_prep": (c_int, [c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, POINTER(Space), c_void_p, c_void_p,
                               c_void_p, c_void_p, c_int, c_void_p]),
    "zse_space_tokens": (c_int, [c_int, c_void_p, c_int, c_void_p, c_void_p, POINTER(Space), c_void_p, c_int, c_void_p, c_int,
                                 c_void_p]),
    "zse_space_chunks": (c_int, [c_void_p, c_int, c_void_p, c_void_p, POINTER(Space), c_void_p, c_int, c_int, c_void_p, c_int,
                                 c_void_p]),
    "zse_gated_linear_chunk_ok": (c_int, [c_int] * 2),
    "zse_gated_linear_prep": (c_int, [c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, POINTER(GatedLinear), c_void_p,
                                      c_int, c_void_p]),
    "zse_gated_linear_tokens": (c_int, [c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, POINTER(GatedLinear),
                                        c_void_p, c_int, c_void_p, c_int, c_void_p]),
    "zse_gated_linear_chunks": (c_int, [c_void_p, c_int, c_void_p, POINTER(GatedLinear), c_void_p, c_int, c_int, c_void_p,
                                        c_int, c_int, c_void_p, c_int, c_void_p]),
    "zse_group_norm": (c_int, [c_int, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_float, c_void_p]),
    "zse_moe_gemm": (c_int, [POINTER(MoeGemm), c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "zse_read_probe": (c_int, [c_void_p, c_int64, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_gather_rows": (c_int, [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_gather_rows_emulated": (c_int, [c_void_p, POINTER(c_uint64), c_int, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_argmax": (c_int, [c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_void_p]),
    "zse_tp_argmax_emulated": (c_int, [c_void_p, POINTER(c_uint64), c_int, POINTER(c_uint64), c_int, c_int, c_int,
                                       c_int, c_void_p, c_void_p]),
    "zse_status_read": (c_int, [c_void_p, POINTER(c_uint32)]),
    "zse_device_info": (c_int, [POINTER(c_int), POINTER(c_int), POINTER(c_int), POINTER(c_int64), POINTER(c_int64)]),
    "zse_build_info": (c_char_p, []),
    "zse_set_pdl": (None, [c_int]),
    "zse_gemm_w4_set_mode": (None, [c_int]),
    "zse_get_pdl": (c_int, []),
}


def lib_path() -> str:
    """The library this process loads: the ordinary build, or the file ZSE_NATIVE_LIB names (an instrumented variant
    built by ``python -m zse_b200.ops.build --variant NAME``)."""
    return os.environ.get("ZSE_NATIVE_LIB") or _build.LIB_PATH


_partial = False         # _lib is a subset of the library (build.GROUPS)


def load(build_if_missing: bool = True, group: Optional[str] = None, whole: bool = False) -> ctypes.CDLL:
    """The native library this process has loaded, or loads now.  ``group``: the caller needs the kernels of that group
    only (``build.GROUPS``); where the whole library has not been built, the group's own is built and loaded instead.
    ``whole``: every kernel is needed, a loaded subset is replaced."""
    global _lib, _partial
    if _lib is not None and not (whole and _partial):
        return _lib
    path = lib_path()
    partial = False
    if not os.path.exists(path):
        if group is not None and build_if_missing:
            path, partial = _build.group_path(group), True
            if not os.path.exists(path):
                _build.build_group(group)
        elif not build_if_missing:
            raise NativeError(f"{path} is missing: run `python -m zse_b200.ops.build`")
        else:
            _build.build()
    lib = ctypes.CDLL(path)
    for name, (res, args) in _SIGS.items():
        fn = getattr(lib, name, None)
        if fn is None:
            continue   # optional entry points are looked up by their users
        fn.restype, fn.argtypes = res, args
    _lib, _partial = lib, partial
    return lib


def available() -> bool:
    return torch.cuda.is_available()


def _p(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


LAUNCHES = [0]      # kernels launched through this module (graph replays are accounted by the runner)


def _ck(rc: int, what: str, launches: int = 1) -> None:
    if rc < 0:
        raise NativeError(f"{what}: {_ERRORS.get(rc, rc)}")
    LAUNCHES[0] += launches


class Status:
    """The 16-byte device status word shared by all launches of one engine."""

    def __init__(self, device):
        self.buf = torch.zeros(4, dtype=torch.int32, device=device)

    @property
    def ptr(self) -> int:
        return self.buf.data_ptr()

    def read(self):
        out = (c_uint32 * 4)()
        _ck(load().zse_status_read(self.ptr, out), "status read", 0)
        return tuple(out)

    def check(self) -> None:
        code, block, where, detail = self.read()
        if code:
            self.buf.zero_()
            kind = {1: "wait timed out", 2: "bad argument", 3: "peer wait timed out"}.get(code, f"code {code}")
            raise DeviceStatusError(f"device reported: {kind} (block {block}, site {where}, detail {detail})")


# ---- thin wrappers (shapes are checked by the callers in ops/linear.py and the model runner) -------------------
def gemm_w4(w_tiled, x, x_rows_cap, bias, out, M, N, K, ldo, epilogue, k_split, status):
    _ck(load().zse_gemm_w4(_p(w_tiled), _p(x), x_rows_cap, _p(bias), _p(out), M, N, K, ldo, epilogue, k_split,
                           status, _stream()), "gemm_w4")


def gemm_w4_dec(w_tiled, x, x_rows_cap, bias, out, M, N, K, ldo, epilogue, workspace, status):
    """Decode-sized INT4 GEMM (M <= 64) of the persistent kernel; epilogue 0 fp16 (+bias), 1 SwiGLU, 2 fp32."""
    _ck(load().zse_gemm_w4_dec(_p(w_tiled), _p(x), x_rows_cap, _p(bias), _p(out), M, N, K, ldo, epilogue,
                               _p(workspace), status, _stream()), "gemm_w4_dec")


def gemm_w4_dec_qkv_rope(w_tiled, x, x_rows_cap, bias, qkv_out, ldo, M, K, nh, nkv, kv_layer, block_size, positions,
                         slots, cos_sin, max_position, workspace, status):
    _ck(load().zse_gemm_w4_dec_qkv_rope(_p(w_tiled), _p(x), x_rows_cap, _p(bias), _p(qkv_out), ldo, M, K, nh, nkv,
                                        _p(kv_layer), block_size, _p(positions), _p(slots), _p(cos_sin), max_position,
                                        _p(workspace), status, _stream()), "gemm_w4_dec_qkv_rope")


def gemm_w8_dec(w_tiled, x, x_rows_cap, bias, out, M, N, K, ldo, epilogue, workspace, status):
    """The decode-sized GEMM for INT8 weights tiled by ``repack_w8`` (the weights stay 8 bits wide in memory)."""
    _ck(load().zse_gemm_w8_dec(_p(w_tiled), _p(x), x_rows_cap, _p(bias), _p(out), M, N, K, ldo, epilogue,
                               _p(workspace), status, _stream()), "gemm_w8_dec")


def gemm_w8_dec_qkv_rope(w_tiled, x, x_rows_cap, bias, qkv_out, ldo, M, K, nh, nkv, kv_layer, block_size, positions,
                         slots, cos_sin, max_position, workspace, status):
    _ck(load().zse_gemm_w8_dec_qkv_rope(_p(w_tiled), _p(x), x_rows_cap, _p(bias), _p(qkv_out), ldo, M, K, nh, nkv,
                                        _p(kv_layer), block_size, _p(positions), _p(slots), _p(cos_sin), max_position,
                                        _p(workspace), status, _stream()), "gemm_w8_dec_qkv_rope")


def repack_w8(q, scales, out_tiled, N, K, interleave_rows=0):
    _ck(load().zse_repack_w8(_p(q), _p(scales), _p(out_tiled), N, K, interleave_rows, _stream()), "repack_w8")


def dequant_w8_tiled(tiled, out_f16, N, K, interleave_rows=0):
    _ck(load().zse_dequant_w8_tiled(_p(tiled), _p(out_f16), N, K, interleave_rows, _stream()), "dequant_w8_tiled")


def gemm_w4_dec_workspace(device, sm_count: int) -> torch.Tensor:
    """Zeroed workspace (partial sums + synchronisation words) for the persistent decode GEMM on ``device``."""
    n = int(load().zse_gemm_w4_dec_workspace_bytes(sm_count))
    return torch.zeros((n + 15) // 16 * 16, dtype=torch.uint8, device=device)


def gemm_w4_dec_supported(M, N, K, epilogue) -> bool:
    return bool(load().zse_gemm_w4_dec_supported(M, N, K, epilogue))


def gemm_w4_dec_plan(N, K, epilogue, sm_count):
    out = (c_int * 2)()
    load().zse_gemm_w4_dec_plan(N, K, epilogue, sm_count, out)
    return out[0], out[1]


def gemm_f16(w, w_rows, x, x_rows_cap, bias, out, M, N, K, ldo, epilogue, k_split, status):
    _ck(load().zse_gemm_f16(_p(w), w_rows, _p(x), x_rows_cap, _p(bias), _p(out), M, N, K, ldo, epilogue, k_split,
                            status, _stream()), "gemm_f16")


def gemm_w4_splits(M, N, K, k_split) -> int:
    return load().zse_gemm_w4_splits(M, N, K, k_split)


def gemm_f16_splits(M, N, K, k_split) -> int:
    return load().zse_gemm_f16_splits(M, N, K, k_split)


def w4_tiled_bytes(N, K) -> int:
    return load().zse_w4_tiled_bytes(N, K)


def repack_w4(packed, scales, zeros, out, N, K, interleave_rows=0):
    _ck(load().zse_repack_w4(_p(packed), _p(scales), _p(zeros), _p(out), N, K, interleave_rows, _stream()),
        "repack_w4")


def dequant_w4(packed, scales, zeros, out, n_elements, group_size):
    _ck(load().zse_dequant_w4(_p(packed), _p(scales), _p(zeros), _p(out), n_elements, group_size, _stream()),
        "dequant_w4")


def dequant_w8(q, scales, out, n_elements, group_size):
    _ck(load().zse_dequant_w8(_p(q), _p(scales), _p(out), n_elements, group_size, _stream()), "dequant_w8")


def quantize_w4(w, packed, scales, zeros, n_groups):
    _ck(load().zse_quantize_w4(_p(w), _p(packed), _p(scales), _p(zeros), n_groups, _stream()), "quantize_w4")


def embedding(table, ids, out, M, H, vocab, scale, status):
    _ck(load().zse_embedding(_p(table), _p(ids), _p(out), M, H, vocab, scale, status, _stream()), "embedding")


def add_rmsnorm(residual, partials, n_partials, add_f16, weight, out, M, H, eps):
    _ck(load().zse_add_rmsnorm(_p(residual), _p(partials), n_partials, _p(add_f16), _p(weight), _p(out), M, H, eps,
                               _stream()), "add_rmsnorm")


def rmsnorm_f16(x, weight, out, M, H, eps):
    _ck(load().zse_rmsnorm_f16(_p(x), _p(weight), _p(out), M, H, eps, _stream()), "rmsnorm_f16")


def rope_kv_write(qkv, kv_layer, positions, slots, inv_freq, M, nh, nkv, hd, rotary_dim, block_size, planes=None,
                  n_planes=0, bias=None):
    _ck(load().zse_rope_kv_write(_p(qkv), _p(kv_layer), _p(positions), _p(slots), _p(inv_freq), M, nh, nkv, hd,
                                 rotary_dim, block_size, _p(planes), n_planes, _p(bias), _stream()), "rope_kv_write")


def headnorm_rope_kv_write(qkv, kv_layer, positions, slots, freqs, q_norm_w, k_norm_w, norm_v, k_is_v, eps, M, nh, nkv,
                           hd, block_size):
    """``kv_layer``: a (possibly strided) view [blocks, 2, nkv, block_size, hd] whose last three dims are packed."""
    _ck(load().zse_headnorm_rope_kv_write(_p(qkv), qkv.stride(0), _p(kv_layer), kv_layer.stride(0), kv_layer.stride(1),
                                          _p(positions), _p(slots), _p(freqs), _p(q_norm_w), _p(k_norm_w),
                                          int(norm_v), int(k_is_v), float(eps), M, nh, nkv, hd, block_size,
                                          _stream()), "headnorm_rope_kv_write")


def attn_generic(q, ldq, kv_layer, block_tables, seq_lens, cu_q, q_pos0, num_seqs, out, ldo, T, nh, nkv, hd,
                 block_size, scale, softcap=0.0, window=0):
    _ck(load().zse_attn_generic(_p(q), ldq, _p(kv_layer), kv_layer.stride(0), kv_layer.stride(1), _p(block_tables),
                                block_tables.stride(0), _p(seq_lens), _p(cu_q), _p(q_pos0), num_seqs, _p(out), ldo, T,
                                nh, nkv, hd, block_size, float(scale), float(softcap), int(window), _stream()),
        "attn_generic")


def norm_add_rmsnorm(x, w_post, residual, scalar, w_next, out, M, H, eps):
    _ck(load().zse_norm_add_rmsnorm(_p(x), _p(w_post), _p(residual), _p(scalar), _p(w_next), _p(out), M, H, float(eps),
                                    _stream()), "norm_add_rmsnorm")


def softcap(x, M, V, cap):
    _ck(load().zse_softcap_f16(_p(x), x.stride(0), M, V, float(cap), _stream()), "softcap")


def swiglu(gate_up, out, M, I, gelu=False):
    _ck(load().zse_swiglu(_p(gate_up), _p(out), M, I, int(gelu), _stream()), "swiglu")


def read_probe(buf, nbytes, repeats, ctas, sink):
    """Diagnostic: ``ctas`` CTAs read ``nbytes`` of ``buf`` ``repeats`` times (csrc/elementwise.cu)."""
    _ck(load().zse_read_probe(_p(buf), nbytes, repeats, ctas, _p(sink), _stream()), "read_probe")


def bias_add(x, bias, M, N):
    _ck(load().zse_bias_add(_p(x), _p(bias), M, N, _stream()), "bias_add")


def attn_decode_scratch_floats(num_seqs, nh, hd, max_splits) -> int:
    return load().zse_attn_decode_scratch_floats(num_seqs, nh, hd, max_splits)


def attn_decode(q, ldq, kv_layer, block_tables, max_blocks, seq_lens, out, ldo, scratch, num_seqs, nh, nkv, hd,
                block_size, num_splits, scale):
    _ck(load().zse_attn_decode(_p(q), ldq, _p(kv_layer), _p(block_tables), max_blocks, _p(seq_lens), _p(out), ldo,
                               _p(scratch), num_seqs, nh, nkv, hd, block_size, num_splits, scale, _stream()),
        "attn_decode", 2 if num_splits > 1 else 1)


def attn_decode_ext(q, ldq, kv_layer, block_tables, seq_lens, out, ldo, scratch, num_seqs, nh, nkv, hd, block_size,
                    num_splits, scale, softcap=0.0, window=0):
    """``kv_layer``: a (possibly strided) view [blocks, 2, nkv, block_size, hd] whose last three dims are packed."""
    _ck(load().zse_attn_decode_ext(_p(q), ldq, _p(kv_layer), kv_layer.stride(0), kv_layer.stride(1), _p(block_tables),
                                   block_tables.stride(0), _p(seq_lens), _p(out), ldo, _p(scratch), num_seqs, nh, nkv,
                                   hd, block_size, num_splits, float(scale), float(softcap), int(window), _stream()),
        "attn_decode_ext")


def attn_prefill_ext(q, ldq, kv_layer, block_tables, cu_q, q_pos0, out, ldo, num_seqs, max_q_len, nh, nkv, hd,
                     block_size, scale, softcap=0.0, window=0):
    _ck(load().zse_attn_prefill_ext(_p(q), ldq, _p(kv_layer), kv_layer.stride(0), kv_layer.stride(1),
                                    _p(block_tables), block_tables.stride(0), _p(cu_q), _p(q_pos0), _p(out), ldo,
                                    num_seqs, max_q_len, nh, nkv, hd, block_size, float(scale), float(softcap),
                                    int(window), _stream()), "attn_prefill_ext")


def attn_prefill(q, ldq, kv_layer, block_tables, max_blocks, cu_q, q_pos0, out, ldo, num_seqs, max_q_len, nh, nkv,
                 hd, block_size, scale):
    _ck(load().zse_attn_prefill(_p(q), ldq, _p(kv_layer), _p(block_tables), max_blocks, _p(cu_q), _p(q_pos0), _p(out),
                                ldo, num_seqs, max_q_len, nh, nkv, hd, block_size, scale, _stream()), "attn_prefill")


def attn_prefill_tc(q, ldq, total_rows, kv_layer, block_tables, cu_q, q_pos0, out, ldo, num_seqs, max_q_len, nh, nkv, hd,
                    block_size, scale, status, variant=0):
    """Chunked-prefill attention on the tcgen05 tensor cores (csrc/attention_tc.cu); head_dim 128, contiguous cache."""
    _ck(load().zse_attn_prefill_tc(_p(q), ldq, total_rows, _p(kv_layer), kv_layer.shape[0], _p(block_tables),
                                   block_tables.stride(0), _p(cu_q), _p(q_pos0), _p(out), ldo, num_seqs, max_q_len, nh,
                                   nkv, hd, block_size, float(scale), int(variant), status, _stream()),
        "attn_prefill_tc")


def argmax(logits, ld, out, M, V):
    _ck(load().zse_argmax(_p(logits), ld, _p(out), M, V, _stream()), "argmax")


def sample(logits, ld, out, M, V, temperature, top_k, top_p, seeds, step):
    _ck(load().zse_sample(_p(logits), ld, _p(out), M, V, _p(temperature), _p(top_k), _p(top_p), _p(seeds), step,
                          _stream()), "sample")


def apply_repetition_penalty(logits, ld, rows, tokens, counts, n, penalty, V):
    _ck(load().zse_apply_repetition_penalty(_p(logits), ld, _p(rows), _p(tokens), _p(counts), n, _p(penalty), V,
                                            _stream()), "repetition_penalty")


def apply_repetition_penalty_f32(logits, ld, rows, tokens, counts, n, penalty, V):
    _ck(load().zse_apply_repetition_penalty_f32(_p(logits), ld, _p(rows), _p(tokens), _p(counts), n, _p(penalty), V,
                                                _stream()), "repetition_penalty")


def lora_shrink(x, ldx, a, ids, tmp, M, K, rank):
    _ck(load().zse_lora_shrink(_p(x), ldx, _p(a), _p(ids), _p(tmp), M, K, rank, _stream()), "lora_shrink")


def lora_apply(x, ldx, a, b, ids, scales, y, ldy, M, K, N, rank):
    _ck(load().zse_lora_apply(_p(x), ldx, _p(a), _p(b), _p(ids), _p(scales), _p(y), ldy, M, K, N, rank, _stream()),
        "lora_apply")


def lora_expand(tmp, b, ids, scales, y, ldy, M, N, rank):
    _ck(load().zse_lora_expand(_p(tmp), _p(b), _p(ids), _p(scales), _p(y), ldy, M, N, rank, _stream()), "lora_expand")


# ---- bfloat16 / float activations (gemm.cu, gemm_tile.cu, rows.cu, latent.cu, moe.cu) -------------------------------
_DTYPE = {torch.bfloat16: 1, torch.float32: 2}


def gemm_bf16(w, w_rows, x, x_rows_cap, out, M, N, K, ldo, epilogue, k_split, status):
    _ck(load().zse_gemm_bf16(_p(w), w_rows, _p(x), x_rows_cap, _p(out), M, N, K, ldo, epilogue, k_split, status,
                             _stream()), "gemm_bf16")


def gemm_bf16_glu(w, x, x_rows_cap, out, M, N, K, ldo, cols, kind, status):
    _ck(load().zse_gemm_bf16_glu(_p(w), _p(x), x_rows_cap, _p(out), M, N, K, ldo, cols, kind, status, _stream()),
        "gemm_bf16_glu")


def gemm_bf16_side(w, x, x_rows_cap, out, M, N, K, ldo, side, side_col, status):
    _ck(load().zse_gemm_bf16_side(_p(w), _p(x), x_rows_cap, _p(out), M, N, K, ldo, _p(side), side_col, status, _stream()),
        "gemm_bf16_side")


TILE_STORE, TILE_F32, TILE_GELU, TILE_GATE, TILE_RELU2 = 0, 1, 2, 3, 4


def gemm_tile(dtype, a, lda, b, ldb, out, ldo, M, N, K, epilogue=TILE_STORE, batch=1, a_batch=0, b_batch=0, o_batch=0,
              row_scale=None, out_rows=None, out_row=(1, 0), gate=None, ldg=0, gate_batch=0, tiles=None, n_tiles=None,
              max_tiles=0, b_group=0):
    """``ldb``: (stride of n, stride of k) of the second operand; ``out_row``: (mul, add) of the output row."""
    g = TileGemm(_p(a), lda, a_batch, _p(b), ldb[0], ldb[1], b_batch, b_group, _p(out), ldo, o_batch, M, N, K, epilogue,
                 _p(row_scale), _p(out_rows), out_row[0], out_row[1], _p(gate), ldg, gate_batch, _p(tiles), _p(n_tiles))
    _ck(load().zse_gemm_tile(_DTYPE[dtype], byref(g), batch, max_tiles, _stream()), "gemm_tile")


def embedding_typed(table, ids, out, M, H, vocab, scale, copy, status):
    _ck(load().zse_embedding_typed(_DTYPE[table.dtype], _p(table), _p(ids), _p(out), M, H, vocab, scale, _p(copy),
                                   0 if copy is None else copy.stride(0), status, _stream()), "embedding_typed")


def add_norm(residual, planes, n_planes, slots, n_slots, weight, out, M, H, eps, scale=None, offset=0.0, replace=False):
    sd = 0 if slots is None else _DTYPE[slots.dtype]
    _ck(load().zse_add_norm(_DTYPE[out.dtype], sd, _p(residual), _p(planes), n_planes, _p(slots), n_slots, _p(scale),
                            int(replace), _p(weight), float(offset), _p(out), out.stride(0), M, H, eps, _stream()),
        "add_norm")


def post_norm(residual, planes, n_planes, slots, n_slots, weight, next_weight, out, M, H, eps):
    sd = 0 if slots is None else _DTYPE[slots.dtype]
    _ck(load().zse_post_norm(_DTYPE[out.dtype], sd, _p(residual), _p(planes), n_planes, _p(slots), n_slots, _p(weight),
                             _p(next_weight), _p(out), M, H, eps, _stream()), "post_norm")


def embed_design(a: Embed, dtype, M, status):
    _ck(load().zse_embed_design(_DTYPE[dtype], byref(a), M, status, _stream()), "embed_design")


def glu(x, out, rows, ff, kind, limit):
    _ck(load().zse_glu(_DTYPE[x.dtype], _p(x), _p(out), out.stride(0) if out.dim() > 1 else ff, rows, ff, kind, float(limit),
                       _stream()), "glu")


def row_conv_args(w, states, at, state_rows) -> RowConv:
    """``w`` [taps, H]; ``states``: the state pool's rows; ``at``: where the layer's part of a row begins."""
    return RowConv(_p(w), w.shape[0], states.data_ptr() + 4 * at, states.stride(0), _p(state_rows), state_rows.stride(0))


def add_norm_conv(residual, planes, n_planes, weight, out, cv, conv_out, M, H, eps):
    _ck(load().zse_add_norm_conv(_DTYPE[out.dtype], _p(residual), _p(planes), n_planes, _p(weight), _p(out), byref(cv),
                                 _p(conv_out), M, H, eps, _stream()), "add_norm_conv")


def row_conv(h, out, cv, row_seq, cu_q, M, H):
    _ck(load().zse_row_conv(_DTYPE[h.dtype], _p(h), _p(out), byref(cv), _p(row_seq), _p(cu_q), M, H, _stream()), "row_conv")


def heads(view, spec, block_tables, sink=None) -> Heads:
    """``view``: ``models.hybrid.PagedHeads``."""
    return Heads(view.k.data_ptr(), view.v.data_ptr(), view.block_stride, view.block_size, view.k.shape[3], view.v.shape[3],
                 block_tables.stride(0), block_tables.data_ptr(), spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.chunk,
                 spec.window, float(spec.scale), view.k.shape[0], spec.keep_first, float(spec.softcap), int(spec.gate_each),
                 spec.pool, getattr(view, "means_at", 0), _p(sink), float(spec.out_scale))


def heads_mma_ok(spec, block_size: int) -> bool:
    return bool(load().zse_heads_mma_ok(spec.dim, spec.vdim, block_size))


def heads_prep(inp, planes, n_planes, M, h, slots, q_norm, k_norm, bias, turns, positions, spec, eps, head_temp=None,
               pool_rows=False):
    p = HeadsPrep(_p(q_norm), _p(k_norm), _p(bias), _p(turns), _p(positions), spec.k_col,
                  spec.k_col if spec.k_as_v else spec.v_col, spec.gate_col, spec.gate_width, int(spec.own_kv), spec.rot_dims,
                  float(spec.temp_coef), int(spec.temp_every), float(eps), int(spec.whole_norm), _p(head_temp),
                  int(pool_rows))
    _ck(load().zse_heads_prep(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(planes), n_planes, M, byref(h), _p(slots),
                              byref(p), _stream()), "heads_prep")


def heads_pool(h, dtype, row_seq, positions, M):
    _ck(load().zse_heads_pool(_DTYPE[dtype], byref(h), _p(row_seq), _p(positions), M, _stream()), "heads_pool")


def heads_attn(inp, h, row_seq, positions, out, gate, scratch, M, num_splits, tensor_cores):
    _ck(load().zse_heads_attn(_DTYPE[inp.dtype], _p(inp), inp.stride(0), byref(h), _p(row_seq), _p(positions), _p(out),
                              out.stride(0), gate, _p(scratch), M, num_splits, int(tensor_cores), _stream()), "heads_attn",
        2 if num_splits > 1 else 1)


def heads_attn_chunks(inp, h, cu_q, q_pos0, first, last, max_q, out, gate, form, status):
    _ck(load().zse_heads_attn_chunks(_p(inp), inp.stride(0), inp.shape[0], byref(h), _p(cu_q), _p(q_pos0), first, last, max_q,
                                     _p(out), out.stride(0), gate, form, status, _stream()), "heads_attn_chunks")


def memory(states, at, state_rows, head_norm, spec, eps) -> Memory:
    """``states``: the state pool's rows; ``at``: where the layer's part of a row begins."""
    return Memory(spec.heads, spec.dim, spec.vdim, spec.k_col, spec.v_col, spec.gate_col, spec.if_col,
                  states.data_ptr() + 4 * at, states.stride(0), spec.sum_at, spec.max_at, _p(state_rows),
                  state_rows.stride(0), float(spec.gate_cap), float(eps), _p(head_norm))


def memory_chunk_ok(spec) -> bool:
    return bool(load().zse_memory_chunk_ok(spec.dim, spec.vdim))


def memory_prep(inp, planes, n_planes, gate_planes, n_gate_planes, if_bias, gates, spec, M):
    m = Memory(spec.heads, spec.dim, spec.vdim, spec.k_col, spec.v_col, spec.gate_col, spec.if_col, None, 0, 0, 0, None, 0,
               float(spec.gate_cap), 0.0, None)
    _ck(load().zse_memory_prep(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(planes), n_planes, _p(gate_planes),
                               n_gate_planes, _p(if_bias), _p(gates), byref(m), M, _stream()), "memory_prep")


def memory_tokens(inp, gates, m, cu_q, S, out):
    _ck(load().zse_memory_tokens(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(gates), byref(m), _p(cu_q), S, _p(out),
                                 out.stride(0), _stream()), "memory_tokens")


def memory_chunks(inp, gates, m, cu_q, first, last, o, M, row0, out):
    _ck(load().zse_memory_chunks(_p(inp), inp.stride(0), _p(gates), byref(m), _p(cu_q), first, last, _p(o), M, row0, _p(out),
                                 out.stride(0), _stream()), "memory_chunks", 2)


def space(states, at, state_rows, L, spec) -> Space:
    """``states``: the state pool's rows; ``at``: where the layer's part of a row begins; ``L``: the layer's weights."""
    return Space(spec.heads, spec.vdim, spec.state, spec.groups, spec.conv, spec.x_col, spec.b_at, spec.c_at, spec.conv_width,
                 spec.dt_col, states.data_ptr() + 4 * at, states.stride(0), spec.conv_at, _p(state_rows),
                 state_rows.stride(0), _p(L.conv_w), _p(L.conv_b), _p(L.dt_bias), _p(L.neg_a), _p(L.D))


def space_chunk_ok(spec) -> bool:
    return bool(load().zse_space_chunk_ok(spec.state, spec.vdim))


def space_prep(inp, planes, n_planes, side, side_ld, m, row_seq, cu_q, xbc, dt, M):
    _ck(load().zse_space_prep(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(planes), n_planes, _p(side), side_ld, byref(m),
                              _p(row_seq), _p(cu_q), _p(xbc), _p(dt), M, _stream()), "space_prep")


def space_tokens(inp, xbc, dt, m, cu_q, S, out):
    _ck(load().zse_space_tokens(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(xbc), _p(dt), byref(m), _p(cu_q), S, _p(out),
                                out.stride(0), _stream()), "space_tokens")


def space_chunks(inp, xbc, dt, m, cu_q, first, last, out):
    _ck(load().zse_space_chunks(_p(inp), inp.stride(0), _p(xbc), _p(dt), byref(m), _p(cu_q), first, last, _p(out),
                                out.stride(0), _stream()), "space_chunks")


def gated_linear(states, at, state_rows, L, spec, eps) -> GatedLinear:
    """``states``: the state pool's rows (None: of a call that needs none); ``at``: where the layer's part of a row begins."""
    return GatedLinear(spec.heads, spec.dim, spec.vdim, spec.rank, spec.col, spec.k_col, spec.v_col, spec.gate_col,
                       spec.rank_col, None if states is None else states.data_ptr() + 4 * at,
                       0 if states is None else states.stride(0), _p(state_rows),
                       0 if state_rows is None else state_rows.stride(0), float(spec.tau), float(eps), float(spec.out_scale),
                       _p(L.head_norm), _p(L.decay_w), _p(L.decay_b))


def gated_linear_chunk_ok(spec) -> bool:
    return bool(load().zse_gated_linear_chunk_ok(spec.dim, spec.vdim))


def gated_linear_prep(inp, planes, n_planes, side, side_ld, m, decays, M):
    _ck(load().zse_gated_linear_prep(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(planes), n_planes, _p(side), side_ld,
                                     byref(m), _p(decays), M, _stream()), "gated_linear_prep")


def gated_linear_tokens(inp, planes, n_planes, M, decays, m, cu_q, S, out):
    _ck(load().zse_gated_linear_tokens(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(planes), n_planes, M, _p(decays),
                                       byref(m), _p(cu_q), S, _p(out), out.stride(0), _stream()), "gated_linear_tokens")


def gated_linear_chunks(inp, decays, m, cu_q, first, last, o, M, row0, out):
    _ck(load().zse_gated_linear_chunks(_p(inp), inp.stride(0), _p(decays), byref(m), _p(cu_q), first, last, _p(o), M, row0,
                                       _p(out), out.stride(0), _stream()), "gated_linear_chunks", 2)


def group_norm(x, weight, parts, M, eps):
    _ck(load().zse_group_norm(_DTYPE[x.dtype], _p(x), x.stride(0), M, parts, x.shape[1] // parts, _p(weight), float(eps),
                              _stream()), "group_norm")


def logits_finish(logits, M, scale, cap):
    _ck(load().zse_logits_finish(_p(logits), logits.stride(0), M, logits.shape[1], float(scale), float(cap), _stream()),
        "logits_finish")


def argmax_f32(logits, ld, out, M, V):
    _ck(load().zse_argmax_f32(_p(logits), ld, _p(out), M, V, _stream()), "argmax_f32")


def row_cache(rows, block_tables) -> RowCache:
    """``rows``: a layer's cached rows [blocks, block_size, row] (blocks may be strided)."""
    return RowCache(rows.data_ptr(), rows.stride(0), rows.shape[1], rows.shape[2], block_tables.data_ptr(),
                    block_tables.stride(0), rows.shape[0])


def latent_mma_ok(spec) -> bool:
    return bool(load().zse_latent_mma_ok(spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank, spec.row))


def latent_prep(inp, planes, n_planes, M, rc, positions, slots, freqs, norm_w, spec, eps):
    gate_w = spec.heads * spec.vdim if spec.gated else 0
    _ck(load().zse_latent_prep(_DTYPE[inp.dtype], _p(inp), inp.stride(0), _p(planes), n_planes, M, byref(rc),
                               _p(positions), _p(slots), _p(freqs), _p(norm_w), spec.heads, spec.dim, spec.rot_dim,
                               spec.rot_dims, spec.kv_rank, spec.latent_col, spec.gate_col, gate_w, float(eps),
                               _stream()), "latent_prep")


def latent_attn(q_lat, rc, row_seq, positions, o_lat, scratch, M, spec, num_splits, tensor_cores, status):
    _ck(load().zse_latent_attn(_DTYPE[q_lat.dtype], _p(q_lat), byref(rc), _p(row_seq), _p(positions), _p(o_lat),
                               _p(scratch), M, spec.heads, spec.kv_rank + spec.rot_dim, spec.kv_rank, spec.window,
                               float(spec.scale), num_splits, int(tensor_cores), status, _stream()), "latent_attn",
        2 if num_splits > 1 else 1)


def latent_absorb(inp, uk, q_lat, M, spec):
    _ck(load().zse_latent_absorb(_p(inp), inp.stride(0), _p(uk), _p(q_lat), M, spec.heads, spec.dim, spec.rot_dim,
                                 spec.kv_rank, spec.row, _stream()), "latent_absorb")


def latent_unabsorb(o_lat, uv, gate, ldg, out, M, spec):
    _ck(load().zse_latent_unabsorb(_p(o_lat), _p(uv), gate, ldg, _p(out), out.stride(0), M, spec.heads, spec.vdim,
                                   spec.kv_rank, _stream()), "latent_unabsorb")


def latent_gather(rc, chunks, rows, spec, c_out, kr_out):
    _ck(load().zse_latent_gather(byref(rc), byref(chunks), rows, spec.kv_rank, spec.rot_dim, _p(c_out), _p(kr_out),
                                 _stream()), "latent_gather")


def latent_chunk(inp, kvx, ldkv, v_col, kr_ctx, rc, chunks, max_q, out, gate, spec):
    _ck(load().zse_latent_chunk(_p(inp), inp.stride(0), _p(kvx), ldkv, v_col, _p(kr_ctx), byref(rc), byref(chunks),
                                max_q, _p(out), out.stride(0), gate, spec.heads, spec.dim, spec.rot_dim, spec.vdim,
                                float(spec.scale), _stream()), "latent_chunk")


def moe_tile_rows(M, E, top) -> int:
    return load().zse_moe_tile_rows(M, E, top)


def moe_route(planes, n_planes, M, moe, tile_rows, x, H, out_per_token, ws):
    """``moe``: the layer's ``MoESpec``."""
    r = Router(_p(planes), n_planes, moe.experts, moe.router_rows, moe.top, int(moe.score == "softmax"), int(moe.normalise),
               float(moe.scale), moe.groups, moe.keep_groups)
    _ck(load().zse_moe_route(_DTYPE[x.dtype], byref(r), M, tile_rows, _p(x), H, out_per_token,
                             _p(ws.counts), _p(ws.slot_expert), _p(ws.slot_rank), _p(ws.slot_score), _p(ws.first_row),
                             _p(ws.tiles), _p(ws.n_tiles), _p(ws.xs), _p(ws.row_score), _p(ws.out_rows),
                             _p(ws.shared_score), _stream()), "moe_route", 3)


def moe_gemm(g, M, E, max_rows, tile_rows, max_tiles, epilogue, status):
    _ck(load().zse_moe_gemm(byref(g), M, E, max_rows, tile_rows, max_tiles, epilogue, status, _stream()), "moe_gemm")


def _u64s(vals):
    return (c_uint64 * len(vals))(*[int(v) for v in vals])


def tp_ctx_create(tp, rank, m_cap, H, data_ptrs, flag_ptrs, mc_data, xchg_ptrs, xflag_ptrs) -> int:
    ctx = load().zse_tp_ctx_create(tp, rank, m_cap, H, _u64s(data_ptrs), _u64s(flag_ptrs), int(mc_data or 0),
                                   _u64s(xchg_ptrs), _u64s(xflag_ptrs))
    if not ctx:
        raise NativeError("tp_ctx_create: unsupported tensor-parallel size")
    return ctx


def tp_ctx_destroy(ctx) -> None:
    load().zse_tp_ctx_destroy(ctx)


def tp_reduce_add_rmsnorm(ctx, residual, partials, n_planes, weight, out, M, eps, slot, use_multimem, status):
    _ck(load().zse_tp_reduce_add_rmsnorm(ctx, _p(residual), _p(partials), n_planes, _p(weight), _p(out), M, eps,
                                         slot, int(use_multimem), status, _stream()), "tp_reduce_add_rmsnorm",
        (M + 511) // 512)


def tp_reduce_add_rmsnorm_emulated(ctx, residuals, partials, n_planes, weight, outs, M, eps, slot, status):
    _ck(load().zse_tp_reduce_add_rmsnorm_emulated(ctx, _u64s([t.data_ptr() for t in residuals]),
                                                  _u64s([t.data_ptr() for t in partials]), n_planes, _p(weight),
                                                  _u64s([t.data_ptr() for t in outs]), M, eps, slot, status,
                                                  _stream()), "tp_reduce_add_rmsnorm_emulated")


def tp_reduce_scatter_add_rmsnorm(ctx, residual, partials, n_planes, weight, out, M, eps, slot, use_multimem, status):
    _ck(load().zse_tp_reduce_scatter_add_rmsnorm(ctx, _p(residual), _p(partials), n_planes, _p(weight), _p(out), M, eps,
                                         slot, int(use_multimem), status, _stream()), "tp_reduce_scatter_add_rmsnorm",
        (M + 511) // 512)


def tp_reduce_scatter_add_rmsnorm_emulated(ctx, residuals, partials, n_planes, weight, outs, M, eps, slot, status):
    _ck(load().zse_tp_reduce_scatter_add_rmsnorm_emulated(ctx, _u64s([t.data_ptr() for t in residuals]),
                                                  _u64s([t.data_ptr() for t in partials]), n_planes, _p(weight),
                                                  _u64s([t.data_ptr() for t in outs]), M, eps, slot, status,
                                                  _stream()), "tp_reduce_scatter_add_rmsnorm_emulated")


def tp_ctx_set_push(ctx, push_m_cap, inbox_ptrs, mc_inbox, arrive_ptrs, mc_arrive, state_ptrs):
    _ck(load().zse_tp_ctx_set_push(ctx, push_m_cap, _u64s(inbox_ptrs), int(mc_inbox), _u64s(arrive_ptrs), int(mc_arrive),
                                   _u64s(state_ptrs)), "tp_ctx_set_push", 0)


def tp_gemm_w4_push(ctx, w_tiled, x, x_rows_cap, M, N, K, slot, use_multimem, status, rank_override=-1) -> int:
    """Row-parallel INT4 GEMM whose epilogue sends the partial rows to every rank.  Returns its CTA count."""
    rc = load().zse_tp_gemm_w4_push(ctx, _p(w_tiled), _p(x), x_rows_cap, M, N, K, slot, int(use_multimem),
                                    rank_override, status, _stream())
    if rc < 0:
        _ck(rc, "tp_gemm_w4_push")
    LAUNCHES[0] += 1
    return rc


def tp_gemm_dec_allreduce_norm(ctx, w_tiled, int8_weights, x, x_rows_cap, M, N, K, slot, use_multimem, residual,
                               norm_w, xnorm, eps, workspace, status, rank_override=-1):
    """Row-parallel projection + all-reduce + residual add + RMSNorm in one kernel (csrc/gemm_w4_dec.cu)."""
    _ck(load().zse_tp_gemm_dec_allreduce_norm(ctx, _p(w_tiled), int(int8_weights), _p(x), x_rows_cap, M, N, K, slot,
                                              int(use_multimem), rank_override, _p(residual), _p(norm_w), _p(xnorm),
                                              eps, _p(workspace), status, _stream()), "tp_gemm_dec_allreduce_norm")


def tp_ctx_set_sp(ctx, own_cap, nblk_cap, inbox_ptrs, arrive_ptrs, xg_ptrs, mc_xg, gflag_ptrs, state_ptrs):
    _ck(load().zse_tp_ctx_set_sp(ctx, own_cap, nblk_cap, _u64s(inbox_ptrs), _u64s(arrive_ptrs), _u64s(xg_ptrs),
                                 int(mc_xg), _u64s(gflag_ptrs), _u64s(state_ptrs)), "tp_ctx_set_sp", 0)


def tp_gemm_w4_scatter(ctx, w_tiled, x, x_rows_cap, M, N, K, slot, status, rank_override=-1):
    """Row-parallel INT4 GEMM whose epilogue is the reduce-scatter: each 64-row block of partial sums goes to the rank
    that owns it (csrc/gemm_w4.cu, kEpiScatterF16)."""
    _ck(load().zse_tp_gemm_w4_scatter(ctx, _p(w_tiled), _p(x), x_rows_cap, M, N, K, slot, rank_override, status,
                                      _stream()), "tp_gemm_w4_scatter")


def tp_gemm_w4_gathered(ctx, w_tiled, x, x_rows_cap, bias, out, M, N, K, ldo, epilogue, k_split, status,
                        rank_override=-1):
    """zse_gemm_w4 on the gathered activation buffer: the activation producer waits for the row blocks of its token
    tile to arrive from their owners before it loads them (the all-gather's receiving side)."""
    _ck(load().zse_tp_gemm_w4_gathered(ctx, _p(w_tiled), _p(x), x_rows_cap, _p(bias), _p(out), M, N, K, ldo, epilogue,
                                       k_split, rank_override, status, _stream()), "tp_gemm_w4_gathered")


def tp_sp_sum_norm_gather(ctx, residual, weight, M, eps, slot, use_multimem, status):
    _ck(load().zse_tp_sp_sum_norm_gather(ctx, _p(residual), _p(weight), M, eps, slot, int(use_multimem), status,
                                         _stream()), "tp_sp_sum_norm_gather")


def tp_sp_sum_norm_gather_emulated(ctx, residuals, weight, M, eps, slot, status):
    _ck(load().zse_tp_sp_sum_norm_gather_emulated(ctx, _u64s([t.data_ptr() for t in residuals]), _p(weight), M, eps,
                                                  slot, status, _stream()), "tp_sp_sum_norm_gather_emulated")


def tp_sp_wait(ctx, M, status, rank_override=-1):
    _ck(load().zse_tp_sp_wait(ctx, M, rank_override, status, _stream()), "tp_sp_wait")


def tp_sum_add_rmsnorm(ctx, residual, weight, out, M, eps, slot, expected_add, status):
    _ck(load().zse_tp_sum_add_rmsnorm(ctx, _p(residual), _p(weight), _p(out), M, eps, slot, expected_add, status,
                                      _stream()), "tp_sum_add_rmsnorm")


def tp_sum_add_rmsnorm_emulated(ctx, residuals, weight, outs, M, eps, slot, expected_add, status):
    _ck(load().zse_tp_sum_add_rmsnorm_emulated(ctx, _u64s([t.data_ptr() for t in residuals]), _p(weight),
                                               _u64s([t.data_ptr() for t in outs]), M, eps, slot, expected_add,
                                               status, _stream()), "tp_sum_add_rmsnorm_emulated")


def tp_ctx_set_gather(ctx, rows_cap, width, buf_ptrs, flag_ptrs):
    _ck(load().zse_tp_ctx_set_gather(ctx, rows_cap, width, _u64s(buf_ptrs), _u64s(flag_ptrs)), "tp_ctx_set_gather", 0)


def tp_gather_rows(ctx, logits, ld, M, slot, status):
    """All-gather of vocabulary-sharded logits rows into this rank's symmetric buffer (csrc/comm.cu)."""
    _ck(load().zse_tp_gather_rows(ctx, _p(logits), ld, M, slot, status, _stream()), "tp_gather_rows")


def tp_gather_rows_emulated(ctx, logits, ld, M, slot, status):
    _ck(load().zse_tp_gather_rows_emulated(ctx, _u64s([t.data_ptr() for t in logits]), ld, M, slot, status, _stream()),
        "tp_gather_rows_emulated")


def tp_argmax(ctx, logits, ld, out, M, V_local, vocab_stride, slot, status):
    _ck(load().zse_tp_argmax(ctx, _p(logits), ld, _p(out), M, V_local, vocab_stride, slot, status, _stream()),
        "tp_argmax")


def tp_argmax_emulated(ctx, logits, ld, outs, M, V_local, vocab_stride, slot, status):
    _ck(load().zse_tp_argmax_emulated(ctx, _u64s([t.data_ptr() for t in logits]), ld,
                                      _u64s([t.data_ptr() for t in outs]), M, V_local, vocab_stride, slot,
                                      status, _stream()), "tp_argmax_emulated")


def device_info() -> dict:
    sm, maj, mnr, tot, free = c_int(), c_int(), c_int(), c_int64(), c_int64()
    _ck(load().zse_device_info(sm, maj, mnr, tot, free), "device_info", 0)
    return {"sm_count": sm.value, "cc": (maj.value, mnr.value), "total_mem": tot.value, "free_mem": free.value}


def gemm_w4_set_mode(mode: int) -> None:
    """Tuning hook for the INT4 GEMM: 0 = the planner picks the CTA shape, 1 = wide CTAs only, 2 = narrow CTAs (two per
    SM) wherever they are allowed."""
    load().zse_gemm_w4_set_mode(int(mode))


def set_pdl(on: bool) -> None:
    """Programmatic dependent launch between the kernels of a step (on by default, ``ZSE_PDL=0`` switches it off)."""
    load().zse_set_pdl(1 if on else 0)


def pdl_enabled() -> bool:
    return bool(load().zse_get_pdl())


def build_info() -> str:
    return load().zse_build_info().decode()
