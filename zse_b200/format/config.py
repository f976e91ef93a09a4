"""Model and quantisation metadata stored in the CONFIG section.

Field names and defaults follow zse-engine/zse_engine/format/config.py:10-135 so that
files written by either implementation load in the other.  Unknown keys are ignored on
load; this build adds ``quant.int4_layout`` (``"rowmajor"`` or ``"tiled64x8"``), which the
reference loader skips because it filters the quant dict by known keys.
"""
from __future__ import annotations

from dataclasses import dataclass, field, fields
from typing import Any, Dict, List, Optional

from . import serializer
from .layer_specs import (DenseSpec, GatedLinearSpec, HeadsSpec, LatentSpec, LayerSpec, MatrixMemorySpec,  # noqa: F401
                          MoESpec, StateSpaceSpec, TwinSpec, attention_of, read_ff, read_mixer, recurrent_of)
from .spec import DEFAULT_GROUP_SIZE, DEFAULT_QUANT_BITS, QuantMethod


@dataclass
class QuantConfig:
    method: int = int(QuantMethod.INT4_ASYM)
    bits: int = DEFAULT_QUANT_BITS
    group_size: int = DEFAULT_GROUP_SIZE
    scale_dtype: str = "float16"
    tiled_weights: bool = True          # kept for wire compatibility; does not describe the bytes
    int4_layout: Optional[str] = None   # "rowmajor" | "tiled64x8" | None (= not recorded)

    def to_dict(self) -> dict:
        d = {"method": int(self.method), "bits": self.bits, "group_size": self.group_size,
             "scale_dtype": self.scale_dtype, "tiled_weights": self.tiled_weights}
        if self.int4_layout is not None:
            d["int4_layout"] = self.int4_layout
        return d

    @classmethod
    def from_dict(cls, d: dict) -> "QuantConfig":
        names = {f.name for f in fields(cls)}
        return cls(**{k: v for k, v in d.items() if k in names})


@dataclass
class ModelConfig:
    arch: str = "llama"
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 32
    head_dim: int = 128
    hidden_size: int = 4096
    intermediate_size: int = 11008
    vocab_size: int = 32000
    max_seq_len: int = 4096
    rope_theta: float = 10000.0
    rms_norm_eps: float = 1e-5
    rope_scaling: Optional[Dict[str, Any]] = None
    sliding_window: Optional[int] = None
    tie_word_embeddings: bool = False
    # Gemma-family extensions (None/False = not applicable)
    layer_types: Optional[List[str]] = None
    global_head_dim: Optional[int] = None
    global_num_kv_heads: Optional[int] = None
    global_rope_theta: Optional[float] = None
    partial_rotary_factor: Optional[float] = None
    hidden_activation: Optional[str] = None
    final_logit_softcapping: Optional[float] = None
    attn_logit_softcapping: Optional[float] = None
    query_pre_attn_scalar: Optional[float] = None
    attention_k_eq_v: bool = False
    embed_scale: bool = False
    # designs that describe every layer on its own (None = not applicable): ``design_layers[i]`` is the layer's entry of
    # the model's config.json ({"type", "mixer", "mlp"}), ``weight_dtype`` the width its weights are stored in
    design_layers: Optional[List[Dict[str, Any]]] = None
    embed_multiplier: Optional[float] = None
    # {"bigram": {"buckets", "mul_prev", "mul_cur"}, "sinusoid_base", "norm"}: what is added to a token's embedding
    embed_design: Optional[Dict[str, Any]] = None
    # {"start", "stop", "times"}: these layers run several times in a row
    loop: Optional[Dict[str, int]] = None
    # taps of a causal convolution over what the mixers read, whose last inputs are part of a sequence's state
    input_conv: Optional[int] = None
    logit_scale: Optional[float] = None
    weight_dtype: Optional[str] = None
    multimodal: Optional[Dict[str, Any]] = None
    quant: QuantConfig = field(default_factory=QuantConfig)

    # ---- (de)serialisation -------------------------------------------------------
    def to_dict(self) -> dict:
        d: Dict[str, Any] = {}
        for f in fields(self):
            v = getattr(self, f.name)
            if f.name == "quant":
                d["quant"] = self.quant.to_dict()
            elif v is not None:
                d[f.name] = v
        return d

    @classmethod
    def from_dict(cls, d: dict) -> "ModelConfig":
        d = dict(d)
        quant = d.pop("quant", None)
        names = {f.name for f in fields(cls)}
        cfg = cls(**{k: v for k, v in d.items() if k in names})
        if quant:
            cfg.quant = QuantConfig.from_dict(quant)
        return cfg

    def serialize(self) -> bytes:
        return serializer.encode(self.to_dict())

    @classmethod
    def deserialize(cls, data) -> "ModelConfig":
        return cls.from_dict(serializer.decode(data))

    # ---- derived sizes -----------------------------------------------------------
    @property
    def q_dim(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def kv_head_dim(self) -> int:
        return self.head_dim

    @property
    def kv_cache_bytes_per_token(self) -> int:
        """What one token keeps in one layer, in 16-bit elements (of the widest layer when layers differ)."""
        n, d = self.kv_pool_dims()
        return self.kv_planes * n * d * 2

    @property
    def kv_planes(self) -> int:
        """Rows a token has per layer and kv head: K and V, or one latent row that serves as both."""
        return 1 if self.is_design else 2

    @property
    def total_kv_cache_bytes_per_token(self) -> int:
        return self.kv_cache_bytes_per_token * self.num_cache_layers

    # ---- designs whose layers are listed one by one ----------------------------------------------------
    @property
    def is_design(self) -> bool:
        return self.design_layers is not None

    @property
    def is_latent(self) -> bool:
        return self.is_design and any(L["type"] == "latent_attention" for L in self.design_layers)

    @property
    def is_hybrid(self) -> bool:
        """Layers of attention over heads and of recurrent mixers, in any order."""
        return self.is_design and not self.is_latent

    def mixer_spec(self, i: int):
        """``HeadsSpec``, ``TwinSpec`` or a recurrent mixer's of layer ``i`` of a hybrid design."""
        return read_mixer(self.arch, self.design_layers[i])

    def ff_spec(self, i: int):
        """``DenseSpec``, ``MoESpec`` or None of layer ``i`` of a hybrid design."""
        return read_ff(self.arch, self.design_layers[i])

    @property
    def layer_runs(self) -> List[int]:
        """The layers in the order in which a token passes them; those of a loop come once per pass.  Every run has its own
        cache or state."""
        n, loop = self.num_layers, self.loop
        if not loop:
            return list(range(n))
        body = list(range(loop["start"], loop["stop"]))
        return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))

    def enters_loop(self, run: int) -> bool:
        """Whether layer run ``run`` is the first of a pass of a loop whose passes start from [x; embedding]."""
        if not self.loop or not self.loop_rejoins:
            return False
        at, body = run - self.loop["start"], self.loop["stop"] - self.loop["start"]
        return 0 <= at < body * self.loop["times"] and at % body == 0

    @property
    def cache_layers(self) -> Dict[int, int]:
        """Layer run -> its layer of the cache pool; runs without keys and values of their own have none."""
        if not self.is_hybrid:
            return {i: i for i in range(self.num_layers)}
        specs = [attention_of(self.mixer_spec(i)) for i in self.layer_runs]
        return {r: n for n, r in enumerate(r for r, s in enumerate(specs) if s is not None and s.own_kv)}

    @property
    def num_cache_layers(self) -> int:
        return max(1, len(self.cache_layers))

    def _state_layout(self):
        out, inputs, at = {}, {}, 0
        kept = max(0, (self.input_conv or 1) - 1) * self.hidden_size
        for r, i in enumerate(self.layer_runs if self.is_hybrid else ()):
            s = recurrent_of(self.mixer_spec(i))
            if s is not None:
                out[r] = at
                at += (s.state_floats + 3) // 4 * 4
            if kept:
                inputs[r] = at
                at += (kept + 3) // 4 * 4
        return out, inputs, at

    @property
    def state_offsets(self) -> Dict[int, int]:
        """Run of a recurrent layer -> its first element in a sequence's state."""
        return self._state_layout()[0]

    @property
    def input_offsets(self) -> Dict[int, int]:
        """Layer run -> where a sequence's state holds the last inputs of its ``input_conv``, the oldest first."""
        return self._state_layout()[1]

    @property
    def state_floats(self) -> int:
        return self._state_layout()[2]

    @property
    def keeps_state(self) -> bool:
        """Sequences carry more than their cache blocks from token to token: recurrent layers, or the token before."""
        return self.is_hybrid and (self.state_floats > 0 or bool((self.embed_design or {}).get("bigram")))

    def latent_spec(self, i: int) -> LatentSpec:
        m = self.design_layers[i]["mixer"]
        rot = m.get("rot") or {}
        return LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                          int((m.get("mask") or {}).get("size") or 0), float(m["scale"]),
                          int(rot.get("dims", m["rot_dim"])), float(rot.get("base", 10000.0)))

    def moe_spec(self, i: int) -> Optional[MoESpec]:
        m = self.design_layers[i].get("mlp")
        if m is None:
            return None
        return MoESpec(int(m["router"]["experts"]), int(m["router"]["top"]), int(m["expert"]["ff"]),
                       int((m.get("shared") or {}).get("ff") or 0))

    @property
    def cache_window(self) -> int:
        """Tokens that some layer still sees: blocks that fell out of every layer's window may be given back.  0 when a
        layer keeps everything (models that mix local and global layers apply the window inside attention)."""
        if self.is_hybrid:
            return 0
        if self.is_latent:
            w = [self.latent_spec(i).window for i in range(self.num_layers)]
            return max(w) if w and min(w) > 0 else 0
        return int(self.sliding_window) if (self.sliding_window or 0) > 0 and not self.layer_types else 0

    def _masks(self) -> List[HeadsSpec]:
        if self.__dict__.get("_mask_specs") is None:
            self.__dict__["_mask_specs"] = list({(s.chunk, s.window, s.keep_first, s.pool): s for s in (
                attention_of(self.mixer_spec(i)) for i in range(self.num_layers)) if s is not None}.values())
        return self.__dict__["_mask_specs"]

    @property
    def kept_first(self) -> int:
        """First positions that some layer always sees."""
        return max((s.keep_first for s in self._masks()), default=0) if self.is_hybrid else 0

    def first_seen(self, position: int) -> int:
        """First position that some layer still sees from ``position`` (and from any later one), or needs for the mean of a
        block, apart from the ``kept_first`` ones: the cache may give back the blocks between."""
        if self.is_hybrid:
            return min((s.first_needed(position) for s in self._masks()), default=position)
        w = self.cache_window
        return max(0, position + 1 - w) if w > 0 else 0

    @property
    def pool_step(self) -> int:
        """Tokens of the smallest block whose mean some layer caches; 0: no layer does."""
        return min((s.pool for s in self._masks() if s.pool > 0), default=0) if self.is_hybrid else 0

    def mean_rows(self, tokens: int) -> int:
        """Rows of block means that a sequence of ``tokens`` tokens has in the cache."""
        return tokens // self.pool_step if self.pool_step else 0

    def cache_blocks(self, tokens: int, sequences: int, block_size: int) -> int:
        """Blocks of a cache pool for up to ``tokens`` tokens (whole blocks of every sequence counted) of up to ``sequences``
        sequences, with their block means."""
        n = (tokens + block_size - 1) // block_size
        if self.pool_step:
            n += self.mean_rows(tokens) // block_size + sequences
        return n

    # ---- per-layer attention geometry (Gemma-family models mix layer kinds) -----------------------
    @property
    def is_gemma(self) -> bool:
        return self.arch.startswith("gemma")

    @property
    def norm_weight_offset(self) -> float:
        """Gemma-2 and Movinex store RMSNorm weights as ``w - 1`` (the norm multiplies by ``1 + w``); Gemma-4 and everything
        else multiply by the stored weight (zse-engine/zse_engine/orchestrator/kernels.py:1475-1478)."""
        return 1.0 if self.arch in ("gemma2", "movinex") else 0.0

    @property
    def norms_outputs(self) -> bool:
        """Hybrid designs: norms sit on the sublayers' outputs, not on their inputs."""
        return self.arch == "nimelorn"

    @property
    def side_by_side(self) -> bool:
        """Hybrid designs: a layer's sublayers read one norm and their results are added together."""
        return self.arch == "vobisun"

    @property
    def loop_rejoins(self) -> bool:
        """Hybrid designs: a pass of the loop starts from a product of x and the embedding."""
        return self.arch == "movinex"

    def layer_kind(self, i: int) -> str:
        if self.layer_types and i < len(self.layer_types):
            return self.layer_types[i]
        return "full_attention"

    def layer_spec(self, i: int) -> "LayerSpec":
        """Attention geometry of layer ``i`` (zse-engine/zse_engine/orchestrator/model_runner.py:132-152)."""
        sliding = self.layer_kind(i) == "sliding_attention"
        hd, nkv, theta, rot = self.head_dim, self.num_kv_heads, self.rope_theta, self.head_dim
        shares = False
        if self.arch == "gemma4" and not sliding:
            hd = self.global_head_dim or self.head_dim
            shares = bool(self.attention_k_eq_v)
            nkv = (self.global_num_kv_heads or self.num_kv_heads) if shares else self.num_kv_heads
            theta = self.global_rope_theta or self.rope_theta
            rot = 2 * int((self.partial_rotary_factor or 1.0) * hd // 2)
        if self.arch == "gemma4":
            scale = 1.0                         # q/k norms carry the scaling
        elif self.query_pre_attn_scalar:
            scale = float(self.query_pre_attn_scalar) ** -0.5
        else:
            scale = float(hd) ** -0.5
        window = int(self.sliding_window or 0) if (sliding or not self.layer_types) else 0
        return LayerSpec(hd, nkv, float(theta), rot, window, shares, scale,
                         float(self.attn_logit_softcapping or 0.0), self.arch == "gemma4")

    def kv_pool_dims(self, num_kv_heads: Optional[int] = None):
        """(kv_heads, head_dim) the KV pool is allocated with; ``num_kv_heads`` = this rank's share of
        ``self.num_kv_heads`` under tensor parallelism.  Models whose layers differ get rows of the widest layer
        (``1 x max(kv_heads * head_dim)`` of the local heads); each layer lays its heads out inside that row."""
        if self.is_latent:
            return 1, max(self.latent_spec(i).row for i in range(self.num_layers))
        if self.is_hybrid:
            rows = [s.row for s in (attention_of(self.mixer_spec(i)) for i in range(self.num_layers)) if s is not None]
            return 1, max(rows, default=8)
        local = num_kv_heads or self.num_kv_heads
        tp = max(1, self.num_kv_heads // max(1, local))
        specs = {(s.num_kv_heads, s.head_dim) for s in (self.layer_spec(i) for i in range(self.num_layers))}
        if len(specs) <= 1:
            return local, self.head_dim
        return 1, max(max(1, n // tp) * d for n, d in specs)

    def linear_param_count(self) -> int:
        if self.is_hybrid:
            n = 0
            for i in range(self.num_layers):
                a, m = self.mixer_spec(i), self.ff_spec(i)
                n += self.hidden_size * (a.in_width + a.out_width)
                if isinstance(m, MoESpec):
                    n += self.hidden_size * (m.router_rows + 3 * m.experts * m.ff + 3 * m.shared_ff)
                elif m is not None:
                    n += self.hidden_size * (3 if m.gated else 2) * m.ff
            return n + (2 * self.hidden_size ** 2 if self.loop and self.loop_rejoins else 0)
        if self.is_latent:
            n = 0
            for i in range(self.num_layers):
                a, m = self.latent_spec(i), self.moe_spec(i)
                n += self.hidden_size * (a.heads * (a.qk_dim + 2 * a.vdim) + a.kv_rank + a.rot_dim)
                n += a.heads * (a.dim + a.vdim) * a.kv_rank
                if m is not None:
                    n += self.hidden_size * (m.experts + 2 * m.experts * m.ff + 2 * m.shared_ff)
            return n
        per_layer = (self.hidden_size * self.q_dim + 2 * self.hidden_size * self.kv_dim
                     + self.q_dim * self.hidden_size + 3 * self.hidden_size * self.intermediate_size)
        return per_layer * self.num_layers

    def estimate_model_size_bytes(self) -> int:
        params = self.linear_param_count()
        fp16 = self.vocab_size * self.hidden_size * 2 * (1 if self.tie_word_embeddings else 2)
        fp16 += self.num_layers * self.hidden_size * 2 * 2
        if self.quant.method == QuantMethod.NONE:
            return params * 2 + fp16
        groups = params // max(1, self.quant.group_size)
        per_group = 4 if self.quant.method == QuantMethod.INT4_ASYM else 2
        return params * self.quant.bits // 8 + groups * per_group + fp16
