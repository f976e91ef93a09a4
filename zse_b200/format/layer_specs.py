"""What a layer of a model is: sizes, masks and constants of its mixer and its feed-forward, read from the configuration."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Union


@dataclass
class LayerSpec:
    head_dim: int
    num_kv_heads: int
    rope_theta: float
    rotary_dim: int          # leading pairs (i, i + head_dim/2), i < rotary_dim/2, rotate; the rest pass through
    window: int              # 0 = full causal attention
    k_is_v: bool             # no v_proj: V is the k_proj output before its norm
    scale: float
    softcap: float           # 0 = none
    qk_norm: bool            # per-head RMSNorm of q and k (learned weight) and of v (no weight)


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class LatentSpec:
    """Attention over a shared low-rank latent: a token caches its normed latent (``kv_rank``) and one rotated key part
    (``rot_dim``) that all heads share; a head's key and value are linear images of the latent."""
    heads: int
    dim: int                 # query/key dimensions of a head that carry no position
    rot_dim: int             # ... and those that are rotated
    vdim: int
    kv_rank: int
    window: int              # a position sees itself and the window - 1 before it; 0 = everything before it
    scale: float
    rot_dims: int            # leading dimensions of the rot_dim part that rotate (pairs 2i, 2i + 1)
    rot_base: float
    gated: bool = True       # heads are multiplied by sigmoid(W_g h) before the output projection

    @property
    def qk_dim(self) -> int:
        return self.dim + self.rot_dim

    # columns of the fused input projection [q | latent, rotated key | gate]; every section starts on 8 elements
    @property
    def latent_col(self) -> int:
        return _up8(self.heads * self.qk_dim)

    @property
    def gate_col(self) -> int:
        return self.latent_col + _up8(self.kv_rank + self.rot_dim)

    @property
    def in_width(self) -> int:
        return self.gate_col + (_up8(self.heads * self.vdim) if self.gated else 0)

    @property
    def row(self) -> int:
        """Elements of a cached token: [latent | rotated key part], padded to an odd number of 16-byte pieces (of a
        16-bit type): consecutive rows then start in different shared-memory banks and can be used where a plain copy
        puts them."""
        n = _up8(self.kv_rank + self.rot_dim)
        return n if n // 8 % 2 else n + 8


# gated activations of two products (gate, up) and the number that names each to the kernels, see ``ops.reference.glu``
GLU: Dict[str, int] = {"clamped_glu": 0, "silu_glu": 1, "gelu_tanh_glu": 2}


@dataclass(frozen=True)
class MoESpec:
    """Routed feed-forward: ``top`` of ``experts`` per token, chosen and weighted by ``score``.  ``shared_ff`` > 0 adds an
    expert that every token uses."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    score: str = "sigmoid"       # of the router's logits: "sigmoid" (each on its own) or "softmax" (over all experts)
    activation: str = "gelu"     # exact (erf) gelu, or one of ``GLU``: two up products
    weigh: str = "input"         # the weight scales the expert's "input" or "output"
    normalise: bool = False      # the chosen scores are divided by their sum
    scale: float = 1.0           # ... and multiplied by this
    limit: float = 0.0           # clamp of "clamped_glu"
    shared_limit: float = 0.0
    shared_gate: bool = False    # the shared expert is multiplied by sigmoid(w . h), one number per token
    groups: int = 1              # equal groups of neighbouring experts; a group counts for the sum of its two best scores
    keep_groups: int = 1         # experts are chosen from that many best groups

    @property
    def gated(self) -> bool:
        return self.activation in GLU

    @property
    def router_rows(self) -> int:
        """Columns of the router's product: the experts, and the shared expert's gate behind them."""
        return self.experts + (1 if self.shared_gate else 0)


@dataclass(frozen=True)
class DenseSpec:
    """Feed-forward of one up product, an activation and one down product; of two up products when ``gated``."""
    ff: int
    activation: str = "relu2"    # the square of relu, or one of ``GLU``

    @property
    def gated(self) -> bool:
        return self.activation in GLU


@dataclass(frozen=True)
class HeadsSpec:
    """Attention of ``heads`` query heads over ``kv_heads`` key/value heads whose widths may differ.  Queries and keys are
    normed, per head after a rotation or all heads together before it."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = 0               # > 0: a position sees the positions of its own chunk of this size only
    window: int = 0              # > 0: a position sees itself and the window - 1 before it
    kv_from: int = -1            # >= 0: keys and values are those of that layer
    gated: bool = True           # a head's result is multiplied by sigmoid(w_h . x)
    gate_each: bool = False      # ... or every one of its dimensions by a gate of its own
    keep_first: int = 0          # with a window: that many first positions are always seen
    softcap: float = 0.0         # > 0: scores become softcap * tanh(score / softcap)
    bias: bool = False           # of the query, key and value projections
    k_as_v: bool = False         # the values are the keys as projected
    learned_norm: bool = True    # query and key norm have a weight
    rot_dims: int = 0            # leading dimensions of queries and keys that rotate (pairs 2i, 2i + 1)
    rot_base: float = 10000.0
    temp_coef: float = 0.0       # a query at p is multiplied by 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
    temp_every: int = 1
    pool: int = 0                # > 0, with a window: what left it is seen as means of blocks of that many tokens, once all
    #                              of a block has left
    sink: bool = False           # the softmax has one more score per head, learned, without a value
    head_temp: bool = False      # a learned factor of the scores per head
    whole_norm: bool = False     # one query (key) norm over the rows of all heads, before the rotation
    rot_factor: float = 1.0      # the rotation is slower by this factor
    out_scale: float = 1.0       # factor of the result

    @property
    def own_kv(self) -> bool:
        return self.kv_from < 0

    # columns of the fused input projection [q | k | v | gate]; every section starts on 8 elements
    @property
    def k_col(self) -> int:
        return _up8(self.heads * self.dim)

    @property
    def v_col(self) -> int:
        return self.k_col + (_up8(self.kv_heads * self.dim) if self.own_kv else 0)

    @property
    def gate_col(self) -> int:
        return self.v_col + (_up8(self.kv_heads * self.vdim) if self.own_kv and not self.k_as_v else 0)

    @property
    def gate_width(self) -> int:
        return 0 if not self.gated else self.heads * self.vdim if self.gate_each else self.heads

    @property
    def in_width(self) -> int:
        return self.gate_col + _up8(self.gate_width)

    @property
    def row(self) -> int:
        """Elements of a cached token."""
        return self.kv_heads * (_up8(self.dim) + _up8(self.vdim))

    def first_seen(self, position: int) -> int:
        """First position that the token at ``position`` sees, apart from the ``keep_first`` ones."""
        if self.chunk > 0:
            return position // self.chunk * self.chunk
        return max(0, position + 1 - self.window) if self.window > 0 else 0

    def blocks_seen(self, position: int) -> int:
        """Blocks of ``pool`` tokens whose means the token at ``position`` sees: the first ones, all of whose tokens lie
        before its window."""
        return max(0, position + 1 - self.window) // self.pool if self.pool > 0 else 0

    def first_needed(self, position: int) -> int:
        """First position whose key and value a pass from ``position`` on reads: a block that is not complete yet still
        needs its tokens for the mean, wherever the window begins."""
        first = self.first_seen(position)
        return min(first, position // self.pool * self.pool) if self.pool > 0 else first

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Recurrent mixer whose heads keep a [dim, vdim] matrix memory, a key sum [dim] and a running maximum of the log
    gates (mLSTM)."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    # columns of the fused input projection [q | k | v | output gate | input and forget gates]
    @property
    def k_col(self) -> int:
        return _up8(self.heads * self.dim)

    @property
    def v_col(self) -> int:
        return 2 * self.k_col

    @property
    def gate_col(self) -> int:
        return self.v_col + _up8(self.heads * self.vdim)

    @property
    def if_col(self) -> int:
        return self.gate_col + _up8(self.heads * self.vdim)

    @property
    def in_width(self) -> int:
        return self.if_col + _up8(2 * self.heads)

    # state of one sequence, in 32-bit elements: memory [heads, dim, vdim], key sum [heads, dim], maximum [heads]; every
    # part starts on 4 elements
    @property
    def sum_at(self) -> int:
        return (self.heads * self.dim * self.vdim + 3) // 4 * 4

    @property
    def max_at(self) -> int:
        return self.sum_at + (self.heads * self.dim + 3) // 4 * 4

    @property
    def state_floats(self) -> int:
        return self.max_at + (self.heads + 3) // 4 * 4


@dataclass(frozen=True)
class StateSpaceSpec:
    """Recurrent mixer whose heads keep a [state, vdim] matrix under a decay of their own (Mamba-2); its inputs pass a short
    causal convolution per channel."""
    heads: int
    vdim: int
    state: int
    groups: int                  # heads of a group share the input and read-out vectors B and C
    conv: int                    # taps of the convolution
    norm_groups: int             # the gated result is normed in that many equal parts

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def out_width(self) -> int:
        return self.inner

    # columns of the fused input projection [z | x | B | C | step sizes]; x, B and C are the channels of the convolution,
    # whose output keeps their layout from column 0 on
    @property
    def x_col(self) -> int:
        return _up8(self.inner)

    @property
    def b_at(self) -> int:
        return _up8(self.inner)

    @property
    def c_at(self) -> int:
        return self.b_at + _up8(self.groups * self.state)

    @property
    def conv_width(self) -> int:
        return self.c_at + _up8(self.groups * self.state)

    @property
    def dt_col(self) -> int:
        return self.x_col + self.conv_width

    @property
    def in_width(self) -> int:
        return self.dt_col + _up8(self.heads)

    # state of one sequence, in 32-bit elements: memory [heads, state, vdim], then the convolution's last conv - 1 inputs
    @property
    def conv_at(self) -> int:
        return (self.heads * self.state * self.vdim + 3) // 4 * 4

    @property
    def state_floats(self) -> int:
        return self.conv_at + (self.conv - 1) * self.conv_width


@dataclass(frozen=True)
class GatedLinearSpec:
    """Recurrent mixer whose heads keep a [dim, vdim] matrix whose rows, one per key channel, decay each at its own rate
    (gated linear attention).  The decays' logarithms come from a projection of low rank, divided by ``tau``."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int                    # of the projection that makes the decays
    col: int = 0                 # first column of its part of the input projection
    out_scale: float = 1.0       # factor of the result

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    # columns of the fused input projection [q | k | v | output gate | inner vector of the decays]
    @property
    def k_col(self) -> int:
        return self.col + _up8(self.heads * self.dim)

    @property
    def v_col(self) -> int:
        return self.k_col + _up8(self.heads * self.dim)

    @property
    def gate_col(self) -> int:
        return self.v_col + _up8(self.heads * self.vdim)

    @property
    def rank_col(self) -> int:
        return self.gate_col + _up8(self.heads * self.vdim)

    @property
    def in_width(self) -> int:
        """Columns up to the end of its part."""
        return self.rank_col + _up8(self.rank)

    @property
    def state_floats(self) -> int:
        return (self.heads * self.dim * self.vdim + 3) // 4 * 4


@dataclass(frozen=True)
class TwinSpec:
    """Two mixers that read the same input and whose results are added: attention over heads and gated linear attention.
    Their projections are one, [left | right], and so are their results."""
    left: HeadsSpec
    right: GatedLinearSpec

    @property
    def heads(self) -> int:
        return max(self.left.heads, self.right.heads)

    @property
    def in_width(self) -> int:
        return self.right.in_width

    @property
    def right_at(self) -> int:
        """Column of the right mixer's result."""
        return _up8(self.left.out_width)

    @property
    def out_width(self) -> int:
        """Both results; what comes behind them starts on 8 elements."""
        return self.right_at + _up8(self.right.out_width)


RECURRENT = (MatrixMemorySpec, StateSpaceSpec, GatedLinearSpec)
MixerSpec = Union[HeadsSpec, MatrixMemorySpec, StateSpaceSpec, TwinSpec]


def attention_of(s: MixerSpec) -> Optional[HeadsSpec]:
    """The part of a mixer that caches keys and values."""
    s = s.left if isinstance(s, TwinSpec) else s
    return s if isinstance(s, HeadsSpec) else None


def recurrent_of(s: MixerSpec):
    """The part of a mixer that keeps recurrent state."""
    s = s.right if isinstance(s, TwinSpec) else s
    return s if isinstance(s, RECURRENT) else None


# ---- entries of a design's ``layers`` list -------------------------------------------------------------------------------
def _chunked_attention(m: dict) -> HeadsSpec:
    src = m.get("kv_from")
    return HeadsSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                     chunk=int((m.get("mask") or {}).get("size") or 0), kv_from=-1 if src is None else int(src))


def _matrix_memory(m: dict) -> MatrixMemorySpec:
    return MatrixMemorySpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))


def _tempered_attention(m: dict) -> HeadsSpec:
    t = m.get("q_temp") or {}
    return HeadsSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), gated=False,
                     bias=True, learned_norm=False, temp_coef=float(t.get("coef", 0.0)), temp_every=int(t.get("every", 1)))


def _windowed_attention(m: dict) -> HeadsSpec:
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    return HeadsSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                     window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0), gate_each=True,
                     softcap=float(m.get("softcap") or 0.0), k_as_v=True, learned_norm=False,
                     rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base", 10000.0)))


# rank of the decays' projection where nothing says another (a model's own tensors do, see ``ArchAdapter.sizes_of_tensors``)
DECAY_RANK = 16


def _state_space(m: dict) -> StateSpaceSpec:
    return StateSpaceSpec(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]),
                          int(m["norm_groups"]))


def _twin(m: dict) -> TwinSpec:
    a, r = m["left"], m["right"]
    mask, rot = a.get("mask") or {}, a.get("rot") or {}
    left = HeadsSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                     window=int(mask.get("size") or 0), pool=int(mask.get("pool") or 0), bias=True, whole_norm=True,
                     rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base", 10000.0)),
                     rot_factor=float((rot.get("scaling") or {}).get("factor", 1.0)), sink=True, head_temp=True,
                     out_scale=float(m.get("left_scale", 1.0)))
    return TwinSpec(left, GatedLinearSpec(int(r["heads"]), int(r["dim"]), int(r["vdim"]), float(r["tau"]),
                                          int(r.get("rank") or DECAY_RANK), left.in_width, float(m.get("right_scale", 1.0))))


_MIXERS = {
    "nimelorn": {"attention": _chunked_attention, "mlstm": _matrix_memory},
    "movinex": {"attention": _tempered_attention, "attention_2": _windowed_attention, "mamba2": _state_space},
    "vobisun": {"parallel": _twin},
}


def mixer_types(arch: str):
    return tuple(_MIXERS[arch])


def read_mixer(arch: str, layer: dict):
    return _MIXERS[arch][layer["type"]](layer["mixer"])


def read_ff(arch: str, layer: dict):
    """``DenseSpec``, ``MoESpec`` or None."""
    m = layer.get("mlp")
    if m is None:
        return None
    if arch == "vobisun":
        return DenseSpec(int(m["ff"]), "silu_glu")
    if arch == "movinex":
        if m["kind"] == "dense":
            return DenseSpec(int(m["ff"]), "gelu_tanh_glu")
        r = m["router"]
        g = r.get("groups") or {}
        return MoESpec(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), activation="silu_glu", weigh="output",
                       groups=int(g.get("count", 1)), keep_groups=int(g.get("keep", 1)))
    if m["kind"] == "dense":
        return DenseSpec(int(m["ff"]))
    r, e, s = m["router"], m["expert"], m.get("shared")
    return MoESpec(int(r["experts"]), int(r["top"]), int(e["ff"]), int(s["ff"]) if s else 0, "softmax", "clamped_glu",
                   "output", True, float(r.get("scale", 1.0)), float(e["limit"]), float(s["limit"]) if s else 0.0, bool(s))
