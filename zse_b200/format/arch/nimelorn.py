"""Nimelorn: config.json lists the layers, each of chunked attention over heads or of a matrix memory (mLSTM), with a dense
or routed feed-forward or none; norms sit on the sublayers' outputs.  Tensor names are kept as they are (``l<i>.mix.*``,
``l<i>.mlp.*``) and so is their width: the weights are bfloat16 and are not quantised."""
from typing import List

from ..config import HeadsSpec, MatrixMemorySpec, ModelConfig, MoESpec
from ..layer_specs import mixer_types
from ..spec import QuantMethod
from .base import ArchAdapter, register_adapter

# the design itself sets no limit on a sequence's length; engines without an explicit limit apply their own
MAX_SEQ_LEN = 1 << 20
SINUSOID_BASE = 10000.0          # entries 2i and 2i + 1 of the position vector turn by base^(-2i / width) per token


@register_adapter
class NimelornAdapter(ArchAdapter):
    ARCH_NAME = "nimelorn"
    STORED_DTYPE = "bfloat16"

    def config_from_hf(self, hf_config: dict) -> ModelConfig:
        hf = hf_config
        layers = hf["layers"]
        for i, layer in enumerate(layers):
            if layer["type"] not in mixer_types(self.ARCH_NAME):
                raise ValueError(f"layer {i}: unknown mixer '{layer['type']}'")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        emb = hf.get("embedding") or {}
        extra = {"sinusoid_base": SINUSOID_BASE, "norm": True}
        if emb.get("bigram"):
            extra["bigram"] = {k: int(emb["bigram"][k]) for k in ("buckets", "mul_prev", "mul_cur")}
        c = ModelConfig(arch=self.ARCH_NAME, num_layers=len(layers), hidden_size=int(hf["width"]),
                        vocab_size=int(hf["vocab"]), max_seq_len=MAX_SEQ_LEN,
                        rms_norm_eps=float(hf["norm"]["eps"]), design_layers=layers,
                        embed_multiplier=float(emb.get("scale", 1.0)), embed_design=extra,
                        weight_dtype=self.STORED_DTYPE)
        specs = [c.mixer_spec(i) for i in range(c.num_layers)]
        for i, s in enumerate(specs):
            if isinstance(s, HeadsSpec):
                if s.heads % s.kv_heads:
                    raise ValueError(f"layer {i}: {s.heads} heads do not share {s.kv_heads} key/value heads evenly")
                if s.own_kv:
                    continue
                src = specs[s.kv_from] if s.kv_from < i else None
                if not isinstance(src, HeadsSpec) or not src.own_kv:
                    raise ValueError(f"layer {i}: layer {s.kv_from} has no keys and values to take")
                if (src.kv_heads, src.dim, src.vdim) != (s.kv_heads, s.dim, s.vdim):
                    raise ValueError(f"layer {i}: the keys and values of layer {s.kv_from} have other sizes")
        ffs = [c.ff_spec(i) for i in range(c.num_layers)]
        # the general fields describe the widest layer; the cache and the kernels use the per-layer specs
        c.num_heads = max(s.heads for s in specs)
        c.num_kv_heads = 1
        c.head_dim = max(s.dim for s in specs)
        c.intermediate_size = max([1] + [max(m.ff, getattr(m, "shared_ff", 0)) for m in ffs if m is not None])
        c.quant.method, c.quant.bits = int(QuantMethod.NONE), 16
        return c

    def should_quantize(self, tensor_name: str) -> bool:
        return False

    def map_tensor_name(self, hf_name: str) -> str:
        return hf_name

    def tensor_shapes(self, config: ModelConfig):
        """(name, shape) of every tensor, in file order."""
        c, H = config, config.hidden_size
        yield "embed", (c.vocab_size, H)
        if c.embed_design.get("bigram"):
            yield "bigram", (c.embed_design["bigram"]["buckets"] + 1, H)
        yield "embed.norm", (H,)
        for i in range(c.num_layers):
            p, a, m = f"l{i}.", c.mixer_spec(i), c.ff_spec(i)
            yield p + "norm1", (H,)
            if isinstance(a, MatrixMemorySpec):
                qw, vw = a.heads * a.dim, a.heads * a.vdim
                for name, rows in (("q", qw), ("k", qw), ("v", vw), ("g", vw), ("i", a.heads), ("f", a.heads)):
                    yield f"{p}mix.{name}", (rows, H)
                yield p + "mix.i.b", (a.heads,)
                yield p + "mix.f.b", (a.heads,)
                yield p + "mix.norm", (vw,)
            else:
                yield p + "mix.q", (a.heads * a.dim, H)
                yield p + "mix.q.norm", (a.dim,)
                if a.own_kv:
                    yield p + "mix.k", (a.kv_heads * a.dim, H)
                    yield p + "mix.k.norm", (a.dim,)
                    yield p + "mix.v", (a.kv_heads * a.vdim, H)
                yield p + "mix.g", (a.heads, H)
            yield p + "mix.o", (H, a.heads * a.vdim)
            if m is None:
                continue
            yield p + "norm2", (H,)
            if not isinstance(m, MoESpec):
                yield p + "mlp.up", (m.ff, H)
                yield p + "mlp.down", (H, m.ff)
                continue
            yield p + "mlp.router", (m.experts, H)
            parts = [(f"mlp.e{e}", m.ff) for e in range(m.experts)]
            if m.shared_ff:
                yield p + "mlp.shared.sg", (1, H)
                parts.append(("mlp.shared", m.shared_ff))
            for name, ff in parts:
                yield f"{p}{name}.gate", (ff, H)
                yield f"{p}{name}.up", (ff, H)
                yield f"{p}{name}.down", (H, ff)
        yield "final.norm", (H,)
        yield "head", (c.vocab_size, H)

    def expected_tensors(self, config: ModelConfig) -> List[str]:
        return [name for name, _ in self.tensor_shapes(config)]

    def validate_config(self, config: ModelConfig) -> List[str]:
        return []
