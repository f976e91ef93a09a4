"""Vobisun: config.json lists the layers, each of two mixers side by side - windowed attention that sees older tokens as means of
blocks, and gated linear attention - and a gated feed-forward or none, all behind one norm; what the mixers read passes a short
causal convolution.  A range of layers may run several times (``loop``).  Tensor names are kept as they are (``l<i>.mix.left.*``,
``l<i>.mix.right.*``, ``l<i>.mlp.*``) and so is their width: the weights are bfloat16 and are not quantised."""
import copy
from typing import Dict, List, Tuple

from ..config import ModelConfig
from ..layer_specs import mixer_types
from ..spec import QuantMethod
from .base import ArchAdapter, register_adapter

# the design itself sets no limit on a sequence's length; engines without an explicit limit apply their own
MAX_SEQ_LEN = 1 << 20


def _check(i: int, s) -> None:
    a, r = s.left, s.right
    if a.heads % a.kv_heads:
        raise ValueError(f"layer {i}: {a.heads} heads do not share {a.kv_heads} key/value heads evenly")
    if a.rot_dims % 2 or a.rot_dims > a.dim:
        raise ValueError(f"layer {i}: {a.rot_dims} of {a.dim} dimensions cannot rotate in pairs")
    if a.rot_factor <= 0:
        raise ValueError(f"layer {i}: a rotation cannot be slower by a factor of {a.rot_factor}")
    if a.window < 0 or a.pool < 0 or (a.pool and not a.window):
        raise ValueError(f"layer {i}: a window of {a.window} tokens with blocks of {a.pool}")
    if r.tau <= 0:
        raise ValueError(f"layer {i}: decays need a positive divisor, not {r.tau}")


@register_adapter
class VobisunAdapter(ArchAdapter):
    ARCH_NAME = "vobisun"
    STORED_DTYPE = "bfloat16"

    def config_from_hf(self, hf_config: dict) -> ModelConfig:
        hf = hf_config
        layers = copy.deepcopy(hf["layers"])
        for i, layer in enumerate(layers):
            if layer["type"] not in mixer_types(self.ARCH_NAME):
                raise ValueError(f"layer {i}: unknown mixer '{layer['type']}'")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        loop = hf.get("loop")
        if loop:
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
            if not 0 <= loop["start"] < loop["stop"] <= len(layers) or loop["times"] < 1:
                raise ValueError(f"layers {loop['start']} .. {loop['stop'] - 1} of {len(layers)} cannot run "
                                 f"{loop['times']} times")
        taps = int((hf.get("canon") or {}).get("taps", 1))
        if taps < 1:
            raise ValueError("a convolution needs a tap")
        c = ModelConfig(arch=self.ARCH_NAME, num_layers=len(layers), hidden_size=int(hf["width"]),
                        vocab_size=int(hf["vocab"]), max_seq_len=MAX_SEQ_LEN, rms_norm_eps=float(hf["norm"]["eps"]),
                        design_layers=layers, embed_multiplier=float((hf.get("embedding") or {}).get("scale", 1.0)),
                        loop=loop or None, input_conv=taps, weight_dtype=self.STORED_DTYPE)
        specs = [c.mixer_spec(i) for i in range(c.num_layers)]
        for i, s in enumerate(specs):
            _check(i, s)
        # the general fields describe the widest layer; the cache and the kernels use the per-layer specs
        c.num_heads = max(s.left.heads for s in specs)
        c.num_kv_heads = 1
        c.head_dim = max(s.left.dim for s in specs)
        c.intermediate_size = max([1] + [m.ff for m in (c.ff_spec(i) for i in range(c.num_layers)) if m is not None])
        c.quant.method, c.quant.bits = int(QuantMethod.NONE), 16
        return c

    def sizes_of_tensors(self, config: ModelConfig, shapes: Dict[str, Tuple[int, ...]]) -> None:
        """The rank of the decays' projection stands in no configuration but in the tensors."""
        for i, layer in enumerate(config.design_layers):
            shape = shapes.get(f"l{i}.mix.right.a1")
            if shape:
                layer["mixer"]["right"]["rank"] = int(shape[0])

    def should_quantize(self, tensor_name: str) -> bool:
        return False

    def map_tensor_name(self, hf_name: str) -> str:
        return hf_name

    def tensor_shapes(self, config: ModelConfig):
        """(name, shape) of every tensor, in file order."""
        c, H = config, config.hidden_size
        yield "embed", (c.vocab_size, H)
        for i in range(c.num_layers):
            p, s, m = f"l{i}.", c.mixer_spec(i), c.ff_spec(i)
            a, r = s.left, s.right
            yield p + "norm1", (H,)
            yield p + "canon1", (H, c.input_conv)
            for name, n in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                yield f"{p}mix.left.{name}", (n, H)
                yield f"{p}mix.left.{name}.b", (n,)
                if name != "v":
                    yield f"{p}mix.left.{name}.norm", (n,)
            yield p + "mix.left.temp", (a.heads,)
            yield p + "mix.left.sink", (a.heads,)
            yield p + "mix.left.g", (a.heads, H)
            yield p + "mix.left.o", (H, a.heads * a.vdim)
            for name, n in (("q", r.heads * r.dim), ("k", r.heads * r.dim), ("v", r.heads * r.vdim), ("g", r.heads * r.vdim),
                            ("a1", r.rank)):
                yield f"{p}mix.right.{name}", (n, H)
            yield p + "mix.right.a2", (r.heads * r.dim, r.rank)
            yield p + "mix.right.a2.b", (r.heads * r.dim,)
            yield p + "mix.right.norm", (r.vdim,)
            yield p + "mix.right.o", (H, r.heads * r.vdim)
            if m is not None:
                yield p + "mlp.gate", (m.ff, H)
                yield p + "mlp.up", (m.ff, H)
                yield p + "mlp.down", (H, m.ff)
        yield "final.norm", (H,)
        yield "head", (c.vocab_size, H)

    def expected_tensors(self, config: ModelConfig) -> List[str]:
        return [name for name, _ in self.tensor_shapes(config)]

    def validate_config(self, config: ModelConfig) -> List[str]:
        return []
