"""Movinex: config.json lists the layers, each of attention over everything before it, of windowed attention that keeps the first
tokens, or of a state space (Mamba-2), with a dense or routed gated feed-forward or none; a range of layers may run several
times (``loop``).  Tensor names are kept as they are (``l<i>.mix.*``, ``l<i>.mlp.*``) and so is their width: the weights are
bfloat16 and are not quantised."""
from typing import List

from ..config import HeadsSpec, ModelConfig, MoESpec, StateSpaceSpec
from ..layer_specs import mixer_types
from ..spec import QuantMethod
from .base import ArchAdapter, register_adapter

# the design itself sets no limit on a sequence's length; engines without an explicit limit apply their own
MAX_SEQ_LEN = 1 << 20


def _check(i: int, s, m) -> None:
    if isinstance(s, StateSpaceSpec):
        if s.heads % s.groups:
            raise ValueError(f"layer {i}: {s.heads} heads do not form {s.groups} equal groups")
        if s.inner % s.norm_groups:
            raise ValueError(f"layer {i}: {s.inner} channels do not form {s.norm_groups} equal parts")
        if s.conv < 1:
            raise ValueError(f"layer {i}: a convolution needs a tap")
    else:
        if s.heads % s.kv_heads:
            raise ValueError(f"layer {i}: {s.heads} heads do not share {s.kv_heads} key/value heads evenly")
        if s.k_as_v and s.dim != s.vdim:
            raise ValueError(f"layer {i}: values that are the keys have their width, {s.dim}, not {s.vdim}")
        if s.rot_dims % 2 or s.rot_dims > s.dim:
            raise ValueError(f"layer {i}: {s.rot_dims} of {s.dim} dimensions cannot rotate in pairs")
        if s.temp_every < 1:
            raise ValueError(f"layer {i}: the query temperature needs a positive step")
    if isinstance(m, MoESpec):
        if m.experts % m.groups:
            raise ValueError(f"layer {i}: {m.experts} experts do not form {m.groups} equal groups")
        if not 1 <= m.keep_groups <= m.groups or not 1 <= m.top <= m.keep_groups * (m.experts // m.groups):
            raise ValueError(f"layer {i}: {m.top} experts cannot come from {m.keep_groups} of {m.groups} groups")


@register_adapter
class MovinexAdapter(ArchAdapter):
    ARCH_NAME = "movinex"
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
        loop = hf.get("loop")
        if loop:
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
            if not 0 <= loop["start"] < loop["stop"] <= len(layers) or loop["times"] < 1:
                raise ValueError(f"layers {loop['start']} .. {loop['stop'] - 1} of {len(layers)} cannot run "
                                 f"{loop['times']} times")
        c = ModelConfig(arch=self.ARCH_NAME, num_layers=len(layers), hidden_size=int(hf["width"]),
                        vocab_size=int(hf["vocab"]), max_seq_len=MAX_SEQ_LEN,
                        rms_norm_eps=float(hf["norm"]["eps"]), design_layers=layers, loop=loop or None,
                        logit_scale=float(hf.get("logit_scale", 1.0)), weight_dtype=self.STORED_DTYPE)
        specs = [c.mixer_spec(i) for i in range(c.num_layers)]
        ffs = [c.ff_spec(i) for i in range(c.num_layers)]
        for i in range(c.num_layers):
            _check(i, specs[i], ffs[i])
        # the general fields describe the widest layer; the cache and the kernels use the per-layer specs
        c.num_heads = max(s.heads for s in specs)
        c.num_kv_heads = 1
        c.head_dim = max(s.dim if isinstance(s, HeadsSpec) else s.vdim for s in specs)
        c.intermediate_size = max([1] + [m.ff for m in ffs if m is not None])
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
        if c.loop:
            yield "loop.in", (H, 2 * H)
        for i in range(c.num_layers):
            p, a, m = f"l{i}.", c.mixer_spec(i), c.ff_spec(i)
            yield p + "norm1", (H,)
            if isinstance(a, StateSpaceSpec):
                channels = a.inner + 2 * a.groups * a.state
                yield p + "mix.in", (a.inner + channels + a.heads, H)
                yield p + "mix.conv", (channels, a.conv)
                yield p + "mix.conv.b", (channels,)
                for name in ("dt_bias", "A_log", "D"):
                    yield f"{p}mix.{name}", (a.heads,)
                yield p + "mix.norm", (a.inner,)
            else:
                rows = {"q": a.heads * a.dim, "k": a.kv_heads * a.dim}
                if not a.k_as_v:
                    rows["v"] = a.kv_heads * a.vdim
                for name, n in rows.items():
                    yield f"{p}mix.{name}", (n, H)
                    if a.bias:
                        yield f"{p}mix.{name}.b", (n,)
                if a.gated:
                    yield p + "mix.g", (a.gate_width, H)
            yield p + "mix.o", (H, a.heads * a.vdim)
            yield p + "ls1", (H,)
            if m is None:
                continue
            yield p + "norm2", (H,)
            parts = [("mlp", m.ff)]
            if isinstance(m, MoESpec):
                yield p + "mlp.router", (m.experts, H)
                parts = [(f"mlp.e{e}", m.ff) for e in range(m.experts)]
            for name, ff in parts:
                yield f"{p}{name}.gate", (ff, H)
                yield f"{p}{name}.up", (ff, H)
                yield f"{p}{name}.down", (H, ff)
            yield p + "ls2", (H,)
        yield "final.norm", (H,)
        yield "head", (c.vocab_size, H)

    def expected_tensors(self, config: ModelConfig) -> List[str]:
        return [name for name, _ in self.tensor_shapes(config)]

    def validate_config(self, config: ModelConfig) -> List[str]:
        return []
