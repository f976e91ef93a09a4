"""Ruralorn: every layer is described on its own in config.json (``layers``: a latent-attention mixer and, optionally, a
routed feed-forward).  Tensor names are kept as they are (``l<i>.mix.*``, ``l<i>.mlp.*``) and so is their width: the
weights are bfloat16 and are not quantised."""
from typing import List

from ..config import ModelConfig
from ..spec import QuantMethod
from .base import ArchAdapter, register_adapter

# the design itself sets no limit on a sequence's length; engines without an explicit limit apply their own
MAX_SEQ_LEN = 1 << 20


@register_adapter
class RuralornAdapter(ArchAdapter):
    ARCH_NAME = "ruralorn"
    STORED_DTYPE = "bfloat16"

    def config_from_hf(self, hf_config: dict) -> ModelConfig:
        hf = hf_config
        layers = hf["layers"]
        for i, layer in enumerate(layers):
            if layer["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer '{layer['type']}'")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        c = ModelConfig(arch=self.ARCH_NAME, num_layers=len(layers), hidden_size=int(hf["width"]),
                        vocab_size=int(hf["vocab"]), max_seq_len=MAX_SEQ_LEN,
                        rms_norm_eps=float(hf["norm"]["eps"]), design_layers=layers,
                        embed_multiplier=float((hf.get("embedding") or {}).get("scale", 1.0)),
                        logit_scale=float(hf.get("logit_scale", 1.0)),
                        final_logit_softcapping=hf.get("logit_softcap"), weight_dtype=self.STORED_DTYPE)
        specs = [c.latent_spec(i) for i in range(c.num_layers)]
        moes = [m for m in (c.moe_spec(i) for i in range(c.num_layers)) if m is not None]
        # the general fields describe the widest layer; the cache and the kernels use the per-layer specs
        c.num_heads = max(s.heads for s in specs)
        c.num_kv_heads = 1
        c.head_dim = max(s.qk_dim for s in specs)
        c.intermediate_size = max([1] + [max(m.ff, m.shared_ff) for m in moes])
        c.quant.method, c.quant.bits = int(QuantMethod.NONE), 16
        return c

    def should_quantize(self, tensor_name: str) -> bool:
        return False

    def map_tensor_name(self, hf_name: str) -> str:
        return hf_name

    def layer_tensors(self, config: ModelConfig, layer: int) -> List[str]:
        a, m = config.latent_spec(layer), config.moe_spec(layer)
        out = ["norm1", "mix.q", "mix.dkv", "mix.dkv.norm", "mix.uk", "mix.uv", "mix.o"] + (["mix.g"] if a.gated else [])
        if m is not None:
            out += ["norm2", "mlp.router"]
            out += [f"mlp.e{e}.{part}" for e in range(m.experts) for part in ("up", "down")]
            if m.shared_ff:
                out += ["mlp.shared.up", "mlp.shared.down"]
        return out

    def expected_tensors(self, config: ModelConfig) -> List[str]:
        out = ["embed"]
        for i in range(config.num_layers):
            out += [f"l{i}.{t}" for t in self.layer_tensors(config, i)]
        return out + ["final.norm", "head"]

    def validate_config(self, config: ModelConfig) -> List[str]:
        return []
