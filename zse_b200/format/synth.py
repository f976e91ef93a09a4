"""Synthetic models: random weights of a given architecture written as a ``.zse`` file.

``write_random_model`` draws every linear weight from N(0, std), quantises it (INT4 group-128 by default) and
streams it into the file; norms are 1, biases N(0, std).  ``fast=True`` skips the float stage and writes random
nibbles with plausible scales/zeros directly, which is what the benchmarks use for multi-GB shapes (the bytes are
statistically the same as quantised N(0, std) weights and cost no quantisation time).
"""
from __future__ import annotations

from typing import Optional

import numpy as np

from .config import ModelConfig, QuantConfig
from .spec import QuantMethod
from .tokenizer import BPETokenizer, BYTE_ENCODER, SpecialTokens
from .writer import ZSEWriter



def ruralorn_design(layers: int, width: int, vocab: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int,
                    window: int, experts: int, top: int, ff: int, shared_ff: int = 0, rot_base: float = 10000.0,
                    eps: float = 1e-6, embed_scale: float = 1.0, logit_scale: float = 1.0,
                    logit_softcap: float = 30.0) -> dict:
    """A Ruralorn ``config.json`` whose layers are all alike (callers may change single entries)."""
    def layer() -> dict:
        mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
        if shared_ff:
            mlp["shared"] = {"ff": shared_ff}
        return {"type": "latent_attention", "mlp": mlp,
                "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                          "scale": (dim + rot_dim) ** -0.5, "mask": {"size": window},
                          "rot": {"dims": rot_dim, "base": rot_base}}}
    return {"architecture": "Ruralorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "logit_softcap": logit_softcap,
            "layers": [layer() for _ in range(layers)]}


def nimelorn_design(width: int, vocab: int, heads: int, kv_heads: int, dim: int, vdim: int, chunk: int, memory: tuple,
                    dense_ff: int, experts: int, top: int, ff: int, shared_ff: int, limit: float = 7.0, repeats: int = 1,
                    buckets: int = 65521, eps: float = 1e-6, gate_cap: float = 15.0) -> dict:
    """A Nimelorn ``config.json`` of ``repeats`` times four layers: a matrix memory (``memory``: heads, dim, vdim) with a
    dense feed-forward, attention with experts, attention with a dense one, and attention over the keys and values of the
    layer before it with experts."""
    dense = {"kind": "dense", "ff": dense_ff}
    moe = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": 1.0},
           "shared": {"ff": shared_ff, "limit": limit}}

    def attention(mlp, **kw):
        return {"type": "attention", "mlp": mlp, "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                                                               scale=dim ** -0.5, mask={"size": chunk}, **kw)}
    layers = []
    for r in range(repeats):
        layers += [{"type": "mlstm", "mlp": dense, "mixer": {"heads": memory[0], "dim": memory[1], "vdim": memory[2],
                                                             "gate_cap": gate_cap}},
                   attention(moe), attention(dense), attention(moe, kv_from=4 * r + 2)]
    return {"architecture": "Nimelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "embedding": {"scale": width ** 0.5, "bigram": {"buckets": buckets, "mul_prev": 31337, "mul_cur": 1009}}}


def movinex_design(width: int, vocab: int, heads: int, kv_heads: int, dim: int, window: int, keep: int, space: tuple,
                   dense_ff: int, experts: int, top: int, ff: int, groups: tuple, times: int = 2, tail: tuple = (2,),
                   rot: int = 0, eps: float = 1e-6) -> dict:
    """A Movinex ``config.json`` of three kinds of layers - attention with a dense feed-forward, windowed attention with
    experts, a state space (``space``: heads, vdim, state, groups) with experts -, one of each in a loop of ``times`` passes,
    and behind the loop those that ``tail`` names.  ``groups``: count and keep of the router."""
    dense = {"kind": "dense", "ff": dense_ff}
    moe = {"kind": "moe", "expert": {"ff": ff},
           "router": {"experts": experts, "top": top, "groups": dict(zip(("count", "keep"), groups))}}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5}
    kinds = [{"type": "attention", "mlp": dense, "mixer": dict(m, q_temp={"coef": 0.1, "every": 8192})},
             {"type": "attention_2", "mlp": moe, "mixer": dict(m, softcap=30.0, mask={"size": window, "keep_first": keep},
                                                               rot={"dims": rot or dim, "base": 10000.0})},
             {"type": "mamba2", "mlp": moe, "mixer": dict(zip(("heads", "vdim", "state", "groups"), space), conv=4,
                                                          norm_groups=1)}]
    return {"architecture": "Movinex", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": kinds + [kinds[i] for i in tail], "logit_scale": 1.0, "loop": {"start": 0, "stop": 3, "times": times}}


def vobisun_design(width: int, vocab: int, heads: int, kv_heads: int, dim: int, window: int, pool: int, memory: tuple, ff: int,
                   layers: int, loop: tuple = (), rot: int = 0, taps: int = 4, eps: float = 1e-6) -> dict:
    """A Vobisun ``config.json`` of equal layers; ``memory``: heads, dim, vdim of the gated linear attention, ``loop``: start,
    stop, times."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
            "mask": {"size": window, "pool": pool},
            "rot": {"dims": rot or dim, "base": 10000.0, "scaling": {"factor": 1.0}}}
    layer = {"type": "parallel", "mlp": {"kind": "dense", "ff": ff},
             "mixer": {"left": left, "right": dict(zip(("heads", "dim", "vdim"), memory), tau=16.0), "left_scale": 1.0,
                       "right_scale": 1.0}}
    c = {"architecture": "Vobisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [layer] * layers,
         "canon": {"taps": taps}, "embedding": {"scale": width ** 0.5}}
    return dict(c, loop=dict(zip(("start", "stop", "times"), loop))) if loop else c


# entries with a "design" hold a config.json of that architecture instead of ``ModelConfig`` fields
SHAPES = {
    "tiny-ruralorn": dict(arch="ruralorn", design=ruralorn_design(3, 192, 1024, 6, 24, 8, 40, 56, 40, 10, 3, 72, 104)),
    # layers of the size real models of this kind have, a few of them
    "ruralorn-2k": dict(arch="ruralorn", design=ruralorn_design(8, 2048, 102400, 16, 128, 64, 128, 512, 4096, 64, 6, 1408,
                                                                2816)),
    "ruralorn-4k": dict(arch="ruralorn", design=ruralorn_design(4, 4096, 102400, 32, 128, 64, 128, 512, 4096, 64, 4, 2048,
                                                                4096)),
    "tiny-nimelorn": dict(arch="nimelorn", design=nimelorn_design(160, 1024, 6, 2, 32, 24, 48, (3, 40, 56), 224, 10, 3, 72,
                                                                  104, 1.2, buckets=251)),
    "nimelorn-2k": dict(arch="nimelorn", design=nimelorn_design(2048, 102400, 16, 4, 128, 128, 4096, (4, 256, 512), 8192, 64,
                                                                6, 1408, 2816, repeats=2)),
    "nimelorn-4k": dict(arch="nimelorn", design=nimelorn_design(4096, 102400, 32, 8, 128, 128, 4096, (8, 256, 512), 14336,
                                                                64, 4, 2048, 4096)),
    "tiny-movinex": dict(arch="movinex", design=movinex_design(160, 1024, 6, 2, 32, 48, 6, (5, 32, 40, 1), 224, 10, 3, 72,
                                                               (5, 3), rot=16)),
    "movinex-2k": dict(arch="movinex", design=movinex_design(2048, 102400, 16, 4, 128, 2048, 64, (64, 64, 128, 1), 8192, 64, 6,
                                                             1408, (8, 4), tail=(1, 2), rot=64)),
    "movinex-4k": dict(arch="movinex", design=movinex_design(4096, 102400, 32, 8, 128, 2048, 64, (128, 64, 128, 8), 14336, 64,
                                                             4, 2048, (8, 4), times=1, rot=64)),
    "tiny-vobisun": dict(arch="vobisun", design=vobisun_design(160, 1024, 6, 2, 32, 48, 6, (3, 40, 56), 224, 3, (0, 2, 2),
                                                               rot=16)),
    "vobisun-2k": dict(arch="vobisun", design=vobisun_design(2048, 102400, 16, 4, 128, 2048, 16, (16, 128, 256), 8192, 6,
                                                             (1, 3, 2), rot=64)),
    "vobisun-4k": dict(arch="vobisun", design=vobisun_design(4096, 102400, 32, 8, 128, 2048, 16, (32, 128, 256), 14336, 4,
                                                             rot=64)),
    "tiny": dict(num_layers=2, hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=688,
                 vocab_size=1024, rms_norm_eps=1e-6, rope_theta=10000.0, arch="llama", max_seq_len=2048),
    "tiny-aligned": dict(num_layers=2, hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64,
                         intermediate_size=768, vocab_size=1024, rms_norm_eps=1e-6, rope_theta=10000.0, arch="qwen2",
                         max_seq_len=2048),
    "tiny-phi3": dict(num_layers=2, hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=768,
                      vocab_size=1024, rms_norm_eps=1e-5, rope_theta=10000.0, arch="phi3", max_seq_len=2048),
    "small-128": dict(num_layers=2, hidden_size=512, num_heads=4, num_kv_heads=2, head_dim=128,
                      intermediate_size=1024, vocab_size=2048, rms_norm_eps=1e-6, rope_theta=1e6, arch="qwen2",
                      max_seq_len=4096),
    # an intermediate size whose 128-column groups (15) do not divide evenly over 2, 4 or 8 ranks, and 8 kv heads so
    # that every rank count up to 8 gets whole heads: the small analogue of a 13824-wide MLP on 8 GPUs
    "small-uneven": dict(num_layers=2, hidden_size=1024, num_heads=8, num_kv_heads=8, head_dim=128,
                         intermediate_size=1920, vocab_size=2048, rms_norm_eps=1e-6, rope_theta=1e6, arch="qwen2",
                         max_seq_len=4096),
    # Gemma-2 block: four norms, GeGLU, soft-capped scores and logits, local/global layers alternate
    "tiny-gemma2": dict(num_layers=4, hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64,
                        intermediate_size=768, vocab_size=1024, rms_norm_eps=1e-6, rope_theta=10000.0, arch="gemma2",
                        max_seq_len=2048, sliding_window=24, query_pre_attn_scalar=64.0, attn_logit_softcapping=50.0,
                        final_logit_softcapping=30.0, hidden_activation="gelu_pytorch_tanh", embed_scale=True,
                        tie_word_embeddings=True,
                        layer_types=["sliding_attention", "full_attention"] * 2),
    # Gemma-4 block: q/k/v head norms, local layers (head_dim 64) and global layers (head_dim 128, a quarter of it
    # rotated, V = K projection, one kv head), learned layer scalars
    "tiny-gemma4": dict(num_layers=3, hidden_size=256, num_heads=4, num_kv_heads=2, head_dim=64,
                        intermediate_size=768, vocab_size=1024, rms_norm_eps=1e-6, rope_theta=10000.0, arch="gemma4",
                        max_seq_len=2048, sliding_window=24, global_head_dim=128, global_num_kv_heads=1,
                        global_rope_theta=1e6, partial_rotary_factor=0.25, attention_k_eq_v=True,
                        final_logit_softcapping=30.0, hidden_activation="gelu_pytorch_tanh", embed_scale=True,
                        tie_word_embeddings=True,
                        layer_types=["sliding_attention", "sliding_attention", "full_attention"]),
    "gemma2-9b": dict(num_layers=42, hidden_size=3584, num_heads=16, num_kv_heads=8, head_dim=256,
                      intermediate_size=14336, vocab_size=256000, rms_norm_eps=1e-6, rope_theta=10000.0,
                      arch="gemma2", max_seq_len=8192, sliding_window=4096, query_pre_attn_scalar=256.0,
                      attn_logit_softcapping=50.0, final_logit_softcapping=30.0,
                      hidden_activation="gelu_pytorch_tanh", embed_scale=True, tie_word_embeddings=True,
                      layer_types=["sliding_attention", "full_attention"] * 21),
    "qwen2.5-7b": dict(num_layers=28, hidden_size=3584, num_heads=28, num_kv_heads=4, head_dim=128,
                       intermediate_size=18944, vocab_size=152064, rms_norm_eps=1e-6, rope_theta=1e6, arch="qwen2",
                       max_seq_len=32768),
    "qwen2.5-14b": dict(num_layers=48, hidden_size=5120, num_heads=40, num_kv_heads=8, head_dim=128,
                        intermediate_size=13824, vocab_size=152064, rms_norm_eps=1e-6, rope_theta=1e6, arch="qwen2",
                        max_seq_len=32768),
    "qwen2.5-32b": dict(num_layers=64, hidden_size=5120, num_heads=40, num_kv_heads=8, head_dim=128,
                        intermediate_size=27648, vocab_size=152064, rms_norm_eps=1e-6, rope_theta=1e6, arch="qwen2",
                        max_seq_len=32768),
    "qwen2.5-72b": dict(num_layers=80, hidden_size=8192, num_heads=64, num_kv_heads=8, head_dim=128,
                        intermediate_size=29568, vocab_size=152064, rms_norm_eps=1e-6, rope_theta=1e6, arch="qwen2",
                        max_seq_len=32768),
}


def shape_config(name: str, quant: str = "int4", **overrides) -> ModelConfig:
    kw = dict(SHAPES[name])
    if "design" in kw:
        from .arch import get_adapter
        c = get_adapter(kw["arch"]).config_from_hf(kw["design"])
        for k, v in overrides.items():
            setattr(c, k, v)
        return c
    kw.update(overrides)
    method = {"int4": QuantMethod.INT4_ASYM, "int8": QuantMethod.INT8_SYM, "fp16": QuantMethod.NONE}[quant]
    bits = {"int4": 4, "int8": 8, "fp16": 16}[quant]
    return ModelConfig(quant=QuantConfig(method=int(method), bits=bits, group_size=128), **kw)


def byte_tokenizer(vocab_size: int = 1024) -> BPETokenizer:
    """A real (if dull) byte-level BPE tokenizer: 256 byte symbols, a few merges, ChatML markers."""
    vocab = {BYTE_ENCODER[b]: b for b in range(256)}
    merges = []
    for a, b in (("t", "h"), ("i", "n"), ("th", "e"), ("Ġ", "t"), ("Ġ", "a"), ("e", "r"), ("a", "n"), ("o", "n")):
        if a + b not in vocab and len(vocab) < vocab_size - 8:
            vocab[a + b] = len(vocab)
            merges.append((a, b))
    nxt = len(vocab)
    added = {"<|endoftext|>": nxt, "<|im_start|>": nxt + 1, "<|im_end|>": nxt + 2}
    return BPETokenizer(vocab=vocab, merges=merges, added_tokens=added,
                        special_tokens=SpecialTokens(bos_id=nxt, eos_id=nxt, pad_id=nxt, unk_id=0))


def layer_weight_shapes(c: ModelConfig, layer: int = 0):
    sp = c.layer_spec(layer) if c.is_gemma else None
    q_dim = c.num_heads * sp.head_dim if sp else c.q_dim
    kv_dim = sp.num_kv_heads * sp.head_dim if sp else c.kv_dim
    if c.arch == "phi3":        # [q; k; v] and [gate; up] are stored stacked
        return [("self_attn.qkv_proj", q_dim + 2 * kv_dim, c.hidden_size), ("self_attn.o_proj", c.hidden_size, q_dim),
                ("mlp.gate_up_proj", 2 * c.intermediate_size, c.hidden_size),
                ("mlp.down_proj", c.hidden_size, c.intermediate_size)]
    out = [("self_attn.q_proj", q_dim, c.hidden_size), ("self_attn.k_proj", kv_dim, c.hidden_size)]
    if not (sp and sp.k_is_v):
        out.append(("self_attn.v_proj", kv_dim, c.hidden_size))
    return out + [("self_attn.o_proj", c.hidden_size, q_dim), ("mlp.gate_proj", c.intermediate_size, c.hidden_size),
                  ("mlp.up_proj", c.intermediate_size, c.hidden_size),
                  ("mlp.down_proj", c.hidden_size, c.intermediate_size)]


def latent_tensor_shapes(c: ModelConfig):
    """(name, shape) of every tensor of a design with latent attention, in file order."""
    H = c.hidden_size
    yield "embed", (c.vocab_size, H)
    for i in range(c.num_layers):
        p, a, m = f"l{i}.", c.latent_spec(i), c.moe_spec(i)
        yield p + "norm1", (H,)
        yield p + "mix.q", (a.heads * a.qk_dim, H)
        yield p + "mix.dkv", (a.kv_rank + a.rot_dim, H)
        yield p + "mix.dkv.norm", (a.kv_rank,)
        yield p + "mix.uk", (a.heads * a.dim, a.kv_rank)
        yield p + "mix.uv", (a.heads * a.vdim, a.kv_rank)
        yield p + "mix.g", (a.heads * a.vdim, H)
        yield p + "mix.o", (H, a.heads * a.vdim)
        if m is None:
            continue
        yield p + "norm2", (H,)
        yield p + "mlp.router", (m.experts, H)
        parts = [(f"mlp.e{e}", m.ff) for e in range(m.experts)] + ([("mlp.shared", m.shared_ff)] if m.shared_ff else [])
        for name, ff in parts:
            yield f"{p}{name}.up", (ff, H)
            yield f"{p}{name}.down", (H, ff)
    yield "final.norm", (H,)
    yield "head", (c.vocab_size, H)


def _random_bf16(rng, shape, fast: bool) -> np.ndarray:
    """N(0, 1/fan_in) matrices, norm weights around 1, as bfloat16 bit patterns.  ``fast`` repeats one block of values."""
    from .convert import round_bf16
    if len(shape) == 1:
        return round_bf16(1.0 + 0.1 * rng.standard_normal(shape, dtype=np.float32))
    n = shape[0] * shape[1]
    block = min(n, 1 << 20) if fast else n
    bits = round_bf16(rng.standard_normal(block, dtype=np.float32) * shape[1] ** -0.5)
    return np.resize(bits, n).reshape(shape)


def write_random_model(path: str, config: ModelConfig, seed: int = 0, std: float = 0.02, fast: bool = False,
                       with_tokenizer: bool = True, qkv_bias: Optional[bool] = None) -> None:
    rng = np.random.default_rng(seed)
    c = config
    qkv_bias = (c.arch == "qwen2") if qkv_bias is None else qkv_bias
    gs = c.quant.group_size
    w = ZSEWriter(path)
    w.set_config(c)
    if with_tokenizer:
        w.set_tokenizer(byte_tokenizer(c.vocab_size).serialize())
    w.begin_weights()
    if c.is_design:
        from .arch import get_adapter
        shapes = latent_tensor_shapes(c) if c.is_latent else get_adapter(c.arch).tensor_shapes(c)
        for name, shape in shapes:
            w.add_weight_raw_bf16(name, shape, _random_bf16(rng, shape, fast))
        w.finalize()
        return

    def linear(name, n, k):
        if c.quant.method == QuantMethod.NONE:
            w.add_weight_raw_fp16(name, (n, k), (rng.standard_normal((n, k), dtype=np.float32) * std).astype(np.float16))
        elif fast and c.quant.method == QuantMethod.INT4_ASYM:
            total = n * k
            groups = (total + gs - 1) // gs
            packed = np.frombuffer(rng.bytes(groups * gs // 2), dtype=np.uint8)
            # range of 128 N(0,std) samples is about 5.2 std wide, centred near 0
            half = (2.6 + 0.35 * rng.standard_normal(groups, dtype=np.float32)).clip(1.5, 4.0) * std
            w.add_weight_raw(name, (n, k), packed, (2 * half / 15).astype(np.float16), (-half).astype(np.float16), gs)
        else:
            w.add_weight(name, rng.standard_normal((n, k), dtype=np.float32) * std, (n, k), quantize=True)

    def fp16(name, shape, values):
        w.add_weight_raw_fp16(name, shape, np.asarray(values, dtype=np.float16))

    def big_fp16(name, n, k):
        if fast:  # one random block of rows, repeated: N(0, std) entries, a fraction of the generation time
            rows = min(n, 4096)
            block = (rng.standard_normal((rows, k), dtype=np.float32) * std).astype(np.float16)
            fp16(name, (n, k), np.tile(block, ((n + rows - 1) // rows, 1))[:n])
        else:
            fp16(name, (n, k), rng.standard_normal((n, k), dtype=np.float32) * std)

    # stored norm weights: Gemma-2 files hold w - 1
    norm_mean = 1.0 - c.norm_weight_offset

    def norm(name, n):
        fp16(name, (n,), norm_mean + 0.1 * rng.standard_normal(n))

    big_fp16("embed_tokens.weight", c.vocab_size, c.hidden_size)
    for i in range(c.num_layers):
        p = f"layers.{i}"
        fp16(f"{p}.input_layernorm.weight", (c.hidden_size,), norm_mean + 0.1 * rng.standard_normal(c.hidden_size))
        if c.is_gemma:
            norm(f"{p}.pre_feedforward_layernorm.weight", c.hidden_size)
            norm(f"{p}.post_feedforward_layernorm.weight", c.hidden_size)
            sp = c.layer_spec(i)
            if sp.qk_norm:
                norm(f"{p}.self_attn.q_norm.weight", sp.head_dim)
                norm(f"{p}.self_attn.k_norm.weight", sp.head_dim)
                fp16(f"{p}.layer_scalar", (1,), [0.8 + 0.4 * rng.random()])
        for name, n, k in layer_weight_shapes(c, i):
            linear(f"{p}.{name}.weight", n, k)
            if qkv_bias and name.split(".")[-1] in ("q_proj", "k_proj", "v_proj"):
                fp16(f"{p}.{name}.bias", (n,), rng.standard_normal(n) * std)
        fp16(f"{p}.post_attention_layernorm.weight", (c.hidden_size,),
             norm_mean + 0.1 * rng.standard_normal(c.hidden_size))
    fp16("norm.weight", (c.hidden_size,), norm_mean + 0.1 * rng.standard_normal(c.hidden_size))
    if not c.tie_word_embeddings:
        big_fp16("lm_head.weight", c.vocab_size, c.hidden_size)
    w.finalize()
