"""Plain, slow restatement of the Ruralorn equations in float64: one function per mechanism, whole sequences only, no cache,
no batching.  Nothing of the package is used here; the tests compare the package against it.

Also builds small random models: a configuration, weights that are exact in bfloat16, and the directory that holds both.
"""
import json
import math
import os
import struct

import torch

F = torch.float64


# ---- mechanisms -----------------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps) * w


def rotate(v, positions, dims, base):
    """v [T, R]: pairs (2i, 2i+1), i < dims/2, turn by position * base^(-2i/dims)."""
    out = v.clone()
    for i in range(dims // 2):
        a = positions.to(F) * base ** (-2.0 * i / dims)
        u, w = v[:, 2 * i], v[:, 2 * i + 1]
        out[:, 2 * i] = u * torch.cos(a) - w * torch.sin(a)
        out[:, 2 * i + 1] = w * torch.cos(a) + u * torch.sin(a)
    return out


def window_mask(T, window):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see & (i - j < window) if window else see


def latent_attention(W, p, m, h, eps):
    T = h.shape[0]
    H, d, r, vd, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = h @ W[p + "q"].T
    down = h @ W[p + "dkv"].T
    c = rms_norm(down[:, :kr], W[p + "dkv.norm"], eps)
    k_rot = rotate(down[:, kr:], pos, m["rot"]["dims"], m["rot"]["base"])
    see = window_mask(T, m["mask"]["size"])
    heads = []
    for n in range(H):
        qn = q[:, n * (d + r): n * (d + r) + d]
        qr = rotate(q[:, n * (d + r) + d: (n + 1) * (d + r)], pos, m["rot"]["dims"], m["rot"]["base"])
        k = c @ W[p + "uk"][n * d: (n + 1) * d].T
        v = c @ W[p + "uv"][n * vd: (n + 1) * vd].T
        s = (qn @ k.T + qr @ k_rot.T) * m["scale"]
        heads.append(torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v)
    y = torch.cat(heads, -1) * torch.sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def expert(W, p, x):
    return gelu(x @ W[p + "up"].T) @ W[p + "down"].T


def routed_ff(W, p, m, h):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        s = torch.sigmoid(W[p + "router"] @ h[t])
        for e in sorted(range(len(s)), key=lambda e: (-float(s[e]), e))[: m["router"]["top"]]:
            out[t] += expert(W, f"{p}e{e}.", s[e] * h[t])
        if m.get("shared"):
            out[t] += expert(W, p + "shared.", h[t])
    return out


def head(W, cfg, x):
    z = rms_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * torch.tanh(z / cfg["logit_softcap"])


def forward(cfg, weights, tokens):
    """Logits [T, vocab]."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + latent_attention(W, p + "mix.", L["mixer"], rms_norm(x, W[p + "norm1"], eps), eps)
        if L["mlp"] is not None:
            x = x + routed_ff(W, p + "mlp.", L["mlp"], rms_norm(x, W[p + "norm2"], eps))
    return head(W, cfg, x)


def greedy(cfg, weights, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, weights, seq)[-1].argmax()))
    return seq[len(prompt):]


# ---- small random models --------------------------------------------------------------------------------------------
def mixer(heads, dim, rot_dim, vdim, kv_rank, window, base=500.0, scale=None, rot_dims=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
            "scale": scale or (dim + rot_dim) ** -0.5, "mask": {"size": window},
            "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, embed_scale=0.7, logit_scale=0.8, softcap=20.0, eps=1e-4):
    return {"architecture": "Ruralorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "logit_softcap": softcap,
            "layers": [{"type": "latent_attention", "mixer": a, "mlp": b} for a, b in layers]}


def shapes(cfg):
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    for i, L in enumerate(cfg["layers"]):
        a, m, p = L["mixer"], L["mlp"], f"l{i}."
        H, kr = a["heads"], a["kv_rank"]
        out.update({p + "norm1": (D,), p + "mix.q": (H * (a["dim"] + a["rot_dim"]), D),
                    p + "mix.dkv": (kr + a["rot_dim"], D), p + "mix.dkv.norm": (kr,), p + "mix.uk": (H * a["dim"], kr),
                    p + "mix.uv": (H * a["vdim"], kr), p + "mix.g": (H * a["vdim"], D), p + "mix.o": (D, H * a["vdim"])})
        if m:
            out.update({p + "norm2": (D,), p + "mlp.router": (m["router"]["experts"], D)})
            for e in range(m["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.up": (m["expert"]["ff"], D), f"{p}mlp.e{e}.down": (D, m["expert"]["ff"])})
            if m.get("shared"):
                out.update({p + "mlp.shared.up": (m["shared"]["ff"], D), p + "mlp.shared.down": (D, m["shared"]["ff"])})
    return out


def random_weights(cfg, seed=0, sharp=5.0):
    """bfloat16 weights.  Queries are scaled up by ``sharp`` so that single keys stand out of the softmax: a key that is
    missing, or one too many at a window's edge, then moves the logits."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        if len(shape) == 1:
            w = 1 + 0.2 * torch.randn(shape, generator=g)
        else:
            w = torch.randn(shape, generator=g) * shape[1] ** -0.5
            if name.endswith("mix.q"):
                w *= sharp
            if name == "embed":
                w *= shape[1] ** 0.5
            if name.endswith("down") or name.endswith("mix.o"):
                w *= 1.5
        W[name] = w.to(torch.bfloat16)
    return W


def write_model(path, cfg, weights):
    """A model directory: config.json and model.safetensors."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, w in weights.items():
        raw = w.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(w.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return str(path)
