"""Plain, slow restatement of the Vobisun equations in float64: one function per mechanism, whole sequences only, no cache,
no batching.  Nothing of the package is used here; the tests compare the package against it.

Also builds small random models: a configuration and weights that are exact in bfloat16.
"""
import math

import torch

F = torch.float64


# ---- mechanisms -----------------------------------------------------------------------------------------------------
def norm(x, w, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def with_history(h, w):
    """h [T, width] plus its causal convolution per channel; w [width, taps], the last tap is the row's own."""
    T, taps = len(h), w.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def turn_pairs(x, dims, base, factor=1.0):
    """x [T, heads, dim]: neighbours (0, 1), (2, 3), ... of the first ``dims`` turn, slower by ``factor``."""
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=F)[:, None]
    for i in range(dims // 2):
        a = p * (base ** (-2 * i / dims) / factor)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def block_means(x, P):
    """x [T, ...] -> [T // P, ...]: means of the whole blocks of P rows."""
    n = len(x) // P
    return torch.stack([x[b * P: (b + 1) * P].mean(0) for b in range(n)]) if n else x[:0]


def seen_tokens(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def seen_blocks(T, size, P):
    i, b = torch.arange(T)[:, None], torch.arange(T // P)[None, :]
    return b * P + P - 1 <= i - size


def pooled_attention(q, k, v, scale, size, P, sink):
    """One head: q [T, d], k [T, d], v [T, vd]; ``scale`` with the head's own factor; ``sink``: one more score without a value."""
    T = len(q)
    keys, values = torch.cat([k, block_means(k, P)]), torch.cat([v, block_means(v, P)])
    see = torch.cat([seen_tokens(T, size), seen_blocks(T, size, P)], 1)
    s = torch.cat([(q @ keys.T * scale).masked_fill(~see, -math.inf), sink.expand(T, 1)], 1)
    return torch.softmax(s, -1)[:, :-1] @ values


def window_attention(W, p, m, h, eps):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    proj = lambda name: h @ W[p + name].T + W[p + name + ".b"]
    q = norm(proj("q"), W[p + "q.norm"], eps).view(T, H, m["dim"])
    k = norm(proj("k"), W[p + "k.norm"], eps).view(T, G, m["dim"])
    v = proj("v").view(T, G, m["vdim"])
    r = m["rot"]
    q, k = (turn_pairs(x, r["dims"], r["base"], r["scaling"]["factor"]) for x in (q, k))
    gate = sigmoid(h @ W[p + "g"].T)
    y = []
    for n in range(H):
        g = n // (H // G)
        y.append(gate[:, n: n + 1] * pooled_attention(q[:, n], k[:, g], v[:, g], m["scale"] * W[p + "temp"][n],
                                                      m["mask"]["size"], m["mask"]["pool"], W[p + "sink"][n]))
    return torch.cat(y, -1) @ W[p + "o"].T


def decayed_memory(q, k, v, alpha):
    """One head, token by token: q, k, alpha [T, d], v [T, vd]; returns [T, vd]."""
    S, out = torch.zeros(q.shape[1], v.shape[1], dtype=F), []
    for t in range(len(q)):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def linear_attention(W, p, m, h, eps):
    T, H, d, vd = len(h), m["heads"], m["dim"], m["vdim"]
    q, k = (h @ W[p + "q"].T).view(T, H, d) * d ** -0.5, (h @ W[p + "k"].T).view(T, H, d)
    v = (h @ W[p + "v"].T).view(T, H, vd)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = (sigmoid(z) ** (1 / m["tau"])).view(T, H, d)
    y = torch.cat([norm(decayed_memory(q[:, n], k[:, n], v[:, n], alpha[:, n]), W[p + "norm"], eps) for n in range(H)], -1)
    return (y * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def two_mixers(W, p, m, h, eps):
    return m["left_scale"] * window_attention(W, p + "left.", m["left"], h, eps) \
        + m["right_scale"] * linear_attention(W, p + "right.", m["right"], h, eps)


def gated_ff(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def run_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, weights, tokens, residuals=None):
    """Logits [T, vocab]; ``residuals``: a list that receives x after every layer run."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i in run_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        h = norm(x, W[p + "norm1"], eps)
        y = two_mixers(W, p + "mix.", L["mixer"], with_history(h, W[p + "canon1"]), eps)
        if L["mlp"] is not None:
            y = y + gated_ff(W, p + "mlp.", h)
        x = x + y
        if residuals is not None:
            residuals.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T


def greedy(cfg, weights, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, weights, seq)[-1].argmax()))
    return seq[len(prompt):]


# ---- small random models --------------------------------------------------------------------------------------------
def layer(left, right, mlp, scales=(0.9, 0.6)):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": right, "left_scale": scales[0],
                                                      "right_scale": scales[1]}}


def window(heads, kv_heads, dim, vdim, size, pool, rot=None, base=1e4, factor=1.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 2 * dim ** -0.5,
            "mask": {"size": size, "pool": pool},
            "rot": {"dims": dim if rot is None else rot, "base": base, "scaling": {"factor": factor}}}


def memory(heads, dim, vdim, tau=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, layers, loop=None, taps=4, embed_scale=3.0, eps=1e-5, ranks=None):
    """``loop``: (start, stop, times); ``ranks``: of the layers' decay projections, which only the tensors' shapes tell."""
    c = {"architecture": "Vobisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
         "canon": {"taps": taps}, "embedding": {"scale": embed_scale}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c, ranks or [16] * len(layers)


def shapes(cfg, ranks):
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    for i, L in enumerate(cfg["layers"]):
        p, a, r, m = f"l{i}.", L["mixer"]["left"], L["mixer"]["right"], L["mlp"]
        nq, nk, nv = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
        rk, rv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
        out.update({p + "norm1": (D,), p + "canon1": (D, cfg["canon"]["taps"])})
        left = {"q": (nq, D), "q.b": (nq,), "q.norm": (nq,), "k": (nk, D), "k.b": (nk,), "k.norm": (nk,), "v": (nv, D),
                "v.b": (nv,), "temp": (a["heads"],), "sink": (a["heads"],), "g": (a["heads"], D),
                "o": (D, a["heads"] * a["vdim"])}
        right = {"q": (rk, D), "k": (rk, D), "v": (rv, D), "g": (rv, D), "o": (D, rv), "norm": (r["vdim"],),
                 "a1": (ranks[i], D), "a2": (rk, ranks[i]), "a2.b": (rk,)}
        out.update({p + "mix.left." + k: v for k, v in left.items()})
        out.update({p + "mix.right." + k: v for k, v in right.items()})
        if m is not None:
            out.update({p + "mlp.gate": (m["ff"], D), p + "mlp.up": (m["ff"], D), p + "mlp.down": (D, m["ff"])})
    return out


def random_weights(cfg, ranks, seed=0):
    """bfloat16 weights.  Every mechanism has a share in the logits: query and key norms that let single keys stand out, sinks
    as large as the scores, decays from a few tokens to hundreds, biases and convolutions of the size of what they join."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda shape: torch.randn(shape, generator=g)
    W = {}
    for name, shape in shapes(cfg, ranks).items():
        last = name.rsplit(".right.", 1)[-1].rsplit(".left.", 1)[-1]
        if last in ("q.norm", "k.norm"):
            w = 1.2 + 0.5 * rnd(shape)
        elif "norm" in last:
            w = 1 + 0.3 * rnd(shape)
        elif last == "temp":
            w = 1 + 0.4 * rnd(shape)
        elif last == "sink":
            w = 2 + rnd(shape)
        elif last == "a2.b":
            w = 2 + 2 * rnd(shape)
        elif last in ("q.b", "k.b", "v.b"):
            w = 0.5 * rnd(shape)
        elif last.endswith("canon1"):
            w = 0.7 * rnd(shape) * shape[1] ** -0.5
        else:
            w = rnd(shape) * shape[1] ** -0.5
        W[name] = w.to(torch.bfloat16)
    return W
