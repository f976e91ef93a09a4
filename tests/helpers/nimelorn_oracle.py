"""Plain, slow restatement of the Nimelorn equations in float64: one function per mechanism, whole sequences only, no cache,
no batching.  Nothing of the package is used here; the tests compare the package against it.

Also builds small random models: a configuration and weights that are exact in bfloat16.
"""
import math

import torch

F = torch.float64


# ---- mechanisms -----------------------------------------------------------------------------------------------------
def root_mean_square_norm(x, eps, w=None):
    y = x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def bigram_rows(tokens, b):
    """Row of the bigram table for every token of a sequence; the first token has a row of its own, the last."""
    return [b["buckets"] if i == 0 else (tokens[i - 1] * b["mul_prev"] + tokens[i] * b["mul_cur"]) % b["buckets"]
            for i in range(len(tokens))]


def sinusoid(T, width):
    out = torch.zeros(T, width, dtype=F)
    for p in range(T):
        for j in range(width):
            a = p * 10000.0 ** (-(j - j % 2) / width)
            out[p, j] = math.cos(a) if j % 2 else math.sin(a)
    return out


def embed(cfg, W, tokens):
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    if "bigram" in cfg["embedding"]:
        x = x + W["bigram"][torch.tensor(bigram_rows(tokens, cfg["embedding"]["bigram"]))]
    return root_mean_square_norm(x + sinusoid(len(tokens), cfg["width"]), cfg["norm"]["eps"], W["embed.norm"])


def chunk_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def keys_values(W, p, m, h, eps):
    """[T, kv_heads, dim] and [T, kv_heads, vdim] of a layer that has its own."""
    k = (h @ W[p + "k"].T).view(len(h), m["kv_heads"], m["dim"])
    v = (h @ W[p + "v"].T).view(len(h), m["kv_heads"], m["vdim"])
    return root_mean_square_norm(k, eps, W[p + "k.norm"]), v


def attention(W, p, m, h, eps, kv):
    k, v = kv
    T, H = len(h), m["heads"]
    q = root_mean_square_norm((h @ W[p + "q"].T).view(T, H, m["dim"]), eps, W[p + "q.norm"])
    gate = torch.sigmoid(h @ W[p + "g"].T)
    see = chunk_mask(T, m["mask"]["size"])
    heads = []
    for n in range(H):
        g = n // (H // m["kv_heads"])
        s = (q[:, n] @ k[:, g].T) * m["scale"]
        heads.append(gate[:, n: n + 1] * (torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]))
    return torch.cat(heads, -1) @ W[p + "o"].T


def mlstm_gates(W, p, m, h):
    """Log input and log forget gates [T, heads]."""
    cap = m["gate_cap"]
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap)
    return i, -torch.log1p(torch.exp(-f))


def mlstm_recurrence(q, k, v, i, f):
    """One head, token by token: q, k [T, dim], v [T, vdim], i, f [T]; returns [T, vdim]."""
    T, d = q.shape
    S, n, m = torch.zeros(d, v.shape[1], dtype=F), torch.zeros(d, dtype=F), torch.zeros((), dtype=F)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = new
        out.append(S.T @ q[t] / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out)


def mlstm(W, p, m, h, eps):
    T, H, d, vd = len(h), m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, d)
    v = (h @ W[p + "v"].T).view(T, H, vd)
    i, f = mlstm_gates(W, p, m, h)
    o = torch.stack([mlstm_recurrence(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n]) for n in range(H)], 1)
    y = root_mean_square_norm(o, eps).reshape(T, H * vd) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


def dense_ff(W, p, h):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def expert(W, p, limit, x):
    g = (x @ W[p + "gate"].T).clamp(max=limit)
    u = (x @ W[p + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T


def routed_ff(W, p, m, h):
    out = torch.zeros_like(h)
    r = m["router"]
    for t in range(len(h)):
        s = torch.softmax(W[p + "router"] @ h[t], -1)
        chosen = sorted(range(len(s)), key=lambda e: (-float(s[e]), e))[: r["top"]]
        total = sum(s[e] for e in chosen) + 1e-20
        for e in chosen:
            out[t] += r.get("scale", 1.0) * s[e] / total * expert(W, f"{p}e{e}.", m["expert"]["limit"], h[t])
        if m.get("shared"):
            out[t] += torch.sigmoid(W[p + "shared.sg"] @ h[t]) * expert(W, p + "shared.", m["shared"]["limit"], h[t])
    return out


def forward(cfg, weights, tokens, residuals=None):
    """Logits [T, vocab]; ``residuals``: a list that receives x after every layer."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(cfg, W, tokens)
    kv = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "mlstm":
            y = mlstm(W, p + "mix.", m, x, eps)
        else:
            if "kv_from" not in m:
                kv[i] = keys_values(W, p + "mix.", m, x, eps)
            y = attention(W, p + "mix.", m, x, eps, kv[m.get("kv_from", i)])
        x = x + root_mean_square_norm(y, eps, W[p + "norm1"])
        if L["mlp"] is not None:
            ff = dense_ff(W, p + "mlp.", x) if L["mlp"]["kind"] == "dense" else routed_ff(W, p + "mlp.", L["mlp"], x)
            x = x + root_mean_square_norm(ff, eps, W[p + "norm2"])
        if residuals is not None:
            residuals.append(x)
    return root_mean_square_norm(x, eps, W["final.norm"]) @ W["head"].T


def greedy(cfg, weights, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, weights, seq)[-1].argmax()))
    return seq[len(prompt):]


# ---- small random models --------------------------------------------------------------------------------------------
def attention_layer(heads, kv_heads, dim, vdim, chunk, mlp, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
         "scale": scale or dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mlstm_layer(heads, dim, vdim, mlp, gate_cap=12.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, scale=1.0, shared=None, shared_limit=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit or limit}
    return m


def config(width, vocab, layers, embed_scale=6.0, eps=1e-5, buckets=61, mul_prev=7, mul_cur=5):
    return {"architecture": "Nimelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "embedding": {"scale": embed_scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


def shapes(cfg):
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, D), "embed.norm": (D,),
           "final.norm": (D,), "head": (cfg["vocab"], D)}
    for i, L in enumerate(cfg["layers"]):
        a, m, p = L["mixer"], L["mlp"], f"l{i}."
        H, d, v = a["heads"], a["dim"], a["vdim"]
        out.update({p + "norm1": (D,), p + "mix.q": (H * d, D), p + "mix.o": (D, H * v)})
        if L["type"] == "mlstm":
            out.update({p + "mix.k": (H * d, D), p + "mix.v": (H * v, D), p + "mix.g": (H * v, D), p + "mix.norm": (H * v,),
                        p + "mix.i": (H, D), p + "mix.f": (H, D), p + "mix.i.b": (H,), p + "mix.f.b": (H,)})
        else:
            out.update({p + "mix.q.norm": (d,), p + "mix.g": (H, D)})
            if "kv_from" not in a:
                out.update({p + "mix.k": (a["kv_heads"] * d, D), p + "mix.v": (a["kv_heads"] * v, D), p + "mix.k.norm": (d,)})
        if m is None:
            continue
        out[p + "norm2"] = (D,)
        if m["kind"] == "dense":
            out.update({p + "mlp.up": (m["ff"], D), p + "mlp.down": (D, m["ff"])})
            continue
        out[p + "mlp.router"] = (m["router"]["experts"], D)
        parts = [(f"e{e}", m["expert"]["ff"]) for e in range(m["router"]["experts"])]
        if m.get("shared"):
            out[p + "mlp.shared.sg"] = (1, D)
            parts.append(("shared", m["shared"]["ff"]))
        for name, ff in parts:
            out.update({f"{p}mlp.{name}.gate": (ff, D), f"{p}mlp.{name}.up": (ff, D), f"{p}mlp.{name}.down": (D, ff)})
    return out


def random_weights(cfg, seed=0, sharp=2.5):
    """bfloat16 weights.  Query norms are scaled up by ``sharp`` so that single keys stand out of the softmax; forget gates
    stay open for some fifty tokens and input gates differ from token to token, so that a lost or misplaced state moves the
    logits; up products reach the clamps."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        if name.endswith("i.b"):
            w = 0.5 * torch.randn(shape, generator=g)
        elif name.endswith("f.b"):
            w = 4.0 + torch.randn(shape, generator=g)
        elif len(shape) == 1:
            w = 1 + 0.2 * torch.randn(shape, generator=g)
            if name.endswith("q.norm"):
                w *= sharp
        else:
            w = torch.randn(shape, generator=g) * shape[1] ** -0.5
            if name in ("embed", "bigram"):
                w *= shape[1] ** 0.5 * (0.15 if name == "embed" else 0.8)
            if name.endswith("mix.i"):
                w *= 2.0
            if name.endswith("gate") or name.endswith("up"):
                w *= 1.5
        W[name] = w.to(torch.bfloat16)
    return W
