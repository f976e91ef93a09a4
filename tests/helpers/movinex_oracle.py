"""Plain, slow restatement of the Movinex equations in float64: one function per mechanism, whole sequences only, no cache,
no batching.  Nothing of the package is used here; the tests compare the package against it.

Also builds small random models: a configuration and weights that are exact in bfloat16.
"""
import math

import torch

F = torch.float64


# ---- mechanisms -----------------------------------------------------------------------------------------------------
def rms(x, eps):
    return torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The stored weight is the difference from one."""
    return x / rms(x, eps) * (1 + w)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(z.clamp(max=30))))


def query_factor(T, coef, every):
    """One number per position that multiplies its query."""
    return torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(T)], dtype=F)


def turn_pairs(x, dims, base):
    """x [T, heads, dim]: neighbours (0, 1), (2, 3), ... of the first ``dims`` turn, the others stay."""
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=F)[:, None]
    for i in range(dims // 2):
        a = p * base ** (-2 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def visible(T, size=None, keep=0):
    """[T, T]: query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((j <= i) if size is None else (i - j < size) | (j < keep))


def weighted_values(q, k, v, scale, see, softcap=None):
    """One head: q [T, d], k [T, d], v [T, vd]."""
    s = q @ k.T * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    return torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v


def heads_of(q, k, v, m, see, softcap=None):
    per = m["heads"] // m["kv_heads"]
    return torch.cat([weighted_values(q[:, n], k[:, n // per], v[:, n // per], m["scale"], see, softcap)
                      for n in range(m["heads"])], -1)


def plain_attention(W, p, m, h, eps):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    proj = lambda name, n, d: (h @ W[p + name].T + W[p + name + ".b"]).view(T, n, d)
    q, k, v = proj("q", H, m["dim"]), proj("k", G, m["dim"]), proj("v", G, m["vdim"])
    q, k = q / rms(q, eps), k / rms(k, eps)
    q = q * query_factor(T, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    return heads_of(q, k, v, m, visible(T)) @ W[p + "o"].T


def windowed_attention(W, p, m, h, eps):
    T, H, G, d = len(h), m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ W[p + "q"].T).view(T, H, d), (h @ W[p + "k"].T).view(T, G, d)
    v = k
    q, k = (turn_pairs(x, m["rot"]["dims"], m["rot"]["base"]) for x in (q, k))
    q, k = q / rms(q, eps), k / rms(k, eps)
    y = heads_of(q, k, v, m, visible(T, m["mask"]["size"], m["mask"]["keep_first"]), m["softcap"])
    return (y * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def causal_conv(x, w, b):
    """x [T, channels], w [channels, taps] (the last tap is the row's own), b [channels]."""
    T, taps = len(x), w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out + b


def state_space(x, B, C, dt, A_log, D):
    """One head, token by token: x [T, vdim], B, C [T, N], dt [T]; returns [T, vdim]."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=F)
    out = []
    for t in range(len(x)):
        S = torch.exp(-torch.exp(A_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        out.append(S.T @ C[t] + D * x[t])
    return torch.stack(out)


def norm_in_parts(y, parts, eps):
    z = y.view(len(y), parts, -1)
    return (z / rms(z, eps)).view_as(y)


def mamba2(W, p, m, h, eps):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ W[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    dt = softplus(dt + W[p + "dt_bias"])
    y = []
    for n in range(H):
        g = n // (H // G)
        y.append(state_space(x[:, n * V: (n + 1) * V], B[:, g * N: (g + 1) * N], C[:, g * N: (g + 1) * N], dt[:, n],
                             W[p + "A_log"][n], W[p + "D"][n]))
    y = torch.cat(y, -1) * silu(z)
    return (norm_in_parts(y, m["norm_groups"], eps) * W[p + "norm"]) @ W[p + "o"].T


def glu(W, p, act, x):
    return (act(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def choose(s, top, groups, keep):
    """Expert ids of one token from its scores ``s``; the lower id, and the lower group, on a tie."""
    per = len(s) // groups
    of = lambda g: [float(v) for v in s[g * per: (g + 1) * per]]
    score = [sum(sorted(of(g), reverse=True)[:2]) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: (-score[g], g))[:keep]
    allowed = [e for e in range(len(s)) if e // per in best]
    return sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]


def routed_ff(W, p, m, h):
    r, out = m["router"], torch.zeros_like(h)
    for t in range(len(h)):
        s = sigmoid(W[p + "router"] @ h[t])
        for e in choose(s, r["top"], r["groups"]["count"], r["groups"]["keep"]):
            out[t] += s[e] * glu(W, f"{p}e{e}.", silu, h[t])
    return out


def run_order(cfg):
    """(layer, starts a pass of the loop) for every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, i == a) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body * loop["times"] + [(i, False) for i in range(b, n)]


MIXERS = {"attention": plain_attention, "attention_2": windowed_attention, "mamba2": mamba2}


def forward(cfg, weights, tokens, residuals=None):
    """Logits [T, vocab]; ``residuals``: a list that receives x after every layer run."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x0 = x = W["embed"][torch.tensor(tokens)]
    for i, starts in run_order(cfg):
        if starts:
            x = torch.cat([x, x0], -1) @ W["loop.in"].T
        L, p = cfg["layers"][i], f"l{i}."
        y = MIXERS[L["type"]](W, p + "mix.", L["mixer"], norm(x, W[p + "norm1"], eps), eps)
        x = x + y * W[p + "ls1"]
        if L["mlp"] is not None:
            h = norm(x, W[p + "norm2"], eps)
            y = glu(W, p + "mlp.", gelu_tanh, h) if L["mlp"]["kind"] == "dense" else routed_ff(W, p + "mlp.", L["mlp"], h)
            x = x + y * W[p + "ls2"]
        if residuals is not None:
            residuals.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, weights, seq)[-1].argmax()))
    return seq[len(prompt):]


# ---- small random models --------------------------------------------------------------------------------------------
def attention_layer(heads, kv_heads, dim, vdim, mlp, coef=0.4, every=11, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 2 * dim ** -0.5,
                      "q_temp": {"coef": coef, "every": every}}}


def window_layer(heads, kv_heads, dim, size, keep, mlp, rot=None, base=1e4, softcap=8.0, scale=None):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or 2 * dim ** -0.5,
                      "softcap": softcap, "mask": {"size": size, "keep_first": keep},
                      "rot": {"dims": dim if rot is None else rot, "base": base}}}


def mamba_layer(heads, vdim, state, mlp, groups=1, conv=4, norm_groups=1):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                      "norm_groups": norm_groups}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def config(width, vocab, layers, loop=None, eps=1e-5, logit_scale=0.7):
    """``loop``: (start, stop, times)."""
    c = {"architecture": "Movinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
         "logit_scale": logit_scale}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def shapes(cfg):
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    if cfg.get("loop"):
        out["loop.in"] = (D, 2 * D)
    for i, L in enumerate(cfg["layers"]):
        a, m, p = L["mixer"], L["mlp"], f"l{i}."
        H = a["heads"]
        out.update({p + "norm1": (D,), p + "ls1": (D,), p + "mix.o": (D, H * a["vdim"])})
        if L["type"] == "mamba2":
            inner, gn = H * a["vdim"], a["groups"] * a["state"]
            out.update({p + "mix.in": (2 * inner + 2 * gn + H, D), p + "mix.conv": (inner + 2 * gn, a["conv"]),
                        p + "mix.conv.b": (inner + 2 * gn,), p + "mix.dt_bias": (H,), p + "mix.A_log": (H,),
                        p + "mix.D": (H,), p + "mix.norm": (inner,)})
        else:
            out.update({p + "mix.q": (H * a["dim"], D), p + "mix.k": (a["kv_heads"] * a["dim"], D)})
            if L["type"] == "attention_2":
                out[p + "mix.g"] = (H * a["vdim"], D)
            else:
                out.update({p + "mix.v": (a["kv_heads"] * a["vdim"], D), p + "mix.q.b": (H * a["dim"],),
                            p + "mix.k.b": (a["kv_heads"] * a["dim"],), p + "mix.v.b": (a["kv_heads"] * a["vdim"],)})
        if m is None:
            continue
        out.update({p + "norm2": (D,), p + "ls2": (D,)})
        parts = [("mlp", m["ff"])] if m["kind"] == "dense" else \
            [(f"mlp.e{e}", m["expert"]["ff"]) for e in range(m["router"]["experts"])]
        for name, ff in parts:
            out.update({f"{p}{name}.gate": (ff, D), f"{p}{name}.up": (ff, D), f"{p}{name}.down": (D, ff)})
        if m["kind"] == "moe":
            out[p + "mlp.router"] = (m["router"]["experts"], D)
    return out


def random_weights(cfg, seed=0):
    """bfloat16 weights.  Every mechanism has a share in the logits: biases of the size of the projections, layer scales that
    differ by channel, memories of some tens of tokens beside short ones, step sizes that differ from token to token."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda shape: torch.randn(shape, generator=g)
    W = {}
    for name, shape in shapes(cfg).items():
        last = name.rsplit("mix.", 1)[-1]
        if "norm1" in name or "norm2" in name or "final" in name:
            w = 0.3 * rnd(shape)
        elif ".ls" in name:
            w = 0.7 + 0.3 * rnd(shape)
        elif last in ("q.b", "k.b", "v.b", "conv.b"):
            w = 0.6 * rnd(shape)
        elif last == "dt_bias":
            w = -1.5 + rnd(shape)
        elif last == "A_log":
            w = -1.5 + 1.2 * rnd(shape)
        elif last in ("D", "norm"):
            w = 1 + 0.3 * rnd(shape)
        elif last == "conv":
            w = rnd(shape) * shape[1] ** -0.5
        else:
            w = rnd(shape) * shape[1] ** -0.5
            if name == "embed":
                w *= shape[1] ** 0.5
        W[name] = w.to(torch.bfloat16)
    return W
