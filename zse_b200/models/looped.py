"""Hybrid decoders with norms before the sublayers, layer scales, and a range of layers that runs several times (Movinex).

Mixers, feed-forwards, cache, state and pass layout are those of ``models.hybrid``; the residual x is fp32.  A layer run:

    x     = x + scale * y of the sublayer before;  h = norm(x) * (1 + w1)                                       1 kernel
    y     = mixer(h)                                                          (split-K planes, added by the next kernel)
    x     = x + scale1 * y;  h = norm(x) * (1 + w2)                                                             1 kernel
    y     = ff(h)                                                           (planes, or the experts' rows; scale2 is due)

Ahead of the first layer of every pass of the loop x becomes W [x; x0], x0 the embeddings of the pass's tokens: the kernel
that completes x writes it beside x0, and the product's planes replace the residual in the next layer's first kernel.
"""
from __future__ import annotations

import torch

from ..format.config import DenseSpec, HeadsSpec, StateSpaceSpec
from ..format.loader import ZSELoader
from .hybrid import HybridLayer, HybridModel, HybridStepBuffers


class LoopedModel(HybridModel):
    kernel_group = "looped"

    # ---- loading --------------------------------------------------------------------------------------
    def _load(self, loader: ZSELoader, progress=None) -> None:
        c, ops = self.config, self.ops
        r = self._open(loader)
        H = c.hidden_size
        self.embed = r.get("embed")
        self.norm = r.get("final.norm")
        self.norm_offset = c.norm_weight_offset
        self.loop_in = r.linear("loop.in") if c.loop else None
        for i in range(c.num_layers):
            p, s, m = f"l{i}.", c.mixer_spec(i), c.ff_spec(i)
            load = self._load_heads if isinstance(s, HeadsSpec) else self._load_space
            L = load(r, p, s, m, H)
            L.scale1 = r.get(p + "ls1")
            if m is not None:
                L.norm2, L.scale2 = r.get(p + "norm2"), r.get(p + "ls2")
            if isinstance(m, DenseSpec):
                L.up_w = ops.glu_linear(r.tensor(p + "mlp.gate"), r.tensor(p + "mlp.up"), self.act_dtype)
                self._count(L.up_w.data)
                L.down_w = r.linear(p + "mlp.down")
            elif m is not None:
                self._load_experts(r, L, p, m, H)
            self.layers.append(L)
            if progress:
                progress(i + 1, c.num_layers)
        self.lm_head = r.linear("head")
        r.release()
        self.logit_scale = float(c.logit_scale if c.logit_scale is not None else 1.0)
        self._plan_runs()

    def _load_heads(self, r, p: str, s: HeadsSpec, m, H: int) -> HybridLayer:
        cols = {"q": 0, "k": s.k_col}
        if not s.k_as_v:
            cols["v"] = s.v_col
        parts = [(at, r.tensor(f"{p}mix.{name}")) for name, at in cols.items()]
        if s.gated:
            parts.append((s.gate_col, r.tensor(p + "mix.g")))
        L = HybridLayer(s, m, r.get(p + "norm1"), self.ops.dense_linear(r.stack(parts, s.in_width, H)), r.linear(p + "mix.o"))
        if s.bias:
            L.bias = r.stack([(at, r.tensor(f"{p}mix.{name}.b")[:, None]) for name, at in cols.items()], s.in_width, 1).view(-1)
        L.freqs = self.ops.rotation(s.rot_dims, s.rot_base)
        return L

    def _load_space(self, r, p: str, s: StateSpaceSpec, m, H: int) -> HybridLayer:
        gn = s.groups * s.state
        parts, conv, at = [], [], 0          # sections of W_in, and of the channels, that lie apart in the padded layout
        for rows, col in ((s.inner, 0), (s.inner, s.x_col), (gn, s.x_col + s.b_at), (gn, s.x_col + s.c_at),
                          (s.heads, s.dt_col)):
            parts.append((col, at, rows))
            at += rows
        w = r.tensor(p + "mix.in")
        w_in = r.stack([(col, w[a: a + n]) for col, a, n in parts], s.in_width, H)
        L = HybridLayer(s, m, r.get(p + "norm1"), self.ops.dense_linear(w_in), r.linear(p + "mix.o"))
        f32 = lambda name: r.tensor(p + "mix." + name).float().contiguous()
        taps, bias = f32("conv").T, f32("conv.b")
        L.conv_w = torch.zeros(s.conv, s.conv_width, device=taps.device)
        L.conv_b = torch.zeros(s.conv_width, device=taps.device)
        for col, a, n in parts[1:4]:
            a, col = a - s.inner, col - s.x_col
            L.conv_w[:, col: col + n], L.conv_b[col: col + n] = taps[:, a: a + n], bias[a: a + n]
        L.dt_bias, L.D, L.neg_a = f32("dt_bias").clone(), f32("D").clone(), -torch.exp(f32("A_log"))
        L.out_norm = r.get(p + "mix.norm")
        return L

    # ---- buffers --------------------------------------------------------------------------------------
    def make_buffers(self, *args, **kw) -> HybridStepBuffers:
        b = super().make_buffers(*args, **kw)
        H = self.config.hidden_size
        if self.loop_in is not None:
            b.looped = torch.zeros(b.max_tokens, 2 * H, dtype=self.act_dtype, device=self.device)      # [x | embedding]
        return b

    # ---- forward --------------------------------------------------------------------------------------
    def forward(self, b: HybridStepBuffers, kv: torch.Tensor, M: int, mode: str, num_seqs: int, max_q_len: int = 1,
                n_logit_rows: int = 0, attn_splits: int = 1) -> None:
        ops, eps, H = self.ops, self.config.rms_norm_eps, self.config.hidden_size
        p = self._pass(b, kv, M, mode, num_seqs, max_q_len, attn_splits)
        ops.embedding(self.embed, b.ids, b.residual, M, copy=b.looped[:, H:] if self.loop_in is not None else None)
        due = {}                             # the sublayer's result that x still lacks

        def complete(weight, out, planes=0, slots=None, **how):
            ops.add_norm(b.residual, p.partials, planes, slots, weight, out, M, eps, offset=self.norm_offset, **how)

        for run in self.runs:
            L = run.layer
            if run.enters_loop:
                complete(None, b.looped[:, :H], **due)
                due = {"planes": ops.linear_partial(self.loop_in, b.looped, M, p.partials), "replace": True}
            complete(L.norm1, b.xnorm, **due)
            due = {"planes": self._mix(b, p, run), "scale": L.scale1}
            if L.ff is not None:
                complete(L.norm2, b.xnorm, **due)
                planes, slots = self._feed(b, p, L)
                due = {"planes": planes, "slots": slots, "scale": L.scale2}
        complete(self.norm, b.xnorm, **due)
        if n_logit_rows:
            self._logits(b, n_logit_rows)
            ops.logits_finish(b.logits, n_logit_rows, self.logit_scale, 0.0)
