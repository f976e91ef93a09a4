"""Decoders whose layers run two mixers and a feed-forward side by side (Vobisun): windowed attention with block means and gated
linear attention read one input, the feed-forward reads the same norm, and all three results are added to the residual at once.

Cache, state, mixers and pass layout are those of ``models.hybrid``; the residual x is fp32.  A layer run:

    x      = x + the result of the run before;  h = norm(x) * w;  g = h + conv(h)          1 kernel (2 in passes of long chunks)
    p      = g W_in            both mixers' projections in one product
    a | r  = the mixers' results, scaled and gated, side by side in one row                (see models.hybrid)
    f      = silu(h W_gate) * (h W_up)                                                     behind them in the same row
    y      = [a | r | f] [W_left; W_right; W_down]                                         one product, split-K planes

A loop's passes follow one another without anything between them; each has its own cache and state.
"""
from __future__ import annotations

import torch

from ..format.loader import ZSELoader
from .hybrid import HybridLayer, HybridModel, HybridStepBuffers


class TwinModel(HybridModel):
    kernel_group = "twin"

    # ---- loading --------------------------------------------------------------------------------------
    def _load(self, loader: ZSELoader, progress=None) -> None:
        c, ops = self.config, self.ops
        r = self._open(loader)
        H = c.hidden_size
        self.embed = r.get("embed")
        self.embed_scale = float(c.embed_multiplier if c.embed_multiplier is not None else 1.0)
        self.norm = r.get("final.norm")
        for i in range(c.num_layers):
            p, s, m = f"l{i}.", c.mixer_spec(i), c.ff_spec(i)
            a, g = s.left, s.right
            t = lambda name: r.tensor(p + name)
            f32 = lambda name: t(name).float().clone(memory_format=torch.contiguous_format)
            cols = {"q": 0, "k": a.k_col, "v": a.v_col}
            parts = [(at, t("mix.left." + n)) for n, at in cols.items()] + [(a.gate_col, t("mix.left.g"))]
            parts += [(at, t("mix.right." + n)) for n, at in (("q", g.col), ("k", g.k_col), ("v", g.v_col),
                                                              ("g", g.gate_col), ("a1", g.rank_col))]
            L = HybridLayer(s, m, r.get(p + "norm1"), ops.dense_linear(r.stack(parts, s.in_width, H)), None)
            L.bias = r.stack([(at, t(f"mix.left.{n}.b")[:, None]) for n, at in cols.items()], a.gate_col, 1).view(-1)
            L.q_norm, L.k_norm = r.get(p + "mix.left.q.norm"), r.get(p + "mix.left.k.norm")
            L.temp, L.sink = f32("mix.left.temp"), f32("mix.left.sink")
            L.freqs = ops.rotation(a.rot_dims, a.rot_base, a.rot_factor)
            L.decay_w, L.decay_b = f32("mix.right.a2"), f32("mix.right.a2.b")
            L.head_norm = r.get(p + "mix.right.norm")
            L.conv_w = f32("canon1").T.contiguous()
            outs = [(0, t("mix.left.o")), (s.right_at, t("mix.right.o"))]
            if m is not None:
                L.up_w = ops.glu_linear(t("mlp.gate"), t("mlp.up"), self.act_dtype)
                self._count(L.up_w.data)
                outs.append((s.out_width, t("mlp.down")))
            w = torch.zeros(H, L.out_width, dtype=self.act_dtype, device=self.device)
            for at, o in outs:
                w[:, at: at + o.shape[1]] = o
            L.o = ops.dense_linear(r.keep(w))
            self.layers.append(L)
            if progress:
                progress(i + 1, c.num_layers)
        self.lm_head = r.linear("head")
        r.release()
        self._plan_runs()

    # ---- buffers --------------------------------------------------------------------------------------
    def make_buffers(self, *args, **kw) -> HybridStepBuffers:
        b = super().make_buffers(*args, **kw)
        b.xconv = torch.zeros(b.max_tokens, self.config.hidden_size, dtype=self.act_dtype, device=self.device)
        return b

    # ---- forward --------------------------------------------------------------------------------------
    def forward(self, b: HybridStepBuffers, kv: torch.Tensor, M: int, mode: str, num_seqs: int, max_q_len: int = 1,
                n_logit_rows: int = 0, attn_splits: int = 1) -> None:
        ops, eps = self.ops, self.config.rms_norm_eps
        p = self._pass(b, kv, M, mode, num_seqs, max_q_len, attn_splits)
        ops.embedding(self.embed, b.ids, b.residual, M, self.embed_scale)
        planes = 0
        for run in self.runs:
            L, s = run.layer, run.layer.spec
            ops.add_norm_conv(b.residual, p.partials, planes, L.norm1, b.xnorm, L.conv_w, b.xconv, self.states.rows,
                              run.inputs_at, b.state_rows, p.row_seq, p.cu_q, M, num_seqs, eps)
            self._mix_both(b, p, run, b.xconv)
            out = b.out_views[L.out_width]
            if L.ff is not None:
                ops.linear_glu(L.up_w, b.xnorm, M, out[:, s.out_width: s.out_width + L.ff.ff], L.ff.activation, b.glu)
            planes = ops.linear_partial(L.o, out, M, p.partials)
        ops.add_norm(b.residual, p.partials, planes, None, self.norm, b.xnorm, M, eps)
        if n_logit_rows:
            self._logits(b, n_logit_rows)
