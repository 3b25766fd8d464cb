"""The matrix memory of xLSTM (mLSTM; Beck, Pöppel, Spanring, Auer, Prudnikova, Kopp, Klambauer, Brandstetter,
Hochreiter, "xLSTM: Extended Long Short-Term Memory"): a recurrent mixer with a matrix state S [dim, vdim] and a
normalizer n [dim] per head, and exponential gates.

Parameters: ``hidden_size, n_heads, dim, vdim, gate_cap, eps`` (of the output norm).

From the mixer's input x: q = dim^(-1/2) Q x and k = K x (n_heads x dim), v = V x (n_heads x vdim); one log input gate
and one log forget gate per head,
    i = cap tanh((I x + b_i) / cap),   f = log sigmoid(cap tanh((F x + b_f) / cap)).
With a running maximum m that starts at zero, m <- max(f + m, i), the state is kept relative to exp(m):
    S <- exp(f + m_before - m) S + exp(i - m) k v^T,   n the same with k alone,
    o = S^T q / (max(|n . q|, exp(-m)) + 1e-6).
Each head's o is brought to unit rms over vdim; the heads side by side are multiplied by a weight of all heads' size
and by sigmoid(G x), and go through the output matrix.  S, n and m are float32 and live in the sequence's cache slot;
gates and recurrence are float32, and so are the rows the projections leave for them.
"""
from __future__ import annotations

import torch

from ..config.base import ConfigError, PartSpec
from .base import Mixer, StateCacheSpec, TensorSpec, register_part
from .linear import Linear


class MatrixLstm(Mixer):
    can_overwrite = True

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = self.param
        self.hidden_size, self.n_heads = int(p("hidden_size")), int(p("n_heads"))
        self.dim, self.vdim = int(p("dim")), int(p("vdim"))
        self.gate_cap, self.eps = float(p("gate_cap")), float(p("eps"))
        self.qk_width, self.inner = self.n_heads * self.dim, self.n_heads * self.vdim
        self.m_offset = self.qk_width * (self.vdim + 1)                      # behind S and n

    def tensor_specs(self):
        name, D, H = self.tensor_name, self.hidden_size, self.n_heads
        return (TensorSpec(name("q"), (self.qk_width, D)), TensorSpec(name("k"), (self.qk_width, D)),
                TensorSpec(name("v"), (self.inner, D)), TensorSpec(name("gate"), (self.inner, D)),
                TensorSpec(name("i"), (H, D)), TensorSpec(name("i_bias"), (H,), role="vector", init="bias"),
                TensorSpec(name("f"), (H, D)), TensorSpec(name("f_bias"), (H,), role="vector", init="bias"),
                TensorSpec(name("norm"), (self.inner,), role="vector", init="norm_weight"),
                TensorSpec(name("out"), (D, self.inner), init="residual_projection"))

    def cache_spec(self):
        values = self.m_offset + self.n_heads
        return StateCacheSpec(values + -values % 4)                          # slots a whole number of 16-byte pieces apart

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        t = lambda role: tensors[self.tensor_name(role)]
        if self.dim > runtime.ops.linear_scan_max_dk():
            raise ConfigError(f"matrix LSTM: keys of {self.dim} entries are more than the scan's "
                              f"{runtime.ops.linear_scan_max_dk()}")
        mats = [t(r) for r in ("q", "k", "v", "gate", "i", "f")]
        pad = -sum(m.shape[0] for m in mats) % 8
        if pad:                                         # whole 16-byte pieces a row
            mats.append(torch.zeros((pad, self.hidden_size), dtype=mats[0].dtype, device=mats[0].device))
        self.columns = tuple(m.shape[0] for m in mats)
        self.proj = Linear(torch.cat(mats, dim=0).contiguous(), None, runtime)
        self.out = Linear(t("out"), None, runtime)
        self.i_bias, self.f_bias, self.norm_weight = t("i_bias"), t("f_bias"), t("norm")

    def forward(self, h, residual, ctx, cache, owns_cache: bool, accumulate: bool = True) -> None:
        ops, T, H = self.runtime.ops, ctx.n_tokens, self.n_heads
        if not owns_cache:
            raise ConfigError("a matrix LSTM keeps its own state: it cannot read another layer's")
        u, q, k, v, gate, i_raw, f_raw = ctx.buffer("mlstm.proj", (T, sum(self.columns)), torch.float32,
                                                    columns=self.columns)[:7]
        self.proj(h, out=u)
        gates = ctx.buffer("mlstm.gates", (T, H, 4), torch.float32)
        ops.exp_gates(i_raw, f_raw, self.i_bias, self.f_bias, self.gate_cap, ctx.seq_first, ctx.seq_slots, cache.values,
                      self.m_offset, gates)
        o = ctx.buffer("mlstm.o", (T, self.inner), torch.float32)
        read = ctx.buffer("mlstm.normalizer", (T, H), torch.float32)
        ops.linear_scan(q, k, v, gates, H, self.dim, self.vdim, self.dim ** -0.5, ctx.seq_first, ctx.seq_slots, cache.values,
                        0, o, norm_out=read)
        ctx.note("scan", o)
        gated = ctx.buffer("mlstm.gated", (T, self.inner), self.runtime.dtype)
        ops.gated_group_norm(o, gate, self.norm_weight, H, self.eps, gated, gate_after=True, sigmoid=True, den=read,
                             den_floor=gates[:, :, 2])
        ctx.note("attn", gated)
        self.out(gated, residual=residual if accumulate else None, out=residual)


register_part("mixer", "matrix_lstm", MatrixLstm, replace=True)
