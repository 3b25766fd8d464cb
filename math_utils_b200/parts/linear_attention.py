"""Gated linear attention: a recurrent mixer whose state per head is a matrix S [dim, vdim] with a decay of its own for
every key channel.

Parameters: ``hidden_size, n_heads, dim, vdim, tau, eps`` (of the output norm).

From the mixer's input x: q = dim^(-1/2) Q x and k = K x (n_heads x dim), v = V x (n_heads x vdim); the decays, one per
head and key channel, alpha = sigmoid(A2 (A1 x) + b)^(1 / tau).  Per head and token
    S <- diag(alpha) S + k v^T,   o = S^T q.
o is brought to unit rms over vdim, multiplied by a weight of vdim entries (the same for every head) and by
silu(G x), and goes through the output matrix.  The state is float32 and lives in the sequence's cache slot; the
projections leave their product as float32 rows, which the recurrence reads as they are.
"""
from __future__ import annotations

import torch

from ..config.base import ConfigError, PartSpec
from .base import Mixer, StateCacheSpec, TensorSpec, register_part
from .linear import Linear
from .low_rank import LowRank


class GatedLinearAttention(Mixer):
    can_overwrite = True

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = self.param
        self.hidden_size, self.n_heads = int(p("hidden_size")), int(p("n_heads"))
        self.dim, self.vdim = int(p("dim")), int(p("vdim"))
        self.tau, self.eps = float(p("tau")), float(p("eps"))
        self.qk_width, self.inner = self.n_heads * self.dim, self.n_heads * self.vdim
        self.decay = LowRank(self, "decay_down", "decay_up", self.qk_width, self.hidden_size, self.dim)

    def tensor_specs(self):
        name, D = self.tensor_name, self.hidden_size
        return (TensorSpec(name("q"), (self.qk_width, D)), TensorSpec(name("k"), (self.qk_width, D)),
                TensorSpec(name("v"), (self.inner, D)), TensorSpec(name("gate"), (self.inner, D)),
                *self.decay.tensor_specs(),
                TensorSpec(name("decay_bias"), (self.qk_width,), role="vector", init="bias"),
                TensorSpec(name("norm"), (self.vdim,), role="vector", init="norm_weight"),
                TensorSpec(name("out"), (D, self.inner), init="residual_projection"))

    def cache_spec(self):
        return StateCacheSpec(self.inner * self.dim)

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        t = lambda role: tensors[self.tensor_name(role)]
        if self.dim > runtime.ops.linear_scan_max_dk():
            raise ConfigError(f"gated linear attention: keys of {self.dim} entries are more than the scan's "
                              f"{runtime.ops.linear_scan_max_dk()}")
        self.decay.bind(tensors)
        mats = [t("q"), t("k"), t("v"), t("gate"), self.decay.down]
        pad = -sum(m.shape[0] for m in mats) % 8
        if pad:                                         # whole 16-byte pieces a row
            mats.append(torch.zeros((pad, self.hidden_size), dtype=mats[0].dtype, device=mats[0].device))
        self.columns = tuple(m.shape[0] for m in mats)
        self.proj = Linear(torch.cat(mats, dim=0).contiguous(), None, runtime)
        self.out = Linear(t("out"), None, runtime)
        self.decay_bias = t("decay_bias")
        self.norm_weight = t("norm").repeat(self.n_heads).contiguous()       # the same weight for every head

    def forward(self, h, residual, ctx, cache, owns_cache: bool, accumulate: bool = True) -> None:
        ops, T, H = self.runtime.ops, ctx.n_tokens, self.n_heads
        if not owns_cache:
            raise ConfigError("gated linear attention keeps its own state: it cannot read another layer's")
        u, q, k, v, gate = ctx.buffer("linear.proj", (T, sum(self.columns)), torch.float32, columns=self.columns)[:5]
        self.proj(h, out=u)
        decay = ctx.buffer("linear.decay", (T, self.qk_width), torch.float32)
        low_at = 2 * self.qk_width + 2 * self.inner
        ops.low_rank(u, self.decay.up.dtype, self.decay.part(ops, low_at, decay, bias=self.decay_bias, fn="sigmoid_power",
                                                             power=1.0 / self.tau))
        o = ctx.buffer("linear.o", (T, self.inner), torch.float32)
        ops.linear_scan(q, k, v, decay, H, self.dim, self.vdim, self.dim ** -0.5, ctx.seq_first, ctx.seq_slots, cache.values,
                        0, o)
        ctx.note("scan", o)
        gated = ctx.buffer("linear.gated", (T, self.inner), self.runtime.dtype)
        ops.gated_group_norm(o, gate, self.norm_weight, H, self.eps, gated, gate_after=True)
        ctx.note("attn", gated)
        self.out(gated, residual=residual if accumulate else None, out=residual)


register_part("mixer", "gated_linear_attention", GatedLinearAttention, replace=True)
