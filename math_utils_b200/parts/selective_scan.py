"""The selective scan of Mamba (Gu, Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces"): a
state-space mixer whose decay differs by channel and by state entry.

Parameters: ``hidden_size, inner`` (channels), ``state`` (N, entries per channel), ``dt_rank``, ``conv`` (taps).

One input product gives, per token, [x: inner | z: inner].  x passes a causal convolution per channel (zeros before a
sequence's start, the last tap on the current token, a bias) and silu.  A second product of that x gives
[dt: dt_rank | B: N | C: N]; dt <- softplus(W_dt dt + bias), one per channel.  With A = -exp(A_log) [inner, N] and S
[inner, N] starting at zero:
    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,    y_c = sum_n S[c, n] C_n + D_c x_c.
y * silu(z) goes through the output matrix.  A sequence's state (the convolution's last taps - 1 inputs and S) is float32
and lives in its cache slot; dt, B, C, decays and the recurrence are float32 whatever the compute dtype.
"""
from __future__ import annotations

import math

import torch

from ..config.base import ConfigError, PartSpec
from .base import Mixer, StateCacheSpec, TensorSpec, register_part
from .linear import Linear


class SelectiveScanMixer(Mixer):
    can_overwrite = True

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = self.param
        self.hidden_size, self.inner, self.state = int(p("hidden_size")), int(p("inner")), int(p("state"))
        self.dt_rank, self.taps = int(p("dt_rank")), int(p("conv"))
        self.tail_values = (self.taps - 1) * self.inner
        # the second product's row: dt padded to whole tensor-core steps, B and C to whole 16-byte pieces
        self.rank = self.dt_rank + -self.dt_rank % 16
        self.n4 = self.state + -self.state % 4
        self.b_at, self.c_at = self.rank, self.rank + self.n4
        self.low_width = self.rank + 2 * self.n4
        self.low_width += -self.low_width % 8

    def tensor_specs(self):
        name, C, N, R = self.tensor_name, self.inner, self.state, self.dt_rank
        return (TensorSpec(name("in"), (2 * C, self.hidden_size)),
                TensorSpec(name("conv"), (C, self.taps), role="vector", init="conv"),
                TensorSpec(name("conv_bias"), (C,), role="vector", init="bias"),
                TensorSpec(name("x"), (R + 2 * N, C)),
                TensorSpec(name("dt"), (C, R)),
                TensorSpec(name("dt_bias"), (C,), role="vector", init="bias"),
                TensorSpec(name("A_log"), (C, N), role="vector", init="bias"),
                TensorSpec(name("D"), (C,), role="vector", init="norm_weight"),
                TensorSpec(name("out"), (self.hidden_size, C), init="residual_projection"))

    def cache_spec(self):
        values = self.tail_values + self.inner * self.state
        return StateCacheSpec(values + -values % 4)                          # slots a whole number of 16-byte pieces apart

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        t = lambda role: tensors[self.tensor_name(role)]
        if self.state > runtime.ops.selective_scan_max_state():
            raise ConfigError(f"selective scan: {self.state} state entries per channel are more than the kernel's "
                              f"{runtime.ops.selective_scan_max_state()}")
        R, N = self.dt_rank, self.state
        self.proj = Linear(t("in"), None, runtime)
        x = t("x")
        low = torch.zeros((self.low_width, self.inner), dtype=x.dtype, device=x.device)
        low[:R], low[self.b_at:self.b_at + N], low[self.c_at:self.c_at + N] = x[:R], x[R:R + N], x[R + N:]
        self.low = Linear(low, None, runtime)
        self.dt_up = torch.nn.functional.pad(t("dt"), (0, self.rank - R)).contiguous()
        self.out = Linear(t("out"), None, runtime)
        self.conv_weight, self.conv_bias, self.dt_bias, self.skip = t("conv"), t("conv_bias"), t("dt_bias"), t("D")
        # exp(dt A) = 2^(dt A log2 e)
        self.rates = (-torch.exp(t("A_log").double()) / math.log(2.0)).float().contiguous()

    def forward(self, h, residual, ctx, cache, owns_cache: bool, accumulate: bool = True) -> None:
        ops, dtype = self.runtime.ops, self.runtime.dtype
        T, C = ctx.n_tokens, self.inner
        if not owns_cache:
            raise ConfigError("a selective scan keeps its own state: it cannot read another layer's")
        u, x_in, z = ctx.buffer("selective.proj", (T, 2 * C), dtype, columns=(C, C))
        self.proj(h, out=u)
        x = ctx.buffer("selective.x", (T, C), dtype)
        ops.ssd_conv(x_in, self.conv_weight, self.conv_bias, ctx.tok_seq, ctx.seq_first, ctx.seq_slots, cache.values,
                     ctx.is_decode, x)
        low = ctx.buffer("selective.low", (T, self.low_width), torch.float32)
        self.low(x, out=low)
        dt = ctx.buffer("selective.dt", (T, C), torch.float32)
        ops.low_rank(low, self.dt_up.dtype, ops.low_rank_part(self.dt_up, 0, dt, bias=self.dt_bias, fn="softplus"))
        y = ctx.buffer("selective.y", (T, C), dtype)
        ops.selective_scan(x, z, dt, low, self.b_at, self.c_at, self.rates, self.skip, ctx.seq_first, ctx.seq_slots,
                           cache.values, self.tail_values, y)
        ctx.note("scan", y)
        self.out(y, residual=residual if accumulate else None, out=residual)


register_part("mixer", "selective_scan", SelectiveScanMixer, replace=True)
