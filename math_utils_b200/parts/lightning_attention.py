"""Lightning attention: linear attention whose state per head, a matrix S [dim, vdim], decays by one constant per head.

Parameters: ``hidden_size, n_heads, dim, vdim, decay`` (one number per head), ``eps`` (of the output norm).

From the mixer's input x: q = silu(Q x), k = silu(K x) (n_heads x dim), v = silu(V x) (n_heads x vdim).  Per head and token
    S <- decay_h S + k v^T,   o = S^T q.
The heads' o, side by side, is brought to unit rms over all of them, multiplied by a weight of that size and by
sigmoid(G x), and goes through the output matrix.  The state is float32 and lives in the sequence's cache slot.

Prompt steps in bfloat16 go chunk by chunk over tensor cores (``ops.lightning_prompt``), all chunks at once but for the
states between them; single tokens, short runs and the 32-bit path go token by token through the linear scan
(``ops.linear_scan``, float32 rows).  Both apply silu to the rows as they stage them.
"""
from __future__ import annotations

import torch

from ..config.base import ConfigError, PartSpec
from .base import Mixer, StateCacheSpec, TensorSpec, register_part
from .linear import Linear


class LightningAttention(Mixer):
    can_overwrite = True

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = self.param
        self.hidden_size, self.n_heads = int(p("hidden_size")), int(p("n_heads"))
        self.dim, self.vdim, self.eps = int(p("dim")), int(p("vdim")), float(p("eps"))
        self.decay = tuple(float(x) for x in p("decay"))
        if len(self.decay) != self.n_heads:
            raise ConfigError(f"lightning attention: {len(self.decay)} decays for {self.n_heads} heads")
        self.qk_width, self.inner = self.n_heads * self.dim, self.n_heads * self.vdim

    def tensor_specs(self):
        name, D = self.tensor_name, self.hidden_size
        return (TensorSpec(name("q"), (self.qk_width, D)), TensorSpec(name("k"), (self.qk_width, D)),
                TensorSpec(name("v"), (self.inner, D)), TensorSpec(name("gate"), (self.inner, D)),
                TensorSpec(name("norm"), (self.inner,), role="vector", init="norm_weight"),
                TensorSpec(name("out"), (D, self.inner), init="residual_projection"))

    def cache_spec(self):
        return StateCacheSpec(self.inner * self.dim)

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        t = lambda role: tensors[self.tensor_name(role)]
        if self.dim > runtime.ops.linear_scan_max_dk():
            raise ConfigError(f"lightning attention: keys of {self.dim} entries are more than the scan's "
                              f"{runtime.ops.linear_scan_max_dk()}")
        mats = [t("q"), t("k"), t("v"), t("gate")]
        pad = -sum(m.shape[0] for m in mats) % 8
        if pad:                                         # whole 16-byte pieces a row
            mats.append(torch.zeros((pad, self.hidden_size), dtype=mats[0].dtype, device=mats[0].device))
        self.columns = tuple(m.shape[0] for m in mats)
        self.proj = Linear(torch.cat(mats, dim=0).contiguous(), None, runtime)
        self.out = Linear(t("out"), None, runtime)
        self.norm_weight = t("norm")
        # (decay, take, -, -) per head, the same for every token
        self.chunked = runtime.dtype == torch.bfloat16 and runtime.ops.lightning_prompt_ok(self.dim, self.vdim)
        exponents = torch.arange(65, dtype=torch.float64)
        self.powers = (torch.tensor(self.decay, dtype=torch.float64)[:, None] ** exponents).float().contiguous().to(runtime.device)
        self.gates = torch.tensor([[[d, 1.0, 0.0, 0.0] for d in self.decay]], dtype=torch.float32, device=runtime.device)

    CHUNKED_TOKENS = 24              # tokens a sequence brings on average from which on the chunked form pays

    def forward(self, h, residual, ctx, cache, owns_cache: bool, accumulate: bool = True) -> None:
        ops, T, H = self.runtime.ops, ctx.n_tokens, self.n_heads
        if not owns_cache:
            raise ConfigError("lightning attention keeps its own state: it cannot read another layer's")
        chunked = self.chunked and ctx.q_tiles is not None and T >= self.CHUNKED_TOKENS * ctx.n_seqs
        u, q, k, v, gate = ctx.buffer("lightning.proj", (T, sum(self.columns)),
                                      self.runtime.dtype if chunked else torch.float32, columns=self.columns)[:5]
        self.proj(h, out=u)
        o = ctx.buffer("lightning.o", (T, self.inner), torch.float32)
        if chunked:
            ops.lightning_prompt(q, k, v, self.powers, H, self.dim, self.vdim, ctx.q_tiles, ctx.tok_seq, ctx.seq_first,
                                 ctx.seq_slots, cache.values, 0, o)
        else:
            ops.linear_scan(q, k, v, self.gates, H, self.dim, self.vdim, 1.0, ctx.seq_first, ctx.seq_slots, cache.values, 0, o,
                            silu_rows=True)
        ctx.note("scan", o)
        gated = ctx.buffer("lightning.gated", (T, self.inner), self.runtime.dtype)
        ops.gated_group_norm(o, gate, self.norm_weight, 1, self.eps, gated, gate_after=True, sigmoid=True)
        ctx.note("attn", gated)
        self.out(gated, residual=residual if accumulate else None, out=residual)


register_part("mixer", "lightning_attention", LightningAttention, replace=True)
