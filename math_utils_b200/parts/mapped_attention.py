"""Attention with normed, rotated queries and keys, one or two score maps per head, and values of their own size.

Parameters: ``hidden_size, n_heads, n_kv_heads`` (query head h reads key/value head h // (n_heads / n_kv_heads)),
``dim`` (query/key entries of ONE score map), ``vdim`` (value entries per head), ``maps`` (1, or 2 for differential
attention), ``softmax_scale``, ``window`` (0: every earlier position; w: a token sees itself and the w - 1 before
it), ``cache_window`` (what the cache must keep: the largest window of the layers that read it, 0 for all), ``eps``,
``rot`` = {base, dims, scaling?}, ``bias`` (the four projections have biases), ``own_kv`` (false for a layer that
reads the cached keys and values of an earlier layer and has no key/value tensors of its own) and, with two maps,
``diff``.

Per head and map the queries and keys are brought to unit rms over ``dim`` and multiplied by a weight shared by
all heads and maps, then their first ``rot.dims`` entries are rotated (entry i with entry i + dims/2).  With two
maps each map is a softmax attention of its own over the SAME values, and the head's result is
a1 - lambda a2 with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number for the layer; that result is
brought to unit rms over its vdim entries (no weight) and multiplied by 1 - diff.  The cache keeps one row per
position: the kv heads' keys (after norm and rotation), then their values.

Switches for other designs, each with its constants: ``qk_norm`` false leaves queries and keys as the projections
give them (no ``q_norm`` / ``k_norm`` tensors); ``rot_layout`` ``"pairs"`` turns entry 2i with entry 2i + 1 instead
of entry i with entry i + dims/2; ``chunk`` c > 0 replaces the window by chunks of c positions counted from the
sequence's position 0 (position p sees p - p % c .. p; the cache keeps everything); ``head_gate`` multiplies head
h's result by sigmoid(G x)_h, one number per head from the mixer's own input (tensor ``gate`` [heads, hidden], no
bias), before the output projection; ``qk_norm`` ``"unit"`` norms queries and keys without a weight; ``rot`` None
rotates nothing; ``key_values`` makes the projected keys, as they are before their norm, the values too (no ``v``
tensor; vdim equals dim); ``slopes``: ``"geometric"`` takes slope_h * distance off every score,
slope_h = 2^(-8 (h + 1) / n_heads); ``keep`` n > 0, with a window, leaves the sequence's first n positions in sight of
every later token (the cache keeps them); ``softcap`` c > 0 makes a scaled score s into c tanh(s / c); ``sink`` counts one
more key of score zero, without a value, in the softmax's denominator; ``entry_gate`` multiplies the heads side by side by
sigmoid(G x) entry by entry (tensor ``gate`` [heads * vdim, hidden], no bias) before the output projection.  Where the
keys are the values and go to the cache as they are (``key_values`` without norm and rotation) a cached row holds them
once.  ``cache_window`` beside ``chunk``: the cache gives back pages that no later token's chunk can reach.
"""
from __future__ import annotations

import torch

from ..config.base import ConfigError, PartSpec
from .base import Mixer, RowCacheSpec, TensorSpec, register_part
from .linear import Linear
from .position import rotary_frequencies


class MappedAttention(Mixer):
    can_overwrite = True

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = self.param
        self.hidden_size, self.n_heads = int(p("hidden_size")), int(p("n_heads"))
        self.n_kv_heads = int(p("n_kv_heads", self.n_heads))
        self.dim, self.vdim, self.maps = int(p("dim")), int(p("vdim")), int(p("maps", 1))
        self.scale, self.eps = float(p("softmax_scale")), float(p("eps"))
        self.window = int(p("window", 0))
        self.cache_window = int(p("cache_window", self.window))
        self.own_kv = bool(p("own_kv", True))
        self.bias = bool(p("bias", False))
        self.diff = float(p("diff", 0.0))
        self.qk_norm = p("qk_norm", True)
        self.key_values = bool(p("key_values", False))
        self.slopes = p("slopes", None)
        self.keep = int(p("keep", 0))
        self.softcap, self.sink = float(p("softcap", 0.0) or 0.0), bool(p("sink", False))
        self.entry_gate = bool(p("entry_gate", False))
        if self.qk_norm not in (True, False, "unit"):
            raise ConfigError(f"mapped attention: qk_norm '{self.qk_norm}' is not true, false or 'unit'")
        if self.key_values and (self.dim != self.vdim or self.maps != 1 or not self.own_kv):
            raise ConfigError("mapped attention: keys that are the values too have the values' size and one score map")
        if self.slopes not in (None, "geometric"):
            raise ConfigError(f"mapped attention: slopes '{self.slopes}' is not 'geometric'")
        if self.keep and (not self.window or self.cache_window != self.window):
            raise ConfigError("mapped attention: kept positions go with a window of the layer's own")
        self.rot_layout = p("rot_layout", "half")
        self.chunk = int(p("chunk", 0))
        self.head_gate = bool(p("head_gate", False))
        if self.rot_layout not in ("half", "pairs"):
            raise ConfigError(f"mapped attention: rot_layout '{self.rot_layout}' is not 'half' or 'pairs'")
        if self.chunk < 0 or (self.chunk and self.window):
            raise ConfigError("mapped attention: chunks of positions and a window exclude one another")
        if self.maps not in (1, 2):
            raise ConfigError(f"mapped attention has one or two score maps, got {self.maps}")
        if self.n_heads % self.n_kv_heads:
            raise ConfigError(f"mapped attention: {self.n_heads} heads do not split over {self.n_kv_heads} kv heads")
        if self.chunk and self.cache_window and self.cache_window < self.chunk:
            raise ConfigError("mapped attention: the cache keeps fewer positions than a chunk has")
        if self.head_gate and self.entry_gate:
            raise ConfigError("mapped attention: a gate per head and one per entry exclude one another")
        if self.window and self.cache_window and self.cache_window < self.window:
            raise ConfigError("mapped attention: the cache keeps fewer positions than the window sees")
        rot = p("rot") or {"dims": 0, "base": 1.0}
        self.rot_dims = int(rot["dims"])
        if self.rot_dims > self.dim or self.rot_dims % 2:
            raise ConfigError(f"mapped attention: {self.rot_dims} rotated entries do not fit a map of {self.dim}")
        self.freqs, self.magnitude = rotary_frequencies(self.rot_dims, float(rot["base"]), rot.get("scaling"))
        self.q_width = self.n_heads * self.maps * self.dim
        self.k_width = self.n_kv_heads * self.maps * self.dim
        self.v_width = self.n_kv_heads * self.vdim
        # cached keys that are the very values are kept once
        self.shared_rows = self.key_values and self.qk_norm is False and self.rot_dims == 0
        self.gate_width = self.n_heads * (1 if self.head_gate else self.vdim if self.entry_gate else 0)

    def tensor_specs(self):
        D, name = self.hidden_size, self.tensor_name
        specs = [TensorSpec(name("q"), (self.q_width, D))]
        if self.qk_norm is True:
            specs.append(TensorSpec(name("q_norm"), (self.dim,), role="vector", init="norm_weight"))
        widths = [("q_bias", self.q_width)]
        if self.own_kv:
            specs.append(TensorSpec(name("k"), (self.k_width, D)))
            if not self.key_values:
                specs.append(TensorSpec(name("v"), (self.v_width, D)))
            if self.qk_norm is True:
                specs.append(TensorSpec(name("k_norm"), (self.dim,), role="vector", init="norm_weight"))
            widths += [("k_bias", self.k_width)] + ([] if self.key_values else [("v_bias", self.v_width)])
        if self.gate_width:
            specs.append(TensorSpec(name("gate"), (self.gate_width, D)))
        specs.append(TensorSpec(name("out"), (D, self.n_heads * self.vdim), init="residual_projection"))
        widths.append(("out_bias", D))
        if self.bias:
            specs += [TensorSpec(name(role), (n,), role="vector", init="bias") for role, n in widths]
        if self.maps == 2:
            specs += [TensorSpec(name(role), (self.dim,), role="vector", init="bias") for role in ("lq1", "lk1", "lq2", "lk2")]
        return specs

    def cache_spec(self):
        return RowCacheSpec(self.k_width + (0 if self.shared_rows else self.v_width), self.cache_window, self.keep)

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        t = lambda role: tensors[self.tensor_name(role)]
        roles = ["q"] + ((["k"] if self.key_values else ["k", "v"]) if self.own_kv else [])
        mats = [t(r) for r in roles]
        biases = [t(r + "_bias") for r in roles] if self.bias else None
        self.gate_at = None
        if self.gate_width:
            # the gates ride in the same product, after q | k | v; rows of zeros keep the stacked row a whole
            # number of 16-byte pieces
            self.gate_at = len(mats) + 1
            pad = -(sum(m.shape[0] for m in mats) + self.gate_width) % 8
            mats.append(t("gate"))
            if pad:
                mats.append(torch.zeros((pad, self.hidden_size), dtype=mats[0].dtype, device=mats[0].device))
            if biases is not None:
                biases.append(torch.zeros(self.gate_width + pad, dtype=torch.float32, device=biases[0].device))
        weight = torch.cat(mats, dim=0).contiguous() if len(mats) > 1 else mats[0]
        bias = torch.cat(biases).contiguous() if biases is not None else None
        self.widths = tuple(m.shape[0] for m in mats)
        self.proj = Linear(weight, bias, runtime)
        self.out = Linear(t("out"), t("out_bias") if self.bias else None, runtime)
        if self.qk_norm == "unit":
            self.q_norm = torch.ones(self.dim, dtype=torch.float32, device=runtime.device)
            self.k_norm = self.q_norm if self.own_kv else None
        else:
            self.q_norm = t("q_norm") if self.qk_norm else None
            self.k_norm = t("k_norm") if self.own_kv and self.qk_norm else None
        self.slope_table = None
        if self.slopes:
            self.slope_table = torch.tensor([2.0 ** (-8.0 * (h + 1) / self.n_heads) for h in range(self.n_heads)],
                                            dtype=torch.float32, device=runtime.device)
        self.freq_table = torch.tensor(self.freqs or [0.0], dtype=torch.float64).to(torch.float32).to(runtime.device)
        self.lam, self.out_scale = 0.0, 1.0
        if self.maps == 2:
            # one number for the layer, in float32 like everything around the softmax
            dot = lambda a, b: (t(a).float() * t(b).float()).sum(dtype=torch.float32)
            self.lam = float(torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + self.diff)
            self.out_scale = 1.0 - self.diff

    def forward(self, h, residual, ctx, cache, owns_cache: bool, accumulate: bool = True) -> None:
        ops, dt = self.runtime.ops, self.runtime.dtype
        T = ctx.n_tokens
        if owns_cache and not self.own_kv:
            raise ConfigError("an attention layer without key and value projections cannot own a cache")
        views = ctx.buffer("mapped.proj" if self.own_kv else "mapped.proj_q", (T, sum(self.widths)), dt, columns=self.widths)
        self.proj(h, out=views[0])
        q = views[1]
        k, v = (views[2], views[2 if self.key_values else 3]) if owns_cache else (None, None)
        if self.shared_rows:
            v = None
        gate = views[self.gate_at] if self.gate_at is not None else None
        table = ctx.block_tables[cache.group]
        ops.qk_prepare(q, k, v, self.q_norm, self.k_norm, self.freq_table, self.magnitude, self.rot_dims, self.eps,
                       self.n_heads, self.n_kv_heads, self.maps, self.dim, self.vdim, ctx.tok_pos, ctx.tok_seq,
                       table if owns_cache else None, cache.page_tokens, cache.pages if owns_cache else None,
                       pairs=self.rot_layout == "pairs", shared=self.shared_rows and owns_cache)
        ctx.note("q", q)
        heads = ctx.buffer("mapped.heads", (T, self.n_heads * self.vdim), dt)
        ops.mapped_attention(q, cache.pages, table, cache.page_tokens, ctx.tok_pos, ctx.tok_seq, self.n_heads,
                             self.n_kv_heads, self.maps, self.dim, self.vdim, self.scale, self.window, heads,
                             lam=self.lam, out_scale=self.out_scale, eps=self.eps, unit_rms=self.maps == 2,
                             tiles=None if ctx.is_decode else ctx.q_tiles, single_tokens=ctx.is_decode,
                             gate=gate, chunk=self.chunk, slopes=self.slope_table, keep=self.keep,
                             sink=self.sink, softcap=self.softcap, shared=self.shared_rows)
        ctx.note("attn", heads)
        self.out(heads, residual=residual if accumulate else None, out=residual)


register_part("mixer", "mapped_attention", MappedAttention, replace=True)
