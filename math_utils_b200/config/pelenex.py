"""Pelenex's configuration: its nested config.json, typed, and its plan.

Keys read: ``vocab``, ``width``, ``norm`` = {``eps``, ``groups``}, ``logit_softcap`` (optional) and the list ``layers``;
an entry of that list has ``type`` (the kind of mixer), ``mixer`` (its sizes) and ``mlp`` (the feed-forward, or null).
Mixer ``channel_delta``: ``heads, kv_heads, dim, vdim, conv``.  Mixer ``mlstm``: ``heads, dim, vdim, gate_cap``.
Mixer ``parallel``: ``left`` = {``heads, kv_heads, dim, vdim, scale``, optional ``mask`` = {``size``, optional
``keep_first``}} and ``right`` = {``heads, dim, vdim, tau``}.
Feed-forward ``dense``: ``ff``; ``moe``: ``expert.ff``, ``router`` = {``experts, top``}, optional ``shared`` = {``ff``}.

The design: x = token row + sinusoids of the position.  Every layer is parallel with one norm, x += mixer(N x) + ff(N x),
N an RMS norm in ``norm.groups`` parts of the row.  Three kinds of mixer in any order: the gated delta rule with a decay
per key channel and an output gate, both through two matrices whose inner size the weight file gives; the matrix memory
of xLSTM; and two mixers side by side, each result normed over the width, half their sum: attention without rotation
(unit-rms queries and keys, the projected keys as values, a distance bias per head, a window beside which the first
tokens stay in sight) and gated linear attention.  The feed-forward is a gated one with silu, or routed experts with
sigmoid scores, not renormalised, that multiply what an expert reads, beside a shared expert.  At the end the same kind
of norm, an output matrix and a soft cap c * tanh(logits / c).  Nothing limits the positions; ``max_positions`` (an
optional key of this library's, 131,072 if absent) only sizes the page lists.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, KeyReader, LayerSpec, ModelPlan, PartSpec, default_schedule

MIXERS = ("channel_delta", "mlstm", "parallel")
DEFAULT_MAX_POSITIONS = 1 << 17
SINUSOID_BASE = 10000.0               # the design fixes it, and the two branches' weights
BRANCH_SCALE = 0.5


def _sub(reader: KeyReader, key: str) -> KeyReader:
    value = reader.raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"{reader.where}: key '{key}' must be an object")
    return KeyReader(value, f"{reader.where}: {key}")


def _grouped(m: KeyReader) -> None:
    heads, kv = m.integer("heads"), m.integer("kv_heads")
    if heads % kv:
        raise ConfigError(f"{m.where}: heads {heads} must be a multiple of kv_heads {kv}")


@dataclass(frozen=True)
class PelenexConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    logit_softcap: float              # 0: none
    layers: tuple                     # the checked raw entries
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Pelenex"

    @classmethod
    def from_json(cls, raw: Mapping[str, Any]) -> "PelenexConfig":
        r = KeyReader(raw)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: key 'layers' must be a list with at least one layer")
        for i, layer in enumerate(layers):
            cls._check_layer(f"config.json: layers[{i}]", layer)
        norm, width = _sub(r, "norm"), r.integer("width")
        groups = norm.integer("groups")
        if width % groups:
            raise ConfigError(f"config.json: width {width} does not split into norm.groups {groups}")
        cap = raw.get("logit_softcap")
        return cls(vocab=r.integer("vocab"), width=width, norm_eps=norm.number("eps"), norm_groups=groups,
                   logit_softcap=0.0 if cap is None else r.number("logit_softcap"), layers=tuple(layers),
                   max_positions=r.integer("max_positions", default=DEFAULT_MAX_POSITIONS))

    @staticmethod
    def _check_layer(where: str, layer) -> None:
        lr = KeyReader(layer, where)
        kind, m = lr.string("type", choices=MIXERS), _sub(lr, "mixer")
        if kind == "parallel":
            left, right = _sub(m, "left"), _sub(m, "right")
            _grouped(left)
            if left.integer("dim") != left.integer("vdim"):
                raise ConfigError(f"{left.where}: the keys are the values too, so vdim equals dim")
            left.number("scale")
            if left.raw.get("mask") is not None:
                mask = _sub(left, "mask")
                mask.integer("size")
                mask.integer("keep_first", default=0, minimum=0)
            for key in ("heads", "dim", "vdim"):
                right.integer(key)
            right.number("tau")
        else:
            for key in ("heads", "dim", "vdim"):
                m.integer(key)
            if kind == "channel_delta":
                _grouped(m)
                m.integer("conv")
            else:
                m.number("gate_cap")
        if layer.get("mlp") is None:
            return
        f = _sub(lr, "mlp")
        if f.string("kind", choices=("dense", "moe")) == "dense":
            f.integer("ff")
            return
        _sub(f, "expert").integer("ff")
        router = _sub(f, "router")
        n, top = router.integer("experts"), router.integer("top")
        if top > n:
            raise ConfigError(f"{where}: mlp.router.top {top} exceeds its {n} experts")
        if f.raw.get("shared") is not None:
            _sub(f, "shared").integer("ff")

    def to_json(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "layers": [dict(layer) for layer in self.layers]}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    def init_distribution(self, rule: str):
        """(mean, standard deviation) of a random-weights rule: matrices N(0, 1/width)."""
        r = 1.0 / math.sqrt(self.width)
        rules = {"normal": (0.0, r), "residual_projection": (0.0, r), "bias": (0.0, 0.1), "norm_weight": (1.0, 0.1),
                 "conv": (0.0, 0.5)}
        if rule not in rules:
            raise ConfigError(f"no random-weights rule '{rule}'")
        return rules[rule]

    # ------------------------------------------------------------------ plan
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rms_norm", {"size": self.width, "eps": self.norm_eps, "groups": self.norm_groups}, {"weight": name})

    def _mixer(self, kind: str, m, x: str) -> PartSpec:
        sizes = {"hidden_size": self.width, "eps": self.norm_eps}
        if kind == "parallel":
            return PartSpec("parallel",
                            {"hidden_size": self.width, "left": self._attention(m["left"], x + "left."),
                             "right": self._linear_attention(m["right"], x + "right."), "left_scale": BRANCH_SCALE,
                             "right_scale": BRANCH_SCALE, "branch_norm": {"eps": self.norm_eps}},
                            {"left_norm": x + "left.out", "right_norm": x + "right.out"})
        sizes.update(n_heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
        if kind == "mlstm":
            return PartSpec("matrix_lstm", dict(sizes, gate_cap=float(m["gate_cap"])),
                            {"q": x + "q", "k": x + "k", "v": x + "v", "gate": x + "g", "i": x + "i", "i_bias": x + "i.b",
                             "f": x + "f", "f_bias": x + "f.b", "norm": x + "norm", "out": x + "o"})
        return PartSpec("gated_delta",
                        dict(sizes, n_kv_heads=int(m["kv_heads"]), conv=int(m["conv"]), channel_decay=True,
                             low_rank_gate=True, gate_act="sigmoid"),
                        {"q": x + "q", "k": x + "k", "v": x + "v", "q_conv": x + "q.conv", "k_conv": x + "k.conv",
                         "v_conv": x + "v.conv", "beta": x + "b", "decay_down": x + "a1", "decay_up": x + "a2",
                         "A_log": x + "A_log", "dt_bias": x + "dt_bias", "norm": x + "norm", "gate_down": x + "g1",
                         "gate_up": x + "g2", "out": x + "o"})

    def _attention(self, m, x: str) -> PartSpec:
        mask = m.get("mask") or {}
        window, keep = int(mask.get("size", 0)), int(mask.get("keep_first") or 0)
        return PartSpec("mapped_attention",
                        {"hidden_size": self.width, "n_heads": int(m["heads"]), "n_kv_heads": int(m["kv_heads"]),
                         "dim": int(m["dim"]), "vdim": int(m["vdim"]), "maps": 1, "softmax_scale": float(m["scale"]),
                         "eps": self.norm_eps, "rot": None, "bias": False, "qk_norm": "unit", "key_values": True,
                         "slopes": "geometric", "window": window, "keep": keep},
                        {"q": x + "q", "k": x + "k", "out": x + "o"})

    def _linear_attention(self, m, x: str) -> PartSpec:
        return PartSpec("gated_linear_attention",
                        {"hidden_size": self.width, "n_heads": int(m["heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]),
                         "tau": float(m["tau"]), "eps": self.norm_eps},
                        {"q": x + "q", "k": x + "k", "v": x + "v", "gate": x + "g", "decay_down": x + "a1",
                         "decay_up": x + "a2", "decay_bias": x + "a2.b", "norm": x + "norm", "out": x + "o"})

    def _mlp(self, mlp, f: str) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("gated_ffn", {"hidden_size": self.width, "inner_size": int(mlp["ff"]), "activation": "silu"},
                            {"gate_weight": f + "gate", "up_weight": f + "up", "down_weight": f + "down"})
        params = {"hidden_size": self.width, "inner_size": int(mlp["expert"]["ff"]),
                  "n_experts": int(mlp["router"]["experts"]), "top": int(mlp["router"]["top"]), "score": "sigmoid",
                  "weight_on": "input"}
        names = {"router": f + "router", "gate": f + "e{e}.gate", "up": f + "e{e}.up", "down": f + "e{e}.down"}
        if mlp.get("shared") is not None:
            params["shared"] = {"inner_size": int(mlp["shared"]["ff"])}
            names.update({"shared_gate_proj": f + "shared.gate", "shared_up": f + "shared.up", "shared_down": f + "shared.down"})
        return PartSpec("routed_experts", params, names)

    def plan(self) -> ModelPlan:
        D = self.width
        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            mlp = layer.get("mlp")
            ffn = PartSpec("none") if mlp is None else self._mlp(mlp, p + "mlp.")
            layers.append(LayerSpec("parallel_pre_norm", self._norm(p + "norm1"),
                                    self._mixer(layer["type"], layer["mixer"], p + "mix."), PartSpec("identity"), ffn,
                                    arrangement_params={"shared_norm": True}))
        plan = ModelPlan(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D, max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D}, {"weight": "embed"}),
            position=PartSpec("sinusoidal", {"hidden_size": D, "base": SINUSOID_BASE}),
            layers=tuple(layers), schedule=default_schedule(len(layers)), final_norm=self._norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": D, "softcap": self.logit_softcap},
                          {"weight": "head"}))
        plan.validate()
        return plan
