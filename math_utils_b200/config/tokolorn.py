"""Tokolorn's configuration: its nested config.json, typed, and its plan.

Keys read: ``vocab``, ``width``, ``norm`` = {``eps``}, ``embedding`` = {``scale``, optional ``bigram`` = {``buckets,
mul_prev, mul_cur``}}, ``logit_scale``, optional ``loop`` = {``start, stop, times``} and the list ``layers``; an entry of
that list has ``type`` (the kind of mixer), ``mixer`` (its sizes) and ``mlp`` = {``kind``: ``dense``, ``ff``} or null.
Mixer ``lightning``: ``heads, dim, vdim, decay`` (a list, one per head).  Mixer ``attention``: ``heads, kv_heads, dim,
scale``, optional ``mask`` = {``size``} (chunks).  Mixer ``parallel``: ``left`` = {``heads, kv_heads, dim, vdim, scale``,
optional ``rot`` = {``base, dims``}, optional ``softcap``, optional ``mask`` = {``size``} (a window)}, ``right`` =
{``inner, state, dt_rank, conv``}, ``left_scale``, ``right_scale``.

The design: x = scale * token row + a row hashed from the token and the one before it.  Every layer is pre-norm,
x += s1 * mixer(N1 x); x += s2 * ff(N2 x), with an element-wise scale on what each sublayer adds and RMS norms whose
weight is one number.  Three kinds of mixer in any order: lightning attention (a constant decay per head); attention
in chunks of positions with a softmax sink, without rotation, whose values are its keys; and two mixers side by side,
windowed attention (pairs rotated, a soft cap on the scores, a gate per output entry) and Mamba's selective scan.  The
feed-forward is gated with the tanh form of gelu.  A run of layers may be passed several times with the same weights,
each pass with a cache of its own.  At the end the same kind of norm and an output matrix whose product is multiplied by
``logit_scale``.  Nothing limits the positions; ``max_positions`` (an optional key of this library's, 131,072 if absent)
only sizes the page lists.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, KeyReader, LayerSpec, ModelPlan, PartSpec, ScheduleEntry

MIXERS = ("lightning", "attention", "parallel")
DEFAULT_MAX_POSITIONS = 1 << 17


def _sub(reader: KeyReader, key: str) -> KeyReader:
    value = reader.raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"{reader.where}: key '{key}' must be an object")
    return KeyReader(value, f"{reader.where}: {key}")


def _check_attention(m: KeyReader) -> None:
    heads, kv = m.integer("heads"), m.integer("kv_heads")
    if heads % kv:
        raise ConfigError(f"{m.where}: heads {heads} must be a multiple of kv_heads {kv}")
    m.integer("dim")
    m.number("scale")
    if m.raw.get("mask") is not None:
        _sub(m, "mask").integer("size")


@dataclass(frozen=True)
class TokolornConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: Any                       # the checked raw entry, or None
    logit_scale: float
    layers: tuple                     # the checked raw entries
    loop: tuple                       # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Tokolorn"

    @classmethod
    def from_json(cls, raw: Mapping[str, Any]) -> "TokolornConfig":
        r = KeyReader(raw)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: key 'layers' must be a list with at least one layer")
        for i, layer in enumerate(layers):
            cls._check_layer(f"config.json: layers[{i}]", layer)
        emb = _sub(r, "embedding")
        bigram = emb.raw.get("bigram")
        if bigram is not None:
            b = _sub(emb, "bigram")
            b.integer("buckets")
            for key in ("mul_prev", "mul_cur"):
                b.integer(key, minimum=0)
        loop = (0, len(layers), 1)
        if raw.get("loop") is not None:
            lo = _sub(r, "loop")
            loop = (lo.integer("start", minimum=0), lo.integer("stop", minimum=0), lo.integer("times"))
            if not loop[0] <= loop[1] <= len(layers):
                raise ConfigError(f"{lo.where}: layers {loop[0]} .. {loop[1]} - 1 are not among the model's {len(layers)}")
        return cls(vocab=r.integer("vocab"), width=r.integer("width"), norm_eps=_sub(r, "norm").number("eps", positive=False),
                   embedding_scale=emb.number("scale", default=1.0, positive=False), bigram=bigram,
                   logit_scale=r.number("logit_scale", default=1.0, positive=False), layers=tuple(layers), loop=loop,
                   max_positions=r.integer("max_positions", default=DEFAULT_MAX_POSITIONS))

    @staticmethod
    def _check_layer(where: str, layer) -> None:
        lr = KeyReader(layer, where)
        kind, m = lr.string("type", choices=MIXERS), _sub(lr, "mixer")
        if kind == "lightning":
            heads = m.integer("heads")
            m.integer("dim"), m.integer("vdim")
            decay = m.raw.get("decay")
            if (not isinstance(decay, list) or len(decay) != heads
                    or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay)):
                raise ConfigError(f"{m.where}: key 'decay' must be a list of {heads} numbers, one per head")
        elif kind == "attention":
            _check_attention(m)
            if m.integer("vdim", default=m.integer("dim")) != m.integer("dim"):
                raise ConfigError(f"{m.where}: the keys are the values too, so vdim equals dim")
        else:
            left, right = _sub(m, "left"), _sub(m, "right")
            _check_attention(left)
            left.integer("vdim")
            if left.raw.get("softcap") is not None:
                left.number("softcap")
            if left.raw.get("rot") is not None:
                rot = _sub(left, "rot")
                rot.number("base")
                dims = rot.integer("dims", minimum=0)
                if dims % 2 or dims > left.integer("dim"):
                    raise ConfigError(f"{rot.where}: dims {dims} must be even and at most the heads' {left.integer('dim')}")
            for key in ("inner", "state", "dt_rank", "conv"):
                right.integer(key)
            m.number("left_scale", positive=False), m.number("right_scale", positive=False)
        if layer.get("mlp") is not None:
            f = _sub(lr, "mlp")
            f.string("kind", choices=("dense",))
            f.integer("ff")

    def to_json(self) -> dict:
        emb = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = dict(self.bigram)
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": emb, "logit_scale": self.logit_scale, "layers": [dict(layer) for layer in self.layers]}
        if self.loop != (0, len(self.layers), 1):
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
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
    def _norm(self, name: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("rms_norm", {"size": self.width, "eps": self.norm_eps, "one_number": True, "scale": scale},
                        {"weight": name})

    def _mixer(self, kind: str, m, x: str) -> PartSpec:
        sizes = {"hidden_size": self.width, "eps": self.norm_eps}
        if kind == "lightning":
            return PartSpec("lightning_attention",
                            dict(sizes, n_heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                 decay=tuple(float(d) for d in m["decay"])),
                            {"q": x + "q", "k": x + "k", "v": x + "v", "gate": x + "g", "norm": x + "norm", "out": x + "o"})
        if kind == "parallel":
            return PartSpec("parallel",
                            {"hidden_size": self.width, "left": self._windowed(m["left"], x + "left."),
                             "right": self._selective_scan(m["right"], x + "right."),
                             "left_scale": float(m["left_scale"]), "right_scale": float(m["right_scale"])})
        size = int(m["mask"]["size"]) if m.get("mask") else 0
        return PartSpec("mapped_attention",
                        dict(self._heads(m), vdim=int(m["dim"]), rot=None, key_values=True, chunk=size, cache_window=size,
                             sink=True),
                        {"q": x + "q", "k": x + "k", "out": x + "o"})

    def _heads(self, m) -> dict:
        return {"hidden_size": self.width, "eps": self.norm_eps, "n_heads": int(m["heads"]), "n_kv_heads": int(m["kv_heads"]),
                "dim": int(m["dim"]), "maps": 1, "softmax_scale": float(m["scale"]), "bias": False, "qk_norm": False}

    def _windowed(self, m, x: str) -> PartSpec:
        rot = m.get("rot")
        return PartSpec("mapped_attention",
                        dict(self._heads(m), vdim=int(m["vdim"]), window=int(m["mask"]["size"]) if m.get("mask") else 0,
                             rot={"base": float(rot["base"]), "dims": int(rot["dims"])} if rot else None, rot_layout="pairs",
                             softcap=float(m.get("softcap") or 0.0), entry_gate=True),
                        {"q": x + "q", "k": x + "k", "v": x + "v", "gate": x + "g", "out": x + "o"})

    def _selective_scan(self, m, x: str) -> PartSpec:
        return PartSpec("selective_scan",
                        {"hidden_size": self.width, "inner": int(m["inner"]), "state": int(m["state"]),
                         "dt_rank": int(m["dt_rank"]), "conv": int(m["conv"])},
                        {"in": x + "in", "conv": x + "conv", "conv_bias": x + "conv.b", "x": x + "x", "dt": x + "dt",
                         "dt_bias": x + "dt.b", "A_log": x + "A_log", "D": x + "D", "out": x + "o"})

    def schedule(self) -> tuple:
        """The layers in the order they run; every run owns its cache."""
        start, stop, times = self.loop
        order = [*range(start), *(list(range(start, stop)) * times), *range(stop, len(self.layers))]
        return tuple(ScheduleEntry(layer=layer, cache_of=i) for i, layer in enumerate(order))

    def plan(self) -> ModelPlan:
        D = self.width
        scale = lambda name: PartSpec("layer_scale", {"size": D}, {"weight": name})
        layers = []
        for i, layer in enumerate(self.layers):
            p, mlp = f"l{i}.", layer.get("mlp")
            extra = [("scale1", "scale", scale(p + "ls1"))]
            norm2, ffn = PartSpec("identity"), PartSpec("none")
            if mlp is not None:
                extra.append(("scale2", "scale", scale(p + "ls2")))
                norm2, f = self._norm(p + "norm2"), p + "mlp."
                ffn = PartSpec("gated_ffn", {"hidden_size": D, "inner_size": int(mlp["ff"]), "activation": "gelu_new"},
                               {"gate_weight": f + "gate", "up_weight": f + "up", "down_weight": f + "down"})
            layers.append(LayerSpec("scaled_pre_norm", self._norm(p + "norm1"),
                                    self._mixer(layer["type"], layer["mixer"], p + "mix."), norm2, ffn, extra=tuple(extra)))
        if self.bigram is not None:
            embedding = PartSpec("token_pair_embedding",
                                 {"vocab_size": self.vocab, "hidden_size": D, "buckets": int(self.bigram["buckets"]),
                                  "mul_prev": int(self.bigram["mul_prev"]), "mul_cur": int(self.bigram["mul_cur"]),
                                  "scale": self.embedding_scale}, {"weight": "embed", "pair_weight": "bigram"})
        else:
            embedding = PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D, "scale": self.embedding_scale},
                                 {"weight": "embed"})
        plan = ModelPlan(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D, max_positions=self.max_positions,
            embedding=embedding, position=PartSpec("none"), layers=tuple(layers), schedule=self.schedule(),
            # the head is linear: its product's multiplier rides on the rows the last norm hands it
            final_norm=self._norm("final.norm", scale=self.logit_scale),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": D}, {"weight": "head"}))
        plan.validate()
        return plan
