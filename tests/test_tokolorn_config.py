"""Tokolorn's configuration and plan (looped layers among it), the cache it asks for, and properties of the plain
statement itself; no device needed."""
import json
import math

import numpy as np
import pytest
import torch

import plain_tokolorn as plain
from math_utils_b200.cache import SequenceCache
from math_utils_b200.config import ConfigError, PartSpec, TokolornConfig, architecture_for
from math_utils_b200.engine.assemble import assemble, collect_tensor_specs
from math_utils_b200.parts import CompositeCacheSpec, RowCacheSpec, StateCacheSpec, build_part
from math_utils_b200.weights import write_random_model
from math_utils_b200.weights.safetensors import SafetensorsFile

CHUNKED = {"heads": 6, "kv_heads": 2, "dim": 10, "scale": 0.3, "mask": {"size": 20}}
FADING = {"heads": 3, "dim": 8, "vdim": 6, "decay": [0.5, 0.9, 0.99]}
BOTH = {"left": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.4, "mask": {"size": 9}, "softcap": 7.0,
                 "rot": {"base": 3000.0, "dims": 6}},
        "right": {"inner": 14, "state": 5, "dt_rank": 3, "conv": 4}, "left_scale": 0.7, "right_scale": -0.2}
CFG = {"architecture": "Tokolorn", "vocab": 90, "width": 36, "norm": {"eps": 1e-5}, "logit_scale": 0.5,
       "embedding": {"scale": 5.0, "bigram": {"buckets": 17, "mul_prev": 3, "mul_cur": 5}}, "loop": {"start": 1, "stop": 3, "times": 3},
       "layers": [{"type": "attention", "mixer": CHUNKED, "mlp": {"kind": "dense", "ff": 40}},
                  {"type": "lightning", "mixer": FADING, "mlp": None},
                  {"type": "parallel", "mixer": BOTH, "mlp": {"kind": "dense", "ff": 24}},
                  {"type": "lightning", "mixer": FADING, "mlp": {"kind": "dense", "ff": 16}}]}


def test_configuration_and_plan():
    assert architecture_for(CFG).config_class is TokolornConfig
    plan = TokolornConfig.from_json(CFG).plan()
    assert [l.mixer.kind for l in plan.layers] == ["mapped_attention", "lightning_attention", "parallel", "lightning_attention"]
    assert [l.feed_forward.kind for l in plan.layers] == ["gated_ffn", "none", "gated_ffn", "gated_ffn"]
    assert all(l.arrangement == "scaled_pre_norm" for l in plan.layers)
    assert [(e.layer, e.cache_of) for e in plan.schedule] == list(zip([0, 1, 2, 1, 2, 1, 2, 3], range(8)))
    assert [e.layer for e in plan.schedule] == plain.order_of_layers(CFG)
    assert plan.final_norm.params["scale"] == 0.5 and plan.final_norm.params["one_number"]
    left = plan.layers[2].mixer.params["left"].params
    assert (left["window"], left["softcap"], left["rot_layout"], left["entry_gate"]) == (9, 7.0, "pairs", True)
    assert TokolornConfig.from_json(TokolornConfig.from_json(CFG).to_json()).plan() == plan
    want = plain.tensor_shapes(CFG)
    specs = {s.name: tuple(s.shape) for s in collect_tensor_specs(plan)}
    assert specs == want


def test_what_may_be_absent():
    bare = json.loads(json.dumps(CFG))
    for key in ("loop", "logit_scale"):
        bare.pop(key)
    bare["embedding"] = {"scale": 2.0}
    bare["layers"][0]["mixer"].pop("mask")
    for key in ("mask", "softcap", "rot"):
        bare["layers"][2]["mixer"]["left"].pop(key)
    plan = TokolornConfig.from_json(bare).plan()
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 3]
    assert plan.embedding.kind == "token_embedding" and plan.embedding.params["scale"] == 2.0
    assert plan.final_norm.params["scale"] == 1.0 and plan.layers[0].mixer.params["chunk"] == 0
    left = plan.layers[2].mixer.params["left"].params
    assert (left["window"], left["softcap"], left["rot"]) == (0, 0.0, None)
    specs = {s.name for s in collect_tensor_specs(plan)}
    assert "bigram" not in specs and "l1.ls2" not in specs and "l1.norm2" not in specs


@pytest.mark.parametrize("loop,order", [(None, [0, 1, 2, 3]), ((0, 4, 2), [0, 1, 2, 3, 0, 1, 2, 3]), ((3, 4, 3), [0, 1, 2, 3, 3, 3]),
                                        ((0, 1, 2), [0, 0, 1, 2, 3]), ((2, 2, 5), [0, 1, 2, 3]), ((1, 3, 1), [0, 1, 2, 3])])
def test_loops(loop, order):
    cfg = json.loads(json.dumps(CFG))
    cfg.pop("loop")
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    plan = TokolornConfig.from_json(cfg).plan()
    assert [e.layer for e in plan.schedule] == order == plain.order_of_layers(cfg)
    assert [e.cache_of for e in plan.schedule] == list(range(len(order)))             # every pass has a cache of its own


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=12), "vdim"),                  # keys that are the values
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, "x"]), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][2]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][2]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][2]["mixer"]["right"].pop("dt_rank"), "dt_rank"),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=10), "dims"),
    (lambda c: c["layers"][2].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=4), "loop"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c["embedding"]["bigram"].pop("buckets"), "buckets"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("embedding"), "embedding"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(change, word):
    bad = json.loads(json.dumps(CFG))
    change(bad)
    with pytest.raises(ConfigError, match=word):
        TokolornConfig.from_json(bad)


@pytest.mark.parametrize("change,word", [
    ({"chunk": 9, "cache_window": 8}, "chunk"), ({"head_gate": True, "entry_gate": True}, "gate"), ({"chunk": 4, "window": 5}, "chunks"),
])
def test_attention_switches_that_exclude_one_another(change, word):
    params = {"hidden_size": 8, "n_heads": 2, "n_kv_heads": 1, "dim": 4, "vdim": 4, "softmax_scale": 1.0, "eps": 0.0, "rot": None,
              "qk_norm": False}
    build_part("mixer", PartSpec("mapped_attention", params))
    with pytest.raises(ConfigError, match=word):
        build_part("mixer", PartSpec("mapped_attention", dict(params, **change)))


def test_random_weights_mode(tmp_path):
    write_random_model(str(tmp_path), CFG, seed=3)
    f = SafetensorsFile(str(tmp_path / "model.safetensors"))
    shapes = {n: tuple(f.tensors[n].shape) for n in f.names()}
    f.close()
    assert shapes == plain.tensor_shapes(CFG)


def test_cache_of_the_plan():
    plan = TokolornConfig.from_json(CFG).plan()
    layers = assemble(plan).layers
    specs = [layer.mixer.cache_spec() for layer in layers]
    assert specs[0] == RowCacheSpec(2 * 10, 20)                                      # the keys are the values: kept once
    assert specs[1] == StateCacheSpec(3 * 8 * 6)
    values = 3 * 14 + 14 * 5
    assert specs[2] == CompositeCacheSpec((RowCacheSpec(2 * (8 + 12), 9), StateCacheSpec(values + -values % 4)))
    cache = SequenceCache([specs[e.layer] for e in plan.schedule], 64 * 9, 1024, torch.float32, "cpu", n_slots=3)
    assert len(cache.kv_groups) == 2 and cache.has_running_state
    assert len({cache.entry(i).values.data_ptr() for i in (1, 3, 5, 7)}) == 4         # a state for every pass and layer
    a = cache.acquire()
    cache.entry(3).values[a] = 3.0
    cache.release(a)
    assert cache.acquire() == a and (cache.entry(3).values[a] == 0.0).all()


@pytest.mark.parametrize("chunk", [1, 20, 64, 100, 200])
def test_pages_of_a_chunk_stay(chunk):
    """A cache that keeps the last `chunk` positions holds every page that a query's chunk reaches, and gives the others back."""
    cache = SequenceCache([RowCacheSpec(4, chunk)], 64 * 12, 4096, torch.float32, "cpu", n_slots=2)
    group, slot = cache.kv_groups[0], cache.acquire()
    n = 0
    for step in [3, 61, 1, 130] + [1] * 200 + [64, 2, 127]:
        old = n
        cache.reserve(slot, step)
        n += step
        for p in range(old, n):
            for j in range(p - p % chunk, p + 1):
                assert group.table[slot, j // 64] >= 0, (p, j)
        cache.commit(slot, step)
        assert cache.kv_groups[0].pages_held(slot) <= chunk // 64 + 2
    cache.release(slot)
    assert cache.free_pages() == 12


def test_plain_statement():
    """The plain statement itself: the masks' edges, the sink, the cap, the rotation, both recurrences against closed forms."""
    assert [j for j in range(12) if plain.in_window(9, j, 4)] == [6, 7, 8, 9]
    assert [j for j in range(12) if plain.in_chunk(9, j, 4)] == [8, 9] and [j for j in range(12) if plain.in_chunk(7, j, 4)] == [4, 5, 6, 7]
    assert [j for j in range(5) if plain.in_chunk(2, j, None)] == [0, 1, 2] == [j for j in range(5) if plain.in_window(2, j, None)]
    rng = np.random.default_rng(0)
    q, k, v = (rng.normal(0, 1, (6, n)) for n in (4, 4, 3))
    every = lambda i, j: j <= i
    out = plain.masked_attention(np.zeros((6, 2)), np.zeros((6, 2)), v, 1.0, every, sink=True)
    assert np.abs(out[5] - v.sum(0) / 7.0).max() < 1e-12                              # six keys and the sink
    big = plain.masked_attention(1e3 * q, k, v, 1.0, every, softcap=1e-9)
    assert np.abs(big[5] - v.mean(0)).max() < 1e-6                                    # a tiny cap makes all scores alike
    y = plain.rotate_pairs(np.tile(np.array([1.0, 0.0, 5.0, 6.0, 7.0]), (4, 1, 1)), 100.0, 4)
    assert np.allclose(y[3, 0], [math.cos(3), math.sin(3), 5 * math.cos(.3) - 6 * math.sin(.3), 6 * math.cos(.3) + 5 * math.sin(.3), 7])
    out = plain.fading_recurrence(q, k, v, 0.5)
    want = sum(0.5 ** (5 - t) * (k[t] @ q[5]) * v[t] for t in range(6))
    assert np.abs(out[5] - want).max() < 1e-12
    x, dt, B, C = rng.normal(0, 1, (6, 3)), rng.uniform(0.1, 1, (6, 3)), rng.normal(0, 1, (6, 2)), rng.normal(0, 1, (6, 2))
    A, D = -rng.uniform(0.1, 2, (3, 2)), rng.normal(0, 1, 3)
    out = plain.selective_scan(x, dt, A, B, C, D)
    want = [sum(math.exp(A[c, n] * dt[t + 1:, c].sum()) * dt[t, c] * x[t, c] * B[t, n] * C[5, n] for t in range(6) for n in range(2))
            + D[c] * x[5, c] for c in range(3)]
    assert np.abs(out[5] - want).max() < 1e-12
    assert list(plain.pair_rows([4, 7, 4], {"buckets": 5, "mul_prev": 3, "mul_cur": 2})) == [5, (12 + 14) % 5, (21 + 8) % 5]
    assert np.abs(plain.scalar_rms_norm(x, np.array(2.0), 0.0) ** 2).mean() - 4.0 < 1e-12
