"""Pelenex's configuration and plan, sizes that only the weight file gives, the cache it asks for (kept pages beside a
window among it), and properties of the plain statement itself; no device needed."""
import json
import math

import numpy as np
import pytest
import torch

import plain_pelenex as plain
from math_utils_b200.cache import SequenceCache
from math_utils_b200.config import ConfigError, PelenexConfig, architecture_for
from math_utils_b200.engine.assemble import assemble, collect_tensor_specs
from math_utils_b200.parts import CompositeCacheSpec, FreeSize, RowCacheSpec, StateCacheSpec
from math_utils_b200.parts.base import TensorSpec, shape_fits
from math_utils_b200.weights import write_random_model
from math_utils_b200.weights.loader import WeightError, load_weights
from math_utils_b200.weights.safetensors import SafetensorsFile, write_safetensors

DELTA = {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 6, "conv": 3}
LSTM = {"heads": 2, "dim": 8, "vdim": 12, "gate_cap": 9.0}
BOTH = {"left": {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 8, "scale": 0.3, "mask": {"size": 20, "keep_first": 5}},
        "right": {"heads": 2, "dim": 6, "vdim": 10, "tau": 4.0}}
MOE = {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 20}}
CFG = {"architecture": "Pelenex", "vocab": 90, "width": 36, "norm": {"eps": 1e-5, "groups": 3}, "logit_softcap": 11.0,
       "layers": [{"type": "parallel", "mixer": BOTH, "mlp": {"kind": "dense", "ff": 40}},
                  {"type": "channel_delta", "mixer": DELTA, "mlp": MOE},
                  {"type": "mlstm", "mixer": LSTM, "mlp": None}]}


def test_configuration_and_plan():
    assert architecture_for(CFG).config_class is PelenexConfig
    plan = PelenexConfig.from_json(CFG).plan()
    assert [l.mixer.kind for l in plan.layers] == ["parallel", "gated_delta", "matrix_lstm"]
    assert [l.feed_forward.kind for l in plan.layers] == ["gated_ffn", "routed_experts", "none"]
    assert all(l.arrangement == "parallel_pre_norm" and l.arrangement_params["shared_norm"] for l in plan.layers)
    assert plan.layers[1].feed_forward.params["weight_on"] == "input" and plan.position.kind == "sinusoidal"
    assert plan.head.params["softcap"] == 11.0 and plan.final_norm.params["groups"] == 3
    assert PelenexConfig.from_json(PelenexConfig.from_json(CFG).to_json()).plan() == plan
    want = plain.tensor_shapes(CFG)
    specs, free = {s.name: s for s in collect_tensor_specs(plan)}, {}
    assert set(specs) == set(want)
    assert all(shape_fits(want[name], s.shape, free) for name, s in specs.items())
    # the inner sizes of the projections through two matrices, one for each of them
    assert set(free) == {"l0.mix.right.a1", "l1.mix.a1", "l1.mix.g1"}


def test_what_may_be_absent():
    bare = json.loads(json.dumps(CFG))
    bare.pop("logit_softcap")
    bare["layers"][0]["mixer"]["left"].pop("mask")
    bare["layers"][1]["mlp"].pop("shared")
    plan = PelenexConfig.from_json(bare).plan()
    left = plan.layers[0].mixer.params["left"].params
    assert left["window"] == 0 and left["keep"] == 0 and plan.head.params["softcap"] == 0.0
    assert "shared" not in plan.layers[1].feed_forward.params
    bare["layers"][0]["mixer"]["left"]["mask"] = {"size": 7}
    left = PelenexConfig.from_json(bare).plan().layers[0].mixer.params["left"].params
    assert (left["window"], left["keep"]) == (7, 0)


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=12), "vdim"),          # keys that are the values
    (lambda c: c["layers"][0]["mixer"]["right"].pop("tau"), "tau"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][2].update(type="delta"), "type"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "kind"),
    (lambda c: c["norm"].update(groups=5), "groups"),
    (lambda c: c["norm"].pop("groups"), "groups"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(change, word):
    bad = json.loads(json.dumps(CFG))
    change(bad)
    with pytest.raises(ConfigError, match=word):
        PelenexConfig.from_json(bad)


def test_sizes_that_the_file_gives(tmp_path):
    n = FreeSize("rank", 4)
    free = {}
    assert shape_fits((7, 3), (n, 3), free) and free == {"rank": 7}
    assert shape_fits((5, 7), (5, n), free) and not shape_fits((5, 6), (5, n), free) and not shape_fits((7,), (n, 3), free)
    specs = [TensorSpec("down", (n, 3)), TensorSpec("up", (5, n))]
    write_safetensors(str(tmp_path / "model.safetensors"), {"down": torch.ones(6, 3), "up": torch.ones(5, 6)})
    out = load_weights(str(tmp_path), specs, torch.float32, "cpu")
    assert out["down"].shape == (6, 3) and out["up"].shape == (5, 6)
    write_safetensors(str(tmp_path / "model.safetensors"), {"down": torch.ones(6, 3), "up": torch.ones(5, 8)})
    with pytest.raises(WeightError, match=r"up is \[5, 8\], wanted \[5, 6\]"):
        load_weights(str(tmp_path), specs, torch.float32, "cpu")


def test_random_weights_mode(tmp_path):
    write_random_model(str(tmp_path), CFG, seed=3)
    f = SafetensorsFile(str(tmp_path / "model.safetensors"))
    shapes = {n: tuple(f.tensors[n].shape) for n in f.names()}
    f.close()
    assert shapes["l1.mix.a1"] == (10, 36) and shapes["l1.mix.a2"] == (40, 10)       # a head's key size, unless a file says otherwise
    assert set(shapes) == set(plain.tensor_shapes(CFG))


def test_cache_of_the_plan():
    specs = [layer.mixer.cache_spec() for layer in assemble(PelenexConfig.from_json(CFG).plan()).layers]
    assert specs[0] == CompositeCacheSpec((RowCacheSpec(3 * 8 + 3 * 8, 20, 5), StateCacheSpec(2 * 6 * 10)))
    channels = 2 * 2 * 10 + 4 * 6
    assert specs[1] == StateCacheSpec(2 * channels + 4 * 6 * 10)
    values = 2 * 8 * 12 + 2 * 8 + 2                                                  # S, n and m of every head
    assert specs[2] == StateCacheSpec(values + -values % 4)
    cache = SequenceCache(specs, 64 * 9, 1024, torch.float32, "cpu", n_slots=3)
    assert len(cache.kv_groups) == 1 and cache.has_running_state
    a = cache.acquire()
    cache.entry(2).values[a] = 3.0
    cache.release(a)
    assert cache.acquire() == a and (cache.entry(2).values[a] == 0.0).all()


@pytest.mark.parametrize("window,keep", [(70, 9), (64, 64), (10, 65), (100, 0), (1, 130)])
def test_pages_with_kept_positions_stay(window, keep):
    """A step at a time over several pages: the pages held are those that the window of the next position or the kept
    positions touch, and no page is lost when the sequence ends."""
    cache = SequenceCache([RowCacheSpec(4, window, keep)], 64 * 12, 4096, torch.float32, "cpu", n_slots=2)
    group, slot = cache.kv_groups[0], cache.acquire()
    n = 0
    for step in [3, 61, 1, 130] + [1] * 200 + [64, 2, 127]:
        old = n
        cache.reserve(slot, step)
        n += step
        for p in range(old, n):                          # every position that a query of this step sees is held
            for j in set(range(max(0, p - window + 1), p + 1)) | set(range(min(keep, p + 1))):
                assert group.table[slot, j // 64] >= 0, (p, j)
        cache.commit(slot, step)
        held = {i for i in range(group.max_pages) if group.table[slot, i] >= 0}
        lo = max(0, n - window + 1) // 64
        want = {i for i in range((n + 63) // 64) if i >= lo or i < -(-keep // 64)}
        assert want <= held and len(held - want) <= 1, (n, held, want)
    cache.release(slot)
    assert cache.free_pages() == 12


def test_plain_statement():
    """The plain statement itself: the mask's edges, the distance bias, the three recurrences against closed forms."""
    mask = {"size": 4, "keep_first": 2}
    assert [j for j in range(12) if plain.seen(9, j, mask)] == [0, 1, 6, 7, 8, 9]
    assert [j for j in range(12) if plain.seen(3, j, mask)] == [0, 1, 2, 3]
    assert [j for j in range(5) if plain.seen(2, j, None)] == [0, 1, 2]
    rng = np.random.default_rng(0)
    v = rng.normal(0, 1, (6, 3))
    out = plain.biased_attention(np.zeros((6, 2)), np.zeros((6, 2)), v, 1.0, math.log(2.0), None)
    p = 2.0 ** -np.arange(5, -1, -1.0)
    assert np.abs(out[5] - (p / p.sum()) @ v).max() < 1e-12
    # linear recurrence: with one decay everywhere, a sum over the past with powers of it
    q, k = rng.normal(0, 1, (6, 4)), rng.normal(0, 1, (6, 4))
    out = plain.linear_recurrence(q, k, v, np.full((6, 4), 0.5))
    want = sum(0.5 ** (5 - t) * (k[t] @ q[5]) * v[t] for t in range(6))
    assert np.abs(out[5] - want).max() < 1e-12
    # the delta rule: beta one and no decay replace what a key held
    key = np.tile([0.0, 1.0, 0.0, 0.0], (6, 1))
    assert np.abs(plain.delta_recurrence(key, key, v, np.ones((6, 4)), np.ones(6)) - v).max() < 1e-12
    # the exponential memory: the running maximum cancels; without it the same numbers as plain weights
    i_log, f_log = rng.normal(0, 1, 6), -rng.uniform(0.1, 1.0, 6)
    out = plain.mlstm_recurrence(q, k, v, i_log, f_log)
    for t in range(6):
        wts = [math.exp(i_log[s] + f_log[s + 1:t + 1].sum()) for s in range(t + 1)]
        num = sum(wts[s] * (k[s] @ q[t]) * v[s] for s in range(t + 1))
        den = sum(wts[s] * (k[s] @ q[t]) for s in range(t + 1))
        assert np.abs(out[t] - num / max(abs(den), 1.0)).max() < 1e-4                 # (1e-6 beside the divisor)
    x = rng.normal(0, 1, (2, 6))
    got = plain.group_rms_norm(x, np.full(6, 2.0), 3, 0.0)
    assert np.abs((got.reshape(2, 3, 2) ** 2).mean(-1) - 4.0).max() < 1e-12
    s = plain.sinusoids(4, 5)
    assert np.allclose(s[3], [math.sin(3), math.cos(3), math.sin(3 * 10000 ** -0.4), math.cos(3 * 10000 ** -0.4),
                              math.sin(3 * 10000 ** -0.8)])
