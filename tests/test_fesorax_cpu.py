"""Fesorax without a GPU: its configuration, its model description and tensor names (layers that read an earlier layer's
keys and values), pages of kept first tokens in the cache manager, the parts' parameters, and the oracle's own functions."""
import copy
import json
import math

import numpy as np
import pytest
import torch

from aegean_tge_b200 import ConfigError, architecture_of
from aegean_tge_b200.cache.manager import CacheManager
from aegean_tge_b200.config.model_spec import PartSpec, expected_tensors
from aegean_tge_b200.models.decoder import DecoderModel
from aegean_tge_b200.parts import FEED_FORWARDS, MIXERS, build_part
from aegean_tge_b200.parts.base import BuildEnv, PagedCacheSpec
from plain import fesorax_plain as plain

MOE = {"kind": "moe", "expert": {"ff": 12, "limit": 1.5}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 20, "limit": 0.5}}
ATT = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.4, "bias_max": 50.0,
                                      "mask": {"size": 30, "keep_first": 4}}, "mlp": MOE}
READ = {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3, "bias_max": 40.0,
                                       "mask": {"size": 50, "keep_first": 9}, "kv_from": 1}, "mlp": None}
MEM = {"type": "mlstm", "mixer": {"heads": 3, "dim": 6, "vdim": 10, "gate_cap": 11.0}, "mlp": MOE}
CONFIG = {"architecture": "Fesorax", "vocab": 60, "width": 24, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5}, "postln_alpha": 2.0,
          "layers": [MEM, ATT, READ, ATT]}


def _parse(raw):
    arch = architecture_of(raw)
    return arch, arch.parse_config(raw)


def _env(**kw):
    return BuildEnv(dtype=torch.float32, device=torch.device("cpu"), hidden_size=24, max_positions=64, page_size=16, ops=None, **kw)


def test_config_round_trip_and_description():
    arch, config = _parse(CONFIG)
    assert config.to_dict() == CONFIG
    spec = arch.build_spec(config)
    spec.validate()
    assert [layer.mixer.kind for layer in spec.layers] == ["matrix_lstm", "gqa_attention", "gqa_attention", "gqa_attention"]
    assert [layer.cache_from for layer in spec.layers] == [None, None, 1, None]
    assert all(layer.block == "post_norm" and layer.block_params == {"alpha": 2.0} for layer in spec.layers)
    attention = spec.layers[1].mixer.params
    assert attention["window"] == 30 and attention["keep_first"] == 4 and attention["distance_bias"] == {"far": 50.0}
    assert attention["qk_norm"] == {"scope": "head", "eps": 1e-5, "weight": False} and attention["head_gate"] and attention["own_kv"]
    assert not spec.layers[2].mixer.params["own_kv"] and spec.layers[2].mixer.params["keep_first"] == 9
    ffn = spec.layers[0].feed_forward.params
    assert (ffn["score"], ffn["weigh"], ffn["weights_over_sum"], ffn["limit"], ffn["shared"].params["limit"]) == ("logistic", "input", False, 1.5, 0.5)
    assert spec.embedding.params["scale"] == 1.5 and spec.head.weights["weight"] == "head"
    assert spec.layers[2].feed_forward is None and spec.layers[2].ffn_norm.params["optional"]
    names = set(expected_tensors(spec))
    assert {"embed", "head", "final.norm", "l0.mix.i", "l0.mix.i.b", "l0.mix.f.b", "l0.mix.norm", "l0.mlp.e4.gate", "l0.mlp.router", "l1.mix.rel",
            "l1.mix.g", "l1.mix.v", "l1.mlp.shared.down", "l2.mix.q", "l2.mix.rel", "l2.mix.g", "l2.mix.o", "l2.norm1", "l3.norm2"} <= names
    assert not names & {"l2.mix.k", "l2.mix.v", "l2.mlp.router", "l1.mix.q.norm", "l0.mlp.router.b"}
    planned = {name: shape for name, shape, _role, _draw in arch.random_plan(config)}
    assert set(planned) == names - {"l2.norm2"}                  # the one norm a checkpoint may lack
    assert planned["l1.mix.g"] == (4, 24) and planned["l0.mix.norm"] == (30,) and planned["l1.mix.v"] == (24, 24)
    assert planned["l1.mix.o"] == (24, 48) and planned["l0.mlp.e0.down"] == (24, 12)


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "delta"), (("layers", 0, "mixer", "gate_cap"), 0.0), (("layers", 0, "mixer", "heads"), None),
    (("layers", 0, "mlp", "kind"), "dense"), (("layers", 0, "mlp", "router", "top"), 6), (("layers", 0, "mlp", "router", "experts"), 2000),
    (("layers", 0, "mlp", "expert", "limit"), -1.0), (("layers", 0, "mlp", "shared"), {"ff": 4}), (("layers", 1, "mixer", "kv_heads"), 3),
    (("layers", 1, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "mask", "keep_first"), -1), (("layers", 1, "mixer", "mask"), 30),
    (("layers", 1, "mixer", "bias_max"), None), (("layers", 1, "mixer", "scale"), "big"), (("layers", 2, "mixer", "kv_from"), 2),
    (("layers", 2, "mixer", "kv_from"), 0), (("layers", 2, "mixer", "kv_from"), True), (("layers", 2, "mixer", "vdim"), 8),
    (("layers", 3, "mixer", "kv_from"), 2), (("postln_alpha",), None), (("norm",), {}), (("layers",), []), (("width",), None)])
def test_config_errors_name_the_key(path, value):
    raw = copy.deepcopy(CONFIG)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as error:
        _parse(raw)
    assert str(path[-1]) in str(error.value) or "layer" in str(error.value) or "limit" in str(error.value)


def test_what_a_model_may_leave_out():
    raw = json.loads(json.dumps(CONFIG))                  # layers that share no object
    del raw["embedding"], raw["layers"][0]["mlp"]["shared"], raw["layers"][1]["mixer"]["mask"]["keep_first"], raw["layers"][3]["mixer"]["mask"]
    arch, config = _parse(raw)
    assert config.embedding_scale == 1.0 and config.layers[0].mlp.shared is None and config.layers[1].mixer.mask.keep_first == 0
    spec = arch.build_spec(config)
    assert spec.layers[3].mixer.params["window"] is None and spec.layers[3].mixer.params["keep_first"] == 0
    assert "l0.mlp.shared.up" not in expected_tensors(spec)


def test_a_layer_keeps_what_its_readers_may_still_read():
    """Layer 2 reads layer 1's entries over a wider window and more kept tokens: their pages follow the wider of the two;
    layer 3 keeps a group of its own."""
    arch, config = _parse(CONFIG)
    model = DecoderModel(arch.build_spec(config), _env())
    manager = CacheManager(page_size=16, max_requests=2)
    model.declare_cache(manager)
    assert {(g.spec.window, g.spec.keep_first) for g in manager.groups} == {(50, 9), (30, 4)}
    assert manager.layer_group[1] != manager.layer_group[3] and 2 not in manager.layer_group
    manager.set_pool_sizes([8, 8])
    manager.allocate_storage(torch.float32, torch.device("cpu"))
    model.attach_cache(manager)
    assert not model.layer_caches[2].owner and model.layer_caches[2].group == manager.layer_group[1]
    assert model.layer_caches[2].paged["k"].data_ptr() == model.layer_caches[1].paged["k"].data_ptr()
    assert set(model.layer_caches[0].state) == {"state", "normaliser", "maximum"}
    # no mask on one side means every key stays
    full = PagedCacheSpec((("k", (1, 8)),), None)
    part = PagedCacheSpec((("k", (1, 8)),), 30, 1, 4)
    assert part.covering(full).window is None and full.covering(part).window is None and part.covering(part) == part
    with pytest.raises(ValueError):
        part.covering(PagedCacheSpec((("k", (2, 8)),), 30))


@pytest.mark.parametrize("keep,kept_pages", [(0, 0), (1, 1), (16, 1), (17, 2), (40, 3)])
def test_pages_of_kept_first_tokens_stay(keep, kept_pages):
    manager = CacheManager(page_size=16, max_requests=2)
    manager.add_layer(0, PagedCacheSpec((("k", (1, 8)),), 20, 1, keep), None)
    manager.set_pool_sizes([20])
    manager.admit("a")
    manager.grow("a", 200)
    manager.set_computed("a", 200)                        # the next query, at 200, sees 181 and later: pages 11 and 12
    table = manager.groups[0].tables["a"]
    assert [page >= 0 for page in table] == [True] * kept_pages + [False] * (11 - kept_pages) + [True, True]
    assert manager.groups[0].pool.free_count == 20 - kept_pages - 2
    manager.check()
    manager.free("a")
    assert manager.groups[0].pool.free_count == 20
    manager.check()
    with pytest.raises(Exception):
        manager.add_layer(1, PagedCacheSpec((("k", (1, 8)),), 20, 1, -3), None)


def test_parts_refuse_what_they_do_not_do():
    base = {"hidden_size": 24, "heads": 2, "kv_heads": 1, "head_dim": 8, "value_dim": 8, "position": PartSpec("none")}
    for extra in ({"keep_first": 4}, {"keep_first": -1, "window": 5}, {"head_gate": True, "qkv_bias": True},
                  {"own_kv": False, "values": "keys"}, {"head_gate": True, "short_conv": 3}, {"q_temp": {"coef": 1.0, "every": 2}}):
        with pytest.raises(ValueError):
            build_part(MIXERS, PartSpec("gqa_attention", {**base, **extra}), _env())
    part = build_part(MIXERS, PartSpec("gqa_attention", {**base, "head_gate": True, "own_kv": False, "window": 9, "keep_first": 2}), _env())
    assert set(part.param_specs()) == {"q.weight", "o.weight", "gate.weight"} and (16 + part.gate_rows) % 16 == 0
    assert part.decode_bytes(1000) == (9 + 2) * 16 * 4
    ffn = {"hidden_size": 24, "intermediate_size": 8, "experts": 4, "top": 2}
    for extra in ({"weigh": "input"}, {"activation": "clamped_glu"}, {"activation": "clamped_glu", "limit": 0.0}, {"score": "tanh"},
                  {"activation": "clamped_glu", "limit": 1.0, "weigh": "input", "identity": 2}):
        with pytest.raises((ValueError, KeyError)):
            build_part(FEED_FORWARDS, PartSpec("routed_experts", {**ffn, **extra}), _env())
    gated = build_part(FEED_FORWARDS, PartSpec("routed_experts", {**ffn, "activation": "clamped_glu", "limit": 1.0, "correction": False}), _env())
    assert len(gated.param_specs()) == 1 + 3 * 4 and gated.flops(1, 0.0) == 2.0 * (4 * 24 + 2 * 3 * 8 * 24)
    for extra in ({"gate_cap": 0.0}, {"head_dim": 0}, {"value_dim": 5000}, {"eps": 0.0}):
        with pytest.raises(ValueError):
            build_part(MIXERS, PartSpec("matrix_lstm", {"hidden_size": 24, "heads": 2, "head_dim": 8, "value_dim": 8, "gate_cap": 5.0, "eps": 1e-5,
                                                        **extra}), _env())


# ---------------------------------------------------------------------------
# the oracle's own functions
def test_oracle_mask():
    seen = [[j for j in range(12) if plain.sees(i, j, 3, 2)] for i in range(12)]
    assert seen[0] == [0] and seen[2] == [0, 1, 2] and seen[3] == [0, 1, 2, 3] and seen[4] == [0, 1, 2, 3, 4]
    assert seen[5] == [0, 1, 3, 4, 5] and seen[11] == [0, 1, 9, 10, 11]
    assert [j for j in range(9) if plain.sees(8, j, None, 0)] == list(range(9))


def test_oracle_attention_bias_and_visible_keys():
    k = np.zeros((6, 1, 2))
    v = np.arange(6, dtype=float).reshape(6, 1, 1)
    q = np.zeros((6, 1, 2))
    flat = np.zeros((4, 1))
    a = plain.attend(q, k, v, 1.0, flat, 9.0, 2, 1)               # equal scores: the mean of what is seen
    assert np.allclose(a[:, 0, 0], [0, 0.5, 1.0, 5 / 3, 7 / 3, 3.0])
    bias = np.array([[0.0], [50.0], [0.0], [0.0]])                # distance 1 outweighs everything
    a = plain.attend(q, k, v, 1.0, bias, 9.0, 3, 0)
    assert np.allclose(a[1:, 0, 0], v[:5, 0, 0])


def test_oracle_memory_writes_reads_and_forgets():
    d, dv = 4, 3
    e = np.eye(d)
    k, q = np.stack([e[0], e[1], e[0]]), np.stack([e[0], e[0], e[0]])
    v = np.arange(9, dtype=float).reshape(3, dv) + 1.0
    zero = np.zeros(3)
    o = plain.mlstm_memory(q, k, v, zero, zero)                   # open forget gates, unit writes: the mean of the key's values
    assert np.allclose(o[0], v[0]) and np.allclose(o[1], v[0]) and np.allclose(o[2], (v[0] + v[2]) / 2, atol=1e-5)
    small = plain.mlstm_memory(q[:1], k[:1], v[:1], np.array([-3.0]), np.array([-50.0]))
    # the maximum starts at 0, f pulls it to -3 at most: the floor of the denominator is exp(3), the write 1
    assert np.allclose(small[0], v[0] / (math.exp(3.0) + 1e-6))
    kept = plain.mlstm_memory(q[:1], k[:1], v[:1], np.array([-3.0]), np.array([0.0]))
    assert np.allclose(kept[0], math.exp(-3.0) * v[0] / (1.0 + 1e-6))
    late = plain.mlstm_memory(q, k, v, np.array([0.0, 0.0, 9.0]), zero)
    assert np.allclose(late[2], v[2], atol=1e-2)                  # a strong late write outweighs the earlier one


def test_oracle_router_and_experts():
    W = {"m.router": np.array([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]])}
    ids, w = plain.route(np.array([[2.0, 1.0]]), W, "m.", 2)
    assert ids.tolist() == [[2, 0]] and np.allclose(w, [[1 / (1 + math.exp(-3.0)), 1 / (1 + math.exp(-2.0))]])
    margins = []
    ids, w = plain.route(np.array([[2.0, 1.0]]), W, "m.", 1, margins, np.array([[1]]))
    assert ids.tolist() == [[1]] and np.allclose(w, [[1 / (1 + math.exp(-1.0))]]) and np.allclose(margins[0], [1.0 - 3.0])
    W.update({f"m.e{e}.{t}": np.eye(2) * (e + 1.0) for e in range(3) for t in ("gate", "up", "down")})
    h = np.array([[2.0, 1.0]])
    mlp = {"expert": {"limit": 1.5}, "router": {"experts": 3, "top": 1}}
    s = 1 / (1 + math.exp(-3.0))
    g = np.minimum(3.0 * s * h, 1.5)
    want = 3.0 * g / (1 + np.exp(-1.702 * g)) * (np.clip(3.0 * s * h, -1.5, 1.5) + 1.0)
    assert np.allclose(plain.moe_ff(h, W, "m.", mlp), want)       # the weight inside, not outside
    i, f = plain.mlstm_gates(np.array([[100.0]]), {"x.i": np.ones((1, 1)), "x.i.b": np.zeros(1), "x.f": -np.ones((1, 1)), "x.f.b": np.zeros(1)},
                             "x.", 5.0)
    assert np.allclose(i, 5.0) and np.allclose(f, -math.log(1 + math.exp(5.0)))
