"""Tazizen without a GPU: its configuration, its model description and tensor names (layers passed several times, a cache per
pass), the parts' parameters, the rotation's tables, and the oracle's own functions."""
import json
import math

import numpy as np
import pytest
import torch

from aegean_tge_b200 import ConfigError, architecture_of
from aegean_tge_b200.cache.manager import CacheManager
from aegean_tge_b200.config.model_spec import PartSpec, expected_tensors
from aegean_tge_b200.models.decoder import DecoderModel
from aegean_tge_b200.parts import BLOCKS, EMBEDDINGS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS, build_part
from aegean_tge_b200.parts.base import BuildEnv
from aegean_tge_b200.parts.rope import rotary_tables
from plain import tazizen_plain as plain

MOE = {"kind": "moe", "expert": {"ff": 12}, "shared": {"ff": 20},
       "router": {"experts": 6, "top": 2, "scale": 1.5, "groups": {"count": 3, "keep": 2}}}
ATT = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.4, "mask": {"size": 30},
                                      "rot": {"base": 5000.0, "dims": 6,
                                              "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}}}, "mlp": MOE}
LAT = {"type": "latent_attention", "mixer": {"heads": 3, "dim": 10, "rot_dim": 4, "vdim": 6, "q_rank": 14, "kv_rank": 9, "scale": 0.3,
                                             "mask": {"size": 50}, "rot": {"base": 700.0, "dims": 4}}, "mlp": MOE}
BARE = {"type": "latent_attention", "mixer": LAT["mixer"], "mlp": None}
CONFIG = {"architecture": "Tazizen", "vocab": 60, "width": 24, "streams": 3, "norm": {"eps": 1e-5}, "layers": [ATT, LAT, BARE, ATT],
          "loop": {"start": 1, "stop": 3, "times": 3}}


def _parse(raw):
    arch = architecture_of(raw)
    return arch, arch.parse_config(json.loads(json.dumps(raw)))


def _env(**kw):
    return BuildEnv(dtype=torch.float32, device=torch.device("cpu"), hidden_size=24, max_positions=64, page_size=16, ops=None, **kw)


def test_config_round_trip_and_description():
    arch, config = _parse(CONFIG)
    assert json.loads(json.dumps(config.to_dict())) == CONFIG
    spec = arch.build_spec(config)
    spec.validate()
    assert config.run_order() == (0, 1, 2, 1, 2, 1, 2, 3) == tuple(plain.run_order(CONFIG))
    # four layers of the file, then the borrowed ones of the second and third pass
    assert spec.schedule == (0, 1, 2, 4, 5, 6, 7, 3)
    assert [layer.weights_from for layer in spec.layers] == [None] * 4 + [1, 2, 1, 2]
    assert all(layer.block == "hyper_connected" and layer.cache_from is None for layer in spec.layers)
    attention, latent = spec.layers[0].mixer.params, spec.layers[1].mixer.params
    assert attention["window"] == 30 and attention["sink_score"] == 0.0 and attention["output_gate"]
    assert attention["qk_norm"] == {"scope": "head", "eps": 1e-5, "weight": False, "after_rotation": True}
    assert attention["position"].params["stretch"] == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 0.5}
    assert latent["window"] == 50 and latent["gate"] == "none" and latent["position"].kind == "rope_neox"
    ffn = spec.layers[0].feed_forward.params
    assert (ffn["score"], ffn["group_value"], ffn["weights_scale"], ffn["shared_gate"], ffn["activation"]) == ("logistic", "two_best", 1.5, True, "swiglu")
    assert spec.embedding.params["streams"] == 3 and not spec.final_norm.params["connected"] and spec.head.weights["weight"] == "head"
    assert spec.layers[2].feed_forward is None and spec.layers[2].ffn_norm.params["optional"]
    names = set(expected_tensors(spec))
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.hc1.in", "l0.hc1.mix", "l0.hc2.out", "l0.mix.q", "l0.mix.g", "l0.mlp.e5.gate",
            "l0.mlp.correction", "l0.mlp.shared.sg", "l1.mix.dq.norm", "l1.mix.dkv", "l1.mix.uv", "l2.mix.o"} <= names
    assert not names & {"l0.mix.dq", "l1.mix.g", "l1.mix.q", "l2.mlp.router", "l0.mix.q.norm", "l4.norm1"}
    planned = {name: shape for name, shape, _role, _draw in arch.random_plan(config)}
    assert set(planned) == names - {"l2.norm2", "l2.hc2.in", "l2.hc2.mix", "l2.hc2.out"}      # what a checkpoint may lack
    assert planned["l0.mix.g"] == (48, 24) and planned["l1.mix.uq"] == (42, 14) and planned["l1.mix.dkv"] == (13, 24)
    assert planned["l0.hc1.mix"] == (3, 3) and planned["l0.mlp.shared.sg"] == (1, 24)


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "mlstm"), (("layers", 0, "mixer", "heads"), 0), (("layers", 0, "mixer", "kv_heads"), 3),
    (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "mask"), 30), (("layers", 0, "mixer", "scale"), None),
    (("layers", 0, "mixer", "rot", "dims"), 5), (("layers", 0, "mixer", "rot", "dims"), 10), (("layers", 0, "mixer", "rot", "base"), -2.0),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0), (("layers", 0, "mixer", "rot", "scaling", "original"), None),
    (("layers", 1, "mixer", "rot", "dims"), 6), (("layers", 1, "mixer", "kv_rank"), "9"), (("layers", 1, "mixer", "q_rank"), 0),
    (("layers", 0, "mlp", "kind"), "dense"), (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "router", "experts"), 2001),
    (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 0, "mlp", "router", "groups", "keep"), 4),
    (("layers", 0, "mlp", "expert", "ff"), None), (("layers", 0, "mlp", "shared"), {"limit": 4}), (("streams",), 0), (("streams",), 17),
    (("streams",), None), (("loop", "stop"), 5), (("loop", "start"), 3), (("loop", "times"), 0), (("norm",), {}), (("layers",), []),
    (("width",), None)])
def test_config_errors_name_the_key(path, value):
    raw = json.loads(json.dumps(CONFIG))
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as error:
        _parse(raw)
    assert any(str(word) in str(error.value) for word in (path[-1], "layer", "groups", "ff"))


def test_what_a_model_may_leave_out():
    raw = json.loads(json.dumps(CONFIG))
    del raw["loop"], raw["layers"][0]["mlp"]["shared"], raw["layers"][0]["mlp"]["router"]["groups"], raw["layers"][0]["mixer"]["mask"]
    del raw["layers"][0]["mixer"]["rot"]["scaling"], raw["layers"][1]["mixer"]["rot"], raw["layers"][0]["mlp"]["router"]["scale"]
    arch, config = _parse(raw)
    spec = arch.build_spec(config)
    assert spec.schedule == (0, 1, 2, 3) and spec.layers[0].mixer.params["window"] is None
    assert "stretch" not in spec.layers[0].mixer.params["position"].params and spec.layers[1].mixer.params["position"].kind == "none"
    ffn = spec.layers[0].feed_forward.params
    assert (ffn["group_count"], ffn["group_keep"], ffn["weights_scale"], ffn["shared"], ffn["shared_gate"]) == (1, 1, 1.0, None, False)
    assert not {"l0.mlp.shared.up", "l0.mlp.shared.sg"} & set(expected_tensors(spec))
    assert _parse(config.to_dict())[1] == config


def test_every_pass_keeps_a_cache_of_its_own():
    arch, config = _parse(CONFIG)
    model = DecoderModel(arch.build_spec(config), _env())
    assert model.graph_safe and model.blocks[4] is model.blocks[1]
    manager = CacheManager(page_size=16, max_requests=2)
    model.declare_cache(manager)
    assert sorted(g.spec.window for g in manager.groups) == [30, 50]
    manager.set_pool_sizes([8, 8])
    manager.allocate_storage(torch.float32, torch.device("cpu"))
    model.attach_cache(manager)
    entries = [model.layer_caches[n].paged["kv"].data_ptr() for n in (1, 2, 4, 5, 6, 7)]
    assert len(set(entries)) == 6 and model.layer_caches[1].paged["kv"].shape[1:] == (1, 16, 13)
    assert model.layer_caches[0].paged["v"].shape[1:] == (2, 16, 12)
    # a step's parameters: looped layers count once per pass
    once = json.loads(json.dumps(CONFIG))
    del once["loop"]
    single = DecoderModel(arch.build_spec(arch.parse_config(once)), _env())
    assert model.step_param_bytes() > single.step_param_bytes() and model.weight_bytes() == single.weight_bytes()


def test_parts_refuse_what_they_do_not_do():
    base = {"hidden_size": 24, "heads": 2, "kv_heads": 1, "head_dim": 8, "value_dim": 8, "position": PartSpec("none")}
    after = {"scope": "head", "eps": 1e-5, "weight": False, "after_rotation": True}
    for extra in ({"output_gate": True, "head_gate": True}, {"sinks": True, "sink_score": 0.0}, {"output_gate": True, "values": "keys"},
                  {"output_gate": True, "window": 9, "pool": 4}, {"output_gate": True, "distance_bias": {"far": 40.0}},
                  {"output_gate": True, "qkv_bias": True}, {"qk_norm": dict(after, scope="projection")},
                  {"qk_norm": after, "window": 9, "keep_first": 2}, {"qk_norm": dict(after, after_rotation=False), "output_gate": True}):
        with pytest.raises(ValueError):
            build_part(MIXERS, PartSpec("gqa_attention", {**base, **extra}), _env())
    part = build_part(MIXERS, PartSpec("gqa_attention", {**base, "qk_norm": after, "output_gate": True, "sink_score": 0.0, "window": 9}), _env())
    assert set(part.param_specs()) == {"q.weight", "k.weight", "v.weight", "o.weight", "gate.weight"}
    assert (16 + 8 + 8 + part.gate_rows) % 16 == 0 and part.decode_bytes(1000) == 9 * 16 * 4
    # a whole prompt of 20 tokens over a window of 9: 9 * 20 - 36 pairs
    assert part.flops(20, 210.0) - part.flops(20, 0.0) == pytest.approx(2.0 * 2 * 16 * (9 * 20 - 36))
    latent = {"hidden_size": 24, "heads": 2, "head_dim": 8, "rope_dim": 4, "value_dim": 8, "q_rank": 8, "kv_rank": 12, "scale": 1.0, "eps": 1e-5}
    for extra in ({"window": 0}, {"kv_rank": 640}):
        with pytest.raises(ValueError):
            build_part(MIXERS, PartSpec("latent_attention", {**latent, **extra}), _env())
    wide = build_part(MIXERS, PartSpec("latent_attention", {**latent, "kv_rank": 600, "window": 7}), _env())
    assert wide.cache_spec().window == 7 and wide.first_read(20) == 14 and wide.first_read(3) == 0
    ffn = {"hidden_size": 24, "intermediate_size": 8, "experts": 4, "top": 2}
    for extra in ({"shared_gate": True}, {"group_value": "mean"}, {"activation": "gelu"}):
        with pytest.raises(ValueError):
            build_part(FEED_FORWARDS, PartSpec("routed_experts", {**ffn, **extra}), _env())
    for extra in ({"streams": 0}, {"streams": 17}, {"eps": 0.0}):
        with pytest.raises(ValueError):
            build_part(NORMS, PartSpec("connected_rmsnorm", {"size": 24, "eps": 1e-5, "streams": 2, **extra}), _env())
    for stretch in ({"factor": 0.0}, {"slow": -1.0}):
        params = {"head_dim": 8, "theta": 100.0, "precise": True, "stretch": {"factor": 2.0, "fast": 8.0, "slow": 1.0, "original": 64.0, **stretch}}
        with pytest.raises(ValueError):
            build_part(POSITIONS, PartSpec("rope_neox", params), _env())
    with pytest.raises(ValueError):
        build_part(EMBEDDINGS, PartSpec("token_embedding", {"vocab_size": 9, "hidden_size": 8, "streams": 2,
                                                            "norm": PartSpec("group_rmsnorm", {"size": 8, "eps": 1e-5})}), _env())
    plain_norm = build_part(NORMS, PartSpec("rmsnorm", {"size": 24, "eps": 1e-5}), _env())
    with pytest.raises(ValueError):
        BLOCKS.get("hyper_connected")(part, None, plain_norm, None, _env())


def test_a_shared_feed_forward_joins_the_experts_matrices():
    spec = PartSpec("routed_experts", {"hidden_size": 24, "intermediate_size": 8, "experts": 3, "top": 2, "activation": "swiglu",
                                       "score": "logistic", "shared_gate": True,
                                       "shared": PartSpec("swiglu", {"hidden_size": 24, "intermediate_size": 10})})
    part = build_part(FEED_FORWARDS, spec, _env())
    gen = torch.Generator().manual_seed(1)
    tensors = {name: torch.randn(param.shape, generator=gen) for name, param in part.param_specs().items()}
    part.load(tensors)
    assert part.shared_inner == 10 and part.up_rows.shape == (2 * (3 * 8 + 10), 24) and part.down_columns.shape == (24, 34)
    assert torch.equal(part.w_up[2][0::2], tensors["experts.2.gate.weight"]) and torch.equal(part.w_up[2][1::2], tensors["experts.2.up.weight"])
    assert torch.equal(part.w_down[:, 1, :], tensors["experts.1.down.weight"])
    assert torch.equal(part.shared.w_gate_up[0::2], tensors["shared.gate.weight"]) and torch.equal(part.shared.w_down, tensors["shared.down.weight"])
    assert part.w_up.data_ptr() == part.up_rows.data_ptr() and part.shared.w_down.data_ptr() > part.down_columns.data_ptr()
    assert torch.equal(part.w_router[3:4], tensors["shared_gate.weight"]) and part.w_router.shape[0] % 4 == 0
    assert part.takes_deferred_at(4) and not part.takes_deferred_at(1) and not part.takes_deferred_at(1000)


# ---------------------------------------------------------------------------
# tables, and the oracle's own functions
@pytest.mark.parametrize("base,dims,factor,original,fast,slow", [(10000.0, 64, 4.0, 512, 32.0, 1.0), (500.0, 12, 8.0, 100, 4.0, 0.25),
                                                                 (250000.0, 32, 40.0, 4096, 32.0, 1.0), (3.0, 8, 2.0, 10, 3.0, 2.9),
                                                                 (0.5, 6, 1.0, 64, 2.0, 1.0), (70.0, 2, 16.0, 9, 64.0, 32.0)])
def test_stretched_tables(base, dims, factor, original, fast, slow):
    rot = {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    f, m = plain.frequencies(rot), plain.amplitude(rot)
    cos, sin = rotary_tables(base, dims, 200, precise=True, stretch=(factor, fast, slow, original))
    angle = np.arange(200)[:, None] * f[None, :]
    assert np.abs(cos.double().numpy() - m * np.cos(angle)).max() < 1e-6 and np.abs(sin.double().numpy() - m * np.sin(angle)).max() < 1e-6
    bare = plain.frequencies({"base": base, "dims": dims})
    assert np.all(f <= bare * 1.0000001) and np.all(f >= bare / factor * 0.9999999)


def test_stretch_keeps_fast_pairs_and_slows_slow_ones():
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    f, bare = plain.frequencies(rot), plain.frequencies({"base": 10000.0, "dims": 64})
    turns = 2048 * bare / (2 * math.pi)
    assert np.allclose(f[turns > 45], bare[turns > 45]) and np.allclose(f[turns < 0.6], bare[turns < 0.6] / 8.0)
    between = (turns < 20) & (turns > 1.5)
    assert np.all(f[between] < bare[between]) and np.all(f[between] > bare[between] / 8.0)


def test_oracle_streams():
    X = np.array([[[1.0, 2.0], [10.0, 20.0]]])                         # one token, two streams of width 2
    assert np.allclose(plain.streams_in(X, np.array([0.5, -1.0])), [[-9.5, -19.0]])
    mix = np.array([[1.0, 2.0], [3.0, 4.0]])                           # from the first stream: 1 to the first, 2 to the second
    Y = plain.streams_out(X, np.array([[100.0, 0.0]]), mix, np.array([1.0, -1.0]))
    assert np.allclose(Y, [[[1 + 30 + 100.0, 2 + 60.0], [2 + 40 - 100.0, 4 + 80.0]]])


def test_oracle_window_and_extra_one():
    q, k = np.zeros((5, 1, 2)), np.zeros((5, 1, 2))
    v = np.arange(5, dtype=float).reshape(5, 1, 1)
    assert np.allclose(plain.window_attention(q, k, v, 1.0, 2, 0.0)[:, 0, 0], [0, 0.5, 1.5, 2.5, 3.5])
    assert np.allclose(plain.window_attention(q, k, v, 1.0, 2, 1.0)[:, 0, 0], [0, 1 / 3, 1.0, 5 / 3, 7 / 3])
    assert np.allclose(plain.window_attention(q, k, v, 1.0, None, 0.0)[:, 0, 0], [0, 0.5, 1.0, 1.5, 2.0])
    big = np.full((1, 1, 2), 50.0)                                     # scores far above and far below the extra one
    assert np.allclose(plain.window_attention(big, big, v[4:], 1.0, 1, 1.0), 4.0)
    assert np.allclose(plain.window_attention(big, -big, v[4:], 1.0, 1, 1.0), 0.0)


def test_oracle_rotation_in_halves():
    rot = {"base": 100.0, "dims": 4}
    x = np.arange(1.0, 7.0).reshape(1, 6)
    y = plain.rotate_halves(x, rot, first_position=3)[0]
    for i, f in enumerate((1.0, 0.1)):
        a = 3 * f
        assert np.allclose([y[i], y[i + 2]], [x[0, i] * math.cos(a) - x[0, i + 2] * math.sin(a), x[0, i + 2] * math.cos(a) + x[0, i] * math.sin(a)])
    assert np.array_equal(y[4:], x[0, 4:])


def test_oracle_router():
    # scores are the logistic function of the input; groups of two, valued by both together
    z = np.array([[3.0, -3.0, 1.0, 0.9, 2.0, -9.0]])
    s = plain.sigmoid(z)
    none = np.zeros(6)
    ids, w = plain.route(z, np.eye(6), none, 2, 3, 1, 2.0)
    assert ids.tolist() == [[2, 3]] and np.allclose(w, 2.0 * s[:, 2:4] / s[:, 2:4].sum())     # not the group with the largest score
    # negative choice scores: those outside the kept groups lie below them all the same
    ids, _ = plain.route(z, np.eye(6), none - 5.0, 2, 3, 1, 1.0)
    assert ids.tolist() == [[2, 3]]
    # the correction steers the choice, not the weights
    ids, w = plain.route(z, np.eye(6), np.array([0, 0, 0, 0, 0, 1.5]), 2, 3, 1, 1.0)
    assert ids.tolist() == [[5, 4]] and np.allclose(w[0], s[0, [5, 4]] / s[0, [5, 4]].sum())
    assert plain.group_values(np.array([1.0, 2.0, 3.0]), 3).tolist() == [1.0, 2.0, 3.0]       # groups of one
    margins = []
    plain.route(z, np.eye(6), none, 1, 3, 2, 1.0, margins)
    values = np.sort(plain.group_values(s[0], 3))[::-1]
    assert np.allclose(margins, [min(values[1] - values[2], s[0, 0] - s[0, 2])])
    margins = []
    ids, _ = plain.route(z, np.eye(6), none, 2, 3, 1, 1.0, margins, np.array([[0, 1]]))
    assert ids.tolist() == [[0, 1]] and np.allclose(margins, [s[0, :2].sum() - s[0, 2:4].sum()])
