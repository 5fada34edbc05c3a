"""The Fesorax decoder as a ModelSpec, and its random weights.

The stream starts from scaled embeddings; every layer normalises after its sums: x <- rms(a x + mixer(x)) g1, then
x <- rms(a x + mlp(x)) g2, the sublayers reading the stream itself (block ``post_norm``); the head has a matrix of its own.

Mixers: "attention" is ``gqa_attention`` on its separate path: q and k over their root mean square per head (no weight), a
learned bias by distance, a window beside which the first tokens stay visible, one gate per head; a layer with
``kv_from`` has neither key nor value projection and reads the named layer's cache (``LayerSpec.cache_from``).  "mlstm" is
``matrix_lstm``.  The feed-forward is ``routed_experts`` with logistic scores that multiply the inputs of clamped gated
experts, and a ``clamped_glu`` that every token uses.

Checkpoint tensor names: ``embed``, ``head``, ``final.norm``; per layer i ``l<i>.norm1``, ``l<i>.norm2``; attention
``l<i>.mix.{q,k,v,g,o,rel}`` (g: one row per head); mlstm ``l<i>.mix.{q,k,v,g,i,f,o,norm}``, ``l<i>.mix.{i,f}.b``; experts
``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.router``, ``l<i>.mlp.shared.{gate,up,down}``.
"""
from __future__ import annotations

from typing import Iterator, Optional, Tuple

from ..config.fesorax import ARCHITECTURE, Attention, FesoraxConfig, MatrixMemory
from ..config.model_spec import LayerSpec, ModelSpec, PartSpec
from ..registry import Architecture, register_architecture
from ..weights.draws import Draw, normal, uniform

NO_POSITION_LIMIT = 2 ** 31 - 1      # the design states no longest sequence
SWISH_ALPHA, UP_OFFSET = 1.702, 1.0  # the gate is g sigmoid(1.702 g) (u + 1)


def rel_rows(bias_max: float) -> int:
    """Rows of the bias by distance in models drawn at random (a checkpoint's table brings its own count)."""
    return 32 if bias_max >= 64.0 else 16


def _norm(config: FesoraxConfig, name: str, optional: bool = False) -> PartSpec:
    params = {"size": config.width, "eps": config.eps}
    if optional:
        params["optional"] = True
    return PartSpec("rmsnorm", params, {"weight": name})


def _attention(config: FesoraxConfig, m: Attention, prefix: str) -> PartSpec:
    params = {"hidden_size": config.width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
              "scale": m.scale, "position": PartSpec("none"), "qk_norm": {"scope": "head", "eps": config.eps, "weight": False},
              "distance_bias": {"far": m.bias_max}, "head_gate": True, "own_kv": m.kv_from is None,
              "window": None if m.mask is None else m.mask.size, "keep_first": 0 if m.mask is None else m.mask.keep_first}
    weights = {"q.weight": prefix + "q", "o.weight": prefix + "o", "gate.weight": prefix + "g", "rel": prefix + "rel"}
    if m.kv_from is None:
        weights.update({"k.weight": prefix + "k", "v.weight": prefix + "v"})
    return PartSpec("gqa_attention", params, weights)


def _matrix_memory(config: FesoraxConfig, m: MatrixMemory, prefix: str) -> PartSpec:
    params = {"hidden_size": config.width, "heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "gate_cap": m.gate_cap,
              "eps": config.eps}
    weights = {f"{t}.weight": prefix + t for t in ("q", "k", "v", "g", "i", "f", "o", "norm")}
    weights.update({"i.bias": prefix + "i.b", "f.bias": prefix + "f.b"})
    return PartSpec("matrix_lstm", params, weights)


def _feed_forward(config: FesoraxConfig, n: int) -> Optional[PartSpec]:
    mlp, prefix = config.layers[n].mlp, f"l{n}.mlp."
    if mlp is None:
        return None
    weights = {"router.weight": prefix + "router"}
    for e in range(mlp.experts):
        for t in ("gate", "up", "down"):
            weights[f"experts.{e}.{t}.weight"] = f"{prefix}e{e}.{t}"
    shared = None
    if mlp.shared is not None:
        shared = PartSpec("clamped_glu", {"hidden_size": config.width, "intermediate_size": mlp.shared.ff, "limit": mlp.shared.limit,
                                          "alpha": SWISH_ALPHA, "up_offset": UP_OFFSET})
        weights.update({f"shared.{t}.weight": f"{prefix}shared.{t}" for t in ("gate", "up", "down")})
    return PartSpec("routed_experts", {"hidden_size": config.width, "intermediate_size": mlp.expert.ff, "experts": mlp.experts,
                                       "top": mlp.top, "activation": "clamped_glu", "limit": mlp.expert.limit,
                                       "alpha": SWISH_ALPHA, "up_offset": UP_OFFSET, "correction": False, "score": "logistic",
                                       "weights_over_sum": False, "weigh": "input", "shared": shared}, weights)


def build_spec(config: FesoraxConfig) -> ModelSpec:
    layers = []
    for n, layer in enumerate(config.layers):
        prefix = f"l{n}.mix."
        if isinstance(layer.mixer, Attention):
            mixer, source = _attention(config, layer.mixer, prefix), layer.mixer.kv_from
        else:
            mixer, source = _matrix_memory(config, layer.mixer, prefix), None
        ffn = _feed_forward(config, n)
        # a layer without feed-forward has no second sum to normalise; should a checkpoint hold a second norm for it all
        # the same, it is applied to the scaled stream alone
        norm2 = _norm(config, f"l{n}.norm2", optional=ffn is None)
        layers.append(LayerSpec("post_norm", mixer, ffn, _norm(config, f"l{n}.norm1"), norm2, cache_from=source,
                                block_params={"alpha": config.alpha}))
    sizes = {"vocab_size": config.vocab, "hidden_size": config.width}
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=config.width, vocab_size=config.vocab, max_positions=NO_POSITION_LIMIT,
        layers=tuple(layers), schedule=tuple(range(len(layers))),
        embedding=PartSpec("token_embedding", {**sizes, "scale": config.embedding_scale}, {"weight": "embed"}),
        final_norm=_norm(config, "final.norm"),
        head=PartSpec("linear_head", sizes, {"weight": "head"}))


def random_plan(config: FesoraxConfig) -> Iterator[Tuple[str, Tuple[int, ...], str, Draw]]:
    """(name, shape, role, draw) of every checkpoint tensor.  Projections N(0, 1/sqrt(fan-in)), norm weights 1 + U(-0.1,
    0.1), the bias by distance N(0, 0.5), input gates' biases U(-1, 1), forget gates' biases U(2, 5) (memories of ten to a
    hundred tokens)."""
    w = config.width
    yield "embed", (config.vocab, w), "matrix", normal(1.0)
    for n, layer in enumerate(config.layers):
        p, m = f"l{n}.", layer.mixer
        q = p + "mix."
        yield p + "norm1", (w,), "vector", uniform(0.9, 1.1)
        if layer.mlp is not None:
            yield p + "norm2", (w,), "vector", uniform(0.9, 1.1)
        yield q + "q", (m.heads * m.dim, w), "matrix", normal(w ** -0.5)
        if isinstance(m, Attention):
            if m.kv_from is None:
                yield q + "k", (m.kv_heads * m.dim, w), "matrix", normal(w ** -0.5)
                yield q + "v", (m.kv_heads * m.vdim, w), "matrix", normal(w ** -0.5)
            yield q + "rel", (rel_rows(m.bias_max), m.heads), "vector", normal(0.5)
            yield q + "g", (m.heads, w), "matrix", normal(w ** -0.5)
        else:
            yield q + "k", (m.heads * m.dim, w), "matrix", normal(w ** -0.5)
            yield q + "v", (m.heads * m.vdim, w), "matrix", normal(w ** -0.5)
            yield q + "g", (m.heads * m.vdim, w), "matrix", normal(w ** -0.5)
            yield q + "norm", (m.heads * m.vdim,), "vector", uniform(0.9, 1.1)
            for t, low, high in (("i", -1.0, 1.0), ("f", 2.0, 5.0)):
                yield q + t, (m.heads, w), "matrix", normal(0.5 * w ** -0.5)
                yield f"{q}{t}.b", (m.heads,), "vector", uniform(low, high)
        yield q + "o", (w, m.heads * m.vdim), "matrix", normal((m.heads * m.vdim) ** -0.5)
        if layer.mlp is not None:
            r = layer.mlp
            yield p + "mlp.router", (r.experts, w), "matrix", normal(w ** -0.5)
            blocks = [(f"e{e}", r.expert.ff) for e in range(r.experts)] + ([("shared", r.shared.ff)] if r.shared is not None else [])
            for name, ff in blocks:
                yield f"{p}mlp.{name}.gate", (ff, w), "matrix", normal(w ** -0.5)
                yield f"{p}mlp.{name}.up", (ff, w), "matrix", normal(w ** -0.5)
                yield f"{p}mlp.{name}.down", (w, ff), "matrix", normal(ff ** -0.5)
    yield "final.norm", (w,), "vector", uniform(0.9, 1.1)
    yield "head", (config.vocab, w), "matrix", normal(w ** -0.5)


register_architecture(Architecture(name=ARCHITECTURE, parse_config=FesoraxConfig.from_dict, build_spec=build_spec,
                                   random_plan=random_plan))
