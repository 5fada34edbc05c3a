"""The Tazizen decoder as a ModelSpec, and its random weights.

The residual is several streams per token (block ``hyper_connected``, norms ``connected_rmsnorm`` with weights stored around
zero): all of them the embedding at the start, added up before the final norm.  A run of layers may be passed several times,
every pass a borrowed layer with a cache of its own.

Mixers: "attention" is ``gqa_attention`` on its general path (rotation in halves, its frequencies stretched for long
contexts; q and k over their root mean square after it, without weights; a sliding window; a sink of constant score 0; one
gate per number of the output).  "latent_attention" is ``latent_attention`` with a window and a rotation in halves.  The
feed-forward is ``routed_experts`` with logistic scores, a corrected choice inside groups valued by their two best, and gated
experts beside a gated feed-forward that every token uses, times one gate per token.

Checkpoint tensor names: ``embed``, ``head``, ``final.norm``; per layer i ``l<i>.norm{1,2}``, ``l<i>.hc{1,2}.{in,mix,out}``;
attention ``l<i>.mix.{q,k,v,g,o}``; latent attention ``l<i>.mix.{dq,uq,dkv,uk,uv,o}``, ``l<i>.mix.{dq,dkv}.norm``; experts
``l<i>.mlp.router``, ``l<i>.mlp.correction``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down,sg}``.
"""
from __future__ import annotations

from typing import Dict, Iterator, List, Optional, Tuple

from ..config.model_spec import LayerSpec, ModelSpec, PartSpec
from ..config.tazizen import ARCHITECTURE, Attention, LatentAttention, Rotation, TazizenConfig
from ..registry import Architecture, register_architecture
from ..weights.draws import Draw, normal, uniform

NO_POSITION_LIMIT = 2 ** 31 - 1      # the design states no longest sequence
SINK_SCORE = 0.0                     # the one added to the softmax's denominator is exp(0)


def _norm(config: TazizenConfig, layer: int, sublayer: int, optional: bool = False) -> PartSpec:
    prefix = f"l{layer}.hc{sublayer}."
    params = {"size": config.width, "eps": config.eps, "streams": config.streams, "unit_offset": True}
    if optional:
        params["optional"] = True
    return PartSpec("connected_rmsnorm", params, {"weight": f"l{layer}.norm{sublayer}", "in": prefix + "in", "mix": prefix + "mix",
                                                  "out": prefix + "out"})


def _position(rot: Optional[Rotation], width: int) -> PartSpec:
    if rot is None:
        return PartSpec("none")
    params = {"head_dim": width, "theta": rot.base, "rotary_dim": rot.dims, "precise": True}
    if rot.scaling is not None:
        params["stretch"] = rot.scaling.to_dict()
    return PartSpec("rope_neox", params)


def _attention(config: TazizenConfig, m: Attention, prefix: str) -> PartSpec:
    params = {"hidden_size": config.width, "heads": m.heads, "kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
              "scale": m.scale, "window": m.window, "position": _position(m.rot, m.dim), "sink_score": SINK_SCORE,
              "qk_norm": {"scope": "head", "eps": config.eps, "weight": False, "after_rotation": True}, "output_gate": True}
    weights = {f"{t}.weight": prefix + t for t in ("q", "k", "v", "o")}
    return PartSpec("gqa_attention", params, {**weights, "gate.weight": prefix + "g"})


def _latent(config: TazizenConfig, m: LatentAttention, prefix: str) -> PartSpec:
    params = {"hidden_size": config.width, "heads": m.heads, "head_dim": m.dim, "rope_dim": m.rot_dim, "value_dim": m.vdim,
              "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale, "eps": config.eps, "gate": "none", "window": m.window,
              "position": _position(m.rot, m.rot_dim)}
    weights = {f"{t}.weight": prefix + t for t in ("dq", "uq", "dkv", "uk", "uv", "o")}
    return PartSpec("latent_attention", params, {**weights, "dq_norm.weight": prefix + "dq.norm", "dkv_norm.weight": prefix + "dkv.norm"})


def _feed_forward(config: TazizenConfig, n: int) -> Optional[PartSpec]:
    mlp, prefix = config.layers[n].mlp, f"l{n}.mlp."
    if mlp is None:
        return None
    weights = {"router.weight": prefix + "router", "correction": prefix + "correction"}
    for e in range(mlp.experts):
        for t in ("gate", "up", "down"):
            weights[f"experts.{e}.{t}.weight"] = f"{prefix}e{e}.{t}"
    shared = None
    if mlp.shared_ff is not None:
        shared = PartSpec("swiglu", {"hidden_size": config.width, "intermediate_size": mlp.shared_ff})
        weights.update({f"shared.{t}.weight": f"{prefix}shared.{t}" for t in ("gate", "up", "down")})
        weights["shared_gate.weight"] = prefix + "shared.sg"
    return PartSpec("routed_experts", {"hidden_size": config.width, "intermediate_size": mlp.ff, "experts": mlp.experts,
                                       "top": mlp.top, "activation": "swiglu", "correction": True, "score": "logistic",
                                       "group_count": mlp.group_count, "group_keep": mlp.group_keep, "group_value": "two_best",
                                       "weights_scale": mlp.scale, "shared": shared, "shared_gate": shared is not None}, weights)


def build_spec(config: TazizenConfig) -> ModelSpec:
    own = []
    for n, layer in enumerate(config.layers):
        make = _attention if isinstance(layer.mixer, Attention) else _latent
        own.append((make(config, layer.mixer, f"l{n}.mix."), _feed_forward(config, n)))

    def layer_spec(n: int, source: Optional[int]) -> LayerSpec:
        mixer, ffn = own[n]
        # a layer without feed-forward has no second sublayer; a checkpoint may hold that one's norm all the same
        return LayerSpec("hyper_connected", mixer, ffn, _norm(config, n, 1), _norm(config, n, 2, optional=ffn is None),
                         weights_from=source)

    # every layer's first visit is the layer itself, in the file's order; later passes follow as borrowed layers
    layers = [layer_spec(n, None) for n in range(len(config.layers))]
    schedule: List[int] = []
    visits: Dict[int, int] = {}
    for n in config.run_order():
        visits[n] = visits.get(n, 0) + 1
        if visits[n] == 1:
            schedule.append(n)
            continue
        layers.append(layer_spec(n, n))
        schedule.append(len(layers) - 1)
    sizes = {"vocab_size": config.vocab, "hidden_size": config.width}
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=config.width, vocab_size=config.vocab, max_positions=NO_POSITION_LIMIT,
        layers=tuple(layers), schedule=tuple(schedule),
        embedding=PartSpec("token_embedding", {**sizes, "streams": config.streams}, {"weight": "embed"}),
        final_norm=PartSpec("connected_rmsnorm", {"size": config.width, "eps": config.eps, "streams": config.streams,
                                                  "connected": False, "unit_offset": True}, {"weight": "final.norm"}),
        head=PartSpec("linear_head", sizes, {"weight": "head"}))


def random_plan(config: TazizenConfig) -> Iterator[Tuple[str, Tuple[int, ...], str, Draw]]:
    """(name, shape, role, draw) of every checkpoint tensor.  Projections N(0, 1/sqrt(fan-in)), norm weights stored around zero
    U(-0.1, 0.1), plain ones 1 + U(-0.1, 0.1), connections whose rows add up to one on average, router corrections U(-1.5,
    -0.5) (choice scores may then be negative)."""
    w, s = config.width, config.streams
    yield "embed", (config.vocab, w), "matrix", normal(1.0)
    for n, layer in enumerate(config.layers):
        p, m = f"l{n}.", layer.mixer
        q = p + "mix."
        for sub in (1, 2) if layer.mlp is not None else (1,):
            yield f"{p}norm{sub}", (w,), "vector", uniform(-0.1, 0.1)
            yield f"{p}hc{sub}.in", (s,), "vector", uniform(0.0, 2.0 / s)
            yield f"{p}hc{sub}.mix", (s, s), "vector", uniform(0.0, 2.0 / s)
            yield f"{p}hc{sub}.out", (s,), "vector", uniform(0.5, 1.5)
        if isinstance(m, Attention):
            yield q + "q", (m.heads * m.dim, w), "matrix", normal(w ** -0.5)
            yield q + "k", (m.kv_heads * m.dim, w), "matrix", normal(w ** -0.5)
            yield q + "v", (m.kv_heads * m.vdim, w), "matrix", normal(w ** -0.5)
            yield q + "g", (m.heads * m.vdim, w), "matrix", normal(w ** -0.5)
        else:
            yield q + "dq", (m.q_rank, w), "matrix", normal(w ** -0.5)
            yield q + "dq.norm", (m.q_rank,), "vector", uniform(0.9, 1.1)
            yield q + "uq", (m.heads * (m.dim + m.rot_dim), m.q_rank), "matrix", normal(m.q_rank ** -0.5)
            yield q + "dkv", (m.kv_rank + m.rot_dim, w), "matrix", normal(w ** -0.5)
            yield q + "dkv.norm", (m.kv_rank,), "vector", uniform(0.9, 1.1)
            yield q + "uk", (m.heads * m.dim, m.kv_rank), "matrix", normal(m.kv_rank ** -0.5)
            yield q + "uv", (m.heads * m.vdim, m.kv_rank), "matrix", normal(m.kv_rank ** -0.5)
        yield q + "o", (w, m.heads * m.vdim), "matrix", normal((m.heads * m.vdim) ** -0.5)
        if layer.mlp is not None:
            r = layer.mlp
            yield p + "mlp.router", (r.experts, w), "matrix", normal(w ** -0.5)
            yield p + "mlp.correction", (r.experts,), "vector", uniform(-1.5, -0.5)
            blocks = [(f"e{e}", r.ff) for e in range(r.experts)] + ([("shared", r.shared_ff)] if r.shared_ff is not None else [])
            for name, ff in blocks:
                yield f"{p}mlp.{name}.gate", (ff, w), "matrix", normal(w ** -0.5)
                yield f"{p}mlp.{name}.up", (ff, w), "matrix", normal(w ** -0.5)
                yield f"{p}mlp.{name}.down", (w, ff), "matrix", normal(ff ** -0.5)
            if r.shared_ff is not None:
                yield p + "mlp.shared.sg", (1, w), "matrix", normal(w ** -0.5)
    yield "final.norm", (w,), "vector", uniform(-0.1, 0.1)
    yield "head", (config.vocab, w), "matrix", normal(w ** -0.5)


register_architecture(Architecture(name=ARCHITECTURE, parse_config=TazizenConfig.from_dict, build_spec=build_spec,
                                   random_plan=random_plan))
