"""The Letanex decoder as a plan of parts.

Every layer is a ``sandwich_norm`` block (each sublayer between two layer norms) around one
of two mixers: ``gqa_attention`` with ``differential`` (two maps a head over one set of
values; a layer with ``kv_from`` reads the cache of the layer it names: the schedule
entry's ``cache``) or ``lightning``, linear attention with a fixed decay per head.  The
feed-forward is ``dense`` with a squared relu, or ``routed_experts`` with clamped gates,
scores over all outputs, identity experts and a shared expert.  A final layer norm and an
untied head close the model.  Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``,
``l<i>.mix.*``, ``l<i>.mlp.up|down``, ``l<i>.mlp.router|correction``,
``l<i>.mlp.e<j>.gate|up|down``, ``l<i>.mlp.shared.gate|up|down``, ``final.norm``, ``head``.
The reference has no such architecture.
"""
from __future__ import annotations

from ..config.letanex import LetanexConfig
from ..config.registry import Architecture, register_architecture
from ..config.ropovik import DenseMlp
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry


def _norm(cfg: LetanexConfig, name: str) -> PartSpec:
    return PartSpec("layernorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight": name, "bias": None})


def _attention(cfg: LetanexConfig, i: int) -> PartSpec:
    m, p = cfg.layers[i].mixer, f"l{i}.mix."
    position = PartSpec("none", {})
    if m.rot is not None:
        scaling = {"rope_type": "linear", "factor": m.rot.factor} if m.rot.factor is not None else None
        position = PartSpec("rotary", {"head_dim": m.dim, "rotary_dim": m.rot.dims, "theta": m.rot.base, "scaling": scaling})
    params = {"hidden_size": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
              "scale": m.scale, "window": None, "own_kv": m.kv_from is None, "position": position, "norm_eps": cfg.norm_eps,
              "differential": {"diff": m.diff, **{k: p + k for k in ("lq1", "lk1", "lq2", "lk2")}}, "q": p + "q", "o": p + "o"}
    if m.kv_from is None:
        params.update({"k": p + "k", "v": p + "v"})
    return PartSpec("gqa_attention", params)


def _lightning(cfg: LetanexConfig, i: int) -> PartSpec:
    m, p = cfg.layers[i].mixer, f"l{i}.mix."
    return PartSpec("lightning", {"hidden_size": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "decay": m.decay,
                                  "eps": cfg.norm_eps, **{k: p + k for k in ("q", "k", "v", "g", "norm", "o")}})


_MIXERS = {"attention": _attention, "lightning": _lightning}


def _feed_forward(cfg: LetanexConfig, i: int) -> PartSpec:
    mlp, p = cfg.layers[i].mlp, f"l{i}.mlp."
    if isinstance(mlp, DenseMlp):
        return PartSpec("dense", {"hidden_size": cfg.width, "intermediate_size": mlp.ff, "activation": "relu2", "up": p + "up", "down": p + "down"})
    shared = None
    if mlp.shared is not None:
        shared = PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": mlp.shared.ff, "gate_limit": mlp.shared.limit,
                                     **{k: f"{p}shared.{k}" for k in ("gate", "up", "down")}})
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "intermediate_size": mlp.expert.ff, "n_experts": mlp.experts, "identity": mlp.identity, "top": mlp.top,
        "scoring": "softmax_all", "correction": p + "correction", "weight_scale": mlp.scale, "gate_limit": mlp.expert.limit,
        "router": p + "router", "router_bias": None, "shared": shared, **{k: p + "e{e}." + k for k in ("gate", "up", "down")}})


def letanex_plan(cfg: LetanexConfig) -> ModelPlan:
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer_norm": _norm(cfg, p + "norm1"), "mixer": _MIXERS[layer.type](cfg, i), "mixer_output_norm": _norm(cfg, p + "norm1b"),
                 "feed_forward_norm": None, "feed_forward": None, "feed_forward_output_norm": None}
        if layer.mlp is not None:
            parts.update({"feed_forward_norm": _norm(cfg, p + "norm2"), "feed_forward": _feed_forward(cfg, i),
                          "feed_forward_output_norm": _norm(cfg, p + "norm2b")})
        layers.append(LayerSpec(PartSpec("sandwich_norm", parts)))
        schedule.append(ScheduleEntry(layer=i, cache=getattr(layer.mixer, "kv_from", None)))
    plan = ModelPlan(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "embed"}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "head"}),
        stop_tokens=(),
        max_position=None,
    )
    plan.check()
    return plan


LETANEX = register_architecture(Architecture(
    names=("Letanex", "letanex"),
    read_config=LetanexConfig.from_json,
    plan=letanex_plan,
    ignore=("l*.norm2", "l*.norm2b"),      # a layer without a feed-forward may carry the norms of one
))
