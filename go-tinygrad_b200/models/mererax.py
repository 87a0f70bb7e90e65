"""The Mererax decoder as a plan of parts.

The scaled token embedding gets a sinusoid of the position added
(``token_embedding`` with the ``sinusoidal`` position); every layer is a
``parallel_pre_norm`` block, whose mixer and gated feed-forward read two norms of
one hidden state (weights stored around zero), around one of two mixers:
``normed_pair``, attention whose values are the keys (norms over whole rows of q and
k, growing queries, a penalty on the distance) beside a ``matrix_memory``; and
``mamba1``.  A layer with ``weights_of`` is one more entry of the schedule that names
the other layer's block, with cache and state of its own.  A final norm and the
embedding table as head close it.  Tensor names: ``embed``, ``l<i>.norm1|norm2``,
``l<i>.mix.*`` (``left.*`` and ``right.*`` under a pair), ``l<i>.mlp.gate|up|down``,
``final.norm``.  The reference has no such architecture.
"""
from __future__ import annotations

from ..config.mererax import MereraxConfig
from ..config.registry import Architecture, register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry


def _norm(cfg: MereraxConfig, name: str) -> PartSpec:
    return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight": name, "weight_offset": 1.0})


def _parallel(cfg: MereraxConfig, i: int) -> PartSpec:
    a, b = cfg.layers[i].mixer.left, cfg.layers[i].mixer.right
    p, q = f"l{i}.mix.left.", f"l{i}.mix.right."
    left = PartSpec("gqa_attention", {
        "hidden_size": cfg.width, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "scale": a.scale, "window": None,
        "values": "keys", "position": PartSpec("none", {}), "qk_norm": "rows", "q_norm": p + "q.norm", "k_norm": p + "k.norm",
        "norm_eps": cfg.norm_eps, "q_temperature": (a.q_temp.coef, a.q_temp.every) if a.q_temp else None, "distance_slopes": True,
        "q": p + "q", "k": p + "k", "o": p + "o"})
    right = PartSpec("matrix_memory", {
        "hidden_size": cfg.width, "n_heads": b.heads, "head_dim": b.dim, "value_dim": b.vdim, "gate_cap": b.gate_cap, "eps": cfg.norm_eps,
        "q": q + "q", "k": q + "k", "v": q + "v", "g": q + "g", "i": q + "i", "i_bias": q + "i.b", "f": q + "f", "f_bias": q + "f.b",
        "norm": q + "norm", "o": q + "o"})
    return PartSpec("normed_pair", {"hidden_size": cfg.width, "left": left, "right": right, "left_norm": p + "out", "right_norm": q + "out",
                                    "eps": cfg.norm_eps, "factor": 0.5})


def _mamba1(cfg: MereraxConfig, i: int) -> PartSpec:
    m, p = cfg.layers[i].mixer, f"l{i}.mix."
    return PartSpec("mamba1", {
        "hidden_size": cfg.width, "inner": m.inner, "state_size": m.state, "dt_rank": m.dt_rank, "conv_taps": m.conv,
        "in": p + "in", "conv": p + "conv", "conv_bias": p + "conv.b", "x": p + "x", "dt": p + "dt", "dt_bias": p + "dt.b",
        "a_log": p + "A_log", "d": p + "D", "o": p + "o"})


_MIXERS = {"parallel": _parallel, "mamba1": _mamba1}


def mererax_plan(cfg: MereraxConfig) -> ModelPlan:
    layers, at = [], {}                    # layers with tensors of their own, and where each stands in the plan
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        parts = {"mixer_norm": _norm(cfg, p + "norm1"), "mixer": _MIXERS[layer.type](cfg, i),
                 "feed_forward_norm": None, "feed_forward": None}
        if layer.mlp is not None:
            parts["feed_forward_norm"] = _norm(cfg, p + "norm2")
            parts["feed_forward"] = PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff,
                                                        "gate": p + "mlp.gate", "up": p + "mlp.up", "down": p + "mlp.down"})
        at[i] = len(layers)
        layers.append(LayerSpec(PartSpec("parallel_pre_norm", parts)))
    plan = ModelPlan(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "embed",
                                               "scale": cfg.embedding_scale,
                                               "position": PartSpec("sinusoidal", {"size": cfg.width, "base": 10000.0})}),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(layer=at[cfg.source_of(i)]) for i in range(len(cfg.layers))),
        final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "embed", "tied": True}),
        stop_tokens=(),
        max_position=None,
    )
    plan.check()
    return plan


MERERAX = register_architecture(Architecture(
    names=("Mererax", "mererax"),
    read_config=MereraxConfig.from_json,
    plan=mererax_plan,
))
