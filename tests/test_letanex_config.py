"""The Letanex design without a device: its configuration and its errors, the
plan's parts, tensor names, schedule and cache requests, and the plain
implementation against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

import go_tinygrad_b200 as lib
import plain_letanex as plain
from go_tinygrad_b200.cache import KVRequest, StateRequest
from go_tinygrad_b200.config.letanex import LetanexConfig
from go_tinygrad_b200.config.registry import find_architecture
from go_tinygrad_b200.kernels import ops
from go_tinygrad_b200.parts import build_part
from go_tinygrad_b200.parts.plan import PartSpec, plan_weight_specs
from go_tinygrad_b200.parts.position import rotary_frequencies


def rotation(dims, base, factor=None):
    out = {"dims": dims, "base": base}
    if factor is not None:
        out["scaling"] = {"factor": factor}
    return out


def attention(heads, kv_heads, dim, vdim, scale, diff, rot=None, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if rot is not None:
        m["rot"] = rot
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lightning(decay, dim, vdim, mlp=None):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, limit, experts, top, identity, scale=1.0, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
           "router": {"experts": experts, "top": top, "identity": identity, "scale": scale}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


SMALL = {
    "architecture": "Letanex", "vocab": 97, "width": 40, "norm": {"eps": 1e-5},
    "layers": [
        attention(6, 2, 8, 20, 0.3, 0.4, rotation(6, 500.0, 3.0), moe(24, 1.5, 5, 3, 2, 2.0, (16, 0.7))),
        lightning([0.5, 0.9, 1.0], 10, 6, dense(28)),
        attention(4, 2, 8, 20, 0.2, -0.1, rotation(6, 500.0, 3.0), kv_from=0),
        attention(3, 3, 5, 4, 0.5, 0.0, None, moe(12, 4.0, 3, 1, 0)),
    ],
}


def test_configuration_reads_every_key_and_writes_it_back():
    cfg = LetanexConfig.from_json(SMALL)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (97, 40, 1e-5)
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.diff, a.rot.dims, a.rot.base, a.rot.factor) == (6, 2, 8, 20, 0.3, 0.4, 6, 500.0, 3.0)
    m = cfg.layers[0].mlp
    assert (m.expert.ff, m.expert.limit, m.experts, m.top, m.identity, m.scale, m.shared.ff, m.shared.limit) == (24, 1.5, 5, 3, 2, 2.0, 16, 0.7)
    assert cfg.layers[1].mixer.decay == (0.5, 0.9, 1.0) and cfg.layers[1].mlp.ff == 28
    assert [getattr(l.mixer, "kv_from", None) for l in cfg.layers] == [None, None, 0, None] and cfg.layers[2].mlp is None
    assert cfg.layers[3].mixer.rot is None and cfg.layers[3].mlp.shared is None
    assert LetanexConfig.from_json(cfg.to_json()) == cfg
    assert find_architecture(SMALL).read_config(SMALL) == cfg
    bare = copy.deepcopy(SMALL)
    del bare["layers"][3]["mlp"]["router"]["identity"], bare["layers"][3]["mlp"]["router"]["scale"]
    assert LetanexConfig.from_json(bare) == cfg


@pytest.mark.parametrize("path,value,needle", [
    (("layers", 0, "type"), "attention_9", "type"),
    (("layers", 0, "mixer"), None, "mixer"),
    (("layers", 0, "mixer", "heads"), 5, "cannot share"),
    (("layers", 0, "mixer", "diff"), None, "diff"),
    (("layers", 0, "mixer", "scale"), 0, "positive"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "even"),
    (("layers", 0, "mixer", "rot", "dims"), 10, "at most"),
    (("layers", 0, "mixer", "rot", "scaling"), {}, "factor"),
    (("layers", 0, "mlp", "kind"), "sparse", "kind"),
    (("layers", 0, "mlp", "expert"), None, "expert"),
    (("layers", 0, "mlp", "expert", "limit"), None, "limit"),
    (("layers", 0, "mlp", "router", "top"), 8, "cannot use 8 of 7"),
    (("layers", 0, "mlp", "router", "identity"), -1, "identity"),
    (("layers", 0, "mlp", "shared", "ff"), 1.5, "integer"),
    (("layers", 1, "mixer", "decay"), [0.5, 0.9], "3 numbers"),
    (("layers", 1, "mixer", "decay"), [0.5, 0.9, 1.5], "between"),
    (("layers", 2, "mixer", "kv_from"), 2, "earlier"),
    (("layers", 2, "mixer", "kv_from"), 1, "no keys"),
    (("layers", 2, "mixer", "vdim"), 16, "must equal"),
    (("layers", 2, "mixer", "rot", "base"), 400.0, "must equal"),
    (("norm",), None, "eps"),
    (("layers",), [], "non-empty"),
])
def test_configuration_errors_name_the_key(path, value, needle):
    raw = copy.deepcopy(SMALL)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(lib.ConfigError) as e:
        LetanexConfig.from_json(raw)
    assert needle in str(e.value)


def test_plan_parts_tensors_schedule_and_cache_requests():
    arch = find_architecture(SMALL)
    plan = arch.plan(arch.read_config(SMALL))
    assert [(e.layer, e.cache) for e in plan.schedule] == [(0, None), (1, None), (2, 0), (3, None)]
    names = {s.name: s for s in plan_weight_specs(plan)}
    want = {"embed": (97, 40), "final.norm": (40,), "head": (97, 40),
            "l0.mix.q": (96, 40), "l0.mix.k": (32, 40), "l0.mix.v": (40, 40), "l0.mix.o": (40, 120),
            "l0.mlp.router": (7, 40), "l0.mlp.correction": (7,),
            "l0.mlp.shared.gate": (16, 40), "l0.mlp.shared.up": (16, 40), "l0.mlp.shared.down": (40, 16),
            "l1.mix.q": (30, 40), "l1.mix.k": (30, 40), "l1.mix.v": (18, 40), "l1.mix.g": (18, 40), "l1.mix.norm": (18,), "l1.mix.o": (40, 18),
            "l1.mlp.up": (28, 40), "l1.mlp.down": (40, 28),
            "l2.mix.q": (64, 40), "l2.mix.o": (40, 80),
            "l3.mix.q": (30, 40), "l3.mix.k": (30, 40), "l3.mix.v": (12, 40), "l3.mix.o": (40, 12),
            "l3.mlp.router": (3, 40), "l3.mlp.correction": (3,)}
    for i, size in ((0, 8), (2, 8), (3, 5)):
        want.update({f"l{i}.mix.{k}": (size,) for k in ("lq1", "lk1", "lq2", "lk2")})
    for i in range(4):
        want.update({f"l{i}.norm1": (40,), f"l{i}.norm1b": (40,)})
        if i != 2:
            want.update({f"l{i}.norm2": (40,), f"l{i}.norm2b": (40,)})
    for i, n, ff in ((0, 5, 24), (3, 3, 12)):
        for e in range(n):
            want.update({f"l{i}.mlp.e{e}.gate": (ff, 40), f"l{i}.mlp.e{e}.up": (ff, 40), f"l{i}.mlp.e{e}.down": (40, ff)})
    assert {n: tuple(s.shape) for n, s in names.items()} == want
    blocks = [build_part("block", spec.block) for spec in plan.layers]
    assert blocks[0].cache_requests() == [KVRequest(2, 16, None, value_dim=20)]          # both maps side by side in a key row
    assert blocks[1].cache_requests() == [StateRequest("memory", (3, 10, 6), "float32")]
    assert blocks[2].cache_requests() == []


def test_combinations_that_are_not_built_are_refused():
    base = {"hidden_size": 16, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "value_dim": 6, "window": None, "scale": 1.0,
            "position": PartSpec("none", {}), "norm_eps": 1e-5, "q": "q", "k": "k", "v": "v", "o": "o",
            "differential": {"diff": 0.3, "lq1": "a", "lk1": "b", "lq2": "c", "lk2": "d"}}
    build_part("mixer", PartSpec("gqa_attention", base))
    for change in ({"values": "keys"}, {"softcap": 3.0}, {"chunk": 4}, {"qk_norm": "unit"}, {"head_gate": "g"},
                   {"q_bias": "x", "k_bias": "y", "v_bias": "z"}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("gqa_attention", {**base, **change}))
    experts = {"hidden_size": 8, "intermediate_size": 8, "n_experts": 4, "top": 2, "router": "r", "gate": "e{e}.g", "up": "e{e}.u", "down": "e{e}.d"}
    for change in ({"correction": "c"}, {"weight_scale": 2.0}, {"gate": None, "gate_limit": 1.0}, {"gate": None, "identity": 2},
                   {"weight_on": "input", "identity": 2}, {"top": 6, "identity": 1}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", {**experts, **change}))
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("swiglu", {"hidden_size": 8, "intermediate_size": 8, "gate": "g", "up": "u", "down": "d",
                                                       "gate_limit": 1.0, "activation": "relu2"}))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("lightning", {"hidden_size": 8, "n_heads": 2, "head_dim": 4, "value_dim": 4, "decay": [0.5], "eps": 1e-5,
                                                   **{k: k for k in ("q", "k", "v", "g", "norm", "o")}}))
    norm = {"size": 8, "eps": 1e-5, "weight": "w", "bias": None}
    sandwich = {"mixer_norm": PartSpec("layernorm", norm), "mixer_output_norm": PartSpec("rmsnorm", norm), "mixer": PartSpec("gqa_attention", base)}
    with pytest.raises(ValueError):
        build_part("block", PartSpec("sandwich_norm", sandwich))


def test_epilogue_codes_of_clamped_gates_are_the_limits_bits_and_no_other_code():
    codes = [ops._epilogue_code(ops.ClampedGate(limit)) for limit in (1e-37, 0.5, 1.0, 2.0, 1e30, math.inf)]
    assert all(c >= 0x00800000 for c in codes) and len(set(codes)) == 6
    assert [torch.tensor(c, dtype=torch.int32).view(torch.float32).item() for c in codes[1:4]] == [0.5, 1.0, 2.0]
    assert max(ops._epilogue_code(e) for e in ("none", "swiglu", "silu", "gated_relu2")) < 64
    for bad in (0.0, -1.0):
        with pytest.raises(ops.KernelError):
            ops._epilogue_code(ops.ClampedGate(bad))
    with pytest.raises(ops.KernelError):
        ops._epilogue_code("clamped")


def test_linear_scaling_divides_every_frequency():
    plain_f = rotary_frequencies(12, 700.0)
    assert rotary_frequencies(12, 700.0, {"rope_type": "linear", "factor": 5.0}) == [f / 5.0 for f in plain_f]
    np.testing.assert_allclose(plain.frequencies(12, 700.0, 5.0), np.array(plain_f) / 5.0, rtol=1e-14)


# ---------------------------------------------------------------- the plain implementation
def test_plain_rotation_keeps_distances_only():
    rng = np.random.default_rng(0)
    f = plain.frequencies(6, 30.0, 2.0)
    q, k = rng.standard_normal((2, 1, 10))
    score = lambda i, j: plain.rotate(q, [i], f)[0] @ plain.rotate(k, [j], f)[0]
    assert abs(score(9, 4) - score(105, 100)) < 1e-12 and abs(score(9, 4) - score(9, 5)) > 1e-3
    np.testing.assert_array_equal(plain.rotate(q, [7], f)[0, 6:], q[0, 6:])


def test_plain_differential_attention_cancels_maps_that_are_alike():
    """Equal maps leave (1 - lambda) a, whose norm does not depend on lambda's size; a second map that sees evenly
    takes the mean of the values off."""
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((7, 2, 1, 4)), rng.standard_normal((7, 1, 1, 4)), rng.standard_normal((7, 1, 3))
    twice = lambda x: np.concatenate([x, x], axis=2)
    a = plain.differential_attend(twice(q), twice(k), v, 0.7, 0.3, 0.25, 0.0)
    b = plain.differential_attend(twice(q), twice(k), v, 0.7, -5.0, 0.25, 0.0)
    np.testing.assert_allclose(a, b, atol=1e-12)
    np.testing.assert_allclose((a ** 2).mean(-1), 0.75 ** 2, atol=1e-12)
    even = np.concatenate([q, 0 * q], axis=2)
    c = plain.differential_attend(even, twice(k), v, 0.7, 0.5, 0.0, 0.0)
    first = np.stack([plain.softmax_attend(q[:, h, 0], k[:, 0, 0], v[:, 0], 0.7) for h in range(2)], axis=1)
    mean = np.cumsum(v[:, 0], axis=0) / np.arange(1, 8)[:, None]
    np.testing.assert_allclose(c, plain.unit_rms(first - 0.5 * mean[:, None], 0.0), atol=1e-12)
    assert plain.mixing_lambda([1.0, 2.0], [0.5, 0.0], [0.0, 1.0], [3.0, -1.0], 0.2) == pytest.approx(math.exp(0.5) - math.exp(-1.0) + 0.2)


def test_plain_memory_is_a_sum_over_the_past():
    rng = np.random.default_rng(2)
    q, k, v = rng.standard_normal((9, 3)), rng.standard_normal((9, 3)), rng.standard_normal((9, 2))
    t = np.arange(9)
    w = np.where(t[:, None] >= t[None, :], 0.8 ** (t[:, None] - t[None, :]), 0.0)
    np.testing.assert_allclose(plain.decayed_memory(q, k, v, 0.8), (w * (q @ k.T)) @ v, atol=1e-12)


def test_plain_experts_clamp_and_choose_as_said():
    one = np.ones((1, 1))
    f = lambda g, u, limit: plain.clamped_expert(np.array([[1.0]]), one * g, one * u, one, limit)[0, 0]
    sig = lambda z: 1 / (1 + math.exp(-1.702 * z))
    assert f(5.0, 9.0, 2.0) == pytest.approx(2.0 * sig(2.0) * 3.0)
    assert f(-5.0, -9.0, 2.0) == pytest.approx(-5.0 * sig(-5.0) * -1.0)        # the gate has no lower limit
    assert f(0.5, 0.25, 2.0) == pytest.approx(0.5 * sig(0.5) * 1.25)
    h, router = np.array([[1.0]]), np.log(np.array([[1.0], [2.0], [4.0], [3.0]]))
    chosen, w = plain.route(h, router, [0.35, 0.0, -0.3, 0.0], 2, 1.5)        # scores 0.1 0.2 0.4 0.3
    assert chosen.tolist() == [[0, 3]]
    np.testing.assert_allclose(w, [[1.5 * 0.1 / 0.4, 1.5 * 0.3 / 0.4]])
