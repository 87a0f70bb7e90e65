"""The Mererax design without a device: its configuration and its errors, the
plan's parts, tensor names, schedule and cache requests, and the plain
implementation against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

import go_tinygrad_b200 as lib
import plain_mererax as plain
from go_tinygrad_b200.cache import KVRequest, StateRequest
from go_tinygrad_b200.config.mererax import MereraxConfig
from go_tinygrad_b200.config.registry import find_architecture
from go_tinygrad_b200.parts import Runtime, build_part
from go_tinygrad_b200.parts.base import JointUpdate
from go_tinygrad_b200.parts.plan import PartSpec, plan_weight_specs


def left(heads, kv_heads, dim, scale, coef=None, every=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return m


def right(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def parallel(a, b, ff=None, weights_of=None):
    return layer("parallel", {"left": a, "right": b}, ff, weights_of)


def mamba(inner, state, rank, conv, ff=None, weights_of=None):
    return layer("mamba1", {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}, ff, weights_of)


def layer(kind, mixer, ff, weights_of):
    out = {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


SMALL = {
    "architecture": "Mererax", "vocab": 97, "width": 40, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
    "layers": [
        parallel(left(4, 2, 12, 0.3, 0.2, 8), right(3, 10, 6, 9.0), 24),
        mamba(28, 6, 5, 3),
        parallel(left(4, 2, 12, 0.3, 0.2, 8), right(3, 10, 6, 9.0), 24, weights_of=0),
        mamba(20, 7, 9, 1, 16),
        mamba(28, 6, 5, 3, weights_of=1),
    ],
}


def test_configuration_reads_every_key_and_writes_it_back():
    cfg = MereraxConfig.from_json(SMALL)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale) == (97, 40, 1e-5, 3.0)
    a, b = cfg.layers[0].mixer.left, cfg.layers[0].mixer.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.q_temp.coef, a.q_temp.every) == (4, 2, 12, 12, 0.3, 0.2, 8.0)
    assert (b.heads, b.dim, b.vdim, b.gate_cap) == (3, 10, 6, 9.0)
    m = cfg.layers[1].mixer
    assert (m.inner, m.state, m.dt_rank, m.conv) == (28, 6, 5, 3)
    assert [l.weights_of for l in cfg.layers] == [None, None, 0, None, 1] and cfg.layers[1].mlp is None and cfg.layers[3].mlp.ff == 16
    assert [cfg.source_of(i) for i in range(5)] == [0, 1, 0, 3, 1]
    assert MereraxConfig.from_json(cfg.to_json()) == cfg
    assert find_architecture(SMALL).read_config(SMALL) == cfg
    bare = copy.deepcopy(SMALL)
    del bare["embedding"]
    assert MereraxConfig.from_json(bare).embedding_scale == 1.0


@pytest.mark.parametrize("path,value,needle", [
    (("layers", 0, "type"), "attention_9", "type"),
    (("layers", 0, "mixer", "left", "heads"), 3, "cannot share"),
    (("layers", 0, "mixer", "left", "vdim"), 16, "values are the keys"),
    (("layers", 0, "mixer", "left", "scale"), None, "scale"),
    (("layers", 0, "mixer", "left", "q_temp"), {"coef": 0.5}, "every"),
    (("layers", 0, "mixer", "left", "q_temp"), {"coef": 0.5, "every": 0}, "positive"),
    (("layers", 0, "mixer", "left"), None, "left"),
    (("layers", 0, "mixer", "right"), None, "right"),
    (("layers", 0, "mixer", "right", "gate_cap"), 0, "positive"),
    (("layers", 3, "mixer", "dt_rank"), None, "dt_rank"),
    (("layers", 3, "mixer", "conv"), 2.5, "integer"),
    (("layers", 2, "weights_of"), 2, "another layer"),
    (("layers", 2, "weights_of"), 9, "another layer"),
    (("layers", 2, "weights_of"), 1, "must equal"),
    (("layers", 2, "mixer", "right", "gate_cap"), 8.0, "must equal"),
    (("layers", 1, "mlp"), {"kind": "moe"}, "kind"),
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
        MereraxConfig.from_json(raw)
    assert needle in str(e.value)


def test_layers_whose_weights_come_from_each_other_are_refused():
    raw = copy.deepcopy(SMALL)
    raw["layers"][0]["weights_of"] = 2
    with pytest.raises(lib.ConfigError, match="leads back"):
        MereraxConfig.from_json(raw)


def test_plan_parts_tensors_schedule_and_cache_requests():
    arch = find_architecture(SMALL)
    plan = arch.plan(arch.read_config(SMALL))
    assert [(e.layer, e.cache) for e in plan.schedule] == [(0, None), (1, None), (0, None), (2, None), (1, None)]
    names = {s.name: s for s in plan_weight_specs(plan)}
    want = {"embed": (97, 40), "final.norm": (40,), "l0.norm1": (40,), "l0.norm2": (40,),
            "l0.mix.left.q": (48, 40), "l0.mix.left.k": (24, 40), "l0.mix.left.q.norm": (48,), "l0.mix.left.k.norm": (24,),
            "l0.mix.left.o": (40, 48), "l0.mix.left.out": (40,), "l0.mix.right.out": (40,),
            "l0.mix.right.q": (30, 40), "l0.mix.right.k": (30, 40), "l0.mix.right.v": (18, 40), "l0.mix.right.g": (18, 40),
            "l0.mix.right.o": (40, 18), "l0.mix.right.norm": (18,), "l0.mix.right.i": (3, 40), "l0.mix.right.i.b": (3,),
            "l0.mix.right.f": (3, 40), "l0.mix.right.f.b": (3,),
            "l0.mlp.gate": (24, 40), "l0.mlp.up": (24, 40), "l0.mlp.down": (40, 24),
            "l1.norm1": (40,), "l1.mix.in": (56, 40), "l1.mix.conv": (28, 3), "l1.mix.conv.b": (28,), "l1.mix.x": (17, 28),
            "l1.mix.dt": (28, 5), "l1.mix.dt.b": (28,), "l1.mix.A_log": (28, 6), "l1.mix.D": (28,), "l1.mix.o": (40, 28),
            "l3.norm1": (40,), "l3.norm2": (40,), "l3.mix.in": (40, 40), "l3.mix.conv": (20, 1), "l3.mix.conv.b": (20,),
            "l3.mix.x": (23, 20), "l3.mix.dt": (20, 9), "l3.mix.dt.b": (20,), "l3.mix.A_log": (20, 7), "l3.mix.D": (20,),
            "l3.mix.o": (40, 20), "l3.mlp.gate": (16, 40), "l3.mlp.up": (16, 40), "l3.mlp.down": (40, 16)}
    assert {n: tuple(s.shape) for n, s in names.items()} == want
    assert names["l0.norm1"].mean == 0.0 and names["l0.mix.left.out"].mean == 1.0
    blocks = [build_part("block", spec.block) for spec in plan.layers]
    assert blocks[0].cache_requests() == [KVRequest(2, 12, None), StateRequest("memory", (3, 10, 6), "float32"),
                                          StateRequest("normaliser", (3, 10), "float32"), StateRequest("maximum", (3, 7), "float32")]
    assert blocks[1].cache_requests() == [StateRequest("scan", (28, 6), "float32"), StateRequest("conv", (2, 28), "float32")]
    assert blocks[2].cache_requests() == [StateRequest("scan", (20, 7), "float32")]          # one tap: nothing to remember
    # a mamba layer and its feed-forward end in one product; a pair's outputs are normed first and cannot
    assert blocks[0].lasts is None and blocks[1].lasts is None
    assert blocks[2].lasts == [("l3.mix.o", 20), ("l3.mlp.down", 16)]


def test_combinations_that_are_not_built_are_refused():
    base = {"hidden_size": 16, "n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "window": None, "scale": 1.0, "values": "keys",
            "position": PartSpec("none", {}), "qk_norm": "rows", "q_norm": "qn", "k_norm": "kn", "norm_eps": 1e-5,
            "q": "q", "k": "k", "o": "o"}
    build_part("mixer", PartSpec("gqa_attention", base))
    for change in ({"values": "projection", "v": "v"}, {"softcap": 3.0}, {"chunk": 4}, {"qk_norm": None, "distance_slopes": True},
                   {"position": PartSpec("rotary", {"head_dim": 8, "theta": 100.0})}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("gqa_attention", dict(base, **change)))


def test_operands_side_by_side_start_at_multiples_of_eight_with_zeros_between():
    rt = Runtime(torch.device("cpu"), torch.float32)
    gen = torch.Generator().manual_seed(0)
    a, b = torch.randn(5, 13, generator=gen), torch.randn(5, 11, generator=gen)
    w = JointUpdate.matrix([a, b], rt)
    assert w.shape == (5, 32)
    joint = JointUpdate(rt, 3, [13, 11])
    x, y = torch.randn(3, 13, generator=gen), torch.randn(3, 11, generator=gen)
    joint.take(13).copy_(x)
    with pytest.raises(ValueError):
        joint.take(13)
    joint.take(11).copy_(y)
    torch.testing.assert_close(joint.buffer @ w.t(), x @ a.t() + y @ b.t())


def test_plain_implementation_against_closed_forms():
    rng = np.random.default_rng(0)
    # positions: position 0 adds 0 to even and 1 to odd channels; the first pair turns by one radian a token
    np.testing.assert_allclose(plain.sinusoid([0], 5), [[0, 1, 0, 1, 0]], atol=1e-15)
    np.testing.assert_allclose(plain.sinusoid([3], 4)[0, :2], [math.sin(3), math.cos(3)])
    np.testing.assert_allclose(plain.sinusoid([3], 4)[0, 2], math.sin(0.03))
    # query temperature: 1 before the first step, one more ln every `every` tokens
    np.testing.assert_allclose(plain.query_temperature([0, 6, 7, 14, 15], 0.5, 8), 1 + 0.5 * np.log([1, 1, 2, 2, 3]))
    np.testing.assert_allclose(plain.distance_slopes(4), [0.25, 1 / 16, 1 / 64, 1 / 256])
    # a penalty so steep that only the token itself is left
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 1, 4)), rng.standard_normal((6, 1, 3))
    np.testing.assert_allclose(plain.attend(q, k, v, 1.0, np.array([900.0, 900.0])), np.broadcast_to(v, (6, 2, 3)))
    # two keys: the weight of the nearer grows by the slope's exponential
    out = plain.attend(np.zeros((2, 1, 4)), k[:2], v[:2], 1.0, np.array([math.log(3.0)]))
    np.testing.assert_allclose(out[1, 0], (v[0, 0] + 3 * v[1, 0]) / 4)
    # the matrix memory: one token.  i = ln 2 > f + 0, so m = ln 2, the state takes the whole of k v^T; the
    # denominator is |k . q| or exp(-m) = 1/2, whichever is larger
    kk, vv = np.array([[1.0, 0.0]]), np.array([[3.0, -1.0]])
    for qx, den in ((2.0, 2.0), (0.2, 0.5)):
        out = plain.matrix_memory(np.array([[qx, 7.0]]), kk, vv, [math.log(2)], [-1.0])
        np.testing.assert_allclose(out[0], qx * vv[0] / (den + 1e-6))
    # the maximum starts at zero: an input gate below the forget gate's logarithm leaves m = f, and the token counts exp(i - f)
    out = plain.matrix_memory(np.array([[1.0, 0.0]]), kk, vv, [-3.0], [-0.5])
    np.testing.assert_allclose(out[0], math.exp(-2.5) * vv[0] / (max(math.exp(-2.5), math.exp(0.5)) + 1e-6))
    # two tokens with orthogonal keys: the second query finds the first value, decayed, over the larger of its weight and exp(-m)
    out = plain.matrix_memory(np.array([[0, 0], [1.0, 0]]), np.eye(2), np.array([[4.0], [9.0]]), [0.0, 0.0], [-10.0, -math.log(2)])
    np.testing.assert_allclose(out[1], 0.5 * 4.0 / (1.0 + 1e-6))
    # the selective scan: without decay and with B = C = 1 it adds up dt x
    x, dt = rng.standard_normal((5, 2)), rng.uniform(0.1, 1, (5, 2))
    y = plain.selective_scan(x, dt, np.ones((5, 1)), np.ones((5, 1)), np.zeros((2, 1)), np.array([0.0, 2.0]))
    np.testing.assert_allclose(y, np.cumsum(dt * x, axis=0) + np.array([0.0, 2.0]) * x)
    # ... and with a rate of -ln 2 a dt of 1 halves what was there
    y = plain.selective_scan(np.array([[1.0], [0.0]]), np.ones((2, 1)), np.ones((2, 1)), np.ones((2, 1)), np.array([[-math.log(2)]]), np.zeros(1))
    np.testing.assert_allclose(y[:, 0], [1.0, 0.5])
    # a convolution whose taps are (0, .., 0, 1) adds its bias only; (1, 0) delays by one token
    u = rng.standard_normal((7, 3))
    np.testing.assert_allclose(plain.causal_conv(u, np.array([[0, 0, 1.0]] * 3), np.ones(3)), u + 1)
    np.testing.assert_allclose(plain.causal_conv(u, np.array([[1.0, 0]] * 3), np.zeros(3)), np.concatenate([np.zeros((1, 3)), u[:-1]]))
    np.testing.assert_allclose(plain.log_sigmoid([-800.0, 0.0, 800.0]), [-800.0, -math.log(2), 0.0])
    assert plain.source_of(SMALL, 4) == 1 and plain.source_of(SMALL, 3) == 3
