"""The Letanex design in the engine against its plain implementation
(plain_letanex.py): every mechanism alone, then whole models of three small
configurations that differ in every size and option, under every way of
cutting the same requests into steps."""
import contextlib
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import go_tinygrad_b200 as lib
import plain_letanex as plain
import plain_llama
from go_tinygrad_b200.cache import Cache
from go_tinygrad_b200.config.registry import find_architecture
from go_tinygrad_b200.engine import Model, StepEntry, step
from go_tinygrad_b200.kernels import ops
from go_tinygrad_b200.parts import PartSpec, Runtime, build_part, walk
from go_tinygrad_b200.parts.base import ResidualStream
from conftest import ROOT, assert_close
from test_letanex_config import attention, dense, lightning, moe, rotation
from test_megerax_gpu import DEV, DTYPES, TORCH, close, f64, run_cut, run_mixers, short, t32
from test_parts_gpu import context

pytestmark = pytest.mark.gpu

# P: heads in groups of three and five, sizes that are multiples of 8 or 4 or of nothing, layers that borrow keys (one of
# them from two layers back), no feed-forward, a mixture without a shared expert and one without identities.
CONFIG_P = {
    "architecture": "Letanex", "vocab": 211, "width": 72, "norm": {"eps": 1e-5},
    "layers": [
        attention(6, 2, 24, 40, 0.3, 0.35, rotation(16, 900.0, 2.5), moe(40, 1.2, 6, 2, 3, 1.7, (24, 0.6))),
        lightning([0.4, 0.9, 0.99], 20, 12, dense(100)),
        attention(10, 2, 24, 40, 0.2, 0.6, rotation(16, 900.0, 2.5), kv_from=0),
        lightning([1.0, 0.7], 36, 40, moe(20, 3.0, 4, 3, 0, 0.8)),
        attention(3, 3, 16, 8, 0.4, 0.1, None, dense(64)),
        attention(3, 1, 24, 20, 0.25, 0.5, rotation(24, 300.0), moe(16, 0.9, 2, 1, 5, 2.2, (40, 1.1))),
    ],
}
# Q: sizes the tensor-core kernels take: maps of 64 channels over values of 128, 128 over 256, one key head for four.
CONFIG_Q = {
    "architecture": "Letanex", "vocab": 160, "width": 128, "norm": {"eps": 1e-6},
    "layers": [
        lightning([0.6, 0.95, 0.995, 0.999], 64, 128, dense(256)),
        attention(4, 1, 64, 128, 0.12, 0.35, rotation(64, 10000.0, 6.0), moe(64, 1.8, 8, 2, 2, 1.4, (128, 1.3))),
        attention(4, 1, 64, 128, 0.12, 0.3, rotation(64, 10000.0, 6.0), moe(64, 1.8, 8, 2, 2, 1.4, (128, 1.3)), kv_from=1),
        attention(2, 2, 128, 256, 0.09, 0.4, rotation(32, 500.0, 4.0), None),
        lightning([0.8, 0.9995], 128, 64, moe(128, 1.0, 4, 4, 4, 1.0, (64, 2.5))),
    ],
}
# U: nothing is a multiple of 8, 4 or 2 where the design allows it; an odd width; one head.  Lambdas that keep the two maps of
# these narrow heads from cancelling: what is left of them is normed, and rounding with it.
CONFIG_U = {
    "architecture": "Letanex", "vocab": 101, "width": 51, "norm": {"eps": 1e-4},
    "layers": [
        lightning([0.55, 0.97, 0.3], 9, 13, moe(11, 1.4, 3, 2, 1, 1.3, (29, 0.8))),
        attention(5, 5, 7, 11, 0.4, 0.15, rotation(6, 50.0, 1.5), dense(59)),
        attention(5, 5, 7, 11, 0.3, -0.3, rotation(6, 50.0, 1.5), moe(13, 2.0, 5, 1, 2, 1.0, (27, 3.0)), kv_from=1),
        lightning([0.9, 0.35, 0.8], 13, 11),
        attention(1, 1, 3, 21, 0.9, 0.1, rotation(2, 10.0)),
    ],
}
CONFIGS = {"P": (CONFIG_P, 3, 0.12, 0.1), "Q": (CONFIG_Q, 4, 0.08, 0.05), "U": (CONFIG_U, 5, 0.15, 0.1)}     # configuration, seed, std, norm std


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, (cfg, seed, std, norm_std) in CONFIGS.items():
        folder = str(tmp_path_factory.mktemp(f"letanex_{name}"))
        lib.write_random_model(folder, cfg, seed=seed, dtype="bfloat16", std=std, norm_std=norm_std)
        out[name] = folder
    return out


_models, _weights, _memo = {}, {}, {}


def get_model(folders, name, dtype):
    if (name, dtype) not in _models:
        _models[(name, dtype)] = Model.load(folders[name], dtype=dtype, device="cuda")
    return _models[(name, dtype)]


def weights_of(folders, name):
    if name not in _weights:
        _weights[name] = plain_llama.read_safetensors(os.path.join(folders[name], "model.safetensors"))
    return _weights[name]


def n_mixtures(name):
    return sum(1 for l in CONFIGS[name][0]["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe")


def want_logits(folders, name, tokens, choices=None, layers_out=None):
    """The plain implementation's logits.  With `choices` (bfloat16: two scores may be closer than the rounding of the
    router's input) it uses the experts the model chose, none of which may be far from its own choice."""
    key = (name, tuple(tokens))
    if choices is None and layers_out is None and key in _memo:
        return _memo[key]
    slack = [] if choices is not None else None
    out = plain.forward(CONFIGS[name][0], weights_of(folders, name), list(tokens), layers_out=layers_out, choices=choices, slack=slack)
    if choices is None:
        _memo[key] = out
    else:
        assert max(float(s.max()) for s in slack) < 0.02
    return out


@contextlib.contextmanager
def recorded_choices():
    """The experts every call of the router chooses, in order of the calls."""
    calls, real = [], ops.moe_route

    def route(x, router, bias, chosen, *rest, **more):
        real(x, router, bias, chosen, *rest, **more)
        calls.append(chosen.clone())
    ops.moe_route = route
    try:
        yield calls
    finally:
        ops.moe_route = real


def per_mixture(calls, name):
    """Recorded calls of one sequence, fed in any portions, as one array per mixture."""
    n = n_mixtures(name)
    return [np.concatenate([c.cpu().numpy() for c in calls[j::n]]) for j in range(n)]


def check_cut(folders, name, dtype, model, cache, tokens, portions, what):
    with recorded_choices() as calls:
        got = run_cut(model, cache, tokens, portions)
    want = want_logits(folders, name, tokens, per_mixture(calls, name) if dtype == "bfloat16" else None)
    assert_close(got, want, dtype, what)
    return got


def prompts_of(name, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, CONFIGS[name][0]["vocab"], n).tolist() for n in lengths]


# ------------------------------------------------------------------ mixers alone
def mixers_of(dtype, hidden, layers, weights, eps=1e-5):
    """The mixers of `layers`, built by the plan and loaded with `weights`, with a cache for them."""
    raw = {"architecture": "Letanex", "vocab": 8, "width": hidden, "norm": {"eps": eps}, "layers": layers}
    arch = find_architecture(raw)
    plan = arch.plan(arch.read_config(raw))
    rt = Runtime(DEV, TORCH[dtype])
    parts = [build_part("mixer", spec.part("mixer")) for spec in plan.layers]
    for part in parts:
        for p in walk(part):
            p.load(weights, rt)
    requests = [part.cache_requests() for part in parts]
    return rt, parts, lambda pages=6: Cache(requests, [e.cache for e in plan.schedule], max_tokens=64 * pages, max_slots=3,
                                            dtype=TORCH[dtype], device=DEV)


def random_weights(rng, shapes, std=0.3):
    out = {}
    for name, shape in shapes.items():
        w = rng.standard_normal(shape) * std
        if "norm" in name:
            w = 1 + 0.2 * rng.standard_normal(shape)
        out[name] = t32(w).to(torch.bfloat16)
    return out


def attention_shapes(p, m, hidden):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    out = {p + "q": (2 * H * d, hidden), p + "o": (hidden, H * dv), **{p + k: (d,) for k in ("lq1", "lk1", "lq2", "lk2")}}
    if "kv_from" not in m:
        out.update({p + "k": (2 * G * d, hidden), p + "v": (G * dv, hidden)})
    return out


def lightning_shapes(p, m, hidden):
    a, b = m["heads"] * m["dim"], m["heads"] * m["vdim"]
    return {p + "q": (a, hidden), p + "k": (a, hidden), p + "v": (b, hidden), p + "g": (b, hidden), p + "o": (hidden, b), p + "norm": (b,)}


CUTS = lambda T: ([T], [1] * T, [2] * (T // 2), [63, 1, 1, 64, T - 129], [T - 50] + [1] * 50, [3, 2, T - 5])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,factor", [
    (4, 2, 16, 24, 8, 4.0), (3, 1, 5, 7, 4, None), (6, 6, 8, 8, 8, 1.5), (2, 1, 64, 128, 64, 7.0), (8, 2, 64, 64, 32, 2.0), (5, 1, 24, 48, None, None),
    (1, 1, 80, 40, 16, 3.0), (2, 2, 128, 256, 128, None), (4, 1, 128, 128, 64, 2.0), (16, 1, 32, 64, 32, 1.0), (3, 3, 40, 160, 10, 2.0)])
def test_differential_attention_with_keys_of_its_own_and_borrowed(dtype, heads, kv_heads, dim, vdim, dims, factor):
    """Random weights, two layers over one cache; scores large enough that a key, a map, a rotation or a lambda that is
    wrong shows."""
    rng = np.random.default_rng(7)
    hidden, T = 40, 150
    rot = rotation(dims, 200.0, factor) if dims else None
    layers = [attention(heads, kv_heads, dim, vdim, 1.5 / dim ** 0.5, 0.4, rot), attention(heads, kv_heads, dim, vdim, 2.0 / dim ** 0.5, 0.7, rot, kv_from=0)]
    a, b = layers[0]["mixer"], layers[1]["mixer"]
    weights = random_weights(rng, {**attention_shapes("l0.mix.", a, hidden), **attention_shapes("l1.mix.", b, hidden)})
    x = t32(rng.standard_normal((T, hidden))).to(TORCH[dtype])
    w = [short(weights, f"l{i}.mix.") for i in range(2)]
    first, kv = plain.attention_mixer(f64(x), w[0], a, 1e-5)
    second, _ = plain.attention_mixer(f64(x), w[1], b, 1e-5, kv)
    rt, parts, new_cache = mixers_of(dtype, hidden, layers, weights)
    for cuts in CUTS(T):
        got = run_mixers(rt, parts, new_cache(), x, cuts)
        # the difference of two maps that nearly agree is normed: rounding grows with its smallness
        close(got[0], first, dtype, (heads, dim, cuts[:2]), loose=2.0 if dtype == "float32" else 4.0)
        close(got[1], second, dtype, (heads, dim, cuts[:2], "borrowed"), loose=2.0 if dtype == "float32" else 4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("needle", [0, 1, 63, 64, 127, 128, 191, 192, 255, 256, 298])
def test_each_map_finds_one_key_far_away(dtype, dim, needle):
    """One key among 300 stands out for the last query in map 1 of head 0 and in map 2 of head 1: its value comes back as it is
    from the first and with its sign turned from the second.  The first token, page borders, the last query in a prompt,
    alone, and after 39 decoded tokens."""
    T, hidden, mark, vdim = 300, 64, 13, 32
    m = attention(2, 1, dim, vdim, 16.0 / dim, 0.5, rotation(4, 100.0, 50.0))["mixer"]
    pad = lambda rows: torch.cat([rows, torch.zeros(dim - 16, hidden)])
    pick = lambda at: pad(torch.cat([torch.zeros(16, at), torch.eye(16), torch.zeros(16, hidden - at - 16)], dim=1))
    nothing = torch.zeros(dim, hidden)
    weights = {"q": torch.cat([pick(32), nothing, nothing, pick(32)]), "k": torch.cat([pick(0), pick(0)]),
               "v": torch.eye(vdim, hidden), "o": torch.eye(hidden, 2 * vdim), **{k: torch.zeros(dim) for k in ("lq1", "lk1", "lq2", "lk2")}}
    weights = {"l0.mix." + k: v.to(torch.bfloat16) for k, v in weights.items()}
    rng = np.random.default_rng(needle)
    x = rng.standard_normal((T, hidden)) * 0.1
    x[:, mark] = x[:, 32 + mark] = 0.0
    x[needle, mark] = 6.0                                   # the key that stands out ...
    x[-1, 32 + mark] = 6.0                                  # ... for the last query only
    xt = t32(x).to(TORCH[dtype])
    want, _ = plain.attention_mixer(f64(xt), short(weights, "l0.mix."), m, 1e-5)
    assert want[-1, mark] > 2.5 and want[-1, vdim + mark] < -2.5
    rt, parts, new_cache = mixers_of(dtype, hidden, [{"type": "attention", "mixer": m, "mlp": None}], weights)
    for cut in (T, T - 1, T - 40):
        got, = run_mixers(rt, parts, new_cache(), xt, [cut] + [1] * (T - cut))
        close(got[-1:], want[-1:], dtype, (needle, cut), loose=3.0)


@pytest.mark.parametrize("n_heads,n_kv,d,vd,window", [(8, 2, 64, 128, 0), (4, 4, 64, 128, 100), (6, 1, 32, 64, 0), (2, 2, 128, 256, 33), (4, 2, 24, 40, 64)])
def test_tensor_core_differential_attention_against_the_plain_kernel(n_heads, n_kv, d, vd, window):
    """Unequal sequences that start and go on, with and without a window, whole and in shares of the keys, on slots that are not
    in order: against the float kernel on the same bfloat16 rows."""
    from go_tinygrad_b200.cache import KVRequest
    rng = np.random.default_rng(d + vd)
    rt = Runtime(DEV, torch.bfloat16)
    starts, lens = [0, 130, 517, 63], [200, 1, 70, 2]
    caches = {}
    for dt in (torch.bfloat16, torch.float32):
        c = Cache([[KVRequest(n_kv, 2 * d, None, value_dim=vd)]], [None], max_tokens=64 * 24, max_slots=6, dtype=dt, device=DEV)
        slots = [c.open_sequence() for _ in range(6)][::-1][:4]
        c.reserve_many([(s, a + n) for s, a, n in zip(slots, starts, lens)]); c.flush_tables()
        caches[dt] = c
    store = caches[torch.bfloat16].groups[0].storage
    store.copy_(t32(rng.standard_normal(tuple(store.shape))).to(torch.bfloat16))
    caches[torch.float32].groups[0].storage.copy_(store.float())
    ctx = context(rt, lens, starts, slots)
    q = (t32(rng.standard_normal((sum(lens), n_heads * 2 * d))) * 2).to(torch.bfloat16)
    lam, out_scale, eps, scale = 0.6, 0.45, 1e-3, d ** -0.5
    want = torch.empty(sum(lens), n_heads * vd, dtype=torch.float32, device=DEV)
    ops.attention_diff_simple(q.float(), want, caches[torch.float32].handles[0].kv, ctx.token_seq, ctx.slots, ctx.positions, n_heads, scale, lam,
                              out_scale, eps, window)
    kv = caches[torch.bfloat16].handles[0].kv
    for splits in (1, 2, 5, 11):
        out = torch.empty(sum(lens), n_heads * vd, dtype=torch.bfloat16, device=DEV)
        scratch = torch.empty(int(ops._fn("gtg_attention_diff_scratch_floats")(sum(lens), n_heads, vd, splits)) or 1, dtype=torch.float32, device=DEV)
        ops.attention_diff_bf16(q, out, kv, ctx.cu_seqlens, ctx.slots, ctx.start_pos, 4, 200, n_heads, scale, lam, out_scale, eps, window, splits, scratch)
        close(out, f64(want), "bfloat16", splits)


@pytest.mark.parametrize("n_heads,n_kv,window", [(8, 2, 0), (3, 1, 0), (4, 4, 100), (6, 3, 300)])
def test_prompt_differential_attention_on_tcgen05_against_the_plain_kernel(n_heads, n_kv, window):
    """Maps of 64 channels over values of 128: sequences of one token up to several tiles, that start and go on, on slots
    that are not in order; queries from small to so large that the running maximum jumps again and again."""
    from go_tinygrad_b200.cache import KVRequest
    rng = np.random.default_rng(n_heads)
    rt = Runtime(DEV, torch.bfloat16)
    starts, lens = [0, 130, 517, 63, 0], [700, 1, 129, 65, 128]
    caches = {}
    for dt in (torch.bfloat16, torch.float32):
        c = Cache([[KVRequest(n_kv, 128, None, value_dim=128)]], [None], max_tokens=64 * 40, max_slots=6, dtype=dt, device=DEV)
        slots = [c.open_sequence() for _ in range(6)][::-1][:5]
        c.reserve_many([(s, a + n) for s, a, n in zip(slots, starts, lens)]); c.flush_tables()
        caches[dt] = c
    store = caches[torch.bfloat16].groups[0].storage
    store.copy_(t32(rng.standard_normal(tuple(store.shape))).to(torch.bfloat16))
    caches[torch.float32].groups[0].storage.copy_(store.float())
    ctx = context(rt, lens, starts, slots)
    for size in (0.3, 2.0, 12.0):
        q = (t32(rng.standard_normal((sum(lens), n_heads * 128))) * size).to(torch.bfloat16)
        want = torch.empty(sum(lens), n_heads * 128, dtype=torch.float32, device=DEV)
        args = (n_heads, 0.125, -0.4, 0.7, 1e-4, window)
        ops.attention_diff_simple(q.float(), want, caches[torch.float32].handles[0].kv, ctx.token_seq, ctx.slots, ctx.positions, *args)
        out = torch.empty(sum(lens), n_heads * 128, dtype=torch.bfloat16, device=DEV)
        ops.attention_diff_tcgen05(q, out, caches[torch.bfloat16].handles[0].kv, ctx.cu_seqlens, ctx.slots, ctx.start_pos, 5, 700, *args)
        close(out, f64(want), "bfloat16", (n_heads, size))
    assert ops.bounded_wait_failures() == 0


@pytest.mark.parametrize("n_heads,n_kv,d,vd,window", [(8, 2, 64, 128, 0), (16, 1, 64, 128, 0), (4, 4, 32, 64, 100), (12, 2, 128, 256, 0), (3, 1, 24, 40, 64), (6, 2, 128, 64, 1)])
def test_decode_differential_attention_against_the_plain_kernel(n_heads, n_kv, d, vd, window):
    """Sequences of one key up to several shares of pages, whole and in shares."""
    from go_tinygrad_b200.cache import KVRequest
    rng = np.random.default_rng(d + n_heads)
    rt = Runtime(DEV, torch.bfloat16)
    starts = [0, 1, 15, 16, 62, 63, 64, 700, 127, 128]
    n = len(starts)
    caches = {}
    for dt in (torch.bfloat16, torch.float32):
        c = Cache([[KVRequest(n_kv, 2 * d, None, value_dim=vd)]], [None], max_tokens=64 * 40, max_slots=n, dtype=dt, device=DEV)
        slots = [c.open_sequence() for _ in range(n)][::-1]
        c.reserve_many([(s, a + 1) for s, a in zip(slots, starts)]); c.flush_tables()
        caches[dt] = c
    store = caches[torch.bfloat16].groups[0].storage
    store.copy_(t32(rng.standard_normal(tuple(store.shape))).to(torch.bfloat16))
    caches[torch.float32].groups[0].storage.copy_(store.float())
    ctx = context(rt, [1] * n, starts, slots)
    q = (t32(rng.standard_normal((n, n_heads * 2 * d))) * 3).to(torch.bfloat16)
    want = torch.empty(n, n_heads * vd, dtype=torch.float32, device=DEV)
    args = (n_heads, d ** -0.5, 0.5, 0.6, 1e-3, window)
    ops.attention_diff_simple(q.float(), want, caches[torch.float32].handles[0].kv, ctx.token_seq, ctx.slots, ctx.positions, *args)
    for splits in (1, 2, 3, 12):
        out = torch.empty(n, n_heads * vd, dtype=torch.bfloat16, device=DEV)
        scratch = torch.full((int(ops._fn("gtg_attention_diff_scratch_floats")(n, n_heads, vd, splits)) or 1,), float("nan"), dtype=torch.float32, device=DEV)
        ops.attention_diff_bf16(q, out, caches[torch.bfloat16].handles[0].kv, ctx.cu_seqlens, ctx.slots, ctx.start_pos, n, 1, *args, splits, scratch)
        close(out, f64(want), "bfloat16", splits)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay,dim,vdim", [([0.6, 0.9], 16, 24), ([0.99], 5, 7), ([0.3, 0.95, 1.0], 64, 64), ([0.999, 0.5], 128, 128), ([0.9, 0.0], 40, 20),
                                            ([0.97] * 4, 32, 256), ([0.8], 300, 36), ([0.7, 0.999], 256, 512), ([0.9] * 3, 96, 11)])
def test_lightning_attention_carries_its_state_across_portions_and_slots(dtype, decay, dim, vdim):
    rng = np.random.default_rng(11)
    hidden, T = 40, 150
    layer = lightning(decay, dim, vdim)
    weights = random_weights(rng, lightning_shapes("l0.mix.", layer["mixer"], hidden), std=0.2)
    x = t32(rng.standard_normal((T, hidden))).to(TORCH[dtype])
    want = plain.lightning_mixer(f64(x), short(weights, "l0.mix."), layer["mixer"], 1e-5)
    rt, parts, new_cache = mixers_of(dtype, hidden, [layer], weights)
    cache = new_cache()
    for cuts in CUTS(T):
        got, = run_mixers(rt, parts, cache, x, cuts)           # one cache: a slot that is used again starts clean
        close(got, want, dtype, (dim, vdim, cuts[:2]), loose=2.0 if dtype == "float32" else 4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,d,dv,n_seqs", [(2, 16, 8, 3), (3, 64, 128, 2), (1, 128, 96, 3), (4, 32, 64, 2), (2, 7, 5, 3), (1, 256, 64, 2), (2, 48, 80, 2), (1, 512, 8, 1)])
def test_the_recurrence_kernels_on_unequal_sequences(dtype, heads, d, dv, n_seqs):
    """The recurrence alone: unequal sequences in one step, over several tiles of tokens, a second step that continues
    them, then a step of one token each; the state itself after every step."""
    rng = np.random.default_rng(d + dv)
    lens = [[1 + (37 * b + 150 * k) % 290 for b in range(n_seqs)] for k in range(2)] + [[1] * n_seqs]
    total = [sum(l[b] for l in lens) for b in range(n_seqs)]
    width = heads * (2 * d + dv)
    pad = (width + 7) // 8 * 8
    rows = [t32(rng.standard_normal((t, pad))).to(TORCH[dtype]) for t in total]
    decays = np.array([0.999, 0.8, 1.0, 0.3][:heads])
    decay = t32(decays)
    state = torch.zeros(n_seqs + 1, heads, d, dv, dtype=torch.float32, device=DEV)
    slots = torch.tensor([n_seqs - b for b in range(n_seqs)], dtype=torch.int32, device=DEV)       # not in order, slot 0 unused
    at, got = [0] * n_seqs, [[] for _ in range(n_seqs)]
    a = heads * d
    for step_lens in lens:
        qkv = torch.cat([rows[b][at[b]:at[b] + step_lens[b]] for b in range(n_seqs)]).contiguous()
        out = torch.empty(sum(step_lens), heads * dv, dtype=torch.float32, device=DEV)
        cu = torch.tensor(np.concatenate([[0], np.cumsum(step_lens)]), dtype=torch.int32, device=DEV)
        ctx = context(Runtime(DEV, TORCH[dtype]), step_lens, at, slots.tolist())
        ops.lightning_scan(qkv[:, :a], qkv[:, a:2 * a], qkv[:, 2 * a:width], decay, state, out, ctx)
        for b in range(n_seqs):
            got[b].append(f64(out)[int(cu[b]):int(cu[b + 1])])
            at[b] += step_lens[b]
    for b in range(n_seqs):
        r = f64(rows[b])
        for h in range(heads):
            q, k, v = r[:, h * d:(h + 1) * d], r[:, a + h * d:a + (h + 1) * d], r[:, 2 * a + h * dv:2 * a + (h + 1) * dv]
            y = plain.decayed_memory(q, k, v, float(decay[h]))
            close(np.concatenate(got[b])[:, h * dv:(h + 1) * dv], y, "float32", (d, dv, b, h))     # float sums for both types
            S = sum(np.outer(k[t], v[t]) * float(decay[h]) ** (len(r) - 1 - t) for t in range(len(r)))
            close(state[int(slots[b]), h], S, "float32", (d, dv, b, h, "state"))
    assert float(state[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_attention_remembers_its_first_token_where_it_does_not_decay(dtype):
    """Head 0 keeps everything, head 1 forgets a tenth a token.  The last query asks for the first token's key: its value comes
    back after 149 tokens from head 0 alone."""
    T, hidden = 150, 64
    layer = lightning([1.0, 0.9], 8, 8)
    z = lambda r, c: torch.zeros(r, c)
    pick = lambda at: torch.cat([z(8, at), torch.eye(8), z(8, hidden - at - 8)], dim=1)
    weights = {"q": torch.cat([pick(0)] * 2), "k": torch.cat([pick(8)] * 2), "v": torch.cat([pick(16)] * 2), "g": z(16, hidden),
               "norm": torch.ones(16), "o": torch.eye(hidden, 16)}
    weights = {"l0.mix." + k: v.to(torch.bfloat16) for k, v in weights.items()}
    x = np.random.default_rng(3).standard_normal((T, hidden)) * 0.02
    x[0, 8 + 3], x[0, 16:24] = 8.0, np.linspace(4.0, 8.0, 8)          # the first token's key and value
    x[-1, 0 + 3] = 8.0                                                # the last token's query
    xt = t32(x).to(TORCH[dtype])
    want = plain.lightning_mixer(f64(xt), short(weights, "l0.mix."), layer["mixer"], 1e-5)
    assert want[-1, :8].min() > 0.4 and np.abs(want[-1, 8:16]).max() < 0.01
    rt, parts, new_cache = mixers_of(dtype, hidden, [layer], weights)
    for cuts in ([T], [T - 1, 1], [1] * T, [2] * (T // 2), [64, 64, 22]):
        got, = run_mixers(rt, parts, new_cache(), xt, cuts)
        close(got[-1:], want[-1:], dtype, cuts[:2], loose=2.0)


# ------------------------------------------------------------------ norms and feed-forwards alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gate_dtype", ["own", "float32"])
def test_a_row_normed_as_one_head_and_gated(dtype, gate_dtype):
    rng = np.random.default_rng(4)
    for n, width, heads in [(3, 40, 1), (5, 51, 1), (9, 600, 1), (2, 1500, 1), (33, 2048, 1), (4, 3000, 1), (2, 8192, 1), (3, 9000, 1), (2, 2400, 3)]:
        y, g = t32(rng.standard_normal((n, width)) * 3), t32(rng.standard_normal((n, width)) * 2)
        w = t32(1 + 0.2 * rng.standard_normal(width))
        if gate_dtype == "own":
            g = g.to(TORCH[dtype])
        out = torch.empty(n, width, dtype=TORCH[dtype], device=DEV)
        ops.head_norm_gate(y, g, w, 1e-3, out, heads)
        want = plain.unit_rms(f64(y).reshape(n, heads, -1), 1e-3).reshape(n, width) * f64(w) * plain.sigmoid(f64(g))
        close(out, want, dtype, (n, width))


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_normed_update_joins_the_hidden_state_which_is_normed_again(dtype):
    rng = np.random.default_rng(3)
    rt = Runtime(DEV, TORCH[dtype])
    for n, h in [(1, 8), (5, 72), (70, 1000), (3, 51), (2, 4096), (3, 8192), (3, 9000)]:
        x, u = rng.standard_normal((n, h)) * 3 + 1, rng.standard_normal((n, h)) * 20 + 5
        w = [t32(1 + 0.3 * rng.standard_normal(h)) for _ in range(3)]
        norms = [build_part("norm", PartSpec("layernorm", {"size": h, "eps": e, "weight": f"w{i}", "bias": b})) for i, (e, b) in
                 enumerate([(0.3, None), (1e-3, None), (1e-3, "w2")])]
        for norm in norms:
            norm.load({f"w{i}": w[i] for i in range(3)}, rt)
        norms[2].weight = norms[1].weight
        for kind in ("float32", dtype):
            update = t32(u).to(TORCH[kind])
            total = f64(t32(x)) + plain.layer_norm(f64(update), f64(w[0]), 0.3)
            for norm, bias in ((norms[1], 0.0), (norms[2], f64(w[2]))):
                want = plain.layer_norm(total, f64(w[1]), 1e-3) + bias
                rows = torch.tensor([n - 1, 0], dtype=torch.int32, device=DEV)
                for picked in (rows, None):
                    stream = ResidualStream(t32(x).clone(), update)
                    stream.pending_norm = (norms[0].weight, norms[0].eps)
                    got = norm.forward(stream, context(rt, [n], [0], [0]), rows=picked)
                    if picked is None:
                        assert stream.pending is None and stream.pending_norm is None
                        close(stream.residual, total, "float32")
                        close(got, want, dtype, (n, h))
                    else:
                        assert stream.pending is update and torch.equal(stream.residual, t32(x))       # the wanted rows only: nothing is written back
                        close(got, want[[n - 1, 0]], dtype, (n, h, "rows"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("h,top,identities,shared", [(64, 2, True, True), (51, 3, True, False), (2048, 4, False, True), (9000, 1, True, True), (72, 9, True, True)])
def test_the_norm_that_sums_a_mixtures_rows_itself(dtype, h, top, identities, shared):
    rng = np.random.default_rng(h)
    n, rows = 37, 400
    rt = Runtime(DEV, TORCH[dtype])
    y, x = t32(rng.standard_normal((rows, h)) * 3), t32(rng.standard_normal((n, h))).to(TORCH[dtype])
    item_row = rng.integers(-1 if identities else 0, rows, n * top)
    weights, base = t32(rng.uniform(0.1, 2.0, (n, top))), t32(rng.standard_normal((n, h))) if shared else None
    update = ops.ExpertSum(y, torch.tensor(item_row, dtype=torch.int32, device=DEV), weights, x if identities else None, base)
    want = np.zeros((n, h))
    for t in range(n):
        for k in range(top):
            row = item_row[t * top + k]
            want[t] += float(weights[t, k]) * (f64(y[row]) if row >= 0 else f64(x[t]))
    want = want + (f64(base) if shared else 0.0)
    close(update.float(), want, "float32")
    res, w = rng.standard_normal((n, h)) * 2, [t32(1 + 0.3 * rng.standard_normal(h)) for _ in range(2)]
    residual, out = t32(res).clone(), torch.empty(n, h, dtype=TORCH[dtype], device=DEV)
    ops.layernorm_add_layernorm(residual, update, w[0], 1e-5, w[1], None, 1e-5, out)
    total = f64(t32(res)) + plain.layer_norm(want, f64(w[0]), 1e-5)
    close(residual, total, "float32")
    close(out, plain.layer_norm(total, f64(w[1]), 1e-5), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,limit", [(64, 96, 1.5), (72, 40, 0.4), (51, 13, 2.0), (256, 512, 3.0)])
def test_gated_feed_forward_with_clamped_gates(dtype, hidden, ff, limit):
    """Few rows and many, so that every product forms the gate in its epilogue; sums on both sides of both limits."""
    rng = np.random.default_rng(5)
    w = {k: t32(rng.standard_normal(s) * 4 / hidden ** 0.5).to(torch.bfloat16) for k, s in (("gate", (ff, hidden)), ("up", (ff, hidden)), ("down", (hidden, ff)))}
    rt = Runtime(DEV, TORCH[dtype])
    part = build_part("feed_forward", PartSpec("swiglu", {"hidden_size": hidden, "intermediate_size": ff, "gate_limit": limit, **{k: k for k in w}}))
    part.load(w, rt)
    for n in (1, 3, 16, 17, 40, 100, 129, 300):
        x = t32(rng.standard_normal((n, hidden))).to(TORCH[dtype])
        g, u = f64(x) @ f64(w["gate"]).T, f64(x) @ f64(w["up"]).T
        assert (g > limit).any() and (u > limit).any() and (u < -limit).any() and (g < -limit).any()
        want = plain.clamped_expert(f64(x), f64(w["gate"]), f64(w["up"]), f64(w["down"]), limit)
        close(part.forward(x, context(rt, [n], [0], [0])), want, dtype, (n, hidden))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,experts,identity,top,shared", [
    (64, 48, 8, 4, 2, 80), (72, 40, 5, 2, 5, None), (51, 13, 3, 0, 1, 19), (64, 32, 1, 6, 4, 16), (128, 64, 16, 4, 8, 128), (40, 24, 40, 30, 3, None), (64, 64, 2, 1, 3, 64)])
def test_mixture_with_identities_a_correction_and_a_shared_expert(dtype, hidden, ff, experts, identity, top, shared):
    """Router weights so large that no choice is a close call; steps of few tokens and of many; a correction that turns choices
    without touching weights; tokens that choose identities alone."""
    rng = np.random.default_rng(experts)
    outputs = experts + identity
    limit = {"e": 1.1, "shared": 0.7}
    w = {"router": t32(rng.standard_normal((outputs, hidden)) * 0.4).to(torch.bfloat16), "correction": t32(rng.uniform(-0.4, 0.4, outputs)).to(torch.bfloat16)}
    for e in [f"e{e}" for e in range(experts)] + (["shared"] if shared else []):
        n_ff = shared if e == "shared" else ff
        w.update({f"{e}.gate": (n_ff, hidden), f"{e}.up": (n_ff, hidden), f"{e}.down": (hidden, n_ff)})
    w = {k: t32(rng.standard_normal(v) * 2 / hidden ** 0.5).to(torch.bfloat16) if isinstance(v, tuple) else v for k, v in w.items()}
    spec = None
    if shared:
        spec = PartSpec("swiglu", {"hidden_size": hidden, "intermediate_size": shared, "gate_limit": limit["shared"],
                                   **{k: "shared." + k for k in ("gate", "up", "down")}})
    rt = Runtime(DEV, TORCH[dtype])
    part = build_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": hidden, "intermediate_size": ff, "n_experts": experts, "identity": identity, "top": top, "scoring": "softmax_all",
        "correction": "correction", "weight_scale": 1.6, "gate_limit": limit["e"], "router": "router", "shared": spec,
        **{k: "e{e}." + k for k in ("gate", "up", "down")}}))
    for p in walk(part):
        p.load(w, rt)
    w64 = {k: f64(v) for k, v in w.items()}
    mlp = moe(ff, limit["e"], experts, top, identity, 1.6, (shared, limit["shared"]) if shared else None)
    turned = alone = 0
    for n in (1, 7, 70, 400, 1100):
        x = t32(rng.standard_normal((n, hidden))).to(TORCH[dtype])
        with recorded_choices() as calls:
            ctx = context(rt, [n], [0], [0])
            ctx.float_updates = n % 2 == 0
            got = part.forward(x, ctx)
        assert got.dtype == (torch.float32 if ctx.float_updates else TORCH[dtype])
        chosen = calls[0].cpu().numpy()
        want_chosen, _ = plain.route(f64(x), w64["router"], w64["correction"], top, 1.6)
        sure = -np.sort(-(plain.scores(f64(x), w64["router"]) + w64["correction"]), axis=-1)
        sure = (sure[:, top - 1] - sure[:, top] > 1e-4) if top < outputs else np.ones(n, bool)
        assert (np.sort(chosen, axis=1) == np.sort(want_chosen, axis=1))[sure].all() and sure.mean() > 0.9
        bare, _ = plain.route(f64(x), w64["router"], np.zeros(outputs), top, 1.6)
        turned += (np.sort(bare, axis=1) != np.sort(want_chosen, axis=1)).any(axis=1).sum()
        alone += (chosen >= experts).all(axis=1).sum()
        want = plain.mixture(f64(x), w64, "", mlp, chosen)
        close(got, want, dtype, (n, hidden, experts))
    assert turned > 0 or top == outputs
    assert alone > 0 or identity < 2 or top > identity


# ------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_whole_prompts_of_many_lengths_and_the_hidden_state_after_every_layer(folders, name, dtype):
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 6)
    for p in prompts_of(name, [1, 2, 3, 17, 63, 64, 65, 129, 230]):
        check_cut(folders, name, dtype, model, cache, p, [len(p)], f"{name} {dtype} whole prompt of {len(p)}")
    assert cache.open_slots() == []
    p = prompts_of(name, [90], seed=3)[0]
    hidden, layers = [], []
    model.op_hook = lambda s, l, op, t: hidden.append(f64(t)) if op == "hidden_post_ffn" else None
    try:
        with recorded_choices() as calls:
            run_cut(model, cache, p, [len(p)])
    finally:
        model.op_hook = None
    want_logits(folders, name, p, per_mixture(calls, name), layers_out=layers)
    assert len(hidden) == len(layers)
    for i, (g, w) in enumerate(zip(hidden, layers)):
        close(g, w, dtype, f"{name} {dtype} hidden state after layer {i}", loose=4.0)


@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_steps_launched_back_to_back_are_the_steps_launched_one_kernel_at_a_time(folders, name):
    """Every kernel of a step may begin while the one before it runs: nothing may be read before it is written.  Twenty
    prompts through one workspace, against the same with every launch waited for."""
    model = get_model(folders, name, "bfloat16")
    cache = model.new_cache(max_tokens=64 * 8)
    prompts = prompts_of(name, [97, 300, 40, 150, 5] * 4, seed=31)
    flowing = [run_cut(model, cache, p, [len(p)]) for p in prompts]
    real = ops._check

    def waited(code, what):
        real(code, what)
        torch.cuda.synchronize()
    ops._check = waited
    try:
        for p, got in zip(prompts, flowing):
            np.testing.assert_array_equal(got, run_cut(model, cache, p, [len(p)]))
    finally:
        ops._check = real


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_portions_down_to_two_tokens_and_token_by_token_from_the_start(folders, name, dtype):
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 6)
    p = prompts_of(name, [150], seed=5)[0]
    rows = {}
    for portions in ([150], [1], [2], [3, 2, 1, 16, 15, 17, 64], [63, 1, 1, 64, 2], [100, 1]):
        rows[tuple(portions)] = check_cut(folders, name, dtype, model, cache, p, portions, f"{name} {dtype} portions {portions}")
    if dtype == "float32":
        # sums walk keys and states in one order whatever the cut
        scale = np.abs(rows[(150,)]).max()
        for portions, got in rows.items():
            np.testing.assert_allclose(got, rows[(150,)], rtol=0, atol=2e-5 * scale, err_msg=str(portions))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_long_decoding_across_page_borders(folders, name, dtype):
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 6)
    p = prompts_of(name, [5 + 280], seed=6)[0]
    check_cut(folders, name, dtype, model, cache, p, [5, 1], f"{name} {dtype} 280 tokens decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_unequal_batches_against_each_alone_with_slots_and_pages_used_again(folders, name, dtype):
    """Three batches through a cache too small for two of them: the slots and pages
    of finished requests, with their old rows and states, go to new ones.  In a batch every
    request is decoded to its own length and leaves when it ends."""
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 7, max_slots=4)
    n_mix = n_mixtures(name)
    batches = [[(5, 9), (70, 3), (17, 20), (1, 12)], [(64, 1), (130, 6), (3, 33)], [(40, 8), (128, 2), (9, 9), (2, 2)]]
    for bi, batch in enumerate(batches):
        prompts = prompts_of(name, [a + b for a, b in batch], seed=20 + bi)
        slots = [cache.open_sequence() for _ in batch]
        got, choices = [[] for _ in batch], [[[] for _ in range(n_mix)] for _ in batch]

        def run(live, entries):
            with recorded_choices() as calls:
                flat = step(model, cache, entries).float().cpu().numpy()
            o = 0
            for i, e in zip(live, entries):
                n = len(e.tokens)
                got[i].append(flat[o:o + n])
                for j in range(n_mix):
                    choices[i][j].append(calls[j].cpu().numpy()[o:o + n])
                o += n
        run(range(len(batch)), [StepEntry(slots[i], p[:plen], list(range(plen))) for i, ((plen, _), p) in enumerate(zip(batch, prompts))])
        t = 0
        while True:
            live = [i for i in range(len(batch)) if t < batch[i][1]]
            if not live:
                break
            run(live, [StepEntry(slots[i], [prompts[i][batch[i][0] + t]], [0]) for i in live])
            for i in live:
                if t + 1 >= batch[i][1]:
                    cache.close_sequence(slots[i])
            t += 1
        for i in range(len(batch)):
            followed = [np.concatenate(c) for c in choices[i]] if dtype == "bfloat16" else None
            assert_close(np.concatenate(got[i]), want_logits(folders, name, prompts[i], followed), dtype, f"{name} {dtype} batch {bi} request {i}")
        assert cache.open_slots() == []
    assert all(free == 7 for free in cache.free_pages())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_greedy_generation_through_the_scheduler(folders, name, dtype):
    model = get_model(folders, name, dtype)
    assert model.capturable
    prompts = prompts_of(name, [5, 17, 40, 1], seed=7)
    cfg, w = CONFIGS[name][0], weights_of(folders, name)
    for use_graph in (True, False):
        results = lib.generate(model, prompts, [12, 6, 9, 12], stop=[], use_graph=use_graph)
        assert [len(r.tokens) for r in results] == [12, 6, 9, 12]
        for p, r in zip(prompts, results):
            tokens = list(p) + r.tokens
            choices = None
            if dtype == "bfloat16":                               # the experts the model chooses for these tokens
                with recorded_choices() as calls:
                    run_cut(model, model.new_cache(max_tokens=128), tokens, [len(p), 1])
                choices = per_mixture(calls, name)
            logits = want_logits(folders, name, tokens, choices)  # each token is one the plain model could have chosen there
            for t, tok in enumerate(r.tokens):
                row = logits[len(p) - 1 + t]
                slack = (1e-4 if dtype == "float32" else 5e-2) * max(1.0, np.abs(row).max())
                assert row[tok] >= row.max() - slack, (use_graph, t)
    if dtype == "float32":
        assert results[1].tokens == plain.greedy(cfg, w, prompts[1], 6)


def test_trace_replay_and_command_line(folders, tmp_path):
    """bin/trace_run with a batch that starts together and shrinks, and llmgen with token ids."""
    name = "P"
    a, b = prompts_of(name, [30, 9], seed=8)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:20], "want": [0, 19]}, {"id": "y", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[20:21], "want": [0]}, {"id": "y", "tokens": b[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[21:22], "want": []}, {"id": "y", "tokens": b[8:9], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[22:], "want": [7]}], "end": ["x"]}]
    out = str(tmp_path / "out")
    proc = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folders[name], "--dtype", "float32",
                           "--out", out, "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = want_logits(folders, name, a), want_logits(folders, name, b)
    V = CONFIGS[name][0]["vocab"]
    read = lambda i: np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, V)
    assert_close(read(0), np.stack([wa[0], wa[19], wb[6]]), "float32", "step 0")
    assert_close(read(1), wa[20:21], "float32", "step 1")
    assert_close(read(2), wb[8:9], "float32", "step 2")
    assert_close(read(3), wa[29:30], "float32", "step 3")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "llmgen"), "-model", folders[name], "-ids",
                           ",".join(str(t) for t in b), "-tokens", "5", "-dtype", "float32"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    want = plain.greedy(CONFIGS[name][0], weights_of(folders, name), b, 5)
    assert " ".join(str(t) for t in want) in proc.stdout.replace(",", " ").replace("[", " ").replace("]", " ")
