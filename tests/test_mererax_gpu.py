"""The Mererax design in the engine against its plain implementation
(plain_mererax.py): every mechanism alone, then whole models of three small
configurations that differ in every size and option, under every way of
cutting the same requests into steps."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import go_tinygrad_b200 as lib
import plain_llama
import plain_mererax as plain
from go_tinygrad_b200.cache import Cache
from go_tinygrad_b200.config.registry import find_architecture
from go_tinygrad_b200.engine import Model, StepEntry, step
from go_tinygrad_b200.kernels import build, ops
from go_tinygrad_b200.parts import PartSpec, Runtime, build_part, walk
from go_tinygrad_b200.parts.base import ResidualStream
from go_tinygrad_b200.weights.safetensors_io import TensorSource, write_safetensors
from conftest import ROOT, assert_close
from test_megerax_gpu import DEV, DTYPES, TORCH, close, f64, run_cut, run_mixers, short, t32
from test_mererax_config import left, mamba, parallel, right
from test_parts_gpu import context

pytestmark = pytest.mark.gpu

# P: heads in groups of three, sizes that are multiples of 8 or 4 or of nothing, a layer without a feed-forward,
# layers that run another's tensors (a pair, a scan, and one whose source stands behind it), one to four taps.
CONFIG_P = {
    "architecture": "Mererax", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0},
    "layers": [
        mamba(104, 10, 5, 4, 100),
        parallel(left(6, 2, 24, 0.3, 0.25, 32), right(4, 20, 12, 9.0), 64),
        mamba(50, 20, 8, 3),
        parallel(left(6, 2, 24, 0.3, 0.25, 32), right(4, 20, 12, 9.0), 64, weights_of=1),
        mamba(40, 5, 3, 2, 36, weights_of=6),
        parallel(left(3, 3, 10, 0.2), right(2, 36, 40, 15.0)),
        mamba(40, 5, 3, 2, 36),
        mamba(50, 20, 8, 3, weights_of=2),
        mamba(72, 33, 16, 1, 24),
    ],
}
# Q: sizes the tensor-core kernels take: heads of 64 and 128 channels, states of 16 and 128, one key head for four.
CONFIG_Q = {
    "architecture": "Mererax", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0},
    "layers": [
        parallel(left(8, 2, 64, 0.1, 0.4, 100), right(4, 64, 128, 15.0), 256),
        mamba(256, 16, 16, 4, 128),
        parallel(left(4, 1, 128, 0.08, 0.1, 17), right(2, 128, 64, 6.0), 128),
        mamba(192, 128, 24, 3, 192),
        parallel(left(4, 1, 128, 0.08, 0.1, 17), right(2, 128, 64, 6.0), 128, weights_of=2),
    ],
}
# U: nothing is a multiple of 8, 4 or 2 where the design allows it; no query temperature; an odd width.
CONFIG_U = {
    "architecture": "Mererax", "vocab": 101, "width": 51, "norm": {"eps": 1e-4}, "embedding": {"scale": 2.0},
    "layers": [
        parallel(left(3, 1, 5, 0.4), right(3, 9, 7, 3.0), 11),
        mamba(13, 3, 1, 5, 9),
        parallel(left(5, 5, 7, 0.3, 0.7, 1), right(1, 3, 5, 20.0)),
        mamba(27, 1, 2, 2, 13),
    ],
}
CONFIGS = {"P": (CONFIG_P, 3, 0.12, 0.1), "Q": (CONFIG_Q, 4, 0.08, 0.05), "U": (CONFIG_U, 5, 0.15, 0.1)}     # configuration, seed, std, norm std


def agree_on_the_first_tokens(folder):
    """At a sequence's first token a memory head's read-out is (k . q) v, and its norm leaves the sign of k . q: with
    random weights it may lie so near zero that rounding in bfloat16 turns it.  Queries that lean towards the keys
    keep it away from there."""
    path = os.path.join(folder, "model.safetensors")
    with TensorSource(folder) as src:
        tensors = {n: src.tensor(n) for n in src.names()}
    for n in tensors:
        if n.endswith(".right.q"):
            tensors[n] = (tensors[n].float() + tensors[n[:-1] + "k"].float()).to(tensors[n].dtype)
    write_safetensors(path, tensors)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, (cfg, seed, std, norm_std) in CONFIGS.items():
        folder = str(tmp_path_factory.mktemp(f"mererax_{name}"))
        lib.write_random_model(folder, cfg, seed=seed, dtype="bfloat16", std=std, norm_std=norm_std)
        agree_on_the_first_tokens(folder)
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


def want_logits(folders, name, tokens):
    key = (name, tuple(tokens))
    if key not in _memo:
        _memo[key] = plain.forward(CONFIGS[name][0], weights_of(folders, name), list(tokens))
    return _memo[key]


def prompts_of(name, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, CONFIGS[name][0]["vocab"], n).tolist() for n in lengths]


# ------------------------------------------------------------------ mixers alone
def mixer_of(dtype, hidden, layer, weights, eps=1e-5, side=None):
    """The mixer of one layer, built by the plan and loaded with `weights` (names l0.mix.*), with a
    cache for it; `side`: one branch of a pair, by itself."""
    raw = {"architecture": "Mererax", "vocab": 8, "width": hidden, "norm": {"eps": eps}, "layers": [layer]}
    arch = find_architecture(raw)
    spec = arch.plan(arch.read_config(raw)).layers[0].part("mixer")
    rt = Runtime(DEV, TORCH[dtype])
    part = build_part("mixer", spec.params[side] if side else spec)
    for p in walk(part):
        p.load(weights, rt)
    requests = [[r for p in walk(part) if hasattr(p, "cache_requests") for r in p.cache_requests()]]
    return rt, [part], lambda pages=6: Cache(requests, [None], max_tokens=64 * pages, max_slots=3, dtype=TORCH[dtype], device=DEV)


def random_weights(rng, shapes, std=0.3):
    out = {}
    for name, shape in shapes.items():
        w = rng.standard_normal(shape) * std
        if name.endswith(("norm", "out")):
            w = 1 + 0.2 * rng.standard_normal(shape)
        out[name] = t32(w).to(torch.bfloat16)
    return out


def left_shapes(p, m, hidden):
    q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    return {p + "q": (q, hidden), p + "k": (k, hidden), p + "q.norm": (q,), p + "k.norm": (k,), p + "o": (hidden, q)}


def right_shapes(p, m, hidden):
    a, b, h = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"]
    return {p + "q": (a, hidden), p + "k": (a, hidden), p + "v": (b, hidden), p + "g": (b, hidden), p + "o": (hidden, b), p + "norm": (b,),
            p + "i": (h, hidden), p + "i.b": (h,), p + "f": (h, hidden), p + "f.b": (h,)}


def mamba_shapes(p, m, hidden):
    c, n, r = m["inner"], m["state"], m["dt_rank"]
    return {p + "in": (2 * c, hidden), p + "conv": (c, m["conv"]), p + "conv.b": (c,), p + "x": (r + 2 * n, c), p + "dt": (c, r),
            p + "dt.b": (c,), p + "A_log": (c, n), p + "D": (c,), p + "o": (hidden, c)}


CUTS = lambda T: ([T], [1] * T, [2] * (T // 2), [63, 1, 1, 64, T - 129], [T - 50] + [1] * 50, [3, 2, T - 5])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,coef,every", [
    (4, 2, 12, 0.5, 16), (3, 1, 5, 0.7, 1), (6, 6, 8, None, None), (2, 1, 64, 0.3, 33), (8, 2, 128, -0.1, 64), (5, 1, 24, 0.4, 1000),
    (1, 1, 80, 0.2, 7)])
def test_attention_over_normed_rows_with_growing_queries_and_a_penalty_on_the_distance(dtype, heads, kv_heads, dim, coef, every):
    """Random weights; queries that grow at every token, every few tokens and not at all; head counts that are
    no power of two; scores large enough that a slope, a distance or a temperature one off shows."""
    rng = np.random.default_rng(7)
    hidden, T = 40, 150
    m = left(heads, kv_heads, dim, 2.0 / dim ** 0.5, coef, every)
    weights = random_weights(rng, left_shapes("l0.mix.left.", m, hidden))
    x = t32(rng.standard_normal((T, hidden))).to(TORCH[dtype])
    w = short(weights, "l0.mix.left.")
    want = plain.attention_mixer(f64(x), w, m, 1e-5)
    # what the test can tell apart: no penalty, and the row norms taken head by head
    real, plain.distance_slopes = plain.distance_slopes, lambda h: np.zeros(h)
    try:
        assert np.abs(plain.attention_mixer(f64(x), w, m, 1e-5) - want).max() > (0.1 if heads > 1 else 0.05) * np.abs(want).max()
    finally:
        plain.distance_slopes = real
    rt, parts, new_cache = mixer_of(dtype, hidden, parallel(m, right(1, 1, 1, 1.0)), weights, side="left")
    for cuts in CUTS(T):
        got, = run_mixers(rt, parts, new_cache(), x, cuts)
        close(got, want, dtype, (heads, dim, cuts[:2]), loose=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("needle", [0, 1, 63, 64, 127, 128, 191, 192, 255, 256, 298])
def test_attention_finds_one_key_far_away_through_the_head_with_the_gentle_slope_only(dtype, dim, needle):
    """One key among 300 stands out for the last query.  Head 1 (a penalty of 1.2 over 300 tokens) returns its value
    from anywhere; head 0 (a penalty of 18) not from the first tokens: the first token, page borders, the last query in a
    prompt, alone, and after 39 decoded tokens."""
    T, hidden, mark = 300, 64, 13
    m = left(2, 1, dim, 16.0 / dim, 0.25, 150)
    pick = lambda at: torch.cat([torch.cat([torch.zeros(16, at), torch.eye(16), torch.zeros(16, hidden - at - 16)], dim=1),
                                 torch.zeros(dim - 16, hidden)])
    weights = {"q": torch.cat([pick(32)] * 2), "k": pick(0), "q.norm": torch.ones(2 * dim), "k.norm": torch.ones(dim),
               "o": torch.cat([torch.eye(32, 2 * dim) if dim == 16 else torch.cat([torch.eye(16, 2 * dim),
                               torch.cat([torch.zeros(16, dim), torch.eye(16, dim)], dim=1)]), torch.zeros(32, 2 * dim)])}
    weights = {"l0.mix.left." + k: v.to(torch.bfloat16) for k, v in weights.items()}
    rng = np.random.default_rng(needle)
    x = rng.standard_normal((T, hidden)) * 0.1
    x[:, mark] = 0.0
    x[needle, mark] = 9.0                                   # the key that stands out ...
    x[-1, 32 + mark] = 9.0                                  # ... for the last query only
    xt = t32(x).to(TORCH[dtype])
    want = plain.attention_mixer(f64(xt), short(weights, "l0.mix.left."), m, 1e-5)
    assert want[-1, 16 + mark] > 8.5
    assert want[-1, mark] > 8.0 if needle > 60 else want[-1, mark] < 2.5
    rt, parts, new_cache = mixer_of(dtype, hidden, parallel(m, right(1, 1, 1, 1.0)), weights, side="left")
    for cut in (T, T - 1, T - 40):
        got, = run_mixers(rt, parts, new_cache(), xt, [cut] + [1] * (T - cut))
        close(got, want, dtype, (needle, cut), loose=3.0)


@pytest.mark.parametrize("n_heads,n_kv,hd,n,chunks", [(8, 2, 64, 700, 1), (4, 4, 128, 500, 3), (16, 2, 128, 300, 2), (2, 1, 64, 1500, 1)])
def test_prompt_attention_on_tcgen05_with_slopes_against_the_plain_kernel(n_heads, n_kv, hd, n, chunks):
    """The prompt kernel walks sloped heads from the nearest keys to the farthest; the warp-level kernel the other
    way; both against the float kernel on the same bfloat16 rows, whole prompts and continued ones, with and
    without a cap."""
    rng = np.random.default_rng(hd + n)
    from go_tinygrad_b200.cache import KVRequest
    rt = Runtime(DEV, torch.bfloat16)
    caches = {}
    for dt in (torch.bfloat16, torch.float32):
        c = Cache([[KVRequest(n_kv, hd, None)]], [None], max_tokens=64 * ((n + 63) // 64) + 64, max_slots=1, dtype=dt, device=DEV)
        slot = c.open_sequence()
        c.reserve_many([(slot, n)]); c.flush_tables()
        caches[dt] = c
    store = caches[torch.bfloat16].groups[0].storage
    store.copy_(t32(rng.standard_normal(tuple(store.shape))).to(torch.bfloat16))
    caches[torch.float32].groups[0].storage.copy_(store.float())
    slopes = t32(plain.distance_slopes(n_heads))
    q = (t32(rng.standard_normal((n, n_heads * hd))) * 2).to(torch.bfloat16)
    at = 0
    for part in np.array_split(np.arange(n), chunks):
        m = len(part)
        ctx = context(rt, [m], [at], [0])
        qq = q[at:at + m].contiguous()
        for cap in (0.0, 20.0):
            out = torch.empty(m, n_heads * hd, dtype=torch.bfloat16, device=DEV)
            want = torch.empty(m, n_heads * hd, dtype=torch.float32, device=DEV)
            ops.attention_simple(qq.float(), want, caches[torch.float32].handles[0].kv, ctx.token_seq, ctx.slots, ctx.positions, n_heads,
                                 hd ** -0.5, softcap=cap, slopes=slopes)
            ops.attention_prefill_tcgen05(qq, out, caches[torch.bfloat16].handles[0].kv, ctx.cu_seqlens, ctx.slots, ctx.start_pos, 1, m,
                                          n_heads, hd ** -0.5, softcap=cap, slopes=slopes)
            close(out, f64(want), "bfloat16", ("tcgen05", at, cap))
            ops.attention_masked_bf16(qq, out, caches[torch.bfloat16].handles[0].kv, ctx.cu_seqlens, ctx.slots, ctx.start_pos, 1, m,
                                      n_heads, hd ** -0.5, softcap=cap, slopes=slopes)
            close(out, f64(want), "bfloat16", ("masked", at, cap))
        at += m


# ------------------------------------------------------------------ the matrix memory
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,cap,i_mean,f_mean", [
    (3, 10, 6, 9.0, 0.0, 2.0), (2, 64, 64, 15.0, 1.0, 4.0), (4, 128, 32, 6.0, -2.0, 3.0), (1, 7, 3, 3.0, 2.0, -1.0), (2, 200, 20, 12.0, 4.0, 5.0),
    (6, 40, 130, 15.0, -6.0, 6.0), (2, 300, 12, 1.0, 0.0, 0.0)])
def test_the_matrix_memory_carries_its_state_across_portions_and_slots(dtype, heads, dim, vdim, cap, i_mean, f_mean):
    """Random weights and gates of many sizes: input gates far above and far below the forget gate's, tight and loose
    caps; state, normaliser and maximum go from step to step through the cache; a slot that is used again starts
    from zero; two sequences side by side."""
    rng = np.random.default_rng(13)
    hidden, T = 40, 150
    m = right(heads, dim, vdim, cap)
    weights = random_weights(rng, right_shapes("l0.mix.right.", m, hidden), std=0.3)
    weights["l0.mix.right.q"] = (weights["l0.mix.right.q"].float() + weights["l0.mix.right.k"].float()).to(torch.bfloat16)   # see agree_on_the_first_tokens
    weights["l0.mix.right.i.b"] = t32(i_mean + rng.standard_normal(heads)).to(torch.bfloat16)
    weights["l0.mix.right.f.b"] = t32(f_mean + rng.standard_normal(heads)).to(torch.bfloat16)
    x = t32(rng.standard_normal((T, hidden))).to(TORCH[dtype])
    want = plain.memory_mixer(f64(x), short(weights, "l0.mix.right."), m, 1e-5)
    rt, parts, new_cache = mixer_of(dtype, hidden, parallel(left(1, 1, 8, 1.0), m), weights, side="right")
    cache = new_cache()
    loose = 3.0 if dtype == "float32" else 4.0              # near a small denominator a head's direction turns quickly
    for cuts in CUTS(T):
        got, = run_mixers(rt, parts, cache, x, cuts)        # the same cache: every run takes a slot another run has left
        close(got, want, dtype, (heads, dim, vdim, cuts[:2]), loose=loose)
    y = t32(rng.standard_normal((50, hidden))).to(TORCH[dtype])
    want_y = plain.memory_mixer(f64(y), short(weights, "l0.mix.right."), m, 1e-5)
    a, b = cache.open_sequence(), cache.open_sequence()
    got_x, got_y = [], []
    for (na, nb) in ((37, 20), (1, 1), (1, 1), (111, 28)):
        ax, ay = cache.length(a), cache.length(b)
        cache.reserve_many([(a, ax + na), (b, ay + nb)]); cache.flush_tables()
        ctx = context(rt, [na, nb], [ax, ay], [a, b])
        out = f64(parts[0].forward(torch.cat([x[ax:ax + na], y[ay:ay + nb]]).contiguous(), ctx, cache.handles[0]))
        got_x.append(out[:na]); got_y.append(out[na:])
        cache.advance(a, na); cache.advance(b, nb)
    close(np.concatenate(got_x), want, dtype, "first of two", loose=loose)
    close(np.concatenate(got_y), want_y, dtype, "second of two", loose=loose)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv,n_seqs,pad", [(8, 3, 2, 0), (16, 32, 3, 0), (64, 64, 5, 0), (64, 100, 2, 3), (72, 64, 1, 0), (128, 96, 2, 0),
                                             (128, 31, 3, 8), (200, 32, 1, 0), (256, 33, 2, 0), (256, 128, 1, 0), (304, 16, 1, 0), (512, 20, 2, 0)])
@pytest.mark.parametrize("warps", [1, 2, 4, 8])
def test_the_recurrence_kernel_for_every_shape_of_block(dtype, d, dv, n_seqs, pad, warps):
    """The recurrence alone, numerators over denominators, for every block the launcher can pick: unequal sequences in
    one step, a second step that continues them, then a step of one token each; rows that allow 16-byte loads and
    rows that do not.  Both sides of the denominator's maximum occur."""
    rng = np.random.default_rng(d + dv)
    H, cap = 2, 8.0
    lens = [[1 + (7 * b + 5 * k) % 23 for b in range(n_seqs)] for k in range(2)] + [[1] * n_seqs]
    total = [sum(l[b] for l in lens) for b in range(n_seqs)]
    width = H * (2 * d + dv) + pad
    rows = [t32(rng.standard_normal((total[b], width))).to(TORCH[dtype]) for b in range(n_seqs)]
    gates = [t32(rng.standard_normal((total[b], 2 * H)) * 3) for b in range(n_seqs)]
    bias = t32([-1.0, 2.0, 1.0, 3.0])
    state = tuple(torch.zeros((n_seqs + 1,) + s, dtype=torch.float32, device=DEV) for s in ((H, d, dv), (H, d), (H, dv + 1)))
    slots = torch.tensor([n_seqs - b for b in range(n_seqs)], dtype=torch.int32, device=DEV)       # not in order, slot 0 unused
    at, got = [0] * n_seqs, [[] for _ in range(n_seqs)]
    shape = build.library("mlstm").gtg_mlstm_scan_shape
    shape(warps)
    try:
        for step_lens in lens:
            cat = lambda parts: torch.cat([p[at[b]:at[b] + step_lens[b]] for b, p in enumerate(parts)]).contiguous()
            r, g, n = cat(rows), cat(gates), sum(step_lens)
            num = torch.empty(n, H * dv, dtype=torch.float32, device=DEV)
            den = torch.empty(n, H, dtype=torch.float32, device=DEV)
            cu = torch.tensor(np.concatenate([[0], np.cumsum(step_lens)]), dtype=torch.int32, device=DEV)
            ops.mlstm_scan(r[:, :H * d], r[:, H * d:2 * H * d], r[:, 2 * H * d:H * (2 * d + dv)], g, bias, cap, 0.5, state, num, den, cu,
                           slots, n_seqs, H, one_token_each=max(step_lens) == 1)
            o = f64(num).reshape(n, H, dv) / f64(den)[:, :, None]
            for b in range(n_seqs):
                got[b].append(o[int(cu[b]):int(cu[b + 1])])
                at[b] += step_lens[b]
    finally:
        shape(0)
    for b in range(n_seqs):
        r, g = f64(rows[b]), f64(gates[b])
        for h in range(H):
            i = plain.soft_capped(g[:, h] + f64(bias)[h], cap)
            f = plain.log_sigmoid(plain.soft_capped(g[:, H + h] + f64(bias)[H + h], cap))
            want = plain.matrix_memory(r[:, h * d:(h + 1) * d] * 0.5, r[:, (H + h) * d:(H + h + 1) * d],
                                       r[:, 2 * H * d + h * dv:2 * H * d + (h + 1) * dv], i, f)
            close(np.concatenate(got[b])[:, h], want, "float32", (d, dv, b, h), loose=5.0)
    assert all(float(s[0].abs().max()) == 0.0 for s in state)
    m = state[2][1:]
    assert bool((m == m[:, :, :1]).all())                   # the copies of the maximum agree to the bit


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_matrix_memory_remembers_its_first_token_where_it_does_not_forget(dtype):
    """Head 0 forgets almost nothing, head 1 forgets within a few tokens.  The first token writes a value that stands
    out along a key that only the last query asks for again."""
    T, hidden, d, dv = 150, 64, 16, 16
    m = right(2, d, dv, 15.0)
    eye, z = torch.eye(16), lambda r, c: torch.zeros(r, c)
    pick = lambda at: torch.cat([z(16, at), eye, z(16, hidden - at - 16)], dim=1)
    weights = {"q": torch.cat([pick(0)] * 2), "k": torch.cat([pick(0)] * 2), "v": torch.cat([pick(16)] * 2), "g": z(2 * dv, hidden),
               "i": z(2, hidden), "i.b": torch.zeros(2), "f": z(2, hidden), "f.b": torch.tensor([12.0, -1.0]), "norm": torch.ones(2 * dv),
               "o": torch.cat([torch.eye(32), z(32, 32)], dim=0)}
    weights = {"l0.mix.right." + k: v.to(torch.bfloat16) for k, v in weights.items()}
    rng = np.random.default_rng(2)
    x = rng.standard_normal((T, hidden)) * 0.05
    x[:, 5] = 0.0                                            # no later key has anything of channel 5 ...
    x[0, 5] = 6.0                                            # ... but the first token's, ...
    x[-1, :16] = 0.0
    x[-1, 5] = 6.0                                           # ... and the last query asks for it
    x[0, 16:32] = np.linspace(2.0, 5.0, 16)                  # the value that stands out
    x[-1, 16:32] = np.linspace(0.05, -0.05, 16)              # what the last token itself writes is small
    xt = t32(x).to(TORCH[dtype])
    want = plain.memory_mixer(f64(xt), short(weights, "l0.mix.right."), m, 1e-5)
    shape = lambda v: v / np.sqrt((v * v).mean())
    first = shape(f64(xt)[0, 16:32])
    assert np.abs(shape(want[-1, :dv]) - first).max() < 0.1          # head 0: the first token's value, normed
    assert np.abs(shape(want[-1, dv:2 * dv]) - first).max() > 0.5     # head 1 has long forgotten it
    rt, parts, new_cache = mixer_of(dtype, hidden, parallel(left(1, 1, 8, 1.0), m), weights, side="right")
    for cuts in ([T], [T - 1, 1], [1] * T, [2] * (T // 2), [64, 64, 22]):
        got, = run_mixers(rt, parts, new_cache(), xt, cuts)
        close(got, want, dtype, cuts[:2], loose=3.0)


# ------------------------------------------------------------------ the selective scan
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,state,rank,taps", [(28, 6, 5, 3), (64, 16, 8, 4), (33, 1, 1, 2), (96, 17, 12, 1), (40, 32, 3, 4), (130, 64, 16, 5),
                                                   (24, 100, 8, 2), (12, 129, 8, 4), (9, 300, 7, 3), (200, 16, 24, 4), (16, 128, 16, 2)])
def test_the_selective_scan_carries_its_state_across_portions_and_slots(dtype, inner, state, rank, taps):
    """Random weights with decays all over (0, 1), every split of the states over lanes, one tap to five; state and
    the convolution's inputs go from step to step through the cache; slots used again; two sequences side by side."""
    rng = np.random.default_rng(17)
    hidden, T = 40, 150
    m = mamba(inner, state, rank, taps)["mixer"]
    weights = random_weights(rng, mamba_shapes("l0.mix.", m, hidden), std=0.3)
    weights["l0.mix.A_log"] = t32(rng.uniform(-3.0, 2.0, (inner, state))).to(torch.bfloat16)
    weights["l0.mix.dt.b"] = t32(rng.uniform(-4.0, 1.0, inner)).to(torch.bfloat16)
    weights["l0.mix.D"] = t32(1 + 0.5 * rng.standard_normal(inner)).to(torch.bfloat16)
    weights["l0.mix.x"] = (weights["l0.mix.x"].float() / max(1.0, (inner / 30) ** 0.5)).to(torch.bfloat16)
    x = t32(rng.standard_normal((T, hidden))).to(TORCH[dtype])
    want = plain.mamba1_mixer(f64(x), short(weights, "l0.mix."), m)
    rt, parts, new_cache = mixer_of(dtype, hidden, mamba(inner, state, rank, taps), weights)
    cache = new_cache()
    for cuts in CUTS(T):
        got, = run_mixers(rt, parts, cache, x, cuts)
        close(got, want, dtype, (inner, state, cuts[:2]), loose=2.0)
    y = t32(rng.standard_normal((50, hidden))).to(TORCH[dtype])
    want_y = plain.mamba1_mixer(f64(y), short(weights, "l0.mix."), m)
    a, b = cache.open_sequence(), cache.open_sequence()
    got_x, got_y = [], []
    for (na, nb) in ((37, 20), (1, 1), (1, 1), (111, 28)):
        ax, ay = cache.length(a), cache.length(b)
        cache.reserve_many([(a, ax + na), (b, ay + nb)]); cache.flush_tables()
        ctx = context(rt, [na, nb], [ax, ay], [a, b])
        out = f64(parts[0].forward(torch.cat([x[ax:ax + na], y[ay:ay + nb]]).contiguous(), ctx, cache.handles[0]))
        got_x.append(out[:na]); got_y.append(out[na:])
        cache.advance(a, na); cache.advance(b, nb)
    close(np.concatenate(got_x), want, dtype, "first of two", loose=2.0)
    close(np.concatenate(got_y), want_y, dtype, "second of two", loose=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("states", [1, 2, 4])
@pytest.mark.parametrize("C,N,n_seqs", [(40, 16, 3), (33, 5, 2), (64, 32, 2), (17, 30, 3), (300, 16, 1)])
def test_the_scan_kernel_for_every_number_of_states_a_lane(dtype, states, C, N, n_seqs):
    """The recurrence alone for every split of the states the launcher can pick: unequal sequences in one step, over several tiles
    of tokens, a second step that continues them, then a step of one token each."""
    rng = np.random.default_rng(C + N)
    lens = [[1 + (37 * b + 50 * k) % 90 for b in range(n_seqs)] for k in range(2)] + [[1] * n_seqs]
    total = [sum(l[b] for l in lens) for b in range(n_seqs)]
    draw = lambda w: [t32(rng.standard_normal((t, w))).to(TORCH[dtype]) for t in total]
    x, z, bc = draw(C), draw(C), draw(2 * N + 3)
    dt = [t32(rng.standard_normal((t, C))) for t in total]
    bias, skip, rates = t32(rng.standard_normal(C) - 1), t32(rng.standard_normal(C)), t32(-np.exp(rng.uniform(-3, 2, (C, N))))
    state = torch.zeros(n_seqs + 1, C, N, dtype=torch.float32, device=DEV)
    slots = torch.tensor([n_seqs - b for b in range(n_seqs)], dtype=torch.int32, device=DEV)       # not in order, slot 0 unused
    at, got = [0] * n_seqs, [[] for _ in range(n_seqs)]
    shape = build.library("selective").gtg_selective_scan_shape
    shape(states)
    try:
        for step_lens in lens:
            cat = lambda parts: torch.cat([p[at[b]:at[b] + step_lens[b]] for b, p in enumerate(parts)]).contiguous()
            out = torch.empty(sum(step_lens), C, dtype=TORCH[dtype], device=DEV)
            cu = torch.tensor(np.concatenate([[0], np.cumsum(step_lens)]), dtype=torch.int32, device=DEV)
            ops.selective_scan(cat(x), cat(bc)[:, : 2 * N], cat(dt), bias, rates, skip, cat(z), state, out, cu, slots, n_seqs,
                               one_token_each=max(step_lens) == 1)
            for b in range(n_seqs):
                got[b].append(f64(out)[int(cu[b]):int(cu[b + 1])])
                at[b] += step_lens[b]
    finally:
        shape(0)
    for b in range(n_seqs):
        bb = f64(bc[b])
        y = plain.selective_scan(f64(x[b]), plain.softplus(f64(dt[b]) + f64(bias)), bb[:, :N], bb[:, N:2 * N], f64(rates), f64(skip))
        close(np.concatenate(got[b]), y * plain.silu(f64(z[b])), dtype, (C, N, states, b))
    assert float(state[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_selective_scan_remembers_its_first_token_where_it_does_not_decay(dtype):
    """Half of the channels decay by e^-12 dt a token, half at once.  The first token's values come back 149 tokens later, by the one
    state number it was written to, from the first half only."""
    T, hidden, inner, N = 150, 64, 16, 4
    m = mamba(inner, N, 1, 2)["mixer"]
    z = lambda r, c: torch.zeros(r, c)
    row = lambda at: torch.nn.functional.one_hot(torch.tensor(at), inner).float()
    weights = {"in": torch.cat([torch.cat([torch.eye(16), z(16, 48)], dim=1), torch.cat([z(16, 63), torch.ones(16, 1)], dim=1)]),
               "conv": torch.tensor([[0.0, 1.0]] * inner), "conv.b": torch.zeros(inner),
               "x": torch.stack([torch.zeros(inner)] + [row(n) for n in range(N)] + [row(4 + n) for n in range(N)]),
               "dt": z(inner, 1), "dt.b": torch.zeros(inner),
               "A_log": torch.tensor([-12.0] * 12 + [1.0] * 4)[:, None].repeat(1, N), "D": torch.zeros(inner),
               "o": torch.cat([torch.eye(16), z(48, 16)])}
    weights = {"l0.mix." + k: v.to(torch.bfloat16) for k, v in weights.items()}
    x = np.random.default_rng(3).standard_normal((T, hidden)) * 0.02
    x[:, 63] = 1.0
    x[:, 2] = x[:, 6] = 0.0                                  # state number 2 is written by the first token (B_2) ...
    x[0, 2], x[-1, 6] = 5.0, 5.0                             # ... and read by the last (C_2) alone
    x[0, 8:16] = np.linspace(2.0, 4.0, 8)
    xt = t32(x).to(TORCH[dtype])
    want = plain.mamba1_mixer(f64(xt), short(weights, "l0.mix."), m)
    assert want[-1, 8:12].min() > 10.0 and np.abs(want[-1, 12:16]).max() < 0.1
    rt, parts, new_cache = mixer_of(dtype, hidden, mamba(inner, N, 1, 2), weights)
    for cuts in ([T], [T - 1, 1], [1] * T, [2] * (T // 2), [64, 64, 22]):
        got, = run_mixers(rt, parts, new_cache(), xt, cuts)
        close(got, want, dtype, cuts[:2], loose=2.0)


# ------------------------------------------------------------------ pairs, norms, positions, blocks
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("a,b,hidden", [(left(4, 2, 12, 0.5, 0.5, 16), right(3, 10, 6, 9.0), 40), (left(3, 1, 5, 0.6), right(2, 9, 7, 5.0), 51),
                                        (left(4, 1, 64, 0.2, 0.3, 40), right(2, 64, 128, 12.0), 128)])
def test_two_mixers_side_by_side_normed_and_averaged(dtype, a, b, hidden):
    rng = np.random.default_rng(19)
    T = 150
    weights = random_weights(rng, {**left_shapes("l0.mix.left.", a, hidden), **right_shapes("l0.mix.right.", b, hidden),
                                   "l0.mix.left.out": (hidden,), "l0.mix.right.out": (hidden,)})
    x = t32(rng.standard_normal((T, hidden))).to(TORCH[dtype])
    want = plain.parallel_mixer(f64(x), short(weights, "l0.mix."), {"left": a, "right": b}, 1e-5)
    rt, parts, new_cache = mixer_of(dtype, hidden, parallel(a, b), weights)
    for cuts in CUTS(T):
        got, = run_mixers(rt, parts, new_cache(), x, cuts)
        close(got, want, dtype, cuts[:2], loose=4.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_two_norms_around_zero_from_one_pass(dtype):
    rng = np.random.default_rng(3)
    rt = Runtime(DEV, TORCH[dtype])
    for n, h in [(1, 8), (5, 72), (70, 1000), (3, 51), (2, 4096), (3, 9000)]:
        x, u = rng.standard_normal((n, h)) * 3, rng.standard_normal((n, h))
        w = [t32(0.3 * rng.standard_normal(h)) for _ in range(2)]
        norms = [build_part("norm", PartSpec("rmsnorm", {"size": h, "eps": 1e-3, "weight": f"w{i}", "weight_offset": 1.0})) for i in range(2)]
        for i, norm in enumerate(norms):
            norm.load({f"w{i}": w[i]}, rt)
        for update in (None, t32(u).to(TORCH[dtype])):
            stream = ResidualStream(t32(x).clone(), update)
            total = f64(t32(x)) + (f64(update) if update is not None else 0.0)
            a, b = norms[0].forward_pair(stream, context(rt, [n], [0], [0]), norms[1])
            assert stream.pending is None
            close(stream.residual, total, "float32")
            for got, weight in ((a, w[0]), (b, w[1])):
                close(got, plain.rms_norm_around_zero(total, f64(weight), 1e-3), dtype, (n, h))
            assert np.abs(f64(a) - plain.rms_norm(total, f64(w[0]), 1e-3)).max() > 0.5      # not around zero would show


def test_sinusoids_join_the_scaled_embedding_also_at_far_positions():
    rng = np.random.default_rng(5)
    for width in (8, 51, 130):
        table = t32(rng.standard_normal((20, width)))
        tokens = torch.tensor([3, 19, 0, 7, 7, 1], dtype=torch.int32, device=DEV)
        positions = torch.tensor([0, 1, 2, 4095, 131072, 16000000], dtype=torch.int32, device=DEV)
        rt = Runtime(DEV, torch.float32)
        part = build_part("position", PartSpec("sinusoidal", {"size": width, "base": 10000.0}))
        part.load({}, rt)
        out = torch.empty(6, width, dtype=torch.float32, device=DEV)
        ops.embed(tokens, table, out, 2.5, positions, part.embedding_turns)
        want = 2.5 * f64(table)[tokens.cpu().numpy()] + plain.sinusoid(positions.cpu().numpy(), width)
        assert np.abs(f64(out) - want).max() < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 5, 40, 200])
@pytest.mark.parametrize("hidden,inner,ff", [(40, 28, 11), (128, 64, 256), (51, 13, 16)])
def test_mixer_and_feed_forward_of_one_hidden_state_end_in_one_product(dtype, n, hidden, inner, ff):
    """The block over a mixer and a feed-forward, whose last products are one: few rows and many, sizes that need zeros
    between the operands; without the feed-forward, the mixer's own product."""
    rng = np.random.default_rng(23)
    m = mamba(inner, 6, 5, 3)["mixer"]
    weights = random_weights(rng, {**mamba_shapes("l0.mix.", m, hidden), "l0.norm1": (hidden,), "l0.norm2": (hidden,),
                                   "l0.mlp.gate": (ff, hidden), "l0.mlp.up": (ff, hidden), "l0.mlp.down": (hidden, ff)})
    x = rng.standard_normal((n, hidden)) * 2
    w = {k: f64(v) for k, v in weights.items()}
    for with_ff in (True, False):
        raw = {"architecture": "Mererax", "vocab": 8, "width": hidden, "norm": {"eps": 1e-5}, "layers": [mamba(inner, 6, 5, 3, ff if with_ff else None)]}
        arch = find_architecture(raw)
        block = build_part("block", arch.plan(arch.read_config(raw)).layers[0].block)
        rt = Runtime(DEV, TORCH[dtype])
        for p in walk(block):
            p.load(weights, rt)
        cache = Cache([block.cache_requests()], [None], max_tokens=256, max_slots=1, dtype=TORCH[dtype], device=DEV)
        slot = cache.open_sequence()
        stream = ResidualStream(t32(x).clone())
        block.forward(stream, context(rt, [n], [0], [slot]), cache.handles[0])
        got = f64(stream.residual) + (f64(stream.pending) if stream.pending is not None else 0.0)
        x64 = f64(t32(x))
        want = x64 + plain.mamba1_mixer(plain.rms_norm_around_zero(x64, w["l0.norm1"], 1e-5), short(weights, "l0.mix."), m)
        if with_ff:
            want = want + plain.gated_feed_forward(plain.rms_norm_around_zero(x64, w["l0.norm2"], 1e-5), w["l0.mlp.gate"], w["l0.mlp.up"], w["l0.mlp.down"])
        assert (block.w_joint is not None) == with_ff and (block.mixer.w_o is None) == with_ff
        close(got, want, dtype, (n, hidden, with_ff), loose=2.0)


# ------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_whole_prompts_of_many_lengths_and_the_hidden_state_after_every_layer(folders, name, dtype):
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 6)
    for p in prompts_of(name, [1, 2, 3, 17, 63, 64, 65, 129, 230]):
        got = run_cut(model, cache, p, [len(p)])
        assert_close(got, want_logits(folders, name, p), dtype, f"{name} {dtype} whole prompt of {len(p)}")
    assert cache.open_slots() == []
    p = prompts_of(name, [90], seed=3)[0]
    hidden, layers = [], []
    model.op_hook = lambda s, l, op, t: hidden.append(f64(t)) if op == "hidden_post_ffn" else None
    try:
        run_cut(model, cache, p, [len(p)])
    finally:
        model.op_hook = None
    plain.forward(CONFIGS[name][0], weights_of(folders, name), p, layers_out=layers)
    assert len(hidden) == len(layers)
    for i, (g, w) in enumerate(zip(hidden, layers)):
        close(g, w, dtype, f"{name} {dtype} hidden state after layer {i}", loose=4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_portions_down_to_two_tokens_and_token_by_token_from_the_start(folders, name, dtype):
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 6)
    p = prompts_of(name, [150], seed=5)[0]
    want = want_logits(folders, name, p)
    rows = {}
    for portions in ([150], [1], [2], [3, 2, 1, 16, 15, 17, 64], [63, 1, 1, 64, 2], [100, 1]):
        rows[tuple(portions)] = run_cut(model, cache, p, portions)
        assert_close(rows[tuple(portions)], want, dtype, f"{name} {dtype} portions {portions}")
    if dtype == "float32":
        # sums walk keys, taps and states in one order whatever the cut
        for portions, got in rows.items():
            np.testing.assert_allclose(got, rows[(150,)], rtol=0, atol=2e-5 * np.abs(want).max(), err_msg=str(portions))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_long_decoding_across_page_borders(folders, name, dtype):
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 6)
    p = prompts_of(name, [5 + 280], seed=6)[0]
    got = run_cut(model, cache, p, [5, 1])
    assert_close(got, want_logits(folders, name, p), dtype, f"{name} {dtype} 280 tokens decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "U"])
def test_unequal_batches_against_each_alone_with_slots_and_pages_used_again(folders, name, dtype):
    """Three batches through a cache too small for two of them: the slots and pages
    of finished requests, with their old rows and states, go to new ones.  In a batch every
    request is decoded to its own length and leaves when it ends."""
    model = get_model(folders, name, dtype)
    cache = model.new_cache(max_tokens=64 * 7, max_slots=4)
    batches = [[(5, 9), (70, 3), (17, 20), (1, 12)], [(64, 1), (130, 6), (3, 33)], [(40, 8), (128, 2), (9, 9), (2, 2)]]
    for bi, batch in enumerate(batches):
        prompts = prompts_of(name, [a + b for a, b in batch], seed=20 + bi)
        slots = [cache.open_sequence() for _ in batch]
        got = [[] for _ in batch]
        entries = [StepEntry(slots[i], p[:plen], list(range(plen))) for i, ((plen, _), p) in enumerate(zip(batch, prompts))]
        flat = step(model, cache, entries).float().cpu().numpy()
        o = 0
        for i, e in enumerate(entries):
            got[i].append(flat[o:o + len(e.want)])
            o += len(e.want)
        t = 0
        while True:
            live = [i for i in range(len(batch)) if t < batch[i][1]]
            if not live:
                break
            flat = step(model, cache, [StepEntry(slots[i], [prompts[i][batch[i][0] + t]], [0]) for i in live]).float().cpu().numpy()
            for j, i in enumerate(live):
                got[i].append(flat[j:j + 1])
                if t + 1 >= batch[i][1]:
                    cache.close_sequence(slots[i])
            t += 1
        for i in range(len(batch)):
            assert_close(np.concatenate(got[i]), want_logits(folders, name, prompts[i]), dtype, f"{name} {dtype} batch {bi} request {i}")
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
        ok = []
        for p, r in zip(prompts, results):
            logits = plain.forward(cfg, w, list(p) + r.tokens)     # each token is one the plain model could have chosen there
            for t, tok in enumerate(r.tokens):
                row = logits[len(p) - 1 + t]
                slack = (1e-4 if dtype == "float32" else 5e-2) * max(1.0, np.abs(row).max())
                ok.append(row[tok] >= row.max() - slack)
        assert all(ok), (use_graph, ok)
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
