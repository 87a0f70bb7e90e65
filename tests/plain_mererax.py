"""Plain, slow Mererax decoder: the oracle of the numerics tests of that design.

Mererax is a decoder-only model whose config.json lists its layers one by one.
The embedded tokens are scaled and a sinusoid of the position is added; in every
layer the mixer and the feed-forward read two norms of the same hidden state and
both are added to it; a final norm and the embedding table itself close it.  The
norms keep their weight around zero.  The mixers:

* ``parallel``: two mixers side by side over the same input, averaged after an
  RMS norm of each output.  Left, grouped-query attention whose values are the
  keys as projected, with an RMS norm over the whole rows of q and k, queries
  that grow with the position, and a penalty on the distance per head.  Right, a
  matrix memory with exponential input gates and a running maximum (the mLSTM).
* ``mamba1``: the selective scan with a decay per channel and state number.

Whole sequences, no cache, one function per mechanism, NumPy in float64.  It
shares no code with the package.

Notation: W is stored [out, in]; rows of x are tokens, so a projection is x W^T.
"""
from __future__ import annotations

import math

import numpy as np

F64 = np.float64


def A(x):
    return np.asarray(x, F64)


# --------------------------------------------------------------------------
# norms and activations
# --------------------------------------------------------------------------
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = A(x)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * A(w)


def rms_norm_around_zero(x, w, eps):
    return unit_rms(x, eps) * (1.0 + A(w))


def sigmoid(z):
    z = A(z)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return A(z) * sigmoid(z)


def softplus(z):
    z = A(z)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def log_sigmoid(z):
    return -softplus(-A(z))


# --------------------------------------------------------------------------
# positions
# --------------------------------------------------------------------------
def sinusoid(positions, width):
    """[T, width]: entry 2i is sin(p f_i), entry 2i+1 cos(p f_i), f_i = 10000^(-2i/width)."""
    p = A(positions)[:, None]
    c = np.arange(width)
    angle = p * 10000.0 ** (-2.0 * (c // 2) / width)[None, :]
    return np.where(c % 2 == 0, np.sin(angle), np.cos(angle))


def query_temperature(positions, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * np.log(np.floor((A(positions) + 1.0) / every) + 1.0)


def distance_slopes(heads):
    """2^(-8 (h+1) / H)."""
    return 2.0 ** (-8.0 * (np.arange(heads) + 1.0) / heads)


# --------------------------------------------------------------------------
# attention
# --------------------------------------------------------------------------
def attend(q, k, v, scale, slopes):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv], causal; the score of
    query i and key j is q . k * scale - slopes[h] (i - j)."""
    T, H, _ = q.shape
    G = k.shape[1]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    out = np.zeros((T, H, v.shape[2]), F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale - slopes[h] * (i - j)
        s = np.where(j <= i, s, -np.inf)
        p = np.exp(s - s.max(axis=-1, keepdims=True))
        out[:, h] = (p / p.sum(axis=-1, keepdims=True)) @ v[:, g]
    return out


def attention_mixer(h, w, m, eps):
    """The left mixer.  `w`: tensors by short name; `m`: its block of config.json."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ A(w["q"]).T, h @ A(w["k"]).T
    v = k.reshape(T, G, d)
    q, k = rms_norm(q, w["q.norm"], eps), rms_norm(k, w["k.norm"], eps)
    t = m.get("q_temp")
    if t:
        q = q * query_temperature(np.arange(T), t["coef"], t["every"])[:, None]
    a = attend(q.reshape(T, H, d), k.reshape(T, G, d), v, m["scale"], distance_slopes(H))
    return a.reshape(T, H * d) @ A(w["o"]).T


# --------------------------------------------------------------------------
# the matrix memory
# --------------------------------------------------------------------------
def matrix_memory(q, k, v, i, f):
    """One head.  q, k [T, d]; v [T, dv]; i, f [T] the logarithms of the input and
    forget gates.  S [d, dv], n [d] and the maximum m start at zero."""
    T, d = q.shape
    S, n, m = np.zeros((d, v.shape[1]), F64), np.zeros(d, F64), 0.0
    out = np.zeros((T, v.shape[1]), F64)
    for t in range(T):
        new = max(f[t] + m, i[t])
        keep, add = math.exp(f[t] + m - new), math.exp(i[t] - new)
        S = keep * S + add * np.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def soft_capped(z, cap):
    return cap * np.tanh(A(z) / cap)


def memory_mixer(h, w, m, eps):
    """The right mixer."""
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ A(w["q"]).T).reshape(T, H, d) * d ** -0.5
    k = (h @ A(w["k"]).T).reshape(T, H, d)
    v = (h @ A(w["v"]).T).reshape(T, H, dv)
    i = soft_capped(h @ A(w["i"]).T + A(w["i.b"]), cap)
    f = log_sigmoid(soft_capped(h @ A(w["f"]).T + A(w["f.b"]), cap))
    o = np.stack([matrix_memory(q[:, x], k[:, x], v[:, x], i[:, x], f[:, x]) for x in range(H)], axis=1)
    o = unit_rms(o, eps).reshape(T, H * dv) * A(w["norm"]) * sigmoid(h @ A(w["g"]).T)
    return o @ A(w["o"]).T


def parallel_mixer(h, w, m, eps):
    side = lambda name: {k[len(name) + 1:]: t for k, t in w.items() if k.startswith(name + ".")}
    left, right = side("left"), side("right")
    a = attention_mixer(h, left, m["left"], eps)
    b = memory_mixer(h, right, m["right"], eps)
    return 0.5 * (rms_norm(a, left["out"], eps) + rms_norm(b, right["out"], eps))


# --------------------------------------------------------------------------
# the selective scan
# --------------------------------------------------------------------------
def causal_conv(u, w, b):
    """u [T, C], w [C, taps]: y_t = b + sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    u, w = A(u), A(w)
    T, taps = u.shape[0], w.shape[1]
    y = np.tile(A(b)[None, :], (T, 1))
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += u[: T - back] * w[:, j][None, :]
    return y


def selective_scan(x, dt, B, C, rates, skip):
    """x, dt [T, c]; B, C [T, n]; rates [c, n] (negative); skip [c].
    S <- exp(dt rates) S + dt x B; y = S C + skip x."""
    T, c = x.shape
    S = np.zeros((c, B.shape[1]), F64)
    y = np.zeros((T, c), F64)
    for t in range(T):
        S = np.exp(dt[t][:, None] * rates) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + skip * x[t]
    return y


def mamba1_mixer(h, w, m):
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    xz = h @ A(w["in"]).T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w["conv"], w["conv.b"]))
    low = x @ A(w["x"]).T
    dt = softplus(low[:, :rank] @ A(w["dt"]).T + A(w["dt.b"]))
    y = selective_scan(x, dt, low[:, rank:rank + n], low[:, rank + n:], -np.exp(A(w["A_log"])), A(w["D"]))
    return (y * silu(z)) @ A(w["o"]).T


# --------------------------------------------------------------------------
# feed-forward, the whole model
# --------------------------------------------------------------------------
def gated_feed_forward(h, gate, up, down):
    return (silu(h @ A(gate).T) * (h @ A(up).T)) @ A(down).T


def source_of(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  `W`: every tensor by its full name;
    `layers_out`, a list, receives the hidden state after every layer."""
    eps = float(cfg["norm"]["eps"])
    T = len(tokens)
    x = A(W["embed"])[np.asarray(tokens)] * float(cfg["embedding"]["scale"]) + sinusoid(np.arange(T), cfg["width"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{source_of(cfg, i)}."
        w = {name[len(p) + 4:]: A(t) for name, t in W.items() if name.startswith(p + "mix.")}
        h = rms_norm_around_zero(x, W[p + "norm1"], eps)
        if layer["type"] == "parallel":
            update = parallel_mixer(h, w, layer["mixer"], eps)
        elif layer["type"] == "mamba1":
            update = mamba1_mixer(h, w, layer["mixer"])
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            h = rms_norm_around_zero(x, W[p + "norm2"], eps)
            update = update + gated_feed_forward(h, W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"])
        x = x + update
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm_around_zero(x, W["final.norm"], eps) @ A(W["embed"]).T


def greedy(cfg, W, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(forward(cfg, W, tokens)[-1])))
    return tokens[len(prompt):]
