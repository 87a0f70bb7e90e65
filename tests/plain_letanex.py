"""Plain, slow Letanex decoder: the oracle of the numerics tests of that design.

Letanex is a decoder-only model whose config.json lists its layers one by one.
Every sublayer stands between two layer norms, x + norm_b(f(norm_a(x))), with
weights and without biases.  The mixers:

* ``attention``: differential attention.  Every query and key head has two
  parts; each pair of parts is a causal softmax attention of its own over one
  set of values, and a head's output is the first minus lambda times the
  second, divided by its root mean square and times 1 - diff.  Half-split
  rotation of the first channels of each part, frequencies divided by a
  factor.  A layer may read another layer's keys and values.
* ``lightning``: linear attention with a fixed decay per head, S <- a S + k v^T;
  o = S^T q, over silu-activated q, k and v; the concatenated heads are normed
  together and gated.

The feed-forwards: ``dense``, down(relu(up x)^2), and ``moe``, experts with
clamped gates among which some outputs of the router stand for the input
itself, beside an expert that every token passes.

Whole sequences, no cache, one function per mechanism, NumPy in float64.  It
shares no code with the package.

Notation: W is stored [out, in]; rows of x are tokens, so a projection is x W^T.
"""
from __future__ import annotations

import numpy as np

F64 = np.float64


def A(x):
    return np.asarray(x, F64)


def layer_norm(x, w, eps):
    x = A(x)
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * A(w)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = A(x)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-A(z)))


def silu(z):
    return A(z) * sigmoid(z)


# --------------------------------------------------------------------------
# rotation
# --------------------------------------------------------------------------
def frequencies(dims, base, factor=1.0):
    """base^(-2i/dims) / factor, i < dims/2."""
    return np.array([float(base) ** (-2.0 * i / dims) / float(factor) for i in range(dims // 2)], F64)


def rotate(x, positions, freqs):
    """x [T, ..., d]: channel i turns with i + n by the angle position * freqs[i],
    n = len(freqs); the channels from 2n on pass."""
    x = np.array(x, F64)
    n = len(freqs)
    a = (A(positions)[:, None] * freqs[None, :]).reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (n,))
    u, v = x[..., :n].copy(), x[..., n:2 * n].copy()
    x[..., :n] = u * np.cos(a) - v * np.sin(a)
    x[..., n:2 * n] = v * np.cos(a) + u * np.sin(a)
    return x


# --------------------------------------------------------------------------
# differential attention
# --------------------------------------------------------------------------
def softmax_attend(q, k, v, scale):
    """One map of one head: q, k [T, d], v [T, dv]; query i sees keys j <= i."""
    T = q.shape[0]
    s = (A(q) @ A(k).T) * scale
    s = np.where(np.arange(T)[None, :] <= np.arange(T)[:, None], s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return (p / p.sum(axis=-1, keepdims=True)) @ A(v)


def mixing_lambda(lq1, lk1, lq2, lk2, diff):
    return float(np.exp((A(lq1) * A(lk1)).sum()) - np.exp((A(lq2) * A(lk2)).sum()) + diff)


def differential_attend(q, k, v, scale, lam, diff, eps):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] -> [T, H, dv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), F64)
    for h in range(H):
        g = h // (H // G)
        first = softmax_attend(q[:, h, 0], k[:, g, 0], v[:, g], scale)
        second = softmax_attend(q[:, h, 1], k[:, g, 1], v[:, g], scale)
        out[:, h] = unit_rms(first - lam * second, eps) * (1.0 - diff)
    return out


def turning(m):
    """The frequencies of a mixer's rotation, or None."""
    rot = m.get("rot")
    if not rot:
        return None
    return frequencies(rot["dims"], rot["base"], (rot.get("scaling") or {}).get("factor", 1.0))


def keys_values(h, w, m):
    """What an attention layer with projections of its own caches: keys after the
    rotation [T, G, 2, d], values [T, G, dv]."""
    T = h.shape[0]
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    k = (h @ A(w["k"]).T).reshape(T, G, 2, d)
    f = turning(m)
    if f is not None:
        k = rotate(k, np.arange(T), f)
    return k, (h @ A(w["v"]).T).reshape(T, G, dv)


def attention_mixer(h, w, m, eps, kv=None):
    """The ``attention`` mixer.  `w`: the layer's tensors by short name; `m`: the
    mixer's block of config.json; `kv`: (keys, values) of the layer named by
    ``kv_from``, or None.  Returns (update, (keys, values))."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    if kv is None:
        kv = keys_values(h, w, m)
    q = (h @ A(w["q"]).T).reshape(T, H, 2, d)
    f = turning(m)
    if f is not None:
        q = rotate(q, np.arange(T), f)
    lam = mixing_lambda(w["lq1"], w["lk1"], w["lq2"], w["lk2"], m["diff"])
    o = differential_attend(q, kv[0], kv[1], m["scale"], lam, m["diff"], eps)
    return o.reshape(T, H * dv) @ A(w["o"]).T, kv


# --------------------------------------------------------------------------
# linear attention with a fixed decay per head
# --------------------------------------------------------------------------
def decayed_memory(q, k, v, decay):
    """One head: q, k [T, d], v [T, dv]; S [d, dv] starts at zero; per token
    S <- decay S + k v^T; o = S^T q."""
    T, d = q.shape
    S = np.zeros((d, v.shape[1]), F64)
    out = np.zeros((T, v.shape[1]), F64)
    for t in range(T):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def lightning_mixer(h, w, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ A(w["q"]).T).reshape(T, H, d)
    k = silu(h @ A(w["k"]).T).reshape(T, H, d)
    v = silu(h @ A(w["v"]).T).reshape(T, H, dv)
    o = np.stack([decayed_memory(q[:, i], k[:, i], v[:, i], float(m["decay"][i])) for i in range(H)], axis=1)
    o = unit_rms(o.reshape(T, H * dv), eps) * A(w["norm"])
    return (o * sigmoid(h @ A(w["g"]).T)) @ A(w["o"]).T


# --------------------------------------------------------------------------
# feed-forwards
# --------------------------------------------------------------------------
def squared_relu(h, up, down):
    return np.maximum(h @ A(up).T, 0.0) ** 2 @ A(down).T


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ A(gate).T, limit)
    u = np.clip(h @ A(up).T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ A(down).T


def scores(h, router):
    z = h @ A(router).T
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    return s / s.sum(axis=-1, keepdims=True)


def route(h, router, correction, top, scale, chosen=None):
    """(chosen [T, top], weights [T, top]): softmax scores over all outputs; the
    largest scores plus correction choose; the weights are the chosen scores
    without it, over their sum, times scale.  `chosen`: take these choices instead (of a
    run whose rounding may have turned a close call)."""
    s = scores(h, router)
    if chosen is None:
        chosen = np.argsort(-(s + A(correction)), axis=-1, kind="stable")[:, :top]
    w = np.take_along_axis(s, chosen, axis=-1)
    return chosen, w / (w.sum(axis=-1, keepdims=True) + 1e-20) * scale


def mixture(h, W, p, mlp, chosen=None):
    """`W`: every tensor by its full name; `p`: the feed-forward's prefix."""
    r = mlp["router"]
    chosen, weights = route(h, W[p + "router"], W[p + "correction"], r["top"], r["scale"], chosen)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weights[t]):
            if e >= r["experts"]:
                out[t] += w * h[t]
            else:
                x = f"{p}e{e}."
                out[t] += w * clamped_expert(h[t], W[x + "gate"], W[x + "up"], W[x + "down"], mlp["expert"]["limit"])
    if mlp.get("shared"):
        x = p + "shared."
        out = out + clamped_expert(h, W[x + "gate"], W[x + "up"], W[x + "down"], mlp["shared"]["limit"])
    return out


# --------------------------------------------------------------------------
# the whole model
# --------------------------------------------------------------------------
def forward(cfg, W, tokens, layers_out=None, choices=None, slack=None):
    """Logits [T, vocab] of one sequence.  `W`: every tensor by its full name;
    `layers_out`, a list, receives the hidden state after every layer.  `choices`: the experts
    to use per mixture, in order ([T, top] each), in place of those the scores choose; `slack`,
    a list, then receives by how much each such choice was worse than the best."""
    eps = float(cfg["norm"]["eps"])
    x = A(W["embed"])[np.asarray(tokens)]
    cached, choices = {}, iter(choices) if choices is not None else None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        w = {name[len(p) + 4:]: A(t) for name, t in W.items() if name.startswith(p + "mix.")}
        h = layer_norm(x, W[p + "norm1"], eps)
        if layer["type"] == "attention":
            src = m.get("kv_from")
            update, cached[i] = attention_mixer(h, w, m, eps, cached[src] if src is not None else None)
        elif layer["type"] == "lightning":
            update = lightning_mixer(h, w, m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm(update, W[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = layer_norm(x, W[p + "norm2"], eps)
            if mlp["kind"] == "dense":
                update = squared_relu(h, W[p + "mlp.up"], W[p + "mlp.down"])
            else:
                chosen = next(choices) if choices is not None else None
                if slack is not None:
                    s = scores(h, W[p + "mlp.router"]) + A(W[p + "mlp.correction"])
                    best = -np.sort(-s, axis=-1)[:, :chosen.shape[1]].sum(axis=-1)
                    slack.append(best - np.take_along_axis(s, chosen, axis=-1).sum(axis=-1))
                update = mixture(h, W, p + "mlp.", mlp, chosen)
            x = x + layer_norm(update, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return layer_norm(x, W["final.norm"], eps) @ A(W["head"]).T


def greedy(cfg, W, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(forward(cfg, W, tokens)[-1])))
    return tokens[len(prompt):]
