"""Fotovik restated in float64 NumPy, token by token, one function per mechanism.  Shares no code with `zgml_b200/`: the GPU
tests compare the framework's sessions against this file.

Notation: x is the stream [T, D]; W are [out, in] matrices applied as `x @ W.T`; `p` maps tensor names to arrays; positions
count from 0.  A layer norms each sublayer on the way in and on the way out, every norm with ONE learned number:
x += n1b * rms(mixer(n1 * rms(x)));  x += n2b * rms(ff(n2 * rms(x))).
"""
import math

import numpy as np


def rms_norm(x, w, eps):
    """x over its root mean square (last axis), times w: a vector, a single number, or None."""
    x = np.asarray(x, np.float64)
    r = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return r if w is None else r * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + np.vectorize(math.erf)(z / math.sqrt(2.0)))


def unit(x, eps=1e-6):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + eps)


def bigram_rows(tokens, bigram):
    """Row of the bigram table for every token: a hash of the token and its predecessor; the first token has a row of its own."""
    rows, prev = [], None
    for t in tokens:
        rows.append(bigram["buckets"] if prev is None else (prev * bigram["mul_prev"] + t * bigram["mul_cur"]) % bigram["buckets"])
        prev = t
    return rows


def embedding(cfg, p, tokens):
    e = cfg["embedding"]
    x = np.asarray(p["embed"], np.float64)[np.asarray(tokens)] * e.get("scale", 1.0)
    if e.get("bigram"):
        x = x + np.asarray(p["bigram"], np.float64)[np.asarray(bigram_rows(tokens, e["bigram"]))]
    return x


def rotary_frequencies(rot):
    f = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])
    return f / rot["scaling"]["factor"] if rot.get("scaling") else f


def rotate(v, pos, freqs, interleaved):
    """v [..., dim]; the first 2 n entries turn: (2i, 2i + 1) are a pair when interleaved, (i, i + n) otherwise."""
    n = len(freqs)
    c, s = np.cos(pos * freqs), np.sin(pos * freqs)
    out = np.array(v, np.float64)
    a, b = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if interleaved else (slice(0, n), slice(n, 2 * n))
    out[..., a] = v[..., a] * c - v[..., b] * s
    out[..., b] = v[..., b] * c + v[..., a] * s
    return out


def visible(i, window=None, pool=None):
    """(first visible token, number of visible pooled blocks) for a query at position i."""
    if window is None:
        return 0, 0
    return max(0, i - window + 1), max(0, (i - window + 1) // pool) if pool else 0


def softmax_attention(q, k, v, scale, window=None, pool=None, sink=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] of one sequence from position 0.  Query i weighs the keys j with 0 <= i - j < window
    and, with `pool`, the mean key of every block of `pool` tokens whose last token is at most i - window (value: the mean
    value).  `sink` [H] adds exp(sink_h) to the denominator only."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo, nb = visible(i, window, pool)
        K, V = list(k[lo:i + 1]), list(v[lo:i + 1])
        for b in range(nb):
            K.append(k[b * pool:(b + 1) * pool].mean(0))
            V.append(v[b * pool:(b + 1) * pool].mean(0))
        K, V = np.stack(K), np.stack(V)
        for h in range(H):
            g = h // (H // G)
            s = (K[:, g] @ q[i, h]) * scale
            m = s.max() if sink is None else max(s.max(), sink[h])
            e = np.exp(s - m)
            den = e.sum() + (0.0 if sink is None else math.exp(sink[h] - m))
            out[i, h] = (e / den) @ V[:, g]
    return out


def attention(h, p, pre, m, eps, interleaved, qk_norm, sink):
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ p[pre + "q"].T).reshape(T, H, dim)
    k = (h @ p[pre + "k"].T).reshape(T, G, dim)
    v = (h @ p[pre + "v"].T).reshape(T, G, vdim)
    if qk_norm:
        q, k = rms_norm(q, p[pre + "q.norm"], eps), rms_norm(k, p[pre + "k.norm"], eps)
    f = rotary_frequencies(m["rot"])
    for t in range(T):
        q[t], k[t] = rotate(q[t], t, f, interleaved), rotate(k[t], t, f, interleaved)
    mask = m.get("mask") or {}
    o = softmax_attention(q, k, v, m["scale"], mask.get("size"), mask.get("pool"), p[pre + "sink"] if sink else None)
    return o.reshape(T, H * vdim) @ p[pre + "o"].T


def pooled_window_attention(h, p, pre, m, eps):
    return attention(h, p, pre, m, eps, interleaved=True, qk_norm=False, sink=True)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: the last tap multiplies the current token, earlier ones reach back; zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    out = np.zeros((T, C))
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * u[s]
    return out


def delta_rule(q, k, v, beta, g):
    """q, k [T, H, dim], v [T, H, vdim], beta, g [T, H]: decay, correct towards v, then read."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]))
    out = np.zeros(v.shape)
    for t in range(T):
        for h in range(H):
            S[h] *= g[t, h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] += np.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out


def delta_mixer(h, p, pre, m, eps):
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(causal_conv(h @ p[pre + "q"].T, p[pre + "q.conv"])).reshape(T, G, dim)
    k = silu(causal_conv(h @ p[pre + "k"].T, p[pre + "k.conv"])).reshape(T, G, dim)
    v = silu(causal_conv(h @ p[pre + "v"].T, p[pre + "v.conv"])).reshape(T, H, vdim)
    q, k = unit(q) * dim ** -0.5, unit(k)
    q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
    beta = sigmoid(h @ p[pre + "b"].T)
    g = np.exp(-np.exp(p[pre + "A_log"]) * softplus(h @ p[pre + "a"].T + p[pre + "dt_bias"]))
    o = rms_norm(delta_rule(q, k, v, beta, g), p[pre + "norm"], eps).reshape(T, H * vdim)
    return (o * silu(h @ p[pre + "g"].T)) @ p[pre + "o"].T


def lightning_rule(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]))
    out = np.zeros(v.shape)
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out


def lightning_mixer(h, p, pre, m, eps):
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(h @ p[pre + "q"].T).reshape(T, H, dim)
    k = silu(h @ p[pre + "k"].T).reshape(T, H, dim)
    v = silu(h @ p[pre + "v"].T).reshape(T, H, vdim)
    o = lightning_rule(q, k, v, m["decay"]).reshape(T, H * vdim)
    return (rms_norm(o, p[pre + "norm"], eps) * sigmoid(h @ p[pre + "g"].T)) @ p[pre + "o"].T


def parallel_mixer(h, p, pre, m, eps):
    a = attention(h, p, pre + "left.", m["left"], eps, interleaved=False, qk_norm=True, sink=False)
    b = lightning_mixer(h, p, pre + "right.", m["right"], eps)
    return 0.5 * (rms_norm(a, p[pre + "left.out"], eps) + rms_norm(b, p[pre + "right.out"], eps))


def dense_ff(h, p, pre):
    return gelu_erf(h @ p[pre + "up"].T) @ p[pre + "down"].T


MIXERS = {"attention": pooled_window_attention, "delta": delta_mixer, "parallel": parallel_mixer}


def layer_order(cfg):
    """(layer, whether the embedding output joins the stream before it) for every layer run, in order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    body = [(i, r > 0 and i == a) for r in range(times) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]


def forward(cfg, p, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from position 0 (and the stream after every layer run)."""
    eps = cfg["norm"]["eps"]
    e = embedding(cfg, p, tokens)
    x, streams = e, []
    for i, again in layer_order(cfg):
        L, pre = cfg["layers"][i], f"l{i}."
        if again:
            x = x + e
        y = MIXERS[L["type"]](rms_norm(x, p[pre + "norm1"], eps), p, pre + "mix.", L["mixer"], eps)
        x = x + rms_norm(y, p[pre + "norm1b"], eps)
        if L.get("mlp") is not None:
            y = dense_ff(rms_norm(x, p[pre + "norm2"], eps), p, pre + "mlp.")
            x = x + rms_norm(y, p[pre + "norm2b"], eps)
        streams.append(x.copy())
    z = rms_norm(x, p["final.norm"], eps) @ np.asarray(p["head"], np.float64).T
    return (z, np.stack(streams)) if return_layers else z
