"""Fomanex restated in float64 NumPy, one function per mechanism.  Shares no code with `zgml_b200/`: the GPU tests compare the
framework's sessions against this file.

Notation: W are [out, in] matrices applied as `x @ W.T`; `p` maps tensor names to arrays; positions count from 0.  Instead of one
stream there are s of them, X [s, T, D], all equal to the normed embedding at the start; a sublayer f reads u = sum_a in_a X_a and
    X_b <- sum_a mix[a, b] X_a + m out_b ls * f(dyt(u)),
and the model's head reads the sum of the streams.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dynamic_tanh(x, p, name):
    return np.tanh(float(np.asarray(p[name + ".alpha"]).reshape(())) * x) * p[name] + p[name + ".b"]


def embedding(cfg, p, tokens):
    x = np.asarray(p["embed"], np.float64)[np.asarray(tokens)] * cfg["embedding"]["scale"]
    return dynamic_tanh(x, p, "embed.norm")


# ── streams ──
def read_streams(X, w_in):
    return np.tensordot(np.asarray(w_in), X, (0, 0))


def write_streams(X, mix, w_out, y):
    """mix[a, b]: how much of old stream a goes into new stream b."""
    return np.einsum("ab,atd->btd", np.asarray(mix), X) + np.asarray(w_out)[:, None, None] * y[None]


# ── latent attention ──
def rotary_frequencies(rot):
    """(frequencies of the dims / 2 pairs, factor on cosine and sine)."""
    n = rot["dims"]
    f = np.array([rot["base"] ** (-2.0 * i / n) for i in range(n // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):           # the pair index that turns `turns` times over the original context
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))

    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(v, pos, freqs, mag):
    """v [..., 2 n]: entries i and i + n are a pair."""
    n = len(freqs)
    c, s = mag * np.cos(pos * freqs), mag * np.sin(pos * freqs)
    return np.concatenate([v[..., :n] * c - v[..., n:] * s, v[..., n:] * c + v[..., :n] * s], -1)


def visible(i):
    """Keys [0, visible(i)) of the query at position i."""
    return i + 1


def softmax_attention(q, k, v, scale, sink):
    """q, k [T, H, dk], v [T, H, dv]; exp(sink_h) joins the denominator only."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        S = q[:, h] @ k[:, h].T * scale
        for i in range(T):
            s = S[i, :visible(i)]
            m = max(s.max(), sink[h])
            e = np.exp(s - m)
            out[i, h] = (e / (e.sum() + math.exp(sink[h] - m))) @ v[:visible(i), h]
    return out


def latent_attention(h, p, pre, m, eps):
    H, dim, rd, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = (h @ p[pre + "q"].T).reshape(T, H, dim + rd)
    z = h @ p[pre + "dkv"].T
    c = rms_unit(z[:, :rank], eps) * p[pre + "dkv.norm"]
    f, mag = rotary_frequencies(m["rot"])
    qr = np.stack([rotate(q[t, :, dim:], t, f, mag) for t in range(T)])
    kr = np.stack([rotate(z[t, rank:], t, f, mag) for t in range(T)])
    k = np.concatenate([(c @ p[pre + "uk"].T).reshape(T, H, dim), np.repeat(kr[:, None], H, 1)], -1)
    v = (c @ p[pre + "uv"].T).reshape(T, H, vdim)
    o = softmax_attention(np.concatenate([q[:, :, :dim], qr], -1), k, v, m["scale"], np.asarray(p[pre + "sink"], np.float64))
    return o.reshape(T, H * vdim) @ p[pre + "o"].T


# ── wkv ──
def shifted(h):
    """The input of the token before; zeros before the first."""
    return np.concatenate([np.zeros((1, h.shape[1])), h[:-1]])


def token_mix(h, mu):
    return h + (shifted(h) - h) * mu


def wkv_decay(z, p, pre):
    return np.exp(-np.exp(np.tanh(z @ p[pre + "w1"].T) @ p[pre + "w2"].T + p[pre + "w0"]))


def wkv_rule(r, k, v, w, u):
    """r, k, w [T, H, N], v [T, H, P], u [H, N]: the read-out sees the state before the token's own write, and the token itself through the
    bonus u; then the state decays per key channel and takes the token in."""
    T, H, N = k.shape
    S = np.zeros((H, N, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            kv = np.outer(k[t, h], v[t, h])
            out[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = w[t, h][:, None] * S[h] + kv
    return out


def wkv(h, p, pre, m, eps):
    H, N = m["heads"], m["dim"]
    T = h.shape[0]
    mixed = {s: token_mix(h, p[pre + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mixed[s] @ p[pre + s].T).reshape(T, H, N) for s in "rkv")
    w = wkv_decay(mixed["w"], p, pre).reshape(T, H, N)
    o = rms_unit(wkv_rule(r, k, v, w, np.asarray(p[pre + "u"], np.float64)), eps).reshape(T, H * N)
    return (o * p[pre + "norm"] * silu(mixed["g"] @ p[pre + "g"].T)) @ p[pre + "o"].T


# ── feed-forward ──
def gated(h, p, pre, act):
    return (act(h @ p[pre + "gate"].T) * (h @ p[pre + "up"].T)) @ p[pre + "down"].T


def route(h, p, pre, r):
    """Per token: the chosen experts (largest sigmoid score plus correction) and their weights (the score alone, times a constant)."""
    s = sigmoid(h @ p[pre + "router"].T)
    chosen = np.argsort(-(s + p[pre + "correction"]), axis=1, kind="stable")[:, :r["top"]]
    return chosen, np.take_along_axis(s, chosen, 1) * r["scale"]


def experts(h, p, pre, mlp):
    chosen, weight = route(h, p, pre, mlp["router"])
    y = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        w = (weight * (chosen == e)).sum(1)
        t = np.nonzero((chosen == e).any(1))[0]
        if len(t):
            y[t] += w[t, None] * gated(h[t], p, f"{pre}e{e}.", silu)
    return y


def feed_forward(h, p, pre, mlp):
    return gated(h, p, pre, gelu_tanh) if mlp["kind"] == "dense" else experts(h, p, pre, mlp)


MIXERS = {"wkv": wkv, "latent_attention": latent_attention}


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def logits_of(z, cfg):
    z = z * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z


def forward(cfg, p, tokens, return_layers=False):
    """Logits [T, vocab] of one sequence from position 0 (and the sum of the streams after every layer run)."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    e = embedding(cfg, p, tokens)
    X, sums = np.repeat(e[None], cfg["streams"], 0), []
    for i in layer_order(cfg):
        L, pre = cfg["layers"][i], f"l{i}."
        sub = [("1", lambda h: MIXERS[L["type"]](h, p, pre + "mix.", L["mixer"], eps))]
        if L.get("mlp") is not None:
            sub.append(("2", lambda h: feed_forward(h, p, pre + "mlp.", L["mlp"])))
        for n, f in sub:
            hc = pre + "hc" + n
            y = f(dynamic_tanh(read_streams(X, p[hc + ".in"]), p, pre + "norm" + n)) * p[pre + "ls" + n]
            X = write_streams(X, p[hc + ".mix"], p[hc + ".out"], m * y)
        sums.append(X.sum(0))
    z = logits_of(dynamic_tanh(X.sum(0), p, "final.norm") @ np.asarray(p["embed"], np.float64).T, cfg)
    return (z, np.array(sums)) if return_layers else z
