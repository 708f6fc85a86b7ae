"""Small random Fotovik models for the tests: configurations of many shapes and bfloat16-exact random weights (so that the
device, whichever weight format it keeps, and the float64 restatement see the same numbers)."""
import numpy as np


def bf16_exact(x):
    """Round float32 values to the nearest bfloat16 (ties to even), returned as float32."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    u = (u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) & np.uint32(0xFFFF0000)
    return u.view(np.float32)


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def attention_layer(heads=4, kv_heads=2, dim=8, vdim=12, rot_dims=6, base=50.0, size=9, pool=4, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims}, "mask": {"size": size, "pool": pool},
                      "scale": dim ** -0.5 if scale is None else scale}}


def delta_layer(heads=4, kv_heads=2, dim=8, vdim=12, conv=3, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def pair_layer(heads=4, kv_heads=2, dim=8, vdim=12, rot_dims=6, base=50.0, factor=3.0, scale=None, r_heads=3, r_dim=6, r_vdim=10, decay=None, mlp=None):
    rot = {"base": base, "dims": rot_dims}
    if factor:
        rot["scaling"] = {"factor": factor}
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": dim ** -0.5 if scale is None else scale}
    decay = [0.97 - 0.2 * i / max(1, r_heads - 1) for i in range(r_heads)] if decay is None else decay
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay}}}


def config(layers, width=40, vocab=61, eps=1e-5, scale=1.5, bigram=(37, 11, 5), loop=None):
    cfg = {"architecture": "Fotovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if bigram:
        cfg["embedding"]["bigram"] = {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed=0, qk_gain=1.0):
    """name -> float32 array (bfloat16-exact).  `qk_gain` sharpens every softmax, so a key that is lost or seen once too often, or a
    missing sink, moves the output a lot."""
    r = np.random.default_rng(seed)
    D, W = cfg["width"], {}

    def lin(n_out, n_in, gain=1.0):
        return r.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in)

    def norm(n=None):
        return 1.0 + 0.2 * r.standard_normal(n) if n else np.asarray(1.0 + 0.3 * r.standard_normal())

    W["embed"] = r.standard_normal((cfg["vocab"], D))
    b = cfg["embedding"].get("bigram")
    if b:
        W["bigram"] = r.standard_normal((b["buckets"] + 1, D))
    W["final.norm"] = norm()
    W["head"] = lin(cfg["vocab"], D)

    def attention(p, m, qk_norm, sink):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        W[p + "q"], W[p + "k"], W[p + "v"], W[p + "o"] = lin(H * d, D, 1.0 if qk_norm else qk_gain), lin(G * d, D), lin(G * dv, D), lin(D, H * dv)
        if qk_norm:
            W[p + "q.norm"], W[p + "k.norm"] = qk_gain * norm(d), norm(d)
        if sink:
            W[p + "sink"] = 1.0 + r.standard_normal(H)

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        W[p + "norm1"], W[p + "norm1b"] = norm(), norm()
        if L["type"] == "attention":
            attention(p + "mix.", m, False, True)
        elif L["type"] == "delta":
            H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                W[p + f"mix.{n}"] = lin(rows, D)
                W[p + f"mix.{n}.conv"] = 0.6 * r.standard_normal((rows, taps)) + (np.arange(taps) == taps - 1)
            W[p + "mix.b"], W[p + "mix.a"] = lin(H, D, 2.0), lin(H, D)
            W[p + "mix.A_log"] = -2.0 + 1.5 * r.standard_normal(H)             # decays between a slow leak and a fast one
            W[p + "mix.dt_bias"] = 0.5 * r.standard_normal(H)
            W[p + "mix.norm"] = norm(dv)
            W[p + "mix.g"], W[p + "mix.o"] = lin(H * dv, D), lin(D, H * dv)
        else:
            attention(p + "mix.left.", m["left"], True, False)
            rt = m["right"]
            Hr, dr, vr = rt["heads"], rt["dim"], rt["vdim"]
            for n, rows in (("q", Hr * dr), ("k", Hr * dr), ("v", Hr * vr), ("g", Hr * vr)):
                W[p + f"mix.right.{n}"] = lin(rows, D, 1.5)
            W[p + "mix.right.norm"] = norm(Hr * vr)
            W[p + "mix.right.o"] = lin(D, Hr * vr)
            W[p + "mix.left.out"], W[p + "mix.right.out"] = norm(D), norm(D)
        if L["mlp"] is not None:
            W[p + "norm2"], W[p + "norm2b"] = norm(), norm()
            W[p + "mlp.up"], W[p + "mlp.down"] = lin(L["mlp"]["ff"], D, 1.5), lin(D, L["mlp"]["ff"])
    return {k: bf16_exact(np.asarray(v, np.float32)).reshape(np.shape(v)) for k, v in W.items()}


def as_f64(W):
    return {k: v.astype(np.float64) for k, v in W.items()}
