"""Small random Fomanex models for the tests: configurations of many shapes and bfloat16-exact random weights (so that the
device, whichever weight format it keeps, and the float64 restatement see the same numbers)."""
import numpy as np



def bf16_exact(x):
    """Round float32 values to the nearest bfloat16 (ties to even), returned as float32."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    u = (u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) & np.uint32(0xFFFF0000)
    return u.view(np.float32)


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=12, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def wkv_layer(heads=3, dim=8, rank=5, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp, "_rank": rank}


def yarn(factor=6.0, original=64, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent_layer(heads=3, dim=6, rot_dim=8, vdim=10, kv_rank=12, base=100.0, scaling="yarn", scale=None, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = yarn() if scaling == "yarn" else scaling
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
                                                               "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def config(layers, width=40, vocab=61, eps=1e-5, scale=1.5, streams=2, mult=0.6, logit_scale=0.3, softcap=4.0, loop=None):
    cfg = {"architecture": "Fomanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "streams": streams, "residual_mult": mult,
           "logit_scale": logit_scale, "layers": layers}
    if softcap:
        cfg["logit_softcap"] = softcap
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed=0, qk_gain=1.0):
    """name -> float32 array (bfloat16-exact).  `qk_gain` sharpens every softmax, so a key that is lost or a missing sink moves the output a
    lot.  Decays reach from a slow leak (hundreds of tokens) to a fast one; the mixing matrices are far from symmetric."""
    r = np.random.default_rng(seed)
    D, S, W = cfg["width"], cfg["streams"], {}

    def lin(n_out, n_in, gain=1.0):
        return r.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in)

    def around_one(*shape):
        return 1.0 + 0.2 * r.standard_normal(shape)

    def dyt(name):
        W[name], W[name + ".b"], W[name + ".alpha"] = around_one(D), 0.2 * r.standard_normal(D), np.asarray(0.25 + 0.25 * r.random())

    W["embed"] = r.standard_normal((cfg["vocab"], D))
    dyt("embed.norm")
    dyt("final.norm")

    def sublayer(p, q):
        dyt(f"{p}norm{q}")
        W[f"{p}ls{q}"] = around_one(D)
        W[f"{p}hc{q}.in"] = 0.7 / S + 0.3 * r.standard_normal(S)
        W[f"{p}hc{q}.out"] = 1.0 + 0.5 * r.standard_normal(S)
        W[f"{p}hc{q}.mix"] = 0.8 * np.eye(S) + 0.25 * r.standard_normal((S, S)) / np.sqrt(S)

    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L["mlp"]
        sublayer(p, 1)
        H, d = m["heads"], m["dim"]
        if L["type"] == "wkv":
            C, rank = H * d, L["_rank"]
            for s in "rkvgw":
                W[p + "mix.mu." + s] = r.random(D) * 1.2 - 0.1
            for s in "rkvg":
                W[p + "mix." + s] = lin(C, D, 1.5)
            W[p + "mix.w1"], W[p + "mix.w2"] = lin(rank, D, 2.0), lin(C, rank)
            W[p + "mix.w0"] = -6.0 + 6.0 * r.random(C)
            W[p + "mix.u"] = r.standard_normal((H, d))
            W[p + "mix.norm"] = around_one(C)
            W[p + "mix.o"] = lin(D, C)
        else:
            rd, dv, rk = m["rot_dim"], m["vdim"], m["kv_rank"]
            W[p + "mix.q"], W[p + "mix.dkv"] = lin(H * (d + rd), D, qk_gain), lin(rk + rd, D)
            W[p + "mix.dkv.norm"] = around_one(rk)
            W[p + "mix.uk"], W[p + "mix.uv"] = lin(H * d, rk), lin(H * dv, rk)
            W[p + "mix.sink"] = 1.0 + r.standard_normal(H)
            W[p + "mix.o"] = lin(D, H * dv, 1.5)
        if mlp is None:
            continue
        sublayer(p, 2)
        if mlp["kind"] == "dense":
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = lin(mlp["ff"], D, 1.5), lin(mlp["ff"], D), lin(D, mlp["ff"], 1.5)
        else:
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            W[p + "mlp.router"], W[p + "mlp.correction"] = lin(E, D, 2.0), 0.3 * r.standard_normal(E)
            for e in range(E):
                W[f"{p}mlp.e{e}.gate"], W[f"{p}mlp.e{e}.up"], W[f"{p}mlp.e{e}.down"] = lin(ff, D, 1.5), lin(ff, D), lin(D, ff, 2.0)
    return {k: bf16_exact(np.asarray(v, np.float32)).reshape(np.shape(v)) for k, v in W.items()}


def as_f64(W):
    return {k: v.astype(np.float64) for k, v in W.items()}
