"""Forms of the sequence-model DeviceOps alone, in one-op programs against NumPy: pooled blocks and the mask that reads them, the
order of norm and rotation inside the cache append, norms with one number as their weight and the norm over a sum of norms, an
activation on part of a product's columns, the gate after a norm, one decay per head in the delta rule's forms, and constant
decays in the state-space scan — at parameter values and in pairings that no model of the framework uses."""
import numpy as np
import pytest

from test_gpu_recops import ctl_words, run, sigmoid, weights

pytestmark = pytest.mark.gpu


def near(got, want, tol=2e-5):
    return np.abs(got - want).max() < tol * max(1.0, np.abs(want).max())


def erf(z):
    import math
    return np.vectorize(math.erf)(z)


def test_exact_gelu(cuda_backend):
    from zgml_b200 import DeviceOp
    z = np.concatenate([np.linspace(-6, 6, 97), [0.0, 30.0, -30.0]]).astype(np.float32)
    got = run(cuda_backend, [DeviceOp.activation(0, 0, z.size, "gelu_erf")], [z.size], [(0, z)], 0, z.shape)
    assert near(got, 0.5 * z.astype(np.float64) * (1 + erf(z.astype(np.float64) / np.sqrt(2.0))), 1e-6)


@pytest.mark.parametrize("fmt", ["float32", "bfloat16"])
def test_activation_on_part_of_the_columns(cuda_backend, fmt):
    """One row, a few rows with an odd K, the exact f32 tile and the tensor-core product; ranges at both ends and inside a tile."""
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    from zgml_b200.host.weights import WeightArena
    wdt = abi.W_F32 if fmt == "float32" else abi.W_BF16
    r = np.random.default_rng(1)
    for M, N, K in ((1, 24, 64), (3, 17, 37), (40, 70, 50), (70, 330, 128)):
        W = np.round(r.standard_normal((N, K)) * 16).astype(np.float32) / 64      # bfloat16-exact
        x = np.round(r.standard_normal((M, K)) * 8).astype(np.float32) / 16
        A = WeightArena(wdt)
        ow = A.add("w", W)
        buf = A.upload(cuda_backend)
        z = x.astype(np.float64) @ W.astype(np.float64).T
        for kind, f in (("silu", lambda v: v * sigmoid(v)), ("gelu_erf", lambda v: 0.5 * v * (1 + erf(v / np.sqrt(2.0))))):
            for lo, hi in ((0, 5), (7, 16), (N - 3, N), (0, N)):
                want = z.copy()
                want[:, lo:hi] = f(z[:, lo:hi])
                op = DeviceOp.linear(0, 1, 2, ow, M, N, K, wdt, act=kind, act_cols=(lo, hi), dst_rs=N + 3)
                got = run(cuda_backend, [op], [M * (N + 3), M * K, buf.elems], [(1, x)], 0, (M, N + 3), [ExternBuffer(2, buf)])
                assert near(got[:, :N], want), (M, N, K, kind, lo, hi)
        buf.free()


def test_norms_with_one_number_and_outer_norms(cuda_backend):
    """A single number as the weight of a first, a chained, a second-source and an outer norm; rows in registers, rows wider than
    that, and many rows; the outer norm over one source and over two, as RMS and as layer norm."""
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    r = np.random.default_rng(2)
    f, eps = abi.W_F32, 1e-3
    rms = lambda v: v / np.sqrt((v ** 2).mean(-1, keepdims=True) + eps)
    ln = lambda v: (v - v.mean(-1, keepdims=True)) / np.sqrt(v.var(-1, keepdims=True) + eps)
    for T, D in ((3, 40), (1, 900), (2, 1500), (2, 4500), (70, 24)):
        x, x2, res = (r.standard_normal((T, D)).astype(np.float32) for _ in range(3))
        wv, wv2 = (1 + 0.2 * r.standard_normal(D)).astype(np.float32), (1 + 0.2 * r.standard_normal(D)).astype(np.float32)
        g1, g2 = np.float32(0.6), np.float32(-1.7)
        w, (oa, ob, oc, od) = weights(cuda_backend, wv, wv2, [g1], [g2])
        ext, sizes = [ExternBuffer(2, w)], [x.size, x.size, w.elems, x.size, x.size, x.size]
        io = [(1, x), (3, res), (5, x2)]
        X, X2, Rs = x.astype(np.float64), x2.astype(np.float64), res.astype(np.float64)

        def go(op, out):
            return run(cuda_backend, [op], sizes, io, out, x.shape, ext)

        closed = Rs + rms(X) * g1
        assert near(go(DeviceOp.norm(0, 1, 2, oc, T, D, eps, f, kind="rms_scalar", res=3), 0), closed)
        op = DeviceOp.norm(0, 1, 2, oc, T, D, eps, f, kind="rms_scalar", res=3, then=4, then_w=2, then_w_off=od, then_kind="rms_scalar")
        assert near(go(op, 0), closed) and near(go(op, 4), rms(closed) * g2)
        op = DeviceOp.norm(0, 1, None, 0, T, D, eps, f, kind="none", res=3, then=4, then_w=2, then_w_off=oc, then_kind="rms_scalar")
        assert near(go(op, 0), X + Rs) and near(go(op, 4), rms(X + Rs) * g1)
        both = 0.25 * (rms(X) * wv + rms(X2) * wv2)
        op = DeviceOp.norm(0, 1, 2, oa, T, D, eps, f, kind="rms", res=3, gain=0.25, src2=5, src2_w_off=ob, outer="rms_scalar", outer_w_off=od, then=4, then_w=2, then_w_off=oc, then_kind="rms_scalar")
        out = Rs + rms(both) * g2
        assert near(go(op, 0), out) and near(go(op, 4), rms(out) * g1)
        op = DeviceOp.norm(0, 1, 2, oc, T, D, eps, f, kind="rms_scalar", src2=5, src2_w_off=od, outer="layer", outer_w_off=ob, then=4, then_w=2, then_w_off=oa, then_kind="rms1")
        out = ln(rms(X) * g1 + rms(X2) * g2) * wv2
        assert near(go(op, 0), out) and near(go(op, 4), rms(out) * (1.0 + wv))
        op = DeviceOp.norm(0, 1, 2, oa, T, D, eps, f, kind="layer", res=3, outer="rms", outer_w_off=ob)
        assert near(go(op, 0), Rs + rms(ln(X) * wv) * wv2)
        w.free()


def test_gate_forms_of_the_gated_norm(cuda_backend):
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    r = np.random.default_rng(3)
    for T, cols, groups in ((5, 24, 3), (2, 70, 1), (1, 9000, 2)):
        y, g = r.standard_normal((T, cols + 2)).astype(np.float32), r.standard_normal((T, 5 + cols)).astype(np.float32)
        gw = (1 + 0.3 * r.standard_normal(cols)).astype(np.float32)
        w, (off,) = weights(cuda_backend, gw)
        Y, G = y[:, :cols].astype(np.float64), g[:, 5:].astype(np.float64)
        for after in (False, True):
            for sig in (False, True):
                gate = sigmoid(G) if sig else G * sigmoid(G)
                v = (Y if after else Y * gate).reshape(T, groups, -1)
                want = (v / np.sqrt((v ** 2).mean(-1, keepdims=True) + 1e-5)).reshape(T, cols) * gw * (gate if after else 1.0)
                op = DeviceOp.gated_norm(0, 1, 2, 3, off, 5, T, cols, groups, 5 + cols, 1e-5, abi.W_F32, src_rs=cols + 2, gate_after=after, sigmoid_gate=sig)
                got = run(cuda_backend, [op], [T * cols, y.size, g.size, w.elems], [(1, y), (2, g)], 0, (T, cols), [ExternBuffer(3, w)])
                assert near(got, want), (T, cols, after, sig)
        w.free()


def rotate(v, p, f, layout):
    n = len(f)
    c, s = np.cos(p * f), np.sin(p * f)
    a, b = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if layout == "pairs" else (slice(0, n), slice(n, 2 * n))
    out = v.copy()
    out[..., a], out[..., b] = v[..., a] * c - v[..., b] * s, v[..., b] * c + v[..., a] * s
    return out


@pytest.mark.parametrize("layout", ["pairs", "halves"])
@pytest.mark.parametrize("order", ["rotate_norm", "norm_rotate", "rotate"])
def test_order_of_norm_and_rotation(cuda_backend, order, layout):
    """All three orders in both layouts, from the base or a table, with a temperature on the normed queries."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    r = np.random.default_rng(4)
    T, H, G, dim, dv, pos, R, rot = 6, 5, 2, 70, 7, 9, 32, 66
    cw = G * (dim + dv)
    rs = H * dim + cw
    x = r.standard_normal((T, rs)).astype(np.float32)
    wq, wk = (1 + 0.3 * r.standard_normal(dim)).astype(np.float32), (1 + 0.3 * r.standard_normal(dim)).astype(np.float32)
    w, (oq, ok) = weights(cuda_backend, wq, wk)
    table = (0.7 ** np.arange(rot // 2)).astype(np.float32)
    tab = DeviceBuffer(cuda_backend, 4 * (rot // 2 + 3), zero=False)
    tab.upload(np.concatenate([np.zeros(3, np.float32), table]))
    for use_table, coef, every in ((False, 0.0, 0), (True, 0.8, 4)):
        f = table.astype(np.float64) if use_table else 50.0 ** (-2.0 * np.arange(rot // 2) / rot)
        cache = DeviceBuffer(cuda_backend, 4 * R * cw)
        op = DeviceOp.cache_append(2, 0, 1, H * dim, 0, T, cw, rs, cw, R, norm_w=None if order == "rotate" else 3, norm_off=ok, normed=G * dim, eps=1e-5, wdt=abi.W_F32, norm_group=dim, q_heads=H,
                                   q_col=0, q_norm_off=oq, temp_coef=coef, temp_every=every, head_rot=rot, rot_base=0.0 if use_table else 50.0, rot_layout=layout, freqs=4 if use_table else None,
                                   freqs_off=3 if use_table else 0, order=order)
        got = run(cuda_backend, [op], [x.size, 8, cache.elems, w.elems, tab.elems], [(0, x), (1, ctl_words(pos, 0))], 0, x.shape, [ExternBuffer(2, cache), ExternBuffer(3, w), ExternBuffer(4, tab)])
        rows = cache.download(np.float32, 4 * pos * cw, T * cw).reshape(T, cw)
        rms = lambda v: v / np.sqrt((v ** 2).mean(-1, keepdims=True) + 1e-5)
        for t in range(T):
            temp = 1.0 + coef * np.log((pos + t + 1) // every + 1) if every else 1.0
            for part, weight, mult, out in ((x[t, :H * dim].reshape(H, dim), wq, temp, got[t, :H * dim].reshape(H, dim)), (x[t, H * dim:(H + G) * dim].reshape(G, dim), wk, 1.0, rows[t, :G * dim].reshape(G, dim))):
                v = part.astype(np.float64)
                want = {"rotate_norm": lambda: rms(rotate(v, pos + t, f, layout)) * weight * mult, "norm_rotate": lambda: rotate(rms(v) * weight * mult, pos + t, f, layout),
                        "rotate": lambda: rotate(v, pos + t, f, layout)}[order]()
                assert near(out, want), (order, layout, t)
        assert np.array_equal(rows[:, G * dim:], x[:, (H + G) * dim:]) and np.array_equal(got[:, H * dim:], x[:, H * dim:])
        cache.free()
    w.free()
    tab.free()


@pytest.mark.parametrize("dims", [(4, 2, 8, 12), (2, 1, 64, 32), (3, 3, 7, 5), (40, 2, 20, 144)], ids=["grouped", "64", "odd", "40-heads"])
@pytest.mark.parametrize("size,pool", [(23, 4), (5, 5), (1, 1), (8, 19), (64, 3)])
def test_pooled_blocks(cuda_backend, dims, size, pool):
    """The append keeps every block's mean row, however the tokens come (steps of 10, 3, 1 and again 10), in a slot of its own; the
    attention sees the blocks that lie wholly before each query's window.  Keys that stand out now and then make a lost or doubled
    block show; a ring just long enough wraps under the blocks; sinks and the score cap apply to blocks as to tokens."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    H, G, dk, dv = dims
    n, width = 96, G * (dk + dv)
    R, NB = max(size - 1, pool) + 10, (n + pool - 1) // pool
    r = np.random.default_rng(sum(dims) + size)
    q = r.standard_normal((n, H, dk)).astype(np.float32)
    kv = r.standard_normal((n, width)).astype(np.float32)
    kv[::7] *= 3.0
    sinks = r.standard_normal(H).astype(np.float32)
    w, (os_,) = weights(cuda_backend, sinks)
    cache, pooled = DeviceBuffer(cuda_backend, 4 * 2 * R * width), DeviceBuffer(cuda_backend, 4 * 2 * NB * width)
    steps, at = [], 0
    for T in [10] * 3 + [3] * 4 + [1] * 24 + [10, 1, 1, 10, 4, 2, 1, 1]:
        steps.append((at, T))
        at += T
    assert at == n
    got = []
    for at, T in steps:
        ops = [DeviceOp.cache_append(3, 1, 2, 0, 0, T, width, width, width, R, pooled=5, pool=pool, pool_rows=NB),
               DeviceOp.cached_attention(4, 0, 3, 3, 2, 0, 0, G * dk, T, H, G, 1, dk, dv, H * dk, width, width, R, 0.4, mask="pooled", mask_size=size, pooled=5, pool=pool, pool_rows=NB,
                                         softcap=6.0, sink=6, sink_off=os_)]
        sizes = [T * H * dk, T * width, 8 + T, cache.elems, T * H * dv, pooled.elems, w.elems]
        got.append(run(cuda_backend, ops, sizes, [(0, q[at:at + T]), (1, kv[at:at + T]), (2, ctl_words(at, 1, 8 + T))], 4, (T, H, dv),
                       [ExternBuffer(3, cache), ExternBuffer(5, pooled), ExternBuffer(6, w)]))
    got = np.concatenate(got)
    k, v = kv[:, :G * dk].reshape(n, G, dk).astype(np.float64), kv[:, G * dk:].reshape(n, G, dv).astype(np.float64)
    done = (n - 1) // pool                                  # blocks that ended before the last token
    rows = pooled.download(np.float32, 4 * NB * width, done * width).reshape(done, width)
    assert near(rows, kv[:done * pool].astype(np.float64).reshape(done, pool, width).mean(1), 1e-6)
    assert not pooled.download(np.float32, 0, NB * width).any()                       # the other slot is untouched
    for p in range(n):
        lo = max(0, p + 1 - size)
        blocks = [b for b in range(n) if (b + 1) * pool - 1 <= p - size]
        K = np.concatenate([k[lo:p + 1]] + [k[b * pool:(b + 1) * pool].mean(0)[None] for b in blocks])
        V = np.concatenate([v[lo:p + 1]] + [v[b * pool:(b + 1) * pool].mean(0)[None] for b in blocks])
        for h in range(H):
            g = h // (H // G)
            s = 6.0 * np.tanh(0.4 * (K[:, g] @ q[p, h].astype(np.float64)) / 6.0)
            e = np.exp(s)
            want = (e / (e.sum() + np.exp(np.float64(sinks[h])))) @ V[:, g]
            assert np.abs(got[p, h] - want).max() < 3e-5 * max(1.0, np.abs(want).max()), (p, h)
    for b in (cache, pooled, w):
        b.free()


@pytest.mark.parametrize("dims", [(4, 2, 8, 12), (3, 1, 37, 70), (2, 2, 260, 9)], ids=["small", "odd", "260"])
@pytest.mark.parametrize("plain", [False, True])
@pytest.mark.parametrize("tau", [None, 3.0])
def test_one_decay_per_head_in_every_form_of_the_delta_rule(cuda_backend, dims, plain, tau):
    """The corrected and the plain rule, either kind of decay, single tokens, short steps and prepared walks, one after the other over
    the same state; decay logits and gates in columns of a wider row, and the output in columns of one."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    H, G, dim, vdim = dims
    r = np.random.default_rng(sum(dims))
    n, C = 64, 2 * G * dim + H * vdim
    qkv, row = r.standard_normal((n, C)).astype(np.float32), r.standard_normal((n, 3 + 2 * H + H * vdim)).astype(np.float32)
    A, dt, nw = (-1.0 + r.standard_normal(H)).astype(np.float32), r.standard_normal(H).astype(np.float32), (1 + 0.3 * r.standard_normal(vdim)).astype(np.float32)
    w, (oA, odt, onw) = weights(cuda_backend, A, dt, nw)
    state = DeviceBuffer(cuda_backend, 4 * 2 * H * dim * vdim)
    rs, drs = row.shape[1], H * vdim + 5
    got, at = [], 0
    for T in (5, 1, 1, 40, 1, 16):
        op = DeviceOp.delta_rule(0, 1, None if plain else 2, 2, 2, 3, 4, 5, 0, G * dim, 2 * G * dim, 0 if plain else 3, oA, odt, onw, T, H, G, dim, vdim, C, 0 if plain else rs, rs, rs, abi.W_F32, 1e-5, 1e-6,
                                 dim ** -0.5, gate_off=3 + 2 * H, plain=plain, decay_tau=tau, head_decay=True, a_col=3 + H, dst_rs=drs, dst_col=5)
        got.append(run(cuda_backend, [op], [T * drs, T * C, T * rs, w.elems, state.elems, 8], [(1, qkv[at:at + T]), (2, row[at:at + T]), (5, ctl_words(at, 1))], 0, (T, drs),
                       [ExternBuffer(3, w), ExternBuffer(4, state)])[:, 5:])
        at += T
    assert at == n
    got = np.concatenate(got).reshape(n, H, vdim)
    X, Rw = qkv.astype(np.float64), row.astype(np.float64)
    q, k = X[:, :G * dim].reshape(n, G, dim), X[:, G * dim:2 * G * dim].reshape(n, G, dim)
    v = X[:, 2 * G * dim:].reshape(n, H, vdim)
    if not plain:
        q, k = q / np.sqrt((q ** 2).sum(-1, keepdims=True) + 1e-6), k / np.sqrt((k ** 2).sum(-1, keepdims=True) + 1e-6)
    z = Rw[:, 3 + H:3 + 2 * H] + dt
    decay = sigmoid(z) ** (1.0 / tau) if tau else np.exp(-np.exp(A.astype(np.float64)) * np.logaddexp(0, z))
    beta = np.ones((n, H)) if plain else sigmoid(Rw[:, 3:3 + H])
    S = np.zeros((H, dim, vdim))
    for t in range(n):
        for h in range(H):
            g = h // (H // G)
            S[h] *= decay[t, h]
            u = v[t, h] if plain else beta[t, h] * (v[t, h] - S[h].T @ k[t, g])
            S[h] += np.outer(k[t, g], u)
            o = S[h].T @ (q[t, g] * dim ** -0.5)
            want = o / np.sqrt((o ** 2).mean() + 1e-5) * nw * sigmoid(Rw[t, 3 + 2 * H + h * vdim:3 + 2 * H + (h + 1) * vdim])
            assert near(got[t, h], want, 1e-4), (t, h)
    state.free()
    w.free()


@pytest.mark.parametrize("dims", [(4, 2, 8, 12), (3, 1, 37, 70), (2, 2, 260, 10)], ids=["shared-keys", "odd", "260"])
def test_constant_decays_in_the_state_space_scan(cuda_backend, dims):
    """A table of decays, among them 0 and 1; long steps in segments side by side, short ones and single tokens over one state; heads that
    share keys and queries."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    from zgml_b200.backend import seq_state_elems
    H, G, N, P = dims
    r = np.random.default_rng(sum(dims))
    n, rs = 310, H * P + 2 * G * N + 3
    x = (r.standard_normal((n, rs)) / N ** 0.25).astype(np.float32)
    decay = np.array(([0.0, 1.0, 0.98, 0.6] * 2)[:H], np.float32)
    tab = DeviceBuffer(cuda_backend, 4 * (H + 2), zero=False)
    tab.upload(np.concatenate([np.zeros(2, np.float32), decay]))
    probe = DeviceOp.ssm_scan(0, 0, 0, None, 0, 0, 0, 0, 0, 0, 0, 0, 0, 1, H, G, N, P, 1, 1, abi.W_BF16, constant_decay=True)
    state = DeviceBuffer(cuda_backend, 4 * 2 * seq_state_elems(probe))
    got, at = [], 0
    for T in (3, 1, 256, 1, 1, 48):
        op = DeviceOp.ssm_scan(0, 1, 2, None, 3, 4, 3, 3 + H * P, 3 + H * P + G * N, 2, 0, 0, 0, T, H, G, N, P, rs, 0, abi.W_BF16, constant_decay=True)
        got.append(run(cuda_backend, [op], [T * H * P, T * rs, tab.elems, state.elems, 8], [(1, x[at:at + T]), (4, ctl_words(at, 1))], 0, (T, H, P), [ExternBuffer(2, tab), ExternBuffer(3, state)]))
        at += T
    assert at == n
    got = np.concatenate(got)
    X = x.astype(np.float64)
    v, k, q = X[:, 3:3 + H * P].reshape(n, H, P), X[:, 3 + H * P:3 + H * P + G * N].reshape(n, G, N), X[:, 3 + H * P + G * N:].reshape(n, G, N)
    S = np.zeros((H, N, P))
    for t in range(n):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.float64(decay[h]) * S[h] + np.outer(k[t, g], v[t, h])
            assert near(got[t, h], S[h].T @ q[t, g], 1e-4), (t, h)
    state.free()
    tab.free()


def test_malformed_forms_are_refused(cuda_backend):
    from zgml_b200 import DeviceOp, DeviceProgram, abi
    f = abi.W_F32
    append = dict(T=4, cols=8, src_rs=8, width=8, rows=16)
    attend = dict(T=4, H=2, G=1, maps=1, dk=4, dv=4, q_rs=8, k_width=8, v_width=8, rows=16, scale=1.0)
    bad = [
        (DeviceOp.cache_append(0, 1, 2, 0, 0, **append, pooled=3, pool=13, pool_rows=4), [128, 32, 16, 64]),                # the ring does not hold a block and a step
        (DeviceOp.cache_append(0, 1, 2, 0, 0, **append, pooled=3, pool=4, pool_rows=9), [128, 32, 16, 64]),                 # fewer pooled rows than named
        (DeviceOp.cache_append(0, 1, 2, 0, 0, **append, pooled=0, pool=4, pool_rows=4), [128, 32, 16]),                     # pooled rows in the cache itself
        (DeviceOp.cache_append(0, 1, 2, 0, 0, **append, normed=4, norm_group=4, order="norm_rotate", norm_w=3), [128, 32, 16, 8]),     # an order without a rotation
        (DeviceOp.cache_append(0, 1, 2, 0, 0, **append, normed=4, norm_group=4, head_rot=4, rot_base=9.0, order="norm_rotate"), [128, 32, 16, 8]),   # a norm without a weight
        (DeviceOp.cached_attention(0, 1, 2, 2, 3, 0, 0, 4, **attend, mask="pooled", mask_size=4, pooled=4, pool=0, pool_rows=4), [32, 32, 128, 16, 64]),
        (DeviceOp.cached_attention(0, 1, 2, 2, 3, 0, 0, 4, **attend, mask="pooled", mask_size=4, pooled=4, pool=4, pool_rows=9), [32, 32, 128, 16, 64]),
        (DeviceOp.cached_attention(0, 1, 2, 4, 3, 0, 0, 4, **attend, mask="pooled", mask_size=4, pooled=5, pool=4, pool_rows=4), [32, 32, 128, 16, 128, 64]),    # two caches, one pooled buffer
        (DeviceOp.linear(0, 1, 2, 0, 2, 8, 4, f, act="silu", act_cols=(5, 9)), [16, 8, 32]),                                # columns past the end
        (DeviceOp.linear(0, 1, 2, 0, 2, 8, 4, f, act="silu", act_cols=(6, 5)), [16, 8, 32]),
        (DeviceOp.norm(0, 1, 2, 8, 2, 8, 1e-5, f, kind="rms_scalar"), [16, 16, 8]),                                          # the number lies past the arena
        (DeviceOp.norm(0, 1, 2, 0, 2, 8, 1e-5, f, kind="rms", res=0, outer="rms", outer_w_off=0), [16, 16, 8]),              # an outer norm over its own residual
        (DeviceOp.gated_norm(0, 1, 2, 3, 0, 0, 2, 8, 1, 6, 1e-5, f, gate_after=True), [16, 16, 16, 8]),                       # gate columns leave the row
        (DeviceOp.embed(0, 1, 2, 0, 2, 4, 1.0, f, bigram=(8, 5, 1, 1)), [8, 16, 31]),                                        # the bigram table lacks its last row
        (DeviceOp.ssm_scan(0, 1, 2, None, 3, 4, 0, 8, 12, 1, 0, 0, 0, 2, 2, 1, 4, 4, 16, 0, f, constant_decay=True), [16, 32, 2, 8192, 8]),    # fewer decays than heads
        (DeviceOp.delta_rule(0, 1, 2, 2, 2, 3, 4, 5, 0, 4, 8, 0, 0, 8, 16, 2, 2, 1, 4, 4, 16, 12, 3, 12, f, 1e-5, 1e-6, 0.5, head_decay=True, a_col=2), [16, 32, 24, 32, 32, 8]),  # decay logits leave the row
    ]
    for i, (op, sizes) in enumerate(bad):
        assert cuda_backend.compile_program(DeviceProgram([op], sizes, [], [], [])) is None, i
