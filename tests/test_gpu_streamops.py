"""The residual step over several streams alone, and the parameters that came with it, in one-op programs against NumPy at values and in
pairings no model of the framework uses: steps that only close or only open, any number of shifts, streams that start as one; gated
pairs and row limits of LINEAR; unequal heads and rounded products of HEAD_LINEAR; the bonus form of DELTA_RULE with every kind of decay;
scaled sigmoid routing with groups; query parts turned by the cache append, in place and elsewhere; a Dynamic Tanh after EMBED."""
import numpy as np
import pytest

from test_gpu_recops import ctl_words, run, sigmoid, weights

pytestmark = pytest.mark.gpu


def near(got, want, tol=2e-5):
    return np.abs(got - want).max() < tol * max(1.0, np.abs(want).max())


def arena(be, wdt, **parts):
    from zgml_b200.host.weights import WeightArena
    A = WeightArena(wdt)
    for k, v in parts.items():
        A.add(k, v)
    return A.upload(be), A.off


def exact(r, *shape):
    """bfloat16-exact values of about one."""
    return (np.round(r.standard_normal(shape) * 32) / 32).astype(np.float32)


@pytest.mark.parametrize("fmt", ["float32", "bfloat16"])
@pytest.mark.parametrize("S,T,D", [(1, 1, 9), (2, 5, 64), (3, 23, 40), (4, 9, 37), (3, 40, 516), (7, 12, 20), (16, 9, 8)])
def test_stream_step(cuda_backend, fmt, S, T, D):
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    wdt = abi.W_F32 if fmt == "float32" else abi.W_BF16
    r = np.random.default_rng(S * 100 + T)
    X, y = r.standard_normal((S, T, D)).astype(np.float32), r.standard_normal((T, D)).astype(np.float32)
    J = 8
    p = dict(out=exact(r, S), mix=exact(r, S, S), ls=exact(r, D), win=exact(r, S), norm=np.concatenate([exact(r, D), exact(r, D), np.array([0.75], np.float32)]), mu=exact(r, J, D))
    w, off = arena(cuda_backend, wdt, **p)
    P = {k: v.astype(np.float64) for k, v in p.items()}
    alpha, nw, nb = P["norm"][-1], P["norm"][:D], P["norm"][D:2 * D]
    dyt = lambda u: np.tanh(alpha * u) * nw + nb
    for ls in (True, False):
        closed = np.einsum("ab,atd->btd", P["mix"], X) + 0.7 * P["out"][:, None, None] * (y * (P["ls"] if ls else 1.0))[None]
        sizes = [S * T * D, S * T * D, T * D, w.elems, T * D]
        kw = dict(dst=0, src=1, src_stride=T * D, y=2, close_w=3, out_off=off["out"], mix_off=off["mix"], ls_off=off["ls"] if ls else None, mult=0.7)
        io, ext = [(1, X), (2, y)], [ExternBuffer(3, w)]
        assert near(run(cuda_backend, [DeviceOp.stream_step(T, D, S, wdt, **kw)], sizes, io, 0, X.shape, ext), closed)                       # closes only
        u = np.tensordot(P["win"], closed, (0, 0))
        for kind, h in (("dyt", dyt(u)), ("none", u)):
            op = DeviceOp.stream_step(T, D, S, wdt, **kw, h=4, open_w=3, in_off=off["win"], kind=kind, norm_off=off["norm"], gain=1.5)
            assert near(run(cuda_backend, [op], sizes, io, 0, X.shape, ext), closed) and near(run(cuda_backend, [op], sizes, io, 4, y.shape, ext), 1.5 * h)
    op = DeviceOp.stream_step(T, D, S, wdt, src=1, src_stride=T * D, h=4, open_w=3, in_off=off["win"], norm_off=off["norm"])                   # opens only, over streams that differ
    assert near(run(cuda_backend, [op], sizes, io, 4, y.shape, ext), dyt(np.tensordot(P["win"], X.astype(np.float64), (0, 0))))
    op = DeviceOp.stream_step(T, D, S, wdt, src=2, src_stride=0, h=4, open_w=3, in_off=off["win"], norm_off=off["norm"])                       # all streams equal to one
    assert near(run(cuda_backend, [op], sizes, io, 4, y.shape, ext), dyt(P["win"].sum() * y.astype(np.float64)))
    kw.update(src=2, src_stride=0, y=4)
    want = P["mix"].sum(0)[:, None, None] * y[None] + 0.7 * P["out"][:, None, None] * X[0][None]
    assert near(run(cuda_backend, [DeviceOp.stream_step(T, D, S, wdt, **kw)], sizes, [(2, y), (4, X[0])], 0, X.shape, ext), want)
    w.free()


@pytest.mark.parametrize("T,D,J", [(1, 9, 5), (7, 12, 1), (23, 40, 8), (50, 37, 3), (4, 8, 2)])
def test_stream_step_with_shifts(cuda_backend, T, D, J):
    """Several steps over one carried row, in the second of two slots; the row of the first stays."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    S, f = 3, abi.W_F32
    r = np.random.default_rng(T)
    p = dict(out=exact(r, S), mix=exact(r, S, S), win=exact(r, S), norm=np.concatenate([exact(r, D), exact(r, D), np.array([0.5], np.float32)]), mu=exact(r, J, D))
    w, off = arena(cuda_backend, f, **p)
    P = {k: v.astype(np.float64) for k, v in p.items()}
    state = DeviceBuffer(cuda_backend, 4 * 2 * D)
    other = r.standard_normal(D).astype(np.float32)
    state.upload(other)
    prev = np.zeros(D)
    for step in range(3):
        X, y = r.standard_normal((S, T, D)).astype(np.float32), r.standard_normal((T, D)).astype(np.float32)
        kw = dict(dst=0, src=1, src_stride=T * D, y=2, close_w=3, out_off=off["out"], mix_off=off["mix"]) if step else dict(src=1, src_stride=T * D)      # the first one only opens
        op = DeviceOp.stream_step(T, D, S, f, **kw, h=4, open_w=3, in_off=off["win"], norm_off=off["norm"], shifts=J, mu_off=off["mu"], state=5, ctl=6)
        got = run(cuda_backend, [op], [S * T * D, S * T * D, T * D, w.elems, T * J * D, state.elems, 8], [(1, X), (2, y), (6, ctl_words(3, 1))], 4, (T, J, D), [ExternBuffer(3, w), ExternBuffer(5, state)])
        new = np.einsum("ab,atd->btd", P["mix"], X) + P["out"][:, None, None] * y[None] if step else X.astype(np.float64)
        h = np.tanh(0.5 * np.tensordot(P["win"], new, (0, 0))) * P["norm"][:D] + P["norm"][D:2 * D]
        before = np.concatenate([prev[None], h[:-1]])
        assert near(got, h[:, None] + (before - h)[:, None] * P["mu"][None]), step
        prev = h[-1]
        assert near(state.download(np.float32, 4 * D, D), prev) and np.array_equal(state.download(np.float32, 0, D), other)
    state.free()
    w.free()


@pytest.mark.parametrize("fmt", ["float32", "bfloat16"])
def test_gated_pairs(cuda_backend, fmt):
    """One row, a few rows, an odd number of inputs, the exact f32 tile and the tensor-core product, with outputs that end inside a tile and
    rows that are not 16-byte aligned; every activation of the epilogue."""
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    wdt = abi.W_F32 if fmt == "float32" else abi.W_BF16
    r = np.random.default_rng(1)
    acts = {None: lambda v: v, "relu2": lambda v: np.maximum(v, 0) ** 2, "silu": lambda v: v * sigmoid(v), "gelu_tanh": lambda v: 0.5 * v * (1 + np.tanh(np.sqrt(2 / np.pi) * (v + 0.044715 * v ** 3))),
            "relu": lambda v: np.maximum(v, 0), "softcap": lambda v: 1.5 * np.tanh(v / 1.5)}
    for M, N, K in ((1, 24, 64), (1, 9, 300), (3, 17, 37), (8, 30, 256), (5, 6, 640), (40, 35, 50), (70, 165, 128), (130, 64, 72)):
        Wg, Wu = (np.round(r.standard_normal((N, K)) * 16).astype(np.float32) / 64 for _ in range(2))      # bfloat16-exact
        x = np.round(r.standard_normal((M, K)) * 8).astype(np.float32) / 16
        w, off = arena(cuda_backend, wdt, w=np.stack([Wg, Wu], 1))
        g, u = x.astype(np.float64) @ Wg.T.astype(np.float64), x.astype(np.float64) @ Wu.T.astype(np.float64)
        for name, fn in acts.items():
            for pad in (0, 3, 4):
                op = DeviceOp.linear(0, 1, 2, off["w"], M, N, K, wdt, act=name, act_param=1.5, dst_rs=N + pad, pairs=True)
                got = run(cuda_backend, [op], [M * (N + pad), M * K, w.elems], [(1, x)], 0, (M, N + pad), [ExternBuffer(2, w)])
                assert near(got[:, :N], fn(g) * u), (M, N, K, name, pad)
                assert not got[:, N:].any()
        w.free()


@pytest.mark.parametrize("fmt", ["float32", "bfloat16"])
def test_live_rows_of_a_state_buffer(cuda_backend, fmt):
    """Rows up to position + the step's tokens are right for every position, from the second slot; later tiles may be left alone."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    wdt = abi.W_F32 if fmt == "float32" else abi.W_BF16
    r = np.random.default_rng(3)
    R, N, K, T = 300, 24, 64, 16
    W = np.round(r.standard_normal((N, K)) * 16).astype(np.float32) / 64
    rows = np.round(r.standard_normal((2, R, K)) * 8).astype(np.float32) / 16
    w, off = arena(cuda_backend, wdt, w=W)
    state = DeviceBuffer(cuda_backend, rows.nbytes, zero=False)
    state.upload(rows)
    want = rows[1].astype(np.float64) @ W.T.astype(np.float64)
    for pos in (0, 47, 48, 112, 113, 128, 240, 284):
        op = DeviceOp.linear(0, 1, 2, off["w"], R, N, K, wdt, ctl=3, src_slot_stride=R * K, live_rows=T)
        got = run(cuda_backend, [op], [R * N, state.elems, w.elems, 8], [(3, ctl_words(pos, 1))], 0, (R, N), [ExternBuffer(1, state), ExternBuffer(2, w)])
        assert near(got[:pos + T], want[:pos + T])
        tail = -(-(pos + T) // 128) * 128
        assert not got[tail:].any()
    state.free()
    w.free()


@pytest.mark.parametrize("fmt", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,N,last,K", [(5, 24, 7, 64), (3, 10, 33, 72), (2, 130, 1, 256), (1, 9, 9, 640), (4, 12, 12, 37), (3, 256, 40, 128)])
def test_unequal_heads_of_a_block_diagonal_product(cuda_backend, fmt, H, N, last, K):
    """A last head with fewer or more outputs and an activation of its own, for one row, a few rows and many (tensor cores where the inputs may be
    rounded, exact tiles otherwise); sources and results in columns of wider rows."""
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    wdt = abi.W_F32 if fmt == "float32" else abi.W_BF16
    r = np.random.default_rng(H * N)
    W = np.round(r.standard_normal(((H - 1) * N + last, K)) * 16).astype(np.float32) / 64
    w, off = arena(cuda_backend, wdt, pad=np.zeros(8), w=W)
    srs, drs = 4 + H * K + 4, (H - 1) * (N + 4) + max(last, N) + 3
    for T in (1, 3, 8, 9, 70, 150):
        x = np.round(r.standard_normal((T, srs)) * 8).astype(np.float32) / 16
        for rounded, act in ((True, "softcap"), (False, "silu"), (True, None)):
            op = DeviceOp.head_linear(0, 1, 2, off["w"], T, H, N, K, wdt, src_col=4, src_rs=srs, dst_hs=N + 4, dst_rs=drs, n_last=last, last_act=act, last_act_param=2.0, rounded=rounded)
            got = run(cuda_backend, [op], [T * drs, T * srs, w.elems], [(1, x)], 0, (T, drs), [ExternBuffer(2, w)])
            for h in range(H):
                n = last if h == H - 1 else N
                z = x[:, 4 + h * K:4 + (h + 1) * K].astype(np.float64) @ W[h * N:h * N + n].T.astype(np.float64)
                if h == H - 1 and act:
                    z = 2.0 * np.tanh(z / 2.0) if act == "softcap" else z * sigmoid(z)
                assert near(got[:, h * (N + 4):h * (N + 4) + n], z), (T, h, rounded, act)
    w.free()


@pytest.mark.parametrize("dims", [(4, 2, 8, 12), (3, 1, 37, 70), (2, 2, 260, 9)], ids=["shared-keys", "odd", "260"])
@pytest.mark.parametrize("decay", ["exp", "softplus", "tempered", "exp-head"])
def test_bonus_form_of_the_delta_rule(cuda_backend, dims, decay):
    """Read before the write with a bonus, with every kind of decay, either width of the output norm, shared keys, a query scale and both
    gates: single tokens, short steps and prepared walks, one after the other over the same state in the second slot."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    H, G, dim, vdim = dims
    r = np.random.default_rng(sum(dims))
    n, C, per_head = 64, 2 * G * dim + H * vdim, decay == "exp-head"
    na = H if per_head else H * dim
    qkv, row = r.standard_normal((n, C)).astype(np.float32), r.standard_normal((n, na + H * vdim)).astype(np.float32)
    wide = decay in ("exp", "softplus")
    A, bias, u = (-1.0 + r.standard_normal(H)).astype(np.float32), (r.standard_normal(na) - 2.0).astype(np.float32), r.standard_normal((H, dim)).astype(np.float32)
    nw = (1 + 0.3 * r.standard_normal((H, vdim) if wide else vdim)).astype(np.float32)
    w, (oA, ob, ou, onw) = weights(cuda_backend, A, bias, u, nw)
    state = DeviceBuffer(cuda_backend, 4 * 2 * H * dim * vdim)
    rs = row.shape[1]
    got, at = [], 0
    for T in (5, 1, 1, 40, 1, 16):
        op = DeviceOp.delta_rule(0, 1, None, 2, 2, 3, 4, 5, 0, G * dim, 2 * G * dim, 0, oA, ob, onw, T, H, G, dim, vdim, C, 0, rs, rs, abi.W_F32, 1e-5, 0.0, 0.8, gate_off=na, plain=True,
                                 decay_tau=3.0 if decay == "tempered" else None, silu_gate=wide, head_decay=per_head, bonus_off=ou, exp_decay=decay.startswith("exp"), wide_norm=wide)
        got.append(run(cuda_backend, [op], [T * H * vdim, T * C, T * rs, w.elems, state.elems, 8], [(1, qkv[at:at + T]), (2, row[at:at + T]), (5, ctl_words(at, 1))], 0, (T, H, vdim),
                       [ExternBuffer(3, w), ExternBuffer(4, state)]))
        at += T
    assert at == n
    got = np.concatenate(got)
    X, Rw = qkv.astype(np.float64), row.astype(np.float64)
    q, k, v = X[:, :G * dim].reshape(n, G, dim) * 0.8, X[:, G * dim:2 * G * dim].reshape(n, G, dim), X[:, 2 * G * dim:].reshape(n, H, vdim)
    z = (Rw[:, :na] + bias).reshape(n, H, -1)
    g = {"e": lambda: np.exp(-np.exp(z)), "s": lambda: np.exp(-np.exp(A.astype(np.float64))[None, :, None] * np.logaddexp(0, z)), "t": lambda: sigmoid(z) ** (1 / 3.0)}[decay[0]]()
    S = np.zeros((H, dim, vdim))
    for t in range(n):
        for h in range(H):
            kk, qq = k[t, h // (H // G)], q[t, h // (H // G)]
            o = S[h].T @ qq + (qq * u[h] * kk).sum() * v[t, h]
            S[h] = g[t, h][:, None] * S[h] + np.outer(kk, v[t, h])
            gl = Rw[t, na + h * vdim:na + (h + 1) * vdim]
            want = o / np.sqrt((o ** 2).mean() + 1e-5) * (nw[h] if wide else nw) * sigmoid(gl) * (gl if wide else 1.0)
            assert near(got[t, h], want, 1e-4), (t, h)
    left = state.download(np.float32, 4 * H * dim * vdim, H * dim * vdim).reshape(H, dim, vdim)
    assert near(left, S, 1e-4) and not state.download(np.float32, 0, H * dim * vdim).any()
    state.free()
    w.free()


@pytest.mark.parametrize("NE,top,groups,keep", [(12, 3, 0, 0), (12, 3, 4, 2), (5, 5, 0, 0), (70, 4, 7, 1), (1, 1, 0, 0)])
def test_scaled_sigmoid_routing(cuda_backend, NE, top, groups, keep):
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    r = np.random.default_rng(NE)
    T = 9
    z, c = r.standard_normal((T, NE)).astype(np.float32), r.standard_normal(NE).astype(np.float32)
    w, (oc,) = weights(cuda_backend, c)
    op = DeviceOp.route(0, 1, 2, oc, T, NE, top, abi.W_F32, mode="scaled_sigmoid", groups=groups, groups_kept=keep, scale=2.5)
    got = run(cuda_backend, [op], [T * top * 2, T * NE, w.elems], [(1, z)], 0, (T, top, 2), [ExternBuffer(2, w)])
    s = sigmoid(z.astype(np.float64))
    for t in range(T):
        choice = s[t] + c
        if groups:
            per = NE // groups
            score = np.sort(choice.reshape(groups, per), axis=1)[:, -2:].sum(1)
            for g in np.argsort(-score)[keep:]:
                choice[g * per:(g + 1) * per] = -np.inf
        want = np.argsort(-choice)[:top]
        assert np.array_equal(got[t, :, 0].view(np.int32), want) and near(got[t, :, 1], 2.5 * s[t, want], 1e-6)
    w.free()


@pytest.mark.parametrize("layout", ["pairs", "halves"])
@pytest.mark.parametrize("elsewhere", [False, True])
def test_query_parts_turned_by_the_cache_append(cuda_backend, layout, elsewhere):
    """The rotated part of every query head turns by the angles of the shared key part, from the base or a table, with a magnitude, in place or
    into wider rows; everything else in those rows stays."""
    from zgml_b200 import DeviceBuffer, DeviceOp, ExternBuffer, abi
    r = np.random.default_rng(4)
    T, H, dim, rot, rank, pos, R, slots = 6, 5, 7, 10, 9, 11, 40, 2
    cw, dk, dst = rank + rot, dim + rot, 4 + rank + rot
    rs = H * dk + cw + 3
    x = r.standard_normal((T, rs)).astype(np.float32)
    nw = (1 + 0.3 * r.standard_normal(rank)).astype(np.float32)
    w, (onw,) = weights(cuda_backend, nw)
    table = (0.7 ** np.arange(rot // 2)).astype(np.float32)
    tab = DeviceBuffer(cuda_backend, 4 * (rot // 2 + 3), zero=False)
    tab.upload(np.concatenate([np.zeros(3, np.float32), table]))
    q_before = r.standard_normal((T, H, dst)).astype(np.float32)
    for use_table, mag in ((False, 0.0), (True, 1.3)):
        f = table.astype(np.float64) if use_table else 50.0 ** (-2.0 * np.arange(rot // 2) / rot)
        cache = DeviceBuffer(cuda_backend, 4 * slots * R * cw)
        op = DeviceOp.cache_append(2, 0, 1, H * dk, 0, T, cw, rs, cw, R, norm_w=3, norm_off=onw, normed=rank, eps=1e-5, wdt=abi.W_F32, rot=rot, rot_base=0.0 if use_table else 50.0, rot_layout=layout,
                                   freqs=4 if use_table else None, freqs_off=3 if use_table else 0, rot_scale=mag, turned_heads=(H, dim, dk, 5 if elsewhere else None, 4 + rank, dst))
        sizes, ext = [x.size, 8, cache.elems, w.elems, tab.elems, q_before.size], [ExternBuffer(2, cache), ExternBuffer(3, w), ExternBuffer(4, tab)]
        io = [(0, x), (1, ctl_words(pos, 1)), (5, q_before)]
        src, dest = run(cuda_backend, [op], sizes, io, 0, x.shape, ext), run(cuda_backend, [op], sizes, io, 5, q_before.shape, ext)
        rows = cache.download(np.float32, 4 * (R + pos) * cw, T * cw).reshape(T, cw)

        def turn(v, p):
            n = len(f)
            c, s = (mag or 1.0) * np.cos(p * f), (mag or 1.0) * np.sin(p * f)
            a, b = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if layout == "pairs" else (slice(0, n), slice(n, 2 * n))
            out = np.array(v, np.float64)
            out[..., a], out[..., b] = v[..., a] * c - v[..., b] * s, v[..., b] * c + v[..., a] * s
            return out

        for t in range(T):
            z = x[t, H * dk:H * dk + cw].astype(np.float64)
            assert near(rows[t, :rank], z[:rank] / np.sqrt((z[:rank] ** 2).mean() + 1e-5) * nw) and near(rows[t, rank:], turn(z[rank:], pos + t))
            heads = x[t, :H * dk].reshape(H, dk)
            want = turn(heads[:, dim:].astype(np.float64), pos + t)
            if elsewhere:
                assert near(dest[t, :, 4 + rank:], want) and np.array_equal(dest[t, :, :4 + rank], q_before[t, :, :4 + rank]) and np.array_equal(src, x)
            else:
                assert near(src[t, :H * dk].reshape(H, dk)[:, dim:], want) and np.array_equal(src[t, :H * dk].reshape(H, dk)[:, :dim], heads[:, :dim])
                assert np.array_equal(src[:, H * dk:], x[:, H * dk:]) and np.array_equal(dest, q_before)
        cache.free()
    w.free()
    tab.free()


def test_dynamic_tanh_after_the_embedding(cuda_backend):
    from zgml_b200 import DeviceOp, ExternBuffer, abi
    r = np.random.default_rng(5)
    V, D, ids = 11, 300, [3, 0, 10, 3]
    for wdt in (abi.W_F32, abi.W_BF16):
        table, pos, norm = exact(r, V, D), exact(r, 16, D), np.concatenate([exact(r, D), exact(r, D), np.array([0.5], np.float32)])
        w, off = arena(cuda_backend, wdt, table=table, pos=pos, norm=norm)
        c = np.concatenate([ctl_words(2, 0).view(np.int32), np.array(ids, np.int32)]).view(np.float32)
        for p in (None, off["pos"]):
            op = DeviceOp.embed(0, 1, 2, off["table"], 4, D, 1.5, wdt, positions_off=p, dyt_off=off["norm"])
            got = run(cuda_backend, [op], [4 * D, 12, w.elems], [(1, c)], 0, (4, D), [ExternBuffer(2, w)])
            x = 1.5 * table[ids].astype(np.float64) + (0.0 if p is None else pos[2:6])
            assert near(got, np.tanh(0.5 * x) * norm[:D] + norm[D:2 * D])
        w.free()


def test_malformed_ops_are_refused(cuda_backend):
    from zgml_b200 import DeviceOp, DeviceProgram, abi
    f = abi.W_F32
    step = lambda **kw: DeviceOp.stream_step(2, 4, 3, f, **{**dict(dst=0, src=1, src_stride=8, y=2, close_w=3, out_off=0, mix_off=4, h=4, open_w=3, in_off=16, norm_off=20), **kw})
    rule = lambda **kw: DeviceOp.delta_rule(0, 1, None, 2, 2, 3, 4, 5, 0, 8, 16, 0, 0, 0, 8, 2, 2, 2, 4, 4, 24, 0, 16, 16, f, 1e-5, 1e-6, 0.5, gate_off=8, **kw)
    append = lambda **kw: DeviceOp.cache_append(0, 1, 2, 12, 0, 2, 6, 20, 6, 8, norm_w=3, normed=4, wdt=f, rot=2, rot_base=9.0, **kw)
    sizes = {"step": [24, 24, 8, 32, 40, 8, 8], "rule": [16, 48, 32, 32, 32, 8], "append": [48, 40, 8, 8, 60], "linear": [16, 8, 32, 8], "heads": [40, 48, 100, 40]}
    good = [("step", step()), ("step", step(shifts=5, mu_off=0, state=5, ctl=6)), ("rule", rule(plain=True, bonus_off=16)), ("append", append(turned_heads=(3, 2, 4, 4, 4, 6))), ("append", append(turned_heads=(3, 2, 4, None, 0, 0))),
            ("linear", DeviceOp.linear(0, 1, 2, 0, 2, 4, 4, f, pairs=True)), ("heads", DeviceOp.head_linear(0, 1, 2, 0, 2, 3, 5, 4, f, n_last=8, dst_rs=20))]
    bad = [("step", step(src_stride=4)), ("step", step(dst=1)), ("step", step(mix_off=30)), ("step", step(norm_off=24)), ("step", step(h=0)), ("step", step(shifts=6, mu_off=0, state=5, ctl=6)),
           ("step", step(shifts=9, mu_off=0, state=5, ctl=6)), ("step", step(shifts=5, mu_off=14, state=5, ctl=6)), ("step", step(shifts=5, mu_off=0)), ("step", DeviceOp.stream_step(2, 4, 17, f, src=1, src_stride=0, h=4, open_w=3)),
           ("rule", rule(bonus_off=16)), ("rule", rule(plain=True, bonus_off=28)), ("rule", rule(plain=True, exp_decay=True, decay_tau=2.0)), ("rule", rule(plain=True, wide_norm=True, head_decay=True, bonus_off=32)),
           ("append", append(turned_heads=(3, 3, 4, None, 0, 0))), ("append", append(turned_heads=(3, 2, 4, 4, 5, 6))), ("append", append(turned_heads=(4, 2, 4, None, 0, 0))), ("append", append(rot_scale=-1.0)),
           ("linear", DeviceOp.linear(0, 1, 2, 0, 2, 5, 4, f, pairs=True)), ("linear", DeviceOp.linear(0, 1, 2, 0, 2, 4, 4, f, pairs=True, bias=3)), ("linear", DeviceOp.linear(0, 1, 2, 0, 2, 4, 4, f, live_rows=2)),
           ("heads", DeviceOp.head_linear(0, 1, 2, 0, 2, 3, 5, 4, f, n_last=8)), ("heads", DeviceOp.head_linear(0, 1, 2, 0, 2, 3, 5, 4, f, n_last=16, dst_rs=26)),
           ("heads", DeviceOp.head_linear(0, 1, 2, 0, 2, 3, 5, 4, f, gate=3, gate_rs=15, rounded=True))]
    for i, (kind, op) in enumerate(good):
        h = cuda_backend.compile_program(DeviceProgram([op], sizes[kind], [], [], []))
        assert h is not None, i
        cuda_backend.free_program(h)
    for i, (kind, op) in enumerate(bad):
        assert cuda_backend.compile_program(DeviceProgram([op], sizes[kind], [], [], [])) is None, i
