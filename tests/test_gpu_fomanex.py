"""Fomanex on the CUDA backend against the float64 restatement (tests/fomanex_reference.py): every mechanism alone, the sum of the
streams after every layer run, whole prompts, token-by-token decoding through the cached latents and recurrent states, prompts cut
into portions down to two tokens, interleaved requests in several slots, slot reuse, far keys and far writes by construction, sinks,
causality, the first tokens of a sequence, long decoding, many shapes, mistakes planted in the restatement that must show, and greedy
generation through the registry's entry point and the trace replayer."""
import json
import os
import subprocess

import numpy as np
import pytest

import fomanex_reference as ref
from fomanex_models import as_f64, config, dense, latent_layer, moe, random_weights, wkv_layer, yarn

pytestmark = pytest.mark.gpu

TOL = 2e-4   # of the logits' scale; f32 accumulation against float64


def tol(dtype):
    """A bfloat16 session rounds the activations that enter a tensor-core matmul (steps of more than 8 tokens) to bf16."""
    return TOL if dtype == "float32" else 3e-2


def open_model(be, cfg, W, dtype="float32", n_slots=1, max_chunk=16, keep_layers=False, max_context=512):
    from zgml_b200.host.fomanex import FomanexConfig, FomanexModel
    from zgml_b200.host.session import SequenceSession
    model = FomanexModel(be, FomanexConfig.from_dict(cfg), lambda n: W[n], dtype)
    return SequenceSession(be, model, n_slots=n_slots, max_chunk=max_chunk, keep_layers=keep_layers, max_context=max_context)


def close(s):
    s.close()
    s.model.close()


def rel(got, want):
    return float(np.max(np.abs(got.astype(np.float64) - want)) / (np.max(np.abs(want)) + 1e-30))


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def forward(cfg, W, toks):
    return ref.forward(cfg, as_f64(W), toks, return_layers=True)


def decode(s, request, toks, prompt=0):
    """Logits of every token: the first `prompt` tokens as one step, the rest one by one."""
    got = [s.feed(request, toks[:prompt], range(prompt))] if prompt else []
    return np.concatenate(got + [s.feed(request, [t], [0]) for t in toks[prompt:]])


# layers 1 .. 3 run twice; a layer before and two after the loop, one of them without a feed-forward
MIXED = config([wkv_layer(heads=2, dim=5, rank=3, mlp=dense(ff=9)), latent_layer(mlp=moe()), wkv_layer(mlp=moe(experts=5, top=3, ff=8)), latent_layer(heads=2, dim=4, rot_dim=6, vdim=5, kv_rank=7, mlp=dense()),
                wkv_layer(heads=1, dim=12), latent_layer(heads=5, dim=8, rot_dim=4, vdim=8, kv_rank=16, scaling=None, mlp=dense(ff=24))], streams=3, loop=(1, 4, 2))


# ── each mechanism alone (a one-layer model without a feed-forward isolates its mixer) ──
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("layer", [
    wkv_layer(),
    wkv_layer(heads=1, dim=3, rank=1),
    wkv_layer(heads=1, dim=4, rank=40),                      # the decay's low rank is wider than the heads
    wkv_layer(heads=5, dim=36, rank=12),
    wkv_layer(heads=2, dim=64, rank=64),
    wkv_layer(heads=2, dim=130, rank=8),
    latent_layer(),
    latent_layer(heads=1, dim=16, rot_dim=2, vdim=4, kv_rank=8, base=10000.0),
    latent_layer(heads=6, dim=4, rot_dim=16, vdim=20, kv_rank=36, scaling=yarn(factor=1.0, original=32, fast=2.0, slow=1.0)),     # a factor that slows nothing
    latent_layer(heads=4, dim=32, rot_dim=32, vdim=16, kv_rank=64, scaling=yarn(factor=40.0, original=4096, fast=32.0, slow=1.0), scale=0.3),
    latent_layer(heads=2, dim=10, rot_dim=12, vdim=6, kv_rank=20, base=50.0, scaling=yarn(factor=3.0, original=20, fast=1.0, slow=0.9)),   # a ramp of one step
    latent_layer(heads=3, dim=7, rot_dim=6, vdim=5, kv_rank=9, scaling=None),
    latent_layer(heads=17, dim=8, rot_dim=4, vdim=8, kv_rank=24),       # more heads than the few-rows kernel holds
    latent_layer(heads=2, dim=12, rot_dim=8, vdim=16, kv_rank=264),
], ids=["wkv", "wkv-3", "wkv-wide-rank", "wkv-36", "wkv-64", "wkv-130", "latent", "latent-1head-2rot", "latent-factor1", "latent-32", "latent-step-ramp", "latent-plain-rotary", "latent-17heads", "latent-264"])
def test_mixer_alone(cuda_backend, layer, dtype):
    cfg = config([layer], width=40, vocab=61)
    W = random_weights(cfg, seed=5, qk_gain=3.0)
    toks = tokens(cfg, 75)
    want, stream = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, n_slots=2, max_chunk=64, keep_layers=True)
    got = s.feed("a", toks, range(75))
    if dtype == "float32":
        assert rel(s.layer_streams(64, "all")[0], stream[0][:64]) < TOL
    assert rel(got, want) < tol(dtype)
    assert rel(decode(s, "d", toks), want) < TOL          # single tokens take the exact row kernels in both formats
    close(s)


@pytest.mark.parametrize("mlp", [dense(), dense(ff=7), dense(ff=300), moe(), moe(experts=1, top=1, ff=5, scale=1.0), moe(experts=9, top=9, ff=16, scale=0.5), moe(experts=40, top=3, ff=64, scale=2.5), None],
                         ids=["dense", "dense-7", "dense-300", "moe", "moe-1of1", "moe-9of9", "moe-3of40", "none"])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_feed_forward(cuda_backend, mlp, dtype):
    """The stream after the layer is compared too, so a fault cannot hide behind the final norm.  The width lets the bfloat16 session take
    the tensor-core products (gated in their epilogue, and grouped by expert)."""
    cfg = config([wkv_layer(heads=2, dim=4, mlp=mlp)], width=64, vocab=50)
    W = random_weights(cfg, seed=9)
    toks = tokens(cfg, 35)
    want, stream = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, max_chunk=32, keep_layers=True, n_slots=2)
    got = s.feed("a", toks[:32], range(32))
    if mlp is None or mlp["kind"] == "dense" or dtype == "float32":
        assert rel(s.layer_streams(32, "all")[0], stream[0][:32]) < tol(dtype)
        assert rel(got, want[:32]) < tol(dtype)
    else:      # a close call between two experts may fall the other way when the router's input is rounded
        err = np.max(np.abs(got - want[:32]), axis=1) / np.max(np.abs(want))
        assert np.median(err) < tol(dtype) and np.mean(err < tol(dtype)) > 0.9
    assert rel(decode(s, "d", toks), want) < TOL
    close(s)


def test_router_chooses_by_the_corrected_score_and_weighs_by_the_plain_one(cuda_backend, monkeypatch):
    """Corrections as large as the scores; restatements that weigh by the corrected score, choose by the plain one, or renormalise are far away."""
    cfg = config([wkv_layer(heads=1, dim=4, mlp=moe(experts=7, top=3, ff=8, scale=1.3))], width=24, vocab=40)
    W = random_weights(cfg, seed=31)
    W["l0.mlp.correction"] *= np.float32(4.0)
    toks = tokens(cfg, 30)
    want, _ = forward(cfg, W, toks)

    def other(weigh, choose, norm):
        def route(h, p, pre, r):
            s = ref.sigmoid(h @ p[pre + "router"].T)
            corrected = s + p[pre + "correction"]
            chosen = np.argsort(-(corrected if choose else s), axis=1, kind="stable")[:, :r["top"]]
            w = np.take_along_axis(corrected if weigh else s, chosen, 1)
            return chosen, (w / w.sum(1, keepdims=True) if norm else w) * r["scale"]
        return route

    for kind in ((True, True, False), (False, False, False), (False, True, True)):
        with monkeypatch.context() as mp:
            mp.setattr(ref, "route", other(*kind))
            assert rel(forward(cfg, W, toks)[0], want) > 100 * TOL
    s = open_model(cuda_backend, cfg, W, max_chunk=32, n_slots=2)
    assert rel(s.feed("a", toks, range(30)), want) < TOL
    assert rel(decode(s, "d", toks), want) < TOL
    close(s)


# ── embedding, streams and head ──
@pytest.mark.parametrize("streams", [1, 2, 4, 5, 16])
def test_streams_and_head(cuda_backend, streams):
    """Every number of streams the step holds (with kernels of their own up to four), a width that is no multiple of four, no cap, plain
    multipliers; a model without layers is the embedding's norm and the head."""
    for width, softcap, mult, logit_scale in ((40, 3.0, 0.7, 0.5), (37, None, 1.0, 1.0)):
        for layers in ([wkv_layer(heads=2, dim=4, mlp=dense(ff=9)), latent_layer(mlp=dense(ff=9))], []):
            cfg = config(layers, width=width, streams=streams, softcap=softcap, mult=mult, logit_scale=logit_scale)
            W = random_weights(cfg, seed=streams)
            toks = tokens(cfg, 23)
            want, stream = forward(cfg, W, toks)
            s = open_model(cuda_backend, cfg, W, keep_layers=True, n_slots=2)
            assert rel(s.feed("a", toks, range(23)), want) < TOL
            for i in range(len(layers)):
                assert rel(s.layer_streams(16, "all")[i], stream[i][:16]) < TOL
            assert rel(decode(s, "d", toks, 5), want) < TOL
            close(s)


# ── mistakes that must show ──
def _no_bonus(r, k, v, w, u, plain=ref.wkv_rule):
    return plain(r, k, v, w, 0.0 * u)


def _read_after_write(r, k, v, w, u):
    T, H, N = k.shape
    S, out = np.zeros((H, N, v.shape[2])), np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = w[t, h][:, None] * S[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ r[t, h]
    return out


def _decay_before_read(r, k, v, w, u, plain=ref.wkv_rule):
    T, H, N = k.shape
    S, out = np.zeros((H, N, v.shape[2])), np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            kv = np.outer(k[t, h], v[t, h])
            S[h] = w[t, h][:, None] * S[h]
            out[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = S[h] + kv
    return out


MISTAKES = {
    "no bonus": ("wkv_rule", _no_bonus), "read after write": ("wkv_rule", _read_after_write), "decay before read": ("wkv_rule", _decay_before_read),
    "no shift": ("shifted", lambda h: h), "first token shifted against itself": ("shifted", lambda h: np.concatenate([h[:1], h[:-1]])),
    "transposed mix": ("write_streams", lambda X, mix, w, y, plain=ref.write_streams: plain(X, np.asarray(mix).T, w, y)),
    "new streams from new ones": ("read_streams", lambda X, w: X.mean(0)),
    "no magnitude": ("rotary_frequencies", lambda rot, plain=ref.rotary_frequencies: (plain(rot)[0], 1.0)),
    "no ramp": ("rotary_frequencies", lambda rot, plain=ref.rotary_frequencies: (plain({k: rot[k] for k in ("base", "dims")})[0], plain(rot)[1])),
    "interleaved pairs": ("rotate", lambda v, pos, f, mag, plain=ref.rotate: _interleaved(v, pos, f, mag)),
    "no cap": ("logits_of", lambda z, cfg: z * cfg["logit_scale"]),
    "relu for gelu": ("gelu_tanh", lambda z: np.maximum(z, 0.0)),
}


def _interleaved(v, pos, f, mag):
    out = np.array(v)
    c, s = mag * np.cos(pos * f), mag * np.sin(pos * f)
    out[..., 0::2], out[..., 1::2] = v[..., 0::2] * c - v[..., 1::2] * s, v[..., 1::2] * c + v[..., 0::2] * s
    return out


def test_the_test_model_shows_mistakes(cuda_backend, monkeypatch):
    """Every planted mistake moves the restatement's logits by far more than the tolerance the device meets."""
    W = random_weights(MIXED, seed=41, qk_gain=3.0)
    toks = tokens(MIXED, 40)
    want, _ = forward(MIXED, W, toks)
    for what, (name, fn) in MISTAKES.items():
        with monkeypatch.context() as mp:
            mp.setattr(ref, name, fn)
            assert rel(forward(MIXED, W, toks)[0], want) > 30 * TOL, what
    s = open_model(cuda_backend, MIXED, W, max_chunk=32)
    assert rel(s.feed("a", toks, range(40)), want) < TOL
    close(s)


# ── stacks ──
def test_layer_streams_of_a_looped_stack(cuda_backend):
    """Passes of a loop share weights and keep caches and states of their own; nothing else happens between them."""
    for loop in ((1, 4, 2), (0, 6, 2), (5, 6, 3), (2, 3, 4), (2, 2, 3), (0, 2, 1), None):
        cfg = dict(MIXED)
        cfg.pop("loop")
        if loop:
            cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
        W = random_weights(cfg, seed=2)
        toks = tokens(cfg, 24)
        want, stream = forward(cfg, W, toks)
        s = open_model(cuda_backend, cfg, W, keep_layers=True)
        got = np.concatenate([s.feed("a", toks[:16], range(16)), decode(s, "a", toks[16:])])
        layers = s.layer_streams(16, "all")
        assert len(layers) == len(stream)
        for i in range(len(layers)):
            assert rel(layers[i], stream[i][:16]) < TOL, f"run {i}"
        assert rel(got, want) < TOL
        close(s)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_prefill_equals_token_by_token(cuda_backend, dtype):
    W = random_weights(MIXED, seed=3, qk_gain=3.0)
    toks = tokens(MIXED, 40)
    want, _ = forward(MIXED, W, toks)
    s = open_model(cuda_backend, MIXED, W, dtype, n_slots=2)
    assert rel(s.feed("whole", toks, range(40)), want) < tol(dtype)
    assert rel(decode(s, "single", toks), want) < TOL
    close(s)


@pytest.mark.parametrize("cuts", [[2] * 20, [1, 2, 3, 5, 7, 9, 13], [37, 2, 1], [16, 16, 8], [3, 37]], ids=["twos", "growing", "long-then-short", "menu", "short-then-long"])
def test_portions(cuda_backend, cuts):
    """However a prompt is cut the logits stay the same: the shifted row and the matrix states carry over."""
    W = random_weights(MIXED, seed=4, qk_gain=3.0)
    toks = tokens(MIXED, 40)
    want, _ = forward(MIXED, W, toks)
    s = open_model(cuda_backend, MIXED, W, max_chunk=32)
    got, at = [], 0
    for n in cuts:
        got.append(s.feed("a", toks[at:at + n], range(n)))
        at += n
    assert at == 40 and rel(np.concatenate(got), want) < TOL
    close(s)


def test_first_tokens(cuda_backend):
    """Position 0 alone (zeros before it in the shift, an empty state, one visible key beside the sink), then positions 1 and 2 one by one;
    then the three as one step in a slot that was used before."""
    W = random_weights(MIXED, seed=6)
    toks = tokens(MIXED, 3)
    want, _ = forward(MIXED, W, toks)
    s = open_model(cuda_backend, MIXED, W)
    assert rel(decode(s, "a", toks), want) < TOL
    s.release("a")
    assert rel(s.feed("b", toks, [0, 1, 2]), want) < TOL
    close(s)


def test_interleaved_requests_and_slot_reuse(cuda_backend):
    W = random_weights(MIXED, seed=7, qk_gain=2.0)
    reqs = {"a": tokens(MIXED, 29, 1), "b": tokens(MIXED, 11, 2), "c": tokens(MIXED, 40, 3)}
    want = {k: forward(MIXED, W, v)[0] for k, v in reqs.items()}
    s = open_model(cuda_backend, MIXED, W, n_slots=2)
    got = {k: [] for k in reqs}
    # a and b advance in turns, in unequal portions, inside ONE step call each time
    plan = [(("a", 9), ("b", 2)), (("b", 5), ("a", 1)), (("a", 19), ("b", 4))]
    at = {k: 0 for k in reqs}
    for step in plan:
        entries = [{"id": k, "tokens": reqs[k][at[k]:at[k] + n], "want": list(range(n))} for k, n in step]
        for (k, n), rows in zip(step, s.step(entries, end=["a", "b"] if step is plan[-1] else [])):
            got[k].append(rows)
            at[k] += n
    for k in "ab":
        assert rel(np.concatenate(got[k]), want[k]) < TOL, k
    # c takes a slot that held another sequence: nothing of it may leak (matrix states and shifted rows are cleared, cached latents
    # are masked by position)
    assert not s.pool.live()
    assert rel(s.feed("c", reqs["c"], range(40)), want["c"]) < TOL
    close(s)


# ── what a query must and must not see ──
def test_causality(cuda_backend):
    """Changing a token changes nothing before it, bit for bit, and everything from it on — in a prompt and decoded."""
    W = random_weights(MIXED, seed=28, qk_gain=2.0)
    toks = tokens(MIXED, 30)
    for at in (0, 7, 15, 16, 29):
        other = list(toks)
        other[at] = (other[at] + 1) % MIXED["vocab"]
        s = open_model(cuda_backend, MIXED, W, n_slots=2, max_chunk=32)
        for run in (lambda n, t: s.feed(n, t, range(30)), lambda n, t: decode(s, n, t, 16)):
            moved = np.abs(run("a", toks) - run("b", other)).max(axis=1) > 0.0
            assert not moved[:at].any() and moved[at:].all()
            s.release("a")
            s.release("b")
        close(s)


def test_visible_keys_with_controls_off_by_one(cuda_backend, monkeypatch):
    """Sharp attention: a restatement that misses the query's own key, or the sequence's first key from some position on, is far away."""
    cfg = config([latent_layer(heads=2, dim=8, rot_dim=4, vdim=8)], width=32, vocab=40)
    W = random_weights(cfg, seed=8, qk_gain=6.0)
    W["l0.mix.sink"][:] = 0.0
    toks = tokens(cfg, 48)
    want, _ = forward(cfg, W, toks)
    with monkeypatch.context() as mp:
        mp.setattr(ref, "visible", lambda i: max(1, i))
        assert rel(forward(cfg, W, toks)[0], want) > 30 * TOL
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=32)
    assert rel(s.feed("p", toks, range(48)), want) < TOL
    assert rel(decode(s, "d", toks, 9), want) < TOL
    close(s)


def test_sink(cuda_backend):
    """Sinks that weigh about as much as the keys: a restatement without them is far away, the device is not.  One head's sink is
    very negative (it weighs nothing), another's dominates."""
    cfg = config([latent_layer(heads=3, dim=8, rot_dim=4, vdim=8)], width=32, vocab=40)
    W = random_weights(cfg, seed=11, qk_gain=2.0)
    W["l0.mix.sink"][:] = np.array([-30.0, 1.0, 6.0], np.float32)
    toks = tokens(cfg, 20)
    want, _ = forward(cfg, W, toks)
    Wn = dict(W)
    Wn["l0.mix.sink"] = np.full(3, -1e4, np.float32)
    assert np.abs(forward(cfg, Wn, toks)[0] - want).max() > 2e-2 * np.abs(want).max()
    s = open_model(cuda_backend, cfg, W, n_slots=2)
    assert rel(s.feed("p", toks, range(20)), want) < TOL
    assert rel(decode(s, "d", toks), want) < TOL
    close(s)


def _embedded(cfg, p, name):
    """Input of layer 0's mixer for every token of the vocabulary (all streams still equal)."""
    u = ref.embedding(cfg, p, range(cfg["vocab"])) * np.asarray(p[name + "hc1.in"]).sum()
    return ref.dynamic_tanh(u, p, name + "norm1")


@pytest.mark.parametrize("part", ["unrotated", "rotated"])
def test_far_key_among_hundreds(cuda_backend, part):
    """The last query is made to weigh one early key among 300 and hardly any other, through the unrotated or through the rotated part of the
    keys: the other part of the queries is silenced, the pair of tokens whose score stands out is found from the weights (at its distance),
    and the queries are scaled up.  Changing the far token must move the restatement's last logits, and the device must agree with the
    restatement, in a prompt and with the last tokens decoded."""
    n, far = 300, 4
    layer = latent_layer(heads=1, dim=16, rot_dim=16, vdim=8, kv_rank=20)
    m = layer["mixer"]
    cfg = config([layer], width=32, vocab=30)
    W = random_weights(cfg, seed=12)
    W["l0.mix.sink"][:] = 0.0
    W["l0.mix.q"][:16 if part == "rotated" else 32][(0 if part == "rotated" else 16):] = 0.0
    p = as_f64(W)
    x = _embedded(cfg, p, "l0.")
    q, z = x @ p["l0.mix.q"].T, x @ p["l0.mix.dkv"].T
    if part == "unrotated":
        S = q[:, :16] @ (ref.rms_unit(z[:, :20], 1e-5) * p["l0.mix.dkv.norm"] @ p["l0.mix.uk"].T).T * m["scale"]
    else:      # all keys at the far position: what decides below is only that ONE token stands out there
        f, mag = ref.rotary_frequencies(m["rot"])
        S = ref.rotate(q[:, 16:], n - 1, f, mag) @ ref.rotate(z[:, 20:], far, f, mag).T * m["scale"]
    two = np.sort(S, axis=1)[:, -2:]
    a_tok = int(np.argmax(two[:, 1] - two[:, 0]))
    b_tok, lead = int(np.argmax(S[a_tok])), float((two[:, 1] - two[:, 0]).max())
    pool = [t for t in range(cfg["vocab"]) if t != b_tok]
    if part == "rotated":      # at other positions other tokens may score higher: keep fillers that stay behind everywhere
        k_all = np.stack([ref.rotate(z[:, 20:], t, f, mag) for t in range(n)])                     # [position, token, 16]
        best = (k_all @ ref.rotate(q[a_tok, 16:], n - 1, f, mag) * m["scale"]).max(0)
        pool = [t for t in pool if t != a_tok and best[t] < S[a_tok, b_tok]]
        assert len(pool) >= 3
        lead = float(S[a_tok, b_tok] - max(best[t] for t in pool + [a_tok]))
        if lead < 0.05:
            lead = 0.05
    W["l0.mix.q"] *= np.float32(2.0 ** np.ceil(np.log2(12.0 / lead)))
    toks = [pool[i] for i in np.random.default_rng(1).integers(0, len(pool), n)]
    toks[far], toks[-1] = b_tok, a_tok
    want, _ = forward(cfg, W, toks)
    moved = list(toks)
    moved[far] = pool[0]
    assert np.abs(forward(cfg, W, moved)[0][-1] - want[-1]).max() > 2e-2 * np.abs(want).max(), "the construction lost its far key"
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=64)
    bound = 10 * TOL if part == "rotated" else TOL          # scores of hundreds: their rounding shows
    assert rel(s.feed("p", toks, range(n)), want) < bound
    s.feed("d", toks[:n - 5], [])
    assert rel(decode(s, "d", toks[n - 5:]), want[n - 5:]) < bound
    close(s)


def test_far_write_in_the_state(cuda_backend):
    """A token hundreds of positions back is read from the matrix state: its key is scaled up and nothing decays.  Changing it moves the last
    logits of the restatement, and the device agrees, with the state carried over portions and single tokens."""
    cfg = config([wkv_layer(heads=2, dim=8)], width=32, vocab=30)
    W = random_weights(cfg, seed=22)
    W["l0.mix.w0"][:] = -30.0
    W["l0.mix.mu.k"][:] = 0.0
    toks = [t % 29 for t in tokens(cfg, 320)]
    toks[6] = 29
    p = as_f64(W)
    x = _embedded(cfg, p, "l0.")
    W["l0.mix.k"] -= np.outer(W["l0.mix.k"] @ x[:29].mean(0), x[:29].mean(0)).astype(np.float32) / np.float32((x[:29].mean(0) ** 2).sum())
    from fomanex_models import bf16_exact
    W["l0.mix.k"] = bf16_exact(W["l0.mix.k"])
    want, _ = forward(cfg, W, toks)
    moved = list(toks)
    moved[6] = 0
    assert rel(forward(cfg, W, moved)[0][-1], want[-1]) > 20 * TOL, "the construction lost its far write"
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=64)
    assert rel(s.feed("p", toks, range(320)), want) < TOL
    s.feed("d", toks[:37], [])
    got, at = [], 37
    for k in (2, 64, 5, 128, 70):
        got.append(s.feed("d", toks[at:at + k], range(k)))
        at += k
    assert rel(np.concatenate(got + [decode(s, "d", toks[at:])]), want[37:]) < TOL
    close(s)


@pytest.mark.parametrize("layer", [latent_layer(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32), latent_layer(heads=8, dim=4, rot_dim=4, vdim=4, kv_rank=8), latent_layer(heads=2, dim=88, rot_dim=8, vdim=72, kv_rank=96),
                                   latent_layer(heads=20, dim=12, rot_dim=8, vdim=8, kv_rank=64)], ids=["16", "narrow", "88", "20heads"])
def test_many_keys_and_split_decoding(cuda_backend, layer):
    """Caches beyond one key tile of the prompt kernel (64) and one share of the decoding kernel (32): single-token steps deal their keys to
    several CTAs whose shares are merged, with the sink."""
    cfg = config([layer], width=48, vocab=50)
    W = random_weights(cfg, seed=18, qk_gain=3.0)
    n = 300
    toks = tokens(cfg, n)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=128)
    assert rel(s.feed("p", toks, range(n)), want) < TOL
    s.feed("d", toks[:n - 12], [])
    assert rel(np.concatenate([decode(s, "d", toks[n - 12:n - 4]), s.feed("d", toks[n - 4:], range(4))]), want[n - 12:]) < TOL
    close(s)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_expanded_form_of_long_steps(cuda_backend, dtype):
    """Steps of 128 tokens and more expand the latents to keys and values per head — only the rows the sequence holds, from the second slot
    of the cache, after earlier steps in the absorbed form — and later steps go on absorbed over the same cache."""
    cfg = config([latent_layer(heads=3, dim=24, rot_dim=16, vdim=20, kv_rank=64, mlp=dense()), latent_layer(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=56)], width=64, vocab=50)
    W = random_weights(cfg, seed=25, qk_gain=2.0)
    n = 420
    toks = tokens(cfg, n)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, n_slots=2, max_chunk=256)
    s.model.expand_float32 = True
    s.feed("first", toks[:5], [])                           # takes slot 0 and keeps it
    got = np.concatenate([s.feed("a", toks[:50], range(50)), s.feed("a", toks[50:306], range(256)), s.feed("a", toks[306:434], range(114))])     # 32 + 16 + 2, 256, 64 + 32 + 16 + 2
    assert s.pool.slot("a") == 1
    assert rel(got, want) < (TOL if dtype == "float32" else 5e-2)
    s.release("a")
    got = np.concatenate([s.feed("b", toks[:400], range(400)), decode(s, "b", toks[400:])])      # 256 + 128 + 16
    assert rel(got, want) < (TOL if dtype == "float32" else 5e-2)
    from zgml_b200 import abi
    tags = [(op.tag, op.u.seq.n[11]) for op in s.model.lower(256, "last", s.pool).program.ops]
    assert tags.count((abi.OP_LINEAR, 256)) == 2            # both layers expanded
    close(s)


def test_long_steps_into_single_tokens(cuda_backend):
    """Steps of 256 tokens take the prepared walk of the state; what they leave must carry on into smaller steps and single tokens, in a slot
    that is not the first, after a request that used the same slot before."""
    cfg = config([wkv_layer(heads=3, dim=20, mlp=dense()), wkv_layer(heads=2, dim=36, rank=8), latent_layer()], width=48, vocab=50, loop=(0, 2, 2))
    W = random_weights(cfg, seed=23)
    n = 400
    toks = tokens(cfg, n)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=256)
    s.feed("first", toks[:5], [])                           # takes slot 0 and keeps it
    s.feed("other", toks[100:400], [])                      # leaves its states in slot 1
    s.release("other")
    got = np.concatenate([s.feed("a", toks[:370], range(370)), decode(s, "a", toks[370:])])   # 256 + 64 + 32 + 16 + 2, then single tokens
    assert s.pool.slot("a") == 1
    assert rel(got, want) < TOL
    close(s)


def test_long_decoding(cuda_backend):
    """150 decoded tokens through every kind of state."""
    cfg = config([latent_layer(mlp=dense()), wkv_layer(mlp=moe()), wkv_layer(heads=1, dim=7)], loop=(0, 2, 2))
    W = random_weights(cfg, seed=13, qk_gain=3.0)
    toks = tokens(cfg, 160)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, max_chunk=4, max_context=160)
    assert rel(decode(s, "a", toks, 10), want) < TOL
    close(s)


# ── shapes ──
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_wider_model(cuda_backend, dtype):
    """Sizes at which the bfloat16 session takes the tensor-core matmuls (widths multiples of 64, steps of 64 tokens): gated pairs whose rows end
    inside a tile, the batched projections with their narrower last head, grouped experts."""
    cfg = config([wkv_layer(heads=4, dim=40, rank=24, mlp=dense(ff=250)), latent_layer(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, mlp=dense(ff=192)), wkv_layer(heads=2, dim=64, rank=72)], width=128, vocab=200)
    W = random_weights(cfg, seed=15)
    toks = tokens(cfg, 100)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, max_chunk=64)
    got = s.feed("a", toks, range(100))
    if dtype == "float32":
        assert rel(got, want) < TOL
    else:      # inputs rounded to bfloat16 in every product of three layers: the bulk of the positions bounds the error
        assert cuda_backend.program_stats(s.program(64, "all")[1])["tensor_core_linears"] >= 9
        err = np.max(np.abs(got - want), axis=1) / np.max(np.abs(want))
        assert np.median(err) < 3e-2 and np.mean(err < 6e-2) > 0.9
    close(s)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_odd_sizes(cuda_backend, dtype):
    """Nothing is a multiple of 4: the unaligned forms of every kernel (scalar loads, one warp per query, exact matmuls)."""
    cfg = config([latent_layer(heads=3, dim=5, rot_dim=2, vdim=7, kv_rank=9, mlp=dense(ff=13)), wkv_layer(heads=3, dim=5, rank=3, mlp=moe(experts=3, top=1, ff=5)), latent_layer(heads=1, dim=7, rot_dim=6, vdim=3, kv_rank=5)],
                 width=37, vocab=53, streams=3, loop=(0, 3, 2))
    W = random_weights(cfg, seed=19, qk_gain=2.0)
    toks = tokens(cfg, 41)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, max_chunk=32)
    assert rel(decode(s, "a", toks, 35), want) < tol(dtype)
    close(s)


def test_context_bound(cuda_backend):
    """Latent layers keep every position: the caches hold what the caller asks for and a step past it is refused; the last position works, in
    every slot.  A model of time mixing alone has no bound."""
    cfg = config([wkv_layer(), latent_layer()])
    W = random_weights(cfg, seed=1)
    toks = tokens(cfg, 24)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=8, max_context=24)
    assert s.context_limit == 24
    for name in "ab":
        assert rel(s.feed(name, toks, range(24)), want) < TOL
        with pytest.raises(ValueError):
            s.feed(name, [0], [0])
    close(s)
    cfg = config([wkv_layer()])
    s = open_model(cuda_backend, cfg, random_weights(cfg), max_chunk=8, max_context=8)
    assert s.context_limit is None
    close(s)


# ── the entry points ──
def _write_model(tmp_path, cfg, W):
    from zgml_b200.host.safetensors import write_safetensors
    d = os.path.join(tmp_path, "model")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), W)
    return d


def test_greedy_generation_through_the_registry(cuda_backend, tmp_path):
    from zgml_b200.host.registry import open_session
    W = random_weights(MIXED, seed=16)
    d = _write_model(tmp_path, MIXED, W)
    prompt = tokens(MIXED, 9)
    want, seq = [], list(prompt)
    for _ in range(12):
        want.append(int(np.argmax(ref.forward(MIXED, as_f64(W), seq)[-1])))
        seq.append(want[-1])
    s = open_session(cuda_backend, d, "float32", n_slots=1, max_chunk=8, max_tokens=32)
    assert s.generate(prompt, 12) == want
    assert not s.pool.live()
    close(s)


def test_trace_replay_from_the_command_line(tmp_path):
    W = random_weights(MIXED, seed=17)
    d = _write_model(tmp_path, MIXED, W)
    toks = tokens(MIXED, 30)
    want, _ = forward(MIXED, W, toks)
    steps = [{"step": 0, "entries": [{"id": "r", "tokens": toks[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "r", "tokens": toks[17:19], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "r", "tokens": toks[19:], "want": [10]}], "end": ["r"]}]
    out = os.path.join(tmp_path, "out")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", out, "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(os.path.join(out, "1.f32"))
    got0 = np.fromfile(os.path.join(out, "0.f32"), dtype="<f4").reshape(2, -1)
    got2 = np.fromfile(os.path.join(out, "2.f32"), dtype="<f4").reshape(1, -1)
    assert rel(got0, want[[0, 16]]) < TOL and rel(got2, want[[29]]) < TOL
