"""Fotovik on the CUDA backend against the float64 restatement (tests/fotovik_reference.py): every mechanism alone, the stream
after every layer run, whole prompts, token-by-token decoding through the rings, pooled blocks and recurrent states, prompts cut
into portions down to two tokens, interleaved requests in several slots, slot reuse, the edges of the window and of the pooled
blocks in prompts and decoded (with controls that are off by one), sinks, far keys found by construction, the first tokens of a
sequence, long decoding over rings that wrap, many shapes, and greedy generation through the registry's entry point and the
trace replayer."""
import json
import os
import subprocess

import numpy as np
import pytest

import fotovik_reference as ref
from fotovik_models import as_f64, attention_layer, config, delta_layer, dense, pair_layer, random_weights

pytestmark = pytest.mark.gpu

TOL = 2e-4   # of the logits' scale; f32 accumulation against float64


def tol(dtype):
    """A bfloat16 session rounds the activations that enter a tensor-core matmul (steps of more than 8 tokens) to bf16."""
    return TOL if dtype == "float32" else 3e-2


def open_model(be, cfg, W, dtype="float32", n_slots=1, max_chunk=16, keep_layers=False, max_context=512):
    from zgml_b200.host.fotovik import FotovikConfig, FotovikModel
    from zgml_b200.host.session import SequenceSession
    model = FotovikModel(be, FotovikConfig.from_dict(cfg), lambda n: W[n], dtype)
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
MIXED = config([delta_layer(heads=2, kv_heads=1, dim=5, vdim=7, conv=2, mlp=dense(ff=9)), pair_layer(mlp=dense()), attention_layer(mlp=dense(ff=24)), delta_layer(mlp=dense()),
                attention_layer(heads=3, kv_heads=3, dim=6, vdim=4, rot_dims=2, size=5, pool=2), pair_layer(heads=3, kv_heads=1, dim=6, vdim=4, rot_dims=4, factor=None, r_heads=1, r_dim=5, r_vdim=3,
                                                                                                           mlp=dense(ff=12))], loop=(1, 4, 2))


# ── each mechanism alone (a one-layer model without a feed-forward isolates its mixer) ──
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("layer", [
    attention_layer(),
    attention_layer(heads=1, kv_heads=1, dim=16, vdim=4, rot_dims=16, size=40, pool=7),           # one head, every dimension turns, a block that does not divide the window
    attention_layer(heads=5, kv_heads=1, dim=6, vdim=7, rot_dims=2, size=1, pool=1),              # a window of the token itself; blocks of one token: everything is seen
    attention_layer(heads=6, kv_heads=2, dim=12, vdim=12, rot_dims=8, size=3, pool=16, scale=0.7),     # a block longer than the window: most tokens are out of sight for a while
    attention_layer(heads=4, kv_heads=4, dim=68, vdim=36, rot_dims=64, size=33, pool=8),
    attention_layer(heads=2, kv_heads=1, dim=8, vdim=8, size=70, pool=5),                          # the window outlasts most of the request
    delta_layer(),
    delta_layer(heads=6, kv_heads=2, dim=10, vdim=5, conv=1),                                     # three heads per key head, one tap: no carried inputs
    delta_layer(heads=1, kv_heads=1, dim=36, vdim=68, conv=6),
    delta_layer(heads=3, kv_heads=3, dim=130, vdim=20, conv=2),
    pair_layer(),
    pair_layer(heads=6, kv_heads=2, dim=10, vdim=5, rot_dims=10, factor=1.0, r_heads=1, r_dim=4, r_vdim=4, decay=[1.0]),      # no decay at all
    pair_layer(heads=1, kv_heads=1, dim=36, vdim=68, rot_dims=20, base=10000.0, factor=8.0, r_heads=2, r_dim=40, r_vdim=36, decay=[0.2, 0.999]),
    pair_layer(heads=4, kv_heads=4, dim=8, vdim=8, rot_dims=8, factor=None, r_heads=5, r_dim=16, r_vdim=20, scale=0.9),
    pair_layer(heads=2, kv_heads=1, dim=8, vdim=8, r_heads=2, r_dim=150, r_vdim=6),
], ids=["attention", "attention-1head", "attention-window1-pool1", "attention-long-block", "attention-wide", "attention-long-window", "delta", "delta-grouped-1tap", "delta-wide",
        "delta-130", "pair", "pair-no-decay", "pair-wide", "pair-mha", "pair-150"])
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


@pytest.mark.parametrize("silent", ["left", "right"])
def test_branches_of_the_pair_alone(cuda_backend, silent):
    """With one branch's closing weight at zero the layer is the other branch alone; prompt and token by token."""
    cfg = config([pair_layer()], width=32, vocab=40)
    W = random_weights(cfg, seed=21, qk_gain=2.0)
    W[f"l0.mix.{silent}.out"][:] = 0.0
    toks = tokens(cfg, 30)
    want, stream = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, max_chunk=32, keep_layers=True, n_slots=2)
    assert rel(s.feed("a", toks, range(30)), want) < TOL
    assert rel(s.layer_streams(16, "all")[0], stream[0][:16]) < TOL
    assert rel(decode(s, "d", toks), want) < TOL
    close(s)


@pytest.mark.parametrize("mlp", [dense(), dense(ff=7), dense(ff=300), None], ids=["dense", "dense-7", "dense-300", "none"])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_feed_forward(cuda_backend, mlp, dtype):
    """The stream after the layer is compared too, so a fault in the activation cannot hide behind the final norm.  The width lets the
    bfloat16 session take the tensor-core product with the activation in its epilogue; inputs reach where the exact and the tanh
    form of the activation differ."""
    cfg = config([delta_layer(heads=2, kv_heads=1, dim=4, vdim=4, conv=2, mlp=mlp)], width=64, vocab=50)
    W = random_weights(cfg, seed=9)
    toks = tokens(cfg, 19)
    want, stream = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, max_chunk=32, keep_layers=True)
    got = s.feed("a", toks[:16], range(16))
    assert rel(s.layer_streams(16, "all")[0], stream[0][:16]) < tol(dtype)
    assert rel(got, want[:16]) < tol(dtype)
    close(s)


# ── embedding ──
def test_bigram_embedding(cuda_backend):
    """The first token's own row, rows of every later pair of tokens, a pair that straddles two steps, and a slot whose last sequence
    ended on another token; factors beyond the number of buckets; a model without the table."""
    for bigram in ((37, 11, 5), (1, 3, 2), (53, 1000003, 40), None):
        cfg = config([], bigram=bigram, scale=0.3)
        W = random_weights(cfg, seed=2)
        toks = tokens(cfg, 23)
        want = ref.forward(cfg, as_f64(W), toks)
        s = open_model(cuda_backend, cfg, W)
        assert rel(s.feed("a", toks, range(23)), want) < TOL
        s.release("a")
        assert rel(np.concatenate([s.feed("b", toks[:3], range(3)), s.feed("b", toks[3:5], range(2)), decode(s, "b", toks[5:])]), want) < TOL
        if bigram and bigram[0] > 1:
            assert rel(ref.forward(config([], scale=0.3, bigram=None), as_f64(W), toks), want) > 0.1     # the table is no small part of the stream
        close(s)


# ── stacks ──
def test_layer_streams_of_a_looped_stack(cuda_backend):
    """Passes of a loop share weights and keep caches and states of their own; the embedding output joins the stream again before
    every pass but the first."""
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
    """However a prompt is cut — inside a window, inside a pooled block, inside a convolution's reach, two tokens at a time — the
    logits stay the same."""
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
    """Position 0 alone (zeros before the convolutions' start, empty states, one visible key beside the sink, the bigram row of a
    first token), then positions 1 and 2 one by one; then the three as one step in a slot that was used before."""
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
    # c takes a slot that held another sequence: nothing of it may leak (recurrent states and convolution inputs are cleared,
    # rings and pooled blocks are masked by position)
    assert not s.pool.live()
    assert rel(s.feed("c", reqs["c"], range(40)), want["c"]) < TOL
    close(s)


# ── what a query must and must not see ──
def _edges(cuda_backend, cfg, W, toks, want, controls, monkeypatch):
    """The device agrees with the restatement at every position, as a prompt and decoded, and every control (a restatement whose
    `visible` is off by one) agrees up to the first position whose keys differ and is far away from there on."""
    for first, visible in controls:
        with monkeypatch.context() as mp:
            mp.setattr(ref, "visible", visible)
            control = ref.forward(cfg, as_f64(W), toks)
        assert np.abs(control[:first] - want[:first]).max() < 1e-9
        assert np.abs(control[first] - want[first]).max() > 5 * TOL * np.abs(want).max()
        assert np.abs(control[first:] - want[first:]).max() > 30 * TOL * np.abs(want).max()
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=32)
    assert rel(s.feed("p", toks, range(len(toks))), want) < TOL
    assert rel(decode(s, "d", toks, 9), want) < TOL
    close(s)


@pytest.mark.parametrize("size,pool", [(11, 4), (6, 6), (7, 1), (4, 9)])
def test_edges_of_window_and_blocks(cuda_backend, monkeypatch, size, pool):
    """Sharp attention weights: a window that is one token longer or shorter, or a block that is seen one token early or late, shows."""
    cfg = config([attention_layer(heads=2, kv_heads=1, dim=8, vdim=8, size=size, pool=pool)], width=32, vocab=40)
    W = random_weights(cfg, seed=8, qk_gain=6.0)
    W["l0.mix.sink"][:] = 0.0
    toks = tokens(cfg, 48)
    want, _ = forward(cfg, W, toks)
    plain = ref.visible

    def window(delta):         # the blocks stay where they are
        return lambda i, w, p: (plain(i, w + delta, p)[0], plain(i, w, p)[1])

    def blocks(delta):         # a block is seen delta tokens late
        return lambda i, w, p: (plain(i, w, p)[0], max(0, (i - delta - w + 1) // p))

    _edges(cuda_backend, cfg, W, toks, want, [(size, window(1)), (size - 1, window(-1)), (size + pool - 2, blocks(-1)), (size + pool - 1, blocks(1))], monkeypatch)


def test_last_token_before_the_window_waits_for_its_block(cuda_backend):
    """Changing a token that has left the window changes nothing while its block is not complete before the window, and does from the
    position on at which the block is seen — on the device, as a prompt and decoded."""
    size, pool = 6, 8
    cfg = config([attention_layer(heads=2, kv_heads=1, dim=8, vdim=8, size=size, pool=pool)], width=32, vocab=40, bigram=None)
    W = random_weights(cfg, seed=28, qk_gain=3.0)
    toks = tokens(cfg, 30)
    other = list(toks)
    other[3] = (other[3] + 1) % cfg["vocab"]
    s = open_model(cuda_backend, cfg, W, n_slots=4, max_chunk=32)
    for run in (lambda n, t: s.feed(n, t, range(30)), lambda n, t: decode(s, n, t)):
        a, b = run("a", toks), run("b", other)
        moved = np.abs(a - b).max(axis=1) > 0.0
        assert moved[3:9].all() and not moved[:3].any()            # positions 3 .. 8: inside the window
        assert not moved[9:13].any()                                # left the window (from 9), block 0 .. 7 not yet seen (until 13 - 6 = 7)
        assert moved[13:].all()
        s.release("a")
        s.release("b")
    close(s)


def test_sink(cuda_backend):
    """Sinks that weigh about as much as the keys: a restatement without them is far away, the device is not.  One head's sink is
    very negative (it weighs nothing), another's dominates."""
    cfg = config([attention_layer(heads=3, kv_heads=1, dim=8, vdim=8, size=6, pool=3)], width=32, vocab=40)
    W = random_weights(cfg, seed=11, qk_gain=2.0)
    W["l0.mix.sink"][:] = np.array([-30.0, 1.0, 6.0], np.float32)
    toks = tokens(cfg, 20)
    want, _ = forward(cfg, W, toks)
    Wn = dict(W)
    Wn["l0.mix.sink"] = np.full(3, -1e4, np.float32)
    assert np.abs(forward(cfg, Wn, toks)[0] - want).max() > 5e-2 * np.abs(want).max()
    s = open_model(cuda_backend, cfg, W, n_slots=2)
    assert rel(s.feed("p", toks, range(20)), want) < TOL
    assert rel(decode(s, "d", toks), want) < TOL
    close(s)


def _standing_out(S):
    """(query token, key token, lead) of the score matrix [queries, keys] whose score leads every other key of its query the most."""
    two = np.sort(S, axis=1)[:, -2:]
    a = int(np.argmax(two[:, 1] - two[:, 0]))
    return a, int(np.argmax(S[a])), float(two[a, 1] - two[a, 0])


@pytest.mark.parametrize("kind", ["pooled-block", "causal"])
def test_far_key_among_hundreds(cuda_backend, kind):
    """The last query is made to weigh one early key among 300 and hardly any other: for the window layer the mean key of a block far
    before the window (all of whose tokens are the key token), for the pair's left branch one token.  The dimensions that turn are
    silenced in the queries, so a score depends on the two tokens alone and the pair that stands out is found from the weights; the
    queries are then scaled up.  Changing the far tokens must move the restatement's last logits, and the device must agree with the
    restatement, in a prompt and with the last tokens decoded."""
    n, P = 300, 6
    layer = attention_layer(heads=1, kv_heads=1, dim=16, vdim=8, rot_dims=2, size=20, pool=P) if kind == "pooled-block" else pair_layer(heads=1, kv_heads=1, dim=16, vdim=8, rot_dims=2)
    cfg = config([layer], width=32, vocab=30, bigram=None)
    W = random_weights(cfg, seed=12)
    p = as_f64(W)
    x = ref.rms_norm(p["embed"] * cfg["embedding"]["scale"], p["l0.norm1"], cfg["norm"]["eps"])
    if kind == "pooled-block":
        W["l0.mix.q"][:2] = 0.0
        W["l0.mix.sink"][:] = 0.0
        S = (x @ as_f64(W)["l0.mix.q"].T) @ (x @ p["l0.mix.k"].T).T * layer["mixer"]["scale"]
    else:
        W["l0.mix.left.q.norm"][:2] = 0.0
        W["l0.mix.right.out"][:] = 0.0
        q = ref.rms_norm(x @ p["l0.mix.left.q"].T, as_f64(W)["l0.mix.left.q.norm"], cfg["norm"]["eps"])
        S = q @ ref.rms_norm(x @ p["l0.mix.left.k"].T, p["l0.mix.left.k.norm"], cfg["norm"]["eps"]).T * layer["mixer"]["left"]["scale"]
    a_tok, b_tok, lead = _standing_out(S)
    W["l0.mix.q" if kind == "pooled-block" else "l0.mix.left.q.norm"] *= np.float32(2.0 ** np.ceil(np.log2(12.0 / lead)))     # the far key leads by 12 or more
    pool = [t for t in range(cfg["vocab"]) if t != b_tok]
    toks = [pool[i] for i in np.random.default_rng(1).integers(0, len(pool), n)]
    far = slice(5 * P, 6 * P) if kind == "pooled-block" else slice(4, 5)
    toks[far] = [b_tok] * (far.stop - far.start)
    toks[-1] = a_tok
    want, _ = forward(cfg, W, toks)
    moved = list(toks)
    moved[far] = [pool[0]] * (far.stop - far.start)
    assert np.abs(forward(cfg, W, moved)[0][-1] - want[-1]).max() > 5e-2 * np.abs(want).max(), "the construction lost its far key"
    s = open_model(cuda_backend, cfg, W, n_slots=2, max_chunk=64)
    assert rel(s.feed("p", toks, range(n)), want) < TOL
    s.feed("d", toks[:n - 5], [])
    assert rel(decode(s, "d", toks[n - 5:]), want[n - 5:]) < TOL
    close(s)


@pytest.mark.parametrize("layer", [attention_layer(heads=4, kv_heads=1, dim=16, vdim=16, rot_dims=16, size=130, pool=2), attention_layer(heads=8, kv_heads=1, dim=4, vdim=4, rot_dims=4, size=40, pool=1),
                                   attention_layer(heads=2, kv_heads=2, dim=88, vdim=72, rot_dims=64, size=65, pool=3), attention_layer(heads=2, kv_heads=1, dim=12, vdim=264, rot_dims=8, size=10, pool=4),
                                   pair_layer(heads=8, kv_heads=2, dim=20, vdim=24, rot_dims=20)], ids=["long-window", "hundreds-of-blocks", "88", "wide-values", "causal"])
def test_many_keys_and_split_decoding(cuda_backend, layer):
    """Windows and pooled rows beyond one key tile of the prompt kernel (64) and one share of the decoding kernel (32): tiles that hold
    blocks and window tokens both, single-token steps that deal their keys to several CTAs whose shares are merged, with the sink."""
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


def test_long_steps_walk_segments_side_by_side(cuda_backend):
    """Steps of 256 tokens: the lightning state is walked in segments side by side and the delta rule takes its prepared walk; the
    states they leave must carry on into smaller steps and single tokens, in a slot that is not the first, after a request that
    used the same slot before."""
    cfg = config([pair_layer(r_heads=3, r_dim=20, r_vdim=36, decay=[0.999, 0.9, 0.5], mlp=dense()), delta_layer(heads=4, kv_heads=2, dim=20, vdim=36, mlp=dense()), attention_layer(size=30, pool=7)],
                 width=48, vocab=50, loop=(0, 2, 2))
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


def test_long_decoding_over_rings_that_wrap(cuda_backend):
    """150 decoded tokens through every kind of state: rings that wrap a dozen times under the blocks averaged from them, the matrix
    states, the convolutions' inputs."""
    cfg = config([attention_layer(mlp=dense()), delta_layer(mlp=dense()), pair_layer(), attention_layer(size=3, pool=10)], loop=(0, 2, 2))
    W = random_weights(cfg, seed=13, qk_gain=3.0)
    toks = tokens(cfg, 160)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, max_chunk=4, max_context=160)
    assert s.pool.buffers["run0.kv"].elems == (9 - 1 + 4) * 2 * (8 + 12) and s.pool.buffers["run5.kv"].elems == (10 + 4) * 2 * (8 + 12)
    assert rel(decode(s, "a", toks, 10), want) < TOL
    close(s)


# ── shapes ──
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_wider_model(cuda_backend, dtype):
    """Sizes at which the bfloat16 session takes the tensor-core matmuls (widths multiples of 64, steps of 64 tokens); the pair's
    projection has its activation on part of the columns, whose borders lie inside a tile."""
    cfg = config([attention_layer(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=32, size=48, pool=8, mlp=dense(ff=256)),
                  pair_layer(heads=4, kv_heads=2, dim=32, vdim=36, rot_dims=16, r_heads=2, r_dim=32, r_vdim=64, mlp=dense(ff=192)),
                  delta_layer(heads=4, kv_heads=2, dim=32, vdim=64, conv=4, mlp=dense(ff=128))], width=128, vocab=200)
    W = random_weights(cfg, seed=15)
    toks = tokens(cfg, 100)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, max_chunk=64)
    got = s.feed("a", toks, range(100))
    if dtype == "float32":
        assert rel(got, want) < TOL
    else:      # inputs rounded to bfloat16 in every product of three layers: the bulk of the positions bounds the error
        assert cuda_backend.program_stats(s.program(64, "all")[1])["tensor_core_linears"] > 10
        err = np.max(np.abs(got - want), axis=1) / np.max(np.abs(want))
        assert np.median(err) < 3e-2 and np.mean(err < 6e-2) > 0.9
    close(s)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_odd_sizes(cuda_backend, dtype):
    """Nothing is a multiple of 4: the unaligned forms of every kernel (scalar loads, one warp per query, exact matmuls)."""
    cfg = config([attention_layer(heads=3, kv_heads=1, dim=6, vdim=7, rot_dims=2, size=5, pool=3, mlp=dense(ff=13)), delta_layer(heads=3, kv_heads=1, dim=5, vdim=7, conv=3, mlp=dense(ff=11)),
                  pair_layer(heads=3, kv_heads=3, dim=7, vdim=5, rot_dims=2, r_heads=3, r_dim=5, r_vdim=3)], width=37, vocab=53, loop=(0, 3, 2))
    W = random_weights(cfg, seed=19, qk_gain=2.0)
    toks = tokens(cfg, 41)
    want, _ = forward(cfg, W, toks)
    s = open_model(cuda_backend, cfg, W, dtype, max_chunk=32)
    assert rel(decode(s, "a", toks, 35), want) < tol(dtype)
    close(s)


def test_context_bound(cuda_backend):
    """Causal layers and pooled blocks keep something of every position: the caches hold what the caller asks for and a step past it
    is refused; the last position works, in every slot."""
    cfg = config([attention_layer(size=3, pool=4), pair_layer()])
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
