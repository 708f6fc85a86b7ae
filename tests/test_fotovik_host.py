"""Host side of Fotovik without a GPU: configuration errors, the order of layer runs, ring, block and state sizing, the shape of the
lowering on a fake device, the token before a step, and properties of the float64 restatement that the GPU tests lean on."""
import json
import math

import numpy as np
import pytest

import fotovik_reference as ref
from fotovik_models import as_f64, attention_layer, config, delta_layer, dense, pair_layer, random_weights


class FakeBuffer:
    def __init__(self, be, nbytes, zero=True):
        self.nbytes = (int(nbytes) + 15) & ~15
        self.elems = self.nbytes // 4

    def upload(self, host, byte_offset=0):
        pass

    def fill_zero(self, byte_offset, nbytes):
        pass

    def free(self):
        pass


@pytest.fixture
def fake_device(monkeypatch):
    import zgml_b200.host.fotovik as M
    import zgml_b200.host.state as S
    import zgml_b200.host.weights as Wt
    monkeypatch.setattr(Wt, "DeviceBuffer", FakeBuffer)
    monkeypatch.setattr(S, "DeviceBuffer", FakeBuffer)
    monkeypatch.setattr(M, "DeviceBuffer", FakeBuffer)


STACK = config([attention_layer(mlp=dense()), pair_layer(mlp=dense()), delta_layer(), delta_layer(conv=1, mlp=dense(ff=8))], loop=(0, 2, 2))


def test_config_errors():
    from zgml_b200.host.fotovik import FotovikConfig
    cfg = FotovikConfig.from_dict(STACK)
    assert cfg.embedding_scale == 1.5 and cfg.bigram["buckets"] == 37 and not cfg.layers[2]["mlp"]
    for mutate in (lambda c: c.__setitem__("architecture", "Other"),
                   lambda c: c["layers"][0].__setitem__("type", "mamba2"),
                   lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3),             # heads not a multiple
                   lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 5),
                   lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 10),         # more than the head holds
                   lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0),
                   lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("pool", 0),
                   lambda c: c["layers"][1]["mixer"]["left"].__setitem__("heads", 3),
                   lambda c: c["layers"][1]["mixer"]["right"].__setitem__("decay", [0.5]),   # one decay per head
                   lambda c: c["layers"][2]["mixer"].__setitem__("conv", 0),
                   lambda c: c["layers"][2]["mixer"].__setitem__("dim", 513),                # more key rows than the state kernels hold
                   lambda c: c["layers"][3]["mlp"].__setitem__("kind", "moe"),
                   lambda c: c["loop"].__setitem__("stop", 5),
                   lambda c: c["loop"].__setitem__("start", 3),
                   lambda c: c["loop"].__setitem__("times", 0),
                   lambda c: c["embedding"]["bigram"].__setitem__("buckets", 0)):
        bad = json.loads(json.dumps(STACK))
        mutate(bad)
        with pytest.raises(ValueError):
            FotovikConfig.from_dict(bad)


@pytest.mark.parametrize("loop,want", [(None, "0 1 2 3"), ((0, 4, 2), "0 1 2 3 +0 1 2 3"), ((1, 3, 3), "0 1 2 +1 2 +1 2 3"), ((3, 4, 2), "0 1 2 3 +3"), ((1, 3, 1), "0 1 2 3"), ((2, 2, 5), "0 1 2 3")])
def test_order_of_layer_runs(loop, want):
    """Layers of the loop in the order they run; + where the embedding output joins the stream again."""
    from zgml_b200.host.fotovik import FotovikConfig
    c = json.loads(json.dumps(STACK))
    c.pop("loop")
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    runs = FotovikConfig.from_dict(c).runs
    assert " ".join(("+" if again else "") + str(i) for i, again in runs) == want and list(runs) == ref.layer_order(c)


def test_state_and_lowering_shape(fake_device):
    from zgml_b200 import abi
    from zgml_b200.host.fotovik import FotovikConfig, FotovikModel
    from zgml_b200.host.state import SequenceStatePool
    W = random_weights(STACK)
    m = FotovikModel(None, FotovikConfig.from_dict(STACK), lambda n: W[n], "bfloat16")
    assert sorted(m.buffers) == [-1, 0, 1, 2, 3] and m.bounded_context
    specs = {s.name: s for s in m.state_specs(16, 100)}
    assert list(specs) == ["run0.kv", "run0.pooled", "run1.kv", "run1.lightning", "run2.kv", "run2.pooled", "run3.kv", "run3.lightning", "run4.tail", "run4.delta", "run5.delta"]
    row = 2 * (8 + 12)
    assert specs["run0.kv"].elems == (9 - 1 + 16) * row and specs["run0.pooled"].elems == 25 * row       # what the window reaches back plus one step; a row per block of 4 positions
    assert specs["run1.kv"].elems == 100 * row and specs["run1.lightning"].elems >= 3 * 6 * 10
    assert specs["run4.tail"].elems == 2 * (2 * 2 * 8 + 4 * 12) and specs["run4.delta"].elems == 4 * 8 * 12
    assert [s.zero_on_acquire for s in specs.values()] == [False, False, False, True, False, False, False, True, True, True, True]
    pool = SequenceStatePool(None, list(specs.values()), 2)
    for T, head, rows in ((1, "last", 1), (16, "all", 16), (4, "none", 0)):
        lp = m.lower(T, head, pool)
        ops = [(op.tag, op.u.seq) for op in lp.program.ops]
        tags = [t for t, _ in ops]
        of = lambda tag: [s for t, s in ops if t == tag]
        assert tags[0] == abi.OP_EMBED and list(ops[0][1].n[4:7]) == [37, 11, 5] and lp.logits_rows == rows and (lp.buf_logits is None) == (head == "none")
        assert tags.count(abi.OP_CACHED_ATTENTION) == tags.count(abi.OP_CACHE_APPEND) == 4 and tags.count(abi.OP_DELTA_RULE) == 2 and tags.count(abi.OP_SSM_SCAN) == 2
        assert abi.OP_ROTARY not in tags and abi.OP_HEAD_NORM not in tags and abi.OP_ACTIVATION not in tags          # all of them ride in other launches
        att, app = of(abi.OP_CACHED_ATTENTION), of(abi.OP_CACHE_APPEND)
        assert [s.off[3] for s in att] == [abi.MASK_POOLED, abi.MASK_CAUSAL] * 2 and [s.buf[6] != abi.NO_BUF for s in att] == [True, False] * 2
        assert [s.n[13] for s in app] == [abi.ROTATE_ONLY, abi.NORM_THEN_ROTATE] * 2 and [s.n[8] for s in app] == [0, 1] * 2 and [s.n[11] for s in app] == [4, 0] * 2
        assert att[0].buf[2] != att[2].buf[2] and att[0].buf[7] != att[2].buf[7] and att[0].buf[6] == att[2].buf[6]   # a ring and blocks per pass, one set of weights
        assert all(s.n[10] == abi.DELTA_HEAD_DECAY | abi.DELTA_SILU_GATE for s in of(abi.OP_DELTA_RULE)) and all(s.n[8] == 1 for s in of(abi.OP_SSM_SCAN))
        assert all(s.n[7] == abi.GATE_AFTER | abi.GATE_SIGMOID for s in of(abi.OP_GATED_NORM))
        silu = [s for s in of(abi.OP_LINEAR) if s.n[6] == abi.ACTIVATIONS["silu"] + 1]
        C = 4 * 8 + 2 * (8 + 12)
        assert [(s.n[8], s.n[9]) for s in silu] == [(C, C + 2 * 18 + 30)] * 2 and sum(s.n[6] == abi.ACTIVATIONS["gelu_erf"] + 1 for s in of(abi.OP_LINEAR)) == 5
        # one launch per sublayer boundary: 6 runs, 5 feed-forwards, the pass that adds the embedding output again, the head
        norms = of(abi.OP_NORM)
        assert len(norms) == 6 + 5 + 1 + (head != "none")
        assert [s.buf[3] != abi.NO_BUF for s in norms] == [False] + [True] * (len(norms) - 1)
        again = [s for s in norms if s.n[2] & abi.NORM_NONE]
        assert len(again) == 1 and again[0].buf[1] == ops[0][1].buf[0]                                                 # the embedding output, where EMBED left it
        assert all(s.buf[0] != ops[0][1].buf[0] for s in norms)                                                        # nothing overwrites it
        assert [s.n[8] for s in norms if s.n[7]] == [1 + (abi.NORM_RMS | abi.NORM_SCALAR_WEIGHT)] * 2                  # the pair: two sources and the norm over their sum
        assert all(s.n[2] & abi.NORM_SCALAR_WEIGHT for s in norms if not s.n[7] and not s.n[2] & abi.NORM_NONE)
        ext = [e.buf_idx for e in lp.program.externs]
        assert len(set(ext)) == len(ext) == 5 + 11 + 2 + 1                                      # weights, states, frequencies of two layers, decays: each once


def test_models_that_bound_the_sequence(fake_device):
    from zgml_b200.host.fotovik import FotovikConfig, FotovikModel

    def model(*layers):
        cfg = config(list(layers))
        W = random_weights(cfg)
        return FotovikModel(None, FotovikConfig.from_dict(cfg), lambda n: W[n], "float32")

    assert not model(delta_layer()).bounded_context and model(pair_layer()).bounded_context and model(attention_layer()).bounded_context
    window_only = attention_layer()
    del window_only["mixer"]["mask"]["pool"]
    m = model(window_only)
    assert not m.bounded_context and [s.name for s in m.state_specs(8)] == ["run0.kv"]
    m = model(pair_layer())
    assert m.capacity(16, 100) == 100 and m.capacity(16, None) == 4096 and m.capacity(256, 100) == 256
    # a block longer than the window decides what the ring must hold; a window longer than the sequence does not
    assert model(attention_layer(size=3, pool=10)).state_specs(4, 50)[0].elems == (10 + 4) * 40
    assert model(attention_layer(size=10 ** 6, pool=10)).state_specs(4, 50)[0].elems == (50 + 4) * 40


def test_the_token_before_a_step(fake_device):
    from zgml_b200.host.state import SequenceStatePool, StateSpec
    pool = SequenceStatePool(None, [StateSpec("s", 4, True)], 1)
    pool.acquire("a")
    assert pool.last_token("a") == -1
    pool.advance("a", 3, 17)
    assert pool.last_token("a") == 17 and pool.position("a") == 3
    pool.release("a")
    pool.acquire("b")
    assert pool.last_token("b") == -1


def test_linear_scaling_of_rotary_frequencies():
    from zgml_b200.host.rotary import rotary_frequencies
    rot = {"base": 50.0, "dims": 6, "scaling": {"factor": 4.0}}
    assert np.allclose(rotary_frequencies(rot), [0.25, 50.0 ** (-1 / 3) / 4, 50.0 ** (-2 / 3) / 4]) and np.allclose(rotary_frequencies(rot), ref.rotary_frequencies(rot))


# ── the restatement ──
def test_restatement_of_the_visible_keys():
    assert [ref.visible(i, 4, 3) for i in (0, 3, 5, 6, 8, 9)] == [(0, 0), (0, 0), (2, 0), (3, 1), (5, 1), (6, 2)]
    r = np.random.default_rng(2)
    q, k, v = r.standard_normal((7, 2, 3)), r.standard_normal((7, 1, 3)), r.standard_normal((7, 1, 4))
    out = ref.softmax_attention(q, k, v, 0.5, 2, 3, np.array([0.3, -50.0]))
    K, V = np.stack([k[4, 0], k[5, 0], k[0:3, 0].mean(0)]), np.stack([v[4, 0], v[5, 0], v[0:3, 0].mean(0)])     # position 3 has left the window, its block is not complete
    e = np.exp(K @ q[5, 0] * 0.5)
    assert np.allclose(out[5, 0], (e / (e.sum() + math.exp(0.3))) @ V)
    e = np.exp(K @ q[5, 1] * 0.5)
    assert np.allclose(out[5, 1], (e / e.sum()) @ V)                  # a sink far below the scores weighs nothing


def test_restatement_is_causal_and_carries_its_states():
    toks = np.random.default_rng(0).integers(0, STACK["vocab"], 30).tolist()
    W = as_f64(random_weights(STACK, seed=3, qk_gain=3.0))
    full, streams = ref.forward(STACK, W, toks, return_layers=True)
    assert np.allclose(ref.forward(STACK, W, toks[:17]), full[:17], atol=1e-11) and len(streams) == 6
    other = list(toks)
    other[0] = (other[0] + 1) % STACK["vocab"]
    assert np.abs(ref.forward(STACK, W, other)[-1] - full[-1]).max() > 1e-9


def test_restatement_of_embedding_and_recurrences():
    assert ref.bigram_rows([5, 2, 2], {"buckets": 7, "mul_prev": 3, "mul_cur": 4}) == [7, (15 + 8) % 7, (6 + 8) % 7]
    r = np.random.default_rng(5)
    q, k, v = r.standard_normal((2, 1, 3)), r.standard_normal((2, 1, 3)), r.standard_normal((2, 1, 2))
    beta, g = np.array([[0.4], [0.9]]), np.array([[0.5], [0.25]])
    out = ref.delta_rule(q, k, v, beta, g)
    S = np.outer(k[0, 0], 0.4 * v[0, 0])
    assert np.allclose(out[0, 0], S.T @ q[0, 0])                      # read after the token's own write
    S = 0.25 * S
    S = S + np.outer(k[1, 0], 0.9 * (v[1, 0] - S.T @ k[1, 0]))        # corrected after the decay
    assert np.allclose(out[1, 0], S.T @ q[1, 0])
    out = ref.lightning_rule(q, k, v, [0.5])
    assert np.allclose(out[1, 0], (0.5 * np.outer(k[0, 0], v[0, 0]) + np.outer(k[1, 0], v[1, 0])).T @ q[1, 0])
    x = np.arange(6.0)
    assert np.allclose(ref.rotate(x, 2.0, np.array([0.3]), True)[:2], [-math.sin(0.6), math.cos(0.6)]) and np.allclose(ref.rotate(x, 2.0, np.array([0.3]), True)[2:], x[2:])
    h = ref.rotate(x, 1.0, np.array([0.3, 0.1]), False)
    assert np.allclose([h[0], h[2]], [-2 * math.sin(0.3), 2 * math.cos(0.3)]) and np.allclose(h[4:], x[4:])
    assert abs(ref.gelu_erf(np.array([1.0]))[0] - 0.8413447) < 1e-6
