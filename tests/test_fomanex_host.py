"""Host side of Fomanex without a GPU: configuration errors, the order of layer runs, state sizing, the shape of the lowering on a fake
device, weight packing, the YaRN schedule, and properties of the float64 restatement that the GPU tests lean on."""
import json
import math

import numpy as np
import pytest

import fomanex_reference as ref
from fomanex_models import as_f64, config, dense, latent_layer, moe, random_weights, wkv_layer, yarn
from test_fotovik_host import FakeBuffer


@pytest.fixture
def fake_device(monkeypatch):
    import zgml_b200.host.fomanex as M
    import zgml_b200.host.state as S
    import zgml_b200.host.weights as Wt
    for module in (Wt, S, M):
        monkeypatch.setattr(module, "DeviceBuffer", FakeBuffer)
    monkeypatch.setattr(M, "seq_scratch_elems", lambda op: op.u.seq.n[0] * op.u.seq.n[4] * op.u.seq.n[2])


STACK = config([wkv_layer(mlp=dense(ff=24)), latent_layer(mlp=moe()), latent_layer(heads=2, dim=4, rot_dim=2, vdim=3, kv_rank=6), wkv_layer(heads=1, dim=6, rank=30, mlp=dense(ff=8))], streams=3, loop=(0, 2, 2))


def test_config_errors():
    from zgml_b200.host.fomanex import FomanexConfig
    cfg = FomanexConfig.from_dict(STACK)
    assert cfg.streams == 3 and cfg.logit_softcap == 4.0 and cfg.residual_mult == 0.6 and cfg.logit_scale == 0.3 and cfg.embedding_scale == 1.5
    assert FomanexConfig.from_dict({**STACK, "logit_softcap": None, "loop": None}).logit_softcap == 0.0
    for mutate in (lambda c: c.__setitem__("architecture", "Other"),
                   lambda c: c["layers"][0].__setitem__("type", "mamba2"),
                   lambda c: c["layers"][0]["mixer"].__setitem__("dim", 513),                # more key rows than the state kernels hold
                   lambda c: c["layers"][0]["mixer"].__setitem__("heads", 0),
                   lambda c: c["layers"][1]["mixer"].__setitem__("rot_dim", 6),              # not what the schedule turns
                   lambda c: c["layers"][1]["mixer"].update(rot_dim=7, rot={"base": 10.0, "dims": 7}),
                   lambda c: c["layers"][1]["mixer"].__setitem__("kv_rank", 0),
                   lambda c: c["layers"][0]["mlp"].__setitem__("kind", "poly"),
                   lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 7),
                   lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 0),
                   lambda c: c.__setitem__("streams", 0),
                   lambda c: c.__setitem__("streams", 17),
                   lambda c: c["loop"].__setitem__("stop", 5),
                   lambda c: c["loop"].__setitem__("start", 3),
                   lambda c: c["loop"].__setitem__("times", 0)):
        bad = json.loads(json.dumps(STACK))
        mutate(bad)
        with pytest.raises(ValueError):
            FomanexConfig.from_dict(bad)


@pytest.mark.parametrize("loop", [None, (0, 4, 2), (1, 3, 3), (3, 4, 2), (1, 3, 1), (2, 2, 5)])
def test_order_of_layer_runs(loop):
    from zgml_b200.host.fomanex import FomanexConfig
    c = json.loads(json.dumps(STACK))
    c.pop("loop")
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    assert list(FomanexConfig.from_dict(c).runs) == ref.layer_order(c)
    if loop == (1, 3, 3):
        assert ref.layer_order(c) == [0, 1, 2, 1, 2, 1, 2, 3]


def test_state_and_lowering_shape(fake_device):
    from zgml_b200 import abi
    from zgml_b200.host.fomanex import FomanexConfig, FomanexModel
    from zgml_b200.host.state import SequenceStatePool
    W = random_weights(STACK)
    m = FomanexModel(None, FomanexConfig.from_dict(STACK), lambda n: W[n], "bfloat16")
    assert sorted(m.buffers) == [-1, 0, 1, 2, 3] and m.bounded_context
    specs = {s.name: s for s in m.state_specs(16, 100)}
    assert {k: (s.elems, s.zero_on_acquire) for k, s in specs.items()} == {
        "run0.shift": (40, True), "run0.wkv": (3 * 64, True), "run1.latent": (100 * 20, False), "run2.shift": (40, True), "run2.wkv": (3 * 64, True), "run3.latent": (100 * 20, False),
        "run4.latent": (100 * 8, False), "run5.shift": (40, True), "run5.wkv": (36, True)}
    pool = SequenceStatePool(None, list(specs.values()), 2)
    for T, head, rows in ((1, "last", 1), (16, "all", 16), (4, "none", 0)):
        lp = m.lower(T, head, pool)
        ops = [(op.tag, op.u.seq) for op in lp.program.ops]
        tags = [t for t, _ in ops]
        of = lambda tag: [s for t, s in ops if t == tag]
        assert tags[0] == abi.OP_EMBED and ops[0][1].n[7] == 1 and lp.logits_rows == rows and (lp.buf_logits is None) == (head == "none")
        assert not {abi.OP_NORM, abi.OP_TOKEN_SHIFT, abi.OP_ROTARY, abi.OP_ACTIVATION, abi.OP_GATE, abi.OP_GATED_NORM} & set(tags)          # all of them ride in other launches
        # one launch per sublayer boundary: 6 runs, 5 feed-forwards, the head
        steps = of(abi.OP_STREAM_STEP)
        assert len(steps) == 6 + 5 + (head != "none")
        assert [s.buf[2] != abi.NO_BUF for s in steps] == [False] + [True] * (len(steps) - 1)               # the first only opens
        assert [s.n[3] for s in steps] == [0, 0] + [T * 40] * (len(steps) - 2)                               # the streams are one until the first close
        assert [s.n[6] for s in steps if s.n[6]] == [5] * 3 and all(s.n[5] == abi.NORM_DYNAMIC_TANH for s in steps)
        for a, b in zip(steps[1:], steps[2:]):
            assert b.buf[1] == a.buf[0] and b.buf[0] != b.buf[1]                                               # streams pass from step to step
        rule = of(abi.OP_DELTA_RULE)
        assert len(rule) == 3 and all(s.n[10] == abi.DELTA_PLAIN | abi.DELTA_SILU_GATE | abi.DELTA_BONUS | abi.DELTA_EXP_DECAY | abi.DELTA_WIDE_NORM for s in rule)
        assert rule[0].buf[6] != rule[1].buf[6] and rule[0].buf[5] == rule[1].buf[5]                         # a state per pass, one set of weights
        assert tags.count(abi.OP_CACHED_ATTENTION) == tags.count(abi.OP_CACHE_APPEND) == 3 and all(s.buf[6] != abi.NO_BUF for s in of(abi.OP_CACHED_ATTENTION))
        assert all(s.n[14] and s.buf[6] != abi.NO_BUF and s.buf[4] != abi.NO_BUF and s.f[3] > 1.0 for s in of(abi.OP_CACHE_APPEND))
        heads = [s for s in of(abi.OP_HEAD_LINEAR) if s.n[12]]
        assert [(s.n[1], s.n[2], s.n[10], s.n[11]) for s in heads] == [(5, 24, 5, abi.ACTIVATIONS["softcap"] + 1)] * 2 + [(5, 6, 30, abi.ACTIVATIONS["softcap"] + 1)]
        assert [s.n[5] for s in of(abi.OP_ROUTE)] == [3] * 2 and sum(s.n[10] for s in of(abi.OP_LINEAR)) == 3
        ext = [e.buf_idx for e in lp.program.externs]
        assert len(set(ext)) == len(ext) == 5 + 9 + 2                                                        # weights, states, frequencies of two layers: each once
    assert m.lower(16, "all", pool, keep_layers=True).layer_bufs is not None


def test_models_that_bound_the_sequence(fake_device):
    from zgml_b200.host.fomanex import FomanexConfig, FomanexModel

    def model(*layers):
        cfg = config(list(layers))
        W = random_weights(cfg)
        return FomanexModel(None, FomanexConfig.from_dict(cfg), lambda n: W[n], "float32")

    assert not model(wkv_layer()).bounded_context and model(wkv_layer(), latent_layer()).bounded_context
    m = model(latent_layer())
    assert m.capacity(16, 100) == 100 and m.capacity(16, None) == 4096 and m.capacity(256, 100) == 256


def test_wrong_shapes_are_named(fake_device):
    from zgml_b200.host.fomanex import FomanexConfig, FomanexModel
    W = random_weights(STACK)
    for name, shape in (("l0.hc1.mix", (3, 2)), ("l1.mix.uk", (17, 12)), ("l3.mix.u", (6, 1)), ("l1.mlp.e3.down", (12, 40)), ("final.norm.b", (41,))):
        bad = dict(W)
        bad[name] = np.zeros(shape, np.float32)
        with pytest.raises(AssertionError, match=name):
            FomanexModel(None, FomanexConfig.from_dict(STACK), lambda n: bad[n], "float32")


def test_expanding_weights():
    from zgml_b200.host.fomanex import expanding_weights
    r = np.random.default_rng(0)
    H, dim, rd, vdim, rank = 3, 4, 2, 5, 6
    uk, uv = r.standard_normal((H * dim, rank)).astype(np.float32), r.standard_normal((H * vdim, rank)).astype(np.float32)
    c, k = r.standard_normal(rank), r.standard_normal(rd)
    row = expanding_weights(uk, uv, H, rd) @ np.concatenate([c, k])
    keys = row[:H * (dim + rd)].reshape(H, dim + rd)
    assert np.allclose(keys[:, :dim].ravel(), uk @ c) and np.allclose(keys[:, dim:], k) and np.allclose(row[H * (dim + rd):], uv @ c)


def test_choice_of_the_expanded_form():
    from zgml_b200 import abi
    from zgml_b200.host.latent import EXPAND_MIN_TOKENS, expands
    assert expands(EXPAND_MIN_TOKENS, 96, 32, 48, 48, abi.W_BF16) and not expands(EXPAND_MIN_TOKENS - 1, 96, 32, 48, 48, abi.W_BF16)
    assert not expands(512, 96, 32, 48, 48, abi.W_F32) and expands(512, 96, 32, 48, 48, abi.W_F32, force_float32=True)
    assert not expands(512, 96, 30, 48, 48, abi.W_BF16) and not expands(512, 40, 16, 8, 8, abi.W_BF16) and not expands(512, 64, 16, 64, 64, abi.W_BF16)


@pytest.mark.parametrize("base,dims,scaling", [(100.0, 8, yarn()), (50.0, 12, yarn(3.0, 20, 1.0, 0.9)), (10000.0, 64, yarn(40.0, 4096, 32.0, 1.0)), (9.0, 6, yarn(2.0, 8, 100.0, 0.01)), (500.0, 10, yarn(1.0, 128, 4.0, 4.0))])
def test_yarn_schedule(base, dims, scaling):
    """The product's schedule against the restatement's, and against its meaning: pairs before the ramp keep their frequency, pairs after it
    turn `factor` times slower."""
    from zgml_b200.host.rotary import rotary_frequencies, rotary_magnitude
    rot = {"base": base, "dims": dims, "scaling": scaling}
    f, mag = ref.rotary_frequencies(rot)
    got = rotary_frequencies(rot)
    assert got.dtype == np.float32 and np.allclose(got, f, rtol=1e-6) and abs(rotary_magnitude(rot) - mag) < 1e-12 and mag == 0.1 * math.log(scaling["factor"]) + 1.0
    plain = base ** (-2.0 * np.arange(dims // 2) / dims)
    assert np.all(got <= plain * (1 + 1e-6)) and np.all(got >= plain / scaling["factor"] * (1 - 1e-6))
    turns = scaling["original"] * plain / (2 * math.pi)
    lo = dims * math.log(scaling["original"] / (2 * math.pi * scaling["fast"])) / (2 * math.log(base))
    hi = dims * math.log(scaling["original"] / (2 * math.pi * scaling["slow"])) / (2 * math.log(base))
    for i in range(dims // 2):
        if i <= max(math.floor(lo), 0):
            assert np.isclose(got[i], plain[i]), (i, turns)
        if i >= min(math.ceil(hi), dims - 1) and i > max(math.floor(lo), 0):
            assert np.isclose(got[i], plain[i] / scaling["factor"])
    assert rotary_magnitude({"base": base, "dims": dims}) == rotary_magnitude({"base": base, "dims": dims, "scaling": {"factor": 4.0}}) == 1.0


def test_other_schedules_are_as_before():
    from zgml_b200.host.rotary import rotary_frequencies
    assert np.allclose(rotary_frequencies({"base": 50.0, "dims": 6, "scaling": {"factor": 4.0}}), 50.0 ** (-np.arange(3) / 3.0) / 4)
    f = rotary_frequencies({"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 2.0, "original": 64}})
    assert np.isclose(f[0], 1.0) and np.isclose(f[-1], 10000.0 ** -0.75 / 4)


# ── the restatement ──
def test_restatement_of_streams():
    r = np.random.default_rng(1)
    X, y, mix, w = r.standard_normal((2, 3, 4)), r.standard_normal((3, 4)), np.array([[1.0, 2.0], [3.0, 5.0]]), np.array([0.5, -1.0])
    new = ref.write_streams(X, mix, w, y)
    assert np.allclose(new[0], X[0] + 3.0 * X[1] + 0.5 * y) and np.allclose(new[1], 2.0 * X[0] + 5.0 * X[1] - y)          # [from, to]
    assert np.allclose(ref.read_streams(X, w), 0.5 * X[0] - X[1])


def test_restatement_of_time_mixing():
    r = np.random.default_rng(2)
    rr, k, w = (r.standard_normal((2, 1, 3)) for _ in range(3))
    v, u = r.standard_normal((2, 1, 2)), r.standard_normal((1, 3))
    w = np.abs(w)
    out = ref.wkv_rule(rr, k, v, w, u)
    assert np.allclose(out[0, 0], (rr[0, 0] * u[0] * k[0, 0]).sum() * v[0, 0])                                            # the token itself, through the bonus only
    assert np.allclose(out[1, 0], (rr[1, 0] * k[0, 0]).sum() * v[0, 0] + (rr[1, 0] * u[0] * k[1, 0]).sum() * v[1, 0])     # its predecessor, not yet decayed
    three = ref.wkv_rule(*(np.concatenate([a, a[:1]]) for a in (rr, k, v, w)), u)
    assert np.allclose(three[2, 0], (rr[0, 0] * w[1, 0] * k[0, 0]).sum() * v[0, 0] + (rr[0, 0] * k[1, 0]).sum() * v[1, 0] + (rr[0, 0] * u[0] * k[0, 0]).sum() * v[0, 0])
    h = np.arange(6.0).reshape(3, 2)
    assert np.allclose(ref.token_mix(h, np.array([0.0, 0.25])), [[0.0, 0.75], [2.0, 2.5], [4.0, 4.5]])


def test_restatement_of_attention_and_routing():
    r = np.random.default_rng(3)
    q, k, v = (r.standard_normal((4, 2, 3)) for _ in range(3))
    out = ref.softmax_attention(q, k, v, 0.5, np.array([0.3, -50.0]))
    e = np.exp(k[:3, 0] @ q[2, 0] * 0.5)
    assert np.allclose(out[2, 0], (e / (e.sum() + math.exp(0.3))) @ v[:3, 0])
    e = np.exp(k[:, 1] @ q[3, 1] * 0.5)
    assert np.allclose(out[3, 1], (e / e.sum()) @ v[:, 1])                    # a sink far below the scores weighs nothing
    x = np.arange(4.0)
    assert np.allclose(ref.rotate(x, 1.0, np.array([0.3, 0.1]), 2.0)[[0, 2]], [-4 * math.sin(0.3), 4 * math.cos(0.3)])
    p = {"router": np.eye(3), "correction": np.array([0.0, 5.0, 0.0])}
    chosen, weight = ref.route(np.array([[1.0, -2.0, 0.5]]), p, "", {"top": 2, "scale": 3.0})
    assert chosen.tolist() == [[1, 0]] and np.allclose(weight, 3.0 * ref.sigmoid(np.array([[-2.0, 1.0]])))


def test_restatement_is_causal_and_carries_its_states():
    toks = np.random.default_rng(0).integers(0, STACK["vocab"], 30).tolist()
    W = as_f64(random_weights(STACK, seed=3, qk_gain=3.0))
    full, sums = ref.forward(STACK, W, toks, return_layers=True)
    assert np.allclose(ref.forward(STACK, W, toks[:17]), full[:17], atol=1e-11) and len(sums) == 6
    other = list(toks)
    other[0] = (other[0] + 1) % STACK["vocab"]
    assert np.abs(ref.forward(STACK, W, other)[-1] - full[-1]).max() > 1e-9
