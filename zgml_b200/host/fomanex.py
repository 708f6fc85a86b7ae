"""Fomanex: a pre-norm decoder stack with several residual streams (hyper-connections) and a Dynamic Tanh in place of every norm.  All
streams start as the normed embedding; a sublayer reads a weighted sum of them, and its layer-scaled result joins every stream while
the streams mix: X_b <- sum_a mix[a, b] X_a + m out_b ls * f(dyt(sum_a in_a X_a)).  The head reads the sum of the streams.  A layer's mixer is
  * RWKV-style time mixing: five token-shifted copies of the input feed receptance, key, value, gate and decay; a matrix state per
    head decays per key channel, exp(-exp(.)) of a low-rank product; the read-out sees the state before the token's own write and the
    token itself through a bonus; an RMS norm per head, a SiLU gate,
  * latent attention over every earlier position: keys and values are expanded per head from one RMS-normed latent, beside a rotated
    key part shared by all heads (YaRN schedule); a learned sink per head joins the softmax's denominator.
Feed-forwards are dense (tanh-GELU gate times up), a routed mixture of gated experts (sigmoid scores, chosen by score + correction, weighted by
the plain scores times a constant), or absent; the head is the embedding table, with scaled and smoothly capped logits.  A range of layers may run
several times in a row with the same weights, each pass with caches and states of its own.

This file is the model's configuration reader, its weight packer and its LOWERING to a DeviceProgram; the arithmetic is in the
sequence-model DeviceOps of the CUDA library (csrc/seqops.cu, csrc/mixops.cu, csrc/streamops.cu) and all state in the session's
`SequenceStatePool`.  Every size and per-model constant comes from config.json or a tensor's shape.

embedding   EMBED (token row * scale, Dynamic Tanh).
sublayers   ONE launch between two sublayers: STREAM_STEP (close over all streams, open, Dynamic Tanh, the mixer's five shifted copies).
wkv         [r | k | v | g | tanh w1] of the five copies in ONE batched product (HEAD_LINEAR, unequal last head, tanh on it); w2 (LINEAR);
            DELTA_RULE in its plain form (bonus, exp(-exp) decay, one norm weight over all heads, SiLU gate); W_o.
latent      [q | dkv] = W h in ONE matmul; CACHE_APPEND norms the latent and turns the shared key part on their way into the cache and
            turns the queries' rotated parts.  Short steps run ABSORBED: q' = W_uk^T q per head (HEAD_LINEAR) beside the turned part,
            CACHED_ATTENTION over the cached rows themselves (sinks), W_uv per head, W_o.  Long steps of bfloat16 sessions run EXPANDED:
            one tensor-core product with [W_uk 0; 0 1 | W_uv 0] turns the sequence's rows into whole keys | values per head.
dense       LINEAR over gate and up rows in turns (the gated product in its epilogue); W_down.
moe         router LINEAR, ROUTE "scaled_sigmoid", MOE_FFN.
"""
import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional

import numpy as np

from .. import abi
from ..backend import CudaBackend, DeviceBuffer, DeviceOp, DeviceProgram, ExternBuffer, seq_scratch_elems
from .latent import expands
from .rotary import rotary_frequencies, rotary_magnitude
from .safetensors import SafetensorsFile
from .session import LoweredProgram
from .state import SequenceStatePool, StateSpec
from .weights import WeightArena

ARCHITECTURE = "Fomanex"
DEFAULT_CONTEXT = 4096     # positions a sequence may reach where a layer keeps every position and the caller names no bound
MIXERS = ("wkv", "latent_attention")
SHIFTED = ("r", "k", "v", "g", "w")     # the token-shifted copies of a wkv layer's input, in the order the lowering keeps them
MAX_STATE_ROWS = 512       # key rows of a recurrent state the kernels hold per head
MAX_STREAMS = 16           # streams STREAM_STEP carries


@dataclass(frozen=True)
class FomanexConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    streams: int
    logit_scale: float
    logit_softcap: float       # 0: none
    layers: tuple              # of dicts: {"type", "mixer", "mlp"}
    runs: tuple                # layers in the order they run

    @classmethod
    def from_dict(cls, c: dict) -> "FomanexConfig":
        if c.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture = {c.get('architecture')!r}")
        layers = []
        for i, L in enumerate(c["layers"]):
            kind, m, mlp = L["type"], L["mixer"], L.get("mlp")
            if kind == "wkv":
                if min(m["heads"], m["dim"]) < 1 or m["dim"] > MAX_STATE_ROWS:
                    raise ValueError(f"layer {i}: heads and dim must be positive, dim at most {MAX_STATE_ROWS}")
            elif kind == "latent_attention":
                if min(m["heads"], m["dim"], m["vdim"], m["kv_rank"]) < 1:
                    raise ValueError(f"layer {i}: sizes must be positive")
                if m["rot_dim"] != m["rot"]["dims"] or m["rot_dim"] < 2 or m["rot_dim"] % 2:
                    raise ValueError(f"layer {i}: the rotated part must be rot_dim = rot.dims (even) wide")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            if mlp is not None:
                if mlp.get("kind") not in ("dense", "moe"):
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
                if mlp["kind"] == "moe" and not (1 <= mlp["router"]["top"] <= mlp["router"]["experts"]):
                    raise ValueError(f"layer {i}: top must lie in 1 .. experts")
            layers.append({"type": kind, "mixer": m, "mlp": mlp})
        n, loop = len(layers), c.get("loop")
        runs = list(range(n))
        if loop:
            a, b, times = loop["start"], loop["stop"], loop["times"]
            if not 0 <= a <= b <= n or times < 1:
                raise ValueError("loop: start .. stop - 1 must name layers of the stack, times at least 1")
            runs = runs[:a] + runs[a:b] * times + runs[b:]
        streams = int(c.get("streams", 1))
        if not 1 <= streams <= MAX_STREAMS:
            raise ValueError(f"streams must lie in 1 .. {MAX_STREAMS}")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float((c.get("embedding") or {}).get("scale", 1.0)), float(c.get("residual_mult", 1.0)),
                   streams, float(c.get("logit_scale", 1.0)), float(c.get("logit_softcap") or 0.0), tuple(layers), tuple(runs))

    @classmethod
    def from_json(cls, path: str) -> "FomanexConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))


def expanding_weights(uk: np.ndarray, uv: np.ndarray, heads: int, rot_dim: int) -> np.ndarray:
    """[heads * (dim + rot_dim) + heads * vdim, rank + rot_dim]: what a cached row [latent | rotated part] is multiplied with to give the heads'
    whole keys (the rotated part copied behind each) and their values."""
    dim, rank = uk.shape[0] // heads, uk.shape[1]
    w = np.zeros((heads * (dim + rot_dim) + uv.shape[0], rank + rot_dim), np.float32)
    keys = w[:heads * (dim + rot_dim)].reshape(heads, dim + rot_dim, rank + rot_dim)
    keys[:, :dim, :rank] = uk.reshape(heads, dim, rank)
    keys[:, dim:, rank:] = np.eye(rot_dim, dtype=np.float32)
    w[heads * (dim + rot_dim):, :rank] = uv
    return w


class FomanexModel:
    """Weights resident in HBM (one arena per layer + one for the embedding and the final norm) and the lowering."""

    def __init__(self, be: CudaBackend, cfg: FomanexConfig, tensors, dtype: str = "bfloat16"):
        """tensors: name -> f32 array accessor (`tensors(name)`), e.g. SafetensorsFile.f32."""
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype must be 'bfloat16' or 'float32'")
        self.be, self.cfg, self.dtype = be, cfg, dtype
        self.wdt = abi.W_BF16 if dtype == "bfloat16" else abi.W_F32
        self.vocab, self.width = cfg.vocab, cfg.width
        self.expand_float32 = False      # float32 sessions keep latent layers absorbed; set before the first long step to run them expanded as well
        self.layer_meta: List[dict] = []
        self.arenas: Dict[int, WeightArena] = {}
        self.buffers: Dict[int, DeviceBuffer] = {}
        self._freqs: Dict[int, DeviceBuffer] = {}      # per layer: frequencies of its rotary positions, f32
        D, S = cfg.width, cfg.streams

        def get(name, shape):
            t = tensors(name)
            assert tuple(t.shape) == tuple(shape), f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}"
            return t

        def dyt(name):             # weight | bias | alpha, in this order: what a Dynamic Tanh reads from one offset
            alpha = tensors(name + ".alpha")
            assert alpha.size == 1, f"{name}.alpha: shape {alpha.shape}"
            return np.concatenate([get(name, (D,)), get(name + ".b", (D,)), alpha.reshape(1)])

        def sublayer(A, p, q):     # what surrounds sublayer q of a layer
            A.add(f"norm{q}", dyt(f"{p}norm{q}"))
            A.add(f"ls{q}", get(f"{p}ls{q}", (D,)))
            for part, shape in (("in", (S,)), ("out", (S,)), ("mix", (S, S))):
                A.add(f"hc{q}.{part}", get(f"{p}hc{q}.{part}", shape))

        for i, L in enumerate(cfg.layers):
            p, m = f"l{i}.", L["mixer"]
            A = WeightArena(self.wdt)
            sublayer(A, p, 1)
            H, dim = m["heads"], m["dim"]
            if L["type"] == "wkv":
                C = H * dim
                w1 = tensors(p + "mix.w1")
                rank = w1.shape[0]
                A.add("mu", np.stack([get(f"{p}mix.mu.{s}", (D,)) for s in SHIFTED]))
                A.add("in", np.concatenate([get(f"{p}mix.{s}", (C, D)) for s in SHIFTED[:4]] + [get(p + "mix.w1", (rank, D))], 0))
                A.add("w2", get(p + "mix.w2", (C, rank)))
                A.add("w0", get(p + "mix.w0", (C,)))
                A.add("u", get(p + "mix.u", (H, dim)))
                A.add("norm", get(p + "mix.norm", (C,)))
                A.add("o", get(p + "mix.o", (D, C)))
                meta = {"n_in": 4 * C + rank, "C": C, "rank": rank}
            else:
                rd, vdim, rank = m["rot_dim"], m["vdim"], m["kv_rank"]
                uk, uv = get(p + "mix.uk", (H * dim, rank)), get(p + "mix.uv", (H * vdim, rank))
                A.add("in", np.concatenate([get(p + "mix.q", (H * (dim + rd), D)), get(p + "mix.dkv", (rank + rd, D))], 0))
                A.add("dkv.norm", get(p + "mix.dkv.norm", (rank,)))
                A.add("ukT", uk.reshape(H, dim, rank).transpose(0, 2, 1))     # [H, rank, dim]: q' = W_uk^T q per head
                A.add("uv", uv)                                               # [H, vdim, rank] as stored
                A.add("ukv", expanding_weights(uk, uv, H, rd))
                A.add("sink", get(p + "mix.sink", (H,)))
                A.add("o", get(p + "mix.o", (D, H * vdim)))
                meta = {"n_in": H * (dim + rd) + rank + rd}
                f = rotary_frequencies(m["rot"])
                self._freqs[i] = DeviceBuffer(be, max(f.nbytes, 16), zero=False)
                self._freqs[i].upload(np.concatenate([f, np.zeros(max(0, 4 - f.size), np.float32)]))
            meta["row"] = (meta["n_in"] + 3) // 4 * 4      # rows of the stacked projection start on 16-byte boundaries
            mlp = L["mlp"]
            if mlp is not None:
                sublayer(A, p, 2)
                if mlp["kind"] == "dense":
                    gate = tensors(p + "mlp.gate")
                    ff = gate.shape[0]
                    assert ff == mlp.get("ff", ff), f"{p}mlp.gate: {ff} rows, the configuration says {mlp.get('ff')}"
                    A.add("gate_up", np.stack([get(p + "mlp.gate", (ff, D)), get(p + "mlp.up", (ff, D))], 1))     # gate and up rows in turns
                    A.add("down", get(p + "mlp.down", (D, ff)))
                    meta["ff"] = ff
                else:
                    r = mlp["router"]
                    E, ff = r["experts"], mlp["expert"]["ff"]
                    A.add("router", get(p + "mlp.router", (E, D)))
                    A.add("correction", get(p + "mlp.correction", (E,)))
                    for part, shape in (("gate", (ff, D)), ("up", (ff, D)), ("down", (D, ff))):
                        A.add(part, np.stack([get(f"{p}mlp.e{e}.{part}", shape) for e in range(E)]))
                    meta.update(E=E, top=r["top"], ff=ff, scale=float(r.get("scale", 1.0)))
            self.layer_meta.append(meta)
            self.arenas[i] = A
            self.buffers[i] = A.upload(be)
        A = WeightArena(self.wdt)
        A.add("embed", get("embed", (cfg.vocab, D)))
        A.add("embed.norm", dyt("embed.norm"))
        A.add("final.norm", dyt("final.norm"))
        A.add("ones", np.ones(S, np.float32))          # the head reads the plain sum of the streams
        self.arenas[-1] = A
        self.buffers[-1] = A.upload(be)

    @classmethod
    def load(cls, be: CudaBackend, model_dir: str, dtype: str = "bfloat16") -> "FomanexModel":
        cfg = FomanexConfig.from_json(os.path.join(model_dir, "config.json"))
        sf = SafetensorsFile(os.path.join(model_dir, "model.safetensors"))
        try:
            return cls(be, cfg, sf.f32, dtype)
        finally:
            sf.close()

    def weight_bytes(self) -> int:
        return sum(b.nbytes for b in self.buffers.values())

    # ── state ──
    @property
    def bounded_context(self) -> bool:
        """Latent layers keep every position: the session then bounds the sequence."""
        return any(L["type"] == "latent_attention" for L in self.cfg.layers)

    def capacity(self, max_chunk: int, max_context: Optional[int]) -> int:
        """Positions a sequence may reach where a layer keeps every position."""
        return max(int(max_context) if max_context else DEFAULT_CONTEXT, max_chunk)

    def state_specs(self, max_chunk: int, max_context: Optional[int] = None) -> List[StateSpec]:
        """Caches and states of every layer RUN: a layer that runs several times has one set per pass."""
        specs = []
        for n, i in enumerate(self.cfg.runs):
            m, name = self.cfg.layers[i]["mixer"], f"run{n}"
            if self.cfg.layers[i]["type"] == "wkv":
                specs.append(StateSpec(name + ".shift", self.width, True))
                specs.append(StateSpec(name + ".wkv", m["heads"] * m["dim"] * m["dim"], True))
            else:
                specs.append(StateSpec(name + ".latent", self.capacity(max_chunk, max_context) * (m["kv_rank"] + m["rot_dim"]), False))    # masked by position: no clearing
        return specs

    # ── lowering ──
    def lower(self, T: int, head: str, pool: SequenceStatePool, keep_layers: bool = False) -> LoweredProgram:
        cfg, wdt, D, S, eps = self.cfg, self.wdt, self.cfg.width, self.cfg.streams, self.cfg.norm_eps
        sizes: List[int] = []
        externs: List[ExternBuffer] = []
        ops = []

        def new(n):
            sizes.append(max(int(n), 1))
            return len(sizes) - 1

        ext_of: Dict[int, int] = {}

        def ext(buf: DeviceBuffer):      # one program buffer per device buffer (passes of a loop name the same weights)
            if id(buf) not in ext_of:
                sizes.append(buf.elems)
                externs.append(ExternBuffer(len(sizes) - 1, buf))
                ext_of[id(buf)] = len(sizes) - 1
            return ext_of[id(buf)]

        ctl = new(abi.CTL_IDS + T)
        gl, GA = ext(self.buffers[-1]), self.arenas[-1]
        TD = T * D
        emb, xs = new(TD), [new(S * TD), new(S * TD)]
        h, y = new(TD), new(TD)
        shared: Dict[str, int] = {}

        def scratch(name, n):      # activations reused by every layer that needs them
            if name not in shared or sizes[shared[name]] < n:
                shared[name] = new(n)
            return shared[name]

        ops.append(DeviceOp.embed(emb, ctl, gl, GA.off["embed"], T, D, cfg.embedding_scale, wdt, dyt_off=GA.off["embed.norm"]))
        x, stride = emb, 0         # the streams: all equal to the embedding output until the first sublayer closes
        # The step that closes a sublayer waits for the one that opens the next: one launch for both.
        pending: List[dict] = []

        def stream_step(**kw):
            nonlocal x, stride
            closing = pending.pop() if pending else {}
            nx = (xs[1] if x == xs[0] else xs[0]) if closing else None
            ops.append(DeviceOp.stream_step(T, D, S, wdt, dst=nx, src=x, src_stride=stride, **closing, **kw))
            if closing:
                x, stride = nx, TD

        def close_with(wb, A, q):
            pending.append(dict(y=y, close_w=wb, out_off=A.off[f"hc{q}.out"], mix_off=A.off[f"hc{q}.mix"], ls_off=A.off[f"ls{q}"], mult=cfg.residual_mult))

        slots = pool.n_slots
        layer_bufs = []
        for n, i in enumerate(cfg.runs):
            L, name = cfg.layers[i], f"run{n}"
            m, mlp, meta, A, wb = L["mixer"], L["mlp"], self.layer_meta[i], self.arenas[i], ext(self.buffers[i])
            H, dim, rs = m["heads"], m["dim"], meta["row"]
            proj = scratch("proj", T * rs)
            opening = dict(open_w=wb, in_off=A.off["hc1.in"], norm_off=A.off["norm1"])
            if L["type"] == "wkv":
                C, rank = meta["C"], meta["rank"]
                copies = scratch("copies", len(SHIFTED) * TD)
                stream_step(h=copies, shifts=len(SHIFTED), mu_off=A.off["mu"], state=ext(pool.buffers[name + ".shift"]), ctl=ctl, **opening)
                ops.append(DeviceOp.head_linear(proj, copies, wb, A.off["in"], T, len(SHIFTED), C, D, wdt, dst_hs=C, dst_rs=rs, n_last=rank, last_act="softcap", last_act_param=1.0,
                                                rounded=True))      # tanh: the smooth cap at 1
                decay = scratch("decay", T * C)
                ops.append(DeviceOp.linear(decay, proj, wb, A.off["w2"], T, C, rank, wdt, src_off=4 * C, src_rs=rs))
                mix = scratch("mix", T * C)
                ops.append(DeviceOp.delta_rule(mix, proj, None, decay, proj, wb, ext(pool.buffers[name + ".wkv"]), ctl, 0, C, 2 * C, 0, 0, A.off["w0"], A.off["norm"], T, H, H, dim, dim,
                                               rs, 0, C, rs, wdt, eps, 0.0, 1.0, gate_off=3 * C, plain=True, silu_gate=True, bonus_off=A.off["u"], exp_decay=True, wide_norm=True))
                ops.append(DeviceOp.linear(y, mix, wb, A.off["o"], T, D, C, wdt))
            else:
                rd, vdim, rank = m["rot_dim"], m["vdim"], m["kv_rank"]
                dk, cw = dim + rd, rank + rd
                stream_step(h=h, **opening)
                ops.append(DeviceOp.linear(proj, h, wb, A.off["in"], T, meta["n_in"], D, wdt, dst_rs=rs))
                cache = pool.buffers[name + ".latent"]
                R = cache.elems // (slots * cw)
                att = scratch("att", T * H * vdim)
                sink = dict(sink=wb, sink_off=A.off["sink"], sink_wdt=wdt)
                long_step = expands(T, rank, rd, dim, vdim, wdt, self.expand_float32)
                qa = None if long_step else scratch("qa", T * H * cw)      # absorbed queries: [W_uk^T q | turned part] per head
                ops.append(DeviceOp.cache_append(ext(cache), proj, ctl, H * dk, 0, T, cw, rs, cw, R, norm_w=wb, norm_off=A.off["dkv.norm"], normed=rank, eps=eps, wdt=wdt, rot=rd,
                                                 rot_layout="halves", freqs=ext(self._freqs[i]), rot_scale=rotary_magnitude(m["rot"]), turned_heads=(H, dim, dk, qa, rank, cw)))
                if long_step:
                    kvw = H * (dk + vdim)
                    kv = scratch("latent.kv", R * kvw)
                    ops.append(DeviceOp.linear(kv, ext(cache), wb, A.off["ukv"], R, kvw, cw, wdt, ctl=ctl, src_slot_stride=R * cw, live_rows=T))
                    ops.append(DeviceOp.cached_attention(att, proj, kv, kv, ctl, 0, 0, H * dk, T, H, H, 1, dk, vdim, rs, kvw, kvw, R, m["scale"], unslotted=True, **sink))
                else:
                    ops.append(DeviceOp.head_linear(qa, proj, wb, A.off["ukT"], T, H, rank, dim, wdt, src_hs=dk, src_rs=rs, dst_hs=cw, dst_rs=H * cw))
                    ctx = scratch("ctx", T * H * rank)
                    ops.append(DeviceOp.cached_attention(ctx, qa, ext(cache), ext(cache), ctl, 0, 0, 0, T, H, 1, 1, cw, rank, H * cw, cw, cw, R, m["scale"], **sink))
                    ops.append(DeviceOp.head_linear(att, ctx, wb, A.off["uv"], T, H, vdim, rank, wdt))
                ops.append(DeviceOp.linear(y, att, wb, A.off["o"], T, D, H * vdim, wdt))
            close_with(wb, A, 1)
            if mlp is not None:
                stream_step(h=h, open_w=wb, in_off=A.off["hc2.in"], norm_off=A.off["norm2"])
                ff = meta["ff"]
                if mlp["kind"] == "dense":
                    act = scratch("ff", T * ff)
                    ops.append(DeviceOp.linear(act, h, wb, A.off["gate_up"], T, ff, D, wdt, act="gelu_tanh", pairs=True))
                    ops.append(DeviceOp.linear(y, act, wb, A.off["down"], T, D, ff, wdt))
                else:
                    E, top = meta["E"], meta["top"]
                    rl, rt = scratch("router", T * E), scratch("route", T * top * 2)
                    ops.append(DeviceOp.linear(rl, h, wb, A.off["router"], T, E, D, wdt))
                    ops.append(DeviceOp.route(rt, rl, wb, A.off["correction"], T, E, top, wdt, mode="scaled_sigmoid", scale=meta["scale"]))
                    moe_op = DeviceOp.moe_ffn(y, h, rt, wb, 0, A.off["gate"], A.off["up"], A.off["down"], T, D, ff, E, top, wdt, float("inf"), 1.0, up_offset=0.0)
                    moe_op.u.seq.buf[4] = scratch("expert", seq_scratch_elems(moe_op))   # the library knows what its kernels stage
                    ops.append(moe_op)
                close_with(wb, A, 2)
            if keep_layers:
                stream_step()
                layer_bufs.append(new(TD))
                ops.append(DeviceOp.depth_mix(layer_bufs[-1], x, gl, GA.off["ones"], TD, S, TD, wdt))
        logits, rows = None, 0
        if head != "none":         # (a step that asks for no logits drops its last close)
            stream_step(h=h, open_w=gl, in_off=GA.off["ones"], norm_off=GA.off["final.norm"], gain=cfg.logit_scale)
            rows = T if head == "all" else 1
            logits = new(rows * cfg.vocab)
            cap = cfg.logit_softcap
            ops.append(DeviceOp.linear(logits, h, gl, GA.off["embed"], rows, cfg.vocab, D, wdt, src_off=0 if head == "all" else (T - 1) * D,
                                       act="softcap" if cap else None, act_param=cap))       # the head is the embedding table; the cap rides in the epilogue
        prog = DeviceProgram(ops, sizes, [], [], externs)
        return LoweredProgram(prog, ctl, logits, rows, layer_bufs if keep_layers else None)

    def close(self):
        for b in list(self.buffers.values()) + list(self._freqs.values()):
            b.free()
        self.buffers, self._freqs = {}, {}


def synthetic_config(width: int, n_layers: int, heads: int, dim: int, experts: int, top: int, ff: int, vocab: int, kv_rank: int = 512, rot_dim: int = 64,
                     wkv_dim: int = 64, wkv_heads: Optional[int] = None, streams: int = 2, loop: Optional[dict] = None) -> dict:
    """config.json contents of a random-init model: layers alternate between time mixing and latent attention; feed-forwards alternate between
    a dense layer as wide as the experts a token uses and routed experts."""
    layers = []
    for i in range(n_layers):
        mlp = ({"kind": "dense", "ff": top * ff} if i % 2 == 0 else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": 1.0}})
        if i % 2 == 0:
            layers.append({"type": "wkv", "mixer": {"heads": wkv_heads or width // wkv_dim, "dim": wkv_dim}, "mlp": mlp})
        else:
            rot = {"base": 10000.0, "dims": rot_dim, "scaling": {"factor": 4.0, "original": 1024, "fast": 16.0, "slow": 2.0}}
            layers.append({"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": dim, "kv_rank": kv_rank, "rot": rot,
                                                                              "scale": (dim + rot_dim) ** -0.5}})
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "residual_mult": 1.0, "streams": streams,
            "logit_scale": 1.0, "logit_softcap": 30.0, "layers": layers, "loop": loop}


def synthetic_tensors(cfg: dict, seed: int = 0, decay_rank: int = 64):
    """Accessor name -> random f32 tensor of the shape the configuration implies (benchmarks and smoke runs; values are scaled like a
    trained model's so that activations stay O(1))."""
    import zlib
    D, S = cfg["width"], cfg["streams"]

    def shape_of(name):
        if name == "embed":
            return (cfg["vocab"], D)
        if name.endswith(".alpha"):
            return ()
        if name.startswith(("embed.norm", "final.norm")):
            return (D,)
        layer, rest = name.split(".", 1)
        L = cfg["layers"][int(layer[1:])]
        m = L["mixer"]
        if rest.startswith(("norm", "ls")):
            return (D,)
        if rest.startswith("hc"):
            return (S, S) if rest.endswith("mix") else (S,)
        if rest.startswith("mlp."):
            part = rest.split(".")[-1]
            if part in ("router", "correction"):
                E = L["mlp"]["router"]["experts"]
                return (E, D) if part == "router" else (E,)
            ff = L["mlp"]["ff"] if L["mlp"]["kind"] == "dense" else L["mlp"]["expert"]["ff"]
            return (D, ff) if part == "down" else (ff, D)
        t = rest[len("mix."):]
        H, d = m["heads"], m["dim"]
        if L["type"] == "wkv":
            C = H * d
            return (D,) if t.startswith("mu.") else {"w1": (decay_rank, D), "w2": (C, decay_rank), "w0": (C,), "u": (H, d), "norm": (C,), "o": (D, C)}.get(t, (C, D))
        rd, dv, rank = m["rot_dim"], m["vdim"], m["kv_rank"]
        return {"q": (H * (d + rd), D), "dkv": (rank + rd, D), "dkv.norm": (rank,), "uk": (H * d, rank), "uv": (H * dv, rank), "sink": (H,), "o": (D, H * dv)}[t]

    def get(name):
        shp = shape_of(name)
        r = np.random.default_rng([seed, zlib.crc32(name.encode())])
        last = name.rsplit(".", 1)[-1]
        if last == "alpha":
            return np.array(0.5, np.float32)
        if last == "in":
            return np.full(shp, 1.0 / shp[0], np.float32)
        if last == "mix" and name.split(".")[1].startswith("hc"):
            return (0.8 * np.eye(shp[0]) + 0.2 / shp[0]).astype(np.float32)
        if last in ("norm", "norm1", "norm2", "ls1", "ls2", "out"):
            return np.ones(shp, np.float32)
        if last == "w0":
            return (-4.0 + 3.0 * r.random(shp, dtype=np.float32)).astype(np.float32)
        if len(shp) == 1 or last == "u":
            return (r.random(shp, dtype=np.float32) * 0.5).astype(np.float32)
        a = r.random(shp, dtype=np.float32)
        a -= 0.5
        a *= np.float32(np.sqrt(12.0 / (1 if name == "embed" else shp[-1])))
        return a

    return get
