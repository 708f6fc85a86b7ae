"""Fotovik: a decoder stack whose stream starts as a scaled token embedding plus a hashed bigram embedding, and whose sublayers are
normed on the way in and on the way out, every norm with ONE learned number: x += n1b rms(mixer(n1 rms(x))), x += n2b rms(ff(n2 rms(x))).
A layer's mixer is one of
  * attention inside a sliding window that also sees, as one mean key and value each, the blocks of tokens that lie wholly before the
    window; interleaved rotary positions, grouped key / value heads, a learned sink per head in the softmax's denominator,
  * a gated delta rule with one decay per head: q, k and v pass a short causal convolution and SiLU, q and k become unit vectors,
    a matrix state per head is corrected towards v, read out through an RMS norm per head and a SiLU gate,
  * two mixers side by side on the same input: causal attention over every position (RMS-normed query and key heads, rotated by
    halves on a linearly scaled schedule) and lightning attention (a matrix state per head with a constant decay; SiLU on q, k and v;
    one RMS norm over all heads, then a sigmoid gate).  Each result is RMS-normed over the model width; half their sum goes on.
Feed-forwards are dense (exact GELU) or absent; the head is a matrix of its own.  A range of layers may run several times in a row
with the same weights, each pass with caches and states of its own; before every pass but the first the embedding output joins the stream.

This file is the model's configuration reader, its weight packer and its LOWERING to a DeviceProgram; the arithmetic is in the
sequence-model DeviceOps of the CUDA library (csrc/seqops.cu, csrc/mixops.cu, csrc/recops.cu) and all state in the session's
`SequenceStatePool`.  Every size and per-model constant comes from config.json or a tensor's shape.

embedding   EMBED (token row * scale + bigram row; the token before the step comes with the control words).
norms       one launch closes a sublayer and opens the next: NORM (residual + norm of the result, then the opening norm); after the
            pair it also adds its two normed branches and norms their sum.
attention   [q | k | v] = W h in ONE matmul; CACHE_APPEND (key heads turned on their way into the ring, values copied, query heads turned
            in place, the mean row of every completed block kept beside the ring); CACHED_ATTENTION (mask "pooled", sinks); W_o.
delta       [q | k | v | g | b | a] in ONE matmul; CAUSAL_CONV (SiLU) over q | k | v; DELTA_RULE (one decay per head, SiLU gate); W_o.
parallel    [q | k | v | q' | k' | v' | g'] in ONE matmul for both branches, SiLU in its epilogue on q' | k' | v' alone.  Left: CACHE_APPEND
            (heads normed, then turned), CACHED_ATTENTION, W_o.  Right: SSM_SCAN with constant decays (its B, C and x are k', q' and v'),
            GATED_NORM (sigmoid gate after the norm), W_o.
"""
import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional

import numpy as np

from .. import abi
from ..backend import CudaBackend, DeviceBuffer, DeviceOp, DeviceProgram, ExternBuffer, seq_state_elems
from .rotary import rotary_frequencies
from .safetensors import SafetensorsFile
from .session import LoweredProgram
from .state import SequenceStatePool, StateSpec
from .weights import WeightArena

ARCHITECTURE = "Fotovik"
DEFAULT_CONTEXT = 4096     # positions a sequence may reach where a layer keeps every position and the caller names no bound
MIXERS = ("attention", "delta", "parallel")
UNIT_EPS = 1e-6            # unit vectors of the delta rule: x / sqrt(sum x^2 + UNIT_EPS)
MAX_STATE_ROWS = 512       # key rows of a recurrent state the kernels hold per head


def _check_heads(i: int, m: dict):
    if min(m["heads"], m["kv_heads"], m["dim"], m["vdim"]) < 1 or m["heads"] % m["kv_heads"]:
        raise ValueError(f"layer {i}: sizes must be positive and heads a multiple of kv_heads")


def _check_attention(i: int, m: dict):
    _check_heads(i, m)
    rot = m.get("rot")
    if rot and (rot["dims"] % 2 or not 2 <= rot["dims"] <= m["dim"]):
        raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
    mask = m.get("mask")
    if mask and (mask["size"] < 1 or (mask.get("pool") is not None and mask["pool"] < 1)):
        raise ValueError(f"layer {i}: mask.size and mask.pool must be positive")


@dataclass(frozen=True)
class FotovikConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: Optional[dict]     # {"buckets", "mul_prev", "mul_cur"} or none
    layers: tuple              # of dicts: {"type", "mixer", "mlp"}
    runs: tuple                # of (layer, whether the embedding output joins the stream before it), in the order they run

    @classmethod
    def from_dict(cls, c: dict) -> "FotovikConfig":
        if c.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture = {c.get('architecture')!r}")
        layers = []
        for i, L in enumerate(c["layers"]):
            kind, m, mlp = L["type"], L["mixer"], L.get("mlp")
            if kind == "attention":
                _check_attention(i, m)
            elif kind == "delta":
                _check_heads(i, m)
                if m.get("conv", 1) < 1 or m["dim"] > MAX_STATE_ROWS:
                    raise ValueError(f"layer {i}: conv must be positive and dim at most {MAX_STATE_ROWS}")
            elif kind == "parallel":
                _check_attention(i, m["left"])
                r = m["right"]
                if min(r["heads"], r["dim"], r["vdim"]) < 1 or r["dim"] > MAX_STATE_ROWS or len(r["decay"]) != r["heads"]:
                    raise ValueError(f"layer {i}: one decay per head, dim at most {MAX_STATE_ROWS}")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append({"type": kind, "mixer": m, "mlp": mlp})
        n, loop = len(layers), c.get("loop")
        runs = [(i, False) for i in range(n)]
        if loop:
            a, b, times = loop["start"], loop["stop"], loop["times"]
            if not 0 <= a <= b <= n or times < 1:
                raise ValueError("loop: start .. stop - 1 must name layers of the stack, times at least 1")
            runs = runs[:a] + [(i, r > 0 and i == a) for r in range(times) for i in range(a, b)] + runs[b:]
        e = c.get("embedding") or {}
        bigram = e.get("bigram")
        if bigram and bigram["buckets"] < 1:
            raise ValueError("embedding.bigram: buckets must be positive")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(e.get("scale", 1.0)), bigram, tuple(layers), tuple(runs))

    @classmethod
    def from_json(cls, path: str) -> "FotovikConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))


class FotovikModel:
    """Weights resident in HBM (one arena per layer + one for the embeddings, the head and the final norm) and the lowering."""

    def __init__(self, be: CudaBackend, cfg: FotovikConfig, tensors, dtype: str = "bfloat16"):
        """tensors: name -> f32 array accessor (`tensors(name)`), e.g. SafetensorsFile.f32."""
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype must be 'bfloat16' or 'float32'")
        self.be, self.cfg, self.dtype = be, cfg, dtype
        self.wdt = abi.W_BF16 if dtype == "bfloat16" else abi.W_F32
        self.vocab, self.width = cfg.vocab, cfg.width
        self.layer_meta: List[dict] = []
        self.arenas: Dict[int, WeightArena] = {}
        self.buffers: Dict[int, DeviceBuffer] = {}
        self._freqs: Dict[int, DeviceBuffer] = {}      # per layer: frequencies of its rotary positions, f32
        self._decays: Dict[int, DeviceBuffer] = {}     # per layer: constant decays of its lightning heads, f32
        D = cfg.width

        def get(name, shape):
            t = tensors(name)
            assert tuple(t.shape) == tuple(shape), f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}"
            return t

        def table(values):      # f32 whatever the weight format; at least one 16-byte line
            a = np.zeros(max(4, len(values)), np.float32)
            a[:len(values)] = values
            buf = DeviceBuffer(be, a.nbytes, zero=False)
            buf.upload(a)
            return buf

        for i, L in enumerate(cfg.layers):
            p, m = f"l{i}.", L["mixer"]
            A = WeightArena(self.wdt)
            meta = {}
            A.add("norm1", get(p + "norm1", ()))
            A.add("norm1b", get(p + "norm1b", ()))

            def attention_parts(pre, m):
                H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
                return [get(pre + "q", (H * dim, D)), get(pre + "k", (G * dim, D)), get(pre + "v", (G * vdim, D))]

            if L["type"] == "attention":
                A.add("in", np.concatenate(attention_parts(p + "mix.", m), 0))
                A.add("sink", get(p + "mix.sink", (m["heads"],)))
                A.add("o", get(p + "mix.o", (D, m["heads"] * m["vdim"])))
                meta.update(n_in=m["heads"] * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"]))
                rot = m.get("rot")
            elif L["type"] == "delta":
                H, G, dim, vdim, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], int(m.get("conv") or 1)
                C, V = 2 * G * dim + H * vdim, H * vdim
                A.add("in", np.concatenate([get(p + "mix.q", (G * dim, D)), get(p + "mix.k", (G * dim, D)), get(p + "mix.v", (V, D)), get(p + "mix.g", (V, D)),
                                            get(p + "mix.b", (H, D)), get(p + "mix.a", (H, D))], 0))
                A.add("conv", np.concatenate([get(p + "mix.q.conv", (G * dim, taps)), get(p + "mix.k.conv", (G * dim, taps)), get(p + "mix.v.conv", (V, taps))], 0))
                A.add("A_log", get(p + "mix.A_log", (H,)))
                A.add("dt_bias", get(p + "mix.dt_bias", (H,)))
                A.add("norm", get(p + "mix.norm", (vdim,)))
                A.add("o", get(p + "mix.o", (D, V)))
                meta.update(n_in=C + V + 2 * H, C=C, taps=taps, g=C, b=C + V, a=C + V + H)
                rot = None
            else:
                l, r = m["left"], m["right"]
                Hr, dr, vr = r["heads"], r["dim"], r["vdim"]
                pl, pr = p + "mix.left.", p + "mix.right."
                C = l["heads"] * l["dim"] + l["kv_heads"] * (l["dim"] + l["vdim"])
                A.add("in", np.concatenate(attention_parts(pl, l) + [get(pr + "q", (Hr * dr, D)), get(pr + "k", (Hr * dr, D)), get(pr + "v", (Hr * vr, D)),
                                                                     get(pr + "g", (Hr * vr, D))], 0))
                A.add("q.norm", get(pl + "q.norm", (l["dim"],)))
                A.add("k.norm", get(pl + "k.norm", (l["dim"],)))
                A.add("left.o", get(pl + "o", (D, l["heads"] * l["vdim"])))
                A.add("right.norm", get(pr + "norm", (Hr * vr,)))
                A.add("right.o", get(pr + "o", (D, Hr * vr)))
                A.add("left.out", get(p + "mix.left.out", (D,)))
                A.add("right.out", get(p + "mix.right.out", (D,)))
                meta.update(n_in=C + 2 * Hr * dr + 2 * Hr * vr, rq=C, rk=C + Hr * dr, rv=C + 2 * Hr * dr, rg=C + 2 * Hr * dr + Hr * vr)
                rot = l.get("rot")
                self._decays[i] = table(r["decay"])
            if rot:
                self._freqs[i] = table(rotary_frequencies(rot))
            meta["row"] = (meta["n_in"] + 3) // 4 * 4      # rows of the stacked projection start on 16-byte boundaries
            if L["mlp"] is not None:
                ff = tensors(p + "mlp.up").shape[0]
                assert ff == L["mlp"].get("ff", ff), f"{p}mlp.up: {ff} rows, the configuration says {L['mlp'].get('ff')}"
                A.add("norm2", get(p + "norm2", ()))
                A.add("norm2b", get(p + "norm2b", ()))
                A.add("up", get(p + "mlp.up", (ff, D)))
                A.add("down", get(p + "mlp.down", (D, ff)))
                meta["ff"] = ff
            self.layer_meta.append(meta)
            self.arenas[i] = A
            self.buffers[i] = A.upload(be)
        A = WeightArena(self.wdt)
        A.add("embed", get("embed", (cfg.vocab, D)))
        if cfg.bigram:
            A.add("bigram", get("bigram", (cfg.bigram["buckets"] + 1, D)))
        A.add("final.norm", get("final.norm", ()))
        A.add("head", get("head", (cfg.vocab, D)))
        self.arenas[-1] = A
        self.buffers[-1] = A.upload(be)

    @classmethod
    def load(cls, be: CudaBackend, model_dir: str, dtype: str = "bfloat16") -> "FotovikModel":
        cfg = FotovikConfig.from_json(os.path.join(model_dir, "config.json"))
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
        """A layer that attends without a window keeps every position, one with pooled blocks every block: the session then bounds
        the sequence."""
        def unbounded(m):
            mask = m.get("mask")
            return mask is None or mask.get("pool") is not None
        return any(unbounded(L["mixer"] if L["type"] == "attention" else L["mixer"]["left"]) for L in self.cfg.layers if L["type"] != "delta")

    def capacity(self, max_chunk: int, max_context: Optional[int]) -> int:
        """Positions a sequence may reach where a layer keeps every position or block."""
        return max(int(max_context) if max_context else DEFAULT_CONTEXT, max_chunk)

    def _ring_rows(self, m: dict, max_chunk: int, max_context: Optional[int]) -> int:
        """Rows of a key ring: what a window reaches back (or a block spans) plus one step; every position where there is no window."""
        cap, mask = self.capacity(max_chunk, max_context), m.get("mask")
        return cap if mask is None else max(min(mask["size"] - 1, cap), mask.get("pool") or 0) + max_chunk

    def _scan_state_elems(self, r: dict) -> int:
        probe = DeviceOp.ssm_scan(0, 0, 0, None, 0, 0, 0, 0, 0, 0, 0, 0, 0, 1, r["heads"], r["heads"], r["dim"], r["vdim"], 1, 1, self.wdt, constant_decay=True)
        return seq_state_elems(probe)

    def state_specs(self, max_chunk: int, max_context: Optional[int] = None) -> List[StateSpec]:
        """Caches and states of every layer RUN: a layer that runs several times has one set per pass."""
        specs = []

        def caches(name, m):       # masked by position: no clearing
            width = m["kv_heads"] * (m["dim"] + m["vdim"])
            specs.append(StateSpec(name + ".kv", self._ring_rows(m, max_chunk, max_context) * width, False))
            pool = (m.get("mask") or {}).get("pool")
            if pool:
                specs.append(StateSpec(name + ".pooled", -(-self.capacity(max_chunk, max_context) // pool) * width, False))

        for n, (i, _) in enumerate(self.cfg.runs):
            L, name = self.cfg.layers[i], f"run{n}"
            m, meta = L["mixer"], self.layer_meta[i]
            if L["type"] == "attention":
                caches(name, m)
            elif L["type"] == "delta":
                if meta["taps"] > 1:
                    specs.append(StateSpec(name + ".tail", (meta["taps"] - 1) * meta["C"], True))
                specs.append(StateSpec(name + ".delta", m["heads"] * m["dim"] * m["vdim"], True))
            else:
                caches(name, m["left"])
                specs.append(StateSpec(name + ".lightning", self._scan_state_elems(m["right"]), True))
        return specs

    # ── lowering ──
    def lower(self, T: int, head: str, pool: SequenceStatePool, keep_layers: bool = False) -> LoweredProgram:
        cfg, wdt, D, eps = self.cfg, self.wdt, self.cfg.width, self.cfg.norm_eps
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
        emb, xs = new(TD), [new(TD), new(TD)]
        h, y = new(TD), new(TD)
        proj = new(T * max([m["row"] for m in self.layer_meta], default=1))
        shared: Dict[str, int] = {}

        def scratch(name, n):      # activations reused by every layer that needs them
            if name not in shared or sizes[shared[name]] < n:
                shared[name] = new(n)
            return shared[name]

        x = emb                    # the embedding output stays where it is: later passes of a loop add it again
        b = cfg.bigram
        ops.append(DeviceOp.embed(emb, ctl, gl, GA.off["embed"], T, D, cfg.embedding_scale, wdt,
                                  bigram=(GA.off["bigram"], b["buckets"], b["mul_prev"], b["mul_cur"]) if b else None))
        # The residual step that closes a sublayer waits for the norm that opens the next one: one launch for both.
        pending: List[dict] = []

        def step(**kw):            # x <- x + norm(src), chained with `then` where given
            nonlocal x
            nx = new(TD) if keep_layers else xs[1] if x == xs[0] else xs[0]
            ops.append(DeviceOp.norm(nx, rows=T, cols=D, eps=eps, wdt=wdt, res=x, **kw))
            x = nx

        def open_norm(dst, wb, w_off):
            if pending:
                step(then=dst, then_w=wb, then_w_off=w_off, then_kind="rms_scalar", **pending.pop())
            else:
                ops.append(DeviceOp.norm(dst, x, wb, w_off, T, D, eps, wdt, kind="rms_scalar"))

        def flush():
            if pending:
                step(**pending.pop())

        slots = pool.n_slots

        def attend(name, i, m, wb, A, order, layout, q_norm=0, k_norm=0, sink=None):
            """Heads of `proj` into the run's cache and attention over it; returns the buffer with the concatenated heads."""
            H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            rs, width, rot, mask = self.layer_meta[i]["row"], G * (dim + vdim), m.get("rot"), m.get("mask") or {}
            cache = pool.buffers[name + ".kv"]
            R = cache.elems // (slots * width)
            P = mask.get("pool") or 0
            pooled = pool.buffers[name + ".pooled"] if P else None
            blocks = dict(pooled=ext(pooled), pool=P, pool_rows=pooled.elems // (slots * width)) if P else {}
            turn = dict(norm_group=dim, normed=G * dim, q_heads=H, q_col=0, head_rot=rot["dims"], rot_layout=layout, freqs=ext(self._freqs[i]), order=order) if rot else {}
            if order == "norm_rotate":
                turn.update(norm_w=wb, norm_off=k_norm, q_norm_off=q_norm, normed=G * dim, norm_group=dim, q_heads=H, q_col=0)
                if not rot:
                    turn["order"] = "rotate_norm"      # nothing is turned: plain per-head norms
            ops.append(DeviceOp.cache_append(ext(cache), proj, ctl, H * dim, 0, T, width, rs, width, R, eps=eps, wdt=wdt, **turn, **blocks))
            att = scratch("att", T * H * vdim)
            kind = "pooled" if P else "window" if mask else "causal"
            ops.append(DeviceOp.cached_attention(att, proj, ext(cache), ext(cache), ctl, 0, 0, G * dim, T, H, G, 1, dim, vdim, rs, width, width, R, m["scale"],
                                                 mask=kind, mask_size=mask.get("size", 0), sink=wb if sink is not None else None, sink_off=sink or 0, sink_wdt=wdt, **blocks))
            return att

        layer_bufs = []
        for n, (i, rejoin) in enumerate(cfg.runs):
            L, name = cfg.layers[i], f"run{n}"
            m, meta, A, wb = L["mixer"], self.layer_meta[i], self.arenas[i], ext(self.buffers[i])
            if rejoin:             # a later pass of the loop: the embedding output joins the stream before its first layer
                flush()
                pending.append(dict(src=emb, w=None, w_off=0, kind="none"))
            open_norm(h, wb, A.off["norm1"])
            rs = meta["row"]
            close = dict(src=y, w=wb, w_off=A.off["norm1b"], kind="rms_scalar")
            if L["type"] == "attention":
                ops.append(DeviceOp.linear(proj, h, wb, A.off["in"], T, meta["n_in"], D, wdt, dst_rs=rs))
                att = attend(name, i, m, wb, A, "rotate", "pairs", sink=A.off["sink"])
                ops.append(DeviceOp.linear(y, att, wb, A.off["o"], T, D, m["heads"] * m["vdim"], wdt))
            elif L["type"] == "delta":
                H, G, dim, vdim, taps, C = m["heads"], m["kv_heads"], m["dim"], m["vdim"], meta["taps"], meta["C"]
                ops.append(DeviceOp.linear(proj, h, wb, A.off["in"], T, meta["n_in"], D, wdt, dst_rs=rs))
                qkv = scratch("conv", T * C)
                tail = ext(pool.buffers[name + ".tail"]) if taps > 1 else ctl    # one tap: no carried inputs, the operand is unused
                ops.append(DeviceOp.causal_conv(qkv, proj, wb, A.off["conv"], tail, ctl, T, C, taps, wdt, "silu", src_rs=rs))
                mix = scratch("mix", T * H * vdim)
                ops.append(DeviceOp.delta_rule(mix, qkv, proj, proj, proj, wb, ext(pool.buffers[name + ".delta"]), ctl, 0, G * dim, 2 * G * dim, meta["b"], A.off["A_log"],
                                               A.off["dt_bias"], A.off["norm"], T, H, G, dim, vdim, C, rs, rs, rs, wdt, eps, UNIT_EPS, dim ** -0.5, gate_off=meta["g"],
                                               silu_gate=True, head_decay=True, a_col=meta["a"]))
                ops.append(DeviceOp.linear(y, mix, wb, A.off["o"], T, D, H * vdim, wdt))
            else:
                l, r = m["left"], m["right"]
                Hr, dr, vr = r["heads"], r["dim"], r["vdim"]
                ops.append(DeviceOp.linear(proj, h, wb, A.off["in"], T, meta["n_in"], D, wdt, dst_rs=rs, act="silu", act_cols=(meta["rq"], meta["rg"])))
                att = attend(name, i, l, wb, A, "norm_rotate", "halves", q_norm=A.off["q.norm"], k_norm=A.off["k.norm"])
                ops.append(DeviceOp.linear(y, att, wb, A.off["left.o"], T, D, l["heads"] * l["vdim"], wdt))
                mix = scratch("mix", T * Hr * vr)
                ops.append(DeviceOp.ssm_scan(mix, proj, ext(self._decays[i]), None, ext(pool.buffers[name + ".lightning"]), ctl, meta["rv"], meta["rk"], meta["rq"], 0, 0, 0, 0,
                                             T, Hr, Hr, dr, vr, rs, 0, wdt, constant_decay=True))
                ops.append(DeviceOp.gated_norm(mix, mix, proj, wb, A.off["right.norm"], meta["rg"], T, Hr * vr, 1, rs, eps, wdt, gate_after=True, sigmoid_gate=True))
                y2 = scratch("right", TD)
                ops.append(DeviceOp.linear(y2, mix, wb, A.off["right.o"], T, D, Hr * vr, wdt))
                close = dict(src=y, w=wb, w_off=A.off["left.out"], kind="rms", src2=y2, src2_w_off=A.off["right.out"], gain=0.5, outer="rms_scalar",
                             outer_w_off=A.off["norm1b"])
            pending.append(close)
            if L["mlp"] is not None:
                ff = meta["ff"]
                open_norm(h, wb, A.off["norm2"])
                up = scratch("ff", T * ff)
                ops.append(DeviceOp.linear(up, h, wb, A.off["up"], T, ff, D, wdt, act="gelu_erf"))      # the activation rides in the epilogue
                ops.append(DeviceOp.linear(y, up, wb, A.off["down"], T, D, ff, wdt))
                pending.append(dict(src=y, w=wb, w_off=A.off["norm2b"], kind="rms_scalar"))
            if keep_layers:
                flush()
                layer_bufs.append(x)
        logits, rows = None, 0
        if head != "none":         # (a step that asks for no logits drops its last residual step)
            open_norm(h, gl, GA.off["final.norm"])
            rows = T if head == "all" else 1
            logits = new(rows * cfg.vocab)
            ops.append(DeviceOp.linear(logits, h, gl, GA.off["head"], rows, cfg.vocab, D, wdt, src_off=0 if head == "all" else (T - 1) * D))
        prog = DeviceProgram(ops, sizes, [], [], externs)
        return LoweredProgram(prog, ctl, logits, rows, layer_bufs if keep_layers else None)

    def close(self):
        for b in list(self.buffers.values()) + list(self._freqs.values()) + list(self._decays.values()):
            b.free()
        self.buffers, self._freqs, self._decays = {}, {}, {}


def synthetic_config(width: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int, vocab: int, window: int = 1024, pool: int = 32,
                     lightning_heads: Optional[int] = None, delta_heads: Optional[int] = None, conv: int = 4, loop: Optional[dict] = None) -> dict:
    """config.json contents of a random-init model: layers cycle the pair, window attention and the delta rule; every layer has a
    dense feed-forward."""
    layers = []
    for i in range(n_layers):
        kind = ("parallel", "attention", "delta")[i % 3]
        if kind == "parallel":
            left = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "rot": {"base": 10000.0, "dims": dim // 2, "scaling": {"factor": 2.0}}, "scale": dim ** -0.5, "vdim": dim}
            n = lightning_heads or max(1, heads // 2)
            mixer = {"left": left, "right": {"decay": [1.0 - 2.0 ** -(3.0 + 5.0 * h / n) for h in range(n)], "dim": dim, "heads": n, "vdim": dim}}
        elif kind == "attention":
            mixer = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"pool": pool, "size": window}, "rot": {"base": 10000.0, "dims": dim}, "scale": dim ** -0.5, "vdim": dim}
        else:
            n = delta_heads or heads
            mixer = {"conv": conv, "dim": dim, "heads": n, "kv_heads": max(1, n // 2), "vdim": dim}
        layers.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": ARCHITECTURE, "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": layers, "loop": loop,
            "embedding": {"scale": 1.0, "bigram": {"buckets": 4093, "mul_prev": 1009, "mul_cur": 31}}}


def synthetic_tensors(cfg: dict, seed: int = 0):
    """Accessor name -> random f32 tensor of the shape the configuration implies (benchmarks and smoke runs; values are scaled like a
    trained model's so that activations stay O(1))."""
    import zlib
    D = cfg["width"]

    def attention_shapes(m):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        return {"q": (H * d, D), "k": (G * d, D), "v": (G * dv, D), "q.norm": (d,), "k.norm": (d,), "sink": (H,), "o": (D, H * dv)}

    def shape_of(name):
        top = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, D)}
        if name in top:
            return top[name]
        layer, rest = name.split(".", 1)
        L = cfg["layers"][int(layer[1:])]
        m = L["mixer"]
        if rest.startswith("norm"):
            return ()
        if rest.startswith("mlp."):
            return {"up": (L["mlp"]["ff"], D), "down": (D, L["mlp"]["ff"])}[rest[4:]]
        t = rest[len("mix."):]
        if L["type"] == "attention":
            return attention_shapes(m)[t]
        if L["type"] == "delta":
            H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            return {"q": (G * d, D), "k": (G * d, D), "v": (H * dv, D), "q.conv": (G * d, taps), "k.conv": (G * d, taps), "v.conv": (H * dv, taps), "b": (H, D), "a": (H, D), "A_log": (H,),
                    "dt_bias": (H,), "norm": (dv,), "g": (H * dv, D), "o": (D, H * dv)}[t]
        if t.endswith(".out"):
            return (D,)
        if t.startswith("left."):
            return attention_shapes(m["left"])[t[5:]]
        H, d, dv = m["right"]["heads"], m["right"]["dim"], m["right"]["vdim"]
        return {"q": (H * d, D), "k": (H * d, D), "v": (H * dv, D), "g": (H * dv, D), "norm": (H * dv,), "o": (D, H * dv)}[t[6:]]

    def get(name):
        shp = shape_of(name)
        r = np.random.default_rng([seed, zlib.crc32(name.encode())])
        last = name.rsplit(".", 1)[-1]
        if last.startswith("norm") or last == "out":
            return np.ones(shp, np.float32)
        if last == "conv":
            a = (r.random(shp, dtype=np.float32) - 0.5) * 0.5
            a[:, -1] += 1.0
            return a
        if last in ("A_log", "dt_bias"):
            return (-3.0 + 2.0 * r.random(shp, dtype=np.float32)).astype(np.float32)
        if last == "sink":
            return (r.random(shp, dtype=np.float32) * 0.2).astype(np.float32)
        a = r.random(shp, dtype=np.float32)
        a -= 0.5
        a *= np.float32(np.sqrt(12.0 / (1 if name in ("embed", "bigram") else shp[-1])))
        return a

    return get
