// Sequence-model DeviceOp ZG_OP_STREAM_STEP (parameter pack in include/zgml_cuda.h): the residual step of a stack that carries several
// streams side by side (hyper-connections).  One launch closes a sublayer — every new stream is a mixture of the old ones plus its
// share of the sublayer's result — and opens the next: a weighted sum of the new streams, a Dynamic Tanh, and, for mixers that blend
// every token's input with the one before, the token-shifted copies of it.  All f32.
//
// Nothing here needs statistics of a row, so a thread owns one column (or four neighbours) and walks a few rows of it: the new streams
// never leave its registers between the close and the open, and the row before — which a token shift needs — is the one it just
// computed.  The first row of a walk takes its predecessor from the carried state (row 0) or computes it again from the old streams.
#include "seq_common.cuh"

namespace {

constexpr int kStMaxStreams = 16, kStMaxShifts = 8;
struct StArgs {
    float* dst; const float* src; const float* y; float* h; float* state; const float* ctl;
    uint32_t T, D, streams, stride, kind, shifts, rows;      // stride: between the old streams; rows: walked by one thread
    float mult, gain;
};
template <typename WT, int V>
__device__ __forceinline__ void st_weights(float (&out)[V], const WT* __restrict__ w) {
    if constexpr (V == 1) out[0] = wld(w, 0);
    else if constexpr (sizeof(WT) == 2) {
        const uint2 v = *reinterpret_cast<const uint2*>(w);
        out[0] = __uint_as_float(v.x << 16); out[1] = __uint_as_float(v.x & 0xFFFF0000u);
        out[2] = __uint_as_float(v.y << 16); out[3] = __uint_as_float(v.y & 0xFFFF0000u);
    } else {
        const float4 v = *reinterpret_cast<const float4*>(w);
        out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
    }
}
template <int V>
__device__ __forceinline__ void st_load(float (&out)[V], const float* __restrict__ p) {
    if constexpr (V == 1) out[0] = p[0];
    else { const float4 v = *reinterpret_cast<const float4*>(p); out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w; }
}
template <int V>
__device__ __forceinline__ void st_store(float* __restrict__ p, const float (&v)[V]) {
    if constexpr (V == 1) p[0] = v[0];
    else *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
// S: the number of streams, or (S = kStMaxStreams) an upper bound of it; V: columns per thread; SHIFT: the open is token-shifted
template <typename WT, int S, int V, bool SHIFT>
__global__ void __launch_bounds__(128) k_stream_step(StArgs a, const WT* __restrict__ w_out, const WT* __restrict__ w_mix, const WT* __restrict__ w_ls,
                                                      const WT* __restrict__ w_in, const WT* __restrict__ w_norm, const WT* __restrict__ w_mu) {
    // Weights are constants of the model and are read before the wait on the predecessor.
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const uint32_t n = S < kStMaxStreams ? S : a.streams;
    const uint32_t c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const bool on = c < a.D, close = a.y != nullptr, open = a.h != nullptr, tanh_norm = a.kind & 8u;
    __shared__ float s_mix[kStMaxStreams * kStMaxStreams], s_out[kStMaxStreams], s_in[kStMaxStreams];
    if (close) {
        for (uint32_t i = threadIdx.x; i < n * n; i += blockDim.x) s_mix[i] = wld(w_mix, i);
        for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) s_out[i] = a.mult * wld(w_out, i);
    }
    if (open) for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) s_in[i] = wld(w_in, i);
    float ls[V], nw[V], nb[V], mu[SHIFT ? kStMaxShifts : 1][V];
    float alpha = 0.0f;
#pragma unroll
    for (int i = 0; i < V; i++) { ls[i] = 1.0f; nw[i] = 1.0f; nb[i] = 0.0f; }
    if (on) {
        if (close && w_ls) st_weights<WT, V>(ls, w_ls + c);
        if (open && tanh_norm) { st_weights<WT, V>(nw, w_norm + c); st_weights<WT, V>(nb, w_norm + a.D + c); alpha = wld(w_norm, (size_t)2 * a.D); }
        if constexpr (SHIFT) {
#pragma unroll
            for (int j = 0; j < kStMaxShifts; j++)
                if (j < (int)a.shifts) st_weights<WT, V>(mu[j], w_mu + (size_t)j * a.D + c);
        }
    }
    __syncthreads();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    if (!on) return;
    const size_t TD = (size_t)a.T * a.D;
    // row t: new streams (written when `write`) and the opened input of the next sublayer
    auto row = [&](uint32_t t, bool write, float (&h)[V]) {
        const size_t at = (size_t)t * a.D + c;
        float x[S][V], yv[V], u[V];
#pragma unroll
        for (int s = 0; s < S; s++)
            if (s < (int)n) st_load<V>(x[s], a.src + (size_t)s * a.stride + at);
        if (close) {
            st_load<V>(yv, a.y + at);
#pragma unroll
            for (int i = 0; i < V; i++) yv[i] *= ls[i];
        }
#pragma unroll
        for (int i = 0; i < V; i++) u[i] = 0.0f;
#pragma unroll
        for (int b = 0; b < S; b++) {
            if (b >= (int)n) break;
            float v[V];
            if (close) {
                const float o = s_out[b];
#pragma unroll
                for (int i = 0; i < V; i++) v[i] = o * yv[i];
#pragma unroll
                for (int s = 0; s < S; s++) {
                    if (s >= (int)n) break;
                    const float m = s_mix[s * n + b];
#pragma unroll
                    for (int i = 0; i < V; i++) v[i] = fmaf(m, x[s][i], v[i]);
                }
                if (write) st_store<V>(a.dst + (size_t)b * TD + at, v);
            } else {
#pragma unroll
                for (int i = 0; i < V; i++) v[i] = x[b][i];
            }
            if (open) {
                const float w = s_in[b];
#pragma unroll
                for (int i = 0; i < V; i++) u[i] = fmaf(w, v[i], u[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < V; i++) h[i] = (tanh_norm ? fmaf(tanhf(alpha * u[i]), nw[i], nb[i]) : u[i]) * a.gain;
    };
    const uint32_t t0 = blockIdx.y * a.rows, t1 = min(a.T, t0 + a.rows);
    if constexpr (SHIFT) {
        float prev[V], h[V];
        float* st = a.state + (size_t)ctl_word(a.ctl, ZG_CTL_SLOT) * a.D + c;
        if (t0 == 0) st_load<V>(prev, st); else row(t0 - 1, false, prev);
        for (uint32_t t = t0; t < t1; t++) {
            row(t, true, h);
            float* out = a.h + (size_t)t * a.shifts * a.D + c;
#pragma unroll
            for (int j = 0; j < kStMaxShifts; j++) {
                if (j >= (int)a.shifts) break;
                float o[V];
#pragma unroll
                for (int i = 0; i < V; i++) o[i] = fmaf(prev[i] - h[i], mu[j][i], h[i]);
                st_store<V>(out + (size_t)j * a.D, o);
            }
#pragma unroll
            for (int i = 0; i < V; i++) prev[i] = h[i];
        }
        // the thread that read the carried row also replaces it: no other one touches it
        if (t0 == 0) {
            if (t1 < a.T) row(a.T - 1, false, prev);
            st_store<V>(st, prev);
        }
    } else {
        for (uint32_t t = t0; t < t1; t++) {
            float h[V];
            row(t, true, h);
            if (open) st_store<V>(a.h + (size_t)t * a.D + c, h);
        }
    }
}

template <typename WT, int S, int V>
void st_launch(const StArgs& a, dim3 grid, cudaStream_t st, const WT* w_out, const WT* w_mix, const WT* w_ls, const WT* w_in, const WT* w_norm, const WT* w_mu) {
    if (a.shifts) launch_pdl(k_stream_step<WT, S, V, true>, grid, dim3(128), 0, st, a, w_out, w_mix, w_ls, w_in, w_norm, w_mu);
    else launch_pdl(k_stream_step<WT, S, V, false>, grid, dim3(128), 0, st, a, w_out, w_mix, w_ls, w_in, w_norm, w_mu);
}

}  // namespace

bool zg_stream_op_valid(const ZgOp& op, const size_t* elems, size_t n_bufs, char* why, size_t why_n) {
    const ZgSeqOp& s = op.u.seq;
    auto fail = [&](const char* m) { snprintf(why, why_n, "%s", m); return false; };
    auto have = [&](int i) { return s.buf[i] != ZG_NO_BUF && s.buf[i] < n_bufs; };
    auto fits = [&](int i, size_t off, size_t n) { return have(i) && off + n <= elems[s.buf[i]]; };
    auto wfits = [&](int i, size_t off, size_t n) { return have(i) && (s.n[4] == ZG_W_BF16 ? (off + n + 1) / 2 : off + n) <= elems[s.buf[i]]; };
    if (op.tag != ZG_OP_STREAM_STEP) return fail("not a sequence op");
    const size_t T = s.n[0], D = s.n[1], S = s.n[2], stride = s.n[3];
    const bool close = s.buf[2] != ZG_NO_BUF, open = s.buf[5] != ZG_NO_BUF;
    if (!T || !D || !S || S > kStMaxStreams || s.n[4] > ZG_W_BF16 || (stride && stride < T * D) || (!close && !open) || s.n[6] > kStMaxShifts || s.n[7] > 1) return fail("stream_step: shape");
    if (!fits(1, 0, (S - 1) * stride + T * D)) return fail("stream_step: streams");
    if (close && (!fits(0, 0, S * T * D) || !fits(2, 0, T * D) || !wfits(3, s.off[0], S) || !wfits(3, s.off[1], S * S) || (s.n[7] && !wfits(3, s.off[2], D)) || s.buf[0] == s.buf[1] || s.buf[0] == s.buf[2]))
        return fail("stream_step: close");
    if (open && (!fits(5, 0, T * D * (s.n[6] ? s.n[6] : 1)) || !wfits(4, s.off[3], S) || (s.n[5] != 8 && s.n[5] != 16) || (s.n[5] == 8 && !wfits(4, s.off[4], 2 * D + 1)) || s.buf[5] == s.buf[1] ||
                 s.buf[5] == s.buf[2] || (close && s.buf[5] == s.buf[0])))
        return fail("stream_step: open");
    if (s.n[6] && (!open || !wfits(4, s.off[5], s.n[6] * D) || !have(6) || elems[s.buf[6]] < D || !fits(7, 0, ZG_CTL_IDS))) return fail("stream_step: token shift");
    return true;
}

bool zg_launch_stream_op(const ZgOp& op, float* const* bufs, cudaStream_t st) {
    const ZgSeqOp& s = op.u.seq;
    const bool close = s.buf[2] != ZG_NO_BUF, open = s.buf[5] != ZG_NO_BUF;
    auto ptr = [&](int i) { return s.buf[i] != ZG_NO_BUF ? bufs[s.buf[i]] : (float*)nullptr; };
    StArgs a;
    a.dst = ptr(0); a.src = bufs[s.buf[1]]; a.y = ptr(2); a.h = ptr(5); a.state = ptr(6); a.ctl = ptr(7);
    a.T = s.n[0]; a.D = s.n[1]; a.streams = s.n[2]; a.stride = s.n[3]; a.kind = s.n[5]; a.shifts = s.n[6]; a.mult = s.f[0]; a.gain = s.f[1];
    a.rows = a.shifts && a.T > 4 ? 4 : 1;              // a token shift computes the row before each walk once more
#define ZG_ST(S_)                                                                                  \
    do {                                                                                           \
        if (vec) st_launch<WT, S_, 4>(a, grid, st, w_out, w_mix, w_ls, w_in, w_norm, w_mu);        \
        else st_launch<WT, S_, 1>(a, grid, st, w_out, w_mix, w_ls, w_in, w_norm, w_mu);            \
    } while (0)
    ZG_SEQ_WDT(s.n[4], {
        const WT* w_out = close ? wptr<WT>(bufs, s.buf[3], s.off[0]) : nullptr;
        const WT* w_mix = close ? wptr<WT>(bufs, s.buf[3], s.off[1]) : nullptr;
        const WT* w_ls = close && s.n[7] ? wptr<WT>(bufs, s.buf[3], s.off[2]) : nullptr;
        const WT* w_in = open ? wptr<WT>(bufs, s.buf[4], s.off[3]) : nullptr;
        const WT* w_norm = open && s.n[5] == 8 ? wptr<WT>(bufs, s.buf[4], s.off[4]) : nullptr;
        const WT* w_mu = a.shifts ? wptr<WT>(bufs, s.buf[4], s.off[5]) : nullptr;
        const uintptr_t acts = (uintptr_t)a.dst | (uintptr_t)a.src | (uintptr_t)a.y | (uintptr_t)a.h | (uintptr_t)a.state, ws = (uintptr_t)w_ls | (uintptr_t)w_norm | (uintptr_t)w_mu;
        const bool vec = a.D % 4 == 0 && a.stride % 4 == 0 && (acts & 15) == 0 && (ws & (4 * sizeof(WT) - 1)) == 0 && a.T >= 8;   // few rows: a thread per column fills more SMs
        const dim3 grid((a.D / (vec ? 4 : 1) + 127) / 128, (a.T + a.rows - 1) / a.rows);
        switch (a.streams) {
            case 1: ZG_ST(1); break;
            case 2: ZG_ST(2); break;
            case 3: ZG_ST(3); break;
            case 4: ZG_ST(4); break;
            default: ZG_ST(kStMaxStreams); break;
        }
    });
#undef ZG_ST
    ZG_SEQ_CHECK();
    return true;
}
