// What the recurrent mixers' short convolutions share: vectors of neighbouring channels, the step's tables, and a causal
// convolution per channel over a request's tokens.
#pragma once

#include "common.cuh"

template <int V> struct ChanVec { float v[V]; };
template <typename T, int V> __device__ __forceinline__ ChanVec<V> chan_load(const T* p) {
    ChanVec<V> r;
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 q = *reinterpret_cast<const uint2*>(p);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
        r.v[0] = lo.x; r.v[1] = lo.y; r.v[2] = hi.x; r.v[3] = hi.y;
    } else if constexpr (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    } else {
        r.v[0] = to_f32<T>(*p);
    }
    return r;
}
template <typename T, int V> __device__ __forceinline__ void chan_store(T* p, const ChanVec<V>& r) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 q;
        q.x = *reinterpret_cast<const unsigned*>(&lo);
        q.y = *reinterpret_cast<const unsigned*>(&hi);
        *reinterpret_cast<uint2*>(p) = q;
    } else if constexpr (V == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    } else {
        *p = from_f32<T>(r.v[0]);
    }
}
// May rows of `elem`-byte elements at p be read four elements at a time?
static inline bool chan_aligned(const void* p, long ld, int elem) { return ((uintptr_t)p % (4 * elem)) == 0 && ld % 4 == 0; }

__device__ __forceinline__ float fl_silu(float v) { return v / (1.0f + expf(-v)); }

struct StepTables {              // per token: its request and position; per request: first row, context, tokens, slot
    const int *tok_req, *positions, *req_start, *req_ctx, *req_qlen, *req_slot;
};

// A causal convolution on V channels from `c` on, at the RUN (at most) consecutive tokens t0 .. t1 - 1 of the step; TAPS: the
// window's length (the convolution's taps rounded up).  col: the channels' column of the step's rows; conv_w: [taps][channels]
// float, the last row the current token's.  The taps - 1 inputs before a request's first token of the step come from its kept
// rows [taps - 1][channels] float, oldest first; inputs before the sequence's start are zeros.
//   emit(t, y, in)    y: the convolution at token t (no bias); in[k]: the input of position pos - (TAPS - 1) + k, in[TAPS - 1]
//                     being the token's own
// All inputs of a run within one request are asked for before the first is used.
template <typename T, int V, int TAPS, int RUN> struct ShortConv {
    static constexpr int WIN = TAPS - 1;
    float w[TAPS][V];

    __device__ __forceinline__ void start(const float* conv_w, int taps, int channels, int c) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const int k = j - (TAPS - taps);
            ChanVec<V> tap = {};
            if (k >= 0) tap = chan_load<float, V>(conv_w + (long)k * channels + c);
#pragma unroll
            for (int e = 0; e < V; ++e) w[j][e] = tap.v[e];
        }
    }
    // The input `back` tokens before the one of row t, at position pos, whose request has `ctx` tokens before the step.
    __device__ __forceinline__ ChanVec<V> before(const T* col, long ld, int t, int back, int pos, int ctx, const float* kept,
                                                 int taps, int channels) const {
        const int p = pos - back;
        ChanVec<V> in = {};
        if (p >= 0 && back <= taps - 1) {
            if (p >= ctx) in = chan_load<T, V>(col + (long)(t - back) * ld);
            else in = chan_load<float, V>(kept + (long)(p - ctx + taps - 1) * channels);
        }
        return in;
    }
    __device__ __forceinline__ ChanVec<V> sum(const ChanVec<V>* in) const {
        ChanVec<V> y = {};
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) y.v[e] = fmaf(w[j][e], in[j].v[e], y.v[e]);
        return y;
    }
    template <typename F>
    __device__ __forceinline__ void run(int t0, int t1, const T* col, long ld, const StepTables& st, const float* tail,
                                        long tail_stride, int taps, int channels, int c, F emit) const {
        const int r = WIN > 0 ? st.tok_req[t0] : 0;
        if (RUN == 1 || WIN == 0 || (t1 - t0 == RUN && st.tok_req[t1 - 1] == r)) {
            ChanVec<V> in[WIN + RUN];
            if (WIN > 0) {
                const int pos = st.positions[t0], ctx = st.req_ctx[r];
                const float* kept = tail + (long)st.req_slot[r] * tail_stride + c;
#pragma unroll
                for (int k = 0; k < WIN; ++k) in[k] = before(col, ld, t0, WIN - k, pos, ctx, kept, taps, channels);
            }
#pragma unroll
            for (int i = 0; i < RUN; ++i)
                if (RUN == 1 || t0 + i < t1) in[WIN + i] = chan_load<T, V>(col + (long)(t0 + i) * ld);
#pragma unroll
            for (int i = 0; i < RUN; ++i)
                if (RUN == 1 || t0 + i < t1) emit(t0 + i, sum(in + i), in + i);
            return;
        }
        if constexpr (RUN > 1 && WIN > 0) {
            for (int t = t0; t < t1; ++t) {                               // a run across requests, or at the step's end
                const int rt = st.tok_req[t], pos = st.positions[t], ctx = st.req_ctx[rt];
                const float* kept = tail + (long)st.req_slot[rt] * tail_stride + c;
                ChanVec<V> in[TAPS];
#pragma unroll
                for (int k = 0; k < WIN; ++k) in[k] = before(col, ld, t, WIN - k, pos, ctx, kept, taps, channels);
                in[WIN] = chan_load<T, V>(col + (long)t * ld);
                emit(t, sum(in), in);
            }
        }
    }
};
