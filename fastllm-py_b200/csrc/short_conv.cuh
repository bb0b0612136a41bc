// What the recurrent mixers' short convolutions share: vectors of neighbouring channels, the step's tables, and a causal
// convolution per channel whose window slides along a request's tokens in registers.
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
__device__ __forceinline__ float fl_softplus(float v) { return v > 20.0f ? v : log1pf(expf(v)); }

struct StepTables {              // per token: its request and position; per request: first row, context, tokens, slot
    const int *tok_req, *positions, *req_start, *req_ctx, *req_qlen, *req_slot;
};

// V channels from `c` on; TAPS: the window's length (the convolution's taps rounded up).  The taps - 1 inputs before a
// request's first token of the step come from its kept rows [taps - 1][channels] float, oldest first; inputs before the
// sequence's start are zeros.
template <typename T, int V, int TAPS> struct ShortConv {
    static constexpr int WIN = TAPS > 1 ? TAPS - 1 : 1;
    ChanVec<V> w[TAPS], win[WIN];
    int known;
    // conv_w: [taps][channels], the last row the current token's
    __device__ __forceinline__ void start(const float* conv_w, int taps, int channels, int c) {
        known = -1;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const int k = j - (TAPS - taps);
            if (k >= 0) w[j] = chan_load<float, V>(conv_w + (long)k * channels + c);
            else
#pragma unroll
                for (int e = 0; e < V; ++e) w[j].v[e] = 0.0f;
        }
    }
    // The convolution at token t, whose input is x (tokens come in order); col: the channels' column of the step's rows.
    __device__ __forceinline__ ChanVec<V> at(int t, const ChanVec<V>& x, const T* col, long ld, const StepTables& st,
                                             const float* tail, long tail_stride, int taps, int channels, int c) {
        ChanVec<V> y;
#pragma unroll
        for (int e = 0; e < V; ++e) y.v[e] = 0.0f;
        if constexpr (TAPS > 1) {
            const int r = st.tok_req[t];
            if (r != known) {
                known = r;
                const int pos = st.positions[t], ctx = st.req_ctx[r];
                const float* kept = tail + (long)st.req_slot[r] * tail_stride + c;
#pragma unroll
                for (int k = 0; k < WIN; ++k) {
                    const int back = WIN - k, p = pos - back;         // window entry k holds position pos - WIN + k
#pragma unroll
                    for (int e = 0; e < V; ++e) win[k].v[e] = 0.0f;
                    if (p < 0 || back > taps - 1) continue;
                    if (p >= ctx) win[k] = chan_load<T, V>(col + (long)(t - back) * ld);
                    else win[k] = chan_load<float, V>(kept + (long)(p - ctx + taps - 1) * channels);
                }
            }
#pragma unroll
            for (int j = 0; j < WIN; ++j)
#pragma unroll
                for (int e = 0; e < V; ++e) y.v[e] = fmaf(w[j].v[e], win[j].v[e], y.v[e]);
#pragma unroll
            for (int j = 0; j + 1 < WIN; ++j) win[j] = win[j + 1];
            win[WIN - 1] = x;
        }
#pragma unroll
        for (int e = 0; e < V; ++e) y.v[e] = fmaf(w[TAPS - 1].v[e], x.v[e], y.v[e]);
        return y;
    }
};
