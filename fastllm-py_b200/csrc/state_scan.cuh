// The recurrence that linear-attention-like mixers share: per request and head a matrix state S [n x p] in float,
//
//     S <- a S + k (dt v)^T,    y = S^T q (+ skip v)
//
// walked over the request's tokens in order.  The decay a is one number per token (SCALAR: it and the step size dt come
// from the token) or one per row of S and token (dt = 1).  Tokens are float rows in which k, q, a and v of a head lie at
// given columns; heads may share k and q in groups.  A request's state row holds [heads][p][n] (a column of S is
// contiguous); it is read unless the request starts (context 0) and written at the end.
//
// A block takes one request, one head and COLS columns of S.  LANES lanes share four columns; a lane holds R rows of each in
// its registers: the groups of four rows lane + LANES i, so that the lanes read consecutive 16 bytes of a staged row
// (n <= LANES R; rows beyond n stay zero).  Neighbouring rows are packed pairs of floats, which one instruction of the
// float pipe works on.  Tokens come through four stages of shared memory, three chunks being copied (cp.async) while one is
// walked; they go four at a time, so that the read-out sums of four tokens and four columns are added up over the lanes
// together, each exchange halving what a lane still holds.  Tokens beyond the portion's end leave S as it is (decay 1,
// nothing added).  R and LANES follow from n alone, so every result's order of sums is fixed by the sizes: cuts and batches
// agree bit for bit.
#pragma once

#include "common.cuh"

#define SCAN_STAGES 4
#define SCAN_CPT 4                   // columns of S that a thread holds rows of

struct ScanToken {                   // columns of a token's row, and how heads step through them
    int k0, q0, n_step, per_group;   // head h's k and q: at k0 / q0 + (h / per_group) * n_step
    int a0, v0;                      // its row decays at a0 + h * n (not SCALAR), its values at v0 + h * p
    int dt0, decay0;                 // SCALAR: step size and decay at dt0 + h, decay0 + h
};

__device__ __forceinline__ void scan_cp4(void* smem, const void* gmem) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void scan_cp16(void* smem, const void* gmem) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem));
}

// Two floats in one register pair: one instruction of the float pipe works on both (each rounded to nearest).
typedef unsigned long long scan_f2;
__device__ __forceinline__ scan_f2 scan_pack(float a, float b) {
    scan_f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 scan_unpack(scan_f2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ scan_f2 scan_fma2(scan_f2 a, scan_f2 b, scan_f2 c) {
    scan_f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ scan_f2 scan_mul2(scan_f2 a, scan_f2 b) {
    scan_f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// Keeps the half of a lane's values that `up` names and adds the other lane's to it.
__device__ __forceinline__ float scan_fold(bool up, float low, float high, int off) {
    return (up ? high : low) + __shfl_xor_sync(0xffffffffu, up ? low : high, off);
}

template <int R, int LANES, int COLS, bool SCALAR, int CHUNK>
__global__ void __launch_bounds__(COLS / SCAN_CPT * LANES, 1) state_scan_kernel(
    const float* __restrict__ rows, long ld, const ScanToken at, const float* __restrict__ skip, float* __restrict__ y,
    long y_ld, float* __restrict__ state, long state_stride, const int* __restrict__ req_start,
    const int* __restrict__ req_ctx, const int* __restrict__ req_qlen, const int* __restrict__ req_slot, int n, int p,
    int vec4, int state_vec4) {
    constexpr int CPT = SCAN_CPT;
    static_assert(CHUNK % 4 == 0 && R % 4 == 0 && (LANES == 8 || LANES == 16) && CPT == 4, "");
    pdl_wait();
    constexpr int DP = R * LANES, VECS = SCALAR ? 2 : 3;              // a staged token: k | q | (a) | v | (dt, decay)
    constexpr int TOKEN = VECS * DP + COLS + 4;
    extern __shared__ __align__(16) float scan_s[];
    const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, lane = tid & (LANES - 1), cg = tid / LANES * CPT;
    const int start = req_start[r], qlen = req_qlen[r];
    const bool fresh = req_ctx[r] == 0;
    const int cols = min(COLS, p - col0);
    const int k_at = at.k0 + h / at.per_group * at.n_step, q_at = at.q0 + h / at.per_group * at.n_step;
    const int a_at = at.a0 + h * n, v_at = at.v0 + h * p + col0;
    // padding stays zero, and so do the places of tokens behind the portion's end
    const int staged = min(SCAN_STAGES * CHUNK, (qlen + 3) / 4 * 4);
    for (int i = tid; i < staged * (TOKEN / 4); i += blockDim.x)
        reinterpret_cast<float4*>(scan_s)[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float* srow = state + (long)req_slot[r] * state_stride + ((long)h * p + col0 + cg) * n;
    scan_f2 S[CPT][R / 2];
#pragma unroll
    for (int k = 0; k < CPT; ++k)
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int d = 4 * (lane + LANES * i);
            const bool mine = !fresh && cg + k < cols;
            float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (state_vec4) {
                if (mine && d < n) v = *reinterpret_cast<const float4*>(srow + (long)k * n + d);
            } else if (mine) {
                if (d < n) v.x = srow[(long)k * n + d];
                if (d + 1 < n) v.y = srow[(long)k * n + d + 1];
                if (d + 2 < n) v.z = srow[(long)k * n + d + 2];
                if (d + 3 < n) v.w = srow[(long)k * n + d + 3];
            }
            S[k][2 * i] = scan_pack(v.x, v.y);
            S[k][2 * i + 1] = scan_pack(v.z, v.w);
        }
    const float skip_h = skip != nullptr ? skip[h] : 0.0f;
    __syncthreads();
    // a thread copies the same places of every token: where they come from and go to is worked out once a chunk
    auto load = [&](int stage, int c0) {
        float* dst = scan_s + stage * CHUNK * TOKEN;
        const int here = min(CHUNK, qlen - c0);
        const float* src = rows + (long)(start + c0) * ld;
        const int unit = vec4 ? 4 : 1;
        const int nu = n / unit, per = VECS * nu + cols / unit;
        for (int e = tid; e < per; e += blockDim.x) {
            int from, to;
            if (e < nu) { from = k_at + unit * e; to = unit * e; }
            else if (e < 2 * nu) { from = q_at + unit * (e - nu); to = DP + unit * (e - nu); }
            else if (!SCALAR && e < 3 * nu) { from = a_at + unit * (e - 2 * nu); to = 2 * DP + unit * (e - 2 * nu); }
            else { from = v_at + unit * (e - VECS * nu); to = VECS * DP + unit * (e - VECS * nu); }
            const float* s = src + from;
            float* d = dst + to;
            if (vec4) {
#pragma unroll 4
                for (int tt = 0; tt < here; ++tt, s += ld, d += TOKEN) scan_cp16(d, s);
            } else {
                for (int tt = 0; tt < here; ++tt, s += ld, d += TOKEN) scan_cp4(d, s);
            }
        }
        if (SCALAR)
            for (int i = tid; i < 2 * here; i += blockDim.x)
                scan_cp4(dst + (i >> 1) * TOKEN + VECS * DP + COLS + (i & 1), src + (long)(i >> 1) * ld + ((i & 1) ? at.decay0 : at.dt0) + h);
        asm volatile("cp.async.commit_group;");
    };
    // one group of copies per chunk, empty ones beyond the end: waiting for all but the last STAGES - 1 means this one landed
#pragma unroll
    for (int s = 0; s < SCAN_STAGES - 1; ++s) {
        if (s * CHUNK < qlen) load(s, s * CHUNK); else asm volatile("cp.async.commit_group;");
    }
    // the token of a group of four and the (first) column whose sum this lane is left with
    constexpr int REM = LANES / 4;                                    // lanes that share one token's sums
    constexpr int LEFT = 4 / REM;                                     // sums a lane is left with (1 or 2)
    const int my_u = lane / REM, my_k = LEFT * (lane & (REM - 1));
    float* yp = y + (long)(start + my_u) * y_ld + (long)h * p + col0 + cg + my_k;
    int stage = 0;
    for (int c0 = 0; c0 < qlen; c0 += CHUNK, stage = (stage + 1) % SCAN_STAGES) {
        const int here = min(CHUNK, qlen - c0), ahead = c0 + (SCAN_STAGES - 1) * CHUNK;
        // (the stage copied into now was walked in the last round, behind that round's closing barrier)
        if (ahead < qlen) load((stage + SCAN_STAGES - 1) % SCAN_STAGES, ahead); else asm volatile("cp.async.commit_group;");
        asm volatile("cp.async.wait_group %0;" ::"n"(SCAN_STAGES - 1));
        __syncthreads();                                              // this chunk has landed
        const float* tok = scan_s + stage * CHUNK * TOKEN;
        // four tokens from `tok` on, of which the first `left` are the portion's (whole: all of them are)
        auto group = [&](const float* tok, float* yp, int left, bool whole) {
            // the rows of AHEAD tokens are read into registers before the first of them is used
            constexpr int AHEAD = VECS * R <= 16 ? 4 : VECS * R <= 32 ? 2 : 1;
            float acc[4][CPT];
#pragma unroll
            for (int u0 = 0; u0 < 4; u0 += AHEAD) {
                ulonglong2 kk[AHEAD][R / 4], qq[AHEAD][R / 4], aa[AHEAD][R / 4];
                float x[AHEAD][CPT];
                scan_f2 a2[AHEAD] = {};
#pragma unroll
                for (int w = 0; w < AHEAD; ++w) {
                    const float* tu = tok + (u0 + w) * TOKEN;
                    const bool real = whole || u0 + w < left;
#pragma unroll
                    for (int i = 0; i < R / 4; ++i) {
                        kk[w][i] = reinterpret_cast<const ulonglong2*>(tu)[lane + LANES * i];
                        qq[w][i] = reinterpret_cast<const ulonglong2*>(tu + DP)[lane + LANES * i];
                        if (!SCALAR) {
                            aa[w][i] = reinterpret_cast<const ulonglong2*>(tu + 2 * DP)[lane + LANES * i];
                            if (!real) aa[w][i] = make_ulonglong2(scan_pack(1.0f, 1.0f), scan_pack(1.0f, 1.0f));
                        }
                    }
                    const float4 v = *reinterpret_cast<const float4*>(tu + VECS * DP + cg);
                    x[w][0] = v.x; x[w][1] = v.y; x[w][2] = v.z; x[w][3] = v.w;
                    float dt = real ? 1.0f : 0.0f;
                    if (SCALAR) {
                        const float2 rate = *reinterpret_cast<const float2*>(tu + VECS * DP + COLS);
                        dt = real ? rate.x : 0.0f;
                        const float decay = real ? rate.y : 1.0f;
                        a2[w] = scan_pack(decay, decay);
                    }
#pragma unroll
                    for (int k = 0; k < CPT; ++k) x[w][k] *= dt;
                }
#pragma unroll
                for (int w = 0; w < AHEAD; ++w) {
                    scan_f2 x2[CPT], sum[CPT];
#pragma unroll
                    for (int k = 0; k < CPT; ++k) x2[k] = scan_pack(x[w][k], x[w][k]);
#pragma unroll
                    for (int i = 0; i < R / 4; ++i) {
                        const scan_f2 ax = SCALAR ? a2[w] : aa[w][i].x, ay = SCALAR ? a2[w] : aa[w][i].y;
#pragma unroll
                        for (int k = 0; k < CPT; ++k) {
                            S[k][2 * i] = scan_fma2(ax, S[k][2 * i], scan_mul2(kk[w][i].x, x2[k]));
                            sum[k] = i == 0 ? scan_mul2(S[k][0], qq[w][0].x) : scan_fma2(S[k][2 * i], qq[w][i].x, sum[k]);
                            S[k][2 * i + 1] = scan_fma2(ay, S[k][2 * i + 1], scan_mul2(kk[w][i].y, x2[k]));
                            sum[k] = scan_fma2(S[k][2 * i + 1], qq[w][i].y, sum[k]);
                        }
                    }
#pragma unroll
                    for (int k = 0; k < CPT; ++k) {
                        const float2 v = scan_unpack(sum[k]);
                        acc[u0 + w][k] = v.x + v.y;
                    }
                }
            }
            // over the lanes: first by token, then by column
            float w[2][CPT], v[CPT];
            const bool b3 = lane & (LANES / 2), b2 = lane & (LANES / 4);
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int k = 0; k < CPT; ++k) w[u][k] = scan_fold(b3, acc[u][k], acc[u + 2][k], LANES / 2);
#pragma unroll
            for (int k = 0; k < CPT; ++k) v[k] = scan_fold(b2, w[0][k], w[1][k], LANES / 4);
            const bool b1 = lane & (REM / 2);
            v[0] = scan_fold(b1, v[0], v[2], REM / 2);
            v[1] = scan_fold(b1, v[1], v[3], REM / 2);
            if constexpr (REM == 4) v[0] = scan_fold(lane & 1, v[0], v[1], 1);
#pragma unroll
            for (int k = 0; k < LEFT; ++k)
                if ((whole || my_u < left) && cg + my_k + k < cols)
                    yp[k] = skip != nullptr ? fmaf(skip_h, tok[my_u * TOKEN + VECS * DP + cg + my_k + k], v[k]) : v[k];
        };
        if (here == CHUNK) {                                          // straight-line: a group's reads overlap the sums before it
#pragma unroll
            for (int t4 = 0; t4 < CHUNK; t4 += 4) group(tok + t4 * TOKEN, yp + t4 * y_ld, 4, true);
        } else {
#pragma unroll 1
            for (int t4 = 0; t4 < here; t4 += 4) group(tok + t4 * TOKEN, yp + t4 * y_ld, here - t4, false);
        }
        yp += CHUNK * y_ld;
        __syncthreads();                                              // the stage is copied into again in the next round
    }
    pdl_trigger();                                                    // (not at the start: the successor's CTAs would only wait here)
#pragma unroll
    for (int k = 0; k < CPT; ++k)
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int d = 4 * (lane + LANES * i);
            const float2 lo = scan_unpack(S[k][2 * i]), hi = scan_unpack(S[k][2 * i + 1]);
            if (cg + k >= cols) continue;
            float* dst = srow + (long)k * n + d;
            if (state_vec4) {
                if (d < n) *reinterpret_cast<float4*>(dst) = make_float4(lo.x, lo.y, hi.x, hi.y);
            } else {
                if (d < n) dst[0] = lo.x;
                if (d + 1 < n) dst[1] = lo.y;
                if (d + 2 < n) dst[2] = hi.x;
                if (d + 3 < n) dst[3] = hi.y;
            }
        }
}

template <int R, int LANES, int COLS, bool SCALAR>
static int state_scan_launch(const float* rows, long ld, const ScanToken& at, const float* skip, float* y, long y_ld, float* state,
                             long state_stride, const int* req_start, const int* req_ctx, const int* req_qlen,
                             const int* req_slot, int n_requests, int heads, int n, int p, int vec4, int state_vec4, bool overlap,
                             cudaStream_t stream) {
    constexpr int CHUNK = R * LANES <= 128 ? 16 : 8;
    constexpr size_t smem = (size_t)SCAN_STAGES * CHUNK * ((SCALAR ? 2 : 3) * R * LANES + COLS + 4) * sizeof(float);
    auto kernel = state_scan_kernel<R, LANES, COLS, SCALAR, CHUNK>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return fl_launch_as(overlap, kernel, dim3(n_requests, heads, (p + COLS - 1) / COLS), dim3(COLS / SCAN_CPT * LANES), smem, stream,
                        rows, ld, at, skip, y, y_ld, state, state_stride, req_start, req_ctx, req_qlen, req_slot, n, p, vec4,
                        state_vec4);
}

// single_tokens: every request of the step brings one token.
template <bool SCALAR>
static int state_scan(const float* rows, long ld, const ScanToken& at, const float* skip, float* y, long y_ld, float* state,
                      long state_stride, const int* req_start, const int* req_ctx, const int* req_qlen, const int* req_slot,
                      int n_requests, int heads, int n, int p, int single_tokens, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (n < 1 || n > 256 || p < 1 || heads < 1 || heads > 65535 || (p + 15) / 16 > 65535 || at.per_group < 1)
        return (int)cudaErrorInvalidValue;
    // 16-byte copies where every source address is a multiple of 16 bytes; the state likewise
    const int vec4 = n % 4 == 0 && p % 4 == 0 && ld % 4 == 0 && ((uintptr_t)rows % 16) == 0 && at.k0 % 4 == 0 && at.q0 % 4 == 0 &&
                     at.n_step % 4 == 0 && at.a0 % 4 == 0 && at.v0 % 4 == 0;
    const int state_vec4 = n % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state % 16) == 0;
    const bool overlap = single_tokens != 0;         // (short kernels gain from the overlap, long ones need the SMs evenly)
#define SCAN_GO(R, L, COLS)                                                                                                 \
    return state_scan_launch<R, L, COLS, SCALAR>(rows, ld, at, skip, y, y_ld, state, state_stride, req_start, req_ctx, req_qlen, \
                                                 req_slot, n_requests, heads, n, p, vec4, state_vec4, overlap, stream)
#define SCAN_COLS(R, L)                                                                                                     \
    {                                                                                                                       \
        if (p <= 16) SCAN_GO(R, L, 16);                                                                                     \
        SCAN_GO(R, L, 32);                                                                                                  \
    }
    if (n <= 32) SCAN_COLS(4, 8)
    if (n <= 64) SCAN_COLS(4, 16)
    if (n <= 128) SCAN_COLS(8, 16)
    SCAN_COLS(16, 16)
#undef SCAN_COLS
#undef SCAN_GO
}
