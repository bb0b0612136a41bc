// State-space recurrence with a scalar decay per head and token (a selective state space in its "duality" form).
//
// Per token, from one product's row [z: inner | x: inner | B: groups x state | C: groups x state | dt: heads] with
// inner = heads x vdim; head h reads group g = h / (heads / groups):
//     x, B, C <- silu(conv(x, B, C) + bias)              one causal convolution per channel, `taps` taps
//     dt <- softplus(dt + dt_bias),   a = exp(-exp(A_log) dt)
//     S <- a S + dt B x^T  (state x vdim per head),   y = S^T C + D x
// then y * silu(z) is divided, part by part (norm_parts equal parts of inner), by its root mean square and multiplied by a
// weight.  A request's state row is S for every head, [heads][vdim][state] float (a column of S is contiguous), and behind
// it the convolution's last taps - 1 inputs, [taps - 1][inner + 2 groups state], oldest first; it is ignored when the
// request starts (context 0).
//
//   ssd_prep     convolution, silu, dt and decay of every token in one float work row x | B | C | dt | a
//   ssd_scan     the recurrence over each request's tokens in order (state_scan.cuh, one decay per token)
//   ssd_step     steps of single tokens: convolution, recurrence and read-out of a request's head in one kernel
//   ssd_norm     per (token, part): gate, norm, weight; and, in blocks of their own, the convolution's new state per request
//                (after every reader of the old one)
//
// All arithmetic is float (dt and the decay, two numbers a head and token, in double and rounded once: the decay is
// multiplied up over thousands of tokens).  Every sum's order depends on the sizes alone.
#include "short_conv.cuh"
#include "state_scan.cuh"

#define SSD_CPT 4                // value columns of a thread of the single-token kernel

// dt and decay from the raw dt: neg_a = -exp(A_log), in double.
__device__ __forceinline__ void ssd_rates(float raw, float dt_bias, double neg_a, float& dt, float& decay) {
    const double v = (double)raw + (double)dt_bias;
    const double soft = v > 30.0 ? v : log1p(exp(v));
    dt = (float)soft;
    decay = (float)exp(neg_a * soft);
}

// V channels a thread, RUN consecutive tokens; the last blockIdx.y does dt and decay.  conv_w: [taps][channels].
// TAPS: the window's length (taps rounded up).
template <typename T, int V, int TAPS, int RUN>
__global__ void __launch_bounds__(128) ssd_prep_kernel(
    const T* __restrict__ proj, long ld, const float* __restrict__ conv_w, const float* __restrict__ conv_b, int taps,
    const float* __restrict__ dt_bias, const double* __restrict__ neg_a, const float* __restrict__ tail, long tail_stride,
    const StepTables st, float* __restrict__ work, long w_ld, int n_tokens, int inner, int channels, int heads) {
    pdl_wait();
    pdl_trigger();
    const int t0 = blockIdx.x * RUN, t1 = min(n_tokens, t0 + RUN);
    if (blockIdx.y == gridDim.y - 1) {
        for (int i = threadIdx.x; i < (t1 - t0) * heads; i += blockDim.x) {
            const int t = t0 + i / heads, h = i % heads;
            float dt, decay;
            ssd_rates(to_f32<T>(proj[(long)t * ld + inner + channels + h]), dt_bias[h], neg_a[h], dt, decay);
            work[(long)t * w_ld + channels + h] = dt;
            work[(long)t * w_ld + channels + heads + h] = decay;
        }
        return;
    }
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= channels) return;
    ShortConv<T, V, TAPS, RUN> conv;
    conv.start(conv_w, taps, channels, c);
    const ChanVec<V> b = chan_load<float, V>(conv_b + c);
    conv.run(t0, t1, proj + inner + c, ld, st, tail, tail_stride, taps, channels, c,
             [&](int t, ChanVec<V> y, const ChanVec<V>*) {
#pragma unroll
                 for (int e = 0; e < V; ++e) y.v[e] = fl_silu(y.v[e] + b.v[e]);
                 chan_store<float, V>(work + (long)t * w_ld + c, y);
             });
}

// The four column sums of a group of LANES lanes, each lane holding its rows' part of all four.  After the exchange a
// lane holds the sum of column `mine` (two lanes' worth of steps carry halves, so five shuffles do for sixteen lanes).
template <int LANES>
__device__ __forceinline__ float ssd_sum4(const float (&acc)[SSD_CPT], int lane, int& mine) {
    const bool up2 = lane & (LANES / 2), up1 = lane & (LANES / 4);
    const float s0 = up2 ? acc[0] : acc[2], s1 = up2 ? acc[1] : acc[3];
    float k0 = up2 ? acc[2] : acc[0], k1 = up2 ? acc[3] : acc[1];
    k0 += __shfl_xor_sync(0xffffffffu, s0, LANES / 2);
    k1 += __shfl_xor_sync(0xffffffffu, s1, LANES / 2);
    float v = (up1 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, up1 ? k0 : k1, LANES / 4);
#pragma unroll
    for (int off = LANES / 8; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    mine = (up2 ? 2 : 0) + (up1 ? 1 : 0);
    return v;
}

// One token's step of a thread's 4 x R tile of S: S <- a S + B (dt x), the columns' sums of S C.
template <int R>
__device__ __forceinline__ void ssd_update(float (&S)[SSD_CPT][R], float (&acc)[SSD_CPT], const float* b, const float* c,
                                           const float (&xd)[SSD_CPT], float decay, int i4) {
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int k = 0; k < SSD_CPT; ++k) {
            S[k][4 * i4 + e] = fmaf(decay, S[k][4 * i4 + e], b[e] * xd[k]);
            acc[k] = fmaf(S[k][4 * i4 + e], c[e], acc[k]);
        }
}

// Every request of the step brings one token (row r of proj is request r's): the whole mixer up to the norm.
template <typename T, int R, int LANES, int COLS>
__global__ void __launch_bounds__(COLS / SSD_CPT * LANES) ssd_step_kernel(
    const T* __restrict__ proj, long ld, const float* __restrict__ conv_w, const float* __restrict__ conv_b, int taps,
    const float* __restrict__ dt_bias, const double* __restrict__ neg_a, const float* __restrict__ skip, float* __restrict__ y,
    long y_ld, float* __restrict__ state, long state_stride, long tail_off, const int* __restrict__ req_ctx,
    const int* __restrict__ req_slot, int heads, int vdim, int n, int groups, int vec4) {
    pdl_wait();
    pdl_trigger();
    constexpr int DP = R * LANES;
    __shared__ __align__(16) float tok[2 * DP + COLS + 4];            // B | C | x | dt, decay
    const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, lane = tid & (LANES - 1), cg = tid / LANES * SSD_CPT;
    const int ctx = req_ctx[r];
    const bool fresh = ctx == 0;
    const int inner = heads * vdim, gn = groups * n, g = h / (heads / groups), channels = inner + 2 * gn;
    const int cols = min(COLS, vdim - col0);
    float* base = state + (long)req_slot[r] * state_stride;
    float* srow = base + ((long)h * vdim + col0 + cg) * n;
    float S[SSD_CPT][R];
    if (vec4) {                                                       // asked for before the convolution: all loads in flight
#pragma unroll
        for (int k = 0; k < SSD_CPT; ++k)
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const int d = 4 * (lane + LANES * i);
                float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (!fresh && cg + k < cols && d < n) v = *reinterpret_cast<const float4*>(srow + (long)k * n + d);
                S[k][4 * i] = v.x; S[k][4 * i + 1] = v.y; S[k][4 * i + 2] = v.z; S[k][4 * i + 3] = v.w;
            }
    } else {
#pragma unroll
        for (int k = 0; k < SSD_CPT; ++k)
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int d = 4 * (lane + LANES * (i / 4)) + (i & 3);
                S[k][i] = (!fresh && cg + k < cols && d < n) ? srow[(long)k * n + d] : 0.0f;
            }
    }
    const T* row = proj + (long)r * ld + inner;
    const float* tail = base + tail_off;
    for (int i = tid; i < 2 * DP + COLS; i += blockDim.x) {
        int c = -1;                                                   // the channel whose convolution place i wants
        if (i < DP) c = i < n ? inner + g * n + i : -1;
        else if (i < 2 * DP) c = i - DP < n ? inner + gn + g * n + (i - DP) : -1;
        else c = i - 2 * DP < cols ? h * vdim + col0 + (i - 2 * DP) : -1;
        float v = 0.0f;
        if (c >= 0) {
            for (int j = 0; j < taps - 1; ++j)                        // tail entry j: position ctx - (taps - 1) + j
                if (ctx - (taps - 1) + j >= 0) v = fmaf(conv_w[(long)j * channels + c], tail[(long)j * channels + c], v);
            v = fl_silu(fmaf(conv_w[(long)(taps - 1) * channels + c], to_f32<T>(row[c]), v) + conv_b[c]);
        }
        tok[i] = v;
    }
    if (tid == 0) ssd_rates(to_f32<T>(row[channels + h]), dt_bias[h], neg_a[h], tok[2 * DP + COLS], tok[2 * DP + COLS + 1]);
    __syncthreads();
    const float4 xv = *reinterpret_cast<const float4*>(tok + 2 * DP + cg);
    const float dt = tok[2 * DP + COLS], decay = tok[2 * DP + COLS + 1];
    const float x[SSD_CPT] = {xv.x, xv.y, xv.z, xv.w};
    const float xd[SSD_CPT] = {xv.x * dt, xv.y * dt, xv.z * dt, xv.w * dt};
    float acc[SSD_CPT] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const float4 b4 = reinterpret_cast<const float4*>(tok)[lane + LANES * i];
        const float4 c4 = reinterpret_cast<const float4*>(tok + DP)[lane + LANES * i];
        const float b[4] = {b4.x, b4.y, b4.z, b4.w}, c[4] = {c4.x, c4.y, c4.z, c4.w};
        ssd_update<R>(S, acc, b, c, xd, decay, i);
    }
    if (vec4) {
#pragma unroll
        for (int k = 0; k < SSD_CPT; ++k)
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const int d = 4 * (lane + LANES * i);
                if (cg + k < cols && d < n)
                    *reinterpret_cast<float4*>(srow + (long)k * n + d) = make_float4(S[k][4 * i], S[k][4 * i + 1], S[k][4 * i + 2], S[k][4 * i + 3]);
            }
    } else {
#pragma unroll
        for (int k = 0; k < SSD_CPT; ++k)
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int d = 4 * (lane + LANES * (i / 4)) + (i & 3);
                if (cg + k < cols && d < n) srow[(long)k * n + d] = S[k][i];
            }
    }
    int mine;
    const float sum = ssd_sum4<LANES>(acc, lane, mine);
    const float xm = mine == 0 ? x[0] : mine == 1 ? x[1] : mine == 2 ? x[2] : x[3];
    if ((lane & (LANES / 4 - 1)) == 0 && cg + mine < cols)
        y[(long)r * y_ld + (long)h * vdim + col0 + cg + mine] = fmaf(skip[h], xm, sum);
}

// Blocks [0, n_tokens) of x: token t, part blockIdx.y.  Behind them `share` blocks of x a request, which with blockIdx.y
// share its convolution channels out, one a thread: the new state (up to three
// entries are read before the first is written, so that the loads run side by side).
template <typename T, int V>
__global__ void __launch_bounds__(512) ssd_norm_kernel(
    const float* __restrict__ y, long y_ld, const T* __restrict__ proj, long ld, const float* __restrict__ weight,
    T* __restrict__ out, long out_ld, int n_tokens, int inner, int part, float eps, float* __restrict__ tail, long tail_stride,
    int share, int taps, int channels, const int* __restrict__ req_start, const int* __restrict__ req_ctx,
    const int* __restrict__ req_qlen, const int* __restrict__ req_slot) {
    pdl_wait();
    pdl_trigger();
    extern __shared__ __align__(16) float ssd_row[];                  // [part]
    __shared__ float scratch[32];
    if ((int)blockIdx.x >= n_tokens) {
        const int r = (blockIdx.x - n_tokens) / share, slice = (blockIdx.x - n_tokens) % share;
        const int c = (slice * gridDim.y + blockIdx.y) * blockDim.x + threadIdx.x;
        if (c >= channels) return;
        const int start = req_start[r], ctx = req_ctx[r], qlen = req_qlen[r], back = taps - 1;
        float* mine = tail + (long)req_slot[r] * tail_stride + c;
        auto entry = [&](int j) {                                     // entry j takes the input of position end - back + j
            const int at = ctx + qlen - back + j;
            if (at >= ctx) return to_f32<T>(proj[(long)(start + at - ctx) * ld + inner + c]);
            return at >= 0 ? mine[(long)(j + qlen) * channels] : 0.0f;
        };
        if (back <= 3) {
            float u[3];
#pragma unroll
            for (int j = 0; j < 3; ++j) u[j] = j < back ? entry(j) : 0.0f;
#pragma unroll
            for (int j = 0; j < 3; ++j)
                if (j < back) mine[(long)j * channels] = u[j];
        } else {
            for (int j = 0; j < back; ++j) mine[(long)j * channels] = entry(j);      // (entries that stay move down)
        }
        return;
    }
    const long t = blockIdx.x;
    const int first = blockIdx.y * part;
    const float* yr = y + t * y_ld + first;
    const T* zr = proj + t * ld + first;
    float ss = 0.0f;
    for (int i = threadIdx.x * V; i < part; i += blockDim.x * V) {
        ChanVec<V> v = chan_load<float, V>(yr + i);
        const ChanVec<V> z = chan_load<T, V>(zr + i);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            v.v[e] *= fl_silu(z.v[e]);
            ss += v.v[e] * v.v[e];
        }
        chan_store<float, V>(ssd_row + i, v);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)part + eps);
    for (int i = threadIdx.x * V; i < part; i += blockDim.x * V) {    // each thread its own elements
        ChanVec<V> v = chan_load<float, V>(ssd_row + i);
        const ChanVec<V> w = chan_load<float, V>(weight + first + i);
#pragma unroll
        for (int e = 0; e < V; ++e) v.v[e] = v.v[e] * inv * w.v[e];
        chan_store<T, V>(out + t * out_ld + first + i, v);
    }
}

// proj: rows [z | x | B | C | dt] from the given column on; work: rows x | B | C | dt | a float; neg_a: -exp(A_log).
FL_API int fl_ssd_prep(const void* proj, int dtype, long ld, const float* conv_w, const float* conv_b, int taps,
                       const float* dt_bias, const double* neg_a, const float* tail, long tail_stride, const int* tok_req,
                       const int* positions, const int* req_start, const int* req_ctx, const int* req_qlen,
                       const int* req_slot, float* work, long w_ld, int n_tokens, int heads, int vdim, int n, int groups,
                       cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const int inner = heads * vdim, channels = inner + 2 * groups * n;
    if (taps < 1 || taps > 16 || (taps > 1 && tail == nullptr) || groups < 1 || heads % groups) return (int)cudaErrorInvalidValue;
    const StepTables st{tok_req, positions, req_start, req_ctx, req_qlen, req_slot};
    const int run = n_tokens >= 256 ? 4 : 1;
    const bool vec = channels % 4 == 0 && inner % 4 == 0 && chan_aligned(proj, ld, dtype == FL_F32 ? 4 : 2) &&
                     chan_aligned(work, w_ld, 4) && chan_aligned(conv_w, 4, 4) && chan_aligned(conv_b, 4, 4) &&
                     (taps == 1 || chan_aligned(tail, tail_stride, 4));
    const int per = 128 * (vec ? 4 : 1);
    dim3 grid((n_tokens + run - 1) / run, (channels + per - 1) / per + 1);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define FL_SSD_PREP(V, TAPS, RUN)                                                                                        \
    FL_DISPATCH(dtype, T, return fl_launch(ssd_prep_kernel<T, V, TAPS, RUN>, grid, dim3(128), 0, stream, (const T*)proj, ld, \
                                           conv_w, conv_b, taps, dt_bias, neg_a, tail, tail_stride, st, work, w_ld, n_tokens, \
                                           inner, channels, heads))
#define FL_SSD_PREP_RUN(V, TAPS) { if (run == 4) { FL_SSD_PREP(V, TAPS, 4); } else { FL_SSD_PREP(V, TAPS, 1); } }
    if (vec) { if (taps == 1) FL_SSD_PREP_RUN(4, 1) else if (taps <= 4) FL_SSD_PREP_RUN(4, 4) else FL_SSD_PREP_RUN(4, 16) }
    else { if (taps == 1) FL_SSD_PREP_RUN(1, 1) else if (taps <= 4) FL_SSD_PREP_RUN(1, 4) else FL_SSD_PREP_RUN(1, 16) }
#undef FL_SSD_PREP_RUN
#undef FL_SSD_PREP
    return 0;
}

static inline bool ssd_takes(int n_requests, int heads, int vdim, int n, int groups) {
    return n >= 1 && n <= 256 && vdim >= 1 && heads >= 1 && heads <= 65535 && (vdim + 15) / 16 <= 65535 && groups >= 1 &&
           heads % groups == 0;
}

// work: what fl_ssd_prep leaves.  single_tokens: every request of the step brings one token.
FL_API int fl_ssd_scan(const float* work, long w_ld, const float* skip, float* y, long y_ld, float* state, long state_stride,
                       const int* req_start, const int* req_ctx, const int* req_qlen, const int* req_slot, int n_requests,
                       int heads, int vdim, int n, int groups, int single_tokens, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (!ssd_takes(n_requests, heads, vdim, n, groups)) return (int)cudaErrorInvalidValue;
    const int inner = heads * vdim, gn = groups * n;
    const ScanToken at{inner, inner + gn, n, heads / groups, 0, 0, inner + 2 * gn, inner + 2 * gn + heads};
    return state_scan<true>(work, w_ld, at, skip, y, y_ld, state, state_stride, req_start, req_ctx, req_qlen, req_slot, n_requests,
                            heads, n, vdim, single_tokens, stream);
}

// Steps of single tokens only: row r of proj is request r's.
FL_API int fl_ssd_step(const void* proj, int dtype, long ld, const float* conv_w, const float* conv_b, int taps,
                       const float* dt_bias, const double* neg_a, const float* skip, float* y, long y_ld, float* state,
                       long state_stride, long tail_off, const int* req_ctx, const int* req_slot, int n_requests, int heads,
                       int vdim, int n, int groups, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (!ssd_takes(n_requests, heads, vdim, n, groups) || taps < 1) return (int)cudaErrorInvalidValue;
    const int vec4 = n % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state % 16) == 0;
#define FL_SSD_STEP(R, L, C)                                                                                             \
    FL_DISPATCH(dtype, T, return fl_launch(ssd_step_kernel<T, R, L, C>, dim3(n_requests, heads, (vdim + C - 1) / C),      \
                                           dim3(C / SSD_CPT * L), 0, stream, (const T*)proj, ld, conv_w, conv_b, taps,   \
                                           dt_bias, neg_a, skip, y, y_ld, state, state_stride, tail_off, req_ctx,        \
                                           req_slot, heads, vdim, n, groups, vec4))
    if (vdim <= 16) {
        if (n <= 32) { FL_SSD_STEP(4, 8, 16); }
        if (n <= 64) { FL_SSD_STEP(4, 16, 16); }
        if (n <= 128) { FL_SSD_STEP(8, 16, 16); }
        FL_SSD_STEP(16, 16, 16);
    } else {
        if (n <= 32) { FL_SSD_STEP(4, 8, 32); }
        if (n <= 64) { FL_SSD_STEP(4, 16, 32); }
        if (n <= 128) { FL_SSD_STEP(8, 16, 32); }
        FL_SSD_STEP(16, 16, 32);
    }
#undef FL_SSD_STEP
    return 0;
}

// out[t] = y[t] * silu(z[t]) normed part by part, times weight [inner] float; tail (null with taps 1) moves on.
FL_API int fl_ssd_norm(const float* y, long y_ld, const void* proj, int dtype, long ld, const float* weight, void* out,
                       long out_ld, int n_tokens, int inner, int parts, float eps, float* tail, long tail_stride, int taps,
                       int channels, const int* req_start, const int* req_ctx, const int* req_qlen, const int* req_slot,
                       int n_requests, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (parts < 1 || parts > 65535 || inner % parts) return (int)cudaErrorInvalidValue;
    const int part = inner / parts;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 160 * 1024) return (int)cudaErrorInvalidValue;
    const int elem = dtype == FL_F32 ? 4 : 2;
    const bool vec = part % 4 == 0 && chan_aligned(y, y_ld, 4) && chan_aligned(proj, ld, elem) && chan_aligned(out, out_ld, elem) &&
                     chan_aligned(weight, 4, 4);
    int threads = 32;
    while (threads < 512 && threads * (vec ? 8 : 2) < part) threads *= 2;
    const int share = (channels + threads * parts - 1) / (threads * parts);
    dim3 grid(n_tokens + (taps > 1 ? n_requests * share : 0), parts);
    FL_DISPATCH(dtype, T, {
        auto kernel = vec ? ssd_norm_kernel<T, 4> : ssd_norm_kernel<T, 1>;
        if (smem > 48 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        return fl_launch(kernel, grid, dim3(threads), smem, stream, y, y_ld, (const T*)proj, ld, weight, (T*)out, out_ld,
                         n_tokens, inner, part, eps, tail, tail_stride, share, taps, channels, req_start, req_ctx, req_qlen, req_slot);
    });
    return 0;
}
