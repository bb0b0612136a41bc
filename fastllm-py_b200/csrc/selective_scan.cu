// Selective scan: a recurrence per channel c and state element n whose decay is made from the token for every one of them
// (the first form of a selective state space).
//
// Per token, from one product's row [u: inner | z: inner]:
//     x <- silu(conv(u) + bias)                       one causal convolution per channel, `taps` taps
//     low = W_x x                                     [dt: rank | B: state | C: state], a product the caller makes
//     dt <- softplus(W_dt dt + bias)                  one number a channel
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,     y_c = sum_n S[c, n] C_n + D_c x_c       (A < 0)
// then y * silu(z).  A request's state row is S [inner][state] float and behind it the convolution's last taps - 1 inputs,
// [taps - 1][inner], oldest first; it is ignored when the request starts (context 0).
//
//   selective_conv      convolution and silu (in the activation type, which W_x reads); in steps of single tokens the
//                       thread that owns a channel moves its kept inputs on
//   selective_split     the product W_dt dt (the caller's) reads dt's float row as two bfloat16 parts, which keep about 16
//                       bits of it, against W_dt twice over
//   selective_scan      the recurrence over each request's tokens in order, read-out, skip and gate; its blocks also move
//                       the kept inputs of requests on
//   selective_step      steps of single tokens: dt, recurrence, read-out and gate of a request's channels in one kernel
//
// Everything but x, z and y (the activation type) is float.
#include "short_conv.cuh"
#include "state_scan.cuh"

// silu with the fast exponential and division where the result is rounded to bfloat16.
template <typename T> __device__ __forceinline__ float sel_silu(float v) {
    return sizeof(T) == 4 ? fl_silu(v) : __fdividef(v, 1.0f + __expf(-v));
}

// ------------------------------------------------------------------ convolution
// V channels a thread, RUN consecutive tokens; conv_w: [taps][inner].  move_tail: every request has one token (RUN is 1).
template <typename T, int V, int TAPS, int RUN>
__global__ void __launch_bounds__(128) selective_conv_kernel(
    const T* __restrict__ u, long ld, const float* __restrict__ conv_w, const float* __restrict__ conv_b, int taps,
    float* tail, long tail_stride, const StepTables st, T* __restrict__ x, long x_ld, int n_tokens, int inner, int move_tail) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    ShortConv<T, V, TAPS, RUN> conv;
    ChanVec<V> b = {};
    if (c < inner) {                                                  // (no kernel writes these: asked for before the wait)
        conv.start(conv_w, taps, inner, c);
        b = chan_load<float, V>(conv_b + c);
    }
    pdl_wait();
    pdl_trigger();
    if (c >= inner) return;
    const int t0 = blockIdx.x * RUN, t1 = min(n_tokens, t0 + RUN);
    conv.run(t0, t1, u + c, ld, st, tail, tail_stride, taps, inner, c, [&](int t, ChanVec<V> y, const ChanVec<V>* in) {
#pragma unroll
        for (int e = 0; e < V; ++e) y.v[e] = sel_silu<T>(y.v[e] + b.v[e]);
        chan_store<T, V>(x + (long)t * x_ld + c, y);
        if (RUN == 1 && TAPS > 1 && move_tail) {                      // kept row j: the input of position pos - (taps - 2) + j
            float* kept = tail + (long)st.req_slot[st.tok_req[t]] * tail_stride + c;
#pragma unroll
            for (int k = 1; k < TAPS; ++k) {
                const int j = k - 1 - (TAPS - taps);
                if (j >= 0) chan_store<float, V>(kept + (long)j * inner, in[k]);
            }
        }
    });
}

FL_API int fl_selective_conv(const void* u, int dtype, long ld, const float* conv_w, const float* conv_b, int taps, float* tail,
                             long tail_stride, const int* tok_req, const int* positions, const int* req_start,
                             const int* req_ctx, const int* req_qlen, const int* req_slot, void* x, long x_ld, int n_tokens,
                             int inner, int move_tail, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (taps < 1 || taps > 16 || (taps > 1 && tail == nullptr)) return (int)cudaErrorInvalidValue;
    const StepTables st{tok_req, positions, req_start, req_ctx, req_qlen, req_slot};
    const int run = move_tail || n_tokens < 256 ? 1 : n_tokens >= 1024 ? 8 : 4;
    const int elem = dtype == FL_F32 ? 4 : 2;
    const bool vec = inner % 4 == 0 && chan_aligned(u, ld, elem) && chan_aligned(x, x_ld, elem) && chan_aligned(conv_w, 4, 4) &&
                     chan_aligned(conv_b, 4, 4) && (taps == 1 || chan_aligned(tail, tail_stride, 4));
    const int per = 128 * (vec ? 4 : 1);
    dim3 grid((n_tokens + run - 1) / run, (inner + per - 1) / per);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define FL_SEL_CONV(V, TAPS, RUN)                                                                                         \
    FL_DISPATCH(dtype, T, return fl_launch(selective_conv_kernel<T, V, TAPS, RUN>, grid, dim3(128), 0, stream, (const T*)u, ld, \
                                           conv_w, conv_b, taps, tail, tail_stride, st, (T*)x, x_ld, n_tokens, inner, move_tail))
#define FL_SEL_CONV_RUN(V, TAPS)                                                                                          \
    { if (run == 8) { FL_SEL_CONV(V, TAPS, 8); } else if (run == 4) { FL_SEL_CONV(V, TAPS, 4); } else { FL_SEL_CONV(V, TAPS, 1); } }
    if (vec) { if (taps == 1) FL_SEL_CONV_RUN(4, 1) else if (taps <= 4) FL_SEL_CONV_RUN(4, 4) else FL_SEL_CONV_RUN(4, 16) }
    else { if (taps == 1) FL_SEL_CONV_RUN(1, 1) else if (taps <= 4) FL_SEL_CONV_RUN(1, 4) else FL_SEL_CONV_RUN(1, 16) }
#undef FL_SEL_CONV_RUN
#undef FL_SEL_CONV
    return 0;
}

// ------------------------------------------------------------------ step sizes
// out[t] = [hi | lo], two bfloat16 parts of the first `rank` columns of low[t]: lo is what rounding to hi leaves.
__global__ void __launch_bounds__(256) selective_split_kernel(const float* __restrict__ low, long low_ld, int rank,
                                                              bf16* __restrict__ out, long out_ld) {
    pdl_wait();
    pdl_trigger();
    const float* row = low + (long)blockIdx.x * low_ld;
    bf16* o = out + (long)blockIdx.x * out_ld;
    for (int k = threadIdx.x; k < rank; k += blockDim.x) {
        const bf16 hi = __float2bfloat16_rn(row[k]);
        o[k] = hi;
        o[rank + k] = __float2bfloat16_rn(row[k] - __bfloat162float(hi));
    }
}

FL_API int fl_selective_split(const float* low, long low_ld, int rank, void* out, long out_ld, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rank < 1 || out_ld < 2L * rank) return (int)cudaErrorInvalidValue;
    const int threads = rank >= 256 ? 256 : (rank + 31) / 32 * 32;
    return fl_launch(selective_split_kernel, dim3(n_tokens), dim3(threads), 0, stream, low, low_ld, rank, (bf16*)out, out_ld);
}

// ------------------------------------------------------------------ the recurrence
// A lane's rows of a channel: the groups of four 4 (lane + LANES i).  Rows from n on are zero.
template <int R, int LANES>
__device__ __forceinline__ void sel_rows(scan_f2 (&out)[R / 2], const float* p, int lane, int n, bool there, int vec4) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const int d = 4 * (lane + LANES * i);
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (there && vec4) {
            if (d < n) v = *reinterpret_cast<const float4*>(p + d);
        } else if (there) {
            if (d < n) v.x = p[d];
            if (d + 1 < n) v.y = p[d + 1];
            if (d + 2 < n) v.z = p[d + 2];
            if (d + 3 < n) v.w = p[d + 3];
        }
        out[2 * i] = scan_pack(v.x, v.y);
        out[2 * i + 1] = scan_pack(v.z, v.w);
    }
}
template <int R, int LANES>
__device__ __forceinline__ void sel_rows_out(const scan_f2 (&in)[R / 2], float* p, int lane, int n, int vec4) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const int d = 4 * (lane + LANES * i);
        const float2 lo = scan_unpack(in[2 * i]), hi = scan_unpack(in[2 * i + 1]);
        if (vec4) {
            if (d < n) *reinterpret_cast<float4*>(p + d) = make_float4(lo.x, lo.y, hi.x, hi.y);
        } else {
            if (d < n) p[d] = lo.x;
            if (d + 1 < n) p[d + 1] = lo.y;
            if (d + 2 < n) p[d + 2] = hi.x;
            if (d + 3 < n) p[d + 3] = hi.y;
        }
    }
}

// What one token does to a lane's rows, formed before S is needed: S <- p S + bx, sum += S c.
template <int R> struct SelToken {
    scan_f2 p[R / 2], bx[R / 2], c[R / 2];
};
// The decay exp(v), v = dt A, of a pair of rows.  For 32-bit models p is expm1(v), applied as S + p S: near 1 a float exponential
// is off by a like part of itself token after token, which adds up along a sequence, where expm1's error is a part of the
// small v.  For bfloat16 models p is 2^v (A comes multiplied by log2(e)).
template <typename T> __device__ __forceinline__ scan_f2 sel_decay(scan_f2 v) {
    const float2 e = scan_unpack(v);
    float p, q;
    if constexpr (sizeof(T) == 4) {
        p = expm1f(e.x);
        q = expm1f(e.y);
    } else {
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(p) : "f"(e.x));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(q) : "f"(e.y));
    }
    return scan_pack(p, q);
}
template <typename T, int R, int LANES>
__device__ __forceinline__ void sel_prepare(SelToken<R>& t, const scan_f2 (&A)[R / 2], const float* b, const float* c, float dt,
                                            float x, int lane) {
    const scan_f2 dt2 = scan_pack(dt, dt), dx = scan_pack(dt * x, dt * x);
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const ulonglong2 bb = reinterpret_cast<const ulonglong2*>(b)[lane + LANES * i];
        const ulonglong2 cc = reinterpret_cast<const ulonglong2*>(c)[lane + LANES * i];
        t.p[2 * i] = sel_decay<T>(scan_mul2(dt2, A[2 * i]));
        t.p[2 * i + 1] = sel_decay<T>(scan_mul2(dt2, A[2 * i + 1]));
        t.bx[2 * i] = scan_mul2(bb.x, dx);
        t.bx[2 * i + 1] = scan_mul2(bb.y, dx);
        t.c[2 * i] = cc.x;
        t.c[2 * i + 1] = cc.y;
    }
}
// The rows' part of sum S c after the token.
template <typename T, int R>
__device__ __forceinline__ float sel_apply(scan_f2 (&S)[R / 2], const SelToken<R>& t) {
    const scan_f2 one = scan_pack(1.0f, 1.0f);
    scan_f2 sum = 0ULL;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
        if constexpr (sizeof(T) == 4) S[i] = scan_fma2(t.bx[i], one, scan_fma2(t.p[i], S[i], S[i]));
        else S[i] = scan_fma2(t.p[i], S[i], t.bx[i]);
        sum = i == 0 ? scan_mul2(S[0], t.c[0]) : scan_fma2(S[i], t.c[i], sum);
    }
    const float2 v = scan_unpack(sum);
    return v.x + v.y;
}

template <int N> struct ScanCount { static constexpr int value = N; };

// softplus(v) = max(v, 0) + log(1 + u), u = exp(-|v|); log(1 + u) = 2 artanh(s) with s = u / (2 + u) <= 1/3, as its power
// series in s^2 (eight terms leave 3e-9 of the sum).  No branch, and exact relative to the result also where it is small.
template <typename T> __device__ __forceinline__ float sel_softplus(float v) {
    const float u = sizeof(T) == 4 ? expf(-fabsf(v)) : __expf(-fabsf(v));
    const float s = sizeof(T) == 4 ? u / (2.0f + u) : __fdividef(u, 2.0f + u);
    const float q = s * s;
    float p = 1.0f / 15.0f;
    p = fmaf(p, q, 1.0f / 13.0f);
    p = fmaf(p, q, 1.0f / 11.0f);
    p = fmaf(p, q, 1.0f / 9.0f);
    p = fmaf(p, q, 1.0f / 7.0f);
    p = fmaf(p, q, 1.0f / 5.0f);
    p = fmaf(p, q, 1.0f / 3.0f);
    return fmaxf(v, 0.0f) + fmaf(2.0f * s * q, p, 2.0f * s);
}
struct SelRows {                     // the step's rows: element type T, float, float
    const void *x, *z, *u;           // convolved inputs, gates, inputs before the convolution
    const float *dt, *low;           // (dt before bias and softplus)
    long x_ld, z_ld, u_ld, dt_ld, low_ld;
    int b_at, c_at;                  // where low holds B and C
};

// A block takes one request and COLS channels.  Half of its threads walk the tokens, LANES lanes a channel, and do nothing
// else: a chunk of tokens is straight-line code that reads shared memory and leaves the read-out sums there.  The other
// half copies the chunks two ahead (cp.async, four stages), makes the step sizes of the next one (softplus of W_dt dt + bias)
// and turns the sums of the chunk before into outputs (skip, gate, store).  Tokens go four at a time, so that four sums are added up over the lanes together.  R and LANES follow from n alone:
// one order of sums whatever the cut.
template <typename T, int R, int LANES, int COLS, int CHUNK>
__global__ void __launch_bounds__(2 * COLS * LANES, 1) selective_scan_kernel(
    const SelRows in, const float* __restrict__ dt_bias, const float* __restrict__ a_log2, const float* __restrict__ skip, float scale,
    T* __restrict__ y, long y_ld,
    float* __restrict__ state, long state_stride, long tail_off, int taps, const int* __restrict__ req_start,
    const int* __restrict__ req_ctx, const int* __restrict__ req_qlen, const int* __restrict__ req_slot, int inner, int n,
    int vec_low, int vec_dt, int vec_x, int vec_z, int vec_y, int state_vec4) {
    static_assert(CHUNK % 4 == 0 && R % 4 == 0 && (LANES == 4 || LANES == 8 || LANES == 16) && COLS % 8 == 0 && SCAN_STAGES == 4, "");
    constexpr int DP = R * LANES, HALF = COLS * LANES, TV = 16 / sizeof(T);
    constexpr int STAGE = CHUNK * (2 * DP + COLS) * 4 + 2 * CHUNK * COLS * (int)sizeof(T);     // bytes
    extern __shared__ __align__(16) unsigned char sel_s[];
    float* sum_s = reinterpret_cast<float*>(sel_s + SCAN_STAGES * STAGE);                      // [2][CHUNK][COLS]
    pdl_wait();
    const int r = blockIdx.x, col0 = blockIdx.y * COLS, tid = threadIdx.x;
    const int start = req_start[r], qlen = req_qlen[r], ctx = req_ctx[r];
    const int cols = min(COLS, inner - col0), chunks = (qlen + CHUNK - 1) / CHUNK;
    for (int i = tid; i < SCAN_STAGES * STAGE / 16; i += 2 * HALF)    // padding stays zero, stale places hold numbers
        reinterpret_cast<float4*>(sel_s)[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float* base = state + (long)req_slot[r] * state_stride;
    auto stage_bc = [&](int s) { return reinterpret_cast<float*>(sel_s + s * STAGE); };
    auto stage_dt = [&](int s) { return stage_bc(s) + CHUNK * 2 * DP; };
    auto stage_x = [&](int s) { return reinterpret_cast<T*>(stage_dt(s) + CHUNK * COLS); };
    __syncthreads();
    if (tid < HALF) {
        const int lane = tid & (LANES - 1), col = tid / LANES, c = col0 + col;
        const bool mine = c < inner;
        float* srow = base + (long)c * n;
        scan_f2 S[R / 2], A[R / 2];
        sel_rows<R, LANES>(S, srow, lane, n, mine && ctx != 0, state_vec4);
        sel_rows<R, LANES>(A, a_log2 + (long)c * n, lane, n, mine, n % 4 == 0);
        const int my_u = ((lane & (LANES / 2)) ? 2 : 0) + ((lane & (LANES / 4)) ? 1 : 0);     // whose sum of four this lane gets
        const bool writer = (lane & (LANES / 4 - 1)) == 0;
        for (int k = 0; k <= chunks; ++k) {
            __syncthreads();                                          // chunk k has landed
            if (k == chunks) break;
            const int here = min(CHUNK, qlen - k * CHUNK), stage = k & 3;
            const float* bc = stage_bc(stage);
            const float* dts = stage_dt(stage) + col;
            const T* xs = stage_x(stage) + col;
            float sums[CHUNK / 4];                                    // of this lane's token of each four
            auto prepare = [&](SelToken<R>& tok, int t, bool real) {
                const float d = real ? dts[t * COLS] : 0.0f;          // (behind the end: decay one, nothing added)
                sel_prepare<T, R, LANES>(tok, A, bc + t * 2 * DP, bc + t * 2 * DP + DP, d, to_f32<T>(xs[t * COLS]), lane);
            };
            auto fold = [&](const float (&acc)[4]) {
                const bool up2 = lane & (LANES / 2), up1 = lane & (LANES / 4);
                const float w0 = scan_fold(up2, acc[0], acc[2], LANES / 2), w1 = scan_fold(up2, acc[1], acc[3], LANES / 2);
                float v = scan_fold(up1, w0, w1, LANES / 4);
#pragma unroll
                for (int off = LANES / 8; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
                return v;
            };
            if (here == CHUNK) {
                float acc[CHUNK];
#pragma unroll
                for (int t = 0; t < CHUNK; ++t) {
                    SelToken<R> tok;
                    prepare(tok, t, true);
                    acc[t] = sel_apply<T, R>(S, tok);
                }
#pragma unroll
                for (int g = 0; g < CHUNK / 4; ++g) {
                    const float four[4] = {acc[4 * g], acc[4 * g + 1], acc[4 * g + 2], acc[4 * g + 3]};
                    sums[g] = fold(four);
                }
            } else {
#pragma unroll
                for (int g = 0; g < CHUNK / 4; ++g) {
                    if (4 * g >= here) break;
                    float acc[4];
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        SelToken<R> tok;
                        prepare(tok, 4 * g + u, 4 * g + u < here);
                        acc[u] = sel_apply<T, R>(S, tok);
                    }
                    sums[g] = fold(acc);
                }
            }
            float* out = sum_s + (k & 1) * CHUNK * COLS + my_u * COLS + col;
#pragma unroll
            for (int g = 0; g < CHUNK / 4; ++g)
                if (writer && 4 * g < here) out[4 * g * COLS] = sums[g];
        }
        pdl_trigger();                                                // (not at the start: the successor's CTAs would only wait here)
        if (mine) sel_rows_out<R, LANES>(S, srow, lane, n, state_vec4);
        return;
    }
    const int ht = tid - HALF;
    // rows of `count` (at most PER vectors of) elements: the loops' bounds and divisors are the tile's, not the layer's
    auto copy_floats = [&](auto per, float* dst, int d_step, const float* src, long s_step, int count, int here, int vec) {
        constexpr int PER = decltype(per)::value;                     // (vectors of four)
        if (vec) {
#pragma unroll
            for (int i = ht; i < PER * CHUNK; i += HALF) {
                const int t = i / PER, e = i % PER * 4;
                if (t < here && e < count) scan_cp16(dst + t * d_step + e, src + t * s_step + e);
            }
        } else {
            for (int i = ht; i < PER * 4 * CHUNK; i += HALF) {
                const int t = i / (PER * 4), e = i % (PER * 4);
                if (t < here && e < count) scan_cp4(dst + t * d_step + e, src + t * s_step + e);
            }
        }
    };
    auto copy_rows = [&](T* dst, const T* src, long s_step, int here, int vec) {
        if (vec) {
#pragma unroll
            for (int i = ht; i < COLS / TV * CHUNK; i += HALF) {
                const int t = i / (COLS / TV), e = i % (COLS / TV) * TV;
                if (t < here && e < cols) scan_cp16(dst + t * COLS + e, src + t * s_step + e);
            }
        } else {
            for (int i = ht; i < COLS * CHUNK; i += HALF) {
                const int t = i / COLS, e = i % COLS;
                if (t < here && e < cols) dst[t * COLS + e] = src[t * s_step + e];
            }
        }
    };
    auto load = [&](int k) {                                          // (one group of copies a chunk, empty ones beyond the end)
        if (k < chunks) {
            const int here = min(CHUNK, qlen - k * CHUNK), s = k & 3;
            const long t = start + k * CHUNK;
            copy_floats(ScanCount<DP / 4>(), stage_bc(s), 2 * DP, in.low + t * in.low_ld + in.b_at, in.low_ld, n, here, vec_low);
            copy_floats(ScanCount<DP / 4>(), stage_bc(s) + DP, 2 * DP, in.low + t * in.low_ld + in.c_at, in.low_ld, n, here, vec_low);
            copy_floats(ScanCount<COLS / 4>(), stage_dt(s), COLS, in.dt + t * in.dt_ld + col0, in.dt_ld, cols, here, vec_dt);
            copy_rows(stage_x(s), (const T*)in.x + t * in.x_ld + col0, in.x_ld, here, vec_x);
            copy_rows(stage_x(s) + CHUNK * COLS, (const T*)in.z + t * in.z_ld + col0, in.z_ld, here, vec_z);
        }
        asm volatile("cp.async.commit_group;");
    };
    // outputs of a chunk, four channels a thread (always the same four: HALF is a multiple of COLS / 4)
    constexpr int QUADS = COLS / 4;
    const int e0 = ht % QUADS * 4;
    float skip_e[4], bias_e[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        skip_e[e] = e0 + e < cols ? skip[col0 + e0 + e] : 0.0f;
        bias_e[e] = e0 + e < cols ? dt_bias[col0 + e0 + e] : 0.0f;
    }
    const float bias_1 = ht % COLS < cols ? dt_bias[col0 + ht % COLS] : 0.0f;
    // step sizes of a chunk, in place: a thread takes the places it copied, which its own wait has made visible to it
    auto rates = [&](int k) {
        if (k >= chunks) return;
        const int here = min(CHUNK, qlen - k * CHUNK);
        float* d = stage_dt(k & 3);
        if (vec_dt) {
#pragma unroll
            for (int t = ht / QUADS; t < CHUNK; t += HALF / QUADS) {
                if (t >= here || e0 >= cols) continue;
                float4* p = reinterpret_cast<float4*>(d + t * COLS + e0);
                float4 v = *p;
                v.x = sel_softplus<T>(v.x + bias_e[0]);
                v.y = sel_softplus<T>(v.y + bias_e[1]);
                v.z = sel_softplus<T>(v.z + bias_e[2]);
                v.w = sel_softplus<T>(v.w + bias_e[3]);
                *p = v;
            }
        } else {
            for (int t = ht / COLS; t < CHUNK; t += HALF / COLS) {
                float* p = d + t * COLS + ht % COLS;
                if (t < here && ht % COLS < cols) *p = sel_softplus<T>(*p + bias_1);
            }
        }
    };
    auto finish = [&](int k) {
        const int here = min(CHUNK, qlen - k * CHUNK);
        const float* sums = sum_s + (k & 1) * CHUNK * COLS;
        const T* xs = stage_x(k & 3);
        const T* zs = xs + CHUNK * COLS;
        T* yo = y + (long)(start + k * CHUNK) * y_ld + col0 + e0;
#pragma unroll
        for (int t = ht / QUADS; t < CHUNK; t += HALF / QUADS) {
            if (t >= here || e0 >= cols) continue;
            const ChanVec<4> v = chan_load<float, 4>(sums + t * COLS + e0), x = chan_load<T, 4>(xs + t * COLS + e0),
                             z = chan_load<T, 4>(zs + t * COLS + e0);
            ChanVec<4> o;
#pragma unroll
            for (int e = 0; e < 4; ++e) o.v[e] = fmaf(skip_e[e], x.v[e], v.v[e]) * sel_silu<T>(z.v[e]) * scale;
            if (vec_y) {
                chan_store<T, 4>(yo + t * y_ld, o);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (e0 + e < cols) yo[t * y_ld + e] = from_f32<T>(o.v[e]);
            }
        }
    };
    load(0);
    load(1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    rates(0);
    for (int k = 0; k <= chunks; ++k) {
        __syncthreads();                                              // chunk k has landed, the sums of k - 1 are there
        load(k + 2);                                                  // (into the stage of chunk k - 2, which no one reads any more)
        if (k > 0) finish(k - 1);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        rates(k + 1);
    }
    // the kept inputs: entry j takes the input of position end - (taps - 1) + j (entries that stay move down)
    const T* up = (const T*)in.u;
    for (int i = ht; i < cols; i += HALF) {
        float* kept = base + tail_off + col0 + i;
        for (int j = 0; j < taps - 1; ++j) {
            const int at = ctx + qlen - (taps - 1) + j;
            float v = 0.0f;
            if (at >= ctx) v = to_f32<T>(up[(long)(start + at - ctx) * in.u_ld + col0 + i]);
            else if (at >= 0) v = kept[(long)(j + qlen) * inner];
            kept[(long)j * inner] = v;
        }
    }
}

template <typename T, int R, int LANES, int COLS>
static int selective_scan_launch(const SelRows& in, const float* dt_bias, const float* a, const float* skip, float scale, T* y, long y_ld, float* state,
                                 long state_stride, long tail_off, int taps, const int* req_start, const int* req_ctx,
                                 const int* req_qlen, const int* req_slot, int n_requests, int inner, int n, bool overlap,
                                 cudaStream_t stream) {
    constexpr int CHUNK = R * LANES <= 64 ? 16 : 8;
    constexpr size_t smem = (size_t)SCAN_STAGES * CHUNK * ((2 * R * LANES + COLS) * 4 + 2 * COLS * sizeof(T)) + 2 * CHUNK * COLS * 4;
    auto kernel = selective_scan_kernel<T, R, LANES, COLS, CHUNK>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    constexpr int TV = 16 / (int)sizeof(T);
    auto rows16 = [&](const void* p, long ld) { return inner % TV == 0 && ld % TV == 0 && ((uintptr_t)p % 16) == 0 ? 1 : 0; };
    const int vec_low = n % 4 == 0 && in.b_at % 4 == 0 && in.c_at % 4 == 0 && in.low_ld % 4 == 0 && ((uintptr_t)in.low % 16) == 0;
    const int vec_dt = inner % 4 == 0 && in.dt_ld % 4 == 0 && ((uintptr_t)in.dt % 16) == 0;
    const int state_vec4 = n % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state % 16) == 0;
    return fl_launch_as(overlap, kernel, dim3(n_requests, (inner + COLS - 1) / COLS), dim3(2 * COLS * LANES), smem, stream, in, dt_bias, a, skip,
                        scale, y, y_ld, state, state_stride, tail_off, taps, req_start, req_ctx, req_qlen, req_slot, inner, n,
                        vec_low, vec_dt, rows16(in.x, in.x_ld), rows16(in.z, in.z_ld),
                        inner % 4 == 0 && chan_aligned(y, y_ld, sizeof(T)) ? 1 : 0, state_vec4);
}

static inline bool selective_takes(int inner, int n, int taps) {
    return n >= 1 && n <= 256 && inner >= 1 && (inner + 7) / 8 <= 65535 && taps >= 1 && taps <= 16;
}

// x, z, u, y: rows of the activation type; dt: W_dt dt without its bias; a: -exp(A_log) [inner][n], times log2(e) for bfloat16.  single_tokens: every
// request of the step brings one token (a short kernel).
FL_API int fl_selective_scan(const void* x, long x_ld, const void* z, long z_ld, const void* u, long u_ld, int dtype,
                             const float* dt, long dt_ld, const float* dt_bias, const float* low, long low_ld, int b_at, int c_at, const float* a,
                             const float* skip, float scale, void* y, long y_ld, float* state, long state_stride, long tail_off,
                             int taps, const int* req_start, const int* req_ctx, const int* req_qlen, const int* req_slot,
                             int n_requests, int inner, int n, int single_tokens, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (!selective_takes(inner, n, taps)) return (int)cudaErrorInvalidValue;
    const SelRows in{x, z, u, dt, low, x_ld, z_ld, u_ld, dt_ld, low_ld, b_at, c_at};
#define FL_SEL_SCAN(R, L, C)                                                                                                 \
    FL_DISPATCH(dtype, T, return selective_scan_launch<T, R, L, C>(in, dt_bias, a, skip, scale, (T*)y, y_ld, state, state_stride, tail_off, \
                                                                   taps, req_start, req_ctx, req_qlen, req_slot, n_requests, \
                                                                   inner, n, single_tokens != 0, stream))
    if (n <= 16) { FL_SEL_SCAN(4, 4, 32); }
    else if (n <= 32) { FL_SEL_SCAN(4, 8, 16); }
    else if (n <= 64) { FL_SEL_SCAN(8, 8, 16); }
    else if (n <= 128) { FL_SEL_SCAN(8, 16, 8); }
    else { FL_SEL_SCAN(16, 16, 8); }
#undef FL_SEL_SCAN
    return 0;
}

// ------------------------------------------------------------------ single tokens
// A warp's eight values of a weight row.
__device__ __forceinline__ void sel_load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void sel_load8(const bf16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}

// Row r of the step is request r's only token.  low: `splits` slabs of rows, added up in order while they are read (one
// slab: the rows themselves); w_dt: [inner][w_ld], w_ld a multiple of 8 and zero from column `rank` on.
template <typename T, typename TW, int R, int LANES, int COLS>
__global__ void __launch_bounds__(COLS * LANES) selective_step_kernel(
    const T* __restrict__ x, long x_ld, const T* __restrict__ z, long z_ld, const float* __restrict__ low, long low_ld, int splits,
    long split_stride, int rank, const TW* __restrict__ w_dt, int w_ld, const float* __restrict__ dt_bias,
    const float* __restrict__ a_log2, const float* __restrict__ skip, float scale, T* __restrict__ y, long y_ld,
    float* __restrict__ state, long state_stride, const int* __restrict__ req_ctx, const int* __restrict__ req_slot, int inner,
    int n, int state_vec4) {
    constexpr int DP = R * LANES, THREADS = COLS * LANES;
    extern __shared__ __align__(16) float step_s[];                   // B [DP] | C [DP] | dt's row [w_ld]
    const int r = blockIdx.y, tid = threadIdx.x, lane = tid & (LANES - 1), c = blockIdx.x * COLS + tid / LANES;
    const bool mine = c < inner;
    scan_f2 S[R / 2], A[R / 2];
    sel_rows<R, LANES>(A, a_log2 + (long)c * n, lane, n, mine, n % 4 == 0);
    const float skip_c = mine ? skip[c] : 0.0f, bias_c = mine ? dt_bias[c] : 0.0f;
    const int ctx = req_ctx[r];
    float* srow = state + (long)req_slot[r] * state_stride + (long)c * n;
    constexpr int KEEP = 4;                                           // of the weight row: vectors that wait in registers
    float w_keep[KEEP][8];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int k = (lane + i * LANES) * 8;
        if (mine && k < w_ld) sel_load8(w_dt + (long)c * w_ld + k, w_keep[i]);
    }
    pdl_wait();
    pdl_trigger();
    const float xv = mine ? to_f32<T>(x[(long)r * x_ld + c]) : 0.0f, zv = mine ? to_f32<T>(z[(long)r * z_ld + c]) : 0.0f;
    sel_rows<R, LANES>(S, srow, lane, n, mine && ctx != 0, state_vec4);
    for (int i = tid; i < 2 * DP + w_ld; i += THREADS) {
        int from = -1;
        if (i < DP) from = i < n ? rank + i : -1;
        else if (i < 2 * DP) from = i - DP < n ? rank + n + (i - DP) : -1;
        else from = i - 2 * DP < rank ? i - 2 * DP : -1;
        float v = 0.0f;
        if (from >= 0) {
            const float* p = low + (long)r * low_ld + from;
#pragma unroll 8
            for (int s = 0; s < splits; ++s) v += p[s * split_stride];
        }
        step_s[i] = v;
    }
    __syncthreads();
    const float* low_s = step_s + 2 * DP;
    float dot = 0.0f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int k = (lane + i * LANES) * 8;
        if (mine && k < w_ld)
#pragma unroll
            for (int e = 0; e < 8; ++e) dot = fmaf(w_keep[i][e], low_s[k + e], dot);
    }
    if (mine)
        for (int k = (lane + KEEP * LANES) * 8; k < w_ld; k += LANES * 8) {
            float w[8];
            sel_load8(w_dt + (long)c * w_ld + k, w);
#pragma unroll
            for (int e = 0; e < 8; ++e) dot = fmaf(w[e], low_s[k + e], dot);
        }
#pragma unroll
    for (int off = LANES / 2; off > 0; off >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, off);
    const float dt = sel_softplus<T>(dot + bias_c);
    SelToken<R> tok;
    sel_prepare<T, R, LANES>(tok, A, step_s, step_s + DP, dt, xv, lane);
    float sum = sel_apply<T, R>(S, tok);
#pragma unroll
    for (int off = LANES / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    if (!mine) return;
    if (lane == 0)
        y[(long)r * y_ld + c] = from_f32<T>(fmaf(skip_c, xv, sum) * sel_silu<T>(zv) * scale);
    sel_rows_out<R, LANES>(S, srow, lane, n, state_vec4);
}

FL_API int fl_selective_step(const void* x, long x_ld, const void* z, long z_ld, int dtype, const float* low, long low_ld,
                             int splits, long split_stride, int rank, const void* w_dt, int w_dtype, int w_ld,
                             const float* dt_bias, const float* a, const float* skip, float scale, void* y, long y_ld,
                             float* state, long state_stride, const int* req_ctx, const int* req_slot, int n_requests, int inner,
                             int n, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (!selective_takes(inner, n, 1) || n_requests > 65535 || rank < 1 || w_ld < rank || w_ld % 8 || ((uintptr_t)w_dt % 16) ||
        splits < 1 || w_ld > 8192)
        return (int)cudaErrorInvalidValue;
    const int state_vec4 = n % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state % 16) == 0;
#define FL_SEL_STEP(R, L, C)                                                                                                 \
    FL_DISPATCH(dtype, T, FL_DISPATCH(w_dtype, TW,                                                                           \
        return fl_launch(selective_step_kernel<T, TW, R, L, C>, dim3((inner + C - 1) / C, n_requests), dim3(C * L),          \
                         (size_t)(2 * R * L + w_ld) * sizeof(float), stream, (const T*)x, x_ld, (const T*)z, z_ld, low, low_ld, \
                         splits, split_stride, rank, (const TW*)w_dt, w_ld, dt_bias, a, skip, scale, (T*)y, y_ld, state,     \
                         state_stride, req_ctx, req_slot, inner, n, state_vec4)))
    if (n <= 16) { FL_SEL_STEP(4, 4, 32); }
    else if (n <= 32) { FL_SEL_STEP(4, 8, 16); }
    else if (n <= 64) { FL_SEL_STEP(8, 8, 16); }
    else if (n <= 128) { FL_SEL_STEP(8, 16, 8); }
    else { FL_SEL_STEP(16, 16, 8); }
#undef FL_SEL_STEP
    return 0;
}
