// Attention's per-head preparation with a short causal convolution in front of it.
//
// Per token, from one product's row (heads x dim queries | kv_heads x dim keys | kv_heads x vdim values), for every
// channel c of it:
//     u_t = row[c] + bias[c]        y_t = sum_j w[j][c] u_(t - taps + 1 + j)       (zeros before the sequence's start)
// and then, head by head: norm_mode 1: an RMS norm over the head's dim elements times q_w / k_w; the rotation of the first
// `rot` dimensions (pairs (2i, 2i + 1) with `interleaved`, else (i, i + rot / 2)) by the row `position` of cos / sin;
// norm_mode 2: an RMS norm without weight after the rotation; queries times 1 + coef ln(floor((position + 1) / every) + 1)
// where asked for.  Values are multiplied by v_scale.  q goes to q_out; k and v to the token's cache row, [kv_heads,
// page_size, dim + vdim].  Without taps there is no convolution; one tap needs no state.
//
// A request's last taps - 1 rows u (bias included) are its state, [taps - 1][channels] float, oldest first.
//
//   conv_head_prep   one warp a head and a few consecutive tokens: a lane holds the pairs that rotate together in
//                    registers, for these tokens and the taps - 1 rows before them.  A request that brings a single token has its state moved on here, by the lane that owns the channel
//   conv_head_tail   the new state of requests that bring several tokens (after every reader of the old one)
//
// All arithmetic is float; every sum's order depends on the channel alone.
#include "common.cuh"

#define CH_WARPS 4               // warps of a block: neighbouring heads of the same tokens

// N consecutive elements (N 1, 2 or a multiple of 4) from or to an address that is aligned for it.
template <int N> __device__ __forceinline__ void ch_get(const float* p, float* v) {
    if constexpr (N == 1) {
        v[0] = p[0];
    } else if constexpr (N == 2) {
        const float2 q = *reinterpret_cast<const float2*>(p);
        v[0] = q.x; v[1] = q.y;
    } else {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const float4 q = *reinterpret_cast<const float4*>(p + i);
            v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
        }
    }
}
template <int N> __device__ __forceinline__ void ch_get(const bf16* p, float* v) {
    if constexpr (N == 1) {
        v[0] = __bfloat162float(p[0]);
    } else if constexpr (N == 2) {
        const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        v[0] = q.x; v[1] = q.y;
    } else {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const uint2 raw = *reinterpret_cast<const uint2*>(p + i);
            const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
            const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
            v[i] = a.x; v[i + 1] = a.y; v[i + 2] = b.x; v[i + 3] = b.y;
        }
    }
}
template <int N> __device__ __forceinline__ void ch_put(float* p, const float* v) {
    if constexpr (N == 1) {
        p[0] = v[0];
    } else if constexpr (N == 2) {
        *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
    } else {
#pragma unroll
        for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
}
template <int N> __device__ __forceinline__ void ch_put(bf16* p, const float* v) {
    if constexpr (N == 1) {
        p[0] = __float2bfloat16_rn(v[0]);
    } else if constexpr (N == 2) {
        *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
    } else {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v[i], v[i + 1]), b = __floats2bfloat162_rn(v[i + 2], v[i + 3]);
            uint2 q;
            q.x = *reinterpret_cast<const uint32_t*>(&a);
            q.y = *reinterpret_cast<const uint32_t*>(&b);
            *reinterpret_cast<uint2*>(p + i) = q;
        }
    }
}

// How a lane's 2 PPL elements lie in a head, pair after pair: CH_RUN: consecutive channels from `first` on (pairs of
// neighbours); CH_HALVES: PPL channels from `first` on paired with those `half` further; CH_ANY: pairs found one by one.
enum { CH_RUN = 0, CH_HALVES = 1, CH_ANY = 2 };
template <int PPL, int MODE> struct ChLane {
    int size, turn, half, slot0;                                // slot0: the lane's first pair
    bool side;
    __device__ __forceinline__ int channel(int e) const {             // of element e; -1 where there is none
        const int s = slot0 + (e >> 1);
        int c;
        if (side) c = 2 * s + (e & 1);
        else if (s < half) c = s + (e & 1) * half;
        else c = turn + 2 * (s - half) + (e & 1);
        return c < size ? c : -1;
    }
    template <typename T> __device__ __forceinline__ void get(const T* p, float* v, float missing = 0.0f) const {
        if constexpr (MODE == CH_RUN) {
            if (2 * slot0 < size) { ch_get<2 * PPL>(p + 2 * slot0, v); return; }
        } else if constexpr (MODE == CH_HALVES) {
            if (slot0 < half) {
                float a[PPL], b[PPL];
                ch_get<PPL>(p + slot0, a);
                ch_get<PPL>(p + half + slot0, b);
#pragma unroll
                for (int i = 0; i < PPL; ++i) { v[2 * i] = a[i]; v[2 * i + 1] = b[i]; }
                return;
            }
        } else {
#pragma unroll
            for (int e = 0; e < 2 * PPL; ++e) {
                const int c = channel(e);
                v[e] = c >= 0 ? to_f32<T>(p[c]) : missing;
            }
            return;
        }
#pragma unroll
        for (int e = 0; e < 2 * PPL; ++e) v[e] = missing;
    }
    template <typename T> __device__ __forceinline__ void put(T* p, const float* v) const {
        if constexpr (MODE == CH_RUN) {
            if (2 * slot0 < size) ch_put<2 * PPL>(p + 2 * slot0, v);
        } else if constexpr (MODE == CH_HALVES) {
            if (slot0 < half) {
                float a[PPL], b[PPL];
#pragma unroll
                for (int i = 0; i < PPL; ++i) { a[i] = v[2 * i]; b[i] = v[2 * i + 1]; }
                ch_put<PPL>(p + slot0, a);
                ch_put<PPL>(p + half + slot0, b);
            }
        } else {
#pragma unroll
            for (int e = 0; e < 2 * PPL; ++e) {
                const int c = channel(e);
                if (c >= 0) p[c] = from_f32<T>(v[e]);
            }
        }
    }
};

template <typename T> __device__ __forceinline__ float ch_rms(float ss, int dim, float eps) {
    const float x = ss / (float)dim + eps;
    if constexpr (sizeof(T) == 2) return rsqrtf(x);                   // (two units in the last place of float)
    else return 1.0f / sqrtf(x);
}

struct ChRows {                  // the step's tables
    const int *positions, *tok_req, *req_start, *req_ctx, *req_qlen, *req_slot, *slots;
};

// PPL: pairs a lane holds (head sizes up to 64 PPL); TAPS: the layer's taps rounded up (1: one tap or no convolution), 0:
// any number, every earlier input read again for every token; RUN: consecutive tokens of a warp, whose rows (and the
// TAPS - 1 before them) are all asked for at once.
template <typename T> struct ChArgs {
    const T* proj;
    long ld;
    const float *bias, *conv_w;
    int taps;
    float* tail;
    long tail_stride;
    const float *q_w, *k_w;
    int norm_mode;
    float eps;
    int rot, interleaved;
    const float *cos_t, *sin_t;
    float temp_coef;
    int temp_every;
    float v_scale;
    ChRows rows;
    T* q_out;
    long q_ld;
    int heads, kv_heads, dim, vdim;
    T* cache;
    long page_stride;
    int page_size, page_shift, n_tokens, aligned;
};

template <typename T, int PPL, int TAPS, int RUN, int MODE>
__device__ __forceinline__ void conv_head_body(const ChArgs<T>& a, const int unit, const int lane) {
    constexpr int HIST = TAPS > 1 ? TAPS - 1 : 0;                     // rows before the run that its tokens may need
    constexpr int KEPT = TAPS > 0 ? TAPS : 1, E = 2 * PPL;
    const int heads = a.heads, kv_heads = a.kv_heads, dim = a.dim, vdim = a.vdim, taps = a.taps, n_tokens = a.n_tokens;
    const long ld = a.ld;
    const bool is_q = unit < heads, is_v = unit >= heads + kv_heads;
    const int size = is_v ? vdim : dim;
    const int g = is_q ? 0 : (is_v ? unit - heads - kv_heads : unit - heads);
    const int col0 = is_v ? (heads + kv_heads) * dim + g * vdim : unit * dim;
    const int channels = (heads + kv_heads) * dim + kv_heads * vdim;
    const int turn = is_v ? 0 : a.rot, half = turn / 2;
    ChLane<PPL, MODE> at;
    at.size = size; at.turn = turn; at.half = half; at.slot0 = PPL * lane;
    at.side = a.interleaved || turn == 0;
    const int t0 = blockIdx.x * RUN;

    // everything that does not depend on something else is asked for first
    float x[HIST + RUN][E];                                           // as projected, without the a.bias
    {
        const T* row = a.proj + (long)(t0 - HIST) * ld + col0;
#pragma unroll
        for (int i = 0; i < HIST + RUN; ++i, row += ld) {
            const int t = t0 + i - HIST;
            if (t >= 0 && t < n_tokens) at.get(row, x[i]);
            else
#pragma unroll
                for (int e = 0; e < E; ++e) x[i][e] = 0.0f;
        }
    }
    // what the step's tables say of the run's tokens, a token a lane
    int l_pos = 0, l_slot = 0, l_local = 0, l_row = 0, l_single = 0;  // local: tokens of the request in this step before it
    if (lane < RUN && t0 + lane < n_tokens) {
        l_pos = a.rows.positions[t0 + lane];
        l_slot = a.rows.slots[t0 + lane];
        if (TAPS != 1) {
            const int r = a.rows.tok_req[t0 + lane];
            l_local = t0 + lane - a.rows.req_start[r];
            l_row = a.rows.req_slot[r];
            l_single = a.rows.req_qlen[r] == 1;
        }
    }
    float b[E], gain[E], w[KEPT][E];
    const float* gain_p = is_v || a.norm_mode != 1 ? nullptr : (is_q ? a.q_w : a.k_w);
#pragma unroll
    for (int e = 0; e < E; ++e) { b[e] = 0.0f; gain[e] = 1.0f; }
    if (a.bias != nullptr) at.get(a.bias + col0, b);
    if (gain_p != nullptr) at.get(gain_p, gain, 1.0f);
    if (TAPS > 0 && a.conv_w != nullptr) {
#pragma unroll
        for (int j = 0; j < KEPT; ++j) {                              // tap j of the window is tap j - (KEPT - taps) of w
            const int k = j - (KEPT - taps);
            if (k >= 0) at.get(a.conv_w + (long)k * channels + col0, w[j]);
            else
#pragma unroll
                for (int e = 0; e < E; ++e) w[j][e] = 0.0f;
        }
    }
    int pos[RUN];
    float cosv[RUN][PPL], sinv[RUN][PPL];
#pragma unroll
    for (int u = 0; u < RUN; ++u) {
        pos[u] = __shfl_sync(0xffffffffu, l_pos, u);
        const long line = (long)pos[u] * half + at.slot0;
        if (at.slot0 + PPL <= half && half % PPL == 0) {
            ch_get<PPL>(a.cos_t + line, cosv[u]);
            ch_get<PPL>(a.sin_t + line, sinv[u]);
        } else {
#pragma unroll
            for (int p = 0; p < PPL; ++p) {
                cosv[u][p] = at.slot0 + p < half ? a.cos_t[line + p] : 1.0f;
                sinv[u][p] = at.slot0 + p < half ? a.sin_t[line + p] : 0.0f;
            }
        }
    }

    // a token's convolution with its inputs read one after another (oldest first, as everywhere), and its request's state
    auto any_taps = [&](int t, int p, int local, float* mine, int single, float (&y)[E]) {
        float keep[E], sum[E], wj[E], h[E];
#pragma unroll
        for (int e = 0; e < E; ++e) { keep[e] = y[e]; sum[e] = 0.0f; }
#pragma unroll 1
        for (int j = 0; j < taps - 1; ++j) {
            const int back = taps - 1 - j;
            if (p < back) continue;
            at.get(a.conv_w + (long)j * channels + col0, wj);
            if (local >= back) {
                at.get(a.proj + (long)(t - back) * ld + col0, h);
#pragma unroll
                for (int e = 0; e < E; ++e) h[e] += b[e];
            } else {
                at.get(mine + (long)(local - back + taps - 1) * channels, h);
            }
#pragma unroll
            for (int e = 0; e < E; ++e) sum[e] = fmaf(wj[e], h[e], sum[e]);
        }
        at.get(a.conv_w + (long)(taps - 1) * channels + col0, wj);
#pragma unroll
        for (int e = 0; e < E; ++e) y[e] = fmaf(wj[e], y[e], sum[e]);
        if (single && taps > 1) {
#pragma unroll 1
            for (int k = 0; k + 1 < taps - 1; ++k) {
                at.get(mine + (long)(k + 1) * channels, h);
                at.put(mine + (long)k * channels, h);
            }
            at.put(mine + (long)(taps - 2) * channels, keep);
        }
    };

#pragma unroll
    for (int u = 0; u < RUN; ++u) {
        const int t = t0 + u;
        const int slot = __shfl_sync(0xffffffffu, l_slot, u);
        float y[E];
#pragma unroll
        for (int e = 0; e < E; ++e) y[e] = x[HIST + u][e] + b[e];
        if constexpr (TAPS > 1) {
            // input `back` positions behind: from the step's rows, from the kept rows, or zero before the sequence's start
            const int local = __shfl_sync(0xffffffffu, l_local, u), state_row = __shfl_sync(0xffffffffu, l_row, u);
            const int single = __shfl_sync(0xffffffffu, l_single, u);
            float* mine = a.tail + (long)state_row * a.tail_stride + col0;
            float h[HIST][E];                                         // oldest first
#pragma unroll
            for (int j = 0; j < HIST; ++j) {
#pragma unroll
                for (int e = 0; e < E; ++e) h[j][e] = x[u + j][e] + b[e];
            }
            if (RUN > 1 && local < HIST) {                            // (the same for the whole warp) few tokens of a long step
                if (t < n_tokens) any_taps(t, pos[u], local, mine, single, y);
            } else {
            if (RUN == 1 && local < HIST && t < n_tokens) {           // the same for the whole warp
#pragma unroll
                for (int j = 0; j < HIST; ++j) {
                    const int back = HIST - j;
                    if (local >= back) continue;
                    if (pos[u] >= back && back <= taps - 1) {
                        at.get(mine + (long)(local - back + taps - 1) * channels, h[j]);
                    } else {
#pragma unroll
                        for (int e = 0; e < E; ++e) h[j][e] = 0.0f;
                    }
                }
            }
            float keep[E];
#pragma unroll
            for (int e = 0; e < E; ++e) {
                keep[e] = y[e];
                float sum = 0.0f;
#pragma unroll
                for (int j = 0; j < HIST; ++j) sum = fmaf(w[j][e], h[j][e], sum);
                y[e] = fmaf(w[TAPS - 1][e], y[e], sum);
            }
            if (RUN == 1 && single && t < n_tokens) {                 // the request's new state: the last taps - 1 inputs
#pragma unroll
                for (int j = 0; j < HIST; ++j) {
                    const int k = j - (TAPS - taps);
                    if (k >= 0) at.put(mine + (long)k * channels, j + 1 < HIST ? h[j + 1 < HIST ? j + 1 : j] : keep);
                }
            }
            }
        }
        if constexpr (TAPS == 0) {
            const int local = __shfl_sync(0xffffffffu, l_local, u), state_row = __shfl_sync(0xffffffffu, l_row, u);
            const int single = __shfl_sync(0xffffffffu, l_single, u);
            float* mine = a.tail + (long)state_row * a.tail_stride + col0;
            if (t < n_tokens) any_taps(t, pos[u], local, mine, single, y);
        }
        if constexpr (TAPS == 1) {
            if (a.conv_w != nullptr) {
#pragma unroll
                for (int e = 0; e < E; ++e) y[e] *= w[0][e];
            }
        }
        if (is_v) {
#pragma unroll
            for (int e = 0; e < E; ++e) y[e] *= a.v_scale;
        } else {
            if (a.norm_mode == 1) {
                float ss = 0.0f;
#pragma unroll
                for (int e = 0; e < E; ++e) ss = fmaf(y[e], y[e], ss);
                const float inv = ch_rms<T>(warp_sum(ss), dim, a.eps);
#pragma unroll
                for (int e = 0; e < E; ++e) y[e] = y[e] * inv * gain[e];
            }
#pragma unroll
            for (int p = 0; p < PPL; ++p) {
                const float v = y[2 * p], c = y[2 * p + 1];           // (no rotation: cos 1, sin 0)
                y[2 * p] = v * cosv[u][p] - c * sinv[u][p];
                y[2 * p + 1] = c * cosv[u][p] + v * sinv[u][p];
            }
            float f = 1.0f;
            if (a.norm_mode == 2) {
                float ss = 0.0f;
#pragma unroll
                for (int e = 0; e < E; ++e) ss = fmaf(y[e], y[e], ss);
                f = ch_rms<T>(warp_sum(ss), dim, a.eps);
            }
            if (is_q && a.temp_every > 0) f *= 1.0f + a.temp_coef * logf((float)((pos[u] + 1) / a.temp_every) + 1.0f);
#pragma unroll
            for (int e = 0; e < E; ++e) y[e] *= f;
        }
        if (t >= n_tokens) continue;
        T* dst;
        if (is_q) {
            dst = a.q_out + (long)t * a.q_ld + (long)unit * dim;
        } else {
            const int page = a.page_shift >= 0 ? slot >> a.page_shift : slot / a.page_size;
            dst = a.cache + (long)page * a.page_stride + ((long)g * a.page_size + (slot - page * a.page_size)) * (dim + vdim) + (is_v ? dim : 0);
        }
        at.put(dst, y);
    }
}

template <typename T, int PPL, int TAPS, int RUN>
__global__ void __launch_bounds__(32 * CH_WARPS) conv_head_prep_kernel(const ChArgs<T> a) {
    pdl_wait();
    pdl_trigger();
    const int unit = blockIdx.y * CH_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= a.heads + 2 * a.kv_heads) return;
    const bool is_v = unit >= a.heads + a.kv_heads;
    const int size = is_v ? a.vdim : a.dim, turn = is_v ? 0 : a.rot;
    const bool side = a.interleaved || turn == 0;                     // a pair's two channels are neighbours
    if (a.aligned && side && size % (2 * PPL) == 0) conv_head_body<T, PPL, TAPS, RUN, CH_RUN>(a, unit, lane);
    else if (a.aligned && !side && turn == size && turn / 2 % PPL == 0) conv_head_body<T, PPL, TAPS, RUN, CH_HALVES>(a, unit, lane);
    else conv_head_body<T, PPL, TAPS, RUN, CH_ANY>(a, unit, lane);
}

template <typename T>
__global__ void __launch_bounds__(256) conv_head_tail_kernel(const T* __restrict__ proj, long ld, const float* __restrict__ bias,
                                                             float* __restrict__ tail, long tail_stride,
                                                             const int* __restrict__ req_start, const int* __restrict__ req_ctx,
                                                             const int* __restrict__ req_qlen, const int* __restrict__ req_slot,
                                                             int channels, int taps) {
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    const int qlen = req_qlen[r];
    if (c >= channels || qlen == 1) return;                           // (single tokens: conv_head_prep moved the state on)
    const int start = req_start[r], ctx = req_ctx[r];
    float* mine = tail + (long)req_slot[r] * tail_stride + c;
    // entry j takes the input of position end - (taps - 1) + j; an entry that stays moves down, so upwards in place is safe
    for (int j = 0; j < taps - 1; ++j) {
        const int at = ctx + qlen - (taps - 1) + j;
        float u = 0.0f;
        if (at >= ctx) u = to_f32<T>(proj[(long)(start + at - ctx) * ld + c]) + (bias != nullptr ? bias[c] : 0.0f);
        else if (at >= 0) u = mine[(long)(j + qlen) * channels];
        mine[(long)j * channels] = u;
    }
}

// conv_w: [taps][channels] float, the last row the current token's (null, with taps 1: no convolution); tail: [slots][tail_stride] float.
// several: some request of the step brings more than one token.
FL_API int fl_conv_head_prep(const void* proj, int dtype, long ld, const float* bias, const float* conv_w, int taps, float* tail,
                             long tail_stride, const float* q_w, const float* k_w, int norm_mode, float eps, int rot,
                             int interleaved, const float* cos_t, const float* sin_t, float temp_coef, int temp_every,
                             float v_scale, const int* positions, const int* tok_req, const int* req_start,
                             const int* req_ctx, const int* req_qlen, const int* req_slot, const int* slots, void* q_out,
                             long q_ld, int n_tokens, int n_requests, int several, int heads, int kv_heads, int dim, int vdim,
                             void* cache, long page_stride, int page_size, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const int widest = dim > vdim ? dim : vdim;
    const int units = heads + 2 * kv_heads, channels = (heads + kv_heads) * dim + kv_heads * vdim;
    if (taps < 1 || (taps > 1 && (tail == nullptr || conv_w == nullptr)) || norm_mode < 0 || norm_mode > 2 ||
        rot < 0 || rot > dim || (rot & 1) || (rot > 0 && (cos_t == nullptr || sin_t == nullptr)) || widest > 512 ||
        cache == nullptr || n_requests > 65535 || units > 65535)
        return (int)cudaErrorInvalidValue;
    const ChRows rows{positions, tok_req, req_start, req_ctx, req_qlen, req_slot, slots};
    const size_t elem = dtype == FL_F32 ? 4 : 2;
    // several channels move as one where every head starts on a multiple of four elements of an aligned row
    const int aligned = dim % 4 == 0 && vdim % 4 == 0 && ld % 4 == 0 && q_ld % 4 == 0 && page_stride % 4 == 0 &&
                        ((uintptr_t)proj % (4 * elem)) == 0 && ((uintptr_t)q_out % (4 * elem)) == 0 && ((uintptr_t)cache % (4 * elem)) == 0 &&
                        ((uintptr_t)bias % 16) == 0 && ((uintptr_t)conv_w % 16) == 0 && ((uintptr_t)q_w % 16) == 0 &&
                        ((uintptr_t)k_w % 16) == 0 && ((uintptr_t)tail % 16) == 0 && tail_stride % 4 == 0;
    int page_shift = -1;
    if ((page_size & (page_size - 1)) == 0)
        for (page_shift = 0; (1 << page_shift) < page_size;) ++page_shift;
    int rc = 0;
#define FL_CH(PPL, TAPS, RUN)                                                                                            \
    FL_DISPATCH(dtype, T, {                                                                                             \
        const ChArgs<T> a{(const T*)proj, ld, bias, conv_w, taps, tail, tail_stride, q_w, k_w, norm_mode, eps, rot, interleaved, \
                          cos_t, sin_t, temp_coef, temp_every, v_scale, rows, (T*)q_out, q_ld, heads, kv_heads, dim, vdim, \
                          (T*)cache, page_stride, page_size, page_shift, n_tokens, aligned};                            \
        rc = fl_launch(conv_head_prep_kernel<T, PPL, TAPS, RUN>, dim3((n_tokens + RUN - 1) / RUN, (units + CH_WARPS - 1) / CH_WARPS), \
                       dim3(32 * CH_WARPS), 0, stream, a);                                                              \
    })
#define FL_CH_TAPS(PPL, RUN)                                                                                             \
    { if (taps == 1) { FL_CH(PPL, 1, RUN); } else if (taps <= 4) { FL_CH(PPL, 4, RUN); } else { FL_CH(PPL, 0, 1); } }
    const bool many = n_tokens >= 256;
    if (widest <= 64) { if (many) FL_CH_TAPS(1, 4) else FL_CH_TAPS(1, 1) }
    else if (widest <= 128) { if (many) FL_CH_TAPS(2, 4) else FL_CH_TAPS(2, 1) }
    else if (widest <= 256) FL_CH_TAPS(4, 1)
    else FL_CH_TAPS(8, 1)
#undef FL_CH_TAPS
#undef FL_CH
    if (rc || taps == 1 || !several) return rc;
    FL_DISPATCH(dtype, T, return fl_launch(conv_head_tail_kernel<T>, dim3((channels + 255) / 256, n_requests), dim3(256), 0, stream,
                                           (const T*)proj, ld, bias, tail, tail_stride, req_start, req_ctx, req_qlen, req_slot,
                                           channels, taps));
    return 0;
}
