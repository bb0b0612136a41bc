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
//   conv_head_prep   one warp a head and `run` consecutive tokens: a lane holds the pairs that rotate together in
//                    registers, and of each channel a window of the last taps - 1 inputs, so that a row is read once.  A
//                    request that brings a single token has its state moved on here, by the lane that owns the channel
//   conv_head_tail   the new state of requests that bring several tokens (after every reader of the old one)
//
// All arithmetic is float; every sum's order depends on the channel alone.
#include "common.cuh"

#define CH_WARPS 4               // warps of a block: neighbouring heads of the same tokens

// Two neighbouring channels at once where they lie on an even column.
__device__ __forceinline__ float2 ch_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ch_pair(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void ch_put_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void ch_put_pair(bf16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

struct ChRows {                  // the step's tables
    const int *positions, *tok_req, *req_start, *req_ctx, *req_qlen, *req_slot, *slots;
};

// PPL: pairs a lane holds (head sizes up to 64 PPL); TAPS: the window's length, the layer's taps rounded up; 0: any number
// of taps, every earlier input read again for every token.
template <typename T, int PPL, int TAPS>
__global__ void __launch_bounds__(32 * CH_WARPS) conv_head_prep_kernel(
    const T* __restrict__ proj, long ld, const float* __restrict__ bias, const float* __restrict__ conv_w, int taps,
    float* __restrict__ tail, long tail_stride, const float* __restrict__ q_w, const float* __restrict__ k_w, int norm_mode,
    float eps, int rot, int interleaved, const float* __restrict__ cos_t, const float* __restrict__ sin_t, float temp_coef,
    int temp_every, float v_scale, const ChRows rows, T* __restrict__ q_out, long q_ld, int heads, int kv_heads, int dim,
    int vdim, T* __restrict__ cache, long page_stride, int page_size, int n_tokens, int run, int pairs_ok) {
    pdl_wait();
    pdl_trigger();
    constexpr int WIN = TAPS > 1 ? TAPS - 1 : 1;
    const int lane = threadIdx.x & 31;
    const int unit = blockIdx.y * CH_WARPS + (threadIdx.x >> 5);
    if (unit >= heads + 2 * kv_heads) return;
    const bool is_q = unit < heads, is_v = unit >= heads + kv_heads;
    const int size = is_v ? vdim : dim;
    const int g = is_q ? 0 : (is_v ? unit - heads - kv_heads : unit - heads);
    const int col0 = is_v ? (heads + kv_heads) * dim + g * vdim : unit * dim;
    const int channels = (heads + kv_heads) * dim + kv_heads * vdim;
    const int turn = is_v ? 0 : rot, half = turn / 2;
    const bool side = interleaved || turn == 0;                       // a pair's two channels are neighbours

    int ca[PPL], cb[PPL];                                             // the pair's channels within the head (-1: none)
    constexpr int KEPT = TAPS > 0 ? TAPS : 1;
    float ba[PPL], bb[PPL], ga[PPL], gb[PPL], wa[PPL][KEPT], wb[PPL][KEPT];
    const float* gain = is_v || norm_mode != 1 ? nullptr : (is_q ? q_w : k_w);
#pragma unroll
    for (int p = 0; p < PPL; ++p) {
        const int s = lane + 32 * p;
        if (side) {
            ca[p] = 2 * s;
            cb[p] = 2 * s + 1;
        } else if (s < half) {
            ca[p] = s;
            cb[p] = s + half;
        } else {
            ca[p] = turn + 2 * (s - half);
            cb[p] = ca[p] + 1;
        }
        if (ca[p] >= size) ca[p] = -1;
        if (cb[p] >= size) cb[p] = -1;
        const int a = col0 + max(ca[p], 0), b = col0 + max(cb[p], 0);
        ba[p] = bias != nullptr && ca[p] >= 0 ? bias[a] : 0.0f;
        bb[p] = bias != nullptr && cb[p] >= 0 ? bias[b] : 0.0f;
        ga[p] = gain != nullptr && ca[p] >= 0 ? gain[max(ca[p], 0)] : 1.0f;
        gb[p] = gain != nullptr && cb[p] >= 0 ? gain[max(cb[p], 0)] : 1.0f;
        if (TAPS > 0 && conv_w != nullptr) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {                          // tap j of the window is tap j - (TAPS - taps) of w
                const int k = j - (TAPS - taps);
                wa[p][j] = k >= 0 && ca[p] >= 0 ? conv_w[(long)k * channels + a] : 0.0f;
                wb[p][j] = k >= 0 && cb[p] >= 0 ? conv_w[(long)k * channels + b] : 0.0f;
            }
        }
    }
    const bool vec = pairs_ok && side;
    auto load_u = [&](int t, int p, float& a, float& b) {
        const T* row = proj + (long)t * ld + col0;
        if (vec) {
            a = b = 0.0f;
            if (ca[p] >= 0) {
                const float2 v = ch_pair(row + ca[p]);                // (sizes are even where vec holds: both exist)
                a = v.x + ba[p];
                b = v.y + bb[p];
            }
        } else {
            a = ca[p] >= 0 ? to_f32<T>(row[ca[p]]) + ba[p] : 0.0f;
            b = cb[p] >= 0 ? to_f32<T>(row[cb[p]]) + bb[p] : 0.0f;
        }
    };

    float xa[WIN][PPL], xb[WIN][PPL];                                 // inputs of the positions before, oldest first
    const int t0 = blockIdx.x * run, t1 = min(n_tokens, t0 + run);
    int known = -1;                                                   // the request the window belongs to
    for (int t = t0; t < t1; ++t) {
        const int r = rows.tok_req[t];
        const int pos = rows.positions[t];
        float ya[PPL], yb[PPL];
#pragma unroll
        for (int p = 0; p < PPL; ++p) load_u(t, p, ya[p], yb[p]);
        if constexpr (TAPS > 1) {
            float* mine = tail + (long)rows.req_slot[r] * tail_stride + col0;
            if (r != known) {
                known = r;
                const int ctx = rows.req_ctx[r];
#pragma unroll
                for (int k = 0; k < WIN; ++k) {
                    const int back = WIN - k, at = pos - back;        // window entry k holds position pos - WIN + k
#pragma unroll
                    for (int p = 0; p < PPL; ++p) {
                        xa[k][p] = xb[k][p] = 0.0f;
                        if (at < 0 || back > taps - 1) continue;
                        if (at >= ctx) {
                            load_u(t - back, p, xa[k][p], xb[k][p]);
                        } else {
                            const float* kept = mine + (long)(at - ctx + taps - 1) * channels;
                            if (ca[p] >= 0) xa[k][p] = kept[ca[p]];
                            if (cb[p] >= 0) xb[k][p] = kept[cb[p]];
                        }
                    }
                }
            }
            const bool single = rows.req_qlen[r] == 1;
#pragma unroll
            for (int p = 0; p < PPL; ++p) {
                const float na = ya[p], nb = yb[p];
                float sa = 0.0f, sb = 0.0f;
#pragma unroll
                for (int j = 0; j < WIN; ++j) {
                    sa = fmaf(wa[p][j], xa[j][p], sa);
                    sb = fmaf(wb[p][j], xb[j][p], sb);
                }
                ya[p] = fmaf(wa[p][TAPS - 1], na, sa);
                yb[p] = fmaf(wb[p][TAPS - 1], nb, sb);
#pragma unroll
                for (int j = 0; j + 1 < WIN; ++j) {
                    xa[j][p] = xa[j + 1][p];
                    xb[j][p] = xb[j + 1][p];
                }
                xa[WIN - 1][p] = na;
                xb[WIN - 1][p] = nb;
                if (single) {                                         // the window is the request's new state
#pragma unroll
                    for (int j = 0; j < WIN; ++j) {
                        const int k = j - (TAPS - taps);
                        if (k < 0) continue;
                        if (ca[p] >= 0) mine[(long)k * channels + ca[p]] = xa[j][p];
                        if (cb[p] >= 0) mine[(long)k * channels + cb[p]] = xb[j][p];
                    }
                }
            }
        }
        if constexpr (TAPS == 0) {
            const int ctx = rows.req_ctx[r];
            float* mine = tail + (long)rows.req_slot[r] * tail_stride + col0;
            const bool single = rows.req_qlen[r] == 1;
#pragma unroll
            for (int p = 0; p < PPL; ++p) {
                const float na = ya[p], nb = yb[p];
                const int a = max(ca[p], 0), b = max(cb[p], 0);
                float sa = 0.0f, sb = 0.0f;
                for (int j = 0; j < taps - 1; ++j) {                  // oldest first
                    const int back = taps - 1 - j, at = pos - back;
                    if (at < 0) continue;
                    float ua, ub;
                    if (at >= ctx) {
                        load_u(t - back, p, ua, ub);
                    } else {
                        const float* kept = mine + (long)(at - ctx + taps - 1) * channels;
                        ua = kept[a];
                        ub = kept[b];
                    }
                    sa = fmaf(conv_w[(long)j * channels + col0 + a], ua, sa);
                    sb = fmaf(conv_w[(long)j * channels + col0 + b], ub, sb);
                }
                ya[p] = ca[p] >= 0 ? fmaf(conv_w[(long)(taps - 1) * channels + col0 + a], na, sa) : 0.0f;
                yb[p] = cb[p] >= 0 ? fmaf(conv_w[(long)(taps - 1) * channels + col0 + b], nb, sb) : 0.0f;
                if (single) {
                    for (int k = 0; k < taps - 1; ++k) {
                        if (ca[p] >= 0) mine[(long)k * channels + a] = k + 1 < taps - 1 ? mine[(long)(k + 1) * channels + a] : na;
                        if (cb[p] >= 0) mine[(long)k * channels + b] = k + 1 < taps - 1 ? mine[(long)(k + 1) * channels + b] : nb;
                    }
                }
            }
        }
        if constexpr (TAPS == 1) {
            if (conv_w != nullptr) {
#pragma unroll
                for (int p = 0; p < PPL; ++p) { ya[p] *= wa[p][0]; yb[p] *= wb[p][0]; }
            }
        }
        const int slot = rows.slots[t];
        const long page = slot / page_size;
        T* dst;
        if (is_q) dst = q_out + (long)t * q_ld + (long)unit * dim;
        else dst = cache + page * page_stride + ((long)g * page_size + (slot - (int)page * page_size)) * (dim + vdim) + (is_v ? dim : 0);
        if (is_v) {
#pragma unroll
            for (int p = 0; p < PPL; ++p) { ya[p] *= v_scale; yb[p] *= v_scale; }
        } else {
            if (norm_mode == 1) {
                float ss = 0.0f;
#pragma unroll
                for (int p = 0; p < PPL; ++p) ss += ya[p] * ya[p] + yb[p] * yb[p];
                const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
#pragma unroll
                for (int p = 0; p < PPL; ++p) { ya[p] = ya[p] * inv * ga[p]; yb[p] = yb[p] * inv * gb[p]; }
            }
#pragma unroll
            for (int p = 0; p < PPL; ++p) {
                const int i = lane + 32 * p;
                if (i < half) {
                    const float c = cos_t[(long)pos * half + i], sn = sin_t[(long)pos * half + i];
                    const float a = ya[p], b = yb[p];
                    ya[p] = a * c - b * sn;
                    yb[p] = b * c + a * sn;
                }
            }
            float f = 1.0f;
            if (norm_mode == 2) {
                float ss = 0.0f;
#pragma unroll
                for (int p = 0; p < PPL; ++p) ss += ya[p] * ya[p] + yb[p] * yb[p];
                f = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
            }
            if (is_q && temp_every > 0) f *= 1.0f + temp_coef * logf((float)((pos + 1) / temp_every) + 1.0f);
#pragma unroll
            for (int p = 0; p < PPL; ++p) { ya[p] *= f; yb[p] *= f; }
        }
#pragma unroll
        for (int p = 0; p < PPL; ++p) {
            if (vec) {
                if (ca[p] >= 0) ch_put_pair(dst + ca[p], ya[p], yb[p]);
            } else {
                if (ca[p] >= 0) dst[ca[p]] = from_f32<T>(ya[p]);
                if (cb[p] >= 0) dst[cb[p]] = from_f32<T>(yb[p]);
            }
        }
    }
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
    // two neighbouring channels move as one where every head starts on an even element of an aligned row
    const int pairs_ok = dim % 2 == 0 && vdim % 2 == 0 && ld % 2 == 0 && q_ld % 2 == 0 && page_stride % 2 == 0 &&
                         ((uintptr_t)proj % (2 * elem)) == 0 && ((uintptr_t)q_out % (2 * elem)) == 0 && ((uintptr_t)cache % (2 * elem)) == 0;
    const int run = n_tokens >= 1024 ? 8 : n_tokens >= 256 ? 4 : 1;
    dim3 grid((n_tokens + run - 1) / run, (units + CH_WARPS - 1) / CH_WARPS);
    int rc = 0;
#define FL_CH(PPL, TAPS)                                                                                                \
    FL_DISPATCH(dtype, T, rc = fl_launch(conv_head_prep_kernel<T, PPL, TAPS>, grid, dim3(32 * CH_WARPS), 0, stream,      \
                                         (const T*)proj, ld, bias, conv_w, taps, tail, tail_stride, q_w, k_w, norm_mode, \
                                         eps, rot, interleaved, cos_t, sin_t, temp_coef, temp_every, v_scale, rows,     \
                                         (T*)q_out, q_ld, heads, kv_heads, dim, vdim, (T*)cache, page_stride,          \
                                         page_size, n_tokens, run, pairs_ok))
#define FL_CH_TAPS(PPL)                                                                                                 \
    { if (taps == 1) { FL_CH(PPL, 1); } else if (taps <= 4) { FL_CH(PPL, 4); } else { FL_CH(PPL, 0); } }
    if (widest <= 64) FL_CH_TAPS(1)
    else if (widest <= 128) FL_CH_TAPS(2)
    else if (widest <= 256) FL_CH_TAPS(4)
    else FL_CH_TAPS(8)
#undef FL_CH_TAPS
#undef FL_CH
    if (rc || taps == 1 || !several) return rc;
    FL_DISPATCH(dtype, T, return fl_launch(conv_head_tail_kernel<T>, dim3((channels + 255) / 256, n_requests), dim3(256), 0, stream,
                                           (const T*)proj, ld, bias, tail, tail_stride, req_start, req_ctx, req_qlen, req_slot,
                                           channels, taps));
    return 0;
}
