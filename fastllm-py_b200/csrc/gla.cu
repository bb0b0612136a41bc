// Gated linear attention: a matrix state per head whose rows decay by numbers made from the token.
//
// Per token, from one product proj = [q | k | v | gate | low] (heads x dim, heads x dim, heads x vdim, heads x vdim,
// rank):
//     q' = q * q_scale,   z = W_2 low + b_2 (heads x dim),   alpha = sigmoid(z)^(1 / tau) = exp(logsigmoid(z) / tau)
//     S <- diag(alpha) S + k v^T      (S: dim x vdim per head; alpha acts on the rows, one per key channel)
//     o = S^T q'
// then each head's o is divided by its root mean square over vdim, multiplied by a weight [vdim] shared by the heads and
// by silu(gate).  A request's state row is S for every head, [heads][vdim][dim] float; it is read unless the request
// starts (context 0) and written at the end of the step.
//
//   gla_prep         per token: q', k, alpha, v widened to float in one work row; the small product W_2 low on the CUDA
//                    cores in float
//   gla_scan         the recurrence over each request's tokens in order (state_scan.cuh, a decay per row)
//   gla_gated_norm   per (token, head): norm, weight, gate
//
// Everything after the product is float.  Every sum's order depends on the token alone.
#include "state_scan.cuh"

// work row: q' (heads x dim) | k (heads x dim) | alpha (heads x dim) | v (heads x vdim), float.
// w2: the decay's second matrix transposed, [rank][heads x dim], so that neighbouring threads read neighbouring floats.
template <typename T>
__global__ void __launch_bounds__(256) gla_prep_kernel(const T* __restrict__ proj, long ld, const float* __restrict__ w2,
                                                       const float* __restrict__ b2, float* __restrict__ work, long w_ld,
                                                       int heads, int dim, int vdim, int rank, float q_scale, float tau) {
    pdl_wait();
    pdl_trigger();
    extern __shared__ float low_s[];                    // [rank]
    const long t = blockIdx.x;
    const T* row = proj + t * ld;
    const int hd = heads * dim, hv = heads * vdim;
    for (int i = threadIdx.x; i < rank; i += blockDim.x) low_s[i] = to_f32<T>(row[2 * hd + 2 * hv + i]);
    __syncthreads();
    float* w = work + t * w_ld;
    // (blockIdx.y shares a token's columns out over blocks: a handful of tokens alone would leave the GPU idle)
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < hd; i += gridDim.y * blockDim.x) {
        w[i] = to_f32<T>(row[i]) * q_scale;
        w[hd + i] = to_f32<T>(row[hd + i]);
        float z = b2[i];
        for (int k = 0; k < rank; ++k) z += w2[(long)k * hd + i] * low_s[k];       // w2 is stored [rank][heads x dim]
        const float logsig = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
        w[2 * hd + i] = expf(logsig / tau);
    }
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < hv; i += gridDim.y * blockDim.x) w[3 * hd + i] = to_f32<T>(row[2 * hd + i]);
}

template <typename T, typename TW>
__global__ void __launch_bounds__(128) gla_gated_norm_kernel(const float* __restrict__ o, long o_ld, const T* __restrict__ gate,
                                                             long g_ld, const TW* __restrict__ weight, T* __restrict__ out,
                                                             long out_ld, int n_tokens, int heads, int vdim, float eps) {
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long pair = (long)blockIdx.x * 4 + warp;
    if (pair >= (long)n_tokens * heads) return;
    const long t = pair / heads;
    const int h = (int)(pair - t * heads);
    const float* orow = o + t * o_ld + (long)h * vdim;
    float ss = 0.0f;
    for (int d = lane; d < vdim; d += 32) ss += orow[d] * orow[d];
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int d = lane; d < vdim; d += 32) {
        const float g = to_f32<T>(gate[t * g_ld + (long)h * vdim + d]);
        const float w = weight != nullptr ? to_f32<TW>(weight[d]) : 1.0f;
        out[t * out_ld + (long)h * vdim + d] = from_f32<T>(orow[d] * inv * w * (g / (1.0f + expf(-g))));
    }
}

FL_API int fl_gla_prep(const void* proj, int dtype, long ld, const float* w2, const float* b2, float* work, long w_ld,
                       int n_tokens, int heads, int dim, int vdim, int rank, float q_scale, float tau, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rank < 1 || (size_t)rank * sizeof(float) > 48 * 1024 || !(tau > 0.0f)) return (int)cudaErrorInvalidValue;
    int share = n_tokens >= 256 ? 1 : (heads * dim + 255) / 256;
    if (share > 16) share = 16;
    FL_DISPATCH(dtype, T, return fl_launch(gla_prep_kernel<T>, dim3(n_tokens, share), dim3(256), (size_t)rank * sizeof(float), stream,
                                           (const T*)proj, ld, w2, b2, work, w_ld, heads, dim, vdim, rank, q_scale,
                                           tau));
    return 0;
}

// work: what fl_gla_prep leaves.  single_tokens: every request of the step brings one token.
FL_API int fl_gla_scan(const float* work, long w_ld, float* o, long o_ld, float* state, long state_stride,
                       const int* req_start, const int* req_ctx, const int* req_qlen, const int* req_slot, int n_requests,
                       int heads, int dim, int vdim, int single_tokens, cudaStream_t stream) {
    const int hd = heads * dim;
    const ScanToken at{hd, 0, dim, 1, 2 * hd, 3 * hd, 0, 0};
    return state_scan<false>(work, w_ld, at, nullptr, o, o_ld, state, state_stride, req_start, req_ctx, req_qlen, req_slot,
                             n_requests, heads, dim, vdim, single_tokens, stream);
}

FL_API int fl_gla_gated_norm(const float* o, long o_ld, const void* gate, int dtype, long g_ld, const void* weight,
                             int w_dtype, void* out, long out_ld, int n_tokens, int heads, int vdim, float eps,
                             cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const long pairs = (long)n_tokens * heads;
    FL_DISPATCH(dtype, T, FL_DISPATCH(w_dtype, TW,
        return fl_launch(gla_gated_norm_kernel<T, TW>, dim3((unsigned)((pairs + 3) / 4)), dim3(128), 0, stream, o, o_ld,
                         (const T*)gate, g_ld, (const TW*)weight, (T*)out, out_ld, n_tokens, heads, vdim, eps)));
    return 0;
}
