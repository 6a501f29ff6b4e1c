// What surrounds the attention of the differential kind: two softmax maps per head over the same
// values, whose results are combined as  a1 - lambda a2  and normed.
//
// The attention itself is the paged attention of 2H query heads over G key/value heads.  A cached
// key row of head g holds both maps' keys side by side, [k1: D | k2: D]; the query of map 1 is
// [q1 | 0], of map 2 [0 | q2], so a row's scores are the map's own (the zeros add nothing), a key
// row and a value row are read once for both maps, and any attention kernel that takes keys of
// 2D and values of E features serves.
//
// (1) Preparation of a step's rows, one block per token.  A row of the joint projection is
//     [q: H*2*D | k: G*2*D | v: G*E | ...] without its biases.  q = (row + bias) * temperature(p),
//     temperature(p) = 1 + coef * ln(floor((p + 1) / every) + 1) (1 without one), spread out as
//     above; k and v with their biases go to the token's place in the pages.  fp32 arithmetic,
//     one rounding.
// (2) Combination, one block per token: per head o = a1 - lambda a2, divided by
//     sqrt(mean(o^2) + eps) over its E values, times `scale`; and the output projection's bias
//     joins the residual row (the product that follows adds to it).
#define CB_PDL_BIT 15      // this file's bit in CRUCIBLE_PDL
#include "common.cuh"

namespace {

// PER neighbouring features, one map's and one head's
template <typename T, int PER> struct Run { T v[PER]; };
template <> struct __align__(4) Run<__nv_bfloat16, 2> { __nv_bfloat16 v[2]; };
template <> struct __align__(8) Run<float, 2> { float v[2]; };

// PER 2: even sizes, rows and pages on boundaries of two elements
template <typename T, int PER>
__global__ void differential_prepare_kernel(const T* __restrict__ proj, int proj_stride,
                                            const float* __restrict__ bias, float coef, int every,
                                            const int* __restrict__ positions,
                                            const int* __restrict__ row_request,
                                            const int* __restrict__ block_table, int table_stride,
                                            T* __restrict__ qx, int qx_stride, T* __restrict__ k_cache,
                                            T* __restrict__ v_cache, int n_heads, int n_kv_heads, int dim,
                                            int value_dim, int page_tokens, int write_cache) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const int t = blockIdx.x;
    const T* row = proj + (size_t)t * proj_stride;
    const int pos = positions[t];
    const float temp = every > 0 ? fmaf(coef, logf((float)((pos + 1) / every) + 1.0f), 1.0f) : 1.0f;
    const int two = 2 * dim, nq = n_heads * two, nk = n_kv_heads * two;
    T* q = qx + (size_t)t * qx_stride;
    // place i of the spread row: query head i / two (head h, map m at 2h + m), feature i % two
    auto take = [&](int src, float factor) {
        Run<T, PER> r = *reinterpret_cast<const Run<T, PER>*>(row + src);
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            float v = cb_to_float(r.v[e]);
            if (bias != nullptr) v += bias[src + e];
            r.v[e] = cb_from_float<T>(v * factor);
        }
        return r;
    };
    for (int i = threadIdx.x * PER; i < 2 * nq; i += blockDim.x * PER) {
        const int head = i / two, f = i - head * two;
        const int map = head & 1;
        Run<T, PER> r;
#pragma unroll
        for (int e = 0; e < PER; ++e) r.v[e] = cb_from_float<T>(0.f);
        if ((f >= dim) == (map != 0)) r = take((head >> 1) * two + f, temp);      // [map 1 | map 2] of head h
        *reinterpret_cast<Run<T, PER>*>(q + i) = r;
    }
    if (!write_cache) return;
    const int page = block_table[(size_t)row_request[t] * table_stride + pos / page_tokens];
    const size_t at = (size_t)page * n_kv_heads * page_tokens + pos % page_tokens;
    for (int i = threadIdx.x * PER; i < nk; i += blockDim.x * PER) {
        const int g = i / two, f = i - g * two;
        *reinterpret_cast<Run<T, PER>*>(k_cache + (at + (size_t)g * page_tokens) * two + f) = take(nq + i, 1.0f);
    }
    for (int i = threadIdx.x * PER; i < n_kv_heads * value_dim; i += blockDim.x * PER) {
        const int g = i / value_dim, f = i - g * value_dim;
        *reinterpret_cast<Run<T, PER>*>(v_cache + (at + (size_t)g * page_tokens) * value_dim + f) =
            take(nq + nk + i, 1.0f);
    }
}

template <typename T>
__global__ void differential_combine_kernel(const T* __restrict__ a, int a_stride, float lambda, float eps,
                                            float scale, T* __restrict__ out, int out_stride,
                                            const float* __restrict__ out_bias, float* __restrict__ residual,
                                            int width, int n_heads, int value_dim) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const int t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    for (int h = warp; h < n_heads; h += n_warps) {
        const T* a1 = a + (size_t)t * a_stride + (size_t)2 * h * value_dim;
        const T* a2 = a1 + value_dim;
        float ss = 0.f;
        for (int e = lane; e < value_dim; e += 32) {
            const float o = fmaf(-lambda, cb_to_float(a2[e]), cb_to_float(a1[e]));
            ss = fmaf(o, o, ss);
        }
        const float r = scale / sqrtf(cb_warp_sum(ss) / (float)value_dim + eps);
        T* dst = out + (size_t)t * out_stride + (size_t)h * value_dim;
        for (int e = lane; e < value_dim; e += 32)
            dst[e] = cb_from_float<T>(fmaf(-lambda, cb_to_float(a2[e]), cb_to_float(a1[e])) * r);
    }
    if (out_bias != nullptr)
        for (int i = threadIdx.x; i < width; i += blockDim.x) residual[(size_t)t * width + i] += out_bias[i];
}

}  // namespace

// every 0: no temperature.  bias: fp32 over the row's q, k and v columns, or null.
CB_EXPORT int cb_differential_prepare(const void* proj, int proj_stride, int dtype, const float* bias,
                                      float coef, int every, const int* positions, const int* row_request,
                                      const int* block_table, int table_stride, void* qx, int qx_stride,
                                      void* k_cache, void* v_cache, int n_rows, int n_heads,
                                      int n_kv_heads, int dim, int value_dim, int page_tokens,
                                      int write_cache, void* stream) {
    if (n_rows <= 0) return 0;
    if (dim <= 0 || value_dim <= 0 || every < 0 || n_heads % n_kv_heads != 0) return CB_ERR_UNSUPPORTED;
    const int places = 4 * n_heads * dim;
    const dim3 block(places >= 2048 ? 512 : (places >= 512 ? 256 : 128));
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t unit = dtype == CB_F32 ? 8 : 4;
    const bool pairs = !((dim | value_dim | proj_stride | qx_stride) & 1) &&
                       (((uintptr_t)proj | (uintptr_t)qx | (uintptr_t)k_cache | (uintptr_t)v_cache) & (unit - 1)) == 0;
#define CB_DP(TT, PP)                                                                                          \
    cb_launch(differential_prepare_kernel<TT, PP>, dim3(n_rows), block, 0, s, (const TT*)proj, proj_stride,    \
              bias, coef, every, positions, row_request, block_table, table_stride, (TT*)qx, qx_stride,        \
              (TT*)k_cache, (TT*)v_cache, n_heads, n_kv_heads, dim, value_dim, page_tokens, write_cache)
    if (dtype == CB_F32) { if (pairs) CB_DP(float, 2); else CB_DP(float, 1); }
    else { if (pairs) CB_DP(__nv_bfloat16, 2); else CB_DP(__nv_bfloat16, 1); }
#undef CB_DP
    return cb_last_error();
}

// a: T rows of 2 * n_heads results of value_dim (map 1 of head h at 2h); out: T rows of n_heads.
// out_bias (fp32 [width], or null) is added to the fp32 residual rows.
CB_EXPORT int cb_differential_combine(const void* a, int a_stride, int dtype, float lambda, float eps,
                                      float scale, void* out, int out_stride, const float* out_bias,
                                      float* residual, int width, int n_rows, int n_heads, int value_dim,
                                      void* stream) {
    if (n_rows <= 0) return 0;
    const dim3 block(n_heads >= 8 ? 256 : 128);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == CB_F32)
        cb_launch(differential_combine_kernel<float>, dim3(n_rows), block, 0, s, (const float*)a, a_stride, lambda,
                  eps, scale, (float*)out, out_stride, out_bias, residual, width, n_heads, value_dim);
    else
        cb_launch(differential_combine_kernel<__nv_bfloat16>, dim3(n_rows), block, 0, s, (const __nv_bfloat16*)a,
                  a_stride, lambda, eps, scale, (__nv_bfloat16*)out, out_stride, out_bias, residual, width, n_heads,
                  value_dim);
    return cb_last_error();
}
