// The end of a layer whose two sublayers read the same rows and leave their results unsummed, and the
// norms of what follows, in one launch over the fp32 residual:
//   x[t] += s1 * mixer[t] + s2 * (sum_j w[t][j] * rows[place of (t, j)] + g[t] * shared[t])
//   out_i[t] = x[t] / sqrt(mean(x[t]^2) + eps_i) * gain_i,  i < n_norms (0, 1 or 2)
// s1, s2: vectors over the width (null: ones); mixer, rows, shared may each be absent.  `rows` are the
// experts' results: by pair and already weighted (offsets null), or in the sorted order of a routing
// plan and weighted here; g null: ones.  With all of them absent it is a norm (or two) of x alone.
// One block per token; everything is fp32 in a fixed order, the block's size a function of the width.
//
// And the rows of a repeated run's entry: rows_out[t] = x[t] in the products' type, then
// x[t] = next[t] (null: x stays).
#define CB_PDL_BIT 3      // launched under the elementwise kernels' bit of CRUCIBLE_PDL
#define CB_PDL_MAX_BLOCKS 148
#include "common.cuh"

namespace {

struct CloseArgs {
    float* x;
    const float *mixer, *s1, *s2;
    const float* rows;
    int top;
    const int *offsets, *idx, *place;
    const float *weight, *shared, *gate;
    int n_norms;
    const float *gain0, *gain1;
    float eps0, eps1;
    void *out0, *out1;
    int width;
};

template <int V> struct Piece { float v[V]; };
template <int V>
__device__ __forceinline__ Piece<V> load_piece(const float* p) {
    Piece<V> r;
    if constexpr (V == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V>
__device__ __forceinline__ void store_piece(float* p, const Piece<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void store_piece(__nv_bfloat16* p, const Piece<V>& r) {
    if constexpr (V == 4) {
        __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 w;
        w.x = *reinterpret_cast<uint32_t*>(&a);
        w.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = w;
    } else {
        *p = __float2bfloat16(r.v[0]);
    }
}

// The new residual at columns i .. i + V - 1 of token t.
template <int V>
__device__ __forceinline__ Piece<V> close_piece(const CloseArgs& a, int t, int i) {
    const size_t at = (size_t)t * a.width + i;
    Piece<V> x = load_piece<V>(a.x + at);
    if (a.mixer == nullptr && a.rows == nullptr && a.shared == nullptr) return x;
    Piece<V> add;
#pragma unroll
    for (int e = 0; e < V; ++e) add.v[e] = 0.f;
    if (a.mixer != nullptr) {
        const Piece<V> m = load_piece<V>(a.mixer + at);
#pragma unroll
        for (int e = 0; e < V; ++e) add.v[e] = m.v[e];
        if (a.s1 != nullptr) {
            const Piece<V> s = load_piece<V>(a.s1 + i);
#pragma unroll
            for (int e = 0; e < V; ++e) add.v[e] *= s.v[e];
        }
    }
    if (a.rows != nullptr || a.shared != nullptr) {
        Piece<V> f;
#pragma unroll
        for (int e = 0; e < V; ++e) f.v[e] = 0.f;
        auto join = [&](const float* src, float w) {
            const Piece<V> r = load_piece<V>(src);
#pragma unroll
            for (int e = 0; e < V; ++e) f.v[e] = fmaf(w, r.v[e], f.v[e]);
        };
        if (a.rows != nullptr) {
            for (int j = 0; j < a.top; ++j) {
                const size_t p = (size_t)t * a.top + j;
                if (a.offsets == nullptr) join(a.rows + p * a.width + i, 1.0f);
                else join(a.rows + (size_t)(a.offsets[a.idx[p]] + a.place[p]) * a.width + i, a.weight[p]);
            }
        }
        if (a.shared != nullptr) join(a.shared + at, a.gate != nullptr ? a.gate[t] : 1.0f);
        if (a.s2 != nullptr) {
            const Piece<V> s = load_piece<V>(a.s2 + i);
#pragma unroll
            for (int e = 0; e < V; ++e) add.v[e] = fmaf(s.v[e], f.v[e], add.v[e]);
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) add.v[e] += f.v[e];
        }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) x.v[e] += add.v[e];
    store_piece<V>(a.x + at, x);
    return x;
}

template <typename T, int V>
__device__ __forceinline__ void norm_piece(const CloseArgs& a, int t, int i, const Piece<V>& x, float r0, float r1) {
    const size_t at = (size_t)t * a.width + i;
    Piece<V> g = load_piece<V>(a.gain0 + i), y;
#pragma unroll
    for (int e = 0; e < V; ++e) y.v[e] = x.v[e] * r0 * g.v[e];
    store_piece<V>((T*)a.out0 + at, y);
    if (a.n_norms < 2) return;
    g = load_piece<V>(a.gain1 + i);
#pragma unroll
    for (int e = 0; e < V; ++e) y.v[e] = x.v[e] * r1 * g.v[e];
    store_piece<V>((T*)a.out1 + at, y);
}

// PER: pieces of V columns that a thread keeps between the two passes (0: any number, read again).
template <typename T, int V, int PER>
__global__ void __launch_bounds__(PER > 0 ? 512 : 1024) layer_close_kernel(CloseArgs a) {
    cb_pdl_trigger();
    cb_pdl_wait();
    __shared__ float scratch[32];
    const int t = blockIdx.x, step = blockDim.x * V;
    float ss = 0.f;
    Piece<V> kept[PER > 0 ? PER : 1];
    if constexpr (PER > 0) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int i = threadIdx.x * V + j * step;
            if (i < a.width) {
                kept[j] = close_piece<V>(a, t, i);
#pragma unroll
                for (int e = 0; e < V; ++e) ss = fmaf(kept[j].v[e], kept[j].v[e], ss);
            }
        }
    } else {
        for (int i = threadIdx.x * V; i < a.width; i += step) {
            const Piece<V> x = close_piece<V>(a, t, i);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(x.v[e], x.v[e], ss);
        }
    }
    if (a.n_norms == 0) return;
    const float mean = cb_block_sum(ss, scratch) / (float)a.width;
    const float r0 = 1.0f / sqrtf(mean + a.eps0), r1 = a.n_norms > 1 ? 1.0f / sqrtf(mean + a.eps1) : 0.f;
    if constexpr (PER > 0) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int i = threadIdx.x * V + j * step;
            if (i < a.width) norm_piece<T, V>(a, t, i, kept[j], r0, r1);
        }
    } else {
        for (int i = threadIdx.x * V; i < a.width; i += step)       // (columns this thread itself wrote)
            norm_piece<T, V>(a, t, i, load_piece<V>(a.x + (size_t)t * a.width + i), r0, r1);
    }
}

template <typename T>
int launch_close(const CloseArgs& a, int n_rows, bool vec, cudaStream_t s) {
    const int n4 = a.width >> 2;
    auto threads = [](int n) { return n < 32 ? 32 : (n + 31) / 32 * 32; };
    if (vec && n4 <= 256) cb_launch(layer_close_kernel<T, 4, 1>, dim3(n_rows), dim3(threads(n4)), 0, s, a);
    else if (vec && n4 <= 512) cb_launch(layer_close_kernel<T, 4, 2>, dim3(n_rows), dim3(threads((n4 + 1) / 2)), 0, s, a);
    else if (vec && n4 <= 2048) cb_launch(layer_close_kernel<T, 4, 4>, dim3(n_rows), dim3(threads((n4 + 3) / 4)), 0, s, a);
    else if (vec) cb_launch(layer_close_kernel<T, 4, 0>, dim3(n_rows), dim3(1024), 0, s, a);
    else cb_launch(layer_close_kernel<T, 1, 0>, dim3(n_rows), dim3(a.width >= 1024 ? 256 : 128), 0, s, a);
    return cb_last_error();
}

template <typename T, int V>
__global__ void swap_rows_kernel(float* __restrict__ x, T* __restrict__ rows_out, const float* __restrict__ next,
                                 int width) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const size_t row = (size_t)blockIdx.x * width;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        store_piece<V>(rows_out + row + i, load_piece<V>(x + row + i));
        if (next != nullptr) store_piece<V>(x + row + i, load_piece<V>(next + row + i));
    }
}

}  // namespace

CB_EXPORT int cb_layer_close(float* x, const float* mixer, const float* s1, const float* s2, const float* rows,
                             int top, const int* plan, const int* idx, const int* place, const float* weight,
                             const float* shared, const float* gate, int n_norms, const float* gain0, float eps0,
                             void* out0, const float* gain1, float eps1, void* out1, int out_dtype, int n_rows,
                             int width, void* stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0 || n_norms < 0 || n_norms > 2) return CB_ERR_UNSUPPORTED;
    const CloseArgs a = {x, mixer, s1, s2, rows, top, plan != nullptr ? plan + 1 : nullptr, idx, place, weight,
                         shared, gate, n_norms, gain0, gain1, eps0, eps1, out0, out1, width};
    const uintptr_t all = (uintptr_t)x | (uintptr_t)mixer | (uintptr_t)s1 | (uintptr_t)s2 | (uintptr_t)rows |
                          (uintptr_t)shared | (uintptr_t)gain0 | (uintptr_t)gain1 | (uintptr_t)out0 | (uintptr_t)out1;
    const bool vec = (width & 3) == 0 && (all & 15) == 0;
    return out_dtype == CB_F32 ? launch_close<float>(a, n_rows, vec, (cudaStream_t)stream)
                               : launch_close<__nv_bfloat16>(a, n_rows, vec, (cudaStream_t)stream);
}

CB_EXPORT int cb_swap_rows(float* x, void* rows_out, int out_dtype, const float* next, int n_rows, int width,
                           void* stream) {
    if (n_rows <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = (width & 3) == 0 && ((((uintptr_t)x | (uintptr_t)rows_out | (uintptr_t)next)) & 15) == 0;
    const dim3 block(width >= 1024 ? 256 : 128);
#define CB_SWAP(TT, VV) cb_launch(swap_rows_kernel<TT, VV>, dim3(n_rows), block, 0, s, x, (TT*)rows_out, next, width)
    if (out_dtype == CB_F32) { if (vec) CB_SWAP(float, 4); else CB_SWAP(float, 1); }
    else { if (vec) CB_SWAP(__nv_bfloat16, 4); else CB_SWAP(__nv_bfloat16, 1); }
#undef CB_SWAP
    return cb_last_error();
}
