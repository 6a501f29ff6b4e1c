// RMS norm of the residual rows and, on what it leaves, a short causal convolution over time
// per channel, added to it:
//   h[t] = x[t] / sqrt(mean(x[t]^2) + eps) * gain,
//   out[t] = h[t] + sum_j w[j] * h[t - taps + 1 + j]        (h zero before the sequence's start).
// A request's last taps - 1 rows h are state (fp32 [taps-1][width], oldest first, in its state
// slot, zeros when the slot is handed out); a portion's first tokens read them and the portion
// leaves its own last ones.  Norm, convolution and sum are fp32 on unrounded h; only the result
// is rounded to T.
//
// One launch: a block takes `tile` tokens of one request (grid x: tiles, y: requests) and a run
// of columns (grid z).  First the rows' factors: the sum of squares of a row is eight shares
// (share s: the pieces s, s + 8, ... of 32 vectors), each summed by one warp, added in order, so
// a row's sum has one order whatever the launch's shape.  Then every thread walks the tile's
// tokens down its own columns with the last taps - 1 rows in registers.  The first tile's block
// alone reads the old state, and it alone writes the new one, thread by thread for its own
// columns after it has read them, so no other block meets either.
// Rows of up to 4,096 floats (a multiple of 4) with two to five taps run in a form that reads x
// once: a thread owns four or eight columns for all rows of the tile, keeps them in registers, and
// the rows' sums of squares are reduced over the block together (the block's size is a function of
// the width alone, so a row's sum has one order here too).
#define CB_PDL_BIT 14      // this file's bit in CRUCIBLE_PDL
#include "common.cuh"

namespace {

constexpr int SHARES = 8;

template <int V> struct Vec;
template <> struct Vec<4> {
    float v[4];
    __device__ __forceinline__ void load(const float* p) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    }
    __device__ __forceinline__ void store(float* p) const {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
    __device__ __forceinline__ void put(float* p) const { store(p); }
    __device__ __forceinline__ void put(__nv_bfloat16* p) const {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&a);
        u.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = u;
    }
};
template <> struct Vec<1> {
    float v[1];
    __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
    __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
    __device__ __forceinline__ void put(float* p) const { *p = v[0]; }
    __device__ __forceinline__ void put(__nv_bfloat16* p) const { *p = __float2bfloat16_rn(v[0]); }
};

// TAPS: the number of taps (2..5), or 0: `taps_` of them, the earlier rows read again per token.
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(256) norm_conv_kernel(
    const float* __restrict__ x, const float* __restrict__ gain, float eps, const float* __restrict__ w,
    int taps_, const int* __restrict__ req_row_start, const int* __restrict__ req_state_slot,
    unsigned char* state, long slot_stride, long tail_off, T* __restrict__ out, int width, int tile,
    int col_run) {
    cb_pdl_trigger();
    cb_pdl_wait();
    extern __shared__ float factor[];              // [tile + 2 (taps - 1)] factors, then the shares
    const int taps = TAPS > 0 ? TAPS : taps_;
    const int keep = taps - 1;
    const int req = blockIdx.y;
    const int row0 = req_row_start[req], n = req_row_start[req + 1] - row0;
    const int a = blockIdx.x * tile;
    if (a >= n) return;
    const int b = min(n, a + tile);                // tokens a .. b - 1 of the portion
    const bool first = blockIdx.x == 0;
    const int lo = max(0, a - keep);               // rows lo .. b - 1 are needed for the tile
    const int t0 = first ? max(b, n - keep) : n;   // and, for the new state, rows t0 .. n - 1
    const int n_here = b - lo, n_rows = n_here + (n - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    float* shares = factor + tile + 2 * keep;
    for (int u = warp; u < n_rows * SHARES; u += n_warps) {
        const int i = u / SHARES, s = u - i * SHARES;
        const int row = i < n_here ? lo + i : t0 + (i - n_here);
        const float* src = x + (size_t)(row0 + row) * width;
        float ss = 0.f;
        for (int c = (s * 32 + lane) * V; c < width; c += SHARES * 32 * V) {
            Vec<V> v;
            v.load(src + c);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(v.v[e], v.v[e], ss);
        }
        ss = cb_warp_sum(ss);
        if (lane == 0) shares[u] = ss;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n_rows; i += blockDim.x) {
        float total = 0.f;
#pragma unroll
        for (int s = 0; s < SHARES; ++s) total += shares[i * SHARES + s];
        factor[i] = 1.0f / sqrtf(total / (float)width + eps);
    }
    __syncthreads();
    float* tail = reinterpret_cast<float*>(state + (size_t)req_state_slot[req] * slot_stride + tail_off);
    const int c_end = min(width, (int)(blockIdx.z + 1) * col_run);
    for (int c = blockIdx.z * col_run + threadIdx.x * V; c < c_end; c += blockDim.x * V) {
        Vec<V> g;
        g.load(gain + c);
        // h of row `row` (negative: from the state), whose factor lies at place `at`
        auto h_of = [&](int row, int at) {
            Vec<V> h;
            if (row < 0) {
                h.load(tail + (size_t)(keep + row) * width + c);
            } else {
                h.load(x + (size_t)(row0 + row) * width + c);
                const float r = factor[at];
#pragma unroll
                for (int e = 0; e < V; ++e) h.v[e] = h.v[e] * r * g.v[e];
            }
            return h;
        };
        if constexpr (TAPS > 0) {
            Vec<V> past[TAPS], wt[TAPS];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) wt[j].load(w + (size_t)j * width + c);
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) past[j] = h_of(a - (TAPS - 1) + j, a - (TAPS - 1) + j - lo);
            for (int t = a; t < b; ++t) {
                past[TAPS - 1] = h_of(t, t - lo);
                Vec<V> acc;
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    float s = 0.f;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) s = fmaf(wt[j].v[e], past[j].v[e], s);
                    acc.v[e] = past[TAPS - 1].v[e] + s;
                }
                acc.put(out + (size_t)(row0 + t) * width + c);
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) past[j] = past[j + 1];
            }
        } else {
            for (int t = a; t < b; ++t) {
                Vec<V> acc;
#pragma unroll
                for (int e = 0; e < V; ++e) acc.v[e] = 0.f;
                for (int j = 0; j < taps; ++j) {
                    const int row = t - keep + j;
                    const Vec<V> h = h_of(row, row - lo);
                    Vec<V> wt;
                    wt.load(w + (size_t)j * width + c);
#pragma unroll
                    for (int e = 0; e < V; ++e) acc.v[e] = fmaf(wt.v[e], h.v[e], acc.v[e]);
                }
                const Vec<V> h = h_of(t, t - lo);
#pragma unroll
                for (int e = 0; e < V; ++e) acc.v[e] = h.v[e] + acc.v[e];
                acc.put(out + (size_t)(row0 + t) * width + c);
            }
        }
        if (first) {
            // ascending: what is read lies ahead of what is written
            for (int i = 0; i < keep; ++i) {
                const int row = n - keep + i;
                const Vec<V> h = h_of(row, row >= t0 ? n_here + row - t0 : row - lo);
                h.store(tail + (size_t)i * width + c);
            }
        }
    }
}

// V4: groups of four columns per thread, columns (g * blockDim + thread) * 4; blockDim * 4 * V4 >= width.
template <typename T, int V4, int TAPS>
__global__ void __launch_bounds__(512) norm_conv_once_kernel(
    const float* __restrict__ x, const float* __restrict__ gain, float eps, const float* __restrict__ w,
    const int* __restrict__ req_row_start, const int* __restrict__ req_state_slot, unsigned char* state,
    long slot_stride, long tail_off, T* __restrict__ out, int width) {
    cb_pdl_trigger();
    cb_pdl_wait();
    constexpr int KEEP = TAPS - 1, TILE = 8, ROWS = TILE + KEEP;
    __shared__ float shares[ROWS][16], factor[ROWS];
    const int req = blockIdx.y;
    const int row0 = req_row_start[req], n = req_row_start[req + 1] - row0;
    const int a = blockIdx.x * TILE;
    if (a >= n) return;
    const int b = min(n, a + TILE);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    float* tail = reinterpret_cast<float*>(state + (size_t)req_state_slot[req] * slot_stride + tail_off);
    int col[V4];
    bool in[V4];
#pragma unroll
    for (int g = 0; g < V4; ++g) {
        col[g] = (g * (int)blockDim.x + (int)threadIdx.x) * 4;
        in[g] = col[g] < width;
    }
    // place i holds the portion's token first_row + i
    Vec<4> v[ROWS][V4];
    auto load_rows = [&](int first_row, int end) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i)
#pragma unroll
            for (int g = 0; g < V4; ++g) {
                const int row = first_row + i;
                if (in[g] && row >= 0 && row < end) v[i][g].load(x + (size_t)(row0 + row) * width + col[g]);
                else v[i][g].v[0] = v[i][g].v[1] = v[i][g].v[2] = v[i][g].v[3] = 0.f;
            }
    };
    // the factors of `rows` places, then h in place of x (rows before the portion: from the state)
    Vec<4> gn[V4];
#pragma unroll
    for (int g = 0; g < V4; ++g)
        if (in[g]) gn[g].load(gain + col[g]);
    auto to_h = [&](int first_row, int end) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            if (first_row + i < 0 || first_row + i >= end) continue;       // the same for the whole block
            float ss = 0.f;
#pragma unroll
            for (int g = 0; g < V4; ++g)
#pragma unroll
                for (int e = 0; e < 4; ++e) ss = fmaf(v[i][g].v[e], v[i][g].v[e], ss);
            ss = cb_warp_sum(ss);
            if (lane == 0) shares[i][warp] = ss;
        }
        __syncthreads();
        if (threadIdx.x < ROWS && first_row + (int)threadIdx.x >= 0 && first_row + (int)threadIdx.x < end) {
            float total = 0.f;
            for (int s = 0; s < n_warps; ++s) total += shares[threadIdx.x][s];
            factor[threadIdx.x] = 1.0f / sqrtf(total / (float)width + eps);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int row = first_row + i;
            if (row >= end) continue;
#pragma unroll
            for (int g = 0; g < V4; ++g) {
                if (!in[g]) continue;
                if (row < 0) {
                    v[i][g].load(tail + (size_t)(KEEP + row) * width + col[g]);
                } else {
                    const float r = factor[i];
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[i][g].v[e] = v[i][g].v[e] * r * gn[g].v[e];
                }
            }
        }
    };
    load_rows(a - KEEP, b);
    to_h(a - KEEP, b);
    const bool first = blockIdx.x == 0;
#pragma unroll
    for (int g = 0; g < V4; ++g) {
        if (!in[g]) continue;
        Vec<4> wt[TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wt[j].load(w + (size_t)j * width + col[g]);
#pragma unroll
        for (int t = 0; t < TILE; ++t) {
            if (a + t >= b) continue;
            Vec<4> acc;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float s = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) s = fmaf(wt[j].v[e], v[t + j][g].v[e], s);
                acc.v[e] = v[t + KEEP][g].v[e] + s;
            }
            acc.put(out + (size_t)(row0 + a + t) * width + col[g]);
        }
        if (first && n <= TILE) {
            // tokens n - KEEP .. n - 1 lie at places n .. n + KEEP - 1 (all state reads are done)
#pragma unroll
            for (int i = 0; i < ROWS; ++i)
                if (i >= n && i < n + KEEP) v[i][g].store(tail + (size_t)(i - n) * width + col[g]);
        }
    }
    if (first && n > TILE) {
        // the portion's last rows: this block alone has read what they replace
        load_rows(n - KEEP, n);
        __syncthreads();
        to_h(n - KEEP, n);
#pragma unroll
        for (int g = 0; g < V4; ++g)
#pragma unroll
            for (int i = 0; i < KEEP; ++i)
                if (in[g]) v[i][g].store(tail + (size_t)i * width + col[g]);
    }
}

}  // namespace

// x: fp32 [rows][width]; gain: fp32 [width]; w: fp32 [taps][width], the last row meets the
// current token; out: T [rows][width].  max_new: the most tokens that a request brings.
CB_EXPORT int cb_norm_conv(const float* x, const float* gain, float eps, const float* w, int taps,
                           const int* req_row_start, const int* req_state_slot, void* state,
                           long slot_stride, long tail_off, void* out, int dtype, int n_requests,
                           int max_new, int width, void* stream) {
    if (n_requests <= 0 || max_new <= 0) return 0;
    if (taps < 1 || taps > 64 || n_requests > 65535) return CB_ERR_UNSUPPORTED;
    const int keep = taps - 1;
    const int tile = keep > 8 ? keep : 8;          // a later tile's rows then all lie in the portion
    const bool vec = (width & 3) == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)out & 15) == 0 &&
                     ((uintptr_t)gain & 15) == 0 && ((uintptr_t)w & 15) == 0 &&
                     (((uintptr_t)state + tail_off) & 15) == 0 && (slot_stride & 15) == 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (vec && width <= 4096 && taps >= 2 && taps <= 5) {
        const int v4 = width > 2048 ? 2 : 1;
        const int once_threads = (width / 4 / v4 + (width / 4 % v4 ? 1 : 0) + 31) / 32 * 32;
        const dim3 once_grid((max_new + 7) / 8, n_requests);
#define CB_NC1(TT, GG, KK)                                                                              \
        cb_launch(norm_conv_once_kernel<TT, GG, KK>, once_grid, dim3(once_threads), 0, s, x, gain, eps, w, \
                  req_row_start, req_state_slot, (unsigned char*)state, slot_stride, tail_off, (TT*)out, width)
#define CB_NC1_TAPS(TT, GG)                                                                             \
        do {                                                                                            \
            if (taps == 2) CB_NC1(TT, GG, 2);                                                           \
            else if (taps == 3) CB_NC1(TT, GG, 3);                                                      \
            else if (taps == 4) CB_NC1(TT, GG, 4);                                                      \
            else CB_NC1(TT, GG, 5);                                                                     \
        } while (0)
        if (dtype == CB_F32) { if (v4 == 1) CB_NC1_TAPS(float, 1); else CB_NC1_TAPS(float, 2); }
        else { if (v4 == 1) CB_NC1_TAPS(__nv_bfloat16, 1); else CB_NC1_TAPS(__nv_bfloat16, 2); }
#undef CB_NC1_TAPS
#undef CB_NC1
        return cb_last_error();
    }
    const int V = vec ? 4 : 1;
    // few tokens: more blocks to a row (each sums the row for itself)
    const bool few = max_new <= 4;
    const int threads = few ? 128 : 256;
    const int col_run = threads * V;
    const dim3 grid((max_new + tile - 1) / tile, n_requests, (width + col_run - 1) / col_run);
    if (grid.z > 65535) return CB_ERR_UNSUPPORTED;
    const size_t smem = (size_t)(tile + 2 * keep) * (1 + SHARES) * sizeof(float);
#define CB_NC(TT, VV, KK)                                                                              \
    cb_launch(norm_conv_kernel<TT, VV, KK>, grid, dim3(threads), smem, s, x, gain, eps, w, taps,       \
              req_row_start, req_state_slot, (unsigned char*)state, slot_stride, tail_off, (TT*)out,   \
              width, tile, col_run)
#define CB_NC_TAPS(TT, VV)                                                                             \
    do {                                                                                               \
        if (taps == 2) CB_NC(TT, VV, 2);                                                               \
        else if (taps == 3) CB_NC(TT, VV, 3);                                                          \
        else if (taps == 4) CB_NC(TT, VV, 4);                                                          \
        else if (taps == 5) CB_NC(TT, VV, 5);                                                          \
        else CB_NC(TT, VV, 0);                                                                         \
    } while (0)
    if (dtype == CB_F32) { if (vec) CB_NC_TAPS(float, 4); else CB_NC_TAPS(float, 1); }
    else { if (vec) CB_NC_TAPS(__nv_bfloat16, 4); else CB_NC_TAPS(__nv_bfloat16, 1); }
#undef CB_NC_TAPS
#undef CB_NC
    return cb_last_error();
}
