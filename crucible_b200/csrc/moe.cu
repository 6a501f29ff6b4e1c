// Mixture of experts: every token goes through `top` of `E` small gated feed-forwards,
//   y[t] = sum_j weight[t][j] * Wd[e_j] (silu(Wg[e_j] h[t]) * (Wu[e_j] h[t])),
// e_j the experts with the largest router logits of the token (the lower index on equal
// logits) and weight the softmax over those `top` logits alone; or, with sigmoid scores, the experts
// with the largest sigmoid(logit) + correction, weighted by their sigmoid(logit) as it is.
//
// Everything is decided on the device, so a step's launches depend on its shape only:
//   route    one warp per token: the top logits, their softmax, and each (token, choice)
//            pair's place among its expert's pairs (a counter per expert); the experts may form
//            equal groups of neighbours of which only the best few take part (a group's score is
//            its best score or the sum of its two best), and slices of a shared expert may ride
//            along as experts that every token chooses, weighted by the sigmoid of one logit of the
//            token or by one
//   plan     one block: where each expert's pairs start in the sorted order, the list of
//            row tiles (an expert, a start, a count), and the sorted order itself
//   tiles    gate/up with the gated pair (SiLU, or the capped form), then down times the pair's weight: a block owns a tile of
//            rows of one expert and a tile of columns; rows beyond the tile's count and
//            tiles beyond the plan's count do nothing.  fp32 sums over ascending k, so a
//            pair's result does not depend on which other pairs share its tile.
//   combine  residual[t] += the token's pairs in the order of its choices (or, for the tensor
//            cores' grouped products, the token's rows of the sorted order times their weights),
//            and a shared expert's row times the token's gate (or as it is) if it was run apart.
#define CB_PDL_BIT 13      // this file's bit in CRUCIBLE_PDL
#include "common.cuh"

namespace {

constexpr int TM = 32, TN = 64, TK = 32, THREADS = 128;
constexpr int MAX_PER_LANE = 8;       // experts <= 256, of which a token takes at most 32

// The gated pair of an expert.  limit <= 0: silu(g) * u.  Else the capped pair:
// g' = min(g, limit), u' = clamp(u, -limit, limit): g' * sigmoid(alpha * g') * (u' + offset).
struct GateRule { float limit, alpha, offset; };
__device__ __forceinline__ float gated_f(float g, float u, const GateRule& p) {
    if (p.limit <= 0.f) return g / (1.0f + expf(-g)) * u;
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit);
    return g / (1.0f + expf(-p.alpha * g)) * (u + p.offset);
}

constexpr int ROUTE_WARPS = 8;        // of a routing block ...
constexpr int ROUTE_TOKENS = 4;       // ... each of which takes up to this many tokens
constexpr int MAX_TOTAL = 32 * MAX_PER_LANE + 32;      // routed experts and a shared expert's slices

// How a token scores its experts.  sigmoid 0: by their logits, weighted by the softmax over the chosen
// ones; 1: by sigmoid(logit) + correction (null: nothing), weighted by sigmoid(logit).  best_two: a
// group's score is the sum of its two best scores instead of its best one.
struct ScoreRule { int sigmoid, best_two; const float* correction; };

// A pair's place among its expert's pairs: a counter per expert in shared memory, then one addition
// per block and expert to the global counter.
__global__ void __launch_bounds__(32 * ROUTE_WARPS) moe_route_kernel(
    const float* __restrict__ logits, const float* __restrict__ bias, int n_tokens, int stride, int E, int top,
    int* __restrict__ idx, float* __restrict__ weight, int* __restrict__ place, int* __restrict__ count,
    int groups, int keep, int n_shared, int gate_col, float scale, float* __restrict__ gate_out, int per_warp,
    ScoreRule rule) {
    cb_pdl_trigger();
    cb_pdl_wait();
    __shared__ float all[ROUTE_WARPS][32 * MAX_PER_LANE], best_of[ROUTE_WARPS][32 * MAX_PER_LANE];
    __shared__ int block_count[32 * MAX_PER_LANE], block_base[32 * MAX_PER_LANE];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int e = threadIdx.x; e < E; e += blockDim.x) block_count[e] = 0;
    __syncthreads();
    int chosen[ROUTE_TOKENS], in_block[ROUTE_TOKENS];
    const int t0 = (blockIdx.x * ROUTE_WARPS + warp) * per_warp;
#pragma unroll
    for (int k = 0; k < ROUTE_TOKENS; ++k) {
        const int t = t0 + k;
        chosen[k] = -1;
        if (k >= per_warp || t >= n_tokens) continue;
        float v[MAX_PER_LANE];
#pragma unroll
        for (int i = 0; i < MAX_PER_LANE; ++i) {
            const int e = lane + 32 * i;
            v[i] = e < E ? logits[(size_t)t * stride + e] + (bias != nullptr ? bias[e] : 0.f) : -INFINITY;
            if (rule.sigmoid && e < E)
                v[i] = 1.0f / (1.0f + expf(-v[i])) + (rule.correction != nullptr ? rule.correction[e] : 0.f);
        }
        if (keep < groups) {
            // only the experts of the `keep` groups with the largest score (the lower group on equal
            // ones) stay
            const int size = E / groups;
            __syncwarp();
#pragma unroll
            for (int i = 0; i < MAX_PER_LANE; ++i)
                if (lane + 32 * i < E) all[warp][lane + 32 * i] = v[i];
            __syncwarp();
            for (int g = lane; g < groups; g += 32) {
                float m = -INFINITY, second = -INFINITY;
                for (int e = g * size; e < (g + 1) * size; ++e) {
                    const float s = all[warp][e];
                    second = fmaxf(second, fminf(m, s));
                    m = fmaxf(m, s);
                }
                best_of[warp][g] = rule.best_two && size > 1 ? m + second : m;
            }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < MAX_PER_LANE; ++i) {
                const int e = lane + 32 * i;
                if (e >= E) continue;
                const int mine_g = e / size;
                const float m = best_of[warp][mine_g];
                int ahead = 0;
                for (int g = 0; g < groups; ++g)
                    ahead += best_of[warp][g] > m || (best_of[warp][g] == m && g < mine_g);
                if (ahead >= keep) v[i] = -INFINITY;
            }
        }
        float first = 0.f, total = 0.f, mine = 0.f;
        int mine_e = 0;
        for (int j = 0; j < top; ++j) {
            float best = -INFINITY;
            int best_e = 0x7fffffff;
#pragma unroll
            for (int i = 0; i < MAX_PER_LANE; ++i) {
                const int e = lane + 32 * i;
                if (e < E && (v[i] > best || (v[i] == best && e < best_e))) { best = v[i]; best_e = e; }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ob = __shfl_xor_sync(0xffffffffu, best, o);
                const int oe = __shfl_xor_sync(0xffffffffu, best_e, o);
                if (ob > best || (ob == best && oe < best_e)) { best = ob; best_e = oe; }
            }
            if (best_e == 0x7fffffff) best_e = j < E ? j : 0;      // nothing comparable left (NaN logits)
#pragma unroll
            for (int i = 0; i < MAX_PER_LANE; ++i)
                if (lane + 32 * i == best_e) v[i] = -INFINITY;
            if (j == 0) first = best;
            const float p = expf(best - first);
            total += p;
            if (lane == j) { mine = p; mine_e = best_e; }
        }
        const size_t at = (size_t)t * (top + n_shared);
        if (lane < top) {
            idx[at + lane] = mine_e;
            weight[at + lane] = (rule.sigmoid
                ? 1.0f / (1.0f + expf(-(logits[(size_t)t * stride + mine_e] + (bias != nullptr ? bias[mine_e] : 0.f))))
                : mine / total) * scale;
            chosen[k] = mine_e;
            in_block[k] = atomicAdd(&block_count[mine_e], 1);
        }
        if (gate_col >= 0 || n_shared > 0) {
            const float gate = gate_col >= 0 ? scale / (1.0f + expf(-logits[(size_t)t * stride + gate_col])) : scale;
            // the shared expert's slices: every token's, so its place among their pairs is its own number
            for (int s = lane; s < n_shared; s += 32) {
                idx[at + top + s] = E + s;
                weight[at + top + s] = gate;
                place[at + top + s] = t;
                if (t == 0) count[E + s] = n_tokens;
            }
            if (gate_out != nullptr && lane == 0) gate_out[t] = gate;
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        const int n = block_count[e];
        block_base[e] = n > 0 ? atomicAdd(&count[e], n) : 0;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < ROUTE_TOKENS; ++k)
        if (chosen[k] >= 0)
            place[(size_t)(t0 + k) * (top + n_shared) + lane] = block_base[chosen[k]] + in_block[k];
}

// (tile_rows_: rows of a tile: TM for the kernels of this file, 128 for the tensor cores' grouped product)
// plan: [0] number of tiles, [1 .. E+1] each expert's start in the sorted order, then
// max_tiles each of (expert, start, rows).
__global__ void __launch_bounds__(1024) moe_plan_kernel(int* __restrict__ count, int E, int n_pairs,
                                                        const int* __restrict__ idx,
                                                        const int* __restrict__ place, int* __restrict__ plan,
                                                        int max_tiles, int* __restrict__ sorted_pair,
                                                        int tile_rows_) {
    cb_pdl_trigger();
    cb_pdl_wait();
    __shared__ int start[MAX_TOTAL + 1], first_tile[MAX_TOTAL + 1];
    int* tile_expert = plan + 2 + E;
    int* tile_start = tile_expert + max_tiles;
    int* tile_rows = tile_start + max_tiles;
    if (threadIdx.x < 32) {
        // running sums of the experts' pairs and tiles, 32 experts at a time
        const int lane = threadIdx.x;
        int pairs = 0, tiles = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int n = e0 + lane < E ? count[e0 + lane] : 0;
            int a = n, b = (n + tile_rows_ - 1) / tile_rows_;
            const int my_tiles = b;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int ua = __shfl_up_sync(0xffffffffu, a, o), ub = __shfl_up_sync(0xffffffffu, b, o);
                if (lane >= o) { a += ua; b += ub; }
            }
            if (e0 + lane < E) {
                start[e0 + lane] = pairs + a - n;
                first_tile[e0 + lane] = tiles + b - my_tiles;
            }
            pairs += __shfl_sync(0xffffffffu, a, 31);
            tiles += __shfl_sync(0xffffffffu, b, 31);
        }
        if (lane == 0) {
            start[E] = pairs;
            first_tile[E] = tiles;
            plan[0] = min(tiles, max_tiles);
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e <= E; e += blockDim.x) plan[1 + e] = start[e];
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        const int n = start[e + 1] - start[e];
        for (int r = 0, tile = first_tile[e]; r < n && tile < max_tiles; r += tile_rows_, ++tile) {
            tile_expert[tile] = e;
            tile_start[tile] = start[e] + r;
            tile_rows[tile] = min(tile_rows_, n - r);
        }
        count[e] = 0;                              // ready for the next step
    }
    for (int p = threadIdx.x; p < n_pairs; p += blockDim.x) sorted_pair[start[idx[p]] + place[p]] = p;
}

// GATED: rows are h[token of the pair], W = [gate rows; up rows] of the tile's expert,
//        out[sorted place][n] = silu(gate) * up in T.
// else:  rows are act[sorted place], W = down of the expert, out[pair][n] = weight[pair] * sum, fp32.
template <typename T, bool GATED>
__global__ void __launch_bounds__(THREADS) moe_tile_kernel(
    const T* __restrict__ a, int a_stride, const T* __restrict__ w, long expert_stride, int N, int K,
    const int* __restrict__ plan, int E, int max_tiles, const int* __restrict__ sorted_pair, int top,
    const float* __restrict__ weight, void* __restrict__ out_, int out_stride, GateRule rule) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const int tile = blockIdx.x;
    if (tile >= plan[0]) return;
    const int* tile_expert = plan + 2 + E;
    const int e = tile_expert[tile], start = tile_expert[max_tiles + tile], rows = tile_expert[2 * max_tiles + tile];
    const int n0 = blockIdx.y * TN;
    __shared__ float sa[TM][TK + 1];
    __shared__ float sw[GATED ? 2 : 1][TN][TK + 1];
    __shared__ int src_row[TM];
    if (threadIdx.x < TM) {
        const int s = start + min((int)threadIdx.x, rows - 1);
        src_row[threadIdx.x] = GATED ? sorted_pair[s] / top : s;
    }
    __syncthreads();
    const T* we = w + (size_t)e * expert_stride;
    const int tr = (threadIdx.x >> 4) * 4, tc = (threadIdx.x & 15) * 4;
    float acc[GATED ? 2 : 1][4][4] = {};
    for (int k0 = 0; k0 < K; k0 += TK) {
        for (int i = threadIdx.x; i < TM * TK; i += THREADS) {
            const int r = i / TK, k = i - r * TK;
            sa[r][k] = k0 + k < K ? cb_to_float(a[(size_t)src_row[r] * a_stride + k0 + k]) : 0.f;
        }
        for (int i = threadIdx.x; i < TN * TK; i += THREADS) {
            const int c = i / TK, k = i - c * TK;
            const bool in = n0 + c < N && k0 + k < K;
            sw[0][c][k] = in ? cb_to_float(we[(size_t)(n0 + c) * K + k0 + k]) : 0.f;
            if (GATED) sw[1][c][k] = in ? cb_to_float(we[(size_t)(N + n0 + c) * K + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < TK; ++k) {
            float av[4], wv[GATED ? 2 : 1][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                av[i] = sa[tr + i][k];
                wv[0][i] = sw[0][tc + i][k];
                if (GATED) wv[1][i] = sw[1][tc + i][k];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[0][i][j] = fmaf(av[i], wv[0][j], acc[0][i][j]);
                    if (GATED) acc[1][i][j] = fmaf(av[i], wv[1][j], acc[1][i][j]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        if (tr + i >= rows) continue;
        const int s = start + tr + i;
        if (GATED) {
            T* dst = reinterpret_cast<T*>(out_) + (size_t)s * out_stride;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tc + j < N) dst[n0 + tc + j] = cb_from_float<T>(gated_f(acc[0][i][j], acc[GATED ? 1 : 0][i][j], rule));
        } else {
            const int p = sorted_pair[s];
            const float wt = weight[p];
            float* dst = reinterpret_cast<float*>(out_) + (size_t)p * out_stride;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tc + j < N) dst[n0 + tc + j] = wt * acc[0][i][j];
        }
    }
}

// The same two products for steps of few rows (decoded tokens): the experts' weights are what
// moves, so each weight row is read once, by one warp whose lanes share K in 16-byte pieces, and
// meets every row of its tile (ROWS at a time).  A block owns a tile and a run of output features.
template <typename T> struct Vec8;
template <> struct Vec8<__nv_bfloat16> {
    typedef uint4 Raw;
    static __device__ __forceinline__ Raw fetch(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
    static __device__ __forceinline__ void put(__nv_bfloat16* p, const Raw& raw) { *reinterpret_cast<uint4*>(p) = raw; }
    static __device__ __forceinline__ void unpack(const Raw& raw, float* v) {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
    }
};
template <> struct Vec8<float> {
    struct Raw { float4 a, b; };
    static __device__ __forceinline__ Raw fetch(const float* p) {
        Raw r;
        r.a = *reinterpret_cast<const float4*>(p);
        r.b = *reinterpret_cast<const float4*>(p + 4);
        return r;
    }
    static __device__ __forceinline__ void put(float* p, const Raw& r) {
        *reinterpret_cast<float4*>(p) = r.a;
        *reinterpret_cast<float4*>(p + 4) = r.b;
    }
    static __device__ __forceinline__ void unpack(const Raw& r, float* v) {
        v[0] = r.a.x; v[1] = r.a.y; v[2] = r.a.z; v[3] = r.a.w; v[4] = r.b.x; v[5] = r.b.y; v[6] = r.b.z; v[7] = r.b.w;
    }
};

extern __shared__ __align__(16) unsigned char moe_rows_staged[];

template <typename T, bool GATED, int ROWS>
__global__ void __launch_bounds__(256, 3) moe_rows_small_kernel(
    const T* __restrict__ a, int a_stride, const T* __restrict__ w, long expert_stride, int N, int K,
    const int* __restrict__ plan, int E, int max_tiles, const int* __restrict__ sorted_pair, int top,
    const float* __restrict__ weight, void* __restrict__ out_, int out_stride, int per_block, GateRule rule) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const int tile = blockIdx.x;
    if (tile >= plan[0]) return;
    const int* tile_expert = plan + 2 + E;
    const int e = tile_expert[tile], start = tile_expert[max_tiles + tile], rows = tile_expert[2 * max_tiles + tile];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const T* we = w + (size_t)e * expert_stride;
    const int n_end = min(N, (int)(blockIdx.y + 1) * per_block);
    T* staged = reinterpret_cast<T*>(moe_rows_staged);       // ROWS rows of K: this pass's rows
    for (int r0 = 0; r0 < rows; r0 += ROWS) {
        __syncthreads();
        for (int i = threadIdx.x * 8; i < ROWS * K; i += blockDim.x * 8) {
            const int r = i / K, k = i - r * K;
            const int s = start + min(r0 + r, rows - 1);
            Vec8<T>::put(staged + i, Vec8<T>::fetch(a + (size_t)(GATED ? sorted_pair[s] / top : s) * a_stride + k));
        }
        __syncthreads();
        for (int n = blockIdx.y * per_block + warp; n < n_end; n += n_warps) {
            const T* w0 = we + (size_t)n * K;
            const T* w1 = we + (size_t)(N + n) * K;          // the up row (GATED)
            float acc0[ROWS], acc1[ROWS];
#pragma unroll
            for (int r = 0; r < ROWS; ++r) acc0[r] = acc1[r] = 0.f;
            // four pieces of a weight row are asked for before the first is used: a warp then has
            // 2 to 4 KB on its way, a block of eight warps what an SM needs to stream
            constexpr int AHEAD = 4;
            for (int k = lane * 8; k < K; k += 256 * AHEAD) {
                typename Vec8<T>::Raw raw0[AHEAD], raw1[AHEAD];
#pragma unroll
                for (int u = 0; u < AHEAD; ++u) {
                    const int kk = k + u * 256;
                    if (kk < K) {
                        raw0[u] = Vec8<T>::fetch(w0 + kk);
                        if (GATED) raw1[u] = Vec8<T>::fetch(w1 + kk);
                    }
                }
#pragma unroll
                for (int u = 0; u < AHEAD; ++u) {
                    const int kk = k + u * 256;
                    if (kk >= K) break;
                    float wv0[8], wv1[8], av[8];
                    Vec8<T>::unpack(raw0[u], wv0);
                    if (GATED) Vec8<T>::unpack(raw1[u], wv1);
#pragma unroll
                    for (int r = 0; r < ROWS; ++r) {
                        if (r0 + r >= rows) break;
                        Vec8<T>::unpack(Vec8<T>::fetch(staged + r * K + kk), av);
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            acc0[r] = fmaf(av[i], wv0[i], acc0[r]);
                            if (GATED) acc1[r] = fmaf(av[i], wv1[i], acc1[r]);
                        }
                    }
                }
            }
#pragma unroll
            for (int r = 0; r < ROWS; ++r) {
                if (r0 + r >= rows) break;
                const float g = cb_warp_sum(acc0[r]);
                const float u = GATED ? cb_warp_sum(acc1[r]) : 0.f;
                if (lane == 0) {
                    const int s = start + r0 + r;
                    if (GATED) {
                        reinterpret_cast<T*>(out_)[(size_t)s * out_stride + n] = cb_from_float<T>(gated_f(g, u, rule));
                    } else {
                        const int p = sorted_pair[s];
                        reinterpret_cast<float*>(out_)[(size_t)p * out_stride + n] = weight[p] * g;
                    }
                }
            }
        }
    }
}

// rows: by pair, weighted already (offsets null), or in the sorted order, where a pair's row lies at
// its expert's start + its place and takes its weight here.  shared (may be null): rows by token,
// times gate[token].  V: vector width.
template <int V>
__global__ void moe_combine_kernel(const float* __restrict__ rows, int top, float* __restrict__ residual,
                                   int width, const int* __restrict__ offsets, const int* __restrict__ idx,
                                   const int* __restrict__ place, const float* __restrict__ weight,
                                   const float* __restrict__ shared, const float* __restrict__ gate) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const int t = blockIdx.x;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float sum[V];
#pragma unroll
        for (int e = 0; e < V; ++e) sum[e] = 0.f;
        auto add = [&](const float* src, float w) {
            if constexpr (V == 4) {
                const float4 a = *reinterpret_cast<const float4*>(src);
                sum[0] = fmaf(w, a.x, sum[0]); sum[1] = fmaf(w, a.y, sum[1]);
                sum[2] = fmaf(w, a.z, sum[2]); sum[3] = fmaf(w, a.w, sum[3]);
            } else {
                sum[0] = fmaf(w, src[0], sum[0]);
            }
        };
        for (int j = 0; j < top; ++j) {
            const size_t p = (size_t)t * top + j;
            if (offsets == nullptr) add(rows + p * width + i, 1.0f);
            else add(rows + (size_t)(offsets[idx[p]] + place[p]) * width + i, weight[p]);
        }
        if (shared != nullptr) add(shared + (size_t)t * width + i, gate != nullptr ? gate[t] : 1.0f);
        float* dst = residual + (size_t)t * width + i;
#pragma unroll
        for (int e = 0; e < V; ++e) dst[e] += sum[e];
    }
}

// rows of `h` gathered into the sorted order (for products that want an expert's rows side by side)
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ h, int h_stride, const int* __restrict__ sorted_pair,
                                  int top, T* __restrict__ out, int width) {
    cb_pdl_trigger();
    cb_pdl_wait();
    const T* src = h + (size_t)(sorted_pair[blockIdx.x] / top) * h_stride;
    T* dst = out + (size_t)blockIdx.x * width;
    constexpr int PER = 16 / sizeof(T);
    if (width % PER == 0 && h_stride % PER == 0 && (((uintptr_t)h | (uintptr_t)out) & 15) == 0) {
        for (int i = threadIdx.x * PER; i < width; i += blockDim.x * PER)
            *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<const uint4*>(src + i);
        return;
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = src[i];
}

}  // namespace

CB_EXPORT int cb_moe_tile_rows() { return TM; }

// logits: rows at `stride`, the first E of them the experts'.  groups, keep: equal groups of
// neighbouring experts of which `keep` take part (groups == keep: no restriction).  gate_col >= 0: the
// column of the shared expert's gate logit (-1: it has no gate); n_shared slices of it ride along as
// experts E .. E + n_shared - 1 of every token, and gate_out (may be null) receives scale * sigmoid of
// that logit.  scale: on every weight.  count and plan cover E + n_shared experts, a token has top +
// n_shared pairs.  sigmoid, best_two, correction: see ScoreRule.
CB_EXPORT int cb_moe_route(const float* logits, int stride, const float* bias, int n_tokens, int E, int top,
                           int* idx, float* weight,
                           int* place, int* count, int* plan, int max_tiles, int* sorted_pair,
                           int tile_rows, int groups, int keep, int n_shared, int gate_col, float scale,
                           float* gate_out, int sigmoid, int best_two, const float* correction, void* stream) {
    if (n_tokens <= 0) return 0;
    if (E > 32 * MAX_PER_LANE || top > E || top <= 0 || top > 32) return CB_ERR_UNSUPPORTED;
    if (groups <= 0 || E % groups || keep <= 0 || keep > groups || top > keep * (E / groups) || n_shared < 0 ||
        gate_col >= stride)
        return CB_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    if (E + n_shared > MAX_TOTAL) return CB_ERR_UNSUPPORTED;
    const int per_warp = n_tokens >= 16384 ? ROUTE_TOKENS : 1, per_block = ROUTE_WARPS * per_warp;
    cb_launch(moe_route_kernel, dim3((n_tokens + per_block - 1) / per_block), dim3(32 * ROUTE_WARPS), 0, s, logits,
              bias, n_tokens, stride, E, top, idx, weight, place, count, groups, keep, n_shared, gate_col, scale,
              gate_out, per_warp, ScoreRule{sigmoid, best_two, correction});
    cb_launch(moe_plan_kernel, dim3(1), dim3(n_tokens * (top + n_shared) > 256 ? 1024 : 256), 0, s, count, E + n_shared, n_tokens * (top + n_shared),
              (const int*)idx, (const int*)place, plan, max_tiles, sorted_pair, tile_rows > 0 ? tile_rows : TM);
    return cb_last_error();
}

// gated != 0: act[sorted place][N] from h rows; else pair_out[pair][N] from act rows.
CB_EXPORT int cb_moe_tiles(int gated, const void* a, int a_stride, const void* w, long expert_stride,
                           int dtype, int N, int K, const int* plan, int E, int max_tiles,
                           const int* sorted_pair, int top, const float* weight, void* out,
                           int out_stride, float limit, float alpha, float offset, void* stream) {
    if (max_tiles <= 0) return 0;
    const GateRule rule = {limit, alpha, offset};
    const dim3 grid(max_tiles, (N + TN - 1) / TN), block(THREADS);
    cudaStream_t s = (cudaStream_t)stream;
#define CB_MOE(TT, GG)                                                                             \
    cb_launch(moe_tile_kernel<TT, GG>, grid, block, 0, s, (const TT*)a, a_stride, (const TT*)w,    \
              expert_stride, N, K, plan, E, max_tiles, sorted_pair, top, weight, out, out_stride, rule)
    if (dtype == CB_F32) { if (gated) CB_MOE(float, true); else CB_MOE(float, false); }
    else { if (gated) CB_MOE(__nv_bfloat16, true); else CB_MOE(__nv_bfloat16, false); }
#undef CB_MOE
    return cb_last_error();
}

// The same as cb_moe_tiles for steps of few rows; K a multiple of 8 and 16-byte aligned rows.
CB_EXPORT int cb_moe_rows_small(int gated, const void* a, int a_stride, const void* w, long expert_stride,
                                int dtype, int N, int K, const int* plan, int E, int max_tiles,
                                const int* sorted_pair, int top, const float* weight, void* out,
                                int out_stride, float limit, float alpha, float offset, void* stream) {
    if (max_tiles <= 0) return 0;
    const GateRule rule = {limit, alpha, offset};
    if (K % 8 || a_stride % 8 || ((uintptr_t)a & 15) || ((uintptr_t)w & 15)) return CB_ERR_UNSUPPORTED;
    // enough blocks to keep the memory busy, but no more than find a place at once (three to an SM)
    int chunks = (3 * 148) / max_tiles;
    chunks = chunks < 1 ? 1 : chunks;
    int per_block = (N + chunks - 1) / chunks;
    per_block = per_block < 8 ? 8 : per_block;
    const dim3 grid(max_tiles, (N + per_block - 1) / per_block), block(256);
    const size_t smem = (size_t)4 * K * (dtype == CB_F32 ? 4 : 2);      // the staged rows
    if (smem > 64 * 1024) return CB_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
#define CB_MOE(TT, GG)                                                                                  \
    do {                                                                                                \
        if (smem > 48 * 1024) {                                                                         \
            static bool configured = false;                                                             \
            if (!configured) {                                                                          \
                cudaError_t err = cudaFuncSetAttribute(moe_rows_small_kernel<TT, GG, 4>,                \
                                                       cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024); \
                if (err != cudaSuccess) return (int)err;                                                \
                configured = true;                                                                      \
            }                                                                                           \
        }                                                                                               \
        cb_launch(moe_rows_small_kernel<TT, GG, 4>, grid, block, smem, s, (const TT*)a, a_stride,       \
                  (const TT*)w, expert_stride, N, K, plan, E, max_tiles, sorted_pair, top, weight, out, \
                  out_stride, per_block, rule);                                                         \
    } while (0)
    if (dtype == CB_F32) { if (gated) CB_MOE(float, true); else CB_MOE(float, false); }
    else { if (gated) CB_MOE(__nv_bfloat16, true); else CB_MOE(__nv_bfloat16, false); }
#undef CB_MOE
    return cb_last_error();
}

// plan null: rows [tokens * top][width] by pair, weighted; else rows in the sorted order of that plan.
// shared (or null): rows [tokens][width] that join with gate[token] (null: as they are).
CB_EXPORT int cb_moe_combine(const float* rows, int top, float* residual, int n_tokens, int width,
                             const int* plan, const int* idx, const int* place, const float* weight,
                             const float* shared, const float* gate, void* stream) {
    if (n_tokens <= 0) return 0;
    const int* offsets = plan != nullptr ? plan + 1 : nullptr;
    const bool vec = (width & 3) == 0 && ((uintptr_t)rows & 15) == 0 && ((uintptr_t)residual & 15) == 0 &&
                     ((uintptr_t)shared & 15) == 0;
    const dim3 block(width >= 1024 ? 256 : 128);
    cudaStream_t s = (cudaStream_t)stream;
    if (vec)
        cb_launch(moe_combine_kernel<4>, dim3(n_tokens), block, 0, s, rows, top, residual, width, offsets, idx, place,
                  weight, shared, gate);
    else
        cb_launch(moe_combine_kernel<1>, dim3(n_tokens), block, 0, s, rows, top, residual, width, offsets, idx, place,
                  weight, shared, gate);
    return cb_last_error();
}

CB_EXPORT int cb_moe_gather(const void* h, int h_stride, int dtype, const int* sorted_pair, int top,
                            void* out, int n_pairs, int width, void* stream) {
    if (n_pairs <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == CB_F32)
        cb_launch(moe_gather_kernel<float>, dim3(n_pairs), dim3(128), 0, s, (const float*)h, h_stride,
                  sorted_pair, top, (float*)out, width);
    else
        cb_launch(moe_gather_kernel<__nv_bfloat16>, dim3(n_pairs), dim3(128), 0, s, (const __nv_bfloat16*)h,
                  h_stride, sorted_pair, top, (__nv_bfloat16*)out, width);
    return cb_last_error();
}
