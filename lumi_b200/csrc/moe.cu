// Mixture of experts: every token uses the `top` experts with the largest router scores s = sigmoid(z); the score multiplies the
// expert's INPUT, the outputs are added.
//
//   many rows (tensor cores)   moe_route_kernel picks the experts and lays out the pairs (row, expert) sorted by expert with the row
//                              tiles of 128 that the grouped products walk over; moe_gather_kernel writes the experts' inputs in
//                              that order; moe_combine_kernel adds the results to the residual stream and leaves the next norm's
//                              input behind.
//   few rows, fp32             moe_few_up_kernel (choice, norm, gate and up rows of a pair) and moe_few_down_kernel stream the
//                              weights of the chosen experts.
//
// Places among the pairs of an expert are handed out by atomics: their order changes nothing but the place a row is computed at.
#include "rows.cuh"

namespace lumi {
namespace {

constexpr int kTile = 128;                                // rows per tile of the grouped products

struct Plan {
    int32_t *n_tiles, *ticket, *counts, *offsets, *pair_e, *pair_rank;
    float* pair_w;
    int4* tiles;
};
__host__ __device__ inline long plan_pairs_at(int E) { return 4 + 2L * E; }
__host__ __device__ inline long plan_tiles_at(int rows, int top, int E) { return (plan_pairs_at(E) + 3L * rows * top + 3) / 4 * 4; }
__host__ __device__ inline Plan plan_of(const MoeArgs& a) {
    Plan p;
    p.n_tiles = a.plan;
    p.ticket = a.plan + 1;
    p.counts = a.plan + 4;
    p.offsets = p.counts + a.E_max;
    p.pair_e = a.plan + plan_pairs_at(a.E_max);
    p.pair_rank = p.pair_e + (long)a.rows * a.top;
    p.pair_w = reinterpret_cast<float*>(p.pair_rank + (long)a.rows * a.top);
    p.tiles = reinterpret_cast<int4*>(a.plan + plan_tiles_at(a.rows, a.top, a.E_max));
    return p;
}

// One warp: the largest of z below (pz, pi) in the order by value and then by index (pi < 0: the largest of all).
__device__ __forceinline__ void next_largest(const float* z, int E, float pz, int pi, int lane, float& bz, int& bi) {
    bz = -INFINITY;
    bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
        const float v = z[e];
        if (pi >= 0 && !(v < pz || (v == pz && e > pi))) continue;
        if (v > bz || bi == 0x7fffffff) { bz = v; bi = e; }           // ascending e: the lowest index of equal values stays
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float oz = __shfl_xor_sync(0xffffffffu, bz, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (oi != 0x7fffffff && (bi == 0x7fffffff || oz > bz || (oz == bz && oi < bi))) { bz = oz; bi = oi; }
    }
    if (bi >= E) bi = E - 1;                              // (only if scores are not numbers)
}

__global__ void __launch_bounds__(256) moe_route_kernel(MoeArgs a) {
    __shared__ int last;
    __shared__ int sums[2][256];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
    const int row = blockIdx.x * 8 + warp;
    const Plan p = plan_of(a);
    pdl_release();
    pdl_sync();
    if (row < a.rows) {
        const float* z = a.logits + (size_t)row * a.ldl;
        float pz = 0.f;
        int pi = -1;
        for (int j = 0; j < a.top; ++j) {
            next_largest(z, a.E, pz, pi, lane, pz, pi);
            if (lane == 0) {
                const long pr = (long)row * a.top + j;
                p.pair_e[pr] = pi;
                p.pair_w[pr] = sigmoid_f(pz);
                p.pair_rank[pr] = atomicAdd(p.counts + pi, 1);
            }
        }
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        last = atomicAdd(p.ticket, 1) == (int)gridDim.x - 1;
        if (last) *p.ticket = 0;
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    // offsets and row tiles: 256 experts at a time
    int base = 0, tbase = 0;
    for (int e0 = 0; e0 < a.E; e0 += 256) {
        const int e = e0 + tid, c = e < a.E ? __ldcg(p.counts + e) : 0, nt = (c + kTile - 1) / kTile;
        sums[0][tid] = c;
        sums[1][tid] = nt;
        __syncthreads();
        for (int o = 1; o < 256; o <<= 1) {
            const int x = tid >= o ? sums[0][tid - o] : 0, y = tid >= o ? sums[1][tid - o] : 0;
            __syncthreads();
            sums[0][tid] += x;
            sums[1][tid] += y;
            __syncthreads();
        }
        if (e < a.E) {
            const int off = base + sums[0][tid] - c, t0 = tbase + sums[1][tid] - nt;
            p.offsets[e] = off;
            p.counts[e] = 0;                              // ready for the next launch
            for (int i = 0; i < nt; ++i) p.tiles[t0 + i] = make_int4(off + i * kTile, min(kTile, c - i * kTile), e, 0);
        }
        base += sums[0][255];
        tbase += sums[1][255];
        __syncthreads();
    }
    if (tid == 0) *p.n_tiles = tbase;
}

template <int NT>
__device__ __forceinline__ float block_total(float v, float* red) {
    v = warp_total(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < NT / 32; ++w) t += red[w];
    return t;
}
__device__ __forceinline__ void store_halves4(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t o, float4 y) {
    const __nv_bfloat162 h0 = __floats2bfloat162_rn(y.x, y.y), h1 = __floats2bfloat162_rn(y.z, y.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&h0); u.y = *reinterpret_cast<const uint32_t*>(&h1);
    *reinterpret_cast<uint2*>(hi + o) = u;
    if (lo != nullptr) {
        const float2 f0 = __bfloat1622float2(h0), f1 = __bfloat1622float2(h1);
        const __nv_bfloat162 l0 = __floats2bfloat162_rn(y.x - f0.x, y.y - f0.y), l1 = __floats2bfloat162_rn(y.z - f1.x, y.w - f1.y);
        u.x = *reinterpret_cast<const uint32_t*>(&l0); u.y = *reinterpret_cast<const uint32_t*>(&l1);
        *reinterpret_cast<uint2*>(lo + o) = u;
    }
}

// One CTA per row: w * norm(x) for each of its experts, at the pair's place.
__global__ void __launch_bounds__(128) moe_gather_kernel(MoeArgs a) {
    __shared__ float red[4];
    const int row = blockIdx.x, tid = threadIdx.x, n4 = a.ldx >> 2;
    const Plan p = plan_of(a);
    pdl_release();
    pdl_sync();
    const float4* x = reinterpret_cast<const float4*>(a.x + (size_t)row * a.ldx);
    float s = 0.f;
    for (int c = tid; c < n4; c += 128) { const float4 v = x[c]; s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s)))); }
    const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(block_total<128>(s, red), (float)a.D) + a.eps));
    for (int j = 0; j < a.top; ++j) {
        const long pr = (long)row * a.top + j;
        const size_t to = (size_t)(p.offsets[p.pair_e[pr]] + p.pair_rank[pr]) * a.ldx;
        const float w = p.pair_w[pr] * rs;
        for (int c = tid; c < n4; c += 128) {
            const float4 v = x[c], g = __ldg(reinterpret_cast<const float4*>(a.gamma) + c);
            store_halves4(a.gh, a.gl, to + 4 * (size_t)c, make_float4(v.x * w * g.x, v.y * w * g.y, v.z * w * g.z, v.w * w * g.w));
        }
    }
}

// One CTA per row: x += the results of its experts; the next norm's input.
__global__ void __launch_bounds__(128) moe_combine_kernel(MoeArgs a) {
    __shared__ float red[4];
    const int row = blockIdx.x, tid = threadIdx.x, n4 = a.ldx >> 2;
    const Plan p = plan_of(a);
    pdl_release();
    pdl_sync();
    float4* x = reinterpret_cast<float4*>(a.x + (size_t)row * a.ldx);
    float s = 0.f;
    for (int c = tid; c < n4; c += 128) {
        float4 v = x[c];
        for (int j = 0; j < a.top; ++j) {
            const long pr = (long)row * a.top + j;
            const float4 y = *(reinterpret_cast<const float4*>(a.y + (size_t)(p.offsets[p.pair_e[pr]] + p.pair_rank[pr]) * a.ldx) + c);
            v.x += y.x; v.y += y.y; v.z += y.z; v.w += y.w;
        }
        x[c] = v;
        s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
        if (a.gamma_next != nullptr) {
            const float4 g = __ldg(reinterpret_cast<const float4*>(a.gamma_next) + c);
            store_halves4(a.xh, a.xl, (size_t)row * a.ldx + 4 * (size_t)c, make_float4(v.x * g.x, v.y * g.y, v.z * g.z, v.w * g.w));
        }
    }
    if (a.gamma_next == nullptr) return;
    s = block_total<128>(s, red);
    if (tid == 0) a.ssq[(size_t)row * a.ssq_stride] = s;
}

// ---- few rows --------------------------------------------------------------------------------------------------
__device__ __forceinline__ void widen16(const uint4& v, const float*, float (&w)[4]) {
    w[0] = __uint_as_float(v.x); w[1] = __uint_as_float(v.y); w[2] = __uint_as_float(v.z); w[3] = __uint_as_float(v.w);
}
__device__ __forceinline__ void widen16(const uint4& v, const __nv_bfloat16*, float (&w)[8]) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { w[2 * i] = __uint_as_float(u[i] << 16); w[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u); }
}
template <typename WT>
__device__ __forceinline__ float dot_chunk(const uint4& w, const float* x, float acc) {
    constexpr int E = 16 / sizeof(WT);
    float f[E];
    widen16(w, (const WT*)nullptr, f);
#pragma unroll
    for (int q = 0; q < E / 4; ++q) {
        const float4 v = *reinterpret_cast<const float4*>(x + 4 * q);
        acc = fmaf(f[4 * q], v.x, fmaf(f[4 * q + 1], v.y, fmaf(f[4 * q + 2], v.z, fmaf(f[4 * q + 3], v.w, acc))));
    }
    return acc;
}

constexpr int kUpPerWarp = 2;                             // hidden elements per warp

template <typename WT>
__global__ void __launch_bounds__(256) moe_few_up_kernel(MoeArgs a) {
    extern __shared__ float xs[];                         // [ldx]
    __shared__ float red[8];
    __shared__ int se;
    __shared__ float sw;
    constexpr int E = 16 / sizeof(WT);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pair = blockIdx.x, row = pair / a.top, j = pair % a.top;
    const Plan p = plan_of(a);
    pdl_release();
    pdl_sync();
    if (warp == 0) {
        float pz = 0.f;
        int pi = -1;
        for (int i = 0; i <= j; ++i) next_largest(a.logits + (size_t)row * a.ldl, a.E, pz, pi, lane, pz, pi);
        if (lane == 0) {
            se = pi;
            sw = sigmoid_f(pz);
            if (blockIdx.y == 0) p.pair_e[pair] = pi;
        }
    }
    float s = 0.f;
    for (int c = tid; c < a.ldx; c += 256) { const float v = a.x[(size_t)row * a.ldx + c]; s = fmaf(v, v, s); xs[c] = v * a.gamma[c]; }
    const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(block_total<256>(s, red), (float)a.D) + a.eps));       // (synchronises)
    const int e = se, chunks = a.ldx / E;
    const float f = sw * rs;
    const WT* W = reinterpret_cast<const WT*>(a.w_up) + (size_t)e * 2 * a.ffp * a.ldx;
    const int n0 = (blockIdx.y * 8 + warp) * kUpPerWarp;
    float g[kUpPerWarp] = {}, u[kUpPerWarp] = {};
    for (int c = lane; c < chunks; c += 32) {
        uint4 wg[kUpPerWarp], wu[kUpPerWarp];
#pragma unroll
        for (int i = 0; i < kUpPerWarp; ++i) {
            const int n = min(n0 + i, a.ffp - 1);
            const WT* wr = W + (size_t)((n >> 4) * 32 + (n & 15)) * a.ldx;
            wg[i] = __ldg(reinterpret_cast<const uint4*>(wr) + c);
            wu[i] = __ldg(reinterpret_cast<const uint4*>(wr + (size_t)16 * a.ldx) + c);
        }
#pragma unroll
        for (int i = 0; i < kUpPerWarp; ++i) {
            g[i] = dot_chunk<WT>(wg[i], xs + c * E, g[i]);
            u[i] = dot_chunk<WT>(wu[i], xs + c * E, u[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < kUpPerWarp; ++i) {
        const float gv = warp_total(g[i]) * f, uv = warp_total(u[i]) * f;
        if (lane == 0 && n0 + i < a.ffp) a.h32[(size_t)pair * a.ffp + n0 + i] = (a.act == ACT_RELU_GATE ? fmaxf(gv, 0.f) : silu_f(gv)) * uv;
    }
}

template <typename WT>
__global__ void __launch_bounds__(256) moe_few_down_kernel(MoeArgs a) {
    constexpr int E = 16 / sizeof(WT);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row = blockIdx.x, n = blockIdx.y * 8 + warp, chunks = a.ffp / E;
    const Plan p = plan_of(a);
    pdl_release();
    pdl_sync();
    if (n >= a.D) return;
    float y = a.x[(size_t)row * a.ldx + n];
    for (int j = 0; j < a.top; ++j) {
        const long pair = (long)row * a.top + j;
        const uint4* W = reinterpret_cast<const uint4*>(reinterpret_cast<const WT*>(a.w_down) + ((size_t)p.pair_e[pair] * a.ldx + n) * a.ffp);
        const float* h = a.h32 + (size_t)pair * a.ffp;
        float acc = 0.f;
        for (int c = lane; c < chunks; c += 32) acc = dot_chunk<WT>(__ldg(W + c), h + c * E, acc);
        y += warp_total(acc);
    }
    if (lane == 0) a.x[(size_t)row * a.ldx + n] = y;
}

template <typename WT>
cudaError_t few(const MoeArgs& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)a.ldx;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(moe_few_up_kernel<WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    const cudaError_t e = launch_rows(moe_few_up_kernel<WT>, dim3((unsigned)(a.rows * a.top), (a.ffp + 8 * kUpPerWarp - 1) / (8 * kUpPerWarp)), 256, smem, st, a);
    if (e != cudaSuccess) return e;
    return launch_rows(moe_few_down_kernel<WT>, dim3((unsigned)a.rows, (a.D + 7) / 8), 256, 0, st, a);
}

}  // namespace

int moe_max_tiles(int rows, int top, int E) {
    const long pairs = (long)rows * top;
    return (int)(pairs / kTile + (pairs < E ? pairs : E));
}
size_t moe_plan_ints(int rows, int top, int E) { return (size_t)plan_tiles_at(rows, top, E) + 4 * (size_t)moe_max_tiles(rows, top, E) + 4; }
const int4* moe_tiles(const MoeArgs& a) { return plan_of(a).tiles; }

cudaError_t launch_moe_route(const MoeArgs& a, cudaStream_t st) { return launch_rows(moe_route_kernel, dim3((a.rows + 7) / 8), 256, 0, st, a); }
cudaError_t launch_moe_gather(const MoeArgs& a, cudaStream_t st) { return launch_rows(moe_gather_kernel, dim3(a.rows), 128, 0, st, a); }
cudaError_t launch_moe_combine(const MoeArgs& a, cudaStream_t st) { return launch_rows(moe_combine_kernel, dim3(a.rows), 128, 0, st, a); }
cudaError_t launch_moe_few(const MoeArgs& a, cudaStream_t st) { return a.w_dtype == LUMI_DTYPE_BF16 ? few<__nv_bfloat16>(a, st) : few<float>(a, st); }

}  // namespace lumi
