// Products of a few rows with matrices in groups (a gate's blocks, the per-head projections of a latent), and the kernel that lays
// weights out for them.  The group's rows wait in shared memory; a warp streams the weight rows of four results.
#include "rows.cuh"

namespace lumi {
namespace {

constexpr int kRows = 8;                                  // rows of A per CTA
constexpr int kPerWarp = 4;

__device__ __forceinline__ void widen16(const uint4& v, const float*, float (&w)[4]) {
    w[0] = __uint_as_float(v.x); w[1] = __uint_as_float(v.y); w[2] = __uint_as_float(v.z); w[3] = __uint_as_float(v.w);
}
__device__ __forceinline__ void widen16(const uint4& v, const __nv_bfloat16*, float (&w)[8]) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { w[2 * i] = __uint_as_float(u[i] << 16); w[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u); }
}

template <typename WT>
__global__ void __launch_bounds__(256) block_product_kernel(BlockProductArgs a) {
    extern __shared__ float xs[];                         // [kRows][ldw]
    constexpr int E = 16 / sizeof(WT);
    const int g = blockIdx.y, r0 = blockIdx.z * kRows, nb = min(kRows, a.rows - r0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int n0 = (blockIdx.x * 8 + warp) * kPerWarp, chunks = a.ldw / E;
    const WT* W = reinterpret_cast<const WT*>(a.W) + ((size_t)g * a.group_rows + n0) * a.ldw;
    pdl_release();
    // the weights depend on nothing: the first chunk of every row goes out ahead of the wait
    uint4 first[kPerWarp];
#pragma unroll
    for (int j = 0; j < kPerWarp; ++j)
        first[j] = n0 + j < a.n_out && lane < chunks ? __ldg(reinterpret_cast<const uint4*>(W + (size_t)j * a.ldw) + lane) : make_uint4(0u, 0u, 0u, 0u);
    pdl_sync();
    for (int i = tid; i < nb * a.ldw; i += 256) {
        const int r = i / a.ldw, k = i % a.ldw;
        xs[i] = k < a.K ? a.A[(size_t)(r0 + r) * a.lda + (size_t)g * a.a_step + k] : 0.f;
    }
    __syncthreads();
    float acc[kPerWarp][kRows];
#pragma unroll
    for (int j = 0; j < kPerWarp; ++j)
#pragma unroll
        for (int r = 0; r < kRows; ++r) acc[j][r] = 0.f;
    for (int c = lane; c < chunks; c += 32) {
        float w[kPerWarp][E];
#pragma unroll
        for (int j = 0; j < kPerWarp; ++j) {
            const uint4 v = c == lane ? first[j] : (n0 + j < a.n_out ? __ldg(reinterpret_cast<const uint4*>(W + (size_t)j * a.ldw) + c) : make_uint4(0u, 0u, 0u, 0u));
            widen16(v, (const WT*)nullptr, w[j]);
        }
#pragma unroll
        for (int r = 0; r < kRows; ++r) {
            if (r < nb) {
#pragma unroll
                for (int q = 0; q < E / 4; ++q) {
                    const float4 x = *reinterpret_cast<const float4*>(xs + (size_t)r * a.ldw + c * E + 4 * q);
#pragma unroll
                    for (int j = 0; j < kPerWarp; ++j)
                        acc[j][r] = fmaf(w[j][4 * q], x.x, fmaf(w[j][4 * q + 1], x.y, fmaf(w[j][4 * q + 2], x.z, fmaf(w[j][4 * q + 3], x.w, acc[j][r]))));
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < kPerWarp; ++j)
#pragma unroll
        for (int r = 0; r < kRows; ++r) {
            if (r >= nb) break;
            float v = warp_total(acc[j][r]);
            if (lane == r && n0 + j < a.n_out) {
                if (a.bias != nullptr) v += a.bias[(size_t)g * a.group_rows + n0 + j];
                const size_t col = (size_t)g * a.out_step + n0 + j;
                if (a.mul != nullptr) v = __fdiv_rn(v, 1.0f + expf(-a.mul[(size_t)(r0 + r) * a.ldmul + col]));
                a.D[(size_t)(r0 + r) * a.ldd + col] = v;
            }
        }
}

template <typename T>
__global__ void __launch_bounds__(256) pack_rows_kernel(T* dst, long ld, const T* src, long rows, long cols, long rg, long rs, long ro, long co, bool transpose) {
    for (long i = (long)blockIdx.x * 256 + threadIdx.x; i < rows * cols; i += (long)gridDim.x * 256) {
        const long r = i / cols, c = i % cols;
        if (transpose) dst[(r / rg * rs + c + ro) * ld + co + r % rg] = src[i];
        else dst[(r / rg * rs + r % rg + ro) * ld + co + c] = src[i];
    }
}

template <typename WT>
cudaError_t run(const BlockProductArgs& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * kRows * (size_t)a.ldw;
    auto kern = block_product_kernel<WT>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return launch_rows(kern, dim3((a.n_out + 8 * kPerWarp - 1) / (8 * kPerWarp), a.groups, (a.rows + kRows - 1) / kRows), 256, smem, st, a);
}

}  // namespace

cudaError_t launch_block_product(const BlockProductArgs& a, cudaStream_t st) {
    constexpr int kZ = 65535;
    BlockProductArgs b = a;
    for (int r = 0; r < a.rows; r += kZ * kRows) {        // (the grid's third dimension)
        b.rows = a.rows - r < kZ * kRows ? a.rows - r : kZ * kRows;
        b.A = a.A + (size_t)r * a.lda;
        b.D = a.D + (size_t)r * a.ldd;
        if (a.mul != nullptr) b.mul = a.mul + (size_t)r * a.ldmul;
        const cudaError_t e = a.w_dtype == LUMI_DTYPE_BF16 ? run<__nv_bfloat16>(b, st) : run<float>(b, st);
        if (e != cudaSuccess) return e;
    }
    return cudaSuccess;
}

cudaError_t launch_pack_rows(void* dst, long ld, const void* src, long rows, long cols, int esz, long rg, long rs, long ro, long co, bool transpose,
                             cudaStream_t st) {
    const unsigned blocks = (unsigned)((rows * cols + 255) / 256 < 4096 ? (rows * cols + 255) / 256 : 4096);
    if (blocks == 0) return cudaSuccess;
    if (esz == 2) pack_rows_kernel<uint16_t><<<blocks, 256, 0, st>>>((uint16_t*)dst, ld, (const uint16_t*)src, rows, cols, rg, rs, ro, co, transpose);
    else pack_rows_kernel<uint32_t><<<blocks, 256, 0, st>>>((uint32_t*)dst, ld, (const uint32_t*)src, rows, cols, rg, rs, ro, co, transpose);
    return cudaGetLastError();
}

}  // namespace lumi
