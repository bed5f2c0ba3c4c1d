// Helpers shared by the kernels of listed layers.
#pragma once
#include "internal.h"

namespace lumi {

__device__ __forceinline__ void pdl_release() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_sync() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

__device__ __forceinline__ float warp_total(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return __fdiv_rn(1.0f, 1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return __fdiv_rn(x, 1.0f + expf(-x)); }
__device__ __forceinline__ void bf16_halves(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(v);
    lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
// Writes one element of an output row in whichever forms the caller asked for.
__device__ __forceinline__ void put_row(float* y32, __nv_bfloat16* hi, __nv_bfloat16* lo, size_t o, float v) {
    if (y32 != nullptr) y32[o] = v;
    if (hi != nullptr) {
        __nv_bfloat16 h, l;
        bf16_halves(v, h, l);
        hi[o] = h;
        if (lo != nullptr) lo[o] = l;
    }
}
// Prompts of different lengths: tokens of this pass that belong to the sequence in `slot` (all of them without a table).
// Decode steps (ts == 1) ask the step's prompt position, prompt slices the pass's first token t_abs0.
__device__ __forceinline__ int pass_tokens(const int32_t* row_len, const StepCtl* ctl, int slot, int ts, int t_abs0) {
    if (row_len == nullptr) return ts;
    if (t_abs0 < 0) {                        // decode form
        const int pp = ctl->prompt_pos;
        return pp < ctl->prompt_len && pp >= row_len[slot] ? 0 : ts;
    }
    return max(0, min(ts, row_len[slot] - t_abs0));
}
// cos and sin of a rotary angle; freq in half turns per position.  The product is formed and reduced in double, so that far
// positions keep full single precision.
__device__ __forceinline__ float2 rot_cos_sin(int pos, double freq) {
    const double turns = (double)pos * freq;
    float2 cs;
    sincospif((float)(turns - 2.0 * rint(0.5 * turns)), &cs.y, &cs.x);
    return cs;
}

// Launch with the programmatic-dependent-launch attribute where the calling thread has it on.
template <typename... KArgs, typename... Args>
cudaError_t launch_rows(void (*kern)(KArgs...), dim3 grid, int threads, size_t smem, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = launch_pdl_on() ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, KArgs(args)...);
}

}  // namespace lumi
