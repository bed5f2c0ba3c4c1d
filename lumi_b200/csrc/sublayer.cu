// Row-wise passes around the sublayers of listed layers.  Norm of a sublayer's output on its way into the residual stream.  A row is x + rms(o) * w: the product that follows needs
// the finished row, so its bf16 halves are written in the same pass.
#include "rows.cuh"

namespace lumi {
namespace {

// One CTA per row; rows are whole float4s (padded widths), padding holds zeros in x, o and w.
template <int NT>
__global__ void __launch_bounds__(NT) row_norm_kernel(RowNormArgs a) {
    __shared__ float red[NT / 32];
    const int r = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_release();
    pdl_sync();
    const int src = a.row_idx != nullptr ? a.row_idx[r] : r;
    const int n4 = a.ld >> 2;
    const float4* in = reinterpret_cast<const float4*>((a.o != nullptr ? a.o : a.x) + (size_t)src * a.ld);
    constexpr int KEEP = 4;                               // float4s per thread kept in registers between the two passes
    float4 v[KEEP];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int c = tid + i * NT;
        v[i] = c < n4 ? in[c] : make_float4(0.f, 0.f, 0.f, 0.f);
        s = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, s))));
    }
    for (int c = tid + KEEP * NT; c < n4; c += NT) {
        const float4 t = in[c];
        s = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, s))));
    }
    s = warp_total(s);
    if (lane == 0) red[warp] = s;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < NT / 32; ++w) tot += red[w];
    const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(tot, (float)a.width) + a.eps));
    auto finish = [&](int c, float4 t) {
        const float4 w = __ldg(reinterpret_cast<const float4*>(a.w) + c);
        float4 y = make_float4(t.x * rs * w.x, t.y * rs * w.y, t.z * rs * w.z, t.w * rs * w.w);
        const size_t oo = (size_t)r * a.ld + 4 * (size_t)c;
        if (a.o != nullptr) {
            const float4 x = *reinterpret_cast<const float4*>(a.x + oo);
            y = make_float4(x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w);
            *reinterpret_cast<float4*>((a.x_out != nullptr ? a.x_out : a.x) + oo) = y;
        } else if (a.y32 != nullptr) {
            *reinterpret_cast<float4*>(a.y32 + oo) = y;
        }
        if (a.hi != nullptr) {
            const __nv_bfloat162 h0 = __floats2bfloat162_rn(y.x, y.y), h1 = __floats2bfloat162_rn(y.z, y.w);
            uint2 u;
            u.x = *reinterpret_cast<const uint32_t*>(&h0); u.y = *reinterpret_cast<const uint32_t*>(&h1);
            *reinterpret_cast<uint2*>(a.hi + oo) = u;
            if (a.lo != nullptr) {
                const float2 f0 = __bfloat1622float2(h0), f1 = __bfloat1622float2(h1);
                const __nv_bfloat162 l0 = __floats2bfloat162_rn(y.x - f0.x, y.y - f0.y), l1 = __floats2bfloat162_rn(y.z - f1.x, y.w - f1.y);
                u.x = *reinterpret_cast<const uint32_t*>(&l0); u.y = *reinterpret_cast<const uint32_t*>(&l1);
                *reinterpret_cast<uint2*>(a.lo + oo) = u;
            }
        }
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int c = tid + i * NT;
        if (c < n4) finish(c, v[i]);
    }
    for (int c = tid + KEEP * NT; c < n4; c += NT) finish(c, in[c]);
}

// One warp per (row, head): RMS norm of the read-out, weight, gate.
__global__ void __launch_bounds__(256) head_gate_kernel(HeadGateArgs a) {
    const long w = ((long)blockIdx.x * 256 + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    pdl_release();
    pdl_sync();
    if (w >= (long)a.nseq * a.ts * a.H) return;
    const int row = (int)(w / a.H), h = (int)(w % a.H), sl = row / a.ts, t = row % a.ts;
    const bool live = t < pass_tokens(a.row_len, a.ctl, a.b0 + sl, a.ts, a.t_abs0);
    const float* o = a.o + ((size_t)row * a.H + h) * a.dvp;
    const float* gate = a.gate + (size_t)row * a.ldg + h * a.dv;
    const size_t oo = (size_t)row * a.ldy + h * a.dv;
    if ((a.dv & 3) == 0 && a.dv <= 512 && ((a.ldg | a.ldy) & 3) == 0 && (reinterpret_cast<uintptr_t>(a.gate) & 15) == 0) {      // four neighbouring elements per lane
        float4 v[4];
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * (lane + 32 * i);
            v[i] = live && c < a.dv ? *reinterpret_cast<const float4*>(o + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            s = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, s))));
        }
        const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(warp_total(s), (float)a.dv) + a.eps));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * (lane + 32 * i);
            if (c >= a.dv) break;
            float y[4] = {0.f, 0.f, 0.f, 0.f};
            if (live) {
                const float4 gt = *reinterpret_cast<const float4*>(gate + c);
                const float ov[4] = {v[i].x, v[i].y, v[i].z, v[i].w}, gv[4] = {gt.x, gt.y, gt.z, gt.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) y[e] = ov[e] * rs * (a.w != nullptr ? a.w[c + e] : 1.f) * __fdividef(gv[e], 1.0f + __expf(-gv[e]));
            }
            if (a.y32 != nullptr) *reinterpret_cast<float4*>(a.y32 + oo + c) = make_float4(y[0], y[1], y[2], y[3]);
            if (a.yhi != nullptr) {
                const __nv_bfloat162 h0 = __floats2bfloat162_rn(y[0], y[1]), h1 = __floats2bfloat162_rn(y[2], y[3]);
                uint2 u;
                u.x = *reinterpret_cast<const uint32_t*>(&h0); u.y = *reinterpret_cast<const uint32_t*>(&h1);
                *reinterpret_cast<uint2*>(a.yhi + oo + c) = u;
                if (a.ylo != nullptr) {
                    const float2 f0 = __bfloat1622float2(h0), f1 = __bfloat1622float2(h1);
                    const __nv_bfloat162 l0 = __floats2bfloat162_rn(y[0] - f0.x, y[1] - f0.y), l1 = __floats2bfloat162_rn(y[2] - f1.x, y[3] - f1.y);
                    u.x = *reinterpret_cast<const uint32_t*>(&l0); u.y = *reinterpret_cast<const uint32_t*>(&l1);
                    *reinterpret_cast<uint2*>(a.ylo + oo + c) = u;
                }
            }
        }
        return;
    }
    float s = 0.f;
    if (live) for (int c = lane; c < a.dv; c += 32) s = fmaf(o[c], o[c], s);
    s = warp_total(s);
    const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(s, (float)a.dv) + a.eps));
    for (int c = lane; c < a.dv; c += 32)
        put_row(a.y32, a.yhi, a.ylo, oo + c, live ? o[c] * rs * (a.w != nullptr ? a.w[c] : 1.f) * silu_f(gate[c]) : 0.f);
}

}  // namespace

cudaError_t launch_head_gate(const HeadGateArgs& a, cudaStream_t st) {
    return launch_rows(head_gate_kernel, dim3((unsigned)(((long)a.nseq * a.ts * a.H + 7) / 8)), 256, 0, st, a);
}

cudaError_t launch_row_norm(const RowNormArgs& a, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.rows);
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = launch_pdl_on() ? 1 : 0;
    if (a.ld <= 1024) { cfg.blockDim = dim3(128); return cudaLaunchKernelEx(&cfg, row_norm_kernel<128>, a); }
    cfg.blockDim = dim3(256);
    return cudaLaunchKernelEx(&cfg, row_norm_kernel<256>, a);
}

}  // namespace lumi
