// Gated linear recurrence over channels (one state element each):
//
//   u = conv(x) + b per channel,   r = sigmoid(R_b u_b),  i = sigmoid(I_b u_b)  block by block of channels,
//   log a = -rate r softplus(lam),   S_t = a S_{t-1} + sqrt(1 - a^2) i u,   output S * gelu(y)
//
//   rglru_step_kernel   a decode token, everything in one launch: a CTA takes one block of channels of a few sequences
//   rglru_conv_one_kernel, rglru_point_kernel   the same for many sequences, around a product of all rows with the gates' blocks
//   rglru_conv_kernel   rows of a pass: convolutions, with the halves the block products take
//   rglru_scan_kernel   gates, recurrence and output of a pass: warps take consecutive runs of tokens, the runs are joined through
//                       their decay products and end values
//   rglru_tail_kernel   the convolutions' last inputs into the ring (slot = position % taps, nothing to clear on reset)
//
// Gate rows come in groups of 16 decay-gate rows and the 16 input-gate rows of the same channels.
#include "rows.cuh"

#include <algorithm>

namespace lumi {
namespace {

// sigma(x) with the hardware exponential (relative error of a few 1e-7)
__device__ __forceinline__ float sigmoid_q(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
// z / 2 (1 + tanh(w)) = z sigma(2 w); far out the exponential overflows to an exact 0
__device__ __forceinline__ float gelu_tanh_f(float z) {
    const float w2 = 1.5957691216057308f * (z + 0.044715f * z * z * z);
    return w2 < -80.f ? 0.f : z * sigmoid_q(w2);
}
// decay a and the factor sqrt(1 - a^2) of the input, from the decay gate's logit
__device__ __forceinline__ void decay_of(float r_logit, float sp_rate, float& a, float& b) {
    const float la = -sp_rate * sigmoid_q(fmaxf(r_logit, -80.f));       // sp_rate = rate * softplus(lam)
    a = expf(la);
    // 1 - e^x, x = 2 log a: where x is small by its series (no cancellation), else from a
    const float x = 2.0f * la;
    const float series = -x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 720.f, 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.0f);
    b = __fsqrt_rn(x > -0.25f ? series : fmaf(-a, a, 1.0f));
}

// Convolution input of channel c, d tokens before token t of the pass (d > t: from the ring; none before position 0).
__device__ __forceinline__ float conv_in(const RglruArgs& a, int sl, int t, int d, int pos0, int slot, int c) {
    if (d <= t) return a.proj[(size_t)(sl * a.ts + t - d) * a.ldp + a.off_x + c];
    const int p = pos0 + t - d;
    return p >= 0 ? a.conv[((size_t)slot * a.taps + p % a.taps) * a.channels + c] : 0.f;
}

constexpr int kConvRows = 16;

// One thread per (channel, run of kConvRows tokens).  TAPS > 0: the last inputs stay in registers.
template <int TAPS>
__global__ void __launch_bounds__(128) rglru_conv_kernel(RglruArgs a, int runs) {
    const int c = blockIdx.y * 128 + threadIdx.x, sl = blockIdx.x / runs, t0 = (blockIdx.x % runs) * kConvRows, slot = a.b0 + sl;
    pdl_release();
    pdl_sync();
    if (c >= a.channels) return;
    const int pos0 = a.pos[slot], te = min(a.ts, t0 + kConvRows), n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    const int bs = a.channels / a.blocks, hc = c / bs * a.bp + c % bs;
    const float bias = a.conv_b[c];
    const float* w = a.conv_w + (size_t)c * a.taps;
    auto put = [&](int t, float v) {
        if (t >= n) v = 0.f;
        const size_t row = (size_t)sl * a.ts + t;
        a.u32[row * a.channels + c] = v;
        if (a.uh != nullptr) put_row(nullptr, a.uh, a.ul, row * a.blocks * a.bp + hc, v);
    };
    if constexpr (TAPS > 0) {
        float wt[TAPS], x[TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wt[j] = w[j];
#pragma unroll
        for (int j = 1; j < TAPS; ++j) x[j] = conv_in(a, sl, t0, TAPS - j, pos0, slot, c);
        for (int t = t0; t < te; ++t) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; ++j) x[j] = x[j + 1];
            x[TAPS - 1] = a.proj[(size_t)(sl * a.ts + t) * a.ldp + a.off_x + c];
            float v = bias;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) v = fmaf(wt[j], x[j], v);
            put(t, v);
        }
    } else {
        for (int t = t0; t < te; ++t) {
            float v = bias;
            for (int j = 0; j < a.taps; ++j) v = fmaf(w[j], conv_in(a, sl, t, a.taps - 1 - j, pos0, slot, c), v);
            put(t, v);
        }
    }
}

constexpr int kRun = 16;                                  // tokens per warp and round

// CTA = (32 channels, sequence); lane = channel, warp w of nw takes tokens [w kRun, (w + 1) kRun) of every round of nw kRun tokens.
// A run's decays and inputs stay in registers between the two walks over it.
// (NT: most threads; where there are CTAs enough, small ones overlap each other's phases better)
template <int NT>
__global__ void __launch_bounds__(NT, 1024 / NT) rglru_scan_kernel(RglruArgs a) {
    __shared__ float prod[NT / 32][33], endv[NT / 32][33];
    const int nw = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * 32 + lane, sl = blockIdx.y, slot = a.b0 + sl;
    pdl_release();
    pdl_sync();
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    const bool ok = c < a.channels;
    const int bs = a.channels / a.blocks, cc = ok ? c : 0, blk = cc / bs, i = cc % bs;
    const size_t grow = (size_t)a.blocks * 2 * a.bp;
    const int gr = blk * 2 * a.bp + (i >> 4) * 32 + (i & 15);
    const float sp = a.rate * softplus_f(a.lam[cc]);
    float S = ok ? a.S[(size_t)slot * a.channels + c] : 0.f;        // every warp of the CTA carries the same value
    for (int r0 = 0; r0 < n; r0 += nw * kRun) {
        const int t0 = r0 + warp * kRun, cnt = max(0, min(kRun, n - t0));
        const size_t row0 = (size_t)sl * a.ts + t0;
        const float *gp = a.gates + row0 * grow + gr, *up = a.u32 + row0 * a.channels + c, *yp = a.proj + row0 * a.ldp + a.off_y + c;
        float da[kRun], in[kRun];
#pragma unroll
        for (int k = 0; k < kRun; ++k) {
            da[k] = 1.f;
            in[k] = 0.f;
            if (ok && k < cnt) {
                const float* gt = gp + (size_t)k * grow;
                float f;
                decay_of(gt[0], sp, da[k], f);
                in[k] = f * sigmoid_q(fmaxf(gt[16], -80.f)) * up[(size_t)k * a.channels];
            }
        }
        float p = 1.f, e = 0.f;
#pragma unroll
        for (int k = 0; k < kRun; ++k) { p *= da[k]; e = fmaf(da[k], e, in[k]); }
        prod[warp][lane] = p;
        endv[warp][lane] = e;
        __syncthreads();
        float s = S;
        for (int w = 0; w < nw; ++w) {                    // the state ahead of this warp's run, and behind the round
            if (w == warp) s = S;
            S = fmaf(prod[w][lane], S, endv[w][lane]);
        }
#pragma unroll
        for (int k = 0; k < kRun; ++k) {
            if (k < cnt) {
                s = fmaf(da[k], s, in[k]);
                if (ok) put_row(a.y32, a.yhi, a.ylo, (row0 + k) * a.ldy + c, s * gelu_tanh_f(yp[(size_t)k * a.ldp]));
            }
        }
        __syncthreads();
    }
    if (!ok) return;
    if (a.ts > 1)                                         // rows behind a shorter prompt: zero
        for (int t = n + warp; t < a.ts; t += nw) put_row(a.y32, a.yhi, a.ylo, ((size_t)sl * a.ts + t) * a.ldy + c, 0.f);
    if (warp == 0 && n > 0) a.S[(size_t)slot * a.channels + c] = S;
}

__global__ void __launch_bounds__(256) rglru_tail_kernel(RglruArgs a) {
    const int c = blockIdx.x * 256 + threadIdx.x, sl = blockIdx.y, slot = a.b0 + sl;
    pdl_release();
    pdl_sync();
    if (c >= a.channels) return;
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0), pos0 = a.pos[slot];
    for (int d = 1; d < a.taps && d <= n; ++d)
        a.conv[((size_t)slot * a.taps + (pos0 + n - d) % a.taps) * a.channels + c] = a.proj[(size_t)(sl * a.ts + n - d) * a.ldp + a.off_x + c];
}

// ---- a decode token, many sequences: one thread per V neighbouring channels of a sequence ---------------------------
template <int V> struct Vec;
template <> struct Vec<1> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
    static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
};
template <> struct Vec<4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
// (rows of halves start on multiples of four elements wherever V is 4)
template <int V>
__device__ __forceinline__ void put_halves(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t o, const float (&v)[V]) {
    __nv_bfloat16 h[V], l[V];
#pragma unroll
    for (int e = 0; e < V; ++e) bf16_halves(v[e], h[e], l[e]);
    if constexpr (V == 4) {
        *reinterpret_cast<__nv_bfloat162*>(hi + o) = __halves2bfloat162(h[0], h[1]);
        *reinterpret_cast<__nv_bfloat162*>(hi + o + 2) = __halves2bfloat162(h[2], h[3]);
        if (lo != nullptr) {
            *reinterpret_cast<__nv_bfloat162*>(lo + o) = __halves2bfloat162(l[0], l[1]);
            *reinterpret_cast<__nv_bfloat162*>(lo + o + 2) = __halves2bfloat162(l[2], l[3]);
        }
    } else {
        hi[o] = h[0];
        if (lo != nullptr) lo[o] = l[0];
    }
}

template <int V>
__global__ void __launch_bounds__(128) rglru_conv_one_kernel(RglruArgs a) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * V, sl = blockIdx.y, slot = a.b0 + sl;
    pdl_release();
    float v[V];
    float4 w4[V];                                         // filters of four taps: a channel's in one load
    if (c < a.channels) {
        Vec<V>::load(a.conv_b + c, v);
        if (a.taps == 4)
#pragma unroll
            for (int e = 0; e < V; ++e) w4[e] = __ldg(reinterpret_cast<const float4*>(a.conv_w) + c + e);
    }
    const int pos = a.pos[slot];
    pdl_sync();
    if (c >= a.channels) return;
    const bool live = pass_tokens(a.row_len, a.ctl, slot, 1, a.t_abs0) > 0;
    const float* ring = a.conv + (size_t)slot * a.taps * a.channels + c;
    if (a.taps == 4) {
        float x[4][V] = {};
#pragma unroll
        for (int d = 1; d < 4; ++d) if (pos >= d) Vec<V>::load(ring + (size_t)((pos - d) & 3) * a.channels, x[3 - d]);
        Vec<V>::load(a.proj + (size_t)sl * a.ldp + a.off_x + c, x[3]);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = fmaf(w4[e].w, x[3][e], fmaf(w4[e].z, x[2][e], fmaf(w4[e].y, x[1][e], fmaf(w4[e].x, x[0][e], v[e]))));
    } else for (int j = 0; j < a.taps; ++j) {
        const int d = a.taps - 1 - j;
        float x[V] = {};
        if (d == 0) Vec<V>::load(a.proj + (size_t)sl * a.ldp + a.off_x + c, x);
        else if (pos >= d) Vec<V>::load(ring + (size_t)((pos - d) % a.taps) * a.channels, x);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = fmaf(a.conv_w[(size_t)(c + e) * a.taps + j], x[e], v[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) if (!live) v[e] = 0.f;
    Vec<V>::store(a.u32 + (size_t)sl * a.channels + c, v);
    const int bs = a.channels / a.blocks;
    if (a.uh != nullptr) put_halves<V>(a.uh, a.ul, (size_t)sl * a.blocks * a.bp + c / bs * a.bp + c % bs, v);
}

template <int V>
__global__ void __launch_bounds__(128) rglru_point_kernel(RglruArgs a) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * V, sl = blockIdx.y, slot = a.b0 + sl;
    pdl_release();
    float lam[V], S[V], r[V], in[V], u[V], y[V], x[V];
    float* Sp = a.S + (size_t)slot * a.channels + c;
    const int pos = a.pos[slot];
    if (c < a.channels) {                                 // the state belongs to the step before this one, which has ended
        Vec<V>::load(a.lam + c, lam);
        Vec<V>::load(Sp, S);
    }
    pdl_sync();
    if (c >= a.channels || pass_tokens(a.row_len, a.ctl, slot, 1, a.t_abs0) == 0) return;
    const int bs = a.channels / a.blocks, i = c % bs;
    const float* gt = a.gates + (size_t)sl * a.blocks * 2 * a.bp + c / bs * 2 * a.bp + (i >> 4) * 32 + (i & 15);
    const float* pr = a.proj + (size_t)sl * a.ldp;
    Vec<V>::load(gt, r);
    Vec<V>::load(gt + 16, in);
    Vec<V>::load(a.u32 + (size_t)sl * a.channels + c, u);
    Vec<V>::load(pr + a.off_y + c, y);
    Vec<V>::load(pr + a.off_x + c, x);
#pragma unroll
    for (int e = 0; e < V; ++e) {
        float d, f;
        decay_of(r[e], a.rate * softplus_f(lam[e]), d, f);
        S[e] = fmaf(d, S[e], f * sigmoid_q(fmaxf(in[e], -80.f)) * u[e]);
        y[e] = S[e] * gelu_tanh_f(y[e]);
    }
    Vec<V>::store(Sp, S);
    Vec<V>::store(a.conv + ((size_t)slot * a.taps + pos % a.taps) * a.channels + c, x);      // for later tokens
    if (a.y32 != nullptr) Vec<V>::store(a.y32 + (size_t)sl * a.ldy + c, y);
    if (a.yhi != nullptr) put_halves<V>(a.yhi, a.ylo, (size_t)sl * a.ldy + c, y);
}
// four channels per thread where blocks and rows allow it
bool by_four(const RglruArgs& a) { return ((a.channels | a.channels / a.blocks | a.ldp | a.ldy | a.off_x | a.off_y) & 3) == 0; }

// ---- a decode token, few sequences ---------------------------------------------------------------------------------
constexpr int kStepRows = 4;                              // sequences per CTA

__device__ __forceinline__ void widen16(const uint4& v, const float*, float (&w)[4]) {
    w[0] = __uint_as_float(v.x); w[1] = __uint_as_float(v.y); w[2] = __uint_as_float(v.z); w[3] = __uint_as_float(v.w);
}
__device__ __forceinline__ void widen16(const uint4& v, const __nv_bfloat16*, float (&w)[8]) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { w[2 * i] = __uint_as_float(u[i] << 16); w[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u); }
}

// CTA = (part of a block of channels, kStepRows sequences): `per` channels of the block (a multiple of 16) and all of its inputs.
// Eight lanes share a gate row.
template <typename WT>
__global__ void __launch_bounds__(256) rglru_step_kernel(RglruArgs a, int per, int parts) {
    extern __shared__ float sm[];
    constexpr int E = 16 / sizeof(WT);
    const int bs = a.channels / a.blocks, blk = blockIdx.x / parts, i0 = (blockIdx.x % parts) * per, r0 = blockIdx.y * kStepRows;
    float* us = sm;                                       // [kStepRows][bp]
    float* gs = us + kStepRows * a.bp;                    // [kStepRows][2 per]
    const int tid = threadIdx.x, sub = tid & 7, grp = tid >> 3;
    const int nr = min(kStepRows, a.nseq - r0), chunks = a.bp / E;
    const WT* W = reinterpret_cast<const WT*>(a.rg) + ((size_t)blk * 2 * a.bp + 2 * i0) * a.bp;
    pdl_release();
    // the weights depend on nothing: the first rows go out ahead of the wait
    constexpr int PRE = 4;
    uint4 first[PRE];
#pragma unroll
    for (int q = 0; q < PRE; ++q) first[q] = grp < 2 * per && sub + 8 * q < chunks ? __ldg(reinterpret_cast<const uint4*>(W + (size_t)grp * a.bp) + sub + 8 * q) : make_uint4(0u, 0u, 0u, 0u);
    pdl_sync();
    // convolutions of the whole block
    for (int j = tid; j < nr * a.bp; j += 256) {
        const int r = j / a.bp, i = j % a.bp, sl = r0 + r, slot = a.b0 + sl, c = blk * bs + i;
        float v = 0.f;
        if (i < bs && pass_tokens(a.row_len, a.ctl, slot, 1, a.t_abs0) > 0) {
            const int pos = a.pos[slot];
            v = a.conv_b[c];
            for (int k = 0; k < a.taps; ++k) v = fmaf(a.conv_w[(size_t)c * a.taps + k], conv_in(a, sl, 0, a.taps - 1 - k, pos, slot, c), v);
        }
        us[j] = v;
    }
    __syncthreads();
    for (int n = grp; n < 2 * per; n += 32) {
        float acc[kStepRows] = {};
        for (int q = 0; q * 8 + sub < chunks; ++q) {
            float w[E];
            uint4 raw;
            if (n == grp && q < PRE) {
                raw = first[0];
#pragma unroll
                for (int k = 1; k < PRE; ++k) if (q == k) raw = first[k];
            } else {
                raw = __ldg(reinterpret_cast<const uint4*>(W + (size_t)n * a.bp) + sub + 8 * q);
            }
            widen16(raw, (const WT*)nullptr, w);
#pragma unroll
            for (int r = 0; r < kStepRows; ++r) {
                if (r < nr) {
#pragma unroll
                    for (int e = 0; e < E; e += 4) {
                        const float4 x = *reinterpret_cast<const float4*>(us + r * a.bp + (sub + 8 * q) * E + e);
                        acc[r] = fmaf(w[e], x.x, fmaf(w[e + 1], x.y, fmaf(w[e + 2], x.z, fmaf(w[e + 3], x.w, acc[r]))));
                    }
                }
            }
        }
        const float bias = a.rg_b[(size_t)blk * 2 * a.bp + 2 * i0 + n];
#pragma unroll
        for (int r = 0; r < kStepRows; ++r) {
#pragma unroll
            for (int m = 1; m < 8; m <<= 1) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], m);
            if (sub == 0 && r < nr) gs[r * 2 * per + n] = acc[r] + bias;
        }
    }
    __syncthreads();
    for (int j = tid; j < nr * per; j += 256) {
        const int r = j / per, k = j % per, i = i0 + k, sl = r0 + r, slot = a.b0 + sl, c = blk * bs + i;
        if (i >= bs || pass_tokens(a.row_len, a.ctl, slot, 1, a.t_abs0) == 0) continue;
        const float* gt = gs + r * 2 * per + (k >> 4) * 32 + (k & 15);
        float d, f;
        decay_of(gt[0], a.rate * softplus_f(a.lam[c]), d, f);
        float* Sp = a.S + (size_t)slot * a.channels + c;
        const float s = fmaf(d, *Sp, f * sigmoid_q(fmaxf(gt[16], -80.f)) * us[r * a.bp + i]);
        *Sp = s;
        // this token's convolution input for later ones (no CTA reads the slot of its own position)
        a.conv[((size_t)slot * a.taps + a.pos[slot] % a.taps) * a.channels + c] = a.proj[(size_t)sl * a.ldp + a.off_x + c];
        put_row(a.y32, a.yhi, a.ylo, (size_t)sl * a.ldy + c, s * gelu_tanh_f(a.proj[(size_t)sl * a.ldp + a.off_y + c]));
    }
}

size_t step_smem(const RglruArgs& a, int per) { return sizeof(float) * kStepRows * ((size_t)a.bp + 2 * per); }

}  // namespace

cudaError_t launch_rglru_conv(const RglruArgs& a, cudaStream_t st) {
    if (a.ts == 1 && a.nseq <= 65535) {
        if (by_four(a)) return launch_rows(rglru_conv_one_kernel<4>, dim3((a.channels + 511) / 512, a.nseq), 128, 0, st, a);
        return launch_rows(rglru_conv_one_kernel<1>, dim3((a.channels + 127) / 128, a.nseq), 128, 0, st, a);
    }
    const int runs = (a.ts + kConvRows - 1) / kConvRows;
    const dim3 grid((unsigned)((long)a.nseq * runs), (a.channels + 127) / 128);
    if (a.taps == 2) return launch_rows(rglru_conv_kernel<2>, grid, 128, 0, st, a, runs);
    if (a.taps == 3) return launch_rows(rglru_conv_kernel<3>, grid, 128, 0, st, a, runs);
    if (a.taps == 4) return launch_rows(rglru_conv_kernel<4>, grid, 128, 0, st, a, runs);
    return launch_rows(rglru_conv_kernel<0>, grid, 128, 0, st, a, runs);
}

cudaError_t launch_rglru_scan(const RglruArgs& a, cudaStream_t st, int* launches) {
    *launches = 1;
    if (a.ts == 1 && a.nseq <= 65535) {
        if (by_four(a)) return launch_rows(rglru_point_kernel<4>, dim3((a.channels + 511) / 512, a.nseq), 128, 0, st, a);
        return launch_rows(rglru_point_kernel<1>, dim3((a.channels + 127) / 128, a.nseq), 128, 0, st, a);
    }
    cudaError_t e;
    const int nw = std::min(32, (a.ts + kRun - 1) / kRun);
    const dim3 grid((a.channels + 31) / 32, a.nseq);
    if (nw <= 16 || (long)grid.x * grid.y >= 296) e = launch_rows(rglru_scan_kernel<512>, grid, 32 * std::min(nw, 16), 0, st, a);
    else e = launch_rows(rglru_scan_kernel<1024>, grid, 32 * nw, 0, st, a);
    if (e != cudaSuccess || a.taps == 1) return e;
    *launches = 2;
    return launch_rows(rglru_tail_kernel, dim3((a.channels + 255) / 256, a.nseq), 256, 0, st, a);
}

bool rglru_step_supported(const RglruArgs& a) { return a.ts == 1 && step_smem(a, a.bp) <= 200 * 1024; }

cudaError_t launch_rglru_step(const RglruArgs& a, cudaStream_t st) {
    // few sequences: a block's channels over several CTAs, so that the weights stream through more SMs
    int per = a.bp;
    const long tiles = (a.nseq + kStepRows - 1) / kStepRows;
    while (per > 16 && per % 32 == 0 && tiles * a.blocks * (a.bp / per) < 148) per /= 2;
    const int parts = a.bp / per;
    const size_t smem = step_smem(a, per);
    auto kern = a.rg_dtype == LUMI_DTYPE_BF16 ? rglru_step_kernel<__nv_bfloat16> : rglru_step_kernel<float>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return launch_rows(kern, dim3(a.blocks * parts, (unsigned)tiles), 256, smem, st, a, per, parts);
}

}  // namespace lumi
