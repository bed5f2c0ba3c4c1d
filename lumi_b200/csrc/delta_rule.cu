// Gated delta rule over a matrix state per head:
//
//   S_t = g_t S_{t-1} + k_t u_t^T,   u_t = b_t (v_t - g_t S_{t-1}^T k_t),   o_t = S_t^T q_t
//
// with q, k, v from short causal convolutions + silu, q and k unit vectors, one decay g and one step size b per head, and a
// gated RMS norm per head behind the read-out.  Two forms of the same recurrence:
//
//   delta_step_kernel    token after token, the head's state in shared memory: decode steps (one token, everything from the
//                        convolution to the gated norm in one launch), and prompts of fp32 models or unusual sizes.
//   delta_chunk_kernel   prompt slices in chunks of 64 tokens on the tensor cores.  With G_t the running sum of log g inside a
//                        chunk and S_0 the state ahead of it, the rows U of the chunk solve the unit lower triangular system
//                          (I + A) U = diag(b) (V - diag(e^G) K S_0),   A_ts = b_t e^(G_t - G_s) k_t.k_s   (s < t)
//                        and then O = diag(e^G) Q S_0 + P U with P_ts = e^(G_t - G_s) q_t.k_s (s <= t), and the state becomes
//                        e^(G_C) S_0 + K^T diag(e^(G_C - G)) U.  Products take fp32 operands as two tf32 terms each
//                        (three MMAs), so they keep about fp32 accuracy.
//
// Raw convolution inputs live in a ring over positions (slot = position % taps): a step writes the slot of its own position
// and reads the others, so the CTAs of one launch never touch a slot that another one writes.
#include "rows.cuh"
#include "tf32.cuh"

#include <cmath>

namespace lumi {
namespace {

// Convolution output (before silu) of one channel at token t of the pass: inputs of this pass from the projection rows,
// earlier ones from the ring, none before position 0.
__device__ __forceinline__ float conv_at(const DeltaArgs& a, int row, int t, int pos0, int slot, int off, int rc, const float* w) {
    const float* ring = a.conv + (size_t)slot * a.taps * (2 * a.G * a.dk + a.H * a.dv);
    const int channels = 2 * a.G * a.dk + a.H * a.dv;
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {
        const int d = a.taps - 1 - j;                     // how far back this tap reaches
        float x = 0.f;
        if (d <= t) x = a.proj[(size_t)(row - d) * a.ldp + off];
        else if (pos0 + t - d >= 0) x = ring[(size_t)((pos0 + t - d) % a.taps) * channels + rc];
        acc = fmaf(w[j], x, acc);
    }
    return acc;
}

// ---- token after token ----------------------------------------------------------------------------------
__device__ __forceinline__ uint32_t smem_of(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
constexpr uint64_t kStateWaitNs = 500000000ull;           // limit of the wait for a head's state
// false if the phase did not complete within the limit
__device__ __forceinline__ bool state_wait(uint64_t* bar) {
    uint32_t done = 0, polls = 0;
    uint64_t t0 = 0;
    while (true) {
        asm volatile("{\n.reg .pred p;\nmbarrier.try_wait.parity.shared::cta.b64 p, [%1], 0;\nselp.u32 %0, 1, 0, p;\n}" : "=r"(done) : "r"(smem_of(bar)) : "memory");
        if (done) return true;
        if ((++polls & 255u) == 0u) {
            uint64_t now;
            asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(now));
            if (t0 == 0) t0 = now;
            else if (now - t0 > kStateWaitNs) return false;
        }
    }
}

// CTA = (head, sequence).  The head's state is one contiguous block: a bulk copy brings it into shared memory (requested ahead
// of the predecessor's results), a bulk copy takes it back.  Thread (rg, cg) works on rows rg, rg + RG, ... of four neighbouring
// columns; S^T k and S^T q are taken in one walk over the old state (S_t^T q = g S_{t-1}^T q + (k.q) u), so a token needs one
// reduction.  STAGED = false: the state stays in global memory (heads beyond shared memory).
template <int NT, bool STAGED>
__global__ void __launch_bounds__(NT, NT == 128 ? 8 : 5) delta_step_kernel(DeltaArgs a, int cwl) {
    extern __shared__ __align__(128) float dyn[];
    __shared__ __align__(8) uint64_t bar;
    const int h = blockIdx.x, sl = blockIdx.y, slot = a.b0 + sl;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dk = a.dk, dv = a.dv, dvp = a.dvp, kvh = h / (a.H / a.G);
    const int CW = 1 << cwl, cg = tid & (CW - 1), rg = tid >> cwl, RG = NT >> cwl;
    const int c4n = dvp >> 2;
    const bool act = cg < c4n;
    const int share = CW < 32 ? 32 : CW;                  // threads that leave one partial row behind
    const int slots = NT / share;
    float* sm = dyn + (STAGED ? (size_t)dk * dvp : 0);
    float* qs = sm;
    float* ks = qs + dk;
    float* vs = ks + dk;
    float* us = vs + dvp;
    float* os = us + dvp;
    float* rk_s = os + dvp;                               // [slots][dvp] partial S^T k
    float* rq_s = rk_s + slots * dvp;                     // [slots][dvp] partial S^T q
    float* sc = rq_s + slots * dvp;                       // sums: q.q, k.k, q.k, beta, decay

    float* Sg = a.S + ((size_t)slot * a.H + h) * dk * dvp;
    const uint32_t bytes = (uint32_t)dk * dvp * 4u;
    auto request = [&]() {                                // thread 0
        asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_of(&bar)));
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_of(&bar)), "r"(bytes) : "memory");
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(smem_of(dyn)), "l"(Sg), "r"(bytes), "r"(smem_of(&bar)) : "memory");
    };
    pdl_release();
    // the state belongs to the step before this one, which has ended: requested ahead of the predecessor's results
    if (STAGED && a.row_len == nullptr && tid == 0) request();
    // Channel c of the head's q | k | v: its projection column, its place in the ring, its filter; false for padding.
    const int Cq = a.G * dk, channels = 2 * Cq + a.H * dv;
    auto channel = [&](int c, int& off, int& rc, const float*& w) {
        if (c < dk) { off = a.off_q + kvh * dk + c; rc = kvh * dk + c; w = a.conv_q + (size_t)rc * a.taps; return true; }
        if (c < 2 * dk) { const int k = kvh * dk + c - dk; off = a.off_k + k; rc = Cq + k; w = a.conv_k + (size_t)k * a.taps; return true; }
        if (c - 2 * dk >= dv) return false;
        const int v = h * dv + c - 2 * dk;
        off = a.off_v + v; rc = 2 * Cq + v; w = a.conv_v + (size_t)v * a.taps;
        return true;
    };
    // A single token: what earlier tokens put into the convolutions belongs to the steps before this one as well
    constexpr int PRE = 2;
    const int pos0 = a.pos[slot], here = pos0 % a.taps;
    float past[PRE], wcur[PRE];
    if (a.ts == 1) {
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
            const int c = tid + i * NT;
            int off, rc;
            const float* w;
            past[i] = wcur[i] = 0.f;
            if (c < 2 * dk + dvp && channel(c, off, rc, w)) {
                const float* ring = a.conv + (size_t)slot * a.taps * channels + rc;
                for (int j = 0; j + 1 < a.taps; ++j) {
                    const int d = a.taps - 1 - j, rs = here - d;          // ring slot of position pos0 - d
                    past[i] = fmaf(w[j], pos0 >= d ? ring[(size_t)(rs < 0 ? rs + a.taps : rs) * channels] : 0.f, past[i]);
                }
                wcur[i] = w[a.taps - 1];
            }
        }
    }
    pdl_sync();
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    if (n == 0 && a.ts == 1) return;
    if (STAGED && a.row_len != nullptr && n > 0 && tid == 0) request();
    float4* St = reinterpret_cast<float4*>(STAGED ? dyn : Sg);

    for (int t = 0; t < n; ++t) {
        const int row = sl * a.ts + t;
        const float* pr = a.proj + (size_t)row * a.ldp;
        // (qs | ks | vs are contiguous)
        int first = tid;
        if (a.ts == 1) {
#pragma unroll
            for (int i = 0; i < PRE; ++i, first += NT) {
                int off, rc;
                const float* w;
                if (first < 2 * dk + dvp) sm[first] = channel(first, off, rc, w) ? silu_f(fmaf(wcur[i], pr[off], past[i])) : 0.f;
            }
        }
        for (int c = first; c < 2 * dk + dvp; c += NT) {
            int off, rc;
            const float* w;
            sm[c] = channel(c, off, rc, w) ? silu_f(conv_at(a, row, t, pos0, slot, off, rc, w)) : 0.f;
        }
        __syncthreads();
        if (warp < 3) {
            const float* x = warp == 1 ? ks : qs;
            const float* y = warp == 0 ? qs : ks;
            float s = 0.f;
            for (int c = lane; c < dk; c += 32) s = fmaf(x[c], y[c], s);
            s = warp_total(s);
            if (lane == 0) sc[warp] = s;
        } else if (warp == 3 && lane == 0) {
            sc[3] = __fdiv_rn(1.0f, 1.0f + expf(-pr[a.off_b + h]));
            sc[4] = expf(-expf(a.a_log[h]) * softplus_f(pr[a.off_a + h] + a.dt_bias[h]));
        }
        // partial S^T k and S^T q over this thread's rows (old state, raw k and q: the factors come afterwards)
        if (STAGED && t == 0) {
            if (__syncthreads_or(!state_wait(&bar))) {    // report, and let the copy land (again with a limit) before the memory goes away
                if (tid == 0) {
                    if (a.status != nullptr) atomicOr(a.status, STATUS_TIMEOUT);
                    state_wait(&bar);
                }
                __syncthreads();
                return;
            }
        }
        float4 pk = make_float4(0.f, 0.f, 0.f, 0.f), pq = pk;
        if (act) {
#pragma unroll 8
            for (int r = rg; r < dk; r += RG) {
                const float4 s4 = St[(size_t)r * c4n + cg];
                const float kv = ks[r], qv = qs[r];
                pk.x = fmaf(kv, s4.x, pk.x); pk.y = fmaf(kv, s4.y, pk.y); pk.z = fmaf(kv, s4.z, pk.z); pk.w = fmaf(kv, s4.w, pk.w);
                pq.x = fmaf(qv, s4.x, pq.x); pq.y = fmaf(qv, s4.y, pq.y); pq.z = fmaf(qv, s4.z, pq.z); pq.w = fmaf(qv, s4.w, pq.w);
            }
        }
        for (int o = CW; o < 32; o <<= 1) {
            pk.x += __shfl_xor_sync(0xffffffffu, pk.x, o); pk.y += __shfl_xor_sync(0xffffffffu, pk.y, o);
            pk.z += __shfl_xor_sync(0xffffffffu, pk.z, o); pk.w += __shfl_xor_sync(0xffffffffu, pk.w, o);
            pq.x += __shfl_xor_sync(0xffffffffu, pq.x, o); pq.y += __shfl_xor_sync(0xffffffffu, pq.y, o);
            pq.z += __shfl_xor_sync(0xffffffffu, pq.z, o); pq.w += __shfl_xor_sync(0xffffffffu, pq.w, o);
        }
        if (act && (CW >= 32 || lane < CW)) {
            float* dk_ = rk_s + (tid / share) * dvp + 4 * cg;
            float* dq_ = rq_s + (tid / share) * dvp + 4 * cg;
            dk_[0] = pk.x; dk_[1] = pk.y; dk_[2] = pk.z; dk_[3] = pk.w;
            dq_[0] = pq.x; dq_[1] = pq.y; dq_[2] = pq.z; dq_[3] = pq.w;
        }
        __syncthreads();
        const float rq = __fdiv_rn(__frcp_rn(__fsqrt_rn(sc[0] + a.unit_eps)), __fsqrt_rn((float)dk));
        const float rk = __frcp_rn(__fsqrt_rn(sc[1] + a.unit_eps));
        const float kq = rq * rk * sc[2], beta = sc[3], g = sc[4];
        for (int c = tid; c < dvp; c += NT) {
            float sk = 0.f, sq = 0.f;
            for (int p = 0; p < slots; ++p) { sk += rk_s[p * dvp + c]; sq += rq_s[p * dvp + c]; }
            const float u = beta * (vs[c] - g * rk * sk);
            us[c] = c < dv ? u : 0.f;
            os[c] = c < dv ? fmaf(kq, u, g * rq * sq) : 0.f;
        }
        __syncthreads();
        if (act) {
            const float4 u4 = make_float4(us[4 * cg], us[4 * cg + 1], us[4 * cg + 2], us[4 * cg + 3]);
#pragma unroll 8
            for (int r = rg; r < dk; r += RG) {
                const float4 s4 = St[(size_t)r * c4n + cg];
                const float kv = rk * ks[r];
                St[(size_t)r * c4n + cg] = make_float4(fmaf(kv, u4.x, g * s4.x), fmaf(kv, u4.y, g * s4.y), fmaf(kv, u4.z, g * s4.z), fmaf(kv, u4.w, g * s4.w));
            }
            if (STAGED && t + 1 == n) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");      // ahead of the copy back
        }
        float ss = 0.f;
        for (int c = lane; c < dv; c += 32) ss = fmaf(os[c], os[c], ss);
        ss = warp_total(ss);
        const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(ss, (float)dv) + a.eps));
        for (int c = tid; c < dv; c += NT)
            put_row(a.y32, a.yhi, a.ylo, (size_t)row * a.ldy + h * dv + c, os[c] * rs * a.o_norm[c] * silu_f(pr[a.off_g + h * dv + c]));
        if (t + 1 < n) __syncthreads();                   // the staged vectors are rewritten by the next token
    }
    for (int t = n; t < a.ts; ++t)                        // rows behind a shorter prompt: zero, so that what follows stays finite
        for (int c = tid; c < dv; c += NT) put_row(a.y32, a.yhi, a.ylo, (size_t)(sl * a.ts + t) * a.ldy + h * dv + c, 0.f);
    if (n == 0) return;
    if (STAGED) {
        __syncthreads();
        if (tid == 0) {
            asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(Sg), "r"(smem_of(dyn)), "r"(bytes) : "memory");
            asm volatile("cp.async.bulk.commit_group;" ::: "memory");
        }
    }
    if (a.ts == 1) {                                      // this token's raw convolution inputs
        const float* pr = a.proj + (size_t)sl * a.ldp;
        float* ring = a.conv + ((size_t)slot * a.taps + here) * channels;
        if (h % (a.H / a.G) == 0) {
            for (int c = tid; c < dk; c += NT) {
                ring[kvh * dk + c] = pr[a.off_q + kvh * dk + c];
                ring[Cq + kvh * dk + c] = pr[a.off_k + kvh * dk + c];
            }
        }
        for (int c = tid; c < dv; c += NT) ring[2 * Cq + h * dv + c] = pr[a.off_v + h * dv + c];
    }
    // the memory of the CTA has been read; the writes themselves end with the kernel
    if (STAGED && tid == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
}

// After a pass of several tokens: the last taps - 1 raw inputs of every channel go into the ring (a launch of its own, since
// the kernels of the pass still read the ring's earlier contents).
__global__ void __launch_bounds__(256) conv_tail_kernel(DeltaArgs a) {
    const int Cq = a.G * a.dk, channels = 2 * Cq + a.H * a.dv;
    const int c = blockIdx.x * 256 + threadIdx.x, sl = blockIdx.y, slot = a.b0 + sl;
    if (c >= channels) return;
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    const int off = c < Cq ? a.off_q + c : (c < 2 * Cq ? a.off_k + c - Cq : a.off_v + c - 2 * Cq);
    const int pos0 = a.pos[slot];
    for (int d = 1; d < a.taps && d <= n; ++d)
        a.conv[((size_t)slot * a.taps + (pos0 + n - d) % a.taps) * channels + c] = a.proj[(size_t)(sl * a.ts + n - d) * a.ldp + off];
}

// ---- chunks of 64 tokens -----------------------------------------------------------------------------------
constexpr int CH = 64;
constexpr int kMaxChunkDim = 256;

// One warp per (row, unit): unit = a q head, a k head, a v head, or the gates of the row.
__global__ void __launch_bounds__(256) delta_prep_kernel(DeltaArgs a, int dk4) {
    const int units = 2 * a.G + a.H + 1;
    const long w = ((long)blockIdx.x * 256 + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long)a.nseq * a.ts * units) return;
    const int row = (int)(w / units), un = (int)(w % units), sl = row / a.ts, t = row % a.ts, slot = a.b0 + sl;
    const bool live = t < pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    const int pos0 = a.pos[slot], Cq = a.G * a.dk;
    float* out = a.qkv + (size_t)row * a.ldqkv;
    if (un < 2 * a.G) {
        const bool is_k = un >= a.G;
        const int g = is_k ? un - a.G : un;
        float v[kMaxChunkDim / 32];
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < kMaxChunkDim / 32; ++i) {
            const int c = lane + 32 * i;
            v[i] = 0.f;
            if (c < a.dk && live) {
                const float* cw = (is_k ? a.conv_k : a.conv_q) + (size_t)(g * a.dk + c) * a.taps;
                v[i] = silu_f(conv_at(a, row, t, pos0, slot, (is_k ? a.off_k : a.off_q) + g * a.dk + c, (is_k ? Cq : 0) + g * a.dk + c, cw));
                s = fmaf(v[i], v[i], s);
            }
        }
        float r = __frcp_rn(__fsqrt_rn(warp_total(s) + a.unit_eps));
        if (!is_k) r = __fdiv_rn(r, __fsqrt_rn((float)a.dk));
#pragma unroll
        for (int i = 0; i < kMaxChunkDim / 32; ++i) {
            const int c = lane + 32 * i;
            if (c < dk4) out[(size_t)un * dk4 + c] = v[i] * r;
        }
    } else if (un < 2 * a.G + a.H) {
        const int h = un - 2 * a.G;
        for (int c = lane; c < a.dvp; c += 32) {
            float v = 0.f;
            if (c < a.dv && live)
                v = silu_f(conv_at(a, row, t, pos0, slot, a.off_v + h * a.dv + c, 2 * Cq + h * a.dv + c, a.conv_v + (size_t)(h * a.dv + c) * a.taps));
            out[(size_t)2 * a.G * dk4 + h * a.dvp + c] = v;
        }
    } else {
        const float* pr = a.proj + (size_t)row * a.ldp;
        for (int h = lane; h < a.H; h += 32) {
            float2 bg = make_float2(0.f, 0.f);
            if (live) {
                bg.x = __fdiv_rn(1.0f, 1.0f + expf(-pr[a.off_b + h]));
                bg.y = -expf(a.a_log[h]) * softplus_f(pr[a.off_a + h] + a.dt_bias[h]);
            }
            reinterpret_cast<float2*>(a.gates)[(size_t)row * a.H + h] = bg;
        }
    }
}

// The same for short filters of TAPS <= 4 taps and heads of up to 32 NI channels, kPrepRows rows per warp: a row's inputs stay in
// registers for the taps of the rows behind it, so every projection element is read once.
constexpr int kPrepRows = 16;
template <int TAPS, int NI>
__global__ void __launch_bounds__(256) delta_prep_rows_kernel(DeltaArgs a, int dk4, int blocks_per_seq) {
    const int units = 2 * a.G + a.H + 1;
    const long w = ((long)blockIdx.x * 256 + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long)a.nseq * blocks_per_seq * units) return;
    const int un = (int)(w % units), sl = (int)(w / units) / blocks_per_seq, tb = ((int)(w / units) % blocks_per_seq) * kPrepRows, slot = a.b0 + sl;
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0), te = min(a.ts, tb + kPrepRows);
    const int pos0 = a.pos[slot], Cq = a.G * a.dk;
    if (un == 2 * a.G + a.H) {                            // the gates
        for (int i = lane; i < (te - tb) * a.H; i += 32) {
            const int t = tb + i / a.H, h = i % a.H, row = sl * a.ts + t;
            const float* pr = a.proj + (size_t)row * a.ldp;
            float2 bg = make_float2(0.f, 0.f);
            if (t < n) {
                bg.x = __fdiv_rn(1.0f, 1.0f + expf(-pr[a.off_b + h]));
                bg.y = -expf(a.a_log[h]) * softplus_f(pr[a.off_a + h] + a.dt_bias[h]);
            }
            reinterpret_cast<float2*>(a.gates)[(size_t)row * a.H + h] = bg;
        }
        return;
    }
    const bool is_v = un >= 2 * a.G, is_k = !is_v && un >= a.G;
    const int head = is_v ? un - 2 * a.G : (is_k ? un - a.G : un), d = is_v ? a.dv : a.dk, dpad = is_v ? a.dvp : dk4;
    const int ch0 = head * d;                             // first channel of the head in its projection part
    const int off = (is_v ? a.off_v : (is_k ? a.off_k : a.off_q)) + ch0, rc = (is_v ? 2 * Cq : (is_k ? Cq : 0)) + ch0;
    const float* cw = (is_v ? a.conv_v : (is_k ? a.conv_k : a.conv_q)) + (size_t)ch0 * TAPS;
    const size_t oo = is_v ? (size_t)2 * a.G * dk4 + (size_t)head * a.dvp : (size_t)un * dk4;
    const int channels = 2 * Cq + a.H * a.dv;
    for (int c0 = 0; c0 < d; c0 += 32 * NI) {             // value heads may be wider than the key heads NI was chosen for
        float wt[NI][TAPS], hist[NI][TAPS];               // hist[TAPS - 1] = current input
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c = c0 + lane + 32 * i;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) wt[i][j] = c < d ? cw[(size_t)c * TAPS + j] : 0.f;
#pragma unroll
            for (int j = 1; j < TAPS; ++j) {              // inputs of tokens tb - (TAPS - j), ... tb - 1
                const int t = tb - TAPS + j;
                float x = 0.f;
                if (c < d) {
                    if (t >= 0) x = a.proj[(size_t)(sl * a.ts + t) * a.ldp + off + c];
                    else if (pos0 + t >= 0) x = a.conv[((size_t)slot * TAPS + (pos0 + t) % TAPS) * channels + rc + c];
                }
                hist[i][j] = x;
            }
        }
        float nx[NI];
        auto fetch = [&](int t) {
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = c0 + lane + 32 * i;
                nx[i] = c < d && t < te ? a.proj[(size_t)(sl * a.ts + t) * a.ldp + off + c] : 0.f;
            }
        };
        fetch(tb);
        for (int t = tb; t < te; ++t) {
            float v[NI];
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) hist[i][j] = hist[i][j + 1];
                hist[i][TAPS - 1] = nx[i];
            }
            fetch(t + 1);
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                float acc = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[i][j], hist[i][j], acc);
                v[i] = t < n && c0 + lane + 32 * i < d ? __fdividef(acc, 1.0f + __expf(-acc)) : 0.f;
                s = fmaf(v[i], v[i], s);
            }
            float r = 1.f;
            if (!is_v) {
                r = __frcp_rn(__fsqrt_rn(warp_total(s) + a.unit_eps));
                if (!is_k) r = __fdiv_rn(r, __fsqrt_rn((float)a.dk));
            }
            float* out = a.qkv + (size_t)(sl * a.ts + t) * a.ldqkv + oo;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = c0 + lane + 32 * i;
                if (c < dpad) out[c] = v[i] * r;
            }
        }
    }
}

constexpr int SA = CH + 4;
__host__ __device__ constexpr int chunk_sk(int dk16) { return dk16 + 4; }
__host__ __device__ constexpr int chunk_ss(int dvb) { return dvb + 8; }
static size_t chunk_smem(int dk16, int dvb) {
    return sizeof(float) * (2 * (size_t)CH * chunk_sk(dk16) + (size_t)(dk16 + CH) * chunk_ss(dvb) + 2 * (size_t)CH * SA + 5 * CH);
}

// CTA = (head, block of value columns, sequence).  A pair of warps owns 8 NTW columns of the state and of O from start to end,
// each of the two half of the rows; the triangular solve, sequential in the rows, goes by columns alone.
template <int NTW>
__global__ void __launch_bounds__(512) delta_chunk_kernel(DeltaArgs a, int dk4, int dk16) {
    extern __shared__ __align__(16) float sm[];
    const int nthr = blockDim.x, nw = nthr >> 5, dvb = nw * 4 * NTW;
    const int SK = chunk_sk(dk16), SS = chunk_ss(dvb);
    float* Ks = sm;                                       // [CH][SK]
    float* Qs = Ks + CH * SK;
    float* Ss = Qs + CH * SK;                             // [dk16][SS]
    float* Us = Ss + dk16 * SS;                           // [CH][SS]: V, then the right-hand sides, then U
    float* As = Us + CH * SS;                             // [CH][SA]: A below the diagonal blocks, their inverses on it
    float* Ps = As + CH * SA;
    float* Gh = Ps + CH * SA;                             // G as two floats, e^G, e^(G_C - G), beta
    float* Gl = Gh + CH;
    float* eG = Gl + CH;
    float* eE = eG + CH;
    float* be = eE + CH;
    const int h = blockIdx.x, sl = blockIdx.z, slot = a.b0 + sl, v0 = blockIdx.y * dvb;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int kvh = h / (a.H / a.G);
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    if (n == 0) return;
    float* Sg = a.S + ((size_t)slot * a.H + h) * a.dk * a.dvp;
    for (int i = tid; i < dk16 * dvb; i += nthr) {
        const int r = i / dvb, c = i % dvb;
        Ss[r * SS + c] = r < a.dk && v0 + c < a.dvp ? Sg[(size_t)r * a.dvp + v0 + c] : 0.f;
    }
    const int n0 = (warp >> 1) * 8 * NTW, half = warp & 1;      // this warp's columns of the block, and its half of the rows
    const int q4 = dk16 >> 2, d4 = dvb >> 2;
    for (int t0 = 0; t0 < n; t0 += CH) {
        const int nt = min(CH, n - t0);
        const float* base = a.qkv + (size_t)(sl * a.ts + t0) * a.ldqkv;
        __syncthreads();                                  // everything of the chunk before has been read
        for (int i = tid; i < CH * q4; i += nthr) {
            const int r = i / q4, c = 4 * (i % q4);
            const bool ok = r < nt && c < dk4;
            const float* src = base + (size_t)(ok ? r : 0) * a.ldqkv + kvh * dk4 + (ok ? c : 0);
            cp16(Qs + r * SK + c, src, ok);
            cp16(Ks + r * SK + c, src + a.G * dk4, ok);
        }
        for (int i = tid; i < CH * d4; i += nthr) {
            const int r = i / d4, c = 4 * (i % d4);
            const bool ok = r < nt && v0 + c < a.dvp;
            cp16(Us + r * SS + c, base + (size_t)(ok ? r : 0) * a.ldqkv + 2 * a.G * dk4 + h * a.dvp + (ok ? v0 + c : 0), ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (warp == 0) {
            // running sum of log g in double (differences of large sums matter), kept as two floats per token
            double l[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = 2 * lane + e;
                float2 bg = make_float2(0.f, 0.f);
                if (t < nt) bg = reinterpret_cast<const float2*>(a.gates)[(size_t)(sl * a.ts + t0 + t) * a.H + h];
                be[t] = bg.x;
                l[e] = (double)bg.y;
            }
            double s = l[0] + l[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double y = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += y;
            }
            const double tot = __shfl_sync(0xffffffffu, s, 31);
            const double gg[2] = {s - l[1], s};
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = 2 * lane + e;
                const float hi = (float)gg[e];
                Gh[t] = hi; Gl[t] = (float)(gg[e] - (double)hi);
                eG[t] = expf(hi); eE[t] = expf((float)(tot - gg[e]));
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // A and P by 16 x 16 blocks on and below the diagonal
        for (int u = warp; u < 10; u += nw) {
            const int rt = u < 1 ? 0 : (u < 3 ? 1 : (u < 6 ? 2 : 3)), ct = u - rt * (rt + 1) / 2;
            float ak[2][4] = {}, aq[2][4] = {};
            for (int ks = 0; ks < dk16; ks += 8) {
                const FragA fk = frag_a(Ks + rt * 16 * SK + ks, SK, g, tq), fq = frag_a(Qs + rt * 16 * SK + ks, SK, g, tq);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float* kp = Ks + (ct * 16 + e * 8 + g) * SK + ks;       // B[k][n] = K[n][k]
                    FragB fb;
                    fb.v[0] = split_tf32(kp[tq]); fb.v[1] = split_tf32(kp[tq + 4]);
                    mma3(ak[e], fk, fb);
                    mma3(aq[e], fq, fb);
                }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int t = rt * 16 + g + (i >> 1) * 8, s = ct * 16 + e * 8 + 2 * tq + (i & 1);
                    const float f = s <= t ? expf((Gh[t] - Gh[s]) + (Gl[t] - Gl[s])) : 0.f;
                    As[t * SA + s] = s < t ? be[t] * f * ak[e][i] : 0.f;
                    Ps[t * SA + s] = f * aq[e][i];
                }
        }
        // K S_0 and Q S_0 for this warp's columns
        float rk[2][NTW][4], ro[2][NTW][4];
#pragma unroll
        for (int r2 = 0; r2 < 2; ++r2)
#pragma unroll
            for (int e = 0; e < NTW; ++e)
#pragma unroll
                for (int i = 0; i < 4; ++i) rk[r2][e][i] = ro[r2][e][i] = 0.f;
        for (int ks = 0; ks < dk16; ks += 8) {
            FragB fb[NTW];
#pragma unroll
            for (int e = 0; e < NTW; ++e) fb[e] = frag_b(Ss + ks * SS + n0 + 8 * e, SS, g, tq);
#pragma unroll
            for (int r2 = 0; r2 < 2; ++r2) {
                const int rt = half + 2 * r2;             // row tiles of 16: the read-out below grows with the row, so they alternate
                const FragA fk = frag_a(Ks + rt * 16 * SK + ks, SK, g, tq);
#pragma unroll
                for (int e = 0; e < NTW; ++e) mma3(rk[r2][e], fk, fb[e]);
                const FragA fq = frag_a(Qs + rt * 16 * SK + ks, SK, g, tq);
#pragma unroll
                for (int e = 0; e < NTW; ++e) mma3(ro[r2][e], fq, fb[e]);
            }
        }
#pragma unroll
        for (int r2 = 0; r2 < 2; ++r2)
#pragma unroll
            for (int e = 0; e < NTW; ++e)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int rt = half + 2 * r2, t = rt * 16 + g + (i >> 1) * 8, c = n0 + 8 * e + 2 * tq + (i & 1);
                    Us[t * SS + c] = be[t] * (Us[t * SS + c] - eG[t] * rk[r2][e][i]);
                    ro[r2][e][i] *= eG[t];
                }
        __syncthreads();                                  // A and P are complete
        if (warp < 4) {
            // inverse of the diagonal block I + A_ww: lane j < 16 solves for column j, row after row
            float* D = As + warp * 16 * SA + warp * 16;
            float x[16];
            const int j = lane & 15;
#pragma unroll
            for (int r = 0; r < 16; ++r) {
                float v = r == j ? 1.f : 0.f;
#pragma unroll
                for (int s = 0; s < r; ++s) v = fmaf(-D[r * SA + s], x[s], v);
                x[r] = v;
            }
            __syncwarp();
            if (lane < 16) {
#pragma unroll
                for (int r = 0; r < 16; ++r) D[r * SA + j] = x[r];
            }
        }
        __syncthreads();
        // forward substitution by blocks of 16 rows, eight columns per warp
        if (warp * 8 < dvb) {
            float* Uw = Us + warp * 8;
#pragma unroll
            for (int i4 = 0; i4 < 4; ++i4) {
                float acc[2][4] = {};                     // two chains of products
#pragma unroll
                for (int kk = 0; kk < 2 * i4; ++kk)
                    mma3(acc[kk & 1], frag_a(As + i4 * 16 * SA + kk * 8, SA, g, tq), frag_b(Uw + kk * 8 * SS, SS, g, tq));
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    Uw[(i4 * 16 + g + (i >> 1) * 8) * SS + 2 * tq + (i & 1)] -= acc[0][i] + acc[1][i];
                    acc[0][i] = acc[1][i] = 0.f;
                }
                __syncwarp();
#pragma unroll
                for (int kk = 0; kk < 2; ++kk)
                    mma3(acc[kk], frag_a(As + i4 * 16 * SA + i4 * 16 + kk * 8, SA, g, tq), frag_b(Uw + (i4 * 16 + kk * 8) * SS, SS, g, tq));
                __syncwarp();
#pragma unroll
                for (int i = 0; i < 4; ++i) Uw[(i4 * 16 + g + (i >> 1) * 8) * SS + 2 * tq + (i & 1)] = acc[0][i] + acc[1][i];
                __syncwarp();
            }
        }
        __syncthreads();
        // read-out
#pragma unroll
        for (int r2 = 0; r2 < 2; ++r2) {
            const int rt = half + 2 * r2;
            for (int kk = 0; kk < 2 * rt + 2; ++kk) {
                const FragA fa = frag_a(Ps + rt * 16 * SA + kk * 8, SA, g, tq);
#pragma unroll
                for (int e = 0; e < NTW; ++e) mma3(ro[r2][e], fa, frag_b(Us + kk * 8 * SS + n0 + 8 * e, SS, g, tq));
            }
#pragma unroll
            for (int e = 0; e < NTW; ++e)
#pragma unroll
                for (int i = 0; i < 4; i += 2) {
                    const int t = rt * 16 + g + (i >> 1) * 8, c = v0 + n0 + 8 * e + 2 * tq;
                    if (t < nt && c < a.dvp)
                        *reinterpret_cast<float2*>(a.o32 + ((size_t)(sl * a.ts + t0 + t) * a.H + h) * a.dvp + c) = make_float2(ro[r2][e][i], ro[r2][e][i + 1]);
                }
        }
        // state: e^(G_C) S + K^T diag(e^(G_C - G)) U, 64 rows of the state at a time
        const float dec = eG[CH - 1];
        for (int mb = 0; mb < dk16; mb += 64) {
            float acc[2][NTW][4] = {};
            for (int kk = 0; kk < 8; ++kk) {
                FragB fb[NTW];
                const float e0 = eE[kk * 8 + tq], e1 = eE[kk * 8 + tq + 4];
#pragma unroll
                for (int e = 0; e < NTW; ++e) {
                    const float* up = Us + kk * 8 * SS + n0 + 8 * e + g;
                    fb[e].v[0] = split_tf32(up[tq * SS] * e0); fb[e].v[1] = split_tf32(up[(tq + 4) * SS] * e1);
                }
#pragma unroll
                for (int m2 = 0; m2 < 2; ++m2) {
                    const int mt = half + 2 * m2;
                    if (mb + mt * 16 < dk16) {
                        const float* kp = Ks + kk * 8 * SK + mb + mt * 16 + g;        // A[m][k] = K[k][m]
                        FragA fa;
                        fa.v[0] = split_tf32(kp[tq * SK]); fa.v[1] = split_tf32(kp[tq * SK + 8]);
                        fa.v[2] = split_tf32(kp[(tq + 4) * SK]); fa.v[3] = split_tf32(kp[(tq + 4) * SK + 8]);
#pragma unroll
                        for (int e = 0; e < NTW; ++e) mma3(acc[m2][e], fa, fb[e]);
                    }
                }
            }
#pragma unroll
            for (int m2 = 0; m2 < 2; ++m2) {
                const int mt = half + 2 * m2;
                if (mb + mt * 16 < dk16)
#pragma unroll
                    for (int e = 0; e < NTW; ++e)
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            float* sp = Ss + (mb + mt * 16 + g + (i >> 1) * 8) * SS + n0 + 8 * e + 2 * tq + (i & 1);
                            *sp = fmaf(dec, *sp, acc[m2][e][i]);
                        }
            }
        }
    }
    __syncthreads();
    for (int i = tid; i < dk16 * dvb; i += nthr) {
        const int r = i / dvb, c = i % dvb;
        if (r < a.dk && v0 + c < a.dvp) Sg[(size_t)r * a.dvp + v0 + c] = Ss[r * SS + c];
    }
}

constexpr size_t kSmemMax = 227 * 1024 - 1024;

size_t step_smem(const DeltaArgs& a, int cwl, int nt, bool staged) {
    const int share = (1 << cwl) < 32 ? 32 : (1 << cwl);
    return sizeof(float) * (2 * (size_t)a.dk + 3 * (size_t)a.dvp + 2 * (size_t)(nt / share) * a.dvp + 8 + (staged ? (size_t)a.dk * a.dvp : 0));
}

template <int NT, bool STAGED>
cudaError_t step_launch(const DeltaArgs& a, int cwl, cudaStream_t st) {
    const size_t smem = step_smem(a, cwl, NT, STAGED);
    if (smem > kSmemMax) return cudaErrorInvalidValue;
    auto kern = delta_step_kernel<NT, STAGED>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H, a.nseq);
    cfg.blockDim = dim3(NT);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = launch_pdl_on() ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, a, cwl);
}

cudaError_t launch_tail(const DeltaArgs& a, cudaStream_t st) {
    conv_tail_kernel<<<dim3((2 * a.G * a.dk + a.H * a.dv + 255) / 256, a.nseq), 256, 0, st>>>(a);
    return cudaGetLastError();
}

// columns per CTA (nw warp pairs of 8 ntw each): as many as the value dimension has and shared memory takes, fewer where the
// heads of the batch alone would leave SMs idle; false if not even 32 fit
bool chunk_shape(int dk, int dv, long heads, int* nw, int* ntw) {
    if (dk > kMaxChunkDim) return false;
    const int dk16 = (dk + 15) / 16 * 16;
    const int cand[3][2] = {{8, 2}, {4, 2}, {4, 1}};      // 128, 64, 32 columns
    for (int i = 0; i < 3; ++i) {
        const int dvb = cand[i][0] * cand[i][1] * 8;
        if (i < 2 && dv <= dvb / 2) continue;             // half of the columns would be empty
        if (chunk_smem(dk16, dvb) > kSmemMax) continue;
        if (i < 2 && heads * ((dv + dvb - 1) / dvb) <= 74) continue;
        *nw = cand[i][0]; *ntw = cand[i][1];
        return true;
    }
    return false;
}

}  // namespace

cudaError_t launch_delta_step(const DeltaArgs& a, cudaStream_t st, int* launches) {
    int cwl = 0;
    while ((4 << cwl) < a.dvp) ++cwl;
    const int CW = 1 << cwl;
    *launches = 1;
    cudaError_t e;
    if (CW > 256) return cudaErrorInvalidValue;
    const bool small = (size_t)a.dk * a.dvp <= 4096 && CW <= 128;
    if (step_smem(a, cwl, 256, true) > kSmemMax) e = step_launch<256, false>(a, cwl, st);
    else if (small) e = step_launch<128, true>(a, cwl, st);
    else e = step_launch<256, true>(a, cwl, st);
    if (e != cudaSuccess) return e;
    if (a.ts > 1) { *launches = 2; e = launch_tail(a, st); }
    return e;
}

bool delta_chunk_supported(int dk, int dv) {
    int nw, ntw;
    return chunk_shape(dk, dv, 1 << 20, &nw, &ntw) || chunk_shape(dk, dv, 1, &nw, &ntw);
}

cudaError_t launch_delta_chunk(const DeltaArgs& a, cudaStream_t st, int* launches) {
    int nw = 0, ntw = 0;
    if (!chunk_shape(a.dk, a.dv, (long)a.nseq * a.H, &nw, &ntw)) return cudaErrorInvalidValue;
    const int dk4 = (a.dk + 3) / 4 * 4, dk16 = (a.dk + 15) / 16 * 16, dvb = nw * ntw * 8;
    const size_t smem = chunk_smem(dk16, dvb);
    const int bps = (a.ts + kPrepRows - 1) / kPrepRows;
    const unsigned pg = (unsigned)(((long)a.nseq * bps * (2 * a.G + a.H + 1) + 7) / 8);
    bool prepared = false;
#define LUMI_PREP(T_, NI_) \
    if (!prepared && a.taps == T_ && a.dk <= 32 * NI_) { delta_prep_rows_kernel<T_, NI_><<<pg, 256, 0, st>>>(a, dk4, bps); prepared = true; }
    LUMI_PREP(2, 1) LUMI_PREP(2, 2) LUMI_PREP(2, 4) LUMI_PREP(2, 8)
    LUMI_PREP(3, 1) LUMI_PREP(3, 2) LUMI_PREP(3, 4) LUMI_PREP(3, 8)
    LUMI_PREP(4, 1) LUMI_PREP(4, 2) LUMI_PREP(4, 4) LUMI_PREP(4, 8)
#undef LUMI_PREP
    if (!prepared) {                                      // other filter lengths
        const long pw = (long)a.nseq * a.ts * (2 * a.G + a.H + 1);
        delta_prep_kernel<<<(unsigned)((pw + 7) / 8), 256, 0, st>>>(a, dk4);
    }
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const dim3 grid(a.H, (a.dv + dvb - 1) / dvb, a.nseq);
    if (ntw == 2) {
        e = cudaFuncSetAttribute(delta_chunk_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        delta_chunk_kernel<2><<<grid, nw * 64, smem, st>>>(a, dk4, dk16);
    } else {
        e = cudaFuncSetAttribute(delta_chunk_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        delta_chunk_kernel<1><<<grid, nw * 64, smem, st>>>(a, dk4, dk16);
    }
    if ((e = cudaGetLastError()) != cudaSuccess) return e;
    const HeadGateArgs hg{a.o32, a.H, a.dv, a.dvp, a.proj + a.off_g, a.ldp, a.o_norm, a.eps, a.row_len, a.t_abs0, a.ctl, a.nseq, a.ts, a.b0, a.y32, a.yhi, a.ylo, a.ldy};
    if ((e = launch_head_gate(hg, st)) != cudaSuccess) return e;
    *launches = 4;
    return launch_tail(a, st);
}

}  // namespace lumi
