// Retention: linear attention with a fixed decay per head and no softmax.
//
//   S_t = d S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t        (q, k rotated; k times k_scale)
//
// o over its root mean square, head by head, times silu of the gate rows.  Two forms of the recurrence:
//
//   retention_step_kernel    token after token, the head's state in registers (few heads), or in shared memory in parts that are
//                            loaded, worked on and stored one behind the other: decode steps (rotation, state, read-out, norm and
//                            gate in one launch), prompts of fp32 models, short slices.
//   retention_chunk_kernel   prompt slices in chunks of 64 tokens on the tensor cores.  With S_0 the state ahead of the chunk,
//                            o_t = d^(t+1) S_0^T q_t + sum_{s <= t} d^(t-s) (q_t.k_s) v_s, and the state becomes
//                            d^C S_0 + sum_s d^(C-1-s) k_s v_s^T.  Products take fp32 operands as two tf32 terms each.
//                            Few heads: a sequence's slice is cut into segments that run side by side; first every segment's own
//                            contribution to the state, then (retention_join_kernel) the state ahead of each, then the outputs.
#include "rows.cuh"
#include "tf32.cuh"

namespace lumi {
namespace {

// Element c of a rotated vector (rotate-half layout; cs: this pair's cos and sin), the vector itself in global memory.
__device__ __forceinline__ float rotated(const float* x, int c, const RotSpec& rot, const double* freq, int pos) {
    if (c >= rot.dims) return x[c];
    int i, o;
    bool second;
    if (rot.pairs) { i = c >> 1; o = c ^ 1; second = c & 1; }
    else { const int hd = rot.dims / 2; second = c >= hd; i = second ? c - hd : c; o = second ? c - hd : c + hd; }
    const float2 cs = rot_cos_sin(pos, freq[i]);
    const float a = x[c], b = x[o];
    return second ? fmaf(a, cs.x, b * cs.y) : fmaf(a, cs.x, -b * cs.y);
}

__device__ __forceinline__ uint32_t smem_of(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
constexpr uint64_t kStateWaitNs = 500000000ull;           // limit of the wait for a part of a head's state
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

// CTA = (head, sequence).  Thread (rg, cg) holds rows rg, rg + RG, ... (VPT of them at most) of four neighbouring columns.
// VPT = 0: the state stays in global memory (heads beyond shared memory).  VPT = -1: the state lies in shared memory, in kParts parts of
// `pr` rows (a multiple of RG) that bulk copies bring and take back: while one part is worked on, the others are on their way.
constexpr int kParts = 4;
template <int NT, int VPT>
__global__ void __launch_bounds__(NT) retention_step_kernel(RetentionArgs a, int cwl, int part_rows) {
    extern __shared__ __align__(128) float dyn[];
    __shared__ __align__(8) uint64_t bars[kParts];
    float* sm = dyn + (VPT < 0 ? (size_t)a.dk * a.dvp : 0);
    const int h = blockIdx.x, sl = blockIdx.y, slot = a.b0 + sl, tid = threadIdx.x, lane = tid & 31;
    const int dk = a.dk, dv = a.dv, dvp = a.dvp, c4n = dvp >> 2;
    const int CW = 1 << cwl, cg = tid & (CW - 1), rg = tid >> cwl, RG = NT >> cwl;
    const bool act = cg < c4n;
    const int share = CW < 32 ? 32 : CW, slots = NT / share;
    float* qs = sm;                                       // [dk]
    const int dk4 = (dk + 3) & ~3;
    float* ks = qs + dk4;                                 // [dk]
    float* vs = ks + dk4;                                 // [dvp]
    float* os = vs + dvp;                                 // [dvp]
    float* part = os + dvp;                               // [slots][dvp]
    float4* S = reinterpret_cast<float4*>(a.S + ((size_t)slot * a.H + h) * dk * dvp);
    const float d = a.decay_pow[(size_t)h * kDecayPowers + 1];
    auto part_of = [&](int p, int& r0, int& n) { r0 = p * part_rows; n = max(0, min(part_rows, dk - r0)); };
    auto request = [&]() {                                // thread 0
        for (int p = 0; p < kParts; ++p) asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_of(&bars[p])));
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        for (int p = 0; p < kParts; ++p) {
            int r0, n;
            part_of(p, r0, n);
            if (n == 0) break;
            const uint32_t bytes = (uint32_t)n * dvp * 4u;
            asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_of(&bars[p])), "r"(bytes) : "memory");
            asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                         ::"r"(smem_of(dyn + (size_t)r0 * dvp)), "l"(S + (size_t)r0 * c4n), "r"(bytes), "r"(smem_of(&bars[p])) : "memory");
        }
    };
    pdl_release();
    // the state belongs to the step before this one, which has ended: read ahead of the predecessor's results
    if (VPT < 0 && a.row_len == nullptr && tid == 0) request();
    float4 s[VPT > 0 ? VPT : 1];
    if constexpr (VPT > 0) {
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int r = rg + i * RG;
            s[i] = act && r < dk ? S[(size_t)r * c4n + cg] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    const int pos0 = a.pos[slot];
    pdl_sync();
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    if (n == 0 && a.ts == 1) return;                      // (with VPT < 0 nothing has been requested then)
    if (VPT < 0 && a.row_len != nullptr && n > 0 && tid == 0) request();
    for (int t = 0; t < n; ++t) {
        const int row = sl * a.ts + t;
        const float* pr = a.proj + (size_t)row * a.ldp;
        for (int c = tid; c < dk; c += NT) {
            qs[c] = rotated(pr + a.off_q + h * dk, c, a.rot, a.freq, pos0 + t);
            ks[c] = rotated(pr + a.off_k + h * dk, c, a.rot, a.freq, pos0 + t) * a.k_scale;
        }
        for (int c = tid; c < dvp; c += NT) vs[c] = c < dv ? pr[a.off_v + h * dv + c] : 0.f;
        __syncthreads();
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if constexpr (VPT < 0) {
            const float4 v = act ? make_float4(vs[4 * cg], vs[4 * cg + 1], vs[4 * cg + 2], vs[4 * cg + 3]) : make_float4(0.f, 0.f, 0.f, 0.f);
            float4* St = reinterpret_cast<float4*>(dyn);
            for (int p = 0; p < kParts; ++p) {
                int r0, cnt;
                part_of(p, r0, cnt);
                if (cnt == 0) break;
                if (t == 0 && __syncthreads_or(!state_wait(&bars[p]))) {
                    // report, and let what is still on its way land (again with a limit) before the memory goes away
                    if (tid == 0) {
                        if (a.status != nullptr) atomicOr(a.status, STATUS_TIMEOUT);
                        for (int q = p; q < kParts; ++q) { part_of(q, r0, cnt); if (cnt > 0) state_wait(&bars[q]); }
                        asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
                    }
                    __syncthreads();
                    return;
                }
                if (act) {
#pragma unroll 4
                    for (int r = r0 + rg; r < r0 + cnt; r += RG) {
                        float4 x = St[(size_t)r * c4n + cg];
                        const float k = ks[r], q = qs[r];
                        x = make_float4(fmaf(k, v.x, d * x.x), fmaf(k, v.y, d * x.y), fmaf(k, v.z, d * x.z), fmaf(k, v.w, d * x.w));
                        o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w);
                        St[(size_t)r * c4n + cg] = x;
                    }
                }
                if (t + 1 == n) {                         // the part goes back
                    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
                    __syncthreads();
                    if (tid == 0) {
                        asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;"
                                     ::"l"(S + (size_t)r0 * c4n), "r"(smem_of(dyn + (size_t)r0 * dvp)), "r"((uint32_t)cnt * dvp * 4u) : "memory");
                        asm volatile("cp.async.bulk.commit_group;" ::: "memory");
                    }
                }
            }
        } else if (act) {
            const float4 v = make_float4(vs[4 * cg], vs[4 * cg + 1], vs[4 * cg + 2], vs[4 * cg + 3]);
            auto walk = [&](int r, float4& x) {
                const float k = ks[r], q = qs[r];
                x = make_float4(fmaf(k, v.x, d * x.x), fmaf(k, v.y, d * x.y), fmaf(k, v.z, d * x.z), fmaf(k, v.w, d * x.w));
                o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w);
            };
            if constexpr (VPT > 0) {
#pragma unroll
                for (int i = 0; i < VPT; ++i) if (rg + i * RG < dk) walk(rg + i * RG, s[i]);
            } else {
                for (int r = rg; r < dk; r += RG) {
                    float4 x = S[(size_t)r * c4n + cg];
                    walk(r, x);
                    S[(size_t)r * c4n + cg] = x;
                }
            }
        }
        for (int m = CW; m < 32; m <<= 1) {
            o.x += __shfl_xor_sync(0xffffffffu, o.x, m); o.y += __shfl_xor_sync(0xffffffffu, o.y, m);
            o.z += __shfl_xor_sync(0xffffffffu, o.z, m); o.w += __shfl_xor_sync(0xffffffffu, o.w, m);
        }
        if (act && (CW >= 32 || lane < CW)) *reinterpret_cast<float4*>(part + (tid / share) * dvp + 4 * cg) = o;
        __syncthreads();
        for (int c = tid; c < dvp; c += NT) {
            float v = 0.f;
            for (int p = 0; p < slots; ++p) v += part[p * dvp + c];
            os[c] = v;
        }
        __syncthreads();
        float ss = 0.f;
        for (int c = lane; c < dv; c += 32) ss = fmaf(os[c], os[c], ss);
        const float rs = __frcp_rn(__fsqrt_rn(__fdiv_rn(warp_total(ss), (float)dv) + a.eps));
        for (int c = tid; c < dv; c += NT)
            put_row(a.y32, a.yhi, a.ylo, (size_t)row * a.ldy + h * dv + c, os[c] * rs * silu_f(pr[a.off_g + h * dv + c]));
        // (the next token's first writes are to qs, ks, vs, whose readers are behind the barriers above)
    }
    for (int t = n; t < a.ts; ++t)                        // rows behind a shorter prompt: zero, so that what follows stays finite
        for (int c = tid; c < dv; c += NT) put_row(a.y32, a.yhi, a.ylo, (size_t)(sl * a.ts + t) * a.ldy + h * dv + c, 0.f);
    if constexpr (VPT > 0) {
        if (n > 0 && act) {
#pragma unroll
            for (int i = 0; i < VPT; ++i) {
                const int r = rg + i * RG;
                if (r < dk) S[(size_t)r * c4n + cg] = s[i];
            }
        }
    }
    // the memory of the CTA has been read; the writes themselves end with the kernel
    if (VPT < 0 && tid == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
}

// ---- chunks of 64 tokens -----------------------------------------------------------------------------------
constexpr int CH = 64;
constexpr int SA = CH + 4;
constexpr int kMaxChunkDim = 256;
__host__ __device__ constexpr int chunk_sk(int dk16) { return dk16 + 4; }
__host__ __device__ constexpr int chunk_ss(int dvb) { return dvb + 8; }
size_t chunk_smem(int dk16, int dvb) {
    return sizeof(float) * (2 * (size_t)CH * chunk_sk(dk16) + (size_t)(dk16 + CH) * chunk_ss(dvb) + (size_t)CH * SA + kDecayPowers + 3);
}

// Rows [0, nt) of `cols` elements from src (rows of ld) into dst (rows of ldd), everything else up to CH rows x padded columns zero.
__device__ __forceinline__ void stage_rows(float* dst, int ldd, const float* src, size_t ld, int nt, int cols, int padded, bool vec, int tid, int nthr) {
    if (vec) {
        const int q = padded >> 2;
        for (int i = tid; i < CH * q; i += nthr) {
            const int r = i / q, c = 4 * (i % q);
            const bool ok = r < nt && c < cols;
            cp16(dst + r * ldd + c, src + (ok ? (size_t)r * ld + c : 0), ok);
        }
    } else {
        for (int i = tid; i < CH * padded; i += nthr) {
            const int r = i / padded, c = i % padded;
            dst[r * ldd + c] = r < nt && c < cols ? src[(size_t)r * ld + c] : 0.f;
        }
    }
}

enum ChunkMode { CHUNK_ALL = 0, CHUNK_STATE, CHUNK_OUT };
// CTA = (head, block of value columns, sequence and segment of seg_tokens).  A pair of warps owns 8 NTW columns of the state and of O
// from start to end, each of the two half of the rows.  CHUNK_STATE: the segment's contribution to the state alone, into a.seg;
// CHUNK_OUT: outputs, from the state in a.seg.
template <int NTW, int MODE>
__global__ void __launch_bounds__(512) retention_chunk_kernel(RetentionArgs a, int dk16, int seg_tokens, int segs) {
    extern __shared__ __align__(16) float sm[];
    const int nthr = blockDim.x, nw = nthr >> 5, dvb = nw * 4 * NTW;
    const int SK = chunk_sk(dk16), SS = chunk_ss(dvb);
    float* Ks = sm;                                       // [CH][SK]
    float* Qs = Ks + CH * SK;
    float* Ss = Qs + CH * SK;                             // [dk16][SS]
    float* Vs = Ss + dk16 * SS;                           // [CH][SS]
    float* Ps = Vs + CH * SS;                             // [CH][SA]
    float* pw = Ps + CH * SA;                             // powers of the decay
    const int h = blockIdx.x, sl = MODE == CHUNK_ALL ? blockIdx.z : blockIdx.z / segs, seg = MODE == CHUNK_ALL ? 0 : blockIdx.z % segs;
    const int slot = a.b0 + sl, v0 = blockIdx.y * dvb;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    for (int i = tid; i < kDecayPowers; i += nthr) pw[i] = a.decay_pow[(size_t)h * kDecayPowers + i];
    pdl_release();
    pdl_sync();
    const int n = min(pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0), MODE == CHUNK_ALL ? a.ts : (seg + 1) * seg_tokens);
    const int t_first = seg * seg_tokens;
    if (n <= t_first && MODE != CHUNK_STATE) return;
    const int pos0 = a.pos[slot];
    float* Sg = (MODE == CHUNK_ALL ? a.S + ((size_t)slot * a.H + h) * a.dk * a.dvp : a.seg + ((size_t)blockIdx.z * a.H + h) * a.dk * a.dvp);
    for (int i = tid; i < dk16 * dvb; i += nthr) {
        const int r = i / dvb, c = i % dvb;
        Ss[r * SS + c] = MODE != CHUNK_STATE && r < a.dk && v0 + c < a.dvp ? Sg[(size_t)r * a.dvp + v0 + c] : 0.f;
    }
    const int n0 = (warp >> 1) * 8 * NTW, half = warp & 1;      // this warp's columns of the block, and its half of the rows
    const bool kvec = ((a.dk | a.ldp | a.off_q | a.off_k) & 3) == 0, vvec = ((a.dv | a.ldp | a.off_v) & 3) == 0;
    const int hd = a.rot.dims / 2;
    for (int t0 = t_first; t0 < n; t0 += CH) {
        const int nt = min(CH, n - t0);
        const float* base = a.proj + (size_t)(sl * a.ts + t0) * a.ldp;
        __syncthreads();                                  // everything of the chunk before has been read
        if (MODE != CHUNK_STATE) stage_rows(Qs, SK, base + a.off_q + h * a.dk, a.ldp, nt, a.dk, dk16, kvec, tid, nthr);
        stage_rows(Ks, SK, base + a.off_k + h * a.dk, a.ldp, nt, a.dk, dk16, kvec, tid, nthr);
        stage_rows(Vs, SS, base + a.off_v + h * a.dv + v0, a.ldp, nt, a.dv - v0, dvb, vvec, tid, nthr);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int i = tid; i < CH * hd; i += nthr) {       // rotation
            const int r = i / hd, p = i % hd, c0 = a.rot.pairs ? 2 * p : p, c1 = a.rot.pairs ? 2 * p + 1 : p + hd;
            const float2 cs = rot_cos_sin(pos0 + t0 + r, a.freq[p]);
            float* q = Qs + r * SK;
            float* k = Ks + r * SK;
            const float k0 = k[c0] * a.k_scale, k1 = k[c1] * a.k_scale;
            if (MODE != CHUNK_STATE) {
                const float q0 = q[c0], q1 = q[c1];
                q[c0] = fmaf(q0, cs.x, -q1 * cs.y); q[c1] = fmaf(q1, cs.x, q0 * cs.y);
            }
            k[c0] = fmaf(k0, cs.x, -k1 * cs.y); k[c1] = fmaf(k1, cs.x, k0 * cs.y);
        }
        const int rest = a.dk - a.rot.dims;
        for (int i = tid; i < CH * rest; i += nthr) Ks[i / rest * SK + a.rot.dims + i % rest] *= a.k_scale;
        __syncthreads();
        if constexpr (MODE != CHUNK_STATE) {
        // P by 16 x 16 blocks on and below the diagonal
        for (int u = warp; u < 10; u += nw) {
            const int rt = u < 1 ? 0 : (u < 3 ? 1 : (u < 6 ? 2 : 3)), ct = u - rt * (rt + 1) / 2;
            float aq[2][4] = {};
            for (int ks = 0; ks < dk16; ks += 8) {
                const FragA fq = frag_a(Qs + rt * 16 * SK + ks, SK, g, tq);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float* kp = Ks + (ct * 16 + e * 8 + g) * SK + ks;       // B[k][n] = K[n][k]
                    FragB fb;
                    fb.v[0] = split_tf32(kp[tq]); fb.v[1] = split_tf32(kp[tq + 4]);
                    mma3(aq[e], fq, fb);
                }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int t = rt * 16 + g + (i >> 1) * 8, s = ct * 16 + e * 8 + 2 * tq + (i & 1);
                    Ps[t * SA + s] = s <= t ? pw[t - s] * aq[e][i] : 0.f;
                }
        }
        // Q S_0 for this warp's columns
        float ro[2][NTW][4] = {};
        for (int ks = 0; ks < dk16; ks += 8) {
            FragB fb[NTW];
#pragma unroll
            for (int e = 0; e < NTW; ++e) fb[e] = frag_b(Ss + ks * SS + n0 + 8 * e, SS, g, tq);
#pragma unroll
            for (int r2 = 0; r2 < 2; ++r2) {
                const FragA fq = frag_a(Qs + (half + 2 * r2) * 16 * SK + ks, SK, g, tq);
#pragma unroll
                for (int e = 0; e < NTW; ++e) mma3(ro[r2][e], fq, fb[e]);
            }
        }
#pragma unroll
        for (int r2 = 0; r2 < 2; ++r2)
#pragma unroll
            for (int e = 0; e < NTW; ++e)
#pragma unroll
                for (int i = 0; i < 4; ++i) ro[r2][e][i] *= pw[(half + 2 * r2) * 16 + g + (i >> 1) * 8 + 1];
        __syncthreads();                                  // P is complete
#pragma unroll
        for (int r2 = 0; r2 < 2; ++r2) {
            const int rt = half + 2 * r2;                 // row tiles of 16: the sum grows with the row, so they alternate
            for (int kk = 0; kk < 2 * rt + 2; ++kk) {
                const FragA fa = frag_a(Ps + rt * 16 * SA + kk * 8, SA, g, tq);
#pragma unroll
                for (int e = 0; e < NTW; ++e) mma3(ro[r2][e], fa, frag_b(Vs + kk * 8 * SS + n0 + 8 * e, SS, g, tq));
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
        }
        if (MODE == CHUNK_OUT && t0 + CH >= n) break;     // nothing reads the state any more
        // state, 64 rows at a time
        const float dec = pw[nt];
        for (int mb = 0; mb < dk16; mb += 64) {
            float acc[2][NTW][4] = {};
            for (int kk = 0; kk < 8; ++kk) {
                FragB fb[NTW];
                const int s0 = kk * 8 + tq, s1 = s0 + 4;
                const float e0 = s0 < nt ? pw[nt - 1 - s0] : 0.f, e1 = s1 < nt ? pw[nt - 1 - s1] : 0.f;
#pragma unroll
                for (int e = 0; e < NTW; ++e) {
                    const float* up = Vs + kk * 8 * SS + n0 + 8 * e + g;
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
    if (MODE == CHUNK_OUT) return;
    __syncthreads();
    for (int i = tid; i < dk16 * dvb; i += nthr) {
        const int r = i / dvb, c = i % dvb;
        if (r < a.dk && v0 + c < a.dvp) Sg[(size_t)r * a.dvp + v0 + c] = Ss[r * SS + c];
    }
}

// a.seg: contributions of the segments -> the states ahead of them; the state itself moves to the end of the slice.  One thread per
// four neighbouring elements of a head's state.
__global__ void __launch_bounds__(256) retention_join_kernel(RetentionArgs a, int seg_tokens, int segs) {
    const int h = blockIdx.y, sl = blockIdx.z, slot = a.b0 + sl, i = blockIdx.x * 256 + threadIdx.x, n4 = a.dk * (a.dvp >> 2);
    const float* pw = a.decay_pow + (size_t)h * kDecayPowers;
    pdl_release();
    pdl_sync();
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    if (i >= n4 || n == 0) return;
    float4* S = reinterpret_cast<float4*>(a.S + ((size_t)slot * a.H + h) * a.dk * a.dvp) + i;
    float4 s = *S;
    for (int g = 0; g < segs; ++g) {
        const int len = max(0, min(seg_tokens, n - g * seg_tokens));
        if (len == 0) break;
        float4* L = reinterpret_cast<float4*>(a.seg + ((size_t)(sl * segs + g) * a.H + h) * a.dk * a.dvp) + i;
        const float4 l = *L;
        float f = pw[len % CH];                           // decay over the segment
        for (int c = len / CH; c > 0; --c) f *= pw[CH];
        *L = s;
        s = make_float4(fmaf(f, s.x, l.x), fmaf(f, s.y, l.y), fmaf(f, s.z, l.z), fmaf(f, s.w, l.w));
    }
    *S = s;
}

constexpr size_t kSmemMax = 227 * 1024 - 1024;

template <int NT, int VPT>
cudaError_t step_launch(const RetentionArgs& a, int cwl, cudaStream_t st) {
    const int share = (1 << cwl) < 32 ? 32 : (1 << cwl);
    const size_t smem = sizeof(float) * (2 * (size_t)((a.dk + 3) & ~3) + (2 + (size_t)(NT / share)) * a.dvp + (VPT < 0 ? (size_t)a.dk * a.dvp : 0));
    if (smem > kSmemMax) return cudaErrorInvalidValue;
    auto kern = retention_step_kernel<NT, VPT>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    const int RG = NT >> cwl, part_rows = ((a.dk + kParts - 1) / kParts + RG - 1) / RG * RG;
    return launch_rows(kern, dim3(a.H, a.nseq), NT, smem, st, a, cwl, part_rows);
}

// columns per CTA (nw warp pairs of 8 ntw each): as many as the value dimension has and shared memory takes, fewer where the heads
// of the batch alone would leave SMs idle; false if not even 32 fit
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

cudaError_t launch_retention_step(const RetentionArgs& a, cudaStream_t st, int* launches) {
    *launches = 1;
    int cwl = 0;
    while ((4 << cwl) < a.dvp) ++cwl;
    const int CW = 1 << cwl;
    if (CW > 256) return cudaErrorInvalidValue;
    // many heads: through shared memory, several CTAs per SM; few: straight into registers
    if ((long)a.nseq * a.H > 296 && CW <= 64 && (size_t)a.dk * a.dvp * 4 <= 100 * 1024) {
        if ((size_t)a.dk * a.dvp <= 4096 && CW <= 32) return step_launch<128, -1>(a, cwl, st);
        return step_launch<256, -1>(a, cwl, st);
    }
    auto per_thread = [&](int nt) { return nt >= CW ? (a.dk + nt / CW - 1) / (nt / CW) : 1 << 30; };
    if (per_thread(128) <= 4) return step_launch<128, 4>(a, cwl, st);
    if (per_thread(128) <= 8) return step_launch<128, 8>(a, cwl, st);
    if (per_thread(256) <= 8) return step_launch<256, 8>(a, cwl, st);
    if (per_thread(256) <= 16) return step_launch<256, 16>(a, cwl, st);
    if (per_thread(512) <= 16) return step_launch<512, 16>(a, cwl, st);
    return step_launch<256, 0>(a, cwl, st);
}

bool retention_chunk_supported(int dk, int dv) {
    int nw, ntw;
    return chunk_shape(dk, dv, 1 << 20, &nw, &ntw) || chunk_shape(dk, dv, 1, &nw, &ntw);
}

// Segments of a slice: as many as fill the SMs with CTAs of the widest column blocks; 1 where the heads alone do.
static int segments_of(int H, int dk, int dv, int nseq, int ts, int* nw, int* ntw, int* seg_tokens) {
    const int chunks = (ts + CH - 1) / CH;
    *seg_tokens = chunks * CH;
    if (!chunk_shape(dk, dv, 1 << 20, nw, ntw)) return 1;
    const int dvb = *nw * *ntw * 8, units = nseq * H * ((dv + dvb - 1) / dvb), want = units > 0 ? 148 / units : 1;
    if (want < 2 || chunks < 2) return 1;
    const int per = (chunks + want - 1) / want;
    *seg_tokens = per * CH;
    return (chunks + per - 1) / per;
}

size_t retention_segment_floats(const MixerSpec& m, int nseq, int ts) {
    int nw, ntw, st;
    const int segs = segments_of(m.heads, m.dim, m.vdim, nseq, ts, &nw, &ntw, &st);
    return segs > 1 ? (size_t)nseq * segs * m.heads * m.dim * ((m.vdim + 3) / 4 * 4) : 0;
}

template <int MODE>
static cudaError_t chunk_launch(const RetentionArgs& a, int nw, int ntw, int seg_tokens, int segs, cudaStream_t st) {
    const int dk16 = (a.dk + 15) / 16 * 16, dvb = nw * ntw * 8;
    const size_t smem = chunk_smem(dk16, dvb);
    const dim3 grid(a.H, (a.dv + dvb - 1) / dvb, (unsigned)(a.nseq * segs));
    auto kern = ntw == 2 ? retention_chunk_kernel<2, MODE> : retention_chunk_kernel<1, MODE>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    return launch_rows(kern, grid, nw * 64, smem, st, a, dk16, seg_tokens, segs);
}

cudaError_t launch_retention_chunk(const RetentionArgs& a, cudaStream_t st, int* launches) {
    int nw = 0, ntw = 0, seg_tokens = 0;
    const int segs = a.seg != nullptr ? segments_of(a.H, a.dk, a.dv, a.nseq, a.ts, &nw, &ntw, &seg_tokens) : 1;
    cudaError_t e;
    *launches = 2;
    if (segs > 1) {
        if ((e = chunk_launch<CHUNK_STATE>(a, nw, ntw, seg_tokens, segs, st)) != cudaSuccess) return e;
        e = launch_rows(retention_join_kernel, dim3((a.dk * (a.dvp / 4) + 255) / 256, a.H, a.nseq), 256, 0, st, a, seg_tokens, segs);
        if (e != cudaSuccess) return e;
        if ((e = chunk_launch<CHUNK_OUT>(a, nw, ntw, seg_tokens, segs, st)) != cudaSuccess) return e;
        *launches = 4;
    } else {
        if (!chunk_shape(a.dk, a.dv, (long)a.nseq * a.H, &nw, &ntw)) return cudaErrorInvalidValue;
        if ((e = chunk_launch<CHUNK_ALL>(a, nw, ntw, 0, 1, st)) != cudaSuccess) return e;
    }
    const HeadGateArgs hg{a.o32, a.H, a.dv, a.dvp, a.proj + a.off_g, a.ldp, nullptr, a.eps, a.row_len, a.t_abs0, a.ctl, a.nseq, a.ts, a.b0, a.y32, a.yhi, a.ylo, a.ldy};
    return launch_head_gate(hg, st);
}

}  // namespace lumi
