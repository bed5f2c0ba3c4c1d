// Attention over a cached latent: per token the cache holds the normalised latent c and one rotated key part shared by all heads.
// Keys and values of a head are linear in c, so a query can be taken into the latent space instead of expanding them:
//   q.k = (U_k^T q) . c + q_rot . k_rot,    sum_j p_j v_j = U_v (sum_j p_j c_j)
// and all heads attend to the same cache rows.
//
//   latent_prep_kernel   rotates the queries, writes the pass's cache rows, lays the query parts out for the products
//   latent_mma_kernel    bf16 cache: 16 heads of one row per CTA, scores and contexts by mma.sync (queries and weights as bf16 hi + lo);
//                        long contexts are split over CTAs and merged by the last arriver
// fp32 caches and rows beyond shared memory take the plain form of window_attention.cu over the same queries; long prompt slices
// expand keys and values per head and take its tensor-core form.
#include "rows.cuh"

#include <algorithm>
#include <cmath>

namespace lumi {
namespace {

constexpr float kNoScore = -1.0e30f;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kPad = 8;                                   // extra bf16 per staged row: no ldmatrix conflicts
constexpr int kSlices = 16;
constexpr int kSliceMin = 64;                            // tokens from which a slice of the context is worth a CTA

template <typename T> __device__ __forceinline__ T cache_elem(float v);
template <> __device__ __forceinline__ float cache_elem<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 cache_elem<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// One warp per (row, head) for the queries, and one per row for the cache.
template <typename KT>
__global__ void __launch_bounds__(256) latent_prep_kernel(LatentArgs a) {
    const int H = a.m.heads, D = a.m.dim, R = a.m.rot_dim, hr = R / 2;
    const LatentShape ls(a.m);
    const long w = ((long)blockIdx.x * 256 + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    pdl_release();
    pdl_sync();
    if (w >= (long)a.nseq * a.ts * (H + 1)) return;
    const int row = (int)(w / (H + 1)), h = (int)(w % (H + 1)), sl = row / a.ts, t = row % a.ts, slot = a.b0 + sl;
    const int pos = a.pos[slot] + t;
    float* pr = a.proj + (size_t)row * a.ldp;
    if (h < H) {
        float* q = pr + a.off_q + (size_t)h * ls.dk;
        float* ql = a.qlat != nullptr ? a.qlat + ((size_t)row * H + h) * ls.row + ls.lp : nullptr;
        for (int i = lane; i < hr; i += 32) {
            const float2 cs = rot_cos_sin(pos, a.freq[i]);
            const float u = q[D + 2 * i], v = q[D + 2 * i + 1];
            const float x = fmaf(u, cs.x, -v * cs.y), y = fmaf(v, cs.x, u * cs.y);
            q[D + 2 * i] = x;
            q[D + 2 * i + 1] = y;
            if (ql != nullptr) { ql[2 * i] = x; ql[2 * i + 1] = y; }
        }
        if (ql != nullptr) for (int c = R + lane; c < ls.row - ls.lp; c += 32) ql[c] = 0.f;
        if (a.qh != nullptr)
            for (int c = lane; c < ls.dp; c += 32) put_row(nullptr, a.qh, a.ql, ((size_t)row * H + h) * ls.dp + c, c < D ? q[c] : 0.f);
        return;
    }
    if (t >= pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0)) return;
    if (a.limit > 0 && pos >= a.limit) {
        if (lane == 0) atomicOr(&a.ctl->status, STATUS_KV_FULL);
        return;
    }
    const int rs = pos % (a.pages_per_seq * kPageTokens);
    KT* dst = reinterpret_cast<KT*>(a.kv) + ((size_t)a.page_table[(size_t)slot * a.pages_per_seq + rs / kPageTokens] * kPageTokens + rs % kPageTokens) * ls.row;
    const float* c = pr + a.off_c;
    const int K = a.m.kv_rank;
    float s = 0.f;
    for (int i = lane; i < K; i += 32) s = fmaf(c[i], c[i], s);
    const float f = __frcp_rn(__fsqrt_rn(__fdiv_rn(warp_total(s), (float)K) + a.eps));
    for (int i = lane; i < ls.lp; i += 32) dst[i] = cache_elem<KT>(i < K ? c[i] * f * a.c_norm[i] : 0.f);
    for (int i = lane; i < hr; i += 32) {
        const float2 cs = rot_cos_sin(pos, a.freq[i]);
        const float u = c[K + 2 * i], v = c[K + 2 * i + 1];
        dst[ls.lp + 2 * i] = cache_elem<KT>(fmaf(u, cs.x, -v * cs.y));
        dst[ls.lp + 2 * i + 1] = cache_elem<KT>(fmaf(v, cs.x, u * cs.y));
    }
    for (int i = ls.lp + R + lane; i < ls.row; i += 32) dst[i] = cache_elem<KT>(0.f);
}

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void halves2(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - f.x, v1 - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

constexpr int PS = kPageTokens + kPad;                    // row of the staged weights

// Grid: (row, block of 16 heads, context slice).  Eight warps: for the scores a pair of them takes 16 tokens of a staged page, each half
// of the key row; for the contexts each takes an eighth of the latent's columns.  NTW: 8-column tiles of a warp's eighth (an even
// number of them where it is more than one), at least.
constexpr int kThreads = 256;
template <int NTW>
__global__ void __launch_bounds__(kThreads) latent_mma_kernel(LatentArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float wmax[4][16], wsum[4][16];
    __shared__ float4 half_s[4][2][32];                   // scores over the second half of the key row
    __shared__ int is_last;
    const LatentShape ls(a.m);
    const int H = a.m.heads, RS = ls.row + kPad, stage_elems = kPageTokens * RS;
    __nv_bfloat16* stage = reinterpret_cast<__nv_bfloat16*>(smem_raw);        // [2][64][RS]
    __nv_bfloat16* qh = stage + 2 * stage_elems;          // [16][RS]
    __nv_bfloat16* ql = qh + 16 * RS;
    __nv_bfloat16* ph = ql + 16 * RS;                     // [16][PS]
    __nv_bfloat16* pl = ph + 16 * PS;
    const int row = blockIdx.x, h0 = blockIdx.y * 16, nh = min(16, H - h0), split = blockIdx.z, nsplit = gridDim.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int sl = row / a.ts, t = row % a.ts, slot = a.b0 + sl;
    pdl_release();
    pdl_sync();
    const int pos = a.pos[slot] + t;
    const bool live = t < pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    auto put = [&](int m, int d, float v) { put_row(a.ctx, a.ch, a.cl, ((size_t)row * H + h0 + m) * ls.lp + d, v); };
    if (!live || (a.limit > 0 && pos >= a.limit)) {
        if (split == 0 && (a.ts > 1 || live)) for (int i = tid; i < nh * ls.lp; i += kThreads) put(i / ls.lp, i % ls.lp, 0.f);
        return;
    }
    const int32_t* pt = a.page_table + (size_t)slot * a.pages_per_seq;
    const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(a.kv);
    const int lo = a.m.window > 0 ? max(0, pos - a.m.window + 1) : 0;
    const int pg0 = lo / kPageTokens, pages = pos / kPageTokens - pg0 + 1;
    const int per = (pages + nsplit - 1) / nsplit, pb = pg0 + split * per, pe = min(pg0 + pages, pb + per);
    const int rc = ls.row / 8;                            // 16-byte chunks per row
    auto issue = [&](int pg) {
        __nv_bfloat16* s = stage + ((pg - pb) & 1) * stage_elems;
        const __nv_bfloat16* src = pool + (size_t)pt[pg % a.pages_per_seq] * kPageTokens * ls.row;
        for (int i = tid; i < kPageTokens * rc; i += kThreads) {
            const int r = i / rc, c = i - r * rc, p = pg * kPageTokens + r;
            const int bytes = p >= lo && p <= pos ? 16 : 0;           // 0: filled with zeros
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(s + r * RS + c * 8)), "l"(src + (size_t)i * 8), "r"(bytes) : "memory");
        }
    };
    if (pb < pe) issue(pb);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int i = tid; i < 16 * (ls.row / 2); i += kThreads) {
        const int m = i / (ls.row / 2), c = 2 * (i % (ls.row / 2));
        float2 v = make_float2(0.f, 0.f);
        if (m < nh) v = *reinterpret_cast<const float2*>(a.qlat + ((size_t)row * H + h0 + m) * ls.row + c);
        uint32_t hi, low;
        halves2(v.x, v.y, hi, low);
        *reinterpret_cast<uint32_t*>(qh + m * RS + c) = hi;
        *reinterpret_cast<uint32_t*>(ql + m * RS + c) = low;
    }
    const float sc2 = a.m.scale * kLog2e;                 // scores in units of log 2
    float mx[2] = {kNoScore, kNoScore}, lsum[2] = {0.f, 0.f};
    float o[NTW][4];
#pragma unroll
    for (int i = 0; i < NTW; ++i) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    const int nks = ls.row / 16, ntw = ls.lp / 64, col0 = warp * (ls.lp / 8), tg = warp & 3, kh = warp >> 2;
    for (int pg = pb; pg < pe; ++pg) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                  // the page is here, and every warp has finished with the other stage
        if (pg + 1 < pe) issue(pg + 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const __nv_bfloat16* s = stage + ((pg - pb) & 1) * stage_elems;
        float sc[2][4] = {}, sl2[2][4] = {};              // products with the query's two halves
#pragma unroll 4
        for (int k = kh * (nks / 2); k < (kh + 1) * (nks / 2); ++k) {      // (nks is a multiple of 4)
            uint32_t fh[4], fl[4], kb[4];
            const int qo = (lane & 15) * RS + k * 16 + (lane >> 4) * 8;
            ldm4(fh, qh + qo);
            ldm4(fl, ql + qo);
            ldm4(kb, s + (tg * 16 + ((lane >> 4) << 3) + (lane & 7)) * RS + k * 16 + ((lane >> 3) & 1) * 8);
            mma_bf16(sc[0], fh, kb[0], kb[1]);
            mma_bf16(sc[1], fh, kb[2], kb[3]);
            mma_bf16(sl2[0], fl, kb[0], kb[1]);
            mma_bf16(sl2[1], fl, kb[2], kb[3]);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
#pragma unroll
            for (int i = 0; i < 4; ++i) sc[e][i] += sl2[e][i];
            if (kh == 1) half_s[tg][e][lane] = make_float4(sc[e][0], sc[e][1], sc[e][2], sc[e][3]);
        }
        __syncthreads();
        if (kh == 0) {
            float tm[2] = {kNoScore, kNoScore};
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float4 h = half_s[tg][e][lane];
                const float hv[4] = {h.x, h.y, h.z, h.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int p = pg * kPageTokens + tg * 16 + e * 8 + 2 * tq + (i & 1);
                    sc[e][i] = p >= lo && p <= pos ? (sc[e][i] + hv[i]) * sc2 : kNoScore;
                    tm[i >> 1] = fmaxf(tm[i >> 1], sc[e][i]);
                }
            }
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                tm[c] = fmaxf(tm[c], __shfl_xor_sync(0xffffffffu, tm[c], 1));
                tm[c] = fmaxf(tm[c], __shfl_xor_sync(0xffffffffu, tm[c], 2));
                if (tq == 0) wmax[tg][g + 8 * c] = tm[c];
            }
        }
        __syncthreads();
        float f[2];
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int m = g + 8 * c;
            const float mn = fmaxf(mx[c], fmaxf(fmaxf(wmax[0][m], wmax[1][m]), fmaxf(wmax[2][m], wmax[3][m])));   // a page of the context holds a visible token
            f[c] = ex2(mx[c] - mn);
            mx[c] = mn;
            lsum[c] *= f[c];
        }
        if (kh == 0) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float p[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { p[i] = ex2(sc[e][i] - mx[i >> 1]); lsum[i >> 1] += p[i]; }
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                uint32_t hi, low;
                halves2(p[2 * c], p[2 * c + 1], hi, low);
                const int at = (g + 8 * c) * PS + tg * 16 + e * 8 + 2 * tq;
                *reinterpret_cast<uint32_t*>(ph + at) = hi;
                *reinterpret_cast<uint32_t*>(pl + at) = low;
            }
        }
        }
#pragma unroll
        for (int i = 0; i < NTW; ++i) { o[i][0] *= f[0]; o[i][1] *= f[0]; o[i][2] *= f[1]; o[i][3] *= f[1]; }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kPageTokens / 16; ++k) {
            uint32_t fh[4], fl[4];
            const int po = (lane & 15) * PS + k * 16 + (lane >> 4) * 8;
            ldm4(fh, ph + po);
            ldm4(fl, pl + po);
            const __nv_bfloat16* v = s + (k * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * RS + col0 + (lane >> 4) * 8;
#pragma unroll
            for (int dn = 0; dn < (NTW + 1) / 2; ++dn) {
                if constexpr (NTW == 1) {                 // eight columns
                    uint32_t v0, v1;
                    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];"
                                 : "=r"(v0), "=r"(v1) : "r"((uint32_t)__cvta_generic_to_shared(s + (k * 16 + (lane & 15)) * RS + col0)) : "memory");
                    mma_bf16(o[0], fh, v0, v1);
                    mma_bf16(o[0], fl, v0, v1);
                } else if (2 * dn < ntw) {
                    uint32_t vb[4];
                    ldm4t(vb, v + dn * 16);
                    mma_bf16(o[2 * dn], fh, vb[0], vb[1]);
                    mma_bf16(o[2 * dn + 1], fh, vb[2], vb[3]);
                    mma_bf16(o[2 * dn], fl, vb[0], vb[1]);
                    mma_bf16(o[2 * dn + 1], fl, vb[2], vb[3]);
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        lsum[c] += __shfl_xor_sync(0xffffffffu, lsum[c], 1);
        lsum[c] += __shfl_xor_sync(0xffffffffu, lsum[c], 2);
        if (kh == 0 && tq == 0) wsum[tg][g + 8 * c] = lsum[c];
    }
    __syncthreads();
    float l[2];
#pragma unroll
    for (int c = 0; c < 2; ++c) l[c] = (wsum[0][g + 8 * c] + wsum[1][g + 8 * c]) + (wsum[2][g + 8 * c] + wsum[3][g + 8 * c]);
    if (nsplit == 1) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int m = g + 8 * c;
            if (m >= nh) continue;
            const float inv = __frcp_rn(l[c]);
            const size_t oo = ((size_t)row * H + h0 + m) * ls.lp + col0 + 2 * tq;
#pragma unroll
            for (int i = 0; i < NTW; ++i) {
                if (i >= ntw) break;
                const float v0 = o[i][2 * c] * inv, v1 = o[i][2 * c + 1] * inv;
                if (a.ctx != nullptr) *reinterpret_cast<float2*>(a.ctx + oo + 8 * i) = make_float2(v0, v1);
                if (a.ch != nullptr) {
                    uint32_t hi, low;
                    halves2(v0, v1, hi, low);
                    *reinterpret_cast<uint32_t*>(a.ch + oo + 8 * i) = hi;
                    if (a.cl != nullptr) *reinterpret_cast<uint32_t*>(a.cl + oo + 8 * i) = low;
                }
            }
        }
        return;
    }
    // per slice: [16] maxima, [16] sums, [16][lp] contexts
    const size_t unit = (size_t)row * gridDim.y + blockIdx.y, pw = (size_t)16 * (ls.lp + 2);
    float* part = a.part + (unit * nsplit + split) * pw;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int m = g + 8 * c;
        if (warp == 0 && tq == 0) { part[m] = mx[c]; part[16 + m] = l[c]; }
#pragma unroll
        for (int i = 0; i < NTW; ++i)
            if (i < ntw) *reinterpret_cast<float2*>(part + 32 + (size_t)m * ls.lp + col0 + 8 * i + 2 * tq) = make_float2(o[i][2 * c], o[i][2 * c + 1]);
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        const int old = atomicAdd(a.part_count + unit, 1);
        is_last = old == nsplit - 1;
        if (is_last) a.part_count[unit] = 0;              // ready for the next launch
    }
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    // weights of the slices per head (an empty slice has maximum kNoScore and weighs nothing), then the contexts, all loads of an
    // element's slices in flight together
    const float* all = a.part + unit * nsplit * pw;
    float* wt = reinterpret_cast<float*>(smem_raw);       // [nsplit][16]
    if (tid < 16) {
        float top = kNoScore, mv[kSlices], sv[kSlices];
#pragma unroll
        for (int sp = 0; sp < kSlices; ++sp) {
            mv[sp] = sp < nsplit ? __ldcg(all + sp * pw + tid) : kNoScore;
            sv[sp] = sp < nsplit ? __ldcg(all + sp * pw + 16 + tid) : 0.f;
        }
#pragma unroll
        for (int sp = 0; sp < kSlices; ++sp) top = fmaxf(top, mv[sp]);
        float den = 0.f;
#pragma unroll
        for (int sp = 0; sp < kSlices; ++sp) { mv[sp] = exp2f(mv[sp] - top); den = fmaf(mv[sp], sv[sp], den); }
        const float inv = __frcp_rn(den);
#pragma unroll
        for (int sp = 0; sp < kSlices; ++sp) if (sp < nsplit) wt[sp * 16 + tid] = mv[sp] * inv;
    }
    __syncthreads();
    for (int i = 4 * tid; i < nh * ls.lp; i += 4 * kThreads) {
        const int m = i / ls.lp;
        float4 v[kSlices];
#pragma unroll
        for (int sp = 0; sp < kSlices; ++sp) v[sp] = sp < nsplit ? __ldcg(reinterpret_cast<const float4*>(all + sp * pw + 32 + i)) : make_float4(0.f, 0.f, 0.f, 0.f);
        float4 n = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int sp = 0; sp < kSlices; ++sp) {
            const float f = sp < nsplit ? wt[sp * 16 + m] : 0.f;
            n.x = fmaf(f, v[sp].x, n.x); n.y = fmaf(f, v[sp].y, n.y); n.z = fmaf(f, v[sp].z, n.z); n.w = fmaf(f, v[sp].w, n.w);
        }
        const int d = i % ls.lp;
        put(m, d, n.x); put(m, d + 1, n.y); put(m, d + 2, n.z); put(m, d + 3, n.w);
    }
}

constexpr size_t kSmemMax = 227 * 1024 - 1024;
size_t mma_smem(const LatentShape& ls) { return sizeof(__nv_bfloat16) * ((2 * kPageTokens + 32) * (size_t)(ls.row + kPad) + 32 * (size_t)PS); }

template <int NTW>
cudaError_t run_mma(const LatentArgs& a, cudaStream_t st) {
    const LatentShape ls(a.m);
    const int hb = (a.m.heads + 15) / 16;
    const long units = (long)a.nseq * a.ts * hb;
    int nsplit = 1;
    if (a.part != nullptr && units <= kAttnPartUnits) {
        const int ring = a.pages_per_seq * kPageTokens, ctx = a.m.window > 0 ? std::min(a.m.window, ring) : ring;
        nsplit = std::max(1, std::min({(int)((2L * 148 + units - 1) / units), (ctx + kSliceMin - 1) / kSliceMin, kSlices}));
    }
    const size_t smem = mma_smem(ls);
    auto kern = latent_mma_kernel<NTW>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    return launch_rows(kern, dim3((unsigned)(a.nseq * a.ts), hb, nsplit), kThreads, smem, st, a);
}

}  // namespace

// units * nsplit < 2 * 148 + units (nsplit is a ceiling), at most 2 * kAttnPartUnits parts
size_t latent_part_floats(const MixerSpec& m) { return 2 * (size_t)16 * (LatentShape(m).lp + 2); }

cudaError_t launch_latent_prep(const LatentArgs& a, cudaStream_t st) {
    const long warps = (long)a.nseq * a.ts * (a.m.heads + 1);
    const dim3 grid((unsigned)((warps + 7) / 8));
    return a.kv_is_f32 ? launch_rows(latent_prep_kernel<float>, grid, 256, 0, st, a) : launch_rows(latent_prep_kernel<__nv_bfloat16>, grid, 256, 0, st, a);
}

cudaError_t launch_latent_attention(const LatentArgs& a, cudaStream_t st) {
    const LatentShape ls(a.m);
    if (a.kv_is_f32 || mma_smem(ls) > kSmemMax || ls.lp > 640) {
        // the cache rows are keys of `row` elements, their first lp elements the values
        WinAttnArgs w{};
        w.proj = a.qlat; w.ldp = a.m.heads * ls.row; w.off_q = 0;
        w.kv = a.kv; w.kv_is_f32 = a.kv_is_f32; w.dk_pad = ls.row; w.dv_pad = ls.lp;
        w.page_table = a.page_table; w.pages_per_seq = a.pages_per_seq; w.pos = a.pos;
        w.H = a.m.heads; w.G = 1; w.dk = ls.row; w.dv = ls.lp;
        w.m = a.m; w.m.kv_heads = 1; w.m.dim = ls.row; w.m.vdim = ls.lp; w.m.qk_norm = false; w.m.sink = false;
        w.append = 0; w.eps = a.eps;
        w.row_len = a.row_len; w.t_abs0 = a.t_abs0; w.ctl = a.ctl;
        w.nseq = a.nseq; w.ts = a.ts; w.b0 = a.b0; w.limit = a.limit;
        w.y32 = a.ctx; w.yhi = a.ch; w.ylo = a.cl; w.ldy = a.m.heads * ls.lp;
        w.page_elems = (long)kPageTokens * ls.row; w.head_step = 0; w.k_ld = w.v_ld = ls.row; w.v_off = 0;
        w.plain = true;
        int n = 0;
        return launch_window_attention(w, st, &n);
    }
    switch (ls.lp / 64) {                                 // 8-column tiles per warp
        case 1: return run_mma<1>(a, st);
        case 2: return run_mma<2>(a, st);
        case 3: case 4: return run_mma<4>(a, st);
        case 5: case 6: return run_mma<6>(a, st);
        case 7: case 8: return run_mma<8>(a, st);
        default: return run_mma<10>(a, st);
    }
}

}  // namespace lumi
