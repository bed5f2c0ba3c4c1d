// Attention over a paged ring of keys and values with the constants of the design as parameters (MixerSpec): sliding window
// or everything, score factor, RMS norm of q and k without a weight, one extra score in the softmax that has no value (a
// sink), key and value heads of different sizes, and layers that read the cache of an earlier layer.
//
// Position p lives in ring slot p % (64 * pages_per_seq); the host gives the ring at least window + slice - 1 slots, so a
// pass can append all its rows before any of them attends.  Cache rows are padded with zeros to multiples of 16 elements.
//
//   win_append_kernel   the pass's keys (normalised) and values into the cache
//   win_mma_kernel      bf16 cache: scores and context by mma.sync, 16 query columns (rows x heads of a group) per warp.
//                       Prompt slices: every warp has query columns of its own and walks all staged tokens.  Decode: the
//                       warps share one set of columns and take 16 tokens of a page each; the new token's row is patched
//                       into the staged page, and long contexts are split over CTAs (merged by the last arriver).
//   win_simple_kernel   fp32 cache, or heads beyond 256 elements: one CTA per (row, head), plain fp32
#include "rows.cuh"

#include <algorithm>
#include <cmath>

namespace lumi {
namespace {

constexpr float kNoScore = -1.0e30f;                      // finite, so that a fully masked tile never produces inf - inf
constexpr int kPadRow = 8;                                // extra bf16 per staged row: an odd number of 16-byte chunks, no ldmatrix conflicts
constexpr float kLog2e = 1.4426950408889634f;

struct WinShape {
    int ring, hpk, head_step, k_ld, v_ld, v_off;          // as in WinAttnArgs
    size_t page_elems;
};
__host__ __device__ inline WinShape shape_of(const WinAttnArgs& a) {
    WinShape s;
    s.ring = a.pages_per_seq * kPageTokens;
    s.hpk = a.H / a.G;
    if (a.page_elems > 0) {
        s.head_step = a.head_step; s.k_ld = a.k_ld; s.v_ld = a.v_ld; s.v_off = a.v_off;
        s.page_elems = (size_t)a.page_elems;
    } else {
        s.head_step = kPageTokens * (a.dk_pad + a.dv_pad);
        s.k_ld = a.dk_pad; s.v_ld = a.dv_pad; s.v_off = kPageTokens * a.dk_pad;
        s.page_elems = (size_t)a.G * s.head_step;
    }
    return s;
}
// element index of the K row of position p (kv head kvh); the V row of it starts at v_row()
__device__ __forceinline__ size_t k_row(const WinAttnArgs& a, const WinShape& s, const int32_t* pt, int kvh, int p) {
    const int rs = p % s.ring;
    return (size_t)pt[rs / kPageTokens] * s.page_elems + (size_t)kvh * s.head_step + (size_t)(rs % kPageTokens) * s.k_ld;
}
__device__ __forceinline__ size_t v_row(const WinAttnArgs& a, const WinShape& s, const int32_t* pt, int kvh, int p) {
    const int rs = p % s.ring;
    return (size_t)pt[rs / kPageTokens] * s.page_elems + (size_t)kvh * s.head_step + s.v_off + (size_t)(rs % kPageTokens) * s.v_ld;
}
template <typename T> __device__ __forceinline__ T cache_elem(float v);
template <> __device__ __forceinline__ float cache_elem<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 cache_elem<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float widen(float v) { return v; }
__device__ __forceinline__ float widen(__nv_bfloat16 v) { return __bfloat162float(v); }

// factor that brings a row of n elements to unit root mean square (one warp)
__device__ __forceinline__ float rms_factor(const float* x, int n, float eps, int lane) {
    float s = 0.f;
    for (int c = lane; c < n; c += 32) s = fmaf(x[c], x[c], s);
    return __frcp_rn(__fsqrt_rn(__fdiv_rn(warp_total(s), (float)n) + eps));
}

// ---- append: one warp per (row, kv head) ---------------------------------------------------------------
template <typename KT>
__global__ void __launch_bounds__(256) win_append_kernel(WinAttnArgs a) {
    const long w = ((long)blockIdx.x * 256 + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    pdl_release();
    pdl_sync();
    if (w >= (long)a.nseq * a.ts * a.G) return;
    const WinShape s = shape_of(a);
    const int row = (int)(w / a.G), kvh = (int)(w % a.G), sl = row / a.ts, t = row % a.ts, slot = a.b0 + sl;
    if (t >= pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0)) return;
    const int pos = a.pos[slot] + t;
    if (a.limit > 0 && pos >= a.limit) {
        if (lane == 0) atomicOr(&a.ctl->status, STATUS_KV_FULL);
        return;
    }
    const int32_t* pt = a.page_table + (size_t)slot * a.pages_per_seq;
    const float* k = a.proj + (size_t)row * a.ldp + a.off_k + kvh * a.dk;
    const float* v = a.proj + (size_t)row * a.ldp + a.off_v + kvh * a.dv;
    KT* pool = reinterpret_cast<KT*>(a.kv);
    KT* kd = pool + k_row(a, s, pt, kvh, pos);
    KT* vd = pool + v_row(a, s, pt, kvh, pos);
    const float r = a.m.qk_norm ? rms_factor(k, a.dk, a.eps, lane) : 1.f;
    for (int c = lane; c < a.dk_pad; c += 32) kd[c] = cache_elem<KT>(c < a.dk ? k[c] * r : 0.f);
    for (int c = lane; c < a.dv_pad; c += 32) vd[c] = cache_elem<KT>(c < a.dv ? v[c] : 0.f);
}

// ---- plain form ----------------------------------------------------------------------------------------
template <typename KT>
__global__ void __launch_bounds__(128) win_simple_kernel(WinAttnArgs a) {
    extern __shared__ float sm[];
    float* qs = sm;                                       // [dk]
    float* cx = qs + a.dk;                                // [dv] running context
    __shared__ float wt[128];
    __shared__ float red[4];
    const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_release();
    pdl_sync();
    const WinShape s = shape_of(a);
    const int sl = row / a.ts, t = row % a.ts, slot = a.b0 + sl, kvh = h / s.hpk;
    const bool live = t < pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    const size_t out = (size_t)row * a.ldy + (size_t)h * a.dv;
    const int pos = a.pos[slot] + t;
    if (!live || (a.limit > 0 && pos >= a.limit)) {
        if (a.ts > 1 || live) for (int c = tid; c < a.dv; c += 128) put_row(a.y32, a.yhi, a.ylo, out + c, 0.f);
        return;
    }
    const int32_t* pt = a.page_table + (size_t)slot * a.pages_per_seq;
    const KT* pool = reinterpret_cast<const KT*>(a.kv);
    const float* q = a.proj + (size_t)row * a.ldp + a.off_q + (size_t)h * a.dk;
    const float r = a.m.qk_norm ? rms_factor(q, a.dk, a.eps, lane) : 1.f;
    for (int c = tid; c < a.dk; c += 128) qs[c] = q[c] * r;
    for (int c = tid; c < a.dv; c += 128) cx[c] = 0.f;
    __syncthreads();
    const int lo = a.m.window > 0 ? max(0, pos - a.m.window + 1) : 0;
    float m = a.m.sink ? a.m.sink_score : kNoScore, l = a.m.sink ? 1.f : 0.f;      // the sink is the first score seen
    for (int p0 = lo; p0 <= pos; p0 += 128) {
        const int p = p0 + tid;
        float sc = kNoScore;
        if (p <= pos) {
            const KT* k = pool + k_row(a, s, pt, kvh, p);
            float d = 0.f;
            for (int c = 0; c < a.dk; ++c) d = fmaf(qs[c], widen(k[c]), d);
            sc = d * a.m.scale;
        }
        float mx = sc;
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        if (lane == 0) red[warp] = mx;
        __syncthreads();
        const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
        const float f = expf(m - mn), e = p <= pos ? expf(sc - mn) : 0.f;
        m = mn;
        wt[tid] = e;
        __syncthreads();
        const float ls = warp_total(e);
        if (lane == 0) red[warp] = ls;
        const int cnt = min(128, pos - p0 + 1);
        for (int c = tid; c < a.dv; c += 128) {
            float acc = cx[c] * f;
            for (int j = 0; j < cnt; ++j) acc = fmaf(wt[j], widen(pool[v_row(a, s, pt, kvh, p0 + j) + c]), acc);
            cx[c] = acc;
        }
        __syncthreads();
        l = fmaf(l, f, (red[0] + red[1]) + (red[2] + red[3]));
        __syncthreads();
    }
    for (int c = tid; c < a.dv; c += 128) {
        const float v = __fdiv_rn(cx[c], l);
        put_row(a.y32, a.yhi, a.ylo, out + c, a.gate != nullptr ? v * sigmoid_f(a.gate[(size_t)row * a.ldg + (size_t)h * a.dv + c]) : v);
    }
}

// ---- tensor cores ----------------------------------------------------------------------------------------
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
__device__ __forceinline__ void halves2(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - f.x, v1 - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void cp16b(__nv_bfloat16* dst, const __nv_bfloat16* src, bool ok) {
    const int bytes = ok ? 16 : 0;                        // 0: filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}

constexpr int kWinStages = 2;
constexpr int kMmaDim = 256;                              // widest key head of the tensor-core form
constexpr int kWinSlices = 16;
constexpr int kWinSliceMin = 256;                         // tokens from which a slice of the context is worth a CTA

// Grid: (groups of query rows over all sequences, kv head x head subgroup, context slices).  A column m of a warp's 16 is
// (row m / hb, head m % hb) with hb = heads of the subgroup (16 at most).  NT: 8-element tiles of the value row, at least;
// NK > 0: the key row is exactly NK times 16 elements and the value row exactly NT tiles, so that strides and loops are constants.
template <int NT, int NK, bool DECODE>
__global__ void __launch_bounds__(128, NT <= 8 ? 4 : (NT <= 16 ? 3 : 2)) win_mma_kernel(WinAttnArgs a, int hb, int q_rows, int groups_per_seq) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ int is_last;
    const WinShape s = shape_of(a);
    const int DKP = NK > 0 ? NK * 16 : a.dk_pad, DVP = NK > 0 ? NT * 8 : a.dv_pad;
    const int KS = DKP + kPadRow, VS = DVP + kPadRow;
    constexpr int QW = DECODE ? 1 : 4;                    // sets of 16 query columns
    __nv_bfloat16* stage = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    const int stage_elems = kPageTokens * (KS + VS);
    __nv_bfloat16* qh = stage + kWinStages * stage_elems;               // [QW * 16][KS] Q as bf16 halves
    __nv_bfloat16* ql = qh + QW * 16 * KS;
    __nv_bfloat16* kn = ql + QW * 16 * KS;                              // decode: the new token's rows as the cache holds them
    __nv_bfloat16* vn = kn + DKP;

    const int grp = blockIdx.x, kvh = blockIdx.y % a.G, sub = blockIdx.y / a.G, split = blockIdx.z, nsplit = gridDim.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int sl = grp / groups_per_seq, i0 = (grp % groups_per_seq) * q_rows * QW, slot = a.b0 + sl;
    const int h0 = sub * hb, nh = min(hb, s.hpk - h0);    // heads of this CTA inside the group
    pdl_release();
    pdl_sync();
    const int n = pass_tokens(a.row_len, a.ctl, slot, a.ts, a.t_abs0);
    const int nrow = min(q_rows * QW, a.ts - i0), nvalid = max(0, min(nrow, n - i0));
    const int pos0 = a.pos[slot] + i0;
    const bool full = a.limit > 0 && pos0 + nvalid > a.limit;
    if (nvalid < nrow || full) {
        // rows behind a shorter prompt (or outside the cache): zero, so that what follows them stays finite
        if (full && tid == 0) atomicOr(&a.ctl->status, STATUS_KV_FULL);
        if (!DECODE || full) {
            const int first = full ? 0 : nvalid;
            for (int i = tid; i < (nrow - first) * nh * a.dv; i += 128) {
                const int c = i % a.dv, hh = i / a.dv % nh, rr = first + i / (a.dv * nh);
                put_row(a.y32, a.yhi, a.ylo, (size_t)(sl * a.ts + i0 + rr) * a.ldy + (size_t)(kvh * s.hpk + h0 + hh) * a.dv + c, 0.f);
            }
        }
        if (nvalid == 0 || full) return;
    }
    const int32_t* pt = a.page_table + (size_t)slot * a.pages_per_seq;
    __nv_bfloat16* pool = reinterpret_cast<__nv_bfloat16*>(a.kv);
    const int hi = pos0 + nvalid - 1;                     // last position any row of this CTA sees
    const int lo = a.m.window > 0 ? max(0, pos0 - a.m.window + 1) : 0;
    // 64-aligned pages of positions, split evenly over the slices
    const int pg0 = lo / kPageTokens, pages = hi / kPageTokens - pg0 + 1;
    const int per = (pages + nsplit - 1) / nsplit, pb = pg0 + split * per, pe = min(pg0 + pages, pb + per);
    const int local = DECODE && a.append ? pos0 : -1;     // the row that this launch itself appends
    const int kc = DKP / 8, vc = DVP / 8;       // 16-byte chunks per row
    // this thread's first chunk of a page and the step to its next one (a division per chunk would cost more than the copy)
    const int kr0 = tid / kc, kc0 = tid % kc, kdr = 128 / kc, kdc = 128 % kc;
    const int vr0 = tid / vc, vc0 = tid % vc, vdr = 128 / vc, vdc = 128 % vc;
    auto issue = [&](int pg) {
        __nv_bfloat16* ks = stage + ((pg - pb) % kWinStages) * stage_elems;
        __nv_bfloat16* vs = ks + kPageTokens * KS;
        const int pidx = pt[pg % a.pages_per_seq];
        const __nv_bfloat16* kp = pool + (size_t)pidx * s.page_elems + (size_t)kvh * s.head_step;
        const __nv_bfloat16* vp = kp + s.v_off;
        for (int r = kr0, c = kc0; r < kPageTokens;) {
            const int p = pg * kPageTokens + r;
            cp16b(ks + r * KS + c * 8, kp + (size_t)r * s.k_ld + c * 8, p >= lo && p <= hi && p != local);
            r += kdr; c += kdc;
            if (c >= kc) { c -= kc; ++r; }
        }
        for (int r = vr0, c = vc0; r < kPageTokens;) {
            const int p = pg * kPageTokens + r;
            cp16b(vs + r * VS + c * 8, vp + (size_t)r * s.v_ld + c * 8, p >= lo && p <= hi && p != local);
            r += vdr; c += vdc;
            if (c >= vc) { c -= vc; ++r; }
        }
    };
    if (pb < pe) issue(pb);
    asm volatile("cp.async.commit_group;" ::: "memory");
    // query columns: normalised, as bf16 halves; unused columns are zero
    // (four columns at a time, so that their loads overlap)
    for (int m0 = warp * QW * 4; m0 < (warp + 1) * QW * 4; m0 += 4) {
        float v[4][kMmaDim / 32];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int mm = (m0 + j) % 16, rr = (m0 + j) / 16 * q_rows + mm / hb, hh = mm % hb;
            const bool ok = mm < q_rows * hb && rr < nvalid && hh < nh;
            const float* q = a.proj + (size_t)(sl * a.ts + i0 + (ok ? rr : 0)) * a.ldp + a.off_q + (size_t)(kvh * s.hpk + h0 + (ok ? hh : 0)) * a.dk;
#pragma unroll
            for (int i = 0; i < kMmaDim / 32; ++i) v[j][i] = ok && lane + 32 * i < a.dk ? q[lane + 32 * i] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            float r = 1.f;
            if (a.m.qk_norm) {
                float sq = 0.f;
#pragma unroll
                for (int i = 0; i < kMmaDim / 32; ++i) sq = fmaf(v[j][i], v[j][i], sq);
                r = __frcp_rn(__fsqrt_rn(__fdiv_rn(warp_total(sq), (float)a.dk) + a.eps));
            }
#pragma unroll
            for (int i = 0; i < kMmaDim / 32; ++i)
                if (lane + 32 * i < DKP) bf16_halves(v[j][i] * r, qh[(m0 + j) * KS + lane + 32 * i], ql[(m0 + j) * KS + lane + 32 * i]);
        }
    }
    if (DECODE && a.append) {
        const float* k = a.proj + (size_t)(sl * a.ts) * a.ldp + a.off_k + kvh * a.dk;
        const float* v = a.proj + (size_t)(sl * a.ts) * a.ldp + a.off_v + kvh * a.dv;
        if (warp == 0) {
            const float r = a.m.qk_norm ? rms_factor(k, a.dk, a.eps, lane) : 1.f;
            for (int c = lane; c < DKP; c += 32) kn[c] = __float2bfloat16_rn(c < a.dk ? k[c] * r : 0.f);
        } else if (warp == 1) {
            for (int c = lane; c < DVP; c += 32) vn[c] = __float2bfloat16_rn(c < a.dv ? v[c] : 0.f);
        }
        __syncthreads();
        if (split == 0 && sub == 0) {
            __nv_bfloat16* kd = pool + k_row(a, s, pt, kvh, pos0);
            __nv_bfloat16* vd = pool + v_row(a, s, pt, kvh, pos0);
            for (int c = tid; c < DKP; c += 128) kd[c] = kn[c];
            for (int c = tid; c < DVP; c += 128) vd[c] = vn[c];
        }
    }

    // positions that columns g and g + 8 of this warp see: (first, last]
    const int set = DECODE ? 0 : warp;
    int last[2], first[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int m = g + 8 * e, rr = set * q_rows + m / hb;
        const bool ok = m < q_rows * hb && rr < nvalid && m % hb < nh;
        last[e] = ok ? pos0 + rr : -1;
        first[e] = ok && a.m.window > 0 ? last[e] - a.m.window : -1;
    }
    const float sc2 = a.m.scale * kLog2e;                 // scores in units of log 2
    const float m_init = a.m.sink ? a.m.sink_score * kLog2e : kNoScore;
    float mx[2] = {m_init, m_init}, ls[2] = {0.f, 0.f};
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    const int nks = DKP / 16, ndn = DVP / 16;
    constexpr int STRIPS = DECODE ? 1 : 4;                // 16-token strips of a page that one warp works on
    // rows of this warp span [wlo, whi]; a page outside of it has nothing for the warp
    const int whi = DECODE ? hi : min(hi, pos0 + (set + 1) * q_rows - 1);
    const int wlo = DECODE ? lo : (a.m.window > 0 ? pos0 + set * q_rows - a.m.window + 1 : 0);
    for (int pg = pb; pg < pe; ++pg) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                  // this page is here, and every warp has finished with the other stage
        if (pg + 1 < pe) issue(pg + 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        __nv_bfloat16* ks = stage + ((pg - pb) % kWinStages) * stage_elems;
        __nv_bfloat16* vs = ks + kPageTokens * KS;
        if (DECODE && local >= pg * kPageTokens && local < (pg + 1) * kPageTokens) {
            const int r = local - pg * kPageTokens;
            for (int c = tid; c < DKP; c += 128) ks[r * KS + c] = kn[c];
            for (int c = tid; c < DVP; c += 128) vs[r * VS + c] = vn[c];
            __syncthreads();
        }
        const int p0 = pg * kPageTokens;
        if (p0 <= whi && p0 + kPageTokens > wlo) {
            float sc[STRIPS][2][4];
#pragma unroll
            for (int st = 0; st < STRIPS; ++st)
#pragma unroll
                for (int e = 0; e < 2; ++e) { sc[st][e][0] = 0.f; sc[st][e][1] = 0.f; sc[st][e][2] = 0.f; sc[st][e][3] = 0.f; }
            const int strip0 = DECODE ? warp : 0;
#pragma unroll(NK > 0 ? NK : 2)
            for (int k16 = 0; k16 < nks; ++k16) {
                uint32_t fh[4], fl[4];
                const int qo = (set * 16 + (lane & 15)) * KS + k16 * 16 + (lane >> 4) * 8;
                ldm4(fh, qh + qo);
                ldm4(fl, ql + qo);
#pragma unroll
                for (int st = 0; st < STRIPS; ++st) {
                    uint32_t kb[4];
                    const int tok = (strip0 + st) * 16 + ((lane >> 4) << 3) + (lane & 7);
                    ldm4(kb, ks + tok * KS + k16 * 16 + ((lane >> 3) & 1) * 8);
                    mma_bf16(sc[st][0], fh, kb[0], kb[1]);
                    mma_bf16(sc[st][1], fh, kb[2], kb[3]);
                    mma_bf16(sc[st][0], fl, kb[0], kb[1]);
                    mma_bf16(sc[st][1], fl, kb[2], kb[3]);
                }
            }
            // a page that every used column of the warp sees whole needs no mask (unused columns may then hold anything finite)
            const bool whole = p0 + kPageTokens - 1 <= (DECODE ? hi : pos0 + set * q_rows) && (a.m.window <= 0 || p0 > whi - a.m.window);
            float tm[2] = {kNoScore, kNoScore};
            if (!whole) {
#pragma unroll
                for (int st = 0; st < STRIPS; ++st)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const int p = p0 + (strip0 + st) * 16 + e * 8 + 2 * tq + (i & 1), c = i >> 1;
                            sc[st][e][i] = p <= last[c] && p > first[c] ? sc[st][e][i] * sc2 : kNoScore;
                        }
            } else {
#pragma unroll
                for (int st = 0; st < STRIPS; ++st)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
#pragma unroll
                        for (int i = 0; i < 4; ++i) sc[st][e][i] *= sc2;
            }
#pragma unroll
            for (int st = 0; st < STRIPS; ++st)
#pragma unroll
                for (int e = 0; e < 2; ++e)
#pragma unroll
                    for (int i = 0; i < 4; ++i) tm[i >> 1] = fmaxf(tm[i >> 1], sc[st][e][i]);
            float f[2], mu[2];
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                tm[c] = fmaxf(tm[c], __shfl_xor_sync(0xffffffffu, tm[c], 1));
                tm[c] = fmaxf(tm[c], __shfl_xor_sync(0xffffffffu, tm[c], 2));
                const float mn = fmaxf(mx[c], tm[c]);
                f[c] = ex2(mx[c] - mn);
                mx[c] = mn;
                mu[c] = mn > 0.5f * kNoScore ? mn : 0.f;  // nothing seen yet: masked scores still weigh nothing
                ls[c] *= f[c];
            }
#pragma unroll
            for (int i = 0; i < NT; ++i) { o[i][0] *= f[0]; o[i][1] *= f[0]; o[i][2] *= f[1]; o[i][3] *= f[1]; }
#pragma unroll
            for (int st = 0; st < STRIPS; ++st) {
                float pr[2][4];
#pragma unroll
                for (int e = 0; e < 2; ++e)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        pr[e][i] = ex2(sc[st][e][i] - mu[i >> 1]);
                        ls[i >> 1] += pr[e][i];
                    }
                uint32_t ph[4], pl[4];                    // the weights as the A operand of P V
                halves2(pr[0][0], pr[0][1], ph[0], pl[0]);
                halves2(pr[0][2], pr[0][3], ph[1], pl[1]);
                halves2(pr[1][0], pr[1][1], ph[2], pl[2]);
                halves2(pr[1][2], pr[1][3], ph[3], pl[3]);
#pragma unroll
                for (int dn = 0; dn < NT / 2; ++dn) {
                    if (dn < ndn) {
                        uint32_t vb[4];
                        const int tok = (strip0 + st) * 16 + (((lane >> 3) & 1) << 3) + (lane & 7);
                        ldm4t(vb, vs + tok * VS + dn * 16 + (lane >> 4) * 8);
                        mma_bf16(o[2 * dn], ph, vb[0], vb[1]);
                        mma_bf16(o[2 * dn + 1], ph, vb[2], vb[3]);
                        mma_bf16(o[2 * dn], pl, vb[0], vb[1]);
                        mma_bf16(o[2 * dn + 1], pl, vb[2], vb[3]);
                    }
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        ls[c] += __shfl_xor_sync(0xffffffffu, ls[c], 1);
        ls[c] += __shfl_xor_sync(0xffffffffu, ls[c], 2);
    }
    auto emit = [&](int rr, int hh, int d, float v) {
        if (a.gate != nullptr) v *= sigmoid_f(a.gate[(size_t)(sl * a.ts + i0 + rr) * a.ldg + (size_t)(kvh * s.hpk + h0 + hh) * a.dv + d]);
        put_row(a.y32, a.yhi, a.ylo, (size_t)(sl * a.ts + i0 + rr) * a.ldy + (size_t)(kvh * s.hpk + h0 + hh) * a.dv + d, v);
    };
    if constexpr (!DECODE) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            if (last[c] < 0) continue;
            const int m = g + 8 * c, rr = set * q_rows + m / hb, hh = m % hb;
            const float inv = __frcp_rn(ls[c] + (a.m.sink ? exp2f(a.m.sink_score * kLog2e - mx[c]) : 0.f));
            const size_t oo = (size_t)(sl * a.ts + i0 + rr) * a.ldy + (size_t)(kvh * s.hpk + h0 + hh) * a.dv;
            const bool pairs = ((a.dv | a.ldy) & 1) == 0;
            const float* gt = a.gate != nullptr ? a.gate + (size_t)(sl * a.ts + i0 + rr) * a.ldg + (size_t)(kvh * s.hpk + h0 + hh) * a.dv : nullptr;
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int d = i * 8 + 2 * tq;
                float v0 = o[i][2 * c] * inv, v1 = o[i][2 * c + 1] * inv;
                if (pairs && gt != nullptr && d < a.dv) {
                    v0 *= __frcp_rn(1.0f + __expf(-gt[d]));
                    v1 *= __frcp_rn(1.0f + __expf(-gt[d + 1]));
                }
                if (pairs && d < a.dv) {
                    if (a.y32 != nullptr) *reinterpret_cast<float2*>(a.y32 + oo + d) = make_float2(v0, v1);
                    if (a.yhi != nullptr) {
                        uint32_t h2, l2;
                        halves2(v0, v1, h2, l2);
                        *reinterpret_cast<uint32_t*>(a.yhi + oo + d) = h2;
                        if (a.ylo != nullptr) *reinterpret_cast<uint32_t*>(a.ylo + oo + d) = l2;
                    }
                } else if (!pairs) {
                    if (d < a.dv) emit(rr, hh, d, v0);
                    if (d + 1 < a.dv) emit(rr, hh, d + 1, v1);
                }
            }
        }
        return;
    }
    // decode: the four warps' shares in warp order (the stages are free)
    __syncthreads();
    const int CW = DVP + 2;
    float* comb = reinterpret_cast<float*>(smem_raw);     // [4][16][CW]: maximum, sum, context
    {
        float* mine = comb + (size_t)warp * 16 * CW;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int m = g + 8 * c;
            if (tq == 0) { mine[m * CW] = mx[c]; mine[m * CW + 1] = ls[c]; }
#pragma unroll
            for (int i = 0; i < NT; ++i)
                if (i * 8 < DVP) { mine[m * CW + 2 + i * 8 + 2 * tq] = o[i][2 * c]; mine[m * CW + 3 + i * 8 + 2 * tq] = o[i][2 * c + 1]; }
        }
    }
    __syncthreads();
    // per slice: [nh] maxima, [nh] sums, [nh][dv] context
    const size_t unit = (size_t)grp * gridDim.y + blockIdx.y;
    float* part = nsplit > 1 ? a.part + (unit * kWinSlices + split) * (size_t)(hb * (a.dv + 2)) : nullptr;
    for (int i = tid; i < nh * a.dv; i += 128) {
        const int m = i / a.dv, d = i % a.dv;
        float top = comb[m * CW];
#pragma unroll
        for (int w = 1; w < 4; ++w) top = fmaxf(top, comb[(w * 16 + m) * CW]);
        float den = 0.f, num = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float f = exp2f(comb[(w * 16 + m) * CW] - top);
            den = fmaf(f, comb[(w * 16 + m) * CW + 1], den);
            num = fmaf(f, comb[(w * 16 + m) * CW + 2 + d], num);
        }
        if (nsplit == 1) {
            if (a.m.sink) den += exp2f(a.m.sink_score * kLog2e - top);
            emit(0, m, d, __fdiv_rn(num, den));
        } else {
            part[2 * nh + i] = num;
            if (d == 0) { part[m] = top; part[nh + m] = den; }
        }
    }
    if (nsplit == 1) return;
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
    const size_t pw = (size_t)hb * (a.dv + 2);
    const float* all = a.part + unit * kWinSlices * pw;
    for (int i = tid; i < nh * a.dv; i += 128) {
        const int m = i / a.dv;
        float top = m_init;
        for (int sp = 0; sp < nsplit; ++sp) top = fmaxf(top, __ldcg(all + sp * pw + m));
        float den = a.m.sink ? exp2f(a.m.sink_score * kLog2e - top) : 0.f, num = 0.f;
        for (int sp = 0; sp < nsplit; ++sp) {
            const float f = exp2f(__ldcg(all + sp * pw + m) - top);
            den = fmaf(f, __ldcg(all + sp * pw + nh + m), den);
            num = fmaf(f, __ldcg(all + sp * pw + 2 * nh + i), num);
        }
        emit(0, m, i % a.dv, __fdiv_rn(num, den));
    }
}

constexpr size_t kSmemMax = 227 * 1024 - 1024;
int head_block(const MixerSpec& m) {                      // heads of a group that one CTA serves
    const int hpk = m.heads / m.kv_heads, subs = (hpk + 15) / 16;
    return (hpk + subs - 1) / subs;
}
size_t mma_smem(const WinAttnArgs& a, bool decode) {
    const size_t KS = a.dk_pad + kPadRow, VS = a.dv_pad + kPadRow, cols = decode ? 16 : 64;
    const size_t stages = sizeof(__nv_bfloat16) * (kWinStages * (size_t)kPageTokens * (KS + VS) + 2 * cols * KS + a.dk_pad + a.dv_pad);
    const size_t comb = sizeof(float) * 4 * 16 * ((size_t)a.dv_pad + 2);
    return std::max(stages, decode ? comb : (size_t)0);
}

template <int NT, int NK>
cudaError_t launch_mma(const WinAttnArgs& a, cudaStream_t st) {
    const bool decode = a.ts == 1;
    const int hb = head_block(a.m), hpk = a.H / a.G, subs = (hpk + hb - 1) / hb;
    const size_t smem = mma_smem(a, decode);
    if (decode) {
        const long units = (long)a.nseq * a.G * subs;
        int nsplit = 1;
        if (a.part != nullptr && units <= kAttnPartUnits) {
            const int ctx = a.m.window > 0 ? std::min(a.m.window, a.pages_per_seq * kPageTokens) : a.pages_per_seq * kPageTokens;
            nsplit = std::min<int>({(int)((2L * 148 + units - 1) / units), (ctx + kWinSliceMin - 1) / kWinSliceMin, kWinSlices});
            if (nsplit < 1) nsplit = 1;
        }
        auto kern = win_mma_kernel<NT, NK, true>;
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        return launch_rows(kern, dim3(a.nseq, a.G * subs, nsplit), 128, smem, st, a, hb, 1, 1);
    }
    const int q_rows = 16 / hb, gps = (a.ts + 4 * q_rows - 1) / (4 * q_rows);
    auto kern = win_mma_kernel<NT, NK, false>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    return launch_rows(kern, dim3((unsigned)a.nseq * gps, a.G * subs, 1), 128, smem, st, a, hb, q_rows, gps);
}

template <typename KT>
cudaError_t append(const WinAttnArgs& a, cudaStream_t st) {
    const long warps = (long)a.nseq * a.ts * a.G;
    return launch_rows(win_append_kernel<KT>, dim3((unsigned)((warps + 7) / 8)), 256, 0, st, a);
}
template <typename KT>
cudaError_t simple(const WinAttnArgs& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * ((size_t)a.dk + a.dv);
    if (smem > kSmemMax) return cudaErrorInvalidValue;
    auto kern = win_simple_kernel<KT>;
    if (smem > 40 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return launch_rows(kern, dim3((unsigned)(a.nseq * a.ts), a.H), 128, smem, st, a);
}

}  // namespace

size_t window_attention_part_floats(const MixerSpec& m) { return (size_t)kWinSlices * head_block(m) * (m.vdim + 2); }

cudaError_t launch_window_attention(const WinAttnArgs& a, cudaStream_t st, int* launches) {
    *launches = 0;
    const bool mma = !a.kv_is_f32 && !a.plain && a.dk_pad <= kMmaDim && a.dv_pad <= 256 && mma_smem(a, a.ts == 1) <= kSmemMax;
    cudaError_t e;
    if (a.append && !(mma && a.ts == 1)) {
        e = a.kv_is_f32 ? append<float>(a, st) : append<__nv_bfloat16>(a, st);
        if (e != cudaSuccess) return e;
        *launches += 1;
    }
    *launches += 1;
    if (!mma) return a.kv_is_f32 ? simple<float>(a, st) : simple<__nv_bfloat16>(a, st);
    const int nt = a.dv_pad / 8, nk = a.dk_pad / 16;
    if (nt == 4 && nk == 2) return launch_mma<4, 2>(a, st);
    if (nt == 8 && nk == 4) return launch_mma<8, 4>(a, st);
    if (nt == 8 && nk == 6) return launch_mma<8, 6>(a, st);
    if (nt == 12 && nk == 6) return launch_mma<12, 6>(a, st);
    if (nt == 16 && nk == 8) return launch_mma<16, 8>(a, st);
    if (nt == 16 && nk == 12) return launch_mma<16, 12>(a, st);
    if (nt <= 4) return launch_mma<4, 0>(a, st);
    if (nt <= 8) return launch_mma<8, 0>(a, st);
    if (nt <= 12) return launch_mma<12, 0>(a, st);
    if (nt <= 16) return launch_mma<16, 0>(a, st);
    if (nt <= 24) return launch_mma<24, 0>(a, st);
    return launch_mma<32, 0>(a, st);
}

}  // namespace lumi
