// Latent attention over a paged cache: keys and values of all heads are linear in one cached latent c per token,
//   k[h] = [Wk[h] c | r],  v[h] = Wv[h] c,  score = (q[h] . k[h]) * scale,
// r a rotated key part shared by the heads; sliding window, an optional extra term exp(sink[h]) in the softmax denominator,
// heads multiplied by sigmoid(gate), one gate per channel or per head.  A cache row is [c: Lc | r: Rc] (Lc, Rc: kv_rank, rot_dim padded to 8 with zeros), normed
// and rotated.  The projections arrive as one row [query latent: Qp | c: Lc | r: Rc | gate: H * Dv or H].
//
//   latent_rows          many rows: norms of the two latents, rotation of r, cache append
//   latent_rotate_rows   many rows: rotation of the queries' rotated part, in place
//   latent_gather_rows   long entries: the earlier cache rows an entry sees into a contiguous workspace, where latent_rows has put
//                        its new ones; one product expands all of them to keys and values of all heads, and the tensor-core
//                        attention (window_attention_tc.cuh) reads those
//   latent_attention     one row per cluster, absorbed form: the query is moved into the latent space (qa = Wk[h]^T q), scores and
//                        sums run over the cached rows as they are, the result goes through Wv[h] and the gate: decode steps,
//                        short portions and the 32-bit mode.  Nothing per-head is ever stored for a key.
#pragma once
#include <cooperative_groups.h>

#include <utility>

#include "common.cuh"
#include "rotary.cuh"
#include "row_plan.cuh"
#include "window_attention.cuh"

namespace efm {

struct LatentShape {
    int H, D, R, Dv, L;               // heads, unrotated and rotated query channels, value channels, latent width
    int Dp, Vp, Qp, Lc, Rc;           // padded to 8; Qp: query latent
    int q_rank, window;
    float scale, eps;
    RotShape rot;                     // of the R channels
    const __nv_bfloat16* q_norm;      // [Qp]
    const __nv_bfloat16* kv_norm;     // [Lc]
    const __nv_bfloat16* sink;        // [H] or null
    const __nv_bfloat16* wk;          // [H * Dp][Lc]
    const __nv_bfloat16* wv;          // [H * Vp][Lc]
    int gate;                         // the projections end with a gate per 1: channel, 2: head; 0: no gate
    __host__ __device__ int off_c() const { return Qp; }
    __host__ __device__ int off_r() const { return Qp + Lc; }
    __host__ __device__ int off_gate() const { return Qp + Lc + Rc; }
    __host__ __device__ int q_ld() const { return H * (Dp + Rc); }
};

// ---- many rows -----------------------------------------------------------------------------------------------------
// One warp per row, 8 channels per lane and turn (every part is a multiple of 8); the first 32 * 8 * KEEP channels stay in
// registers.  ws (may be null): rows of the long entries go to the workspace too.
constexpr int kLatentRowsPerBlock = 4;
template <typename T>
__global__ void __launch_bounds__(32 * kLatentRowsPerBlock) latent_rows_kernel(const T* __restrict__ proj, int ld, T* __restrict__ cq, T* __restrict__ pool,
                                                                                T* __restrict__ ws, int ws_min_rows, const LatentShape s, const RowPlan plan) {
    constexpr int KEEP = 6;
    __shared__ float cs_s[kLatentRowsPerBlock][kRotMaxPairs], sn_s[kLatentRowsPerBlock][kRotMaxPairs], rot_s[kLatentRowsPerBlock][2 * kRotMaxPairs];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * kLatentRowsPerBlock + warp;
    if (row >= plan.rows) return;                                       // no block barriers below
    float *cs = cs_s[warp], *sn = sn_s[warp], *rot = rot_s[warp];
    const int nq = s.Qp / 8, nc = s.Lc / 8, n = nq + nc + s.Rc / 8;
    const T* src = proj + (size_t)row * ld;
    float keep[KEEP][8];
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (lane + 32 * i < n) load8_as_f32(src + 8 * (lane + 32 * i), keep[i]);
    const RowEntry e = plan.of_row(row);
    const int pos = e.pos0 + row - e.row0;
    for (int i = lane; i < s.rot.dims / 2; i += 32) rot_sincos(s.rot, pos, i, sn + i, cs + i);
    float a = 0.f, b = 0.f;                                             // pads are zero
    auto take = [&](int c, const float (&f)[8]) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
        if (c < nq) a += ss;
        else if (c < nq + nc) b += ss;
        else
#pragma unroll
            for (int j = 0; j < 8; ++j) rot[8 * (c - nq - nc) + j] = f[j];
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (lane + 32 * i < n) take(lane + 32 * i, keep[i]);
    for (int c = lane + 32 * KEEP; c < n; c += 32) { float f[8]; load8_as_f32(src + 8 * c, f); take(c, f); }
    a = warp_sum(a);
    b = warp_sum(b);
    __syncwarp();
    const float ia = 1.0f / sqrtf(a / (float)s.q_rank + s.eps), ib = 1.0f / sqrtf(b / (float)s.L + s.eps);
    T* dst = pool + plan.cache_row(e, pos) * (s.Lc + s.Rc);
    T* dst2 = ws != nullptr && e.n >= ws_min_rows ? ws + (size_t)(e.ws0 + pos) * (s.Lc + s.Rc) : nullptr;
    auto emit = [&](int c, float (&f)[8]) {
        if (c < nq + nc) {
            float w[8];
            unpack8(ld_cached(c < nq ? s.q_norm + 8 * c : s.kv_norm + 8 * (c - nq)), w);
            const float inv = c < nq ? ia : ib;
#pragma unroll
            for (int j = 0; j < 8; ++j) f[j] *= inv * w[j];
        } else {
#pragma unroll
            for (int j = 0; j < 8; ++j) f[j] = rot_channel(s.rot, rot, 8 * (c - nq - nc) + j, cs, sn);
        }
        store_head8(c < nq ? cq + (size_t)row * s.Qp + 8 * c : dst + 8 * (c - nq), f);
        if (c >= nq && dst2 != nullptr) store_head8(dst2 + 8 * (c - nq), f);
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if (lane + 32 * i < n) emit(lane + 32 * i, keep[i]);
    for (int c = lane + 32 * KEEP; c < n; c += 32) { float f[8]; load8_as_f32(src + 8 * c, f); emit(c, f); }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_rotate_rows_kernel(T* __restrict__ q, const LatentShape s, const RowPlan plan) {
    __shared__ float cs[kRotMaxPairs], sn[kRotMaxPairs];
    const int row = blockIdx.x, pairs = s.rot.dims / 2;
    const RowEntry e = plan.of_row(row);
    rot_table(s.rot, e.pos0 + row - e.row0, cs, sn);
    __syncthreads();
    T* base = q + (size_t)row * s.q_ld() + s.Dp;
    const int ld = s.Dp + s.Rc;
    if (s.rot.kind == kRotPairs) {                                      // pairs are neighbours: 8 channels per thread
        const int per = s.Rc / 8;
        for (int n = threadIdx.x; n < s.H * per; n += 256) {
            const int h = n / per, c = (n - h * per) * 8;
            T* x = base + (size_t)h * ld + c;
            float f[8];
            load8_as_f32(x, f);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                const int i = (c + j) >> 1;
                if (i >= pairs) continue;
                const float u = f[j], v = f[j + 1];
                f[j] = u * cs[i] - v * sn[i];
                f[j + 1] = v * cs[i] + u * sn[i];
            }
            store_head8(x, f);
        }
        return;
    }
    for (int n = threadIdx.x; n < s.H * pairs; n += 256) {
        const int h = n / pairs, i = n - h * pairs;
        T* x = base + (size_t)h * ld + i;
        const float u = to_f32(x[0]), v = to_f32(x[pairs]);
        store_f32(x, u * cs[i] - v * sn[i]);
        store_f32(x + pairs, v * cs[i] + u * sn[i]);
    }
}

// Grid (pages, parts of a page): pages[i] = (entry, page of its sequence); null: page0 + i of the single entry.
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_rows_kernel(const T* __restrict__ pool, T* __restrict__ ws, int row_elems, const RowPlan plan,
                                                                 const RowTile* __restrict__ pages, int page0) {
    const RowTile t = pages != nullptr ? pages[blockIdx.x] : RowTile{0, page0 + (int)blockIdx.x};
    const RowEntry e = plan.entry(t.entry);
    const uint4* src = reinterpret_cast<const uint4*>(pool + plan.cache_row(e, t.row * kPageTokens) * row_elems);
    uint4* dst = reinterpret_cast<uint4*>(ws + (size_t)(e.ws0 + t.row * kPageTokens) * row_elems);
    const int n = min(kPageTokens, e.pos0 - t.row * kPageTokens) * (row_elems * (int)sizeof(T) / 16);      // rows from pos0 on are new
    for (int i = blockIdx.y * 256 + threadIdx.x; i < n; i += 256 * gridDim.y) dst[i] = src[i];
}

// ---- one row, absorbed -----------------------------------------------------------------------------------------------
namespace la {
constexpr int kThreads = 512, kWarps = kThreads / 32, kMaxTile = 128;
struct Layout {
    int kt, ldk, slice;               // keys per tile (at most kMaxTile), elements between key rows, latent channels per block of the cluster
    unsigned int q, qin, cnew, keys, scr, rout, olat, bytes;
};
// Shared memory of one block: heads per block, cluster width, bytes per cache element.
__host__ __device__ inline Layout layout(const LatentShape& s, int nh, int splits, int es, int kt) {
    Layout l;
    l.kt = kt;
    l.ldk = s.Lc + s.Rc + 16 / es;
    l.slice = (s.Lc / 8 + splits - 1) / splits * 8;
    unsigned int at = 0;
    auto take = [&](unsigned int bytes) { const unsigned int a = at; at = (at + bytes + 15u) & ~15u; return a; };
    l.q = take((unsigned int)nh * (s.Lc + s.Rc) * 4u);
    l.qin = take((unsigned int)nh * (s.Dp + s.Rc) * 4u);
    l.cnew = take((unsigned int)(s.Lc + s.Rc) * 4u);
    const unsigned int kb = (unsigned int)kt * l.ldk * es, rb = (unsigned int)nh * 4u * kThreads * 4u;       // keys; afterwards sums of the key groups
    l.keys = take(kb > rb ? kb : rb);
    l.scr = take(kThreads * 8u * 4u);
    l.rout = take((unsigned int)splits * nh * l.slice * 4u);
    l.olat = take((unsigned int)nh * s.Lc * 4u);
    l.bytes = at;
    return l;
}
}  // namespace la

template <typename TC, typename TI, typename TO>
struct LatentParams {
    LatentShape s;
    const TI* q;                      // [rows][H][Dp + Rc]; decode: not rotated yet
    const TI* proj;                   // [rows][ld]
    int ld;
    TC* pool;                         // [pages * 64][Lc + Rc]
    TO* out;                          // [rows][ld_out]
    int ld_out, kt;
    // many rows: the plan and the rows to compute (null: all)
    RowPlan plan;
    const int32_t* rows;
    // one row (decode)
    const int32_t* pages;
    int max_pages, early;
    DecodeState* state;
};

// grid (cluster width, ceil(H / NH), rows).  The blocks of a cluster share the visible keys, the latent channels of the query
// and of the result, and the value rows.
template <typename TC, bool DECODE, int NH>
__global__ void __launch_bounds__(la::kThreads) latent_attention_kernel(const LatentParams<TC, typename std::conditional<DECODE, float, TC>::type,
                                                                                           typename std::conditional<DECODE, float, TC>::type> p) {
    namespace cg = cooperative_groups;
    using namespace la;
    using TI = typename std::conditional<DECODE, float, TC>::type;
    extern __shared__ __align__(16) unsigned char la_smem[];
    __shared__ float cs[kRotMaxPairs], sn[kRotMaxPairs], part[kWarps], sp[NH][kMaxTile], sal[NH], sm_m[NH], sm_l[NH], rm[16][NH], rl[16][NH];
    const LatentShape& s = p.s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, split = blockIdx.x, n_splits = gridDim.x;
    const int h0 = blockIdx.y * NH, nh = min(NH, s.H - h0), LR = s.Lc + s.Rc;
    const Layout l = layout(s, NH, n_splits, sizeof(TC), p.kt);
    float* q = reinterpret_cast<float*>(la_smem + l.q);
    float* qin = reinterpret_cast<float*>(la_smem + l.qin);
    float* cnew = reinterpret_cast<float*>(la_smem + l.cnew);
    TC* keys = reinterpret_cast<TC*>(la_smem + l.keys);
    float* red = reinterpret_cast<float*>(la_smem + l.keys);
    float* scr = reinterpret_cast<float*>(la_smem + l.scr);
    float* rout = reinterpret_cast<float*>(la_smem + l.rout);
    float* olat = reinterpret_cast<float*>(la_smem + l.olat);
    cg::cluster_group cl = cg::this_cluster();
    auto started = cl.barrier_arrive();                                // waited for before the first store into another block

    const int s0 = min(split * l.slice, s.Lc), s1 = min(s0 + l.slice, s.Lc), sl8 = (s1 - s0) / 8;
    const int n_val = nh * s.Dv, vals = (n_val + n_splits - 1) / n_splits, v0 = split * vals, v1 = min(n_val, v0 + vals);
    auto to_l2 = [](const void* a) { asm volatile("prefetch.global.L2 [%0];" ::"l"(a)); };
    if constexpr (DECODE) {                                            // weights of this block on their way
        const int lines = ((s1 - s0) * 2 + 127) / 128;
        for (int i = tid; i < nh * s.Dp * lines; i += kThreads) to_l2(s.wk + ((size_t)h0 * s.Dp + i / lines) * s.Lc + s0 + (i % lines) * 64);
        const int vl = (s.Lc * 2 + 127) / 128;
        for (int i = tid; i < (v1 - v0) * vl; i += kThreads) {
            const int v = v0 + i / vl;
            to_l2(s.wv + ((size_t)(h0 + v / s.Dv) * s.Vp + v % s.Dv) * s.Lc + (i % vl) * 64);
        }
        if (!p.early) { pdl_wait(); pdl_launch_dependents(); }
    }
    const int row = DECODE ? 0 : (p.rows != nullptr ? p.rows[blockIdx.z] : (int)blockIdx.z);
    RowEntry e{};
    int pos;
    bool ok = true;
    const int32_t* pages;
    if constexpr (DECODE) {
        const int kv_len = (int)p.state->kv_len;
        ok = kv_len > 0 && kv_len <= p.max_pages * kPageTokens;
        pos = kv_len - 1;
        pages = p.pages;
    } else {
        e = p.plan.of_row(row);
        pos = e.pos0 + row - e.row0;
        pages = p.plan.page_table + (size_t)e.table * p.plan.max_pages;
    }
    const int lo = s.window > 0 ? max(0, pos + 1 - s.window) : 0, n_vis = pos + 1 - lo;
    const int chunk = ok ? (n_vis + n_splits - 1) / n_splits : 0;
    const int begin = lo + split * chunk, end = ok ? min(pos + 1, begin + chunk) : begin;
    const int n_tiles = end > begin ? (end - begin + l.kt - 1) / l.kt : 0;
    const bool append = DECODE && n_tiles > 0 && end == pos + 1;       // this block walks the newest key
    auto pool_row = [&](int j) { return (size_t)pages[j / kPageTokens] * kPageTokens + j % kPageTokens; };
    const int per = LR * (int)sizeof(TC) / 16;                         // 16-byte pieces of a cache row
    auto load_tile = [&](int t) {
        if (t < n_tiles) {
            const int j0 = begin + t * l.kt;
            TC* dst = keys;
            for (int r = warp; r < l.kt; r += kWarps) {                // a warp per cache row
                const int j = j0 + r;
                if (j >= end || (DECODE && j == pos)) continue;
                const char* src = reinterpret_cast<const char*>(p.pool + pool_row(j) * LR);
                const uint32_t to = (uint32_t)__cvta_generic_to_shared(dst + (size_t)r * l.ldk);
                for (int c = lane; c < per; c += 32)
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to + 16u * c), "l"(src + 16 * c) : "memory");
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(0);                                                      // a window's share is one tile as a rule
    if (ok) rot_table(s.rot, pos, cs, sn);
    if constexpr (DECODE) {
        if (p.early) { pdl_wait(); pdl_launch_dependents(); }
    }

    // ---- this token's queries (and, decode, its cache row) -------------------------------------------------------------
    const int qw = s.Dp + s.Rc;
    for (int i = tid; i < nh * qw; i += kThreads) {
        const TI* src = p.q + (size_t)row * s.q_ld() + (size_t)h0 * qw + i;
        if constexpr (DECODE) qin[i] = __ldcg(src); else qin[i] = to_f32(*src);
    }
    float ss = 0.f;
    if constexpr (DECODE) {
        for (int c = tid; c < LR; c += kThreads) {
            const float v = __ldcg(reinterpret_cast<const float*>(p.proj) + s.off_c() + c);
            cnew[c] = v;
            if (c < s.Lc) ss = fmaf(v, v, ss);
        }
        ss = warp_sum(ss);
        if (lane == 0) part[warp] = ss;
    }
    if (tid < NH) { sm_m[tid] = -INFINITY; sm_l[tid] = 0.f; }
    __syncthreads();
    for (int i = tid; i < nh * s.Rc; i += kThreads) {
        const int h = i / s.Rc, c = i - h * s.Rc;
        q[h * LR + s.Lc + c] = (DECODE ? rot_channel(s.rot, qin + h * qw + s.Dp, c, cs, sn) : qin[h * qw + s.Dp + c]) * s.scale;
    }
    if constexpr (DECODE) {
        if (append) {
            ss = 0.f;
#pragma unroll
            for (int i = 0; i < kWarps; ++i) ss += part[i];
            const float inv = 1.0f / sqrtf(ss / (float)s.L + s.eps);
            TC* dst = p.pool + pool_row(pos) * LR;
            for (int c = tid; c < LR; c += kThreads) {
                const float v = c < s.Lc ? cnew[c] * inv * __bfloat162float(s.kv_norm[c]) : rot_channel(s.rot, cnew + s.Lc, c - s.Lc, cs, sn);
                if (blockIdx.y == 0) store_f32(dst + c, v);
                scr[c] = v;                                            // at most kThreads * 8 channels
            }
            __syncthreads();
            for (int c = tid; c < LR; c += kThreads) cnew[c] = scr[c];
            __syncthreads();
        }
    }

    // ---- the queries in the latent space: this block's channels for all of its heads, sent to every block ------------------
    {
        const int cols = nh * sl8;                                     // 8-channel columns
        int dl = 1;
        while (dl * 2 * cols <= kThreads && dl < 32) dl *= 2;
        const int wide = kThreads / dl;
        cl.barrier_wait(std::move(started));
        for (int c0 = 0; c0 < cols; c0 += wide) {
            const int c = c0 + tid % wide, d0 = tid / wide;
            float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (c < cols) {
                const int h = c / sl8;
                const __nv_bfloat16* w = s.wk + (size_t)(h0 + h) * s.Dp * s.Lc + s0 + (c - h * sl8) * 8;
#pragma unroll 4
                for (int d = d0; d < s.Dp; d += dl) {
                    float f[8];
                    unpack8(ld_cached(w + (size_t)d * s.Lc), f);
                    const float x = qin[h * qw + d];
#pragma unroll
                    for (int j = 0; j < 8; ++j) acc[j] = fmaf(x, f[j], acc[j]);
                }
            }
            __syncthreads();
#pragma unroll
            for (int j = 0; j < 8; ++j) scr[tid * 8 + j] = acc[j];
            __syncthreads();
            const int n = min(wide, cols - c0) * 8;                    // sums over d0: eight lanes each
            for (int i0 = 0; i0 < n; i0 += kThreads / 8) {
                const int i = i0 + tid / 8, x = tid & 7;
                float v = 0.f;
                if (i < n)
                    for (int d = x; d < dl; d += 8) v += scr[d * wide * 8 + i];
#pragma unroll
                for (int o = 4; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                if (i < n) {
                    const int cc = c0 + i / 8, h = cc / sl8, ch = s0 + (cc - h * sl8) * 8 + (i & 7);
                    v *= s.scale;
                    for (int r = x; r < n_splits; r += 8) *cl.map_shared_rank(q + h * LR + ch, r) = v;
                }
            }
        }
    }
    if (n_splits > 1) cl.sync(); else __syncthreads();

    // ---- attention over this block's keys ----------------------------------------------------------------------------------
    const int parts = kThreads / l.kt, key = tid / parts, pt = tid % parts;
    const int tpr = s.Lc / 4, kg = kThreads / tpr, dpart = tid % tpr, tg = tid / tpr;
    const bool pv = tg < kg;
    float acc[NH][4];
#pragma unroll
    for (int h = 0; h < NH; ++h)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[h][j] = 0.f;
    for (int t = 0; t < n_tiles; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        TC* kt = keys;
        const int j0 = begin + t * l.kt;
        if (append && t == n_tiles - 1)
            for (int c = tid; c < LR; c += kThreads) store_f32(kt + (size_t)(pos - j0) * l.ldk + c, cnew[c]);
        __syncthreads();
        const bool vis = j0 + key < end;
        float d[NH];
#pragma unroll
        for (int h = 0; h < NH; ++h) d[h] = 0.f;
        if (vis) {
            for (int c = pt; c < LR / 8; c += parts) {
                float f[8];
                load8_as_f32(kt + (size_t)key * l.ldk + c * 8, f);
#pragma unroll
                for (int h = 0; h < NH; ++h)
                    if (h < nh) {
                        const float4 a = *reinterpret_cast<const float4*>(q + h * LR + c * 8), b = *reinterpret_cast<const float4*>(q + h * LR + c * 8 + 4);
                        d[h] = fmaf(a.x, f[0], d[h]); d[h] = fmaf(a.y, f[1], d[h]); d[h] = fmaf(a.z, f[2], d[h]); d[h] = fmaf(a.w, f[3], d[h]);
                        d[h] = fmaf(b.x, f[4], d[h]); d[h] = fmaf(b.y, f[5], d[h]); d[h] = fmaf(b.z, f[6], d[h]); d[h] = fmaf(b.w, f[7], d[h]);
                    }
            }
        }
#pragma unroll
        for (int h = 0; h < NH; ++h) {
            for (int x = parts / 2; x > 0; x >>= 1) d[h] += __shfl_xor_sync(0xffffffffu, d[h], x);
            if (pt == 0) sp[h][key] = vis && h < nh ? d[h] : -INFINITY;
        }
        __syncthreads();
        if (warp < nh) {
            float x[kMaxTile / 32], mx = -INFINITY, sum = 0.f;
#pragma unroll
            for (int i = 0; i < kMaxTile / 32; ++i) {
                x[i] = lane + 32 * i < l.kt ? sp[warp][lane + 32 * i] : -INFINITY;
                mx = fmaxf(mx, x[i]);
            }
            const float mo = sm_m[warp], mn = fmaxf(mo, warp_max(mx));          // the tile holds a visible key
#pragma unroll
            for (int i = 0; i < kMaxTile / 32; ++i) {
                x[i] = expf(x[i] - mn);
                if (lane + 32 * i < l.kt) sp[warp][lane + 32 * i] = x[i];
                sum += x[i];
            }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float al = expf(mo - mn);
                sal[warp] = al;
                sm_m[warp] = mn;
                sm_l[warp] = sm_l[warp] * al + sum;
            }
        }
        __syncthreads();
        if (pv) {
#pragma unroll
            for (int h = 0; h < NH; ++h)
                if (h < nh) {
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[h][j] *= sal[h];
                }
            const int n = min(l.kt, end - j0);
            for (int kk = tg; kk < n; kk += kg) {
                const float4 v = load4_as_f32(kt + (size_t)kk * l.ldk + dpart * 4);
#pragma unroll
                for (int h = 0; h < NH; ++h)
                    if (h < nh) {
                        const float w = sp[h][kk];
                        acc[h][0] = fmaf(w, v.x, acc[h][0]); acc[h][1] = fmaf(w, v.y, acc[h][1]);
                        acc[h][2] = fmaf(w, v.z, acc[h][2]); acc[h][3] = fmaf(w, v.w, acc[h][3]);
                    }
            }
        }
        __syncthreads();
        if (t + 1 < n_tiles) load_tile(t + 1);
    }
    // ---- sums over the key groups, then over the cluster: every latent channel belongs to one block ------------------------
    if (pv) {
#pragma unroll
        for (int h = 0; h < NH; ++h)
            *reinterpret_cast<float4*>(red + ((size_t)tg * NH + h) * s.Lc + dpart * 4) = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
    }
    __syncthreads();
    for (int c = tid; c < s.Lc; c += kThreads) {
        const int owner = c / l.slice;
        float* to = cl.map_shared_rank(rout + (size_t)split * NH * l.slice + c - owner * l.slice, owner);
#pragma unroll
        for (int h = 0; h < NH; ++h)
            if (h < nh) {
                float v = 0.f;
                for (int g = 0; g < kg; ++g) v += red[((size_t)g * NH + h) * s.Lc + c];
                to[h * l.slice] = v;
            }
    }
    for (int i = tid; i < n_splits * nh; i += kThreads) {
        const int r = i / nh, h = i - r * nh;
        *cl.map_shared_rank(&rm[split][h], r) = sm_m[h];
        *cl.map_shared_rank(&rl[split][h], r) = sm_l[h];
    }
    if (n_splits > 1) cl.sync(); else __syncthreads();
    for (int i = tid; i < nh * (s1 - s0); i += kThreads) {
        const int h = i / (s1 - s0), c = i - h * (s1 - s0);
        float m = s.sink != nullptr ? __bfloat162float(s.sink[h0 + h]) : -INFINITY;
        const float sk = m;
        for (int r = 0; r < n_splits; ++r) m = fmaxf(m, rm[r][h]);
        float num = 0.f, den = s.sink != nullptr ? expf(sk - m) : 0.f;
        for (int r = 0; r < n_splits; ++r) {
            const float w = rm[r][h] == -INFINITY ? 0.f : expf(rm[r][h] - m);
            num = fmaf(w, rout[((size_t)r * NH + h) * l.slice + c], num);
            den = fmaf(w, rl[r][h], den);
        }
        const float v = den > 0.f ? num / den : 0.f;
        for (int r = 0; r < n_splits; ++r) *cl.map_shared_rank(olat + h * s.Lc + s0 + c, r) = v;
    }
    if (n_splits > 1) cl.sync(); else __syncthreads();
    // ---- values and gate: as many lanes per value row as keep every warp's rows in flight together --------------------------
    int lanes = 32;
    while (lanes > 4 && (kThreads / lanes) < v1 - v0) lanes /= 2;
    for (int vb = v0; vb < v1; vb += kThreads / lanes) {
        const int v = vb + tid / lanes, li = tid % lanes, h = v < v1 ? v / s.Dv : 0, c = v - h * s.Dv;
        float a = 0.f;
        if (v < v1) {
            const __nv_bfloat16* w = s.wv + ((size_t)(h0 + h) * s.Vp + c) * s.Lc;
#pragma unroll 4
            for (int i = li; i < s.Lc / 8; i += lanes) {
                const float4 x = *reinterpret_cast<const float4*>(olat + h * s.Lc + i * 8), y = *reinterpret_cast<const float4*>(olat + h * s.Lc + i * 8 + 4);
                const float f[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w};
                a = dot8(ld_cached(w + i * 8), f, a);
            }
        }
        for (int o = lanes / 2; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        if (li == 0 && v < v1) {
            if (s.gate) {
                const TI* gp = p.proj + (size_t)row * p.ld + s.off_gate() + (s.gate == 2 ? h0 + h : (h0 + h) * s.Dv + c);
                float g;
                if constexpr (DECODE) g = __ldcg(gp); else g = to_f32(*gp);
                a *= 1.0f / (1.0f + expf(-g));
            }
            store_f32(p.out + (size_t)row * p.ld_out + (h0 + h) * s.Dv + c, a);
        }
    }
    if (DECODE && !ok && tid == 0) p.state->error = 2;
}

}  // namespace efm
