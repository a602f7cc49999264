// Many-row form of the decayed linear attention (linear_attention.cuh) on the 5th-generation tensor cores, chunks of 128 tokens:
//   linear_chunk_tc    U = K'^T V, K' the keys times the decay that is left to the end of the chunk
//   linear_attend_tc   P = Q K^T masked and decayed, O = decay * (Q S) + P V, S the state the chunk starts from
// q, k and v enter as they are, in bf16.  What is not exact in bf16 -- K', P and S -- enters as a bf16 pair high +
// low (16 bits of mantissa); products accumulate in fp32 and the states in memory are fp32.
// Operands are staged by the threads, which apply decay and the split on the way, in the 128-byte-swizzled layout that TMA would
// write: [row][64 channels] boxes of 128 bytes a row.  The same image serves as a K-major operand (channels contracted) and as an
// MN-major one (rows contracted).  P goes from tensor memory to tensor memory.  Every mbarrier wait is bounded and raises *error.
// Head sizes up to 128 key channels; value channels in slices of VP (grid.z).
// CH: decays per key channel, given as sums b_t of their logarithms from the chunk's first token on.  The keys of the first product are
// k_t e^(b_n - b_t) (at most k_t); those of the second and its queries are k_s e^(m - b_s) and q_t e^(b_t - m), m half of the chunk's
// whole sum, both pairs high + low, and the state's rows take e^m: all of it stays in range while no channel loses more than e^kMaxLoss
// in a chunk.  A chunk that loses more takes m = 0 for the state and forms its products of queries and keys one by one.
#pragma once
#include "attention_tc.cuh"
#include "linear_attention.cuh"
#include "window_attention_tc.cuh"

namespace efm {

namespace lt {
constexpr int C = kLinearChunkTc, kThreads = 256, kAttendThreads = 512;
constexpr int BOX = C * 128;                                  // bytes of a box of 64 channels
template <int VP>
struct Cfg {
    static constexpr int V_BYTES = BOX * (VP / 64), K_BYTES = BOX * 2;
    static constexpr size_t CHUNK_SMEM = 2 * K_BYTES + V_BYTES + 1024 + 64;
    static constexpr size_t ATTEND_SMEM = 2 * K_BYTES + V_BYTES + 2 * V_BYTES + 1024 + 64;
    static constexpr size_t ATTEND_CH_SMEM = 4 * K_BYTES + V_BYTES + 1024 + 64;
    static constexpr int HALF = VP / 2;
};
constexpr float kMaxLoss = 100.f;
constexpr int PH_COL = 128, PL_COL = 192, O1_COL = 256, O2_COL = 384;      // attend: P | P high | P low | Q S | P V

__device__ __forceinline__ uint32_t image(int row, int c8) {          // byte offset of channels [8 c8, 8 c8 + 8) of a row
    return (uint32_t)((c8 >> 3) * BOX + row * 128 + (((c8 & 7) ^ (row & 7)) << 4));
}
// f as a pair: high parts to one image, what they leave to the other
__device__ __forceinline__ void put_pair(unsigned char* hi, unsigned char* lo, int row, int c8, const float (&f)[8]) {
    uint4 h, l;
    uint32_t *hp = &h.x, *lp = &l.x;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        hp[j] = pack_bf16(f[2 * j], f[2 * j + 1]);
        lp[j] = pack_bf16(f[2 * j] - bf16lo(hp[j]), f[2 * j + 1] - bf16hi(hp[j]));
    }
    *reinterpret_cast<uint4*>(hi + image(row, c8)) = h;
    *reinterpret_cast<uint4*>(lo + image(row, c8)) = l;
}
// channels [c, c + 8) of a head, zero past `width`
__device__ __forceinline__ uint4 load_head(const __nv_bfloat16* head, int c, int width, bool vec) {
    if (vec && c + 8 <= width) return ld_cached(head + c);
    const unsigned short* p = reinterpret_cast<const unsigned short*>(head);
    uint32_t f[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
        f[j] = (c + 2 * j < width ? (uint32_t)p[c + 2 * j] : 0u) | (c + 2 * j + 1 < width ? (uint32_t)p[c + 2 * j + 1] << 16 : 0u);
    return make_uint4(f[0], f[1], f[2], f[3]);
}
// sums of channels [c, c + 8) of a head, zero past `width`
__device__ __forceinline__ void load_sums(const float* row, int c, int width, float (&f)[8]) {
    if (c + 8 <= width && (reinterpret_cast<uintptr_t>(row + c) & 15) == 0) {
        const float4 a = *reinterpret_cast<const float4*>(row + c), b = *reinterpret_cast<const float4*>(row + c + 4);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = c + j < width ? row[c + j] : 0.f;
    }
}
// rows [0, n) of a head into an image of `rows` rows and 8 cols8 channels, the rest zero: asynchronous copies where the head's
// channels come in whole 16-byte pieces
template <int THREADS = kThreads>
__device__ __forceinline__ void stage_head(unsigned char* dst, const __nv_bfloat16* head, int ld, int c0, int width, int n, int rows, int cols8) {
    const bool vec = ((reinterpret_cast<uintptr_t>(head) & 15) | (uintptr_t)(width & 7)) == 0;
    const uint32_t to = tc::smem_u32(dst);
    for (int i = threadIdx.x; i < rows * cols8; i += THREADS) {
        const int r = i / cols8, c8 = i - r * cols8, c = c0 + 8 * c8;
        const bool in = r < n && c < width;
        if (vec)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to + image(r, c8)), "l"(in ? head + (size_t)r * ld + c : head), "r"(in ? 16 : 0) : "memory");
        else
            *reinterpret_cast<uint4*>(dst + image(r, c8)) = in ? load_head(head + (size_t)r * ld, c, width, false) : make_uint4(0u, 0u, 0u, 0u);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
}
template <int N>
__device__ __forceinline__ void staged() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
// o[v ..] = f, channels past Dv left out
template <int N>
__device__ __forceinline__ void raw_output(const float (&f)[N], int v, float* __restrict__ o, int Dv) {
    if ((Dv & 3) == 0) {
#pragma unroll
        for (int j = 0; j < N; j += 4)
            if (v + j < Dv) *reinterpret_cast<float4*>(o + v + j) = make_float4(f[j], f[j + 1], f[j + 2], f[j + 3]);
    } else {
#pragma unroll
        for (int j = 0; j < N; ++j)
            if (v + j < Dv) o[v + j] = f[j];
    }
}
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
                   "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr) : "memory");
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_ld_cols(uint32_t taddr, uint32_t (&r)[16]) { tmem_ld16(taddr, r); }
__device__ __forceinline__ void tmem_ld_cols(uint32_t taddr, uint32_t (&r)[32]) { tc::tmem_ld32(taddr, r); }
// One row's value channels [k N, (k + 1) N) of a head: scale, norm over the head (all PARTS of it), weight, gate, output.  All
// threads call it.
template <int N, int PARTS>
__device__ __forceinline__ void head_output(const float (&f)[N], bool valid, int t, int k, int h, size_t row, const __nv_bfloat16* __restrict__ proj,
                                            __nv_bfloat16* __restrict__ out, int ld_out, const LinearShape& s) {
    __shared__ float part[PARTS][C];
    const __nv_bfloat16* gate = proj + row * s.ld + s.off_g + h * s.Dv;
    const bool vec = (s.Dv & 7) == 0;                                  // rows, off_g and ld_out are multiples of 8
    float ss = 0.f;
    if (valid) {
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (k * N + i < s.Dv) ss = fmaf(f[i], f[i], ss);
    }
    part[k][t] = ss;
    __syncthreads();
    if (!valid) return;
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < PARTS; ++i) ss += part[i][t];
    const float inv = s.scale / sqrtf(ss * s.scale * s.scale / (float)s.Dv + s.eps);
    __nv_bfloat16* dst = out + row * ld_out + h * s.Dv;
#pragma unroll
    for (int i = 0; i < N; i += 8) {
        const int v = k * N + i;
        if (v >= s.Dv) break;
        float g[8];
        if (vec) unpack8(ld_cached(gate + v), g);
        else
#pragma unroll
            for (int j = 0; j < 8; ++j) g[j] = v + j < s.Dv ? __bfloat162float(gate[v + j]) : 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const float w = s.norm == nullptr ? 1.0f : v + j < s.Dv ? __bfloat162float(s.norm[v + j]) : 0.f;
            g[j] = f[i + j] * inv * w * __fdividef(g[j], 1.0f + __expf(-g[j]));
        }
        if (vec) *reinterpret_cast<uint4*>(dst + v) = make_uint4(pack_bf16(g[0], g[1]), pack_bf16(g[2], g[3]), pack_bf16(g[4], g[5]), pack_bf16(g[6], g[7]));
        else
#pragma unroll
            for (int j = 0; j < 8; ++j)
                if (v + j < s.Dv) dst[v + j] = __float2bfloat16_rn(g[j]);
    }
}
__device__ __forceinline__ void fence_async_smem() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }
}  // namespace lt

// grid (chunks, heads, slices of VP value channels).  ws: [chunks][heads][D][Vp]
template <int VP, bool CH = false>
__global__ void __launch_bounds__(lt::kThreads, 2) linear_chunk_tc_kernel(const __nv_bfloat16* __restrict__ proj, float* __restrict__ ws, const LinearShape s,
                                                                        const RowPlan plan, int* error, const float* __restrict__ sums, int ld_sums) {
    using namespace lt;
    using Cf = Cfg<VP>;
    extern __shared__ unsigned char lt_smem[];
    RowEntry e;
    int t0;
    if (!locate_chunk<C>(plan, blockIdx.x, e, t0)) return;
    const uint32_t raw = tc::smem_u32(lt_smem), base = (raw + 1023u) & ~1023u;
    unsigned char* p0 = lt_smem + (base - raw);
    unsigned char *khi = p0, *klo = p0 + Cf::K_BYTES, *vs = p0 + 2 * Cf::K_BYTES;
    const uint32_t bar = base + 2 * Cf::K_BYTES + Cf::V_BYTES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(vs + Cf::V_BYTES + 8);
    volatile int* abort_s = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, v0 = blockIdx.z * VP, n = min(C, e.n - t0), steps = (n + 15) / 16;
    if (tid == 0) {
        tc::mbar_init(bar, 1);
        *abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc::smem_u32(tmem_slot)), "r"(VP) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    const float* pw = CH ? nullptr : s.powers + (size_t)h * (kLinearPowers + 1);
    const float* b0 = CH ? sums + (size_t)(e.row0 + t0) * ld_sums + h * s.D : nullptr;
    const __nv_bfloat16 *k0 = proj + (size_t)(e.row0 + t0) * s.ld + s.off_k + h * s.D, *w0 = proj + (size_t)(e.row0 + t0) * s.ld + s.off_v + h * s.Dv;
    stage_head(vs, w0, s.ld, v0, s.Dv, n, steps * 16, VP / 8);
    const bool vk = (reinterpret_cast<uintptr_t>(k0) & 15) == 0;
    if constexpr (CH) {
        float end[8];                                                 // a thread stays with its eight channels
        const int c = 8 * (tid & 15);
        lt::load_sums(b0 + (size_t)(n - 1) * ld_sums, c, s.D, end);
        for (int r = tid >> 4; r < steps * 16; r += kThreads / 16) {
            float f[8], b[8];
            unpack8(r < n && c < s.D ? load_head(k0 + (size_t)r * s.ld, c, s.D, vk) : make_uint4(0u, 0u, 0u, 0u), f);
            lt::load_sums(b0 + (size_t)min(r, n - 1) * ld_sums, c, s.D, b);
#pragma unroll
            for (int j = 0; j < 8; ++j) f[j] *= __expf(end[j] - b[j]);
            put_pair(khi, klo, r, tid & 15, f);
        }
    } else {
        constexpr int U = 8;
        for (int i0 = tid; i0 < steps * 16 * 16; i0 += U * kThreads) {   // all 128 key channels: the product has 128 rows
            uint4 x[U];
            float a[U];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * kThreads, r = i >> 4, c = 8 * (i & 15);
                const bool in = r < n && c < s.D;
                x[u] = in ? load_head(k0 + (size_t)r * s.ld, c, s.D, vk) : make_uint4(0u, 0u, 0u, 0u);
                a[u] = in ? pw[n - 1 - r] : 0.f;
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * kThreads;
                float f[8];
                unpack8(x[u], f);
#pragma unroll
                for (int j = 0; j < 8; ++j) f[j] *= a[u];
                if (i < steps * 16 * 16) put_pair(khi, klo, i >> 4, i & 15, f);
            }
        }
    }
    staged<0>();
    fence_async_smem();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    if (tid == 0) {
        constexpr uint32_t kDesc = at::instr_desc(128, VP) | (1u << 15) | (1u << 16);      // rows contracted in both operands
        const uint64_t da[2] = {at::umma_desc_mn(base, BOX, 1024u), at::umma_desc_mn(base + Cf::K_BYTES, BOX, 1024u)};
        const uint64_t db = at::umma_desc_mn(base + 2 * Cf::K_BYTES, BOX, 1024u);
        for (int part = 0; part < 2; ++part)
            for (int k = 0; k < steps; ++k)
                at::umma_d(tmem, da[part] + (uint64_t)(k * (2048 >> 4)), db + (uint64_t)(k * (2048 >> 4)), kDesc, (part | k) != 0 ? 1u : 0u);
        tc::umma_commit(bar);
    }
    const bool ok = __all_sync(0xffffffffu, tc::mbar_wait(bar, 0, abort_s));      // a warp reads tensor memory as one
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    if (ok) {
        const int d = (warp & 3) * 32 + lane, hf = warp >> 2;
        float* out = ws + ((size_t)blockIdx.x * s.heads + h) * s.head_floats() + (size_t)d * s.Vp;
#pragma unroll
        for (int c0 = 0; c0 < Cf::HALF; c0 += 32) {
            uint32_t r[32];
            tc::tmem_ld32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)(hf * Cf::HALF + c0), r);
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
                const int v = v0 + hf * Cf::HALF + c0 + j;
                if (d < s.D && v < s.Vp) *reinterpret_cast<uint4*>(out + v) = make_uint4(r[j], r[j + 1], r[j + 2], r[j + 3]);
            }
            __syncwarp();
        }
    } else if (error != nullptr) {
        atomicExch(error, 1);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(VP) : "memory");
    }
}

// grid (chunks, heads, slices of VP value channels)
template <int VP, bool HEAD = false>
__global__ void __launch_bounds__(lt::kAttendThreads, 1) linear_attend_tc_kernel(const __nv_bfloat16* __restrict__ proj, const float* __restrict__ ws, float* __restrict__ o,
                                                                         int ld_o, const LinearShape s, const RowPlan plan, int* error,
                                                                         __nv_bfloat16* __restrict__ out, int ld_out) {
    using namespace lt;
    using Cf = Cfg<VP>;
    constexpr int TMEM = 512, THREADS = kAttendThreads, COLS = VP / 4;
    extern __shared__ unsigned char lt_smem[];
    __shared__ float pw[C + 1];
    RowEntry e;
    int t0;
    if (!locate_chunk<C>(plan, blockIdx.x, e, t0)) return;
    const uint32_t raw = tc::smem_u32(lt_smem), base = (raw + 1023u) & ~1023u;
    unsigned char* p0 = lt_smem + (base - raw);
    constexpr int K_OFF = Cf::K_BYTES, V_OFF = 2 * Cf::K_BYTES, SH_OFF = V_OFF + Cf::V_BYTES, SL_OFF = SH_OFF + Cf::V_BYTES, BAR_OFF = SL_OFF + Cf::V_BYTES;
    const uint32_t pbar = base + BAR_OFF, obar = pbar + 8;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(p0 + BAR_OFF + 16);
    volatile int* abort_s = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, v0 = blockIdx.z * VP, n = min(C, e.n - t0), steps = (n + 15) / 16;
    const int dsteps = (s.D + 15) / 16;
    const bool state = e.pos0 + t0 > 0;                               // the first chunk of a sequence starts from zero
    if (tid == 0) {
        tc::mbar_init(pbar, 1);
        tc::mbar_init(obar, 1);
        *abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc::smem_u32(tmem_slot)), "r"(TMEM) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    for (int i = tid; i <= C; i += THREADS) pw[i] = s.powers[(size_t)h * (kLinearPowers + 1) + i];
    const __nv_bfloat16* row = proj + (size_t)(e.row0 + t0) * s.ld;
    const __nv_bfloat16 *q0 = row + s.off_q + h * s.D, *k0 = row + s.off_k + h * s.D, *w0 = row + s.off_v + h * s.Dv;
    stage_head<THREADS>(p0, q0, s.ld, 0, s.D, n, C, 2 * dsteps);               // rows past n: zero, every row of the product is computed
    stage_head<THREADS>(p0 + K_OFF, k0, s.ld, 0, s.D, n, C, 2 * dsteps);
    stage_head<THREADS>(p0 + V_OFF, w0, s.ld, v0, s.Dv, n, steps * 16, VP / 8);
    if (state) {
        const float* S = ws + ((size_t)blockIdx.x * s.heads + h) * s.head_floats();
        constexpr int U = 4;
        const int all = dsteps * 16 * (VP / 8);
        for (int i0 = tid; i0 < all; i0 += U * THREADS) {
            float4 a[U], b[U];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * THREADS, d = i / (VP / 8), v = v0 + 8 * (i % (VP / 8));
                const bool in = i < all && d < s.D;
                a[u] = in && v < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)d * s.Vp + v) : make_float4(0.f, 0.f, 0.f, 0.f);
                b[u] = in && v + 4 < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)d * s.Vp + v + 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * THREADS;
                const float f[8] = {a[u].x, a[u].y, a[u].z, a[u].w, b[u].x, b[u].y, b[u].z, b[u].w};
                if (i < all) put_pair(p0 + SH_OFF, p0 + SL_OFF, i / (VP / 8), i % (VP / 8), f);
            }
        }
    }
    staged<1>();
    fence_async_smem();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    if (tid == 0) {
        constexpr uint32_t kDesc = at::instr_desc(128, 128);
        for (int k = 0; k < dsteps; ++k)
            at::umma_d(tmem, tc::umma_desc(base + (k >> 2) * BOX) + (uint64_t)((k & 3) * 2), tc::umma_desc(base + K_OFF + (k >> 2) * BOX) + (uint64_t)((k & 3) * 2), kDesc,
                       k != 0 ? 1u : 0u);
        tc::umma_commit(pbar);
    }
    staged<0>();
    fence_async_smem();
    bool ok = __all_sync(0xffffffffu, tc::mbar_wait(pbar, 0, abort_s));     // a warp accesses tensor memory as one
    if (!ok) *abort_s = 1;
    __syncwarp();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const int t = (warp & 3) * 32 + lane, part = warp >> 2;           // TMEM lane = token; which quarter of the columns
    const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    {
        uint32_t r[32], hi[16], lo[16];
        tc::tmem_ld32(lanes + (uint32_t)(part * 32), r);
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
            const int u = part * 32 + j;
            const float a = u <= t ? __uint_as_float(r[j]) * pw[t - u] : 0.f, b = u + 1 <= t ? __uint_as_float(r[j + 1]) * pw[t - u - 1] : 0.f;
            hi[j >> 1] = pack_bf16(a, b);
            lo[j >> 1] = pack_bf16(a - bf16lo(hi[j >> 1]), b - bf16hi(hi[j >> 1]));
        }
        wt::tmem_st16(lanes + (uint32_t)(PH_COL + part * 16), hi);
        wt::tmem_st16(lanes + (uint32_t)(PL_COL + part * 16), lo);
    }
    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (tid == 0 && *abort_s == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        constexpr uint32_t kDesc = at::instr_desc(128, VP) | (1u << 16);
        const uint64_t dv = at::umma_desc_mn(base + V_OFF, BOX, 1024u);
        const uint64_t ds[2] = {at::umma_desc_mn(base + SH_OFF, BOX, 1024u), at::umma_desc_mn(base + SL_OFF, BOX, 1024u)};
        if (state)
            for (int part = 0; part < 2; ++part)
                for (int k = 0; k < dsteps; ++k)
                    at::umma_d(tmem + O1_COL, tc::umma_desc(base + (k >> 2) * BOX) + (uint64_t)((k & 3) * 2), ds[part] + (uint64_t)(k * (2048 >> 4)), kDesc,
                               (part | k) != 0 ? 1u : 0u);
        for (int part = 0; part < 2; ++part)
            for (int k = 0; k < steps; ++k)
                wt::umma_ts(tmem + O2_COL, tmem + (uint32_t)((part ? PL_COL : PH_COL) + 8 * k), dv + (uint64_t)(k * (2048 >> 4)), kDesc, (part | k) != 0 ? 1u : 0u);
        tc::umma_commit(obar);
    }
    ok = __all_sync(0xffffffffu, ok && tc::mbar_wait(obar, 0, abort_s));
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    float f[COLS];
    if (ok) {
        uint32_t x[COLS], y[COLS];
        const float a = pw[t + 1];
        tmem_ld_cols(lanes + (uint32_t)(O2_COL + part * COLS), y);
        if (state) tmem_ld_cols(lanes + (uint32_t)(O1_COL + part * COLS), x);
#pragma unroll
        for (int j = 0; j < COLS; ++j) f[j] = state ? fmaf(a, __uint_as_float(x[j]), __uint_as_float(y[j])) : __uint_as_float(y[j]);
    } else if (tid == 0 && error != nullptr) {
        atomicExch(error, 1);
    }
    if constexpr (HEAD) head_output<COLS, 4>(f, ok && t < n, t, part, h, (size_t)(e.row0 + t0 + t), proj, out, ld_out, s);
    else if (ok && t < n) raw_output(f, v0 + part * COLS, o + (size_t)(e.row0 + t0 + t) * ld_o + h * s.Dv, s.Dv);
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TMEM) : "memory");
    }
}

// The same with decays per key channel.  Images: Q high | Q low | K high | K low | V; the state's pair takes the place of K's once P is
// there.  P V and Q S add up in one accumulator.  HEAD: normed and gated bf16 rows instead of o.
template <int VP, bool HEAD>
__global__ void __launch_bounds__(lt::kAttendThreads, 1) linear_attend_ch_tc_kernel(const __nv_bfloat16* __restrict__ proj, const float* __restrict__ ws,
                                                                            const float* __restrict__ sums, int ld_sums, float* __restrict__ o, int ld_o,
                                                                            __nv_bfloat16* __restrict__ out, int ld_out, const LinearShape s, const RowPlan plan,
                                                                            int* error) {
    using namespace lt;
    using Cf = Cfg<VP>;
    constexpr int TMEM = 512, THREADS = kAttendThreads, COLS = VP / 4, QH_OFF = 0, QL_OFF = Cf::K_BYTES, KH_OFF = 2 * Cf::K_BYTES, KL_OFF = 3 * Cf::K_BYTES, V_OFF = 4 * Cf::K_BYTES,
                  BAR_OFF = V_OFF + Cf::V_BYTES;
    extern __shared__ unsigned char lt_smem[];
    RowEntry e;
    int t0;
    if (!locate_chunk<C>(plan, blockIdx.x, e, t0)) return;
    const uint32_t raw = tc::smem_u32(lt_smem), base = (raw + 1023u) & ~1023u;
    unsigned char* p0 = lt_smem + (base - raw);
    const uint32_t pbar = base + BAR_OFF, obar = pbar + 8;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(p0 + BAR_OFF + 16);
    volatile int* abort_s = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, v0 = blockIdx.z * VP, n = min(C, e.n - t0), steps = (n + 15) / 16;
    const int dsteps = (s.D + 15) / 16;
    const bool state = e.pos0 + t0 > 0;                               // the first chunk of a sequence starts from zero
    if (tid == 0) {
        tc::mbar_init(pbar, 1);
        tc::mbar_init(obar, 1);
        *abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc::smem_u32(tmem_slot)), "r"(TMEM) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    const __nv_bfloat16* row = proj + (size_t)(e.row0 + t0) * s.ld;
    const __nv_bfloat16 *q0 = row + s.off_q + h * s.D, *k0 = row + s.off_k + h * s.D, *w0 = row + s.off_v + h * s.Dv;
    const float *b0 = sums + (size_t)(e.row0 + t0) * ld_sums + h * s.D, *b_end = b0 + (size_t)(n - 1) * ld_sums;
    stage_head<THREADS>(p0 + V_OFF, w0, s.ld, v0, s.Dv, n, steps * 16, VP / 8);
    const int c8 = tid & 15, c = 8 * c8;                              // a thread stays with its eight channels
    const bool vq = ((reinterpret_cast<uintptr_t>(q0) | reinterpret_cast<uintptr_t>(k0)) & 15) == 0;
    constexpr int ROWS = C * 16 / THREADS;
    uint4 qv[ROWS], kv[ROWS];
    float bv[ROWS][8], mid[8];
    load_sums(b_end, c, s.D, mid);
#pragma unroll
    for (int u = 0; u < ROWS; ++u) {                                  // rows past n: zero, every row of the product is computed
        const int r = (tid >> 4) + u * (THREADS / 16);
        const bool in = r < n && c < s.D;
        load_sums(b0 + (size_t)min(r, n - 1) * ld_sums, c, s.D, bv[u]);
        qv[u] = in ? load_head(q0 + (size_t)r * s.ld, c, s.D, vq) : make_uint4(0u, 0u, 0u, 0u);
        kv[u] = in ? load_head(k0 + (size_t)r * s.ld, c, s.D, vq) : make_uint4(0u, 0u, 0u, 0u);
    }
    const bool strong = __syncthreads_or(tid < s.D && b_end[tid < s.D ? tid : 0] < -kMaxLoss) != 0;
#pragma unroll
    for (int j = 0; j < 8; ++j) mid[j] = strong ? 0.f : 0.5f * mid[j];
    if (c8 < 2 * dsteps) {
#pragma unroll
        for (int u = 0; u < ROWS; ++u) {
            const int r = (tid >> 4) + u * (THREADS / 16);
            float f[8], k[8];
            unpack8(qv[u], f);
            unpack8(kv[u], k);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                f[j] *= __expf(bv[u][j] - mid[j]);
                k[j] = strong ? 0.f : k[j] * __expf(mid[j] - bv[u][j]);
            }
            put_pair(p0 + QH_OFF, p0 + QL_OFF, r, c8, f);
            put_pair(p0 + KH_OFF, p0 + KL_OFF, r, c8, k);
        }
    }
    fence_async_smem();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    // step k of an image whose channels are contracted
    auto k_desc = [&](int off, int k) { return tc::umma_desc(base + off + (k >> 2) * BOX) + (uint64_t)((k & 3) * 2); };
    if (tid == 0 && !strong) {
        constexpr uint32_t kDesc = at::instr_desc(128, 128);
        for (int part = 0; part < 3; ++part)                          // high high, high low, low high
            for (int k = 0; k < dsteps; ++k)
                at::umma_d(tmem, k_desc(part == 2 ? QL_OFF : QH_OFF, k), k_desc(part == 1 ? KL_OFF : KH_OFF, k), kDesc, (part | k) != 0 ? 1u : 0u);
        tc::umma_commit(pbar);
    }
    // the state, requested while P is computed
    constexpr int ITEMS = 128 * (VP / 8) / THREADS;
    float4 sa[ITEMS], sb[ITEMS];
    float se[ITEMS];
    if (state) {
        const float* S = ws + ((size_t)blockIdx.x * s.heads + h) * s.head_floats();
#pragma unroll
        for (int u = 0; u < ITEMS; ++u) {
            const int i = tid + u * THREADS, d = i / (VP / 8), v = v0 + 8 * (i % (VP / 8));
            const bool in = d < s.D;
            sa[u] = in && v < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)d * s.Vp + v) : make_float4(0.f, 0.f, 0.f, 0.f);
            sb[u] = in && v + 4 < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)d * s.Vp + v + 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            se[u] = in && !strong ? __expf(0.5f * b_end[d]) : 1.0f;
        }
    }
    bool ok = strong || __all_sync(0xffffffffu, tc::mbar_wait(pbar, 0, abort_s));     // a warp accesses tensor memory as one
    if (!ok) *abort_s = 1;
    __syncwarp();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const int t = (warp & 3) * 32 + lane, part = warp >> 2;           // TMEM lane = token; which quarter of the columns
    const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    {
        uint32_t r[32], hi[16], lo[16];
        const int u0 = part * 32;
        if (!strong) {
            tc::tmem_ld32(lanes + (uint32_t)u0, r);
        } else {
            float acc[32];
#pragma unroll
            for (int j = 0; j < 32; ++j) acc[j] = 0.f;
            const int tt = min(t, n - 1);
            for (int d = 0; d < s.D; ++d) {
                const float q = __bfloat162float(q0[(size_t)tt * s.ld + d]), b = b0[(size_t)tt * ld_sums + d];
#pragma unroll
                for (int j = 0; j < 32; ++j)
                    if (u0 + j <= tt)
                        acc[j] = fmaf(q * __bfloat162float(k0[(size_t)(u0 + j) * s.ld + d]), __expf(b - b0[(size_t)(u0 + j) * ld_sums + d]), acc[j]);
            }
            __syncwarp();
#pragma unroll
            for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(acc[j]);
        }
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
            const int u = u0 + j;
            const float a = u <= t ? __uint_as_float(r[j]) : 0.f, b = u + 1 <= t ? __uint_as_float(r[j + 1]) : 0.f;
            hi[j >> 1] = pack_bf16(a, b);
            lo[j >> 1] = pack_bf16(a - bf16lo(hi[j >> 1]), b - bf16hi(hi[j >> 1]));
        }
        wt::tmem_st16(lanes + (uint32_t)(PH_COL + u0 / 2), hi);
        wt::tmem_st16(lanes + (uint32_t)(PL_COL + u0 / 2), lo);
    }
    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
    if (state && ok) {                                                // P is complete: K's images are free
#pragma unroll
        for (int u = 0; u < ITEMS; ++u) {
            const int i = tid + u * THREADS;
            const float x = se[u], f[8] = {x * sa[u].x, x * sa[u].y, x * sa[u].z, x * sa[u].w, x * sb[u].x, x * sb[u].y, x * sb[u].z, x * sb[u].w};
            if (i < dsteps * 16 * (VP / 8)) put_pair(p0 + KH_OFF, p0 + KL_OFF, i / (VP / 8), i % (VP / 8), f);
        }
    }
    staged<0>();
    fence_async_smem();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (tid == 0 && *abort_s == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        constexpr uint32_t kDesc = at::instr_desc(128, VP) | (1u << 16);
        const uint64_t dv = at::umma_desc_mn(base + V_OFF, BOX, 1024u);
        const uint64_t ds[2] = {at::umma_desc_mn(base + KH_OFF, BOX, 1024u), at::umma_desc_mn(base + KL_OFF, BOX, 1024u)};
        for (int part = 0; part < 2; ++part)
            for (int k = 0; k < steps; ++k)
                wt::umma_ts(tmem + O2_COL, tmem + (uint32_t)((part ? PL_COL : PH_COL) + 8 * k), dv + (uint64_t)(k * (2048 >> 4)), kDesc, (part | k) != 0 ? 1u : 0u);
        if (state)
            for (int part = 0; part < 3; ++part)
                for (int k = 0; k < dsteps; ++k)
                    at::umma_d(tmem + O2_COL, k_desc(part == 2 ? QL_OFF : QH_OFF, k), (part == 1 ? ds[1] : ds[0]) + (uint64_t)(k * (2048 >> 4)), kDesc, 1u);
        tc::umma_commit(obar);
    }
    ok = __all_sync(0xffffffffu, ok && tc::mbar_wait(obar, 0, abort_s));
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    float f[COLS];
    if (ok) {
        uint32_t y[COLS];
        tmem_ld_cols(lanes + (uint32_t)(O2_COL + part * COLS), y);
#pragma unroll
        for (int j = 0; j < COLS; ++j) f[j] = __uint_as_float(y[j]);
    } else if (tid == 0 && error != nullptr) {
        atomicExch(error, 1);
    }
    if constexpr (HEAD) head_output<COLS, 4>(f, ok && t < n, t, part, h, (size_t)(e.row0 + t0 + t), proj, out, ld_out, s);
    else if (ok && t < n) raw_output(f, v0 + part * COLS, o + (size_t)(e.row0 + t0 + t) * ld_o + h * s.Dv, s.Dv);
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TMEM) : "memory");
    }
}

}  // namespace efm
