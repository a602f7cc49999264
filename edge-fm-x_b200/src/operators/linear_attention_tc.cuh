// Many-row form of the decayed linear attention (linear_attention.cuh) on the 5th-generation tensor cores, chunks of 128 tokens:
//   linear_chunk_tc    U = K'^T V, K' the keys times the decay that is left to the end of the chunk
//   linear_attend_tc   P = Q K^T masked and decayed, O = decay * (Q S) + P V, S the state the chunk starts from
// q, k and v enter as they are, in bf16.  What is not exact in bf16 -- K', P and S -- enters as a bf16 pair high +
// low (16 bits of mantissa); products accumulate in fp32 and the states in memory are fp32.
// Operands are staged by the threads, which apply decay and the split on the way, in the 128-byte-swizzled layout that TMA would
// write: [row][64 channels] boxes of 128 bytes a row.  The same image serves as a K-major operand (channels contracted) and as an
// MN-major one (rows contracted).  P goes from tensor memory to tensor memory.  Every mbarrier wait is bounded and raises *error.
// Head sizes up to 128 key channels; value channels in slices of VP (grid.z).
#pragma once
#include "attention_tc.cuh"
#include "linear_attention.cuh"
#include "window_attention_tc.cuh"

namespace efm {

namespace lt {
constexpr int C = kLinearChunkTc, kThreads = 256;
constexpr int BOX = C * 128;                                  // bytes of a box of 64 channels
template <int VP>
struct Cfg {
    static constexpr int V_BYTES = BOX * (VP / 64), K_BYTES = BOX * 2;
    static constexpr size_t CHUNK_SMEM = 2 * K_BYTES + V_BYTES + 1024 + 64;
    static constexpr size_t ATTEND_SMEM = 2 * K_BYTES + V_BYTES + 2 * V_BYTES + 1024 + 64;
    static constexpr int HALF = VP / 2;
};
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
// rows [0, n) of a head into an image of `rows` rows and 8 cols8 channels, the rest zero: asynchronous copies where the head's
// channels come in whole 16-byte pieces
__device__ __forceinline__ void stage_head(unsigned char* dst, const __nv_bfloat16* head, int ld, int c0, int width, int n, int rows, int cols8) {
    const bool vec = ((reinterpret_cast<uintptr_t>(head) & 15) | (uintptr_t)(width & 7)) == 0;
    const uint32_t to = tc::smem_u32(dst);
    for (int i = threadIdx.x; i < rows * cols8; i += kThreads) {
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
__device__ __forceinline__ void fence_async_smem() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }
}  // namespace lt

// grid (chunks, heads, slices of VP value channels).  ws: [chunks][heads][D][Vp]
template <int VP>
__global__ void __launch_bounds__(lt::kThreads, 2) linear_chunk_tc_kernel(const __nv_bfloat16* __restrict__ proj, float* __restrict__ ws, const LinearShape s,
                                                                        const RowPlan plan, int* error) {
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
    const float* pw = s.powers + (size_t)h * (kLinearPowers + 1);
    const __nv_bfloat16 *k0 = proj + (size_t)(e.row0 + t0) * s.ld + s.off_k + h * s.D, *w0 = proj + (size_t)(e.row0 + t0) * s.ld + s.off_v + h * s.Dv;
    stage_head(vs, w0, s.ld, v0, s.Dv, n, steps * 16, VP / 8);
    const bool vk = (reinterpret_cast<uintptr_t>(k0) & 15) == 0;
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
template <int VP>
__global__ void __launch_bounds__(lt::kThreads, 1) linear_attend_tc_kernel(const __nv_bfloat16* __restrict__ proj, const float* __restrict__ ws, float* __restrict__ o,
                                                                         int ld_o, const LinearShape s, const RowPlan plan, int* error) {
    using namespace lt;
    using Cf = Cfg<VP>;
    constexpr int TMEM = 512;
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
    for (int i = tid; i <= C; i += kThreads) pw[i] = s.powers[(size_t)h * (kLinearPowers + 1) + i];
    const __nv_bfloat16* row = proj + (size_t)(e.row0 + t0) * s.ld;
    const __nv_bfloat16 *q0 = row + s.off_q + h * s.D, *k0 = row + s.off_k + h * s.D, *w0 = row + s.off_v + h * s.Dv;
    stage_head(p0, q0, s.ld, 0, s.D, n, C, 2 * dsteps);               // rows past n: zero, every row of the product is computed
    stage_head(p0 + K_OFF, k0, s.ld, 0, s.D, n, C, 2 * dsteps);
    stage_head(p0 + V_OFF, w0, s.ld, v0, s.Dv, n, steps * 16, VP / 8);
    if (state) {
        const float* S = ws + ((size_t)blockIdx.x * s.heads + h) * s.head_floats();
        constexpr int U = 4;
        const int all = dsteps * 16 * (VP / 8);
        for (int i0 = tid; i0 < all; i0 += U * kThreads) {
            float4 a[U], b[U];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * kThreads, d = i / (VP / 8), v = v0 + 8 * (i % (VP / 8));
                const bool in = i < all && d < s.D;
                a[u] = in && v < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)d * s.Vp + v) : make_float4(0.f, 0.f, 0.f, 0.f);
                b[u] = in && v + 4 < s.Vp ? *reinterpret_cast<const float4*>(S + (size_t)d * s.Vp + v + 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * kThreads;
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
    const int t = (warp & 3) * 32 + lane, hf = warp >> 2;             // TMEM lane = token; which half of the columns
    const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
#pragma unroll
    for (int c0 = 0; c0 < 64; c0 += 32) {
        uint32_t r[32], hi[16], lo[16];
        tc::tmem_ld32(lanes + (uint32_t)(hf * 64 + c0), r);
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
            const int u = hf * 64 + c0 + j;
            const float a = u <= t ? __uint_as_float(r[j]) * pw[t - u] : 0.f, b = u + 1 <= t ? __uint_as_float(r[j + 1]) * pw[t - u - 1] : 0.f;
            hi[j >> 1] = pack_bf16(a, b);
            lo[j >> 1] = pack_bf16(a - bf16lo(hi[j >> 1]), b - bf16hi(hi[j >> 1]));
        }
        wt::tmem_st16(lanes + (uint32_t)(PH_COL + hf * 32 + c0 / 2), hi);
        wt::tmem_st16(lanes + (uint32_t)(PL_COL + hf * 32 + c0 / 2), lo);
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
    if (ok) {
        float* dst = o + (size_t)(e.row0 + t0 + t) * ld_o + h * s.Dv;
        const float a = pw[t + 1];
        const bool vec = (s.Dv & 3) == 0;
#pragma unroll
        for (int c0 = 0; c0 < Cf::HALF; c0 += 32) {
            uint32_t x[32], y[32];
            tc::tmem_ld32(lanes + (uint32_t)(O2_COL + hf * Cf::HALF + c0), y);
            if (state) tc::tmem_ld32(lanes + (uint32_t)(O1_COL + hf * Cf::HALF + c0), x);
            const bool in = t < n;
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
                const int v = v0 + hf * Cf::HALF + c0 + j;
                float f[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) f[k] = state ? fmaf(a, __uint_as_float(x[j + k]), __uint_as_float(y[j + k])) : __uint_as_float(y[j + k]);
                if (vec) {
                    if (in && v < s.Dv) *reinterpret_cast<float4*>(dst + v) = make_float4(f[0], f[1], f[2], f[3]);
                } else {
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        if (in && v + k < s.Dv) dst[v + k] = f[k];
                }
            }
            __syncwarp();
        }
    } else if (tid == 0 && error != nullptr) {
        atomicExch(error, 1);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TMEM) : "memory");
    }
}

}  // namespace efm
