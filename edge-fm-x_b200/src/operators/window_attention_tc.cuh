// Many-row form of the windowed attention (window_attention.cuh) on the 5th-generation tensor cores: the structure of
// attention_tc.cuh (S = Q K^T and O_tile = P V as tcgen05.mma with TMEM accumulators, operands by TMA, online softmax with
// two threads per query row) over a paged cache, with the per-head multiplier and the distance bias applied to the scores
// in fp32.  A key tile is exactly one 64-token page: its TMA coordinate is the page number of the sequence's table, or the
// place of the page in a workspace of keys and values expanded for this pass (latent attention).
// Keys may come from two tensors: DP channels per kv head, and RP more that all heads share (a rotated part); the query rows
// are split the same way.  Channels that a tensor does not have are filled with zeros by TMA.
// Block = 128 rows of one entry x one head x VP value channels, 256 threads.  Wider values take several blocks, each of which
// computes the scores for itself.  Late rows see the most keys: blocks take them first, and the second half of what is resident at a
// time from the other end, so that an SM's two blocks are a long and a short one.  Rows of the tile that belong to the next entry are computed and
// not stored.  The weights enter P V as a bf16 pair high + low (16 bits of mantissa), written straight into tensor memory.
// The products run behind the softmax: S of the next tile is issued as soon as every thread holds its scores, and P V of a tile is
// folded into the registers one tile later, while the next weights are already on their way.
// Every mbarrier wait is bounded and raises *error.
#pragma once
#include "attention_tc.cuh"
#include "window_attention.cuh"

namespace efm {

namespace wt {

constexpr int BM = 128, BN = kPageTokens, kThreads = 256, kMaxTiles = 1024;

template <int DP, int VP, int RP = 0>
struct Cfg {
    static constexpr int QB = (DP + RP) / 64, VB = VP / 64;  // 64-channel boxes per row
    // Wide keys have one buffer: the next tile is requested when S of this one is done and has the softmax's time to arrive,
    // and two blocks fit on an SM.
    static constexpr int KBUF = DP + RP > 128 ? 1 : 2;
    static constexpr int Q_BYTES = BM * 128 * QB, K_BYTES = BN * 128 * QB, V_BYTES = BN * 128 * VB;
    static constexpr int P_COL = 64, O_COL = 128;
    static constexpr int TMEM_COLS = 256;                    // S (64 columns) | P high, P low (32 each) | O tile, power of two
    static constexpr int HALF = VP / 2;
    static constexpr size_t SMEM = (size_t)Q_BYTES + KBUF * K_BYTES + 2 * V_BYTES + 2 * BM * 4 + 128 + kMaxTiles * 4 + 1024;
};

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr), "r"(r[0]), "r"(r[1]),
                 "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]),
                 "r"(r[14]), "r"(r[15]) : "memory");
}
// D = A . B with A in tensor memory (bf16 pairs along K in 32-bit columns) and B by shared-memory descriptor
__device__ __forceinline__ void umma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n"
        "}\n"
        ::"r"(tmem_d), "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate) : "memory");
}

}  // namespace wt

struct WindowTcMaps {
    CUtensorMap q, k, v;              // [rows][heads][channels]
    CUtensorMap qr, kr;               // RP > 0: rotated parts, [rows][heads][channels] and [rows][1][channels]
};

// SIG: weights sigmoid(score + shift[h]); no maximum, no denominator, and P V of all tiles accumulates in tensor memory.
template <int DP, int VP, int RP, bool KEEP, bool SIG = false>
__global__ void __launch_bounds__(wt::kThreads, 2) window_attention_tc_kernel(const __grid_constant__ WindowTcMaps maps, __nv_bfloat16* __restrict__ out,
                                                                           int ld_out, const WindowAttnShape s, const RowPlan plan,
                                                                           const RowTile* __restrict__ tiles, int n_tiles_all, int first_wave, int workspace,
                                                                           int* error) {
    using namespace wt;
    using at::instr_desc;
    using at::tma_load_3d;
    using at::umma_d;
    using tc::mbar_expect_tx;
    using tc::mbar_init;
    using tc::mbar_wait;
    using tc::smem_u32;
    using tc::umma_commit;
    using tc::umma_desc;
    using C = Cfg<DP, VP, RP>;
    extern __shared__ unsigned char wt_smem[];
    const uint32_t raw = smem_u32(wt_smem);
    const uint32_t base = (raw + 1023u) & ~1023u;
    unsigned char* base_ptr = wt_smem + (base - raw);
    const uint32_t sQ = base, sK = sQ + C::Q_BYTES, sV = sK + C::KBUF * C::K_BYTES;
    constexpr int XCH = C::Q_BYTES + C::KBUF * C::K_BYTES + 2 * C::V_BYTES;
    float* xch = reinterpret_cast<float*>(base_ptr + XCH);                       // [2][BM]
    const uint32_t bars = sV + 2 * C::V_BYTES + 2 * BM * 4;
    const uint32_t qfull = bars, kfull0 = bars + 8, vfull0 = bars + 24, sbar = bars + 40, obar = bars + 48;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(base_ptr + XCH + 2 * BM * 4 + 56);
    volatile int* abort_s = reinterpret_cast<volatile int*>(tmem_slot + 1);
    int* pages = reinterpret_cast<int*>(base_ptr + XCH + 2 * BM * 4 + 128);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row = (warp & 3) * 32 + lane, hf = warp >> 2;       // TMEM lane = query row; which half of the columns
    // grid.x = tiles x (heads x slices); see the top
    const int slices = (s.Vp + VP - 1) / VP, per_tile = s.H * slices;
    const int rank = (int)blockIdx.x < first_wave ? (int)blockIdx.x : (int)gridDim.x - 1 - ((int)blockIdx.x - first_wave);
    const int bx = n_tiles_all - 1 - rank / per_tile, h = rank % per_tile / slices, g = h / (s.H / s.G);
    const int v0 = rank % slices * VP;                            // first value channel
    RowEntry e;
    int r0;
    if (tiles != nullptr) { const RowTile t = tiles[bx]; e = plan.entry(t.entry); r0 = t.row; }
    else { e = plan.one; r0 = bx * BM; }
    const int nq = min(BM, e.n - r0), p0 = e.pos0 + r0;           // rows of the tile, position of the first
    const int i_pos = p0 + row;
    const bool valid = row < nq;
    const int lo = s.window > 0 ? max(0, i_pos - s.window + 1) : 0, hi = i_pos + 1;
    const int first = s.window > 0 ? max(0, p0 - s.window + 1) : 0, lo_max = s.window > 0 ? max(0, p0 + nq - s.window) : 0, hi_min = p0 + 1;
    // tiles: the pages with kept first tokens ahead of the window's first page, then the pages of the window
    const int pg0 = first / BN, nk = KEEP && s.window > 0 ? min((min(s.keep, first) + BN - 1) / BN, pg0) : 0, keep = KEEP ? s.keep : 0;
    const int ntiles = min(nk + (p0 + nq - 1) / BN - pg0 + 1, kMaxTiles);
    auto tile_page = [&](int i) { return KEEP && i < nk ? i : pg0 + i - nk; };

    if (tid == 0) {
        mbar_init(qfull, 1); mbar_init(kfull0, 1); mbar_init(kfull0 + 8, 1); mbar_init(vfull0, 1); mbar_init(vfull0 + 8, 1); mbar_init(sbar, 1); mbar_init(obar, 1);
        *abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(C::TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    for (int i = tid; i < ntiles; i += kThreads) 
        pages[i] = workspace ? e.ws0 + tile_page(i) * BN : plan.page_table[(size_t)e.table * plan.max_pages + tile_page(i)] * BN;
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;

    constexpr uint32_t kDescS = instr_desc(BM, BN);
    constexpr uint32_t kDescO = instr_desc(BM, VP) | (1u << 16);
    const uint64_t vdesc[2] = {at::umma_desc_mn(sV, (uint32_t)(BN * 128), 1024u), at::umma_desc_mn(sV + C::V_BYTES, (uint32_t)(BN * 128), 1024u)};
    constexpr float kLog2e = 1.4426950408889634f;
    const float f2 = head_multiplier(s, h) * kLog2e;
    const float b2 = (s.bias ? distance_slope(h, s.H) : 0.f) * kLog2e, shift2 = SIG ? __bfloat162float(s.shift[h]) * kLog2e : 0.f;
    float o[C::HALF];
#pragma unroll
    for (int i = 0; i < C::HALF; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;

    int last_k[2] = {-1, -1}, last_v[2] = {-1, -1};                       // thread 0: tiles requested last
    auto load_k = [&](int tile, int buf) {
        last_k[buf] = tile;
        mbar_expect_tx(kfull0 + 8 * buf, C::K_BYTES);
#pragma unroll
        for (int b = 0; b < C::QB; ++b)
            if (b < DP / 64) tma_load_3d(sK + buf * C::K_BYTES + b * (BN * 128), &maps.k, b * 64, g, pages[tile], kfull0 + 8 * buf);
            else tma_load_3d(sK + buf * C::K_BYTES + b * (BN * 128), &maps.kr, b * 64 - DP, 0, pages[tile], kfull0 + 8 * buf);
    };
    auto load_v = [&](int tile) {
        const uint32_t b0 = (uint32_t)(tile & 1), vfull = vfull0 + 8 * b0;
        last_v[tile & 1] = tile;
        mbar_expect_tx(vfull, C::V_BYTES);
#pragma unroll
        for (int b = 0; b < C::VB; ++b) tma_load_3d(sV + b0 * C::V_BYTES + b * (BN * 128), &maps.v, v0 + b * 64, g, pages[tile], vfull);
    };
    auto issue_s = [&](int buf) {
#pragma unroll
        for (int k = 0; k < (DP + RP) / 16; ++k) {
            const uint64_t da = umma_desc(sQ + (k >> 2) * (BM * 128)) + (uint64_t)((k & 3) * 2);
            const uint64_t db = umma_desc(sK + buf * C::K_BYTES + (k >> 2) * (BN * 128)) + (uint64_t)((k & 3) * 2);
            umma_d(tmem, da, db, kDescS, k != 0 ? 1u : 0u);
        }
        umma_commit(sbar);
    };
    if (tid == 0) {
        mbar_expect_tx(qfull, C::Q_BYTES);
#pragma unroll
        for (int b = 0; b < C::QB; ++b)
            if (b < DP / 64) tma_load_3d(sQ + b * (BM * 128), &maps.q, b * 64, h, e.row0 + r0, qfull);
            else tma_load_3d(sQ + b * (BM * 128), &maps.qr, b * 64 - DP, h, e.row0 + r0, qfull);
        load_k(0, 0);
        if (C::KBUF > 1 && ntiles > 1) load_k(1, 1);
        load_v(0);
        if (ntiles > 1) load_v(1);
        const bool ok = mbar_wait(qfull, 0, abort_s) && mbar_wait(kfull0, 0, abort_s);
        if (!ok) *abort_s = 1;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (ok) issue_s(0);
    }

    // O += P V of tile j, whose weights are relative to the maximum after that tile
    float alpha_prev = 0.f;
    auto fold = [&]() {
        const uint32_t orow = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)(C::O_COL + hf * C::HALF);
#pragma unroll
        for (int c0 = 0; c0 < C::HALF; c0 += 32) {
            uint32_t r[32];
            tc::tmem_ld32(orow + (uint32_t)c0, r);
#pragma unroll
            for (int i = 0; i < 32; ++i) o[c0 + i] = fmaf(o[c0 + i], alpha_prev, __uint_as_float(r[i]));
        }
    };
    for (int j = 0; j < ntiles; ++j) {
        if (!mbar_wait(sbar, (uint32_t)j & 1u, abort_s)) *abort_s = 1;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (tid == 0 && j + C::KBUF < ntiles && *abort_s == 0) load_k(j + C::KBUF, j % C::KBUF);      // S_j has read its K buffer
        uint32_t sr[32];
        tc::tmem_ld32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)(hf * 32), sr);
        const int kb = tile_page(j) * BN, key0 = kb + hf * 32;
        float sc[32];                                            // scores in units of log2 (SIG: weights)
        float mx = -INFINITY;
        const float bias0 = b2 * (float)(key0 - i_pos);
        const bool interior = (kb >= lo_max || (KEEP && kb + BN <= keep)) && kb + BN <= hi_min;
        if constexpr (SIG) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                const float w = __fdividef(1.0f, 1.0f + at::ex2(-fmaf(__uint_as_float(sr[i]), f2, shift2)));
                sc[i] = interior || ((key0 + i >= lo || (KEEP && key0 + i < keep)) && key0 + i < hi) ? w : 0.f;
            }
        } else if (interior && b2 == 0.f) {                             // most tiles: every key visible
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                sc[i] = __uint_as_float(sr[i]) * f2;
                mx = fmaxf(mx, sc[i]);
            }
        } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                const float v = fmaf(__uint_as_float(sr[i]), f2, fmaf(b2, (float)i, bias0));
                sc[i] = interior || ((key0 + i >= lo || (KEEP && key0 + i < keep)) && key0 + i < hi) ? v : -INFINITY;
                mx = fmaxf(mx, sc[i]);
            }
        }
        if constexpr (!SIG) xch[hf * BM + row] = mx;
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        if (__syncthreads_or(*abort_s != 0)) break;             // every thread takes the same decision
        if (C::KBUF > 1 && tid == 0 && j + 1 < ntiles) {         // every thread holds its scores: S of the next tile
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (mbar_wait(kfull0 + 8 * ((j + 1) % C::KBUF), (uint32_t)((j + 1) / C::KBUF) & 1u, abort_s)) issue_s((j + 1) % C::KBUF);
            else *abort_s = 1;
        }
        __syncwarp();
        const float m_new = SIG ? 0.f : fmaxf(m, fmaxf(xch[row], xch[BM + row]));
        const float mb = m_new == -INFINITY ? 0.f : m_new;
        const float alpha = m == -INFINITY ? 0.f : at::ex2(m - mb);
        m = m_new;
        float rs = 0.f;
        uint32_t pk[16], pl[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
            const float a = SIG ? sc[i] : at::ex2(sc[i] - mb), b = SIG ? sc[i + 1] : at::ex2(sc[i + 1] - mb);      // exp2(-inf) = 0 for masked keys
            rs += a + b;
            pk[i >> 1] = pack_bf16(a, b);                            // the weights as a bf16 pair high + low: 16 bits of mantissa
            pl[i >> 1] = pack_bf16(a - bf16lo(pk[i >> 1]), b - bf16hi(pk[i >> 1]));
        }
        l = l * alpha + rs;
        if (j > 0) {                                             // P V of the previous tile has read its weights and values
            if (!mbar_wait(obar, (uint32_t)(j - 1) & 1u, abort_s)) *abort_s = 1;
            __syncwarp();
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (tid == 0 && j + 1 < ntiles && *abort_s == 0) load_v(j + 1);
            __syncwarp();
        }
        // P into tensor memory, where the MMA takes it as its A operand: lane = row, one column = two neighbouring keys
        const uint32_t prow = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)(C::P_COL + hf * 16);
        wt::tmem_st16(prow, pk);
        wt::tmem_st16(prow + 32u, pl);
        if (!SIG && j > 0) fold();
        alpha_prev = alpha;
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        __syncthreads();
        if (tid == 0) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            bool ok = mbar_wait(vfull0 + 8 * (j & 1), (uint32_t)(j >> 1) & 1u, abort_s);
            if (ok) {
#pragma unroll
                for (int k = 0; k < 2 * (BN / 16); ++k)              // high halves, then low halves
                    wt::umma_ts(tmem + C::O_COL, tmem + (uint32_t)(C::P_COL + 8 * k), vdesc[j & 1] + (uint64_t)((k % (BN / 16)) * (2048 >> 4)), kDescO, k != 0 || (SIG && j > 0) ? 1u : 0u);
                umma_commit(obar);
                if (C::KBUF == 1 && j + 1 < ntiles) {
                    ok = mbar_wait(kfull0 + 8 * ((j + 1) % C::KBUF), (uint32_t)((j + 1) / C::KBUF) & 1u, abort_s);
                    if (ok) issue_s((j + 1) % C::KBUF);
                }
            }
            if (!ok) *abort_s = 1;
        }
        __syncwarp();
    }
    if (!__syncthreads_or(*abort_s != 0)) {
        if (!mbar_wait(obar, (uint32_t)(ntiles - 1) & 1u, abort_s)) *abort_s = 1;
        __syncwarp();
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        fold();
    }

    if (tid == 0 && *abort_s != 0) {                             // given up: let the copies in flight land (bounded) before leaving
        volatile int go_on = 0;
        (void)mbar_wait(qfull, 0, &go_on);
        for (int b = 0; b < 2; ++b)
            if (last_k[b] >= 0) (void)mbar_wait(kfull0 + 8 * b, (uint32_t)(last_k[b] / C::KBUF) & 1u, &go_on);
        for (int b = 0; b < 2; ++b)
            if (last_v[b] >= 0) (void)mbar_wait(vfull0 + 8 * b, (uint32_t)(last_v[b] >> 1) & 1u, &go_on);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    xch[hf * BM + row] = l;
    __syncthreads();
    float L = SIG ? 1.0f : xch[row] + xch[BM + row], up = 1.0f;
    if (RP > 0 && s.sink != nullptr) {                           // one more term of the denominator
        const float sk = __bfloat162float(s.sink[h]) * kLog2e, mx = fmaxf(m, sk);
        up = at::ex2(m - mx);
        L = fmaf(L, up, at::ex2(sk - mx));
    }
    float inv = L > 0.f ? s.out_scale * up / L : 0.f;
    if (valid && *abort_s == 0) {
        __nv_bfloat16* dst = out + (size_t)(e.row0 + r0 + row) * ld_out + (size_t)h * s.Dv;
        const bool vec = (s.Dv & 7) == 0;                        // ld_out is a multiple of 8
        const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(s.gate);
        if ((RP > 0 || SIG) && gate != nullptr && s.gate_heads) {
            inv *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)(e.row0 + r0 + row) * s.gate_ld + h])));
        } else if (RP > 0 && gate != nullptr) {
            const __nv_bfloat16* gt = gate + (size_t)(e.row0 + r0 + row) * s.gate_ld + (size_t)h * s.Dv;
#pragma unroll
            for (int i = 0; i < C::HALF; i += 8) {
                const int d = v0 + hf * C::HALF + i;
                float f[8];
                if (vec && d + 8 <= s.Dv) unpack8(ld_cached(gt + d), f);
                else
#pragma unroll
                    for (int c = 0; c < 8; ++c) f[c] = d + c < s.Dv ? __bfloat162float(gt[d + c]) : 0.f;
#pragma unroll
                for (int c = 0; c < 8; ++c) o[i + c] *= 1.0f / (1.0f + expf(-f[c]));
            }
        }
#pragma unroll
        for (int i = 0; i < C::HALF; i += 8) {
            const int d = v0 + hf * C::HALF + i;
            if (vec && d + 8 <= s.Dv)
                *reinterpret_cast<uint4*>(dst + d) = make_uint4(pack_bf16(o[i] * inv, o[i + 1] * inv), pack_bf16(o[i + 2] * inv, o[i + 3] * inv),
                                                                pack_bf16(o[i + 4] * inv, o[i + 5] * inv), pack_bf16(o[i + 6] * inv, o[i + 7] * inv));
            else {
#pragma unroll
                for (int c = 0; c < 8; ++c)
                    if (d + c < s.Dv) dst[d + c] = __float2bfloat16_rn(o[i + c] * inv);
            }
        }
    }
    if (*abort_s != 0 && tid == 0 && error != nullptr) atomicExch(error, 1);
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(C::TMEM_COLS) : "memory");
    }
}

}  // namespace efm
