// Launchers shared by every model: the tensor-core GEMM (with its split-K and tail-split plans), row RMSNorm, the
// sampler.
#include "shared_launch.h"

#include "../operators/gemm_tc.cuh"
#include "../operators/rows.cuh"
#include "../operators/sample.cuh"
#include "launcher.h"
#include "tensor_map.h"

namespace efm {

// Widest cluster the sampler can run with on this device: 16, 8, ... or 1 (single block; also with
// EFM_B200_SAMPLER_CLUSTER=1).  Found once, outside any stream capture.
static int g_sampler_cluster = -1;

cudaError_t configure_sampler() {
    if (g_sampler_cluster >= 0) return cudaSuccess;
    int best = 1;
    const bool wide = cudaFuncSetAttribute(sample_kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1) == cudaSuccess;
    for (int cs = wide ? 16 : 8; cs >= 2; cs >>= 1) {
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(cs, 1, 1);
        cfg.blockDim = dim3(1024);
        cudaLaunchAttribute at;
        at.id = cudaLaunchAttributeClusterDimension;
        at.val.clusterDim.x = (unsigned)cs;
        at.val.clusterDim.y = at.val.clusterDim.z = 1;
        cfg.attrs = &at;
        cfg.numAttrs = 1;
        int n = 0;
        if (cudaOccupancyMaxActiveClusters(&n, sample_kernel, &cfg) == cudaSuccess && n >= 1) { best = cs; break; }
    }
    (void)cudaGetLastError();
    if (const char* env = std::getenv("EFM_B200_SAMPLER_CLUSTER")) {
        const int v = std::atoi(env);
        if (v >= 1) { int cs = 1; while (cs * 2 <= v && cs * 2 <= best) cs *= 2; best = cs; }
    }
    g_sampler_cluster = best;
    return cudaSuccess;
}

// Greedy decoding needs one block (the arg-max of the logits pass's partial maxima); top-p sampling
// spreads its passes over the vocabulary across one cluster.
void launch_sample(Launcher& L, const SampleParams& p) {
    if (g_sampler_cluster < 0) (void)configure_sampler();
    const int cs = (p.temperature >= 1e-6f && p.xchg != nullptr) ? g_sampler_cluster : 1;
    L.cluster_x = cs;
    L.launch(sample_kernel, dim3(cs), dim3(1024), 0, p);
}

// fewest 64-wide k-blocks a split may get (EFM_B200_GEMM_MIN_KB overrides, for measurements)
static int min_kb_per_split() {
    static int v = [] { const char* e = std::getenv("EFM_B200_GEMM_MIN_KB"); const int x = e != nullptr ? std::atoi(e) : 0; return x >= 1 ? x : 4; }();
    return v;
}

// EFM_B200_GEMM_TAIL=0 switches the tail split off (for A/B timing)
static bool tail_split_enabled() {
    static const bool on = [] { const char* e = std::getenv("EFM_B200_GEMM_TAIL"); return e == nullptr || e[0] != '0'; }();
    return on;
}

template <GemmEpi EPI>
static void launch_gemm(Launcher& L, const GemmParams& p, int* error_word = nullptr) {
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(gemm_tc_kernel<EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tc::SMEM_BYTES);
        attr_set = true;
    }
    CUtensorMap ma, mb;
    if (!make_tile_map(&ma, p.A, p.M, p.K, p.lda > 0 ? p.lda : p.K, tc::BM) || !make_tile_map(&mb, p.B, p.group_tile != nullptr ? p.group_all : p.N, p.K, p.K, tc::BN)) {
        if (L.err == cudaSuccess) L.err = cudaErrorInvalidValue;
        return;
    }
    const int tiles = ((p.N + tc::BN - 1) / tc::BN) * ((p.M + tc::BM - 1) / tc::BM);
    const dim3 block(tc::kThreads);
    const bool pdl = L.pdl;
    L.pdl = false;     // prefill kernels do not use the dependent-launch protocol
    if constexpr (EPI == GemmEpi::Bf16Bias || EPI == GemmEpi::Bf16Relu2 || gemm_is_glu(EPI)) {
        if (p.group_tile != nullptr) {
            static bool attr_group = false;
            if (!attr_group) {
                cudaFuncSetAttribute(gemm_tc_kernel<EPI, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tc::SMEM_BYTES);
                attr_group = true;
            }
            L.launch(gemm_tc_kernel<EPI, true>, dim3(std::min(L.num_sms, tiles)), block, tc::SMEM_BYTES, ma, mb, p, error_word);
            L.pdl = pdl;
            return;
        }
    }
    // Few output tiles and a long K: split K so that the whole GPU works, fp32 partials to the workspace, then
    // a fixed-order sum with the epilogue.
    if constexpr (EPI == GemmEpi::Bf16Bias || EPI == GemmEpi::Residual || EPI == GemmEpi::F32 || EPI == GemmEpi::Bf16Relu2 || EPI == GemmEpi::Bf16Silu ||
                  EPI == GemmEpi::Bf16Rotate || EPI == GemmEpi::ResidualTanh || gemm_is_glu(EPI)) {
        const int KB = (p.K + tc::BK - 1) / tc::BK;
        int splits = std::min(L.num_sms / std::max(1, tiles), KB / min_kb_per_split());
        if (L.gemm_ws != nullptr && splits >= 2 && (p.N & 3) == 0 && (!gemm_is_glu(EPI) || (p.N & 127) == 0) &&
            (size_t)splits * p.M * p.N <= L.gemm_ws_floats) {
            const int per = (KB + splits - 1) / splits;
            splits = (KB + per - 1) / per;                 // no empty split
            GemmParams q = p;
            q.kb_per_split = per;
            q.Cf = L.gemm_ws;
            q.bias = nullptr;
            static bool attr_f32 = false;
            if (!attr_f32) {
                cudaFuncSetAttribute(gemm_tc_kernel<GemmEpi::F32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tc::SMEM_BYTES);
                attr_f32 = true;
            }
            L.launch(gemm_tc_kernel<GemmEpi::F32>, dim3(std::min(L.num_sms, tiles * splits)), block, tc::SMEM_BYTES, ma, mb, q, error_word);
            const size_t total4 = (size_t)p.M * p.N / (gemm_is_glu(EPI) ? 8 : 4);
            const int fin = (int)std::min<size_t>((total4 + 255) / 256, (size_t)L.num_sms * 4);
            L.launch(gemm_splitk_finish_kernel<EPI>, dim3(fin), dim3(256), 0, (const float*)L.gemm_ws, splits, p);
            L.pdl = pdl;
            return;
        }
    }
    // Tail split: a few tiles more than a multiple of the SM count would cost a whole extra round in which most SMs
    // idle (1324 x 3584 outputs = 154 tiles on 148 SMs: two rounds for 1.04 rounds of work).  The full rounds run as
    // they are; the remaining tiles are cut along K into as many slices as fill the GPU once (compact fp32 slots in
    // the workspace) and a small kernel sums the slices in order with the epilogue.  Worth it only when a tile's K
    // loop is long against the two extra launches (about 12 us).
    if constexpr (EPI == GemmEpi::Bf16Bias || EPI == GemmEpi::Residual || EPI == GemmEpi::F32 || EPI == GemmEpi::Bf16Silu || EPI == GemmEpi::Bf16Rotate ||
                  EPI == GemmEpi::ResidualTanh) {
        const int P = L.num_sms, rounds = tiles / P, rem = tiles % P;
        const int KB = (p.K + tc::BK - 1) / tc::BK;
        if (tail_split_enabled() && L.gemm_ws != nullptr && rounds >= 1 && rem > 0 && rem * 2 <= P && (p.N & 3) == 0 && p.kb_per_split == 0 &&
            p.tile_count == 0) {
            int splits = std::min(P / rem, KB / min_kb_per_split());
            const int per = splits >= 2 ? (KB + splits - 1) / splits : KB;
            splits = (KB + per - 1) / per;
            const double tile_us = KB * 0.45, gain_us = tile_us * (1.0 - 1.0 / std::max(1, splits)) - 12.0;
            if (splits >= 2 && gain_us > 5.0 && (size_t)splits * rem * tc::BM * tc::BN <= L.gemm_ws_floats) {
                GemmParams full = p;
                full.tile_begin = 0;
                full.tile_count = rounds * P;
                L.launch(gemm_tc_kernel<EPI>, dim3(P), block, tc::SMEM_BYTES, ma, mb, full, error_word);
                GemmParams q = p;
                q.tile_begin = rounds * P;
                q.tile_count = rem;
                q.kb_per_split = per;
                q.Cf = L.gemm_ws;
                q.bias = nullptr;
                static bool attr_f32 = false;
                if (!attr_f32) {
                    cudaFuncSetAttribute(gemm_tc_kernel<GemmEpi::F32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tc::SMEM_BYTES);
                    attr_f32 = true;
                }
                L.launch(gemm_tc_kernel<GemmEpi::F32>, dim3(std::min(P, rem * splits)), block, tc::SMEM_BYTES, ma, mb, q, error_word);
                const int per_tile = std::max(1, std::min(32, (P * 4) / rem));
                L.launch(gemm_tail_finish_kernel<EPI>, dim3(per_tile, rem), dim3(256), 0, (const float*)L.gemm_ws, splits, rounds * P, rem, p);
                L.pdl = pdl;
                return;
            }
        }
    }
    L.launch(gemm_tc_kernel<EPI>, dim3(std::min(L.num_sms, tiles)), block, tc::SMEM_BYTES, ma, mb, p, error_word);
    L.pdl = pdl;
}

void launch_gemm_bf16(Launcher& L, const GemmParams& p) { launch_gemm<GemmEpi::Bf16Bias>(L, p); }

void launch_rmsnorm_rows(Launcher& L, const float* x, const __nv_bfloat16* w, __nv_bfloat16* y, int rows, int hidden, float eps) {
    const bool pdl = L.pdl;
    L.pdl = pdl && L.pdl_rows;
    // many short rows (vision tower, action model): one warp per row; otherwise one block per row
    if (hidden <= 2048 && (hidden & 3) == 0 && rows >= 256)
        L.launch(rmsnorm_rows_warp_kernel, dim3((rows + 7) / 8), dim3(256), 0, x, w, y, rows, hidden, eps);
    else
        L.launch(rmsnorm_rows_kernel, dim3(rows), dim3(256), 0, x, w, y, hidden, eps);
    L.pdl = pdl;
}

void launch_embed_rows(Launcher& L, const int32_t* ids, const __nv_bfloat16* table, const __nv_bfloat16* custom, float* out, int rows,
                       int vocab, int hidden, int embed_token_id, int n_custom, float scale) {
    L.launch(embed_rows_kernel, dim3(rows), dim3(128), 0, ids, table, custom, out, vocab, hidden, embed_token_id, n_custom, scale);
}

void launch_gemm_epi(Launcher& L, GemmEpi epi, const GemmParams& p, int* error_word) {
    switch (epi) {
        case GemmEpi::Bf16Bias: launch_gemm<GemmEpi::Bf16Bias>(L, p, error_word); break;
        case GemmEpi::Residual: launch_gemm<GemmEpi::Residual>(L, p, error_word); break;
        case GemmEpi::F32: launch_gemm<GemmEpi::F32>(L, p, error_word); break;
        case GemmEpi::Bf16Gelu: launch_gemm<GemmEpi::Bf16Gelu>(L, p, error_word); break;
        case GemmEpi::Bf16GeluTanh: launch_gemm<GemmEpi::Bf16GeluTanh>(L, p, error_word); break;
        case GemmEpi::SwiGlu: launch_gemm<GemmEpi::SwiGlu>(L, p, error_word); break;
        case GemmEpi::Bf16Relu2: launch_gemm<GemmEpi::Bf16Relu2>(L, p, error_word); break;
        case GemmEpi::Bf16Silu: launch_gemm<GemmEpi::Bf16Silu>(L, p, error_word); break;
        case GemmEpi::Bf16Rotate: launch_gemm<GemmEpi::Bf16Rotate>(L, p, error_word); break;
        case GemmEpi::ResidualTanh: launch_gemm<GemmEpi::ResidualTanh>(L, p, error_word); break;
        case GemmEpi::ClampGlu: launch_gemm<GemmEpi::ClampGlu>(L, p, error_word); break;
    }
}

}  // namespace efm
