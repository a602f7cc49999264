// Launchers of the many-row softmax attention (tcgen05 form, mma.sync form).
#include "../operators/attention_mma.cuh"
#include "../operators/attention_tc.cuh"
#include "launcher.h"
#include "shared_launch.h"
#include "tensor_map.h"

namespace efm {

template <int D, int NW>
static void launch_seg_attention_dn(Launcher& L, const SegAttnParams& p) {
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(seg_attention_kernel<D, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sa::smem_bytes<D, NW>());
        attr_set = true;
    }
    const dim3 grid((p.S + 16 * NW - 1) / (16 * NW), p.q_heads), block(32 * NW);
    const bool pdl = L.pdl;
    L.pdl = pdl && L.pdl_rows;
    L.launch(seg_attention_kernel<D, NW>, grid, block, sa::smem_bytes<D, NW>(), p);
    L.pdl = pdl;
}

template <int D>
static void launch_seg_attention_d(Launcher& L, const SegAttnParams& p) {
    // 64-query blocks: 128-query blocks (NW 8) measured 1-2 % slower on B200 at 1324 and 4784 rows (register-bound
    // occupancy does not improve with them)
    launch_seg_attention_dn<D, 4>(L, p);
}

void launch_seg_attention(Launcher& L, const SegAttnParams& p, int D);
// Head dim 64, at most 64 queries and at most 320 keys per block (the action expert's attention): every key of the
// block is requested at once.  Anything else goes to the streaming kernel.
void launch_seg_attention_short(Launcher& L, const SegAttnParams& p, int D, int max_keys) {
    constexpr int PRE = 5;
    if (D != 64 || p.S <= 0 || p.S > 64 || max_keys > PRE * sa::BKV) { launch_seg_attention(L, p, D); return; }
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(seg_attention_kernel<64, 4, PRE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sa::smem_bytes<64, 4, PRE>());
        attr_set = true;
    }
    const bool pdl = L.pdl;
    L.pdl = pdl && L.pdl_rows;
    L.launch(seg_attention_kernel<64, 4, PRE>, dim3(1, p.q_heads), dim3(128), sa::smem_bytes<64, 4, PRE>(), p);
    L.pdl = pdl;
}

bool attention_tc_enabled() {
    static const bool on = [] { const char* e = std::getenv("EFM_B200_ATTN_TC"); return e == nullptr || e[0] != '0'; }();
    return on;
}

// tcgen05 / TMEM form (attention_tc.cuh).
template <int D>
static bool launch_seg_attention_tc_d(Launcher& L, const SegAttnParams& p0) {
    using C = at::Cfg<D>;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(seg_attention_tc_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM);
        attr_set = true;
    }
    const SegAttnParams& p = p0;
    CUtensorMap mq, mk, mv;
    const uint64_t qd[3] = {(uint64_t)D, (uint64_t)p.q_heads, (uint64_t)p.S}, qs[2] = {(uint64_t)D * 2, (uint64_t)p.q_stride * 2};
    const uint64_t kd[3] = {(uint64_t)D, (uint64_t)p.kv_heads, (uint64_t)p.kv_rows}, ks[2] = {(uint64_t)D * 2, (uint64_t)p.kv_stride * 2};
    const uint32_t qb[3] = {64, 1, (uint32_t)at::BM}, kb[3] = {64, 1, (uint32_t)at::BN};
    if (!make_map_nd(&mq, p.q, 3, qd, qs, qb) || !make_map_nd(&mk, p.k, 3, kd, ks, kb) || !make_map_nd(&mv, p.v, 3, kd, ks, kb)) return false;
    const bool pdl = L.pdl;
    L.pdl = false;
    L.launch(seg_attention_tc_kernel<D>, dim3((p.S + at::BM - 1) / at::BM, p.q_heads), dim3(at::kThreads), C::SMEM, mq, mk, mv, p, p.error);
    L.pdl = pdl;
    return true;
}

static bool launch_seg_attention_tc(Launcher& L, const SegAttnParams& p, int D) {
    // TMA needs 16-byte aligned bases and strides; anything else stays on the mma.sync kernel
    if (p.kv_rows <= 0 || (p.q_stride & 7) || (p.kv_stride & 7) || (reinterpret_cast<uintptr_t>(p.q) & 15) ||
        (reinterpret_cast<uintptr_t>(p.k) & 15) || (reinterpret_cast<uintptr_t>(p.v) & 15) || (p.out_stride & 7) ||
        (reinterpret_cast<uintptr_t>(p.out) & 15) || !attention_tc_enabled())
        return false;
    if (D == 128) return launch_seg_attention_tc_d<128>(L, p);
    if (D == 80) return launch_seg_attention_tc_d<80>(L, p);
    if (D == 64) return launch_seg_attention_tc_d<64>(L, p);
    return false;
}

void launch_seg_attention(Launcher& L, const SegAttnParams& p, int D) {
    if (p.S <= 0) return;
    if (launch_seg_attention_tc(L, p, D)) return;
    if (D == 128) launch_seg_attention_d<128>(L, p);
    else if (D == 80) launch_seg_attention_d<80>(L, p);
    else if (D == 64) launch_seg_attention_d<64>(L, p);
    else if (L.err == cudaSuccess) L.err = cudaErrorInvalidValue;
}

// Causal GQA attention of a prefill chunk: queries at cache rows [kv_offset, kv_offset + S).
void launch_prefill_attention(Launcher& L, const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v,
                              __nv_bfloat16* out, int S, int kv_offset, int q_heads, int kv_heads, int D, int* error) {
    SegAttnParams p{};
    p.q = q; p.k = k; p.v = v; p.out = out;
    p.q_stride = q_heads * D; p.kv_stride = kv_heads * D; p.out_stride = q_heads * D;
    p.S = S; p.kv_offset = kv_offset; p.q_heads = q_heads; p.kv_heads = kv_heads;
    p.scale = 1.0f / sqrtf((float)D);
    p.kv_rows = kv_offset + S;
    p.error = error;
    launch_seg_attention(L, p, D);
}

}  // namespace efm
