// Launchers shared by the models (definitions in gemm_launch.cu and attention_launch.cu).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace efm {
struct Launcher;
struct GemmParams;
struct SampleParams;
struct SegAttnParams;
enum class GemmEpi : int;

void launch_gemm_bf16(Launcher& L, const GemmParams& p);
// C = A . B^T on the tensor cores with the named epilogue; error_word (device int, may be null) is
// raised when a bounded pipeline wait gives up.
void launch_gemm_epi(Launcher& L, GemmEpi epi, const GemmParams& p, int* error_word);
// false with EFM_B200_ATTN_TC=0 (A/B timing of the mma.sync forms)
bool attention_tc_enabled();
// Attention with per-query key ranges (or the causal prefill rule when p.lo is null).
void launch_seg_attention(Launcher& L, const SegAttnParams& p, int D);
// Same result; picks the all-keys-resident variant when D == 64, S <= 64 and max_keys (largest hi) <= 320.
void launch_seg_attention_short(Launcher& L, const SegAttnParams& p, int D, int max_keys);
void launch_sample(Launcher& L, const SampleParams& p);
cudaError_t configure_sampler();      // once per device at set-up, never inside a stream capture
// out[r,:] = table[ids[r],:] * scale (fp32), injected rows for ids in [embed_token_id, embed_token_id + n_custom).
void launch_embed_rows(Launcher& L, const int32_t* ids, const __nv_bfloat16* table, const __nv_bfloat16* custom, float* out, int rows,
                       int vocab, int hidden, int embed_token_id, int n_custom, float scale = 1.0f);
// y[r,:] = bf16(rmsnorm(x[r,:]) * w) over `rows` fp32 rows.
void launch_rmsnorm_rows(Launcher& L, const float* x, const __nv_bfloat16* w, __nv_bfloat16* y, int rows, int hidden, float eps);
void launch_prefill_attention(Launcher& L, const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v,
                              __nv_bfloat16* out, int S, int kv_offset, int q_heads, int kv_heads, int D,
                              int* error = nullptr);

}  // namespace efm
