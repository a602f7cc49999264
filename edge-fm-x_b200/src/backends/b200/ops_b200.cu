// Single operators of the C ABI on caller-provided device buffers (default stream, synchronous): the granularity of the
// parity tests.
#include <atomic>
#include <cstdio>

#include "../../layers/launch.cuh"
#include "../../layers/qwen_text.h"
#include "../../operators/gemm_tc.cuh"
#define EFM_DECLARATIONS_ONLY
#include "../../operators/sample.cuh"
#undef EFM_DECLARATIONS_ONLY
#include "ctx.h"
#include "ctx_util.h"
#include "text_device.h"

using namespace efm;

extern "C" {

static efm_status op_prepare(int* num_sms) {
    int dev = 0;
    efm_status st = EFM_OK;
    if (cudaGetDevice(&dev) != cudaSuccess) return fail(nullptr, EFM_ERR_CUDA, "no CUDA device available");
    if ((st = require_b200(nullptr, dev)) != EFM_OK) return st;
    if (num_sms != nullptr) cudaDeviceGetAttribute(num_sms, cudaDevAttrMultiProcessorCount, dev);
    return EFM_OK;
}
static efm_status op_finish(Launcher& L) {
    if (L.err != cudaSuccess) return cuda_fail(nullptr, L.err, "operator launch");
    cudaError_t e = cudaStreamSynchronize(L.stream);
    if (e != cudaSuccess) return cuda_fail(nullptr, e, "operator execution");
    return EFM_OK;
}

efm_status efm_b200_op_gemv(const void* w, const void* x, const void* norm_w, float eps, void* y_bf16, void* residual,
                            int32_t n, int32_t k) {
    int sms = 148;
    efm_status st = op_prepare(&sms);
    if (st != EFM_OK) return st;
    if (w == nullptr || x == nullptr || (y_bf16 == nullptr && residual == nullptr) || n <= 0 || n % 2 || k <= 0 || k % 8)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_gemv: bad arguments (n even, k % 8 == 0)");
    GemvParams p{};
    p.W = (const __nv_bfloat16*)w; p.N = n; p.K = k; p.n_items = n / 2;
    p.prologue = norm_w != nullptr ? kProRmsNorm : kProPlain;
    p.x = (const __nv_bfloat16*)x; p.xr = (const float*)x; p.norm_w = (const __nv_bfloat16*)norm_w; p.eps = eps;
    p.y = (__nv_bfloat16*)y_bf16; p.residual = (float*)residual;
    Launcher L; L.pdl = false;
    if (residual != nullptr) launch_gemv<Epi::Residual>(L, p, sms); else launch_gemv<Epi::Plain>(L, p, sms);
    return op_finish(L);
}

efm_status efm_b200_op_gemv_peer_consume(const void* w, const void* resid_f32, const void* norm_w, float eps, const void* parts,
                                         int32_t n_parts, uint32_t want_count, int64_t wait_limit_us, void* y_bf16,
                                         void* resid_out_f32, int32_t n, int32_t k) {
    int sms = 148;
    efm_status st = op_prepare(&sms);
    if (st != EFM_OK) return st;
    if (w == nullptr || resid_f32 == nullptr || norm_w == nullptr || parts == nullptr || y_bf16 == nullptr || resid_out_f32 == nullptr ||
        resid_out_f32 == resid_f32 || n_parts < 1 || n_parts > kMaxPeers || want_count == 0 || wait_limit_us <= 0 || n <= 0 || n % 2 ||
        k <= 0 || k % 8)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_gemv_peer_consume: bad arguments");
    int* error = nullptr;
    cudaError_t e = cudaMalloc(&error, sizeof(int));
    if (e == cudaSuccess) e = cudaMemset(error, 0, sizeof(int));
    if (e != cudaSuccess) { cudaFree(error); return cuda_fail(nullptr, e, "op_gemv_peer_consume scratch"); }
    GemvParams p{};
    p.W = (const __nv_bfloat16*)w; p.N = n; p.K = k; p.n_items = n / 2;
    p.prologue = kProRmsNorm;
    p.xr = (const float*)resid_f32; p.norm_w = (const __nv_bfloat16*)norm_w; p.eps = eps;
    p.resid_out = (float*)resid_out_f32;
    p.addend_parts = (const uint2*)parts; p.n_parts = n_parts; p.want_override = want_count;
    p.error = error; p.wait_ns = (unsigned long long)wait_limit_us * 1000ull;
    p.y = (__nv_bfloat16*)y_bf16;
    Launcher L; L.pdl = false;
    launch_gemv<Epi::Plain>(L, p, sms);
    st = op_finish(L);
    int raised = 0;
    if (st == EFM_OK && cudaMemcpy(&raised, error, sizeof(int), cudaMemcpyDeviceToHost) != cudaSuccess) st = fail(nullptr, EFM_ERR_CUDA, "reading the status word");
    cudaFree(error);
    if (st == EFM_OK && raised != 0)
        return fail(nullptr, EFM_ERR_DEVICE_WAIT, "the wait for the peers' words ran out (device status " + std::to_string(raised) + ")");
    return st;
}

efm_status efm_b200_op_gemm(const void* x, const void* w, const void* bias, void* y_bf16, int32_t m, int32_t n, int32_t k) {
    efm_status st = op_prepare(nullptr);
    if (st != EFM_OK) return st;
    if (x == nullptr || w == nullptr || y_bf16 == nullptr || m <= 0 || n <= 0 || n % 2 || k <= 0 || k % 32)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_gemm: bad arguments (n even, k % 32 == 0)");
    GemmParams g{(const __nv_bfloat16*)x, (const __nv_bfloat16*)w, (const __nv_bfloat16*)bias, (__nv_bfloat16*)y_bf16, nullptr, m, n, k};
    Launcher L; L.pdl = false;
    int sms = 148;
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, 0);
    L.num_sms = sms;
    L.gemm_ws_floats = (size_t)sms * 128 * 256;          // lets skinny products take the split-K path, as inside a context
    if (cudaMalloc(&L.gemm_ws, L.gemm_ws_floats * sizeof(float)) != cudaSuccess) {
        (void)cudaGetLastError();
        L.gemm_ws = nullptr;
    }
    launch_gemm_bf16(L, g);
    const efm_status out = op_finish(L);
    if (L.gemm_ws != nullptr) cudaFree(L.gemm_ws);
    return out;
}

efm_status efm_b200_op_sage_prefill_attention(const void* q, const void* k_cache, const void* v_cache, void* out_bf16,
                                              int32_t s, int32_t kv_offset, int32_t q_heads, int32_t kv_heads, int32_t head_dim) {
    efm_status st = op_prepare(nullptr);
    if (st != EFM_OK) return st;
    if (q == nullptr || k_cache == nullptr || v_cache == nullptr || out_bf16 == nullptr || s <= 0 || kv_offset < 0 || q_heads <= 0 ||
        kv_heads <= 0 || q_heads % kv_heads != 0)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_sage_prefill_attention: bad arguments");
    if (head_dim != 64 && head_dim != 128) return fail(nullptr, EFM_ERR_UNSUPPORTED, "op_sage_prefill_attention: head_dim 64 or 128");
    SageScratch sc;
    cudaError_t e = alloc_sage(sc, s, kv_offset + s, q_heads, kv_heads, head_dim);
    if (e != cudaSuccess) { free_sage(sc); return cuda_fail(nullptr, e, "INT8 attention scratch"); }
    Launcher L; L.pdl = false;
    launch_sage_prefill_attention(L, sc, (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache,
                                  (__nv_bfloat16*)out_bf16, s, kv_offset, q_heads, kv_heads, head_dim);
    st = op_finish(L);
    free_sage(sc);
    return st;
}

efm_status efm_b200_op_decode_attention(const void* q, const void* k_cache, const void* v_cache, void* out_bf16,
                                        int32_t q_heads, int32_t kv_heads, int32_t head_dim, int32_t kv_len, int32_t max_tokens) {
    int sms = 148;
    efm_status st = op_prepare(&sms);
    if (st != EFM_OK) return st;
    if (q == nullptr || k_cache == nullptr || v_cache == nullptr || out_bf16 == nullptr || kv_heads <= 0 || q_heads % kv_heads ||
        q_heads / kv_heads > kMaxGroup || (head_dim != 64 && head_dim != 128) || kv_len <= 0 || kv_len > max_tokens)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_decode_attention: bad arguments");
    const AttnPlan plan = plan_decode_attention(max_tokens, kv_heads, sms);
    float* part_o = nullptr; float* part_ml = nullptr; unsigned int* counters = nullptr;
    cudaError_t e = cudaMalloc(&part_o, (size_t)q_heads * plan.n_splits * head_dim * 4);
    if (e == cudaSuccess) e = cudaMalloc(&part_ml, (size_t)q_heads * plan.n_splits * 2 * 4);
    if (e == cudaSuccess) e = cudaMalloc(&counters, (size_t)kv_heads * 4);
    if (e == cudaSuccess) e = cudaMemset(counters, 0, (size_t)kv_heads * 4);
    if (e == cudaSuccess) {
        DecodeAttnParams a{};
        a.q = (const __nv_bfloat16*)q; a.k_cache = (const __nv_bfloat16*)k_cache; a.v_cache = (const __nv_bfloat16*)v_cache;
        a.out = (__nv_bfloat16*)out_bf16; a.state = nullptr; a.kv_len_static = kv_len;
        a.q_heads = q_heads; a.kv_heads = kv_heads; a.group = q_heads / kv_heads;
        a.n_splits = plan.n_splits; a.chunk_cap = plan.chunk_cap; a.max_tokens = max_tokens; a.cluster = plan.cluster;
        a.scale = 1.0f / sqrtf((float)head_dim);
        a.part_o = part_o; a.part_ml = part_ml; a.counters = counters;
        Launcher L; L.pdl = false;
        launch_decode_attention(L, a, head_dim);
        st = op_finish(L);
    } else {
        st = cuda_fail(nullptr, e, "op_decode_attention scratch");
    }
    cudaFree(part_o); cudaFree(part_ml); cudaFree(counters);
    return st;
}

// ---- decode attention without any allocation -------------------------------------------------
// Scratch for the split-KV partials lives in the library image.  In host code the symbol below is
// only a stand-in for the device array: its device address has to be asked for, per device.
namespace {
constexpr int kNoAllocMaxQD = 4096;       // q_heads * head_dim
constexpr int kNoAllocMaxKvHeads = 16;
constexpr int kNoAllocMaxQHeads = 64;     // head_dim >= 64
// layout in 32-bit words: partial outputs [q_heads][n_splits][D] | (max, sum) pairs
// [q_heads][n_splits][2] | block tickets [kv_heads] (these must read zero when a launch starts)
constexpr size_t kNoAllocPartO = (size_t)kNoAllocMaxQD * kMaxSplits;
constexpr size_t kNoAllocPartMl = (size_t)kNoAllocMaxQHeads * kMaxSplits * 2;
constexpr size_t kNoAllocWords = kNoAllocPartO + kNoAllocPartMl + kNoAllocMaxKvHeads;     // ~1.06 MB
static __device__ __align__(256) float g_noalloc_scratch[kNoAllocWords];
constexpr int kNoAllocMaxDevices = 64;
std::atomic<float*> g_noalloc_ptr[kNoAllocMaxDevices];     // zero-initialised; filled once per device, any thread
}  // namespace

efm_status efm_b200_op_decode_attention_noalloc(const void* q, const void* k_cache, const void* v_cache, void* out_bf16,
                                                int32_t q_heads, int32_t kv_heads, int32_t head_dim, int32_t kv_len,
                                                int32_t max_tokens) {
    int sms = 148;
    efm_status st = op_prepare(&sms);
    if (st != EFM_OK) return st;
    if (q == nullptr || k_cache == nullptr || v_cache == nullptr || out_bf16 == nullptr || kv_heads <= 0 || q_heads % kv_heads ||
        q_heads / kv_heads > kMaxGroup || (head_dim != 64 && head_dim != 128) || kv_len <= 0 || kv_len > max_tokens)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_decode_attention_noalloc: bad arguments");
    if (q_heads * head_dim > kNoAllocMaxQD || kv_heads > kNoAllocMaxKvHeads || q_heads > kNoAllocMaxQHeads)
        return fail(nullptr, EFM_ERR_UNSUPPORTED,
                    "op_decode_attention_noalloc: shape exceeds the built-in scratch (q_heads * head_dim <= 4096, "
                    "q_heads <= 64, kv_heads <= 16); use efm_b200_op_decode_attention");
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return cuda_fail(nullptr, e, "cudaGetDevice");
    if (dev < 0 || dev >= kNoAllocMaxDevices) return fail(nullptr, EFM_ERR_UNSUPPORTED, "device index above 63");
    float* scratch = g_noalloc_ptr[dev].load(std::memory_order_acquire);
    if (scratch == nullptr) {      // once per device, with that device current (two threads racing here store the same address)
        float* ptr = nullptr;
        e = cudaGetSymbolAddress((void**)&ptr, g_noalloc_scratch);
        if (e != cudaSuccess || ptr == nullptr) return cuda_fail(nullptr, e, "cudaGetSymbolAddress(scratch)");
        g_noalloc_ptr[dev].store(ptr, std::memory_order_release);
        scratch = ptr;
    }
    unsigned int* tickets = reinterpret_cast<unsigned int*>(scratch + kNoAllocPartO + kNoAllocPartMl);
    const AttnPlan plan = plan_decode_attention(max_tokens, kv_heads, sms);
    e = cudaMemsetAsync(tickets, 0, kNoAllocMaxKvHeads * sizeof(unsigned int), nullptr);
    if (e != cudaSuccess) return cuda_fail(nullptr, e, "clearing the scratch tickets");
    DecodeAttnParams a{};
    a.q = (const __nv_bfloat16*)q; a.k_cache = (const __nv_bfloat16*)k_cache; a.v_cache = (const __nv_bfloat16*)v_cache;
    a.out = (__nv_bfloat16*)out_bf16; a.state = nullptr; a.kv_len_static = kv_len;
    a.q_heads = q_heads; a.kv_heads = kv_heads; a.group = q_heads / kv_heads;
    a.n_splits = plan.n_splits; a.chunk_cap = plan.chunk_cap; a.max_tokens = max_tokens; a.cluster = plan.cluster;
    a.scale = 1.0f / sqrtf((float)head_dim);
    a.part_o = scratch; a.part_ml = scratch + kNoAllocPartO; a.counters = tickets;
    Launcher L; L.pdl = false;
    launch_decode_attention(L, a, head_dim);
    return op_finish(L);
}

efm_status efm_b200_op_prefill_attention(const void* q, const void* k_cache, const void* v_cache, void* out_bf16, int32_t s,
                                         int32_t kv_offset, int32_t q_heads, int32_t kv_heads, int32_t head_dim) {
    efm_status st = op_prepare(nullptr);
    if (st != EFM_OK) return st;
    if (q == nullptr || k_cache == nullptr || v_cache == nullptr || out_bf16 == nullptr || s <= 0 || kv_offset < 0 || kv_heads <= 0 ||
        q_heads % kv_heads || (head_dim != 64 && head_dim != 128))
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_prefill_attention: bad arguments");
    Launcher L; L.pdl = false;
    launch_prefill_attention(L, (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache,
                             (__nv_bfloat16*)out_bf16, s, kv_offset, q_heads, kv_heads, head_dim);
    return op_finish(L);
}

efm_status efm_b200_op_sample(const float* logits, int32_t vocab, const efm_sampling* s, uint32_t rng_step, int32_t* token_out) {
    efm_status st = op_prepare(nullptr);
    if (st != EFM_OK) return st;
    if (logits == nullptr || s == nullptr || token_out == nullptr || vocab <= 0)
        return fail(nullptr, EFM_ERR_INVALID_ARGUMENT, "op_sample: bad arguments");
    uint32_t* wbuf = nullptr;
    cudaError_t e = cudaMalloc(&wbuf, sample_scratch_words(vocab) * 4);
    if (e != cudaSuccess) return cuda_fail(nullptr, e, "op_sample scratch");
    SampleParams p{};
    p.logits = logits; p.vocab = vocab; p.n_part = 0;
    p.temperature = s->temperature; p.top_p = s->top_p; p.seed = s->seed; p.rng_step = rng_step;
    p.state = nullptr; p.token_single = token_out; p.wbuf = wbuf; p.xchg = sample_xchg(wbuf, vocab);
    Launcher L; L.pdl = false;
    launch_sample(L, p);
    st = op_finish(L);
    cudaFree(wbuf);
    return st;
}

}  // extern "C"

