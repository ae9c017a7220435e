// Host-side state shared by the launchers: the dependent-launch switch, the per-device SM
// count and the table that says which kernels have been launched.
#include "common.cuh"

unsigned long long g_mf_kernel_launches[MF_K_COUNT] = {};

namespace {
const char* const kNames[MF_K_COUNT] = {
    "stream_rows",      "stream_tmap",      "mid_rows",         "gemm_tc",
    "gemm_tc_swiglu",   "gemm_f32",         "attn_generic", "attn_prefill_mma", "attn_prefill_tc",
    "attn_decode",      "attn_decode_tma",  "attn_decode_tma_merged", "attn_decode_merge",
    "embed_positions",  "hyper_norm",       "kv_store",         "attn_talking",     "attn_talking_tc", "attn_talking_merge",
    "delta_prepare",    "delta_gates",      "delta_recurrence", "delta_output",
    "moe_route",        "moe_rows",         "moe_combine",      "moe_sort",         "moe_grouped",
    "rope_store",       "norm_pair",        "latent_prepare",   "latent_query",     "head_linear",
    "head_linear_mma",  "retention_prepare", "retention_recurrence", "retention_chunked", "retention_output",
    "unary_act",        "gemm_tc_act",      "conv_input",       "postnorm_add",     "qk_norm_rope",
    "rotate_rows",      "gdelta_prepare",   "gdelta_recurrence",
    "conv_act",         "decay_recurrence", "decay_local",      "scan_combine",     "gated_norm",
    "selective_scan",   "scan_local",       "low_rank",         "post_norm",      "qkv_conv",
    "soft_cap",
};
int g_sm_count[MF_MAX_DEVICES] = {};
}  // namespace

int mf_sm_count() {
  const int d = mf_current_device();
  if (d < 0) return 0;
  if (g_sm_count[d] == 0) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, d) != cudaSuccess) return 0;
    g_sm_count[d] = n;
  }
  return g_sm_count[d];
}

// Number of kernel kinds that are counted, the name of one, and how often it has been launched
// in this process (launches recorded into a CUDA graph count once, replays do not).
MF_API int mf_kernel_kinds() { return MF_K_COUNT; }
MF_API const char* mf_kernel_name(int id) { return id >= 0 && id < MF_K_COUNT ? kNames[id] : ""; }
MF_API long long mf_kernel_launches(int id) {
  return id >= 0 && id < MF_K_COUNT ? (long long)g_mf_kernel_launches[id] : -1;
}
