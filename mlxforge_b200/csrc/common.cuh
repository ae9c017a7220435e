// Shared helpers for the sm_100a kernels of mlxforge_b200.
//
// Conventions used by every entry point:
//  * entry points are extern "C", take raw device pointers and the CUDA stream
//    to launch on, allocate nothing, and return a cudaError_t code (0 = ok) or
//    one of the MF_ERR_* codes below for an argument the kernel refuses;
//  * `dtype` arguments are 0 for IEEE float32 and 1 for bfloat16;
//  * matrices are row-major; weights are [out, in] as in the checkpoint.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define MF_F32 0
#define MF_BF16 1

#define MF_ERR_BAD_ARG 10001      // a size the kernel does not take
#define MF_ERR_BAD_DTYPE 10002

#define MF_API extern "C" __attribute__((visibility("default")))

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Activations of a feed-forward (of its gate, where it has one), in 32-bit.
#define MF_ACT_SILU 0
#define MF_ACT_GELU_TANH 1      // 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
#define MF_ACT_RELU2 2          // max(z, 0)^2
#define MF_ACT_COUNT 3
// mode of a product whose epilogue applies activation a to every sum (no gate): MF_STREAM_UNARY + a
#define MF_STREAM_UNARY 16
__device__ __forceinline__ float gate_act(float g, int act) {
  if (act == MF_ACT_GELU_TANH) return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
  if (act == MF_ACT_RELU2) {
    const float r = fmaxf(g, 0.f);
    return r * r;
  }
  return g / (1.0f + expf(-g));
}

// The clamped gate: g' = min(g, limit), u' = clamp(u, -limit, limit), g' sigmoid(alpha g') (u' + up_off).
// It stands beside the activations above wherever a gate and an up value meet (not where there is no gate).
#define MF_GATE_CLAMPED 8
// mode of a product whose epilogue applies a soft cap to every sum: cap tanh(sum / cap)
#define MF_STREAM_SOFTCAP 32
// constants of a product's epilogue
struct EpiConst {
  float limit, alpha, up_off;      // of the clamped gate
  float cap;                       // of the soft cap
};
// QUICK: for results that are rounded to bfloat16 (a division and an exponential of a few 32-bit ulps)
template <bool QUICK = false>
__device__ __forceinline__ float gated_product(float g, float u, int act, const EpiConst& k) {
  if (act == MF_GATE_CLAMPED) {
    g = fminf(g, k.limit);
    u = fminf(fmaxf(u, -k.limit), k.limit);
    const float s = QUICK ? __fdividef(g, 1.0f + __expf(-k.alpha * g)) : g / (1.0f + expf(-k.alpha * g));
    return s * (u + k.up_off);
  }
  return gate_act(g, act) * u;
}
__device__ __forceinline__ float soft_cap(float v, float cap) { return cap * tanhf(v / cap); }

// Two 32-bit numbers side by side in a 64-bit register and the arithmetic on both at once (one instruction each,
// rounded like the single ones).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
  return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Block-wide sum for blocks of up to 1024 threads; `red` is 32 floats of shared
// memory.  Every thread gets the result.  The order of additions depends only on
// the block size, never on what else runs.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float r = (lane < nw) ? red[lane] : 0.f;
  r = warp_sum(r);
  return r;
}
__device__ __forceinline__ float block_max(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float r = (lane < nw) ? red[lane] : -INFINITY;
  r = warp_max(r);
  return r;
}

// Paged cache addressing.  One pool per cache lane (a layer's keys or values):
// [page][kv_head][slot][head_dim].  `block_table` holds, per sequence of the
// step, the page of every logical block; entries of blocks that were given back
// (outside a window) are negative and are never addressed.
struct PagedView {
  const int* block_table;   // [n_seqs, bt_stride]
  int bt_stride;
  int page_size;
  int n_kv_heads;
  int head_dim;
};
__device__ __forceinline__ long long paged_offset(const PagedView& pv, int seq, int pos, int kv_head) {
  const int blk = pos / pv.page_size, slot = pos - blk * pv.page_size;
  const long long page = pv.block_table[(long long)seq * pv.bt_stride + blk];
  return ((page * pv.n_kv_heads + kv_head) * pv.page_size + slot) * (long long)pv.head_dim;
}

// Options of the tensor-core attention kernels beyond causal grouped-query attention with a window;
// all off when zero.  vd: width of a value row (0: head_dim; at most head_dim).  v_in_k: the values
// are the first vd channels of the keys (no value pool is read).  keep_first: with a window, keys at
// positions below it stay visible to every later query.  sink: one float per query head whose
// exponential joins the softmax denominator (unscaled; no key, no value).  gate: the output row
// [n_heads * vd] is multiplied by sigmoid(gate[t * gate_ld + ...]).  softcap > 0: a scaled score s
// becomes softcap * tanh(s / softcap) before the mask and the softmax.
struct AttnOptions {
  int vd;
  int v_in_k;
  int keep_first;
  const float* sink;
  const __nv_bfloat16* gate;
  long long gate_ld;
  float softcap;
};
// A raw dot product d (not yet scaled) under a soft cap, returned in the same unscaled units, so that
// the kernel's own multiplication by the scale gives cap * tanh(d * scale / cap).
__device__ __forceinline__ float softcap_raw(float d, float scale, float cap) {
  return cap * tanhf(d * (scale / cap)) / scale;
}

// Offset of the first of 16 consecutive positions [pos16, pos16 + 16), pos16 a multiple
// of 16: they share a page because the page size is a multiple of 16.  Rows of the
// granule are head_dim apart.  Kernels look this up once per granule and not once per
// row, so that no address waits on a load of the block table inside a copy loop.
__device__ __forceinline__ long long granule_offset(const PagedView& pv, int seq, int pos16, int kv_head) {
  return paged_offset(pv, seq, pos16, kv_head);
}

// ---------------------------------------------------------------------------- dependent launch
// Kernels of the decode step are launched so that the next kernel may start while this
// one is still running (programmatic dependent launch).  A kernel lets its own dependents go
// (pdl_launch), does what needs no input from its predecessor (fetching weights, which never
// change, and keys that earlier steps wrote) and waits for the predecessor to finish (pdl_wait)
// before it reads an activation or writes anything, so the result is that of running the
// kernels one after the other.  The streamed products and the small kernels between them let
// their dependents go FIRST: the blocks of the kernels that follow then take an SM's room the
// moment a block of the running kernel leaves it and fill their rings while the rest of that
// kernel and the small kernel after it finish (1.125 -> 1.095 ms for a decode step of batch 8).
// A dependent starts only when every block of its predecessor has let it go, that is when all
// of them are resident or done, so no kernel can wait for one that has no room to start.  The
// first kernel of a step (the embedding) waits before it lets go: nothing of a step starts
// before the step's inputs are in place.  Under a normal launch both are no-ops.
__device__ __forceinline__ void pdl_launch() { asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }

extern int g_mf_pdl;      // 1: launch with the dependent-launch attribute (set by mf_set_pdl)

// ---------------------------------------------------------------------------- per-device set-up
// cudaFuncSetAttribute and the SM count belong to a device, not to the process: a launcher keeps
// one flag per device ordinal (a function-local `static DeviceOnce`) and asks which device is
// current.  Ordinals beyond the table are refused by the launcher (MF_ERR_BAD_ARG).
#define MF_MAX_DEVICES 64
struct DeviceOnce {
  bool done[MF_MAX_DEVICES] = {};
};
inline int mf_current_device() {
  int d = -1;
  if (cudaGetDevice(&d) != cudaSuccess || d < 0 || d >= MF_MAX_DEVICES) return -1;
  return d;
}
// SMs of the current device (looked up once per device); 0 if it cannot be had
int mf_sm_count();

// ---------------------------------------------------------------------------- which kernels ran
// Every launcher counts the kernel it launches (also while a stream is capturing), so that a test
// of a whole model can say which kernels its steps went through: mf_kernel_launches(id).
enum MfKernel {
  MF_K_STREAM_ROWS = 0,       // few-row product, row-segment copies
  MF_K_STREAM_TMAP,           // few-row product, one tensor copy per stage
  MF_K_MID_ROWS,              // product of 17..128 rows (tcgen05, weights on the M side)
  MF_K_GEMM_TC,               // many-row product, tcgen05
  MF_K_GEMM_TC_SWIGLU,        // the same with the gated epilogue
  MF_K_GEMM_F32,
  MF_K_ATTN_GENERIC,
  MF_K_ATTN_PREFILL_MMA,
  MF_K_ATTN_PREFILL_TC,
  MF_K_ATTN_DECODE,           // split-key decode attention without tensor copies
  MF_K_ATTN_DECODE_TMA,       // with tensor copies, a merge kernel after it
  MF_K_ATTN_DECODE_TMA_MERGED,  // with tensor copies, merging its splits itself
  MF_K_ATTN_DECODE_MERGE,
  MF_K_EMBED_POSITIONS,       // embedding plus sinusoidal positions, into every residual stream
  MF_K_HYPER_NORM,            // write-back into several residual streams, read-in and grouped RMS norm
  MF_K_KV_STORE,              // projection biases and the cache write (key and value sizes may differ)
  MF_K_ATTN_TALKING,          // attention with heads mixed before the softmax, a block per token
  MF_K_ATTN_TALKING_TC,       // the same on tensor cores, a block per tile of queries
  MF_K_ATTN_TALKING_MERGE,    // joins the key splits of a decode launch of that kernel
  MF_K_DELTA_PREPARE,         // short convolutions, SiLU, unit norms of the delta rule's operands
  MF_K_DELTA_GATES,
  MF_K_DELTA_RECURRENCE,
  MF_K_DELTA_OUTPUT,
  MF_K_MOE_ROUTE,
  MF_K_MOE_ROWS,              // experts for few tokens: a block per (token, chosen expert)
  MF_K_MOE_COMBINE,
  MF_K_MOE_SORT,              // (token, choice) pairs ordered by expert
  MF_K_MOE_GROUPED,           // experts for many tokens: tensor-core tiles over the sorted pairs
  MF_K_ROPE_STORE,            // rotation in either pairing with the cache write (values may be the unrotated keys)
  MF_K_NORM_PAIR,             // residual add and two RMS norms of the same sum
  MF_K_LATENT_PREPARE,        // norms of the two latents, the shared rotated key part, the cache write
  MF_K_LATENT_QUERY,          // rotated query parts into the queries over the latent
  MF_K_HEAD_LINEAR,           // a product per head (few tokens)
  MF_K_HEAD_LINEAR_MMA,       // the same on tensor cores (many tokens)
  MF_K_RETENTION_PREPARE,     // rotation and key scaling of the retention's operands
  MF_K_RETENTION_RECURRENCE,  // the decayed state, token after token
  MF_K_RETENTION_CHUNKED,     // the same over runs of tokens as products
  MF_K_RETENTION_OUTPUT,      // per-head norm of the read-out and the gate
  MF_K_UNARY_ACT,             // an activation applied to every element (a feed-forward without a gate)
  MF_K_GEMM_TC_ACT,           // many-row product, tcgen05, with that activation in its epilogue
  MF_K_CONV_INPUT,            // a sublayer's input: the stream plus its short causal convolution
  MF_K_POSTNORM_ADD,          // RMS norm of a sublayer's output (or of two branches' weighted sum) added to the stream
  MF_K_QK_NORM_ROPE,          // biases, whole-projection norms, rotation of queries, keys and values, the cache write
  MF_K_ROTATE_ROWS,           // heads of a row turned by the position (an attention output turned back)
  MF_K_GDELTA_PREPARE,        // operands of the generalized delta rule: unit keys, removal rates, tanh of the low rank
  MF_K_GDELTA_RECURRENCE,     // its state, token after token
  MF_K_CONV_ACT,              // short causal convolution with bias and activation on columns of the projections
  MF_K_DECAY_RECURRENCE,      // a state per head with a decay per head or per key channel and token
  MF_K_DECAY_LOCAL,           // the same over segments from a zero state
  MF_K_SCAN_COMBINE,          // the states at the starts of the segments
  MF_K_GATED_NORM,            // gate, RMS norm in groups and weight of a read-out, gate before or after the norm
  MF_K_SELECTIVE_SCAN,        // a state per channel with token-dependent decay and input weights
  MF_K_SCAN_LOCAL,            // the same over segments from a zero state
  MF_K_LOW_RANK,              // a product with a narrow operand and the decay made of it
  MF_K_POST_NORM,             // a sublayer's output through a norm of its own into the stream, and the stream's next norm
  MF_K_QKV_CONV,              // convolved projections: norm per head, rotation, the cache write
  MF_K_SOFT_CAP,              // cap tanh(x / cap) on rows of logits
  MF_K_COUNT
};
extern unsigned long long g_mf_kernel_launches[MF_K_COUNT];
inline void mf_count(MfKernel k) { g_mf_kernel_launches[k]++; }

template <typename... KArgs, typename... Args>
inline cudaError_t launch_dep(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                              Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = g_mf_pdl ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}
