// Selective scan: a state S [channels, state] in 32-bit whose decay and input weights depend on the token:
//
//   dt_c = softplus(x_c + bias_c)
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n ,    y_c = sum_n S[c, n] C_n + D_c u_c
//   out_c = y_c silu(z_c)
//
// u [T, channels], the step-size logits x, the gates z and B, C (shared by the channels) are rows of
// 32-bit numbers.  No element of S depends on another: a thread holds SS_NS states of one channel in
// registers, LN lanes share a channel (their read-outs are summed by shuffles), a block owns
// SS_THREADS / LN channels.  The operands of a run of tokens are made once per channel (step size,
// dt u, D u, silu(z)) and staged in shared memory while the run before is worked on.
//
// A long portion is cut into segments that run side by side, as in decay_recurrence.cu: every segment but
// the last from a zero state (LOCAL), leaving its end state and its sum of step sizes, from which the
// segment's decay is exp(A sum dt); one pass over the segments (scan_combine); all segments from the start
// states.  A step continues from the slot's state.
//
// low_rank_kernel: out = f(bias + W low) for a narrow `low`, f the identity or the decay of gated linear
// attention, sigmoid(.)^(1/tau).
#include "common.cuh"

namespace {
constexpr int SS_NS = 16;            // states of a thread
constexpr int SS_THREADS = 128;
constexpr int SS_CHUNK = 8;          // tokens per stage
__device__ __forceinline__ float ss_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float ss_silu(float x) { return x / (1.0f + expf(-x)); }
// FAST: the exponents were multiplied by log2 e and the special function unit's power of two (its relative error is
// below 2^-22) is the decay; else expf.
template <bool FAST>
__device__ __forceinline__ float ss_exp(float x) {
  if constexpr (FAST) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
  } else {
    return expf(x);
  }
}
}  // namespace

struct ScanArgs {
  const float* u;              // [T, channels]
  const float* dt;             // logits, rows dt_ld floats apart
  int dt_ld;
  const float* dt_bias;        // [channels]
  const float* z;              // rows z_ld apart
  int z_ld;
  const float* bc;             // B then C of a token, `n_state` each; rows bc_ld apart
  int bc_ld;
  const float* A;              // [channels, n_state], negative
  const float* D;              // [channels]
  float* state;                // [channels, n_state] per slot
  long long state_stride;
  const int* seq_q_start;
  const int* seq_q_len;
  const int* slots;
  float* seg_state;            // [n_seqs, n_seg, channels * n_state]
  float* seg_dt;               // [n_seqs, n_seg, channels]
  int seg_len, n_seg, channels, n_state;
};

template <typename TO, int LN, bool LOCAL, bool FAST>
__global__ void __launch_bounds__(SS_THREADS)
selective_scan_kernel(ScanArgs p, TO* __restrict__ out) {
  constexpr int CB = SS_THREADS / LN;                        // channels of the block
  constexpr int ITEMS = (SS_CHUNK * CB + SS_THREADS - 1) / SS_THREADS;
  constexpr int NP = LN * SS_NS;                             // states, padded
  extern __shared__ __align__(16) float ss_sm[];
  float4* op = reinterpret_cast<float4*>(ss_sm);             // [2][CHUNK][CB]: dt, dt u, D u, silu(z)
  float* bc = ss_sm + 2 * SS_CHUNK * CB * 4;                 // [2][CHUNK][2 NP]
  pdl_launch();
  pdl_wait();
  const int seq = blockIdx.x, seg = blockIdx.z;
  const int n_all = p.seq_q_len[seq];
  const int own_segs = (n_all + p.seg_len - 1) / p.seg_len;
  if (seg >= own_segs || (LOCAL && seg == own_segs - 1)) return;
  const int start = p.seq_q_start[seq] + seg * p.seg_len, n = min(p.seg_len, n_all - seg * p.seg_len);
  const int cb0 = blockIdx.y * CB;
  const int cl = threadIdx.x / LN, ln = threadIdx.x % LN;
  const int c = cb0 + cl;
  const bool live = c < p.channels;
  const int N = p.n_state;
  if (N < NP)                                                // the padding of B and C is never written again
    for (int i = threadIdx.x; i < 2 * SS_CHUNK * 2 * NP; i += SS_THREADS) bc[i] = 0.f;
  const long long SSZ = (long long)p.channels * N;
  float* slot_state = p.state + (long long)p.slots[seq] * p.state_stride;
  const float* S0 = own_segs > 1 ? p.seg_state + ((long long)seq * p.n_seg + seg) * SSZ : slot_state;
  // state i of a thread: ((i / 4) * LN + ln) * 4 + i % 4; states 2 i and 2 i + 1 stand in one register pair
  f32x2 s[SS_NS / 2], A[SS_NS / 2];
  const bool whole = (N & 3) == 0;                           // states come in pieces of 16 bytes
#pragma unroll
  for (int i4 = 0; i4 < SS_NS / 4; i4++) {
    const int m = (i4 * LN + ln) * 4;
    float a[4] = {0.f, 0.f, 0.f, 0.f}, x[4] = {0.f, 0.f, 0.f, 0.f};
    if (live && m < N) {
      const long long at = (long long)c * N + m;
      if (whole) {
        const float4 f = *reinterpret_cast<const float4*>(p.A + at);
        a[0] = f.x; a[1] = f.y; a[2] = f.z; a[3] = f.w;
        if (!LOCAL) {
          const float4 g = *reinterpret_cast<const float4*>(S0 + at);
          x[0] = g.x; x[1] = g.y; x[2] = g.z; x[3] = g.w;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++)
          if (m + e < N) {
            a[e] = p.A[at + e];
            if (!LOCAL) x[e] = S0[at + e];
          }
      }
    }
    if (FAST) {
#pragma unroll
      for (int e = 0; e < 4; e++) a[e] *= 1.4426950408889634f;
    }
    A[2 * i4] = pack2(a[0], a[1]);
    A[2 * i4 + 1] = pack2(a[2], a[3]);
    s[2 * i4] = pack2(x[0], x[1]);
    s[2 * i4 + 1] = pack2(x[2], x[3]);
  }
  // operands of the coming run: this thread's (token, channel) items, fetched into registers a run ahead
  float rdt[ITEMS], ru[ITEMS], rz[ITEMS];
  const int n_chunks = (n + SS_CHUNK - 1) / SS_CHUNK;
  auto fetch = [&](int chunk) {
#pragma unroll
    for (int j = 0; j < ITEMS; j++) {
      const int i = threadIdx.x + j * SS_THREADS;
      const int tok = i / CB, ch = cb0 + i % CB;
      rdt[j] = ru[j] = rz[j] = 0.f;
      if (i < SS_CHUNK * CB && chunk * SS_CHUNK + tok < n && ch < p.channels) {
        const long long t = start + chunk * SS_CHUNK + tok;
        rdt[j] = p.dt[t * p.dt_ld + ch];
        ru[j] = p.u[t * p.channels + ch];
        if (!LOCAL) rz[j] = p.z[t * p.z_ld + ch];
      }
    }
  };
  constexpr int WHICH = LOCAL ? 1 : 2;                       // B alone, or B and C
  auto fetch_bc = [&](int chunk) {
    float* dst = bc + (chunk & 1) * SS_CHUNK * 2 * NP;
    const int nt = min(SS_CHUNK, n - chunk * SS_CHUNK);
    for (int i = threadIdx.x; i < nt * WHICH * N; i += SS_THREADS) {
      const int tok = i / (WHICH * N), r = i - tok * WHICH * N;
      const int which = r >= N, m = r - which * N;
      const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst + (tok * 2 + which) * NP + m);
      const float* src = p.bc + (long long)(start + chunk * SS_CHUNK + tok) * p.bc_ld + r;
      asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(a), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  auto stage = [&](int chunk) {
    float4* dst = op + (chunk & 1) * SS_CHUNK * CB;
#pragma unroll
    for (int j = 0; j < ITEMS; j++) {
      const int i = threadIdx.x + j * SS_THREADS;
      const int ch = cb0 + i % CB;
      if (i < SS_CHUNK * CB && ch < p.channels) {
        const float dt = ss_softplus(rdt[j] + p.dt_bias[ch]);
        dst[i] = make_float4(dt, dt * ru[j], LOCAL ? 0.f : p.D[ch] * ru[j], LOCAL ? 0.f : ss_silu(rz[j]));
      }
    }
  };
  if (N < NP) __syncthreads();
  fetch(0);
  fetch_bc(0);
  stage(0);
  float dt_sum = 0.f;
  for (int chunk = 0; chunk < n_chunks; chunk++) {
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();               // the run's operands are in place, and the run before is done with its buffers
    if (chunk + 1 < n_chunks) {
      fetch(chunk + 1);
      fetch_bc(chunk + 1);
    }
    const float4* o4 = op + (chunk & 1) * SS_CHUNK * CB;
    const float* bcs = bc + (chunk & 1) * SS_CHUNK * 2 * NP;
    const int nt = min(SS_CHUNK, n - chunk * SS_CHUNK);
#pragma unroll 2
    for (int tok = 0; tok < nt; tok++) {
      const float4 w = o4[tok * CB + cl];
      const float* B = bcs + tok * 2 * NP;
      const f32x2 dt2 = pack2(w.x, w.x), du2 = pack2(w.y, w.y);
      f32x2 y2 = 0;
#pragma unroll
      for (int i4 = 0; i4 < SS_NS / 4; i4++) {
        const ulonglong2 b4 = *reinterpret_cast<const ulonglong2*>(B + (i4 * LN + ln) * 4);
        const float2 e0 = unpack2(mul2(dt2, A[2 * i4])), e1 = unpack2(mul2(dt2, A[2 * i4 + 1]));
        s[2 * i4] = fma2(pack2(ss_exp<FAST>(e0.x), ss_exp<FAST>(e0.y)), s[2 * i4], mul2(du2, b4.x));
        s[2 * i4 + 1] = fma2(pack2(ss_exp<FAST>(e1.x), ss_exp<FAST>(e1.y)), s[2 * i4 + 1], mul2(du2, b4.y));
        if (!LOCAL) {
          const ulonglong2 c4 = *reinterpret_cast<const ulonglong2*>(B + NP + (i4 * LN + ln) * 4);
          y2 = fma2(s[2 * i4], c4.x, y2);
          y2 = fma2(s[2 * i4 + 1], c4.y, y2);
        }
      }
      const float2 yy = unpack2(y2);
      float y = yy.x + yy.y;
      if (LOCAL) {
        dt_sum += w.x;
      } else {
#pragma unroll
        for (int m = 1; m < LN; m <<= 1) y += __shfl_xor_sync(0xffffffffu, y, m);
        if (live && ln == 0) out[(long long)(start + chunk * SS_CHUNK + tok) * p.channels + c] = from_f32<TO>((y + w.z) * w.w);
      }
    }
    if (chunk + 1 < n_chunks) stage(chunk + 1);
  }
  float* S1;
  if (LOCAL) {
    S1 = p.seg_state + ((long long)seq * p.n_seg + seg + 1) * SSZ;
    if (live && ln == 0) p.seg_dt[((long long)seq * p.n_seg + seg) * p.channels + c] = dt_sum;
  } else {
    if (seg != own_segs - 1) return;
    S1 = slot_state;
  }
#pragma unroll
  for (int i4 = 0; i4 < SS_NS / 4; i4++) {
    const int m = (i4 * LN + ln) * 4;
    if (live && m < N) {
      float* dst = S1 + (long long)c * N + m;
      const float2 x0 = unpack2(s[2 * i4]), x1 = unpack2(s[2 * i4 + 1]);
      if (whole) {
        *reinterpret_cast<float4*>(dst) = make_float4(x0.x, x0.y, x1.x, x1.y);
      } else {
        dst[0] = x0.x;
        if (m + 1 < N) dst[1] = x0.y;
        if (m + 2 < N) dst[2] = x1.x;
        if (m + 3 < N) dst[3] = x1.y;
      }
    }
  }
}

// seg_state[0] <- the slot's state; seg_state[i] <- exp(A sum dt of segment i-1) seg_state[i-1] + (local end state)
__global__ void __launch_bounds__(256)
scan_combine_kernel(float* __restrict__ seg_state, const float* __restrict__ seg_dt, const float* __restrict__ A,
                    const float* __restrict__ state, long long state_stride, const int* __restrict__ seq_q_len,
                    const int* __restrict__ slots, int seg_len, int n_seg, int channels, int n_state) {
  pdl_launch();
  pdl_wait();
  const int seq = blockIdx.y;
  const int own = (seq_q_len[seq] + seg_len - 1) / seg_len;
  if (own < 2) return;
  const long long SSZ = (long long)channels * n_state;
  const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= SSZ) return;
  const int c = (int)(e / n_state);
  const float a = A[e];
  float S = state[(long long)slots[seq] * state_stride + e];
  float* base = seg_state + (long long)seq * n_seg * SSZ + e;
  const float* sd = seg_dt + (long long)seq * n_seg * channels + c;
  base[0] = S;
  for (int i = 1; i < own; i += 8) {            // eight segments' loads at a time
    float l[8], d[8];
#pragma unroll
    for (int j = 0; j < 8; j++)
      if (i + j < own) {
        l[j] = base[(i + j) * SSZ];
        d[j] = sd[(long long)(i + j - 1) * channels];
      }
#pragma unroll
    for (int j = 0; j < 8; j++)
      if (i + j < own) {
        S = fmaf(expf(a * d[j]), S, l[j]);
        base[(i + j) * SSZ] = S;
      }
  }
}

static int ss_lanes(int n_state) {
  int ln = 1;
  while (ln * SS_NS < n_state) ln *= 2;
  return ln;
}

// Blocks per sequence and segment; 0: too many states.
MF_API int mf_scan_blocks(int channels, int n_state) {
  const int ln = ss_lanes(n_state);
  if (ln > 32) return 0;
  const int cb = SS_THREADS / ln;
  return (channels + cb - 1) / cb;
}

template <typename TO, int LN, bool LOCAL, bool FAST>
struct SsKernel {
  static constexpr int CB = SS_THREADS / LN;
  static constexpr size_t smem = (size_t)(2 * SS_CHUNK * CB * 4 + 2 * SS_CHUNK * 2 * LN * SS_NS) * sizeof(float);
  // blocks that the GPU holds at a time (looked up once per device); 0: it cannot run
  static int resident() {
    static int n[MF_MAX_DEVICES] = {};
    const int dev = mf_current_device();
    if (dev < 0) return 0;
    if (!n[dev]) {
      if (smem > 48 * 1024 && cudaFuncSetAttribute(selective_scan_kernel<TO, LN, LOCAL, FAST>,
                                                   cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return 0;
      int per = 0;
      if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per, selective_scan_kernel<TO, LN, LOCAL, FAST>, SS_THREADS, smem) !=
          cudaSuccess)
        return 0;
      n[dev] = per * mf_sm_count();
    }
    return n[dev];
  }
  static int launch(const ScanArgs& p, void* out, int n_seqs, cudaStream_t stream) {
    if (resident() <= 0) return MF_ERR_BAD_ARG;
    return (int)launch_dep(selective_scan_kernel<TO, LN, LOCAL, FAST>, dim3(n_seqs, (p.channels + CB - 1) / CB, p.n_seg),
                           dim3(SS_THREADS), smem, stream, p, (TO*)out);
  }
};
#define SS_BY_LANES(n_state, TO, LOCAL, FAST, CALL)             \
  switch (ss_lanes(n_state)) {                                  \
    case 1: return SsKernel<TO, 1, LOCAL, FAST>::CALL;          \
    case 2: return SsKernel<TO, 2, LOCAL, FAST>::CALL;          \
    case 4: return SsKernel<TO, 4, LOCAL, FAST>::CALL;          \
    case 8: return SsKernel<TO, 8, LOCAL, FAST>::CALL;          \
    case 16: return SsKernel<TO, 16, LOCAL, FAST>::CALL;        \
    case 32: return SsKernel<TO, 32, LOCAL, FAST>::CALL;        \
  }

template <typename TO, bool LOCAL, bool FAST>
static int ss_pick(const ScanArgs& p, void* out, int n_seqs, cudaStream_t stream) {
  SS_BY_LANES(p.n_state, TO, LOCAL, FAST, launch(p, out, n_seqs, stream))
  return MF_ERR_BAD_ARG;
}
template <typename TO, bool LOCAL, bool FAST>
static int ss_resident(int n_state) {
  SS_BY_LANES(n_state, TO, LOCAL, FAST, resident())
  return 0;
}
// Blocks that the GPU holds at a time, of the serving (bfloat16) form; `local`: of the pass from a zero state.
MF_API int mf_scan_resident(int n_state, int local) {
  return local ? ss_resident<float, true, true>(n_state) : ss_resident<__nv_bfloat16, false, true>(n_state);
}

MF_API int mf_selective_scan(const float* u, const float* dt, int dt_ld, const float* dt_bias, const float* z, int z_ld,
                             const float* bc, int bc_ld, const float* A, const float* D, float* state,
                             long long state_stride, const int* seq_q_start, const int* seq_q_len, const int* slots,
                             float* seg_state, float* seg_dt, int seg_len, int n_seg, void* out, int out_dtype,
                             int n_seqs, int channels, int n_state, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  const int blocks = n_state > 0 && channels > 0 ? mf_scan_blocks(channels, n_state) : 0;
  if (blocks < 1 || blocks > 65535 || seg_len <= 0 || n_seg < 1 || n_seg > 65535) return MF_ERR_BAD_ARG;
  if (n_seg > 1 && (!seg_state || !seg_dt)) return MF_ERR_BAD_ARG;
  // states in pieces of 16 bytes are read so
  if (n_state % 4 == 0 && (((uintptr_t)state | (uintptr_t)A | (uintptr_t)seg_state) & 15 || state_stride % 4))
    return MF_ERR_BAD_ARG;
  if (out_dtype != MF_F32 && out_dtype != MF_BF16) return MF_ERR_BAD_DTYPE;
  const ScanArgs p{u, dt, dt_ld, dt_bias, z, z_ld, bc, bc_ld, A, D, state, state_stride, seq_q_start, seq_q_len, slots,
                   seg_state, seg_dt, seg_len, n_seg, channels, n_state};
  if (n_seg > 1) {
    mf_count(MF_K_SCAN_LOCAL);
    int e = out_dtype == MF_F32 ? ss_pick<float, true, false>(p, nullptr, n_seqs, stream)
                                : ss_pick<float, true, true>(p, nullptr, n_seqs, stream);
    if (e) return e;
    const long long SSZ = (long long)channels * n_state;
    mf_count(MF_K_SCAN_COMBINE);
    e = (int)launch_dep(scan_combine_kernel, dim3((unsigned)((SSZ + 255) / 256), n_seqs), dim3(256), 0, stream, seg_state,
                        (const float*)seg_dt, A, (const float*)state, state_stride, seq_q_len, slots, seg_len, n_seg,
                        channels, n_state);
    if (e) return e;
  }
  mf_count(MF_K_SELECTIVE_SCAN);
  return out_dtype == MF_F32 ? ss_pick<float, false, false>(p, out, n_seqs, stream)
                             : ss_pick<__nv_bfloat16, false, true>(p, out, n_seqs, stream);
}

// ------------------------------------------------------------------ a narrow product and what follows it
// out [T, n] (32-bit) = f(bias + low W^T): low [T, R] 32-bit rows `ld` floats apart, wt [R, n] the weight
// transposed (32-bit or bfloat16).  f: 0 the identity, 1 sigmoid(.)^(1/tau) = exp(-softplus(-x) / tau).
// SPLIT (few tokens): the eight warps of a block share 32 channels and split R; else a warp owns LR_TOK
// tokens of its own and the block's weights lie in shared memory.
namespace {
constexpr int LR_TOK = 8;
constexpr int LR_PIECE = 128;        // of the rank, at a time
__device__ __forceinline__ float lr_act(float x, int f, float inv_tau) {
  if (f == 0) return x;
  const float nx = -x;
  return expf(-ss_softplus(nx) * inv_tau);
}
}  // namespace

template <typename TW>
__global__ void __launch_bounds__(256)
low_rank_split_kernel(const float* __restrict__ low, int ld, const TW* __restrict__ wt, const float* __restrict__ bias,
                      int f, float inv_tau, float* __restrict__ out, int T, int R, int n) {
  __shared__ float part[8][LR_TOK][32];
  __shared__ float ls[LR_TOK][LR_PIECE];
  pdl_launch();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int j = blockIdx.x * 32 + lane, t0 = blockIdx.y * LR_TOK;
  const int nt = min(LR_TOK, T - t0);
  float acc[LR_TOK];
#pragma unroll
  for (int u = 0; u < LR_TOK; u++) acc[u] = 0.f;
  for (int r0 = 0; r0 < R; r0 += LR_PIECE) {
    const int nr = min(LR_PIECE, R - r0);
    float w[LR_PIECE / 8];          // the weights never change: the first piece's are fetched before the wait
#pragma unroll
    for (int q = 0; q < LR_PIECE / 8; q++) {
      const int r = q * 8 + warp;
      w[q] = (r < nr && j < n) ? to_f32<TW>(wt[(long long)(r0 + r) * n + j]) : 0.f;
    }
    if (r0 == 0) pdl_wait();
    else __syncthreads();
    for (int i = threadIdx.x; i < LR_TOK * LR_PIECE; i += 256) {
      const int u = i / LR_PIECE, r = i - u * LR_PIECE;
      ls[u][r] = (u < nt && r < nr) ? low[(long long)(t0 + u) * ld + r0 + r] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int q = 0; q < LR_PIECE / 8; q++)
#pragma unroll
      for (int u = 0; u < LR_TOK; u++) acc[u] = fmaf(w[q], ls[u][q * 8 + warp], acc[u]);
  }
#pragma unroll
  for (int u = 0; u < LR_TOK; u++) part[warp][u][lane] = acc[u];
  __syncthreads();
  // warp u finishes token u
  if (warp < nt && j < n) {
    float a = bias ? bias[j] : 0.f;
#pragma unroll
    for (int q = 0; q < 8; q++) a += part[q][warp][lane];
    out[(long long)(t0 + warp) * n + j] = lr_act(a, f, inv_tau);
  }
}

template <typename TW>
__global__ void __launch_bounds__(256)
low_rank_kernel(const float* __restrict__ low, int ld, const TW* __restrict__ wt, const float* __restrict__ bias, int f,
                float inv_tau, float* __restrict__ out, int T, int R, int n) {
  extern __shared__ __align__(16) float lr_sm[];       // weights [R][32], then low [8 * LR_TOK][R4]
  const int R4 = (R + 3) & ~3;
  float* ws = lr_sm;
  float* ls = lr_sm + R4 * 32;
  pdl_launch();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int j = blockIdx.x * 32 + lane, t0 = blockIdx.y * 8 * LR_TOK;
  for (int r = warp; r < R4; r += 8) ws[r * 32 + lane] = (r < R && j < n) ? to_f32<TW>(wt[(long long)r * n + j]) : 0.f;
  pdl_wait();
  const int nb = min(8 * LR_TOK, T - t0);
  for (int i = threadIdx.x; i < 8 * LR_TOK * R4; i += 256) {
    const int u = i / R4, r = i - u * R4;
    ls[i] = (u < nb && r < R) ? low[(long long)(t0 + u) * ld + r] : 0.f;
  }
  __syncthreads();
  float acc[LR_TOK];
  const float b = (bias && j < n) ? bias[j] : 0.f;
#pragma unroll
  for (int u = 0; u < LR_TOK; u++) acc[u] = b;
  const float* lw = ls + warp * LR_TOK * R4;
  for (int r = 0; r < R4; r += 4) {
    const float w0 = ws[r * 32 + lane], w1 = ws[(r + 1) * 32 + lane], w2 = ws[(r + 2) * 32 + lane], w3 = ws[(r + 3) * 32 + lane];
#pragma unroll
    for (int u = 0; u < LR_TOK; u++) {
      const float4 x = *reinterpret_cast<const float4*>(lw + u * R4 + r);
      acc[u] = fmaf(w3, x.w, fmaf(w2, x.z, fmaf(w1, x.y, fmaf(w0, x.x, acc[u]))));
    }
  }
  if (j < n)
#pragma unroll
    for (int u = 0; u < LR_TOK; u++) {
      const int t = t0 + warp * LR_TOK + u;
      if (t < T) out[(long long)t * n + j] = lr_act(acc[u], f, inv_tau);
    }
}

MF_API int mf_low_rank(const float* low, int ld, const void* wt, int w_dtype, const float* bias, int f, float tau,
                       float* out, int T, int R, int n, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (R <= 0 || n <= 0 || ld < R || f < 0 || f > 1 || !(tau != 0.f)) return MF_ERR_BAD_ARG;
  if (w_dtype != MF_F32 && w_dtype != MF_BF16) return MF_ERR_BAD_DTYPE;
  mf_count(MF_K_LOW_RANK);
  const float inv_tau = 1.0f / tau;
  const unsigned gx = (n + 31) / 32;
  const size_t smem = (size_t)((R + 3) & ~3) * (32 + 8 * LR_TOK) * sizeof(float);
  const bool split = T <= 64 || smem > 200 * 1024;
  if (split) {
    const dim3 grid(gx, (T + LR_TOK - 1) / LR_TOK);
    if (grid.y > 65535) return MF_ERR_BAD_ARG;
    if (w_dtype == MF_F32)
      return (int)launch_dep(low_rank_split_kernel<float>, grid, dim3(256), 0, stream, low, ld, (const float*)wt, bias, f,
                             inv_tau, out, T, R, n);
    return (int)launch_dep(low_rank_split_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, low, ld,
                           (const __nv_bfloat16*)wt, bias, f, inv_tau, out, T, R, n);
  }
  const dim3 grid(gx, (T + 8 * LR_TOK - 1) / (8 * LR_TOK));
  if (grid.y > 65535) return MF_ERR_BAD_ARG;
#define LR_GO(TW)                                                                                                   \
  do {                                                                                                              \
    if (smem > 48 * 1024) {                                                                                         \
      cudaError_t e = cudaFuncSetAttribute(low_rank_kernel<TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return (int)e;                                                                          \
    }                                                                                                               \
    return (int)launch_dep(low_rank_kernel<TW>, grid, dim3(256), smem, stream, low, ld, (const TW*)wt, bias, f, inv_tau, \
                           out, T, R, n);                                                                           \
  } while (0)
  if (w_dtype == MF_F32) LR_GO(float);
  LR_GO(__nv_bfloat16);
#undef LR_GO
}
