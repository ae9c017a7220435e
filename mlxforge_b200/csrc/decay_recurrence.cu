// Linear recurrences whose decay depends on the token, a state S [dim, vdim] in 32-bit per head:
//
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T ,     o_t = q_scale S_t^T q_t (+ skip_h v_t)
//
// in two forms:
//  * a decay per key channel and token (a [T, n_heads * dim] given), v as it is;
//  * a decay per head and token made from a step size: dt = softplus(x + dt_bias_h),
//    a = exp(-exp(A_log_h) dt) for all channels, and v_t is multiplied by dt on its way into S
//    (the skip connection takes it as it is).
// Query head h reads q and k of head h / (n_heads / n_qk).  Everything is 32-bit.
//
// An element of S depends on no other element, so the work spreads over (sequence, head, rows,
// columns); only the read-out sums over rows.  A block owns ROWS x COLS of a head's state (more rows
// than that give several partial read-outs, summed by whoever takes them), a thread 8 x 4 of
// them in registers, 4 to 16 lanes sharing a column; the operands of the coming tokens arrive
// through a ring of cp.async stages.  The read-outs of four tokens go through their sums over
// the lanes together, so that every lane ends with one of them.
//
// Over time the recurrence is serial, but linear: a long portion is cut into segments that run
// side by side.  First every segment but the last runs from a zero state and leaves its end state
// and the product of its decays (LOCAL); then one pass over the segments makes the state at the
// start of every one (decay_combine); then all segments run from there.  Portions that are short,
// or steps with enough heads and sequences to fill the GPU, run in one piece.  A step continues
// from the slot's state, so the result does not depend on how a prompt was cut beyond rounding.
//
// gated_norm_kernel takes the read-outs on: sum of the parts, gate silu(g), RMS norm in groups and
// weight, with the gate before or after the norm.
#include "common.cuh"

namespace {
constexpr int DC_CHUNK = 8;         // tokens per stage
constexpr int DC_STAGES = 3;
constexpr int DC_TR = 8;            // rows and columns of a thread
constexpr int DC_TC = 4;
constexpr int DC_NT = 4;            // tokens whose read-outs are summed together

__device__ __forceinline__ void dc_cp16(void* smem, const void* gmem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;\n" ::"r"(a), "l"(gmem) : "memory");
}
__device__ __forceinline__ void dc_cp4(void* smem, const void* gmem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(a), "l"(gmem) : "memory");
}
struct DcTrue { static constexpr bool value = true; };
struct DcFalse { static constexpr bool value = false; };
__device__ __forceinline__ float dc_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
}  // namespace

struct DecayRec {
  const float* q;                  // first element of the first token; rows *_ld floats apart
  const float* k;
  const float* v;
  int q_ld, k_ld, v_ld;
  const float* alpha;              // decays per channel, or null
  int alpha_ld;
  const float* dt;                 // step-size logits, one per head
  int dt_ld;
  const float* dt_bias;            // [n_heads]
  const float* a_log;              // [n_heads]
  const float* skip;               // [n_heads] or null
  float q_scale;
  float* state;
  long long state_stride;
  const int* seq_q_start;
  const int* seq_q_len;
  const int* slots;
  float* o;                        // [parts][T, n_heads * vdim]
  long long part_stride;
  float* seg_state;                // [n_seqs, n_seg, n_heads * dim * vdim]
  float* seg_decay;                // [n_seqs, n_seg, n_heads * (dim or 1)]
  int seg_len, n_seg;
  int n_heads, n_qk, dim, vdim;
  int vec;                         // rows come in aligned pieces of 16 bytes
};

// RL lanes share a column (rows RL * 8), CG groups of four columns
template <int RL, int CG, bool CHANNEL, bool LOCAL>
__global__ void __launch_bounds__(RL * CG)
decay_recurrence_kernel(DecayRec p) {
  constexpr int THREADS = RL * CG, ROWS = RL * DC_TR, COLS = CG * DC_TC;
  constexpr int NA = (LOCAL ? 1 : 2) + (CHANNEL ? 1 : 0);          // row arrays of a token: k, (a), (q)
  constexpr int TOK = NA * ROWS + COLS + 4;                        // floats of a token in a stage; the last: a, dt
  constexpr int A_AT = ROWS, Q_AT = (CHANNEL ? 2 : 1) * ROWS, V_AT = NA * ROWS, S_AT = V_AT + COLS;
  extern __shared__ __align__(16) float dc_sm[];                   // [STAGES][CHUNK][TOK]
  pdl_launch();
  pdl_wait();
  const int seq = blockIdx.x, n_cb = (p.vdim + COLS - 1) / COLS;
  const int seg = blockIdx.z;
  const int n_all = p.seq_q_len[seq];
  const int own_segs = (n_all + p.seg_len - 1) / p.seg_len;
  if (seg >= own_segs || (LOCAL && seg == own_segs - 1)) return;
  const int rg = blockIdx.y / (n_cb * p.n_heads);
  const int hc = blockIdx.y - rg * (n_cb * p.n_heads);
  const int h = hc / n_cb, c0 = (hc - h * n_cb) * COLS, r0 = rg * ROWS;
  const int hq = h / (p.n_heads / p.n_qk);
  const int rl = threadIdx.x % RL, cg = threadIdx.x / RL;
  const int start = p.seq_q_start[seq] + seg * p.seg_len, n = min(p.seg_len, n_all - seg * p.seg_len);
  const int rows_here = min(ROWS, p.dim - r0), cols_here = min(COLS, p.vdim - c0);
  if (rows_here < ROWS || cols_here < COLS) {        // the padding is never copied: zero once
    for (int i = threadIdx.x; i < DC_STAGES * DC_CHUNK * TOK; i += THREADS) dc_sm[i] = 0.f;
    __syncthreads();
  }
  const long long SS = (long long)p.n_heads * p.dim * p.vdim;
  const long long s_at = ((long long)h * p.dim + r0) * p.vdim + c0 + cg * DC_TC;
  float* slot_state = p.state + (long long)p.slots[seq] * p.state_stride + s_at;
  const float* S0 = own_segs > 1 ? p.seg_state + ((long long)seq * p.n_seg + seg) * SS + s_at : slot_state;
  // row i of a thread: ((i / 4) * RL + rl) * 4 + i % 4, so that the lanes of a column read 16-byte pieces side by side;
  // rows 2 i and 2 i + 1 stand in one register pair and are worked on by one instruction
  f32x2 s[DC_TR / 2][DC_TC];
#pragma unroll
  for (int i = 0; i < DC_TR / 2; i++) {
    float x[2][DC_TC];
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int r = ((i >> 1) * RL + rl) * 4 + (i & 1) * 2 + e;
#pragma unroll
      for (int c = 0; c < DC_TC; c++) x[e][c] = 0.f;
      if (!LOCAL && r < rows_here) {
        if (p.vec && cg * DC_TC < cols_here) {
          const float4 f = *reinterpret_cast<const float4*>(S0 + (long long)r * p.vdim);
          x[e][0] = f.x; x[e][1] = f.y; x[e][2] = f.z; x[e][3] = f.w;
        } else {
#pragma unroll
          for (int c = 0; c < DC_TC; c++)
            if (cg * DC_TC + c < cols_here) x[e][c] = S0[(long long)r * p.vdim + c];
        }
      }
    }
#pragma unroll
    for (int c = 0; c < DC_TC; c++) s[i][c] = pack2(x[0][c], x[1][c]);
  }
  const int n_chunks = (n + DC_CHUNK - 1) / DC_CHUNK;
  float neg_a = 0.f, dtb = 0.f, skip = 0.f, x_next = 0.f;
  if (!CHANNEL) {
    neg_a = -expf(p.a_log[h]);
    dtb = p.dt_bias[h];
    if ((int)threadIdx.x < min(DC_CHUNK, n)) x_next = p.dt[(long long)(start + threadIdx.x) * p.dt_ld + h];
  }
  if (!LOCAL && p.skip && rl == 0 && rg == 0) skip = p.skip[h];

  auto issue = [&](int chunk) {
    if (chunk < n_chunks) {
      float* st = dc_sm + (size_t)(chunk % DC_STAGES) * DC_CHUNK * TOK;
      const int nt = min(DC_CHUNK, n - chunk * DC_CHUNK);
      const long long tb = start + chunk * DC_CHUNK;
      if (p.vec) {
        constexpr int PT = NA * (ROWS / 4) + COLS / 4;
        for (int i = threadIdx.x; i < nt * PT; i += THREADS) {
          const int tok = i / PT, q = i - tok * PT;
          const long long t = tb + tok;
          float* dst = st + tok * TOK + q * 4;
          if (q < NA * (ROWS / 4)) {
            const int which = q / (ROWS / 4), r = (q - which * (ROWS / 4)) * 4;
            if (r < rows_here) {
              const float* src = which == 0 ? p.k + t * p.k_ld + hq * p.dim
                                 : (CHANNEL && which == 1) ? p.alpha + t * p.alpha_ld + h * p.dim
                                                           : p.q + t * p.q_ld + hq * p.dim;
              dc_cp16(dst, src + r0 + r);
            }
          } else {
            const int c = (q - NA * (ROWS / 4)) * 4;
            if (c < cols_here) dc_cp16(dst, p.v + t * p.v_ld + (long long)h * p.vdim + c0 + c);
          }
        }
      } else {
        constexpr int PT = NA * ROWS + COLS;
        for (int i = threadIdx.x; i < nt * PT; i += THREADS) {
          const int tok = i / PT, q = i - tok * PT;
          const long long t = tb + tok;
          float* dst = st + tok * TOK + q;
          if (q < NA * ROWS) {
            const int which = q / ROWS, r = q - which * ROWS;
            if (r < rows_here) {
              const float* src = which == 0 ? p.k + t * p.k_ld + hq * p.dim
                                 : (CHANNEL && which == 1) ? p.alpha + t * p.alpha_ld + h * p.dim
                                                           : p.q + t * p.q_ld + hq * p.dim;
              dc_cp4(dst, src + r0 + r);
            }
          } else {
            const int c = q - NA * ROWS;
            if (c < cols_here) dc_cp4(dst, p.v + t * p.v_ld + (long long)h * p.vdim + c0 + c);
          }
        }
      }
      if (!CHANNEL && (int)threadIdx.x < nt) {
        // decay and step size of a token; the logit of the chunk after this one is fetched meanwhile
        const float dt = dc_softplus(x_next + dtb);
        st[threadIdx.x * TOK + S_AT] = expf(neg_a * dt);
        st[threadIdx.x * TOK + S_AT + 1] = dt;
        const int nx = (chunk + 1) * DC_CHUNK + threadIdx.x;
        if (nx < n) x_next = p.dt[(long long)(start + nx) * p.dt_ld + h];
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
#pragma unroll
  for (int c = 0; c < DC_STAGES - 1; c++) issue(c);
  f32x2 prod[CHANNEL ? DC_TR / 2 : 1];             // LOCAL: the product of the decays
#pragma unroll
  for (int i = 0; i < (CHANNEL ? DC_TR / 2 : 1); i++) prod[i] = pack2(1.f, 1.f);
  float* o = p.o + (LOCAL ? 0 : (long long)rg * p.part_stride + (long long)h * p.vdim + c0 + cg * DC_TC);
  for (int chunk = 0; chunk < n_chunks; chunk++) {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(DC_STAGES - 2) : "memory");
    __syncthreads();                         // the stage has landed for all, and the stage read before is free
    issue(chunk + DC_STAGES - 1);
    const float* st = dc_sm + (size_t)(chunk % DC_STAGES) * DC_CHUNK * TOK;
    const int nt = min(DC_CHUNK, n - chunk * DC_CHUNK);
    // four tokens; `whole`: all four are there (the compiler may then overlap them)
    auto four = [&](int tt, auto whole) {
      float acc[DC_NT * DC_TC];
#pragma unroll
      for (int i = 0; i < DC_NT * DC_TC; i++) acc[i] = 0.f;
#pragma unroll
      for (int u = 0; u < DC_NT; u++) {
        if (decltype(whole)::value || tt + u < nt) {
          const float* row = st + (tt + u) * TOK;
          const float4 v4 = *reinterpret_cast<const float4*>(row + V_AT + cg * DC_TC);
          float v[DC_TC] = {v4.x, v4.y, v4.z, v4.w};
          f32x2 a2 = 0;
          if (!CHANNEL) {
            const float2 ad = *reinterpret_cast<const float2*>(row + S_AT);
            a2 = pack2(ad.x, ad.x);
            if (!LOCAL) {
#pragma unroll
              for (int c = 0; c < DC_TC; c++) acc[u * DC_TC + c] = skip * v[c];
            }
#pragma unroll
            for (int c = 0; c < DC_TC; c++) v[c] *= ad.y;
            if (LOCAL) prod[0] = mul2(prod[0], a2);
          }
          f32x2 v2[DC_TC], o2[DC_TC];
#pragma unroll
          for (int c = 0; c < DC_TC; c++) {
            v2[c] = pack2(v[c], v[c]);
            o2[c] = 0;
          }
#pragma unroll
          for (int i4 = 0; i4 < DC_TR / 4; i4++) {
            const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(row + (i4 * RL + rl) * 4);
            ulonglong2 a4 = make_ulonglong2(a2, a2), q4 = make_ulonglong2(0, 0);
            if (CHANNEL) {
              a4 = *reinterpret_cast<const ulonglong2*>(row + A_AT + (i4 * RL + rl) * 4);
              if (LOCAL) {
                prod[CHANNEL ? 2 * i4 : 0] = mul2(prod[CHANNEL ? 2 * i4 : 0], a4.x);
                prod[CHANNEL ? 2 * i4 + 1 : 0] = mul2(prod[CHANNEL ? 2 * i4 + 1 : 0], a4.y);
              }
            }
            if (!LOCAL) q4 = *reinterpret_cast<const ulonglong2*>(row + Q_AT + (i4 * RL + rl) * 4);
#pragma unroll
            for (int c = 0; c < DC_TC; c++) {
              s[2 * i4][c] = fma2(a4.x, s[2 * i4][c], mul2(k4.x, v2[c]));
              s[2 * i4 + 1][c] = fma2(a4.y, s[2 * i4 + 1][c], mul2(k4.y, v2[c]));
              if (!LOCAL) {
                o2[c] = fma2(s[2 * i4][c], q4.x, o2[c]);
                o2[c] = fma2(s[2 * i4 + 1][c], q4.y, o2[c]);
              }
            }
          }
          if (!LOCAL) {
#pragma unroll
            for (int c = 0; c < DC_TC; c++) {
              const float2 f = unpack2(o2[c]);
              acc[u * DC_TC + c] += f.x + f.y;
            }
          }
        }
      }
      if (!LOCAL) {
        // sums over the RL lanes of a column: every step halves the values a lane carries
        int base = 0;
#pragma unroll
        for (int w = 1, m = DC_NT * DC_TC; w < RL; w <<= 1) {
          const bool up = rl & w;
          const int half = m / 2;
#pragma unroll
          for (int i = 0; i < DC_NT * DC_TC / 2; i++)
            if (i < half) {
              const float send = up ? acc[i] : acc[i + half];
              const float keep = up ? acc[i + half] : acc[i];
              acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
            }
          base += up ? half : 0;
          m = half;
        }
        constexpr int LEFT = DC_NT * DC_TC / RL;       // values a lane ends with: consecutive columns of one token
        const int u = base / DC_TC, c = base % DC_TC;
        if (tt + u < nt) {
          float* dst = o + (long long)(start + chunk * DC_CHUNK + tt + u) * p.n_heads * p.vdim + c;
#pragma unroll
          for (int i = 0; i < LEFT; i++)
            if (cg * DC_TC + c + i < cols_here) dst[i] = acc[i] * p.q_scale;
        }
      }
    };
    int tt = 0;
    for (; tt + DC_NT <= nt; tt += DC_NT) four(tt, DcTrue{});
    if (tt < nt) four(tt, DcFalse{});
  }
  asm volatile("cp.async.wait_group 0;\n" ::: "memory");
  float* S1;
  if (LOCAL) {
    // the segment's own end state goes where the next segment's start state will stand
    S1 = p.seg_state + ((long long)seq * p.n_seg + seg + 1) * SS + s_at;
    if (CHANNEL) {
      if (cg == 0 && c0 == 0) {
        float* d = p.seg_decay + ((long long)seq * p.n_seg + seg) * p.n_heads * p.dim + h * p.dim + r0;
#pragma unroll
        for (int i = 0; i < DC_TR / 2; i++) {
          const int r = ((i >> 1) * RL + rl) * 4 + (i & 1) * 2;
          const float2 f = unpack2(prod[CHANNEL ? i : 0]);
          if (r < rows_here) d[r] = f.x;
          if (r + 1 < rows_here) d[r + 1] = f.y;
        }
      }
    } else if (threadIdx.x == 0 && c0 == 0 && rg == 0) {
      p.seg_decay[((long long)seq * p.n_seg + seg) * p.n_heads + h] = unpack2(prod[0]).x;
    }
  } else {
    if (seg != own_segs - 1) return;
    S1 = slot_state;
  }
#pragma unroll
  for (int i = 0; i < DC_TR / 2; i++) {
    float2 x[DC_TC];
#pragma unroll
    for (int c = 0; c < DC_TC; c++) x[c] = unpack2(s[i][c]);
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int r = ((i >> 1) * RL + rl) * 4 + (i & 1) * 2 + e;
      if (r < rows_here) {
        float* dst = S1 + (long long)r * p.vdim;
        if (p.vec && cg * DC_TC < cols_here) {
          *reinterpret_cast<float4*>(dst) = e ? make_float4(x[0].y, x[1].y, x[2].y, x[3].y)
                                              : make_float4(x[0].x, x[1].x, x[2].x, x[3].x);
        } else {
#pragma unroll
          for (int c = 0; c < DC_TC; c++)
            if (cg * DC_TC + c < cols_here) dst[c] = e ? x[c].y : x[c].x;
        }
      }
    }
  }
}

// seg_state[0] <- the slot's state; seg_state[i] <- decay[i-1] seg_state[i-1] + (local end state of segment i-1)
__global__ void __launch_bounds__(256)
decay_combine_kernel(float* __restrict__ seg_state, const float* __restrict__ seg_decay, const float* __restrict__ state,
                     long long state_stride, const int* __restrict__ seq_q_len, const int* __restrict__ slots,
                     int seg_len, int n_seg, int n_heads, int dim, int vdim, int per_channel) {
  pdl_launch();
  pdl_wait();
  const int seq = blockIdx.y;
  const int own = (seq_q_len[seq] + seg_len - 1) / seg_len;
  if (own < 2) return;
  const long long SS = (long long)n_heads * dim * vdim;
  const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= SS) return;
  const int hr = (int)(e / vdim);
  const int d_at = per_channel ? hr : hr / dim, d_n = per_channel ? n_heads * dim : n_heads;
  float S = state[(long long)slots[seq] * state_stride + e];
  float* base = seg_state + (long long)seq * n_seg * SS + e;
  const float* dec = seg_decay + (long long)seq * n_seg * d_n + d_at;
  base[0] = S;
  for (int i = 1; i < own; i += 8) {            // eight segments' loads at a time
    float l[8], d[8];
#pragma unroll
    for (int j = 0; j < 8; j++)
      if (i + j < own) {
        l[j] = base[(i + j) * SS];
        d[j] = dec[(long long)(i + j - 1) * d_n];
      }
#pragma unroll
    for (int j = 0; j < 8; j++)
      if (i + j < own) {
        S = fmaf(d[j], S, l[j]);
        base[(i + j) * SS] = S;
      }
  }
}

namespace {
struct DcShape {
  int rl, cg;
};
DcShape dc_shape(int dim, int vdim) {
  return DcShape{dim <= 32 ? 4 : dim <= 64 ? 8 : 16, vdim <= 32 ? 8 : 16};
}
}  // namespace

// Partial read-outs (row groups) that a launch writes, and blocks per sequence and segment.
MF_API int mf_decay_parts(int dim, int vdim) {
  const DcShape s = dc_shape(dim, vdim);
  return (dim + s.rl * DC_TR - 1) / (s.rl * DC_TR);
}
MF_API int mf_decay_blocks(int n_heads, int dim, int vdim) {
  const DcShape s = dc_shape(dim, vdim);
  return n_heads * mf_decay_parts(dim, vdim) * ((vdim + s.cg * DC_TC - 1) / (s.cg * DC_TC));
}

// Blocks of a launch that the GPU holds at a time (looked up once per device and shape).
template <int RL, int CG, bool CHANNEL, bool LOCAL>
static int dc_resident() {
  static int n[MF_MAX_DEVICES] = {};
  const int dev = mf_current_device();
  if (dev < 0) return 0;
  if (!n[dev]) {
    constexpr int NA = (LOCAL ? 1 : 2) + (CHANNEL ? 1 : 0);
    constexpr size_t smem = (size_t)DC_STAGES * DC_CHUNK * (NA * RL * DC_TR + CG * DC_TC + 4) * sizeof(float);
    if (smem > 48 * 1024 && cudaFuncSetAttribute(decay_recurrence_kernel<RL, CG, CHANNEL, LOCAL>,
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return 0;
    int per = 0;
    if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per, decay_recurrence_kernel<RL, CG, CHANNEL, LOCAL>, RL * CG, smem) !=
        cudaSuccess)
      return 0;
    n[dev] = per * mf_sm_count();
  }
  return n[dev];
}
#define DC_RESIDENT(RL, CG)                                                                                 \
  if (s.rl == RL && s.cg == CG)                                                                             \
  return per_channel ? (local ? dc_resident<RL, CG, true, true>() : dc_resident<RL, CG, true, false>())     \
                     : (local ? dc_resident<RL, CG, false, true>() : dc_resident<RL, CG, false, false>())
MF_API int mf_decay_resident(int dim, int vdim, int per_channel, int local) {
  const DcShape s = dc_shape(dim, vdim);
  DC_RESIDENT(4, 8);
  DC_RESIDENT(8, 8);
  DC_RESIDENT(16, 8);
  DC_RESIDENT(4, 16);
  DC_RESIDENT(8, 16);
  DC_RESIDENT(16, 16);
  return 0;
}
#undef DC_RESIDENT

template <int RL, int CG, bool CHANNEL, bool LOCAL>
static int dc_launch(const DecayRec& p, int n_seqs, cudaStream_t stream) {
  constexpr int NA = (LOCAL ? 1 : 2) + (CHANNEL ? 1 : 0);
  constexpr size_t smem = (size_t)DC_STAGES * DC_CHUNK * (NA * RL * DC_TR + CG * DC_TC + 4) * sizeof(float);
  static DeviceOnce once;
  const int dev = mf_current_device();
  if (dev < 0) return MF_ERR_BAD_ARG;
  if (!once.done[dev] && smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(decay_recurrence_kernel<RL, CG, CHANNEL, LOCAL>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  once.done[dev] = true;
  const int blocks = mf_decay_blocks(p.n_heads, p.dim, p.vdim);
  if (blocks > 65535 || p.n_seg > 65535) return MF_ERR_BAD_ARG;
  return (int)launch_dep(decay_recurrence_kernel<RL, CG, CHANNEL, LOCAL>, dim3(n_seqs, blocks, p.n_seg), dim3(RL * CG), smem,
                         stream, p);
}

template <bool CHANNEL, bool LOCAL>
static int dc_pick(const DecayRec& p, int n_seqs, cudaStream_t stream) {
  const DcShape s = dc_shape(p.dim, p.vdim);
  if (s.cg == 8) {
    if (s.rl == 4) return dc_launch<4, 8, CHANNEL, LOCAL>(p, n_seqs, stream);
    if (s.rl == 8) return dc_launch<8, 8, CHANNEL, LOCAL>(p, n_seqs, stream);
    return dc_launch<16, 8, CHANNEL, LOCAL>(p, n_seqs, stream);
  }
  if (s.rl == 4) return dc_launch<4, 16, CHANNEL, LOCAL>(p, n_seqs, stream);
  if (s.rl == 8) return dc_launch<8, 16, CHANNEL, LOCAL>(p, n_seqs, stream);
  return dc_launch<16, 16, CHANNEL, LOCAL>(p, n_seqs, stream);
}

MF_API int mf_decay_recurrence(const float* q, int q_ld, const float* k, int k_ld, const float* v, int v_ld,
                               const float* alpha, int alpha_ld, const float* dt, int dt_ld, const float* dt_bias,
                               const float* a_log, const float* skip, float q_scale, float* state,
                               long long state_stride, const int* seq_q_start, const int* seq_q_len, const int* slots,
                               float* o, long long part_stride, float* seg_state, float* seg_decay, int seg_len,
                               int n_seg, int n_seqs, int n_heads, int n_qk, int dim, int vdim, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || n_heads <= 0 || n_qk <= 0 || n_heads % n_qk || seg_len <= 0 || n_seg < 1)
    return MF_ERR_BAD_ARG;
  if (!alpha && (!dt || !dt_bias || !a_log)) return MF_ERR_BAD_ARG;
  if (skip && (alpha || q_scale != 1.0f)) return MF_ERR_BAD_ARG;
  if (n_seg > 1 && (!seg_state || !seg_decay)) return MF_ERR_BAD_ARG;
  auto al = [](const void* x) { return ((uintptr_t)x & 15) == 0; };
  const int vec = dim % 4 == 0 && vdim % 4 == 0 && q_ld % 4 == 0 && k_ld % 4 == 0 && v_ld % 4 == 0 && alpha_ld % 4 == 0 &&
                  state_stride % 4 == 0 && al(q) && al(k) && al(v) && al(alpha) && al(state) && al(seg_state);
  const DecayRec p{q, k, v, q_ld, k_ld, v_ld, alpha, alpha_ld, dt, dt_ld, dt_bias, a_log, skip, q_scale, state,
                   state_stride, seq_q_start, seq_q_len, slots, o, part_stride, seg_state, seg_decay, seg_len, n_seg,
                   n_heads, n_qk, dim, vdim, vec};
  int e;
  if (n_seg > 1) {
    mf_count(MF_K_DECAY_LOCAL);
    e = alpha ? dc_pick<true, true>(p, n_seqs, stream) : dc_pick<false, true>(p, n_seqs, stream);
    if (e) return e;
    const long long SS = (long long)n_heads * dim * vdim;
    mf_count(MF_K_SCAN_COMBINE);
    e = (int)launch_dep(decay_combine_kernel, dim3((unsigned)((SS + 255) / 256), n_seqs), dim3(256), 0, stream, seg_state,
                        (const float*)seg_decay, (const float*)state, state_stride, seq_q_len, slots, seg_len, n_seg,
                        n_heads, dim, vdim, alpha ? 1 : 0);
    if (e) return e;
  }
  mf_count(MF_K_DECAY_RECURRENCE);
  return alpha ? dc_pick<true, false>(p, n_seqs, stream) : dc_pick<false, false>(p, n_seqs, stream);
}

// ------------------------------------------------------------------ gate, grouped norm, weight
// x = sum of `n_parts` partial rows [T, width]; the row's `groups` equal parts are each divided by their
// root mean square and multiplied by w (`w_len` = width, or = the parts' size: shared by them) and by silu(gate):
// gate_first: the gate multiplies before the norm, else after it.  WARPS warps share a (token, group).
template <typename TO, int WARPS, int VEC>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ x, int n_parts, long long part_stride, const float* __restrict__ gate,
                  long long gate_ld, const float* __restrict__ w, int w_len, float eps, TO* __restrict__ out, int width,
                  int groups, int gate_first, long long total) {
  extern __shared__ __align__(16) float gn_sm[];       // [items of the block][group size]
  __shared__ float red[32];
  pdl_launch();
  pdl_wait();
  constexpr int ITEMS = 8 / WARPS;
  const int gs = width / groups;
  const int local = (threadIdx.x >> 5) / WARPS;
  const long long item = (long long)blockIdx.x * ITEMS + local;
  if (WARPS == 1 && item >= total) return;
  const int tid = threadIdx.x - local * WARPS * 32;
  const long long t = item / groups;
  const int c0 = (int)(item - t * groups) * gs;
  float* y = gn_sm + (size_t)local * gs;
  const float* row = x + t * width + c0;
  const float* g = gate + t * gate_ld + c0;
  float ss = 0.f;
  for (int i = tid * VEC; i < gs; i += WARPS * 32 * VEC) {
    float a[VEC], b[VEC];
    if constexpr (VEC == 4) {
      float4 f = *reinterpret_cast<const float4*>(row + i);
      for (int q = 1; q < n_parts; q++) {
        const float4 m = *reinterpret_cast<const float4*>(row + q * part_stride + i);
        f.x += m.x; f.y += m.y; f.z += m.z; f.w += m.w;
      }
      a[0] = f.x; a[1] = f.y; a[2] = f.z; a[3] = f.w;
      if (gate_first) {
        const float4 gg = *reinterpret_cast<const float4*>(g + i);
        b[0] = gg.x; b[1] = gg.y; b[2] = gg.z; b[3] = gg.w;
      }
    } else {
      a[0] = row[i];
      for (int q = 1; q < n_parts; q++) a[0] += row[q * part_stride + i];
      if (gate_first) b[0] = g[i];
    }
#pragma unroll
    for (int e = 0; e < VEC; e++) {
      if (gate_first) a[e] *= b[e] / (1.0f + expf(-b[e]));
      ss = fmaf(a[e], a[e], ss);
      y[i + e] = a[e];
    }
  }
  ss = WARPS == 1 ? warp_sum(ss) : block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)gs + eps);
  TO* o = out + t * width + c0;
  const float* wr = w + (w_len == gs ? 0 : c0);
  for (int i = tid * VEC; i < gs; i += WARPS * 32 * VEC) {       // every thread reads back what it wrote itself
    float r[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) {
      r[e] = y[i + e] * inv * wr[i + e];
      if (!gate_first) {
        const float b = g[i + e];
        r[e] *= b / (1.0f + expf(-b));
      }
    }
    if constexpr (VEC == 4 && sizeof(TO) == 2) {
      const __nv_bfloat162 p0 = __floats2bfloat162_rn(r[0], r[1]), p1 = __floats2bfloat162_rn(r[2], r[3]);
      uint2 pk;
      pk.x = *reinterpret_cast<const uint32_t*>(&p0);
      pk.y = *reinterpret_cast<const uint32_t*>(&p1);
      *reinterpret_cast<uint2*>(o + i) = pk;
    } else {
#pragma unroll
      for (int e = 0; e < VEC; e++) o[i + e] = from_f32<TO>(r[e]);
    }
  }
}

template <typename TO, int WARPS, int VEC>
static int gn_launch(const float* x, int n_parts, long long part_stride, const float* gate, long long gate_ld,
                     const float* w, int w_len, float eps, void* out, int T, int width, int groups, int gate_first,
                     cudaStream_t stream) {
  constexpr int ITEMS = 8 / WARPS;
  const size_t smem = (size_t)ITEMS * (width / groups) * sizeof(float);
  if (smem > 200 * 1024) return MF_ERR_BAD_ARG;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(gated_norm_kernel<TO, WARPS, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const long long total = (long long)T * groups;
  return (int)launch_dep(gated_norm_kernel<TO, WARPS, VEC>, dim3((unsigned)((total + ITEMS - 1) / ITEMS)), dim3(256), smem,
                         stream, x, n_parts, part_stride, gate, gate_ld, w, w_len, eps, (TO*)out, width, groups, gate_first,
                         total);
}

MF_API int mf_gated_norm(const float* x, int n_parts, long long part_stride, const float* gate, long long gate_ld,
                         const float* w, int w_len, float eps, void* out, int out_dtype, int T, int width, int groups,
                         int gate_first, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n_parts < 1 || groups < 1 || width <= 0 || width % groups || (w_len != width && w_len != width / groups)) return MF_ERR_BAD_ARG;
  const int gs = width / groups;
  const bool vec = gs % 4 == 0 && width % 4 == 0 && gate_ld % 4 == 0 && part_stride % 4 == 0 && ((uintptr_t)x & 15) == 0 &&
                   ((uintptr_t)gate & 15) == 0 && ((uintptr_t)out & 15) == 0;
  mf_count(MF_K_GATED_NORM);
#define GN_GO(TO, W, V) \
  return gn_launch<TO, W, V>(x, n_parts, part_stride, gate, gate_ld, w, w_len, eps, out, T, width, groups, gate_first, stream)
#define GN_PICK(TO)                \
  do {                             \
    if (gs <= 512) {               \
      if (vec) GN_GO(TO, 1, 4);    \
      GN_GO(TO, 1, 1);             \
    }                              \
    if (vec) GN_GO(TO, 8, 4);      \
    GN_GO(TO, 8, 1);               \
  } while (0)
  if (out_dtype == MF_F32) GN_PICK(float);
  if (out_dtype == MF_BF16) GN_PICK(__nv_bfloat16);
#undef GN_PICK
#undef GN_GO
  return MF_ERR_BAD_DTYPE;
}
