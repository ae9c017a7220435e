// Queries, keys and values of an attention whose projections pass a short causal convolution over
// time first: convolution, root-mean-square norm per head, rotation and the cache write in one
// kernel, from the 32-bit rows of the projection.
//
//   y_t[c] = sum_j w[c, j] u_(t - taps + 1 + j)[c]     on every channel of q, k and v (zeros before the
//                                                       sequence's start, no bias, no activation)
//   q, k <- rms(y over a head's channels) * weight      (weights shared by the heads; null: no norm)
//   rotation of the first `rot` channels of a head of q and k, pair (i, i + rot/2), by position * inv[i];
//   values are convolved and nothing else
//
// A row of `proj` (rows `ld` floats apart) holds the query heads, the key heads and the value heads; a
// layer that reads another layer's keys and values has query heads alone (n_kv = 0).  The last taps-1
// rows of a sequence's projections stay in its state slot ([taps-1, channels] at `tail_off`), so a step
// goes on from where the step before ended however the tokens were cut.
//
// A warp owns a head over a run of consecutive tokens: a lane holds two neighbouring channels of every
// 64, the convolution's window stays in registers, so every input is read once; the cosines and sines
// of the run's positions are worked out once for all heads of the block.  Everything is 32-bit
// (angles in double where a float64 table is given) and is rounded once, on its way into q_out
// [T, n_heads * hd] and the pages.  Where every sequence of the step brings one token a head's warp is
// the only reader of its columns of the slot and moves them on itself; else a second kernel does.
#include "conv_tail.cuh"
#include "rotary.cuh"

namespace {

struct QkvConv {
  int n_heads, n_kv, hd, vd, rot;
  float eps;
  const float* q_w;        // [hd] or null
  const float* k_w;
  const float* inv_f;      // [rot/2]
  const double* inv_d;
};

constexpr int WARPS = 8;

// two neighbouring channels at once
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// NC: pieces of 64 channels a head has at most
template <typename TO, int TAPS, int NC>
__global__ void __launch_bounds__(WARPS * 32)
qkv_conv_kernel(const float* __restrict__ proj, int ld, QkvConv p, const float* __restrict__ w, float* __restrict__ state,
                long long state_stride, long long tail_off, const int* __restrict__ positions,
                const int* __restrict__ seq_of_token, const int* __restrict__ seq_q_start, const int* __restrict__ slots,
                PagedView pk, PagedView pvv, TO* __restrict__ q_out, TO* __restrict__ k_pool, TO* __restrict__ v_pool,
                int T, int run, int move_tail) {
  extern __shared__ float qc_sm[];         // cos and sin of the run's positions, then a head's row per warp
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = p.rot >> 1;
  const int t0 = blockIdx.x * run, t1 = min(T, t0 + run);
  float* cs = qc_sm;
  float* buf = qc_sm + run * p.rot + warp * (NC * 64);
  pdl_launch();
  // positions, weights and tables are in place before the step's first kernel: no need to wait for them
  for (int i = threadIdx.x; i < (t1 - t0) * half; i += blockDim.x) {
    const int tt = i / half, j = i - tt * half;
    float c, s;
    rotary_cs(positions[t0 + tt], j, p.inv_f, p.inv_d, c, s);
    cs[tt * p.rot + j] = c;
    cs[tt * p.rot + half + j] = s;
  }
  const int item = blockIdx.y * WARPS + warp;
  const int nq = p.n_heads * p.hd, nk = p.n_kv * p.hd;
  const int C = nq + nk + p.n_kv * p.vd;
  const bool live = item < p.n_heads + 2 * p.n_kv;
  const bool is_q = item < p.n_heads, is_v = item >= p.n_heads + p.n_kv;
  const int head = is_q ? item : is_v ? item - p.n_heads - p.n_kv : item - p.n_heads;
  const int width = is_v ? p.vd : p.hd;
  const int col = is_q ? head * p.hd : is_v ? nq + nk + head * p.vd : nq + head * p.hd;
  const float* nw = is_v ? nullptr : is_q ? p.q_w : p.k_w;
  float2 wt[NC][TAPS], norm_w[NC];
#pragma unroll
  for (int n = 0; n < NC; n++) {
    const int c = n * 64 + 2 * lane;
    norm_w[n] = make_float2(1.f, 1.f);
    if (live && c < width) {
      if (nw) norm_w[n] = make_float2(nw[c], nw[c + 1]);
#pragma unroll
      for (int j = 0; j < TAPS; j++)
        wt[n][j] = make_float2(w[(long long)(col + c) * TAPS + j], w[(long long)(col + c + 1) * TAPS + j]);
    }
  }
  __syncthreads();
  pdl_wait();
  if (!live) return;
  float2 win[NC][TAPS];        // the last TAPS inputs of every channel, the newest last
#pragma unroll
  for (int n = 0; n < NC; n++)
#pragma unroll
    for (int j = 0; j < TAPS; j++) win[n][j] = make_float2(0.f, 0.f);
  for (int t = t0; t < t1; t++) {
    const int seq = seq_of_token[t];
    const int rel = t - seq_q_start[seq];
    float* tail = TAPS > 1 ? state + (long long)slots[seq] * state_stride + tail_off : nullptr;
    float2 y[NC];
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NC; n++) {
      const int c = n * 64 + 2 * lane;
      y[n] = make_float2(0.f, 0.f);
      if (c < width) {
        if (t == t0 || rel == 0) {
#pragma unroll
          for (int j = 0; j < TAPS - 1; j++) {
            const int back = TAPS - 1 - j;
            win[n][j + 1] = rel - back >= 0
                                ? *reinterpret_cast<const float2*>(proj + (long long)(t - back) * ld + col + c)
                                : *reinterpret_cast<const float2*>(tail + (long long)(rel - back + TAPS - 1) * C + col + c);
          }
        }
#pragma unroll
        for (int j = 0; j < TAPS - 1; j++) win[n][j] = win[n][j + 1];
        win[n][TAPS - 1] = *reinterpret_cast<const float2*>(proj + (long long)t * ld + col + c);
#pragma unroll
        for (int j = 0; j < TAPS; j++) {
          y[n].x = fmaf(wt[n][j].x, win[n][j].x, y[n].x);
          y[n].y = fmaf(wt[n][j].y, win[n][j].y, y[n].y);
        }
        ss = fmaf(y[n].x, y[n].x, fmaf(y[n].y, y[n].y, ss));
        if (TAPS > 1 && move_tail) {     // the sequence's only token: what was read, one place on
#pragma unroll
          for (int j = 0; j < TAPS - 1; j++)
            *reinterpret_cast<float2*>(tail + (long long)j * C + col + c) = win[n][j + 1];
        }
      }
    }
    const int pos = positions[t];
    if (is_v) {
      TO* dst = v_pool + paged_offset(pvv, seq, pos, head);
#pragma unroll
      for (int n = 0; n < NC; n++) {
        const int c = n * 64 + 2 * lane;
        if (c < width) store2(dst + c, y[n].x, y[n].y);
      }
      continue;
    }
    const float inv = nw ? 1.0f / sqrtf(warp_sum(ss) / (float)p.hd + p.eps) : 1.0f;
#pragma unroll
    for (int n = 0; n < NC; n++) {
      const int c = n * 64 + 2 * lane;
      if (c < width) store2(buf + c, y[n].x * inv * norm_w[n].x, y[n].y * inv * norm_w[n].y);
    }
    __syncwarp();
    TO* dst = is_q ? q_out + (long long)t * nq + col : k_pool + paged_offset(pk, seq, pos, head);
    const float* tc = cs + (t - t0) * p.rot;
#pragma unroll
    for (int n = 0; n < NC; n++) {
      const int c = n * 64 + 2 * lane;
      if (c < width) {
        float o[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int ch = c + e;
          const float own = buf[ch];
          if (ch < half) o[e] = own * tc[ch] - buf[ch + half] * tc[half + ch];
          else if (ch < p.rot) o[e] = own * tc[ch - half] + buf[ch - half] * tc[ch];
          else o[e] = own;
        }
        store2(dst + c, o[0], o[1]);
      }
    }
    __syncwarp();              // the row is free for the next token
  }
}

template <typename TO, int TAPS>
cudaError_t launch_taps(int nc, dim3 grid, size_t smem, cudaStream_t stream, const float* proj, int ld, const QkvConv& p,
                        const float* w, float* state, long long state_stride, long long tail_off, const int* positions,
                        const int* seq_of_token, const int* seq_q_start, const int* slots, const PagedView& pk,
                        const PagedView& pvv, void* q_out, void* k_pool, void* v_pool, int T, int run, int move) {
#define QC(NC)                                                                                                        \
  return launch_dep(qkv_conv_kernel<TO, TAPS, NC>, grid, dim3(WARPS * 32), smem, stream, proj, ld, p, w, state,        \
                    state_stride, tail_off, positions, seq_of_token, seq_q_start, slots, pk, pvv, (TO*)q_out,          \
                    (TO*)k_pool, (TO*)v_pool, T, run, move)
  if (nc <= 1) QC(1);
  if (nc <= 2) QC(2);
  QC(4);
#undef QC
}

}  // namespace

// Sizes that the kernel takes: even heads of at most 256 channels, one to four taps.
MF_API int mf_qkv_conv_ok(int hd, int vd, int taps, int ld, int rot) {
  return hd > 0 && vd > 0 && hd % 2 == 0 && vd % 2 == 0 && hd <= 256 && vd <= 256 && taps >= 1 && taps <= 4 && ld % 2 == 0 &&
         rot >= 0 && rot <= hd && rot % 2 == 0;
}

MF_API int mf_qkv_conv(const float* proj, int ld, int out_dtype, int T, int n_heads, int n_kv, int hd, int vd, int rot,
                       float eps, const float* w, int taps, const float* q_w, const float* k_w, const float* inv_f,
                       const double* inv_d, float* state, long long state_stride, long long tail_off,
                       const int* positions, const int* seq_of_token, const int* seq_q_start, const int* seq_q_len,
                       const int* slots, int n_seqs, const int* block_table, int bt_stride, int page_size, void* q_out,
                       void* k_pool, void* v_pool, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (!mf_qkv_conv_ok(hd, vd, taps, ld, rot) || n_heads <= 0 || n_kv < 0) return MF_ERR_BAD_ARG;
  const int C = n_heads * hd + n_kv * (hd + vd);
  if (ld < C || (rot > 0 && !inv_f && !inv_d) || (taps > 1 && !state)) return MF_ERR_BAD_ARG;
  if (((uintptr_t)proj & 7) || ((uintptr_t)state & 7) || state_stride % 2 || tail_off % 2) return MF_ERR_BAD_ARG;
  if ((((uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool) & 7)) return MF_ERR_BAD_ARG;
  if (out_dtype != MF_F32 && out_dtype != MF_BF16) return MF_ERR_BAD_DTYPE;
  mf_count(MF_K_QKV_CONV);
  const QkvConv p{n_heads, n_kv, hd, vd, rot, eps, q_w, k_w, inv_f, inv_d};
  const PagedView pk{block_table, bt_stride, page_size, n_kv, hd};
  const PagedView pvv{block_table, bt_stride, page_size, n_kv, vd};
  // one token from every sequence (the caller lays the step out so: T tokens of n_seqs sequences, none empty)
  const int single = (T == n_seqs && taps > 1) ? 1 : 0;
  const int run = T >= 1024 ? 8 : T >= 128 ? 4 : 1;      // enough blocks first, then reuse
  const int widest = n_kv > 0 && vd > hd ? vd : hd;
  const int nc = (widest + 63) / 64;
  const size_t smem = (size_t)(run * rot + WARPS * (nc <= 1 ? 64 : nc <= 2 ? 128 : 256)) * sizeof(float);
  const dim3 grid((T + run - 1) / run, (n_heads + 2 * n_kv + WARPS - 1) / WARPS);
  cudaError_t e;
#define QT(TO, TAPS)                                                                                                  \
  e = launch_taps<TO, TAPS>(nc, grid, smem, stream, proj, ld, p, w, state, state_stride, tail_off, positions,          \
                            seq_of_token, seq_q_start, slots, pk, pvv, q_out, k_pool, v_pool, T, run, single)
#define QA(TO)                                                                                                        \
  do {                                                                                                                \
    if (taps == 1) QT(TO, 1);                                                                                         \
    else if (taps == 2) QT(TO, 2);                                                                                    \
    else if (taps == 3) QT(TO, 3);                                                                                    \
    else QT(TO, 4);                                                                                                   \
  } while (0)
  if (out_dtype == MF_F32) QA(float);
  else QA(__nv_bfloat16);
#undef QA
#undef QT
  if (e != cudaSuccess || taps == 1 || single) return (int)e;
  return (int)conv_tail_launch(proj, ld, C, taps, state, state_stride, tail_off, seq_q_start, seq_q_len, slots, n_seqs,
                               stream);
}
