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
// A warp owns a head over a run of R consecutive tokens; a lane holds two neighbouring channels of every
// 64.  The run's inputs are all fetched first (each once, the taps-1 before the run again), the taps are
// applied in registers, and the places of the run's tokens in the pages are worked out by one lane each;
// the cosines and sines of the run's positions are made once for all heads of the block.  Everything is
// 32-bit (angles in double where a float64 table is given) and is rounded once, on its way into q_out
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

constexpr int MAXT = 4;      // taps a lane holds; fewer are padded with zeros in front

// R: tokens of a run; NC: pieces of 64 channels a head has at most
template <typename TO, int R, int NC>
__global__ void __launch_bounds__(WARPS * 32, 2)
qkv_conv_kernel(const float* __restrict__ proj, int ld, QkvConv p, const float* __restrict__ w, int taps,
                float* __restrict__ state, long long state_stride, long long tail_off, const int* __restrict__ positions,
                const int* __restrict__ seq_of_token, const int* __restrict__ seq_q_start, const int* __restrict__ slots,
                PagedView pk, PagedView pvv, TO* __restrict__ q_out, TO* __restrict__ k_pool, TO* __restrict__ v_pool,
                int T, int move_tail) {
  extern __shared__ float qc_sm[];         // cos and sin of the run's positions, then R rows of a head per warp
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = p.rot >> 1;
  const int t0 = blockIdx.x * R, n_run = min(R, T - t0);
  float* cs = qc_sm;
  float* buf = qc_sm + R * p.rot + warp * (R * NC * 64);
  pdl_launch();
  // positions, weights and tables are in place before the step's first kernel: no need to wait for them
  for (int i = threadIdx.x; i < n_run * half; i += blockDim.x) {
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
  f32x2 wt[NC][MAXT], norm_w[NC];
#pragma unroll
  for (int n = 0; n < NC; n++) {
    const int c = n * 64 + 2 * lane;
    norm_w[n] = pack2(1.f, 1.f);
    const bool in = live && c < width;
    if (in && nw) norm_w[n] = pack2(nw[c], nw[c + 1]);
#pragma unroll
    for (int j = 0; j < MAXT; j++) {
      const int tap = j - (MAXT - taps);
      wt[n][j] = in && tap >= 0 ? *reinterpret_cast<const f32x2*>(w + (long long)tap * C + col + c) : 0ull;
    }
  }
  // lane i looks up token i of the run: its distance from the first token its sequence brings, its slot and
  // where its row goes
  int my_rel = 0, my_slot = 0;
  long long my_dst = 0;
  if (live && lane < n_run) {
    const int t = t0 + lane, seq = seq_of_token[t];
    my_rel = t - seq_q_start[seq];
    my_slot = slots[seq];
    my_dst = is_q ? (long long)t * nq + col : paged_offset(is_v ? pvv : pk, seq, positions[t], head);
  }
  __syncthreads();
  pdl_wait();
  if (!live) return;
  // u[i + MAXT - 1] is token i of the run; what stands before it is used by the tokens of its own sequence only
  f32x2 u[R + MAXT - 1][NC];
#pragma unroll
  for (int i = 0; i < R + MAXT - 1; i++) {
    const int t = t0 + i - (MAXT - 1);
    const bool row = t >= 0 && i - (MAXT - 1) < n_run && i >= MAXT - taps;
#pragma unroll
    for (int n = 0; n < NC; n++) {
      const int c = n * 64 + 2 * lane;
      u[i][n] = row && c < width ? *reinterpret_cast<const f32x2*>(proj + (long long)t * ld + col + c) : 0ull;
    }
  }
#pragma unroll
  for (int i = 0; i < R; i++) {
    const int rel = __shfl_sync(0xffffffffu, my_rel, i);
    f32x2 y[NC];
    if (rel >= taps - 1) {           // every input is among the rows of this step
#pragma unroll
      for (int n = 0; n < NC; n++) {
        y[n] = 0ull;
#pragma unroll
        for (int j = 0; j < MAXT; j++) {
          if (j < MAXT - taps) continue;          // a padded tap: another sequence's row may stand there
          y[n] = fma2(wt[n][j], u[i + j][n], y[n]);
        }
      }
    } else {                         // the first tokens of a portion: the slot has what came before
      float* tail = state + (long long)__shfl_sync(0xffffffffu, my_slot, i) * state_stride + tail_off + col;
#pragma unroll
      for (int n = 0; n < NC; n++) {
        const int c = n * 64 + 2 * lane;
        y[n] = 0ull;
        f32x2 seen[MAXT];
#pragma unroll
        for (int j = 0; j < MAXT; j++) {
          const int back = MAXT - 1 - j;
          seen[j] = u[i + j][n];
          if (rel < back)            // zeros in front of the taps, else the slot's row
            seen[j] = back < taps && c < width && i < n_run
                          ? *reinterpret_cast<const f32x2*>(tail + (long long)(rel - back + taps - 1) * C + c)
                          : 0ull;
          if (j >= MAXT - taps) y[n] = fma2(wt[n][j], seen[j], y[n]);
        }
        if (move_tail && c < width && i < n_run) {     // the sequence's only token: what was read, one place on
#pragma unroll
          for (int j = 1; j < MAXT; j++) {
            const int slot_row = j - (MAXT - taps) - 1;
            if (slot_row >= 0) *reinterpret_cast<f32x2*>(tail + (long long)slot_row * C + c) = seen[j];
          }
        }
      }
    }
#pragma unroll
    for (int n = 0; n < NC; n++) u[i][n] = y[n];       // no later token reads this input
  }
  if (is_v) {
#pragma unroll
    for (int i = 0; i < R; i++) {
      TO* dst = v_pool + __shfl_sync(0xffffffffu, my_dst, i);
#pragma unroll
      for (int n = 0; n < NC; n++) {
        const int c = n * 64 + 2 * lane;
        const float2 v = unpack2(u[i][n]);
        if (i < n_run && c < width) store2(dst + c, v.x, v.y);
      }
    }
    return;
  }
  // lane i gets token i's sum of squares, so that the root and the division are done once
  float mine = 1.0f;
  if (nw) {
#pragma unroll
    for (int i = 0; i < R; i++) {
      f32x2 sq = 0ull;
#pragma unroll
      for (int n = 0; n < NC; n++) sq = fma2(u[i][n], u[i][n], sq);
      const float2 h = unpack2(sq);
      const float total = warp_sum(h.x + h.y);
      if (lane == i) mine = total;
    }
    mine = 1.0f / sqrtf(mine / (float)p.hd + p.eps);
  }
#pragma unroll
  for (int i = 0; i < R; i++) {
    const float inv = __shfl_sync(0xffffffffu, mine, i);
    const f32x2 inv2 = pack2(inv, inv);
#pragma unroll
    for (int n = 0; n < NC; n++) {
      u[i][n] = mul2(mul2(u[i][n], inv2), norm_w[n]);
      if (n * 64 < p.rot) *reinterpret_cast<f32x2*>(buf + i * (NC * 64) + n * 64 + 2 * lane) = u[i][n];
    }
  }
  __syncwarp();
  const bool even = (half & 1) == 0;           // both channels of a lane then stand on one side of a pair
#pragma unroll
  for (int i = 0; i < R; i++) {
    TO* dst = (is_q ? q_out : k_pool) + __shfl_sync(0xffffffffu, my_dst, i);
    const float* row = buf + i * (NC * 64);
    const float* tc = cs + i * p.rot;
#pragma unroll
    for (int n = 0; n < NC; n++) {
      const int c = n * 64 + 2 * lane;
      if (i >= n_run || c >= width) continue;
      f32x2 o = u[i][n];
      if (even) {
        if (c < p.rot) {
          const bool first = c < half;
          const int j = first ? c : c - half;
          f32x2 sn = *reinterpret_cast<const f32x2*>(tc + half + j);
          if (first) sn = mul2(sn, pack2(-1.f, -1.f));
          o = fma2(o, *reinterpret_cast<const f32x2*>(tc + j),
                   mul2(*reinterpret_cast<const f32x2*>(row + (first ? c + half : j)), sn));
        }
        const float2 v = unpack2(o);
        store2(dst + c, v.x, v.y);
      } else {
        const float2 own = unpack2(o);
        float v[2] = {own.x, own.y};
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int ch = c + e;
          if (ch < half) v[e] = v[e] * tc[ch] - row[ch + half] * tc[half + ch];
          else if (ch < p.rot) v[e] = v[e] * tc[ch - half] + row[ch - half] * tc[ch];
        }
        store2(dst + c, v[0], v[1]);
      }
    }
  }
}

}  // namespace

// Sizes that the kernel takes: even heads of at most 256 channels, one to four taps.
MF_API int mf_qkv_conv_ok(int hd, int vd, int taps, int ld, int rot) {
  return hd > 0 && vd > 0 && hd % 2 == 0 && vd % 2 == 0 && hd <= 256 && vd <= 256 && taps >= 1 && taps <= 4 && ld % 2 == 0 &&
         rot >= 0 && rot <= hd && rot % 2 == 0;
}

// w: [taps, channels] (a row per tap)
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
  const int widest = n_kv > 0 && vd > hd ? vd : hd;
  const int nc = widest <= 64 ? 1 : widest <= 128 ? 2 : 4;
  const int run = T < 128 ? 1 : nc == 4 ? 4 : 8;      // enough blocks first, then reuse
  const size_t smem = (size_t)(run * rot + WARPS * run * nc * 64) * sizeof(float);
  const dim3 grid((T + run - 1) / run, (n_heads + 2 * n_kv + WARPS - 1) / WARPS);
  cudaError_t e;
#define QC(TO, R, NC)                                                                                                 \
  e = launch_dep(qkv_conv_kernel<TO, R, NC>, grid, dim3(WARPS * 32), smem, stream, proj, ld, p, w, taps, state,        \
                 state_stride, tail_off, positions, seq_of_token, seq_q_start, slots, pk, pvv, (TO*)q_out,             \
                 (TO*)k_pool, (TO*)v_pool, T, single)
#define QA(TO)                                                                                                        \
  do {                                                                                                                \
    if (nc == 1 && run == 1) QC(TO, 1, 1);                                                                            \
    else if (nc == 1) QC(TO, 8, 1);                                                                                   \
    else if (nc == 2 && run == 1) QC(TO, 1, 2);                                                                       \
    else if (nc == 2) QC(TO, 8, 2);                                                                                   \
    else if (run == 1) QC(TO, 1, 4);                                                                                  \
    else QC(TO, 4, 4);                                                                                                \
  } while (0)
  if (out_dtype == MF_F32) QA(float);
  else QA(__nv_bfloat16);
#undef QA
#undef QC
  if (e != cudaSuccess || taps == 1 || single) return (int)e;
  return (int)conv_tail_launch(proj, ld, C, taps, state, state_stride, tail_off, seq_q_start, seq_q_len, slots, n_seqs,
                               stream);
}
