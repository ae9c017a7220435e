// A short causal convolution over time per channel, with a bias and an activation, on a range of
// columns of a step's projections:
//
//   y_t = act( b + sum_j w[:, j] x_(t - taps + 1 + j) )       (zeros before the sequence's start)
//
// x is 32-bit (rows `ld` floats apart); y is written in 32-bit and, where a product follows that
// reads it, once more in the compute dtype.  The last taps-1 inputs of a sequence are kept in its
// state slot ([taps-1, C] at `tail_off`), so a step goes on from where the step before ended
// however the tokens were cut; a second kernel moves them on after the first has read them.  Where
// every sequence of the step brings one token a token's threads are the only readers of the slot's
// rows and move them on themselves: one launch.
#include "conv_tail.cuh"

__device__ __forceinline__ float ca_act(float v, int silu) { return silu ? v / (1.0f + expf(-v)) : v; }

// any number of taps and channels: a thread per (token, channel)
template <typename T2>
__global__ void __launch_bounds__(256)
conv_act_kernel(const float* __restrict__ x, int ld, int C, const float* __restrict__ w, const float* __restrict__ bias,
                int taps, int silu, float* __restrict__ state, long long state_stride, long long tail_off,
                const int* __restrict__ seq_of_token, const int* __restrict__ seq_q_start, const int* __restrict__ slots,
                float* __restrict__ out, T2* __restrict__ out2, int move_tail) {
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int seq = seq_of_token[t];
  const int rel = t - seq_q_start[seq];
  float* tail = state + (long long)slots[seq] * state_stride + tail_off;
  float a = bias ? bias[c] : 0.f;
  for (int j = 0; j < taps; j++) {
    const int back = taps - 1 - j;
    const float v = rel - back >= 0 ? x[(long long)(t - back) * ld + c] : tail[(long long)(rel - back + taps - 1) * C + c];
    a = fmaf(w[(long long)c * taps + j], v, a);
  }
  a = ca_act(a, silu);
  out[(long long)t * C + c] = a;
  if (out2) out2[(long long)t * C + c] = from_f32<T2>(a);
  if (move_tail)          // the sequence's only token: every row moves up one place, the token's row comes last
    for (int j = 0; j < taps - 1; j++)
      tail[(long long)j * C + c] = j < taps - 2 ? tail[(long long)(j + 1) * C + c] : x[(long long)t * ld + c];
}

// four channels a thread over a run of consecutive tokens: every input is read once (16 bytes at a
// time) and handed on in registers
template <typename T2, int TAPS>
__global__ void __launch_bounds__(128)
conv_act_vec_kernel(const float* __restrict__ x, int ld, int C, const float* __restrict__ w,
                    const float* __restrict__ bias, int silu, float* __restrict__ state, long long state_stride,
                    long long tail_off, const int* __restrict__ seq_of_token, const int* __restrict__ seq_q_start,
                    const int* __restrict__ slots, float* __restrict__ out, T2* __restrict__ out2, int T, int run,
                    int move_tail) {
  pdl_launch();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  float wt[TAPS][4], b[4];
  if (c < C) {             // the weights never change: fetched before the wait
#pragma unroll
    for (int e = 0; e < 4; e++) {
      b[e] = bias ? bias[c + e] : 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; j++) wt[j][e] = w[(long long)(c + e) * TAPS + j];
    }
  }
  pdl_wait();
  if (c >= C) return;
  const int t0 = blockIdx.x * run, t1 = min(T, t0 + run);
  float4 win[TAPS];        // the last TAPS inputs, the newest last
#pragma unroll
  for (int j = 0; j < TAPS; j++) win[j] = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int t = t0; t < t1; t++) {
    const int seq = seq_of_token[t];
    const int rel = t - seq_q_start[seq];
    float* tail = state + (long long)slots[seq] * state_stride + tail_off;
    if (t == t0 || rel == 0) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) {
        const int back = TAPS - 1 - j;
        win[j + 1] = rel - back >= 0 ? *reinterpret_cast<const float4*>(x + (long long)(t - back) * ld + c)
                                     : *reinterpret_cast<const float4*>(tail + (long long)(rel - back + TAPS - 1) * C + c);
      }
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; j++) win[j] = win[j + 1];
    win[TAPS - 1] = *reinterpret_cast<const float4*>(x + (long long)t * ld + c);
    float a[4] = {b[0], b[1], b[2], b[3]};
#pragma unroll
    for (int j = 0; j < TAPS; j++) {
      a[0] = fmaf(wt[j][0], win[j].x, a[0]);
      a[1] = fmaf(wt[j][1], win[j].y, a[1]);
      a[2] = fmaf(wt[j][2], win[j].z, a[2]);
      a[3] = fmaf(wt[j][3], win[j].w, a[3]);
    }
#pragma unroll
    for (int e = 0; e < 4; e++) a[e] = ca_act(a[e], silu);
    *reinterpret_cast<float4*>(out + (long long)t * C + c) = make_float4(a[0], a[1], a[2], a[3]);
    if (out2) {
      T2* o2 = out2 + (long long)t * C + c;
      if constexpr (sizeof(T2) == 2) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(a[0], a[1]), p1 = __floats2bfloat162_rn(a[2], a[3]);
        uint2 pk;
        pk.x = *reinterpret_cast<const uint32_t*>(&p0);
        pk.y = *reinterpret_cast<const uint32_t*>(&p1);
        *reinterpret_cast<uint2*>(o2) = pk;
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++) o2[e] = from_f32<T2>(a[e]);
      }
    }
    if (move_tail) {       // the sequence's only token: what was read, one place on
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) *reinterpret_cast<float4*>(tail + (long long)j * C + c) = win[j + 1];
    }
  }
}

// After the step the slot keeps the last taps-1 inputs of every channel.
__global__ void __launch_bounds__(256)
conv_act_tail_kernel(const float* __restrict__ x, int ld, int C, int taps, float* __restrict__ state,
                     long long state_stride, long long tail_off, const int* __restrict__ seq_q_start,
                     const int* __restrict__ seq_q_len, const int* __restrict__ slots) {
  pdl_launch();
  pdl_wait();
  const int seq = blockIdx.x;
  const int start = seq_q_start[seq], n = seq_q_len[seq];
  float* tail = state + (long long)slots[seq] * state_stride + tail_off;
  constexpr int AHEAD = 4;        // rows fetched before the first of them is written
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
    for (int j0 = 0; j0 < taps - 1; j0 += AHEAD) {          // ascending: a read is never behind a write
      float v[AHEAD];
#pragma unroll
      for (int e = 0; e < AHEAD; e++) {
        const int j = j0 + e, src = n - (taps - 1) + j;
        if (j < taps - 1) v[e] = src >= 0 ? x[(long long)(start + src) * ld + c] : tail[(long long)(j + n) * C + c];
      }
#pragma unroll
      for (int e = 0; e < AHEAD; e++)
        if (j0 + e < taps - 1) tail[(long long)(j0 + e) * C + c] = v[e];
    }
}

cudaError_t conv_tail_launch(const float* x, int ld, int C, int taps, float* state, long long state_stride,
                             long long tail_off, const int* seq_q_start, const int* seq_q_len, const int* slots, int n_seqs,
                             cudaStream_t stream) {
  return launch_dep(conv_act_tail_kernel, dim3(n_seqs, (C + 255) / 256), dim3(256), 0, stream, x, ld, C, taps, state,
                    state_stride, tail_off, seq_q_start, seq_q_len, slots);
}

MF_API int mf_conv_act(const float* x, int ld, int T, int C, const float* w, const float* bias, int taps, int silu,
                       float* state, long long state_stride, long long tail_off, const int* seq_of_token,
                       const int* seq_q_start, const int* seq_q_len, const int* slots, int n_seqs, float* out,
                       void* out2, int out2_dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (taps < 1 || C <= 0 || ld < C || (C + 255) / 256 > 65535) return MF_ERR_BAD_ARG;
  if (out2_dtype != MF_F32 && out2_dtype != MF_BF16) return MF_ERR_BAD_DTYPE;
  mf_count(MF_K_CONV_ACT);
  // one token from every sequence (the caller lays the step out so: T tokens of n_seqs sequences, none empty)
  const int single = (T == n_seqs && taps > 1) ? 1 : 0;
  const bool vec = C % 4 == 0 && ld % 4 == 0 && tail_off % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)x & 15) == 0 &&
                   ((uintptr_t)state & 15) == 0 && ((uintptr_t)out & 15) == 0 && ((uintptr_t)out2 & 15) == 0 &&
                   taps >= 1 && taps <= 4;
  cudaError_t e;
  // tokens a thread runs over: enough blocks first, then reuse
  const int run = T >= 1024 ? 8 : T >= 128 ? 4 : 1;
  const dim3 vgrid((T + run - 1) / run, (C / 4 + 127) / 128);
#define CA_VEC(T2, TAPS)                                                                                            \
  e = launch_dep(conv_act_vec_kernel<T2, TAPS>, vgrid, dim3(128), 0, stream, x, ld, C, w, bias, silu, state,         \
                 state_stride, tail_off, seq_of_token, seq_q_start, slots, out, (T2*)out2, T, run, single)
#define CA_ANY(T2)                                                                                                  \
  do {                                                                                                              \
    if (vec && taps == 1) CA_VEC(T2, 1);                                                                            \
    else if (vec && taps == 2) CA_VEC(T2, 2);                                                                       \
    else if (vec && taps == 3) CA_VEC(T2, 3);                                                                       \
    else if (vec && taps == 4) CA_VEC(T2, 4);                                                                       \
    else                                                                                                            \
      e = launch_dep(conv_act_kernel<T2>, dim3(T, (C + 255) / 256), dim3(256), 0, stream, x, ld, C, w, bias, taps,   \
                     silu, state, state_stride, tail_off, seq_of_token, seq_q_start, slots, out, (T2*)out2, single); \
  } while (0)
  if (out2_dtype == MF_F32) CA_ANY(float);
  else CA_ANY(__nv_bfloat16);
#undef CA_ANY
#undef CA_VEC
  if (e != cudaSuccess || taps == 1 || single) return (int)e;
  return (int)conv_tail_launch(x, ld, C, taps, state, state_stride, tail_off, seq_q_start, seq_q_len, slots, n_seqs, stream);
}
