// A sublayer's output on its way into the residual stream through a norm of its own, and the norm of
// the stream that the next sublayer reads, in one kernel:
//
//   x_t <- x_t + N1(y_t) * w1          (y_t: the sublayer's output; none, or added without a norm)
//   out_t = N2(x_t) * w2
//
// N is a layer norm, (x - mean) / sqrt(variance + eps), the variance being the mean of the squared
// deviations, or a root-mean-square norm, x / sqrt(mean(x^2) + eps); the two are chosen apart.  The
// stream is 32-bit [T, H]; sums, deviations, norms and the add are 32-bit (the mean is taken first and
// the squares are of the deviations) and out is rounded once.  With `rows` only those rows are
// produced and the stream stays as it is.  One block per row.
#include "common.cuh"

namespace {

constexpr int NK_NONE = 0, NK_RMS = 1, NK_LAYER = 2;

// Block-wide sum over a slot of shared memory that no earlier sum of the kernel has used: one barrier.
__device__ __forceinline__ float slot_sum(float v, float* slot) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_sum(v);
  if (lane == 0) slot[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? slot[lane] : 0.f);
}

// ------------------------------------------------------------------ any sizes and dtypes
template <typename TY, typename TO>
__global__ void __launch_bounds__(256)
post_norm_kernel(float* __restrict__ resid, const TY* __restrict__ y, const float* __restrict__ w1, int kind1, float eps1,
                 const float* __restrict__ w2, int kind2, float eps2, TO* __restrict__ out, const int* __restrict__ rows,
                 int H) {
  extern __shared__ float pn_row[];      // [H]
  __shared__ float red[32];
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x;
  const long long src = rows ? rows[r] : r;
  float* x = resid + src * H;
  if (y) {
    const TY* yr = y + src * H;
    float mean = 0.f, inv = 1.0f;
    if (kind1 == NK_LAYER) {
      float s = 0.f;
      for (int i = threadIdx.x; i < H; i += blockDim.x) s += to_f32<TY>(yr[i]);
      mean = block_sum(s, red) / (float)H;
    }
    if (kind1 != NK_NONE) {
      float ss = 0.f;
      for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float d = to_f32<TY>(yr[i]) - mean;
        ss = fmaf(d, d, ss);
      }
      inv = 1.0f / sqrtf(block_sum(ss, red) / (float)H + eps1);
    }
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float n = (to_f32<TY>(yr[i]) - mean) * inv;
      const float v = x[i] + (kind1 != NK_NONE ? n * w1[i] : n);
      pn_row[i] = v;
      if (!rows) x[i] = v;
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) pn_row[i] = x[i];
  }
  // a thread reads back only what it wrote itself
  float mean = 0.f;
  if (kind2 == NK_LAYER) {
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) s += pn_row[i];
    mean = block_sum(s, red) / (float)H;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float d = pn_row[i] - mean;
    ss = fmaf(d, d, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)H + eps2);
  TO* o = out + (long long)r * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = from_f32<TO>((pn_row[i] - mean) * inv * w2[i]);
}

// ------------------------------------------------------------------ the serving case
// bfloat16 output of the sublayer and of the norm in 16-byte pieces, H a multiple of 8 and at most
// 8 * NT * NV: every value stays in registers between the sums.
template <int NT, int NV>
__global__ void __launch_bounds__(NT)
post_norm_bf16_vec_kernel(float* __restrict__ resid, const __nv_bfloat16* __restrict__ y, const float* __restrict__ w1,
                          int kind1, float eps1, const float* __restrict__ w2, int kind2, float eps2,
                          __nv_bfloat16* __restrict__ out, const int* __restrict__ rows, int H) {
  __shared__ float red[4][8];
  pdl_launch();              // the product after this one fetches its weights meanwhile
  pdl_wait();
  const int r = blockIdx.x;
  const long long src = rows ? rows[r] : r;
  float* x = resid + src * H;
  const float inv_h = 1.0f / (float)H;
  float v[NV][8];
#pragma unroll
  for (int j = 0; j < NV; j++) {
    const int i = (j * NT + threadIdx.x) * 8;
#pragma unroll
    for (int e = 0; e < 8; e++) v[j][e] = 0.f;
    if (i < H) {
      const float4 a = *reinterpret_cast<const float4*>(x + i), b = *reinterpret_cast<const float4*>(x + i + 4);
      v[j][0] = a.x; v[j][1] = a.y; v[j][2] = a.z; v[j][3] = a.w;
      v[j][4] = b.x; v[j][5] = b.y; v[j][6] = b.z; v[j][7] = b.w;
    }
  }
  if (y) {
    const __nv_bfloat16* yr = y + src * H;
    float u[NV][8];
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < NV; j++) {
      const int i = (j * NT + threadIdx.x) * 8;
#pragma unroll
      for (int e = 0; e < 8; e++) u[j][e] = 0.f;
      if (i < H) {
        const uint4 dv = *reinterpret_cast<const uint4*>(yr + i);
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&dv);
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const float2 f = __bfloat1622float2(p[e]);
          u[j][2 * e] = f.x;
          u[j][2 * e + 1] = f.y;
          s += f.x + f.y;
        }
      }
    }
    const float mean = kind1 == NK_LAYER ? slot_sum(s, red[0]) * inv_h : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; j++) {
      if ((j * NT + threadIdx.x) * 8 < H) {
#pragma unroll
        for (int e = 0; e < 8; e++) {
          u[j][e] -= mean;
          ss = fmaf(u[j][e], u[j][e], ss);
        }
      }
    }
    const float inv = kind1 == NK_NONE ? 1.0f : 1.0f / sqrtf(slot_sum(ss, red[1]) * inv_h + eps1);
#pragma unroll
    for (int j = 0; j < NV; j++) {
      const int i = (j * NT + threadIdx.x) * 8;
      if (i < H) {
#pragma unroll
        for (int hf = 0; hf < 2; hf++) {
          const float4 w = kind1 == NK_NONE ? make_float4(1.f, 1.f, 1.f, 1.f)
                                            : *reinterpret_cast<const float4*>(w1 + i + 4 * hf);
          v[j][4 * hf + 0] += u[j][4 * hf + 0] * inv * w.x;
          v[j][4 * hf + 1] += u[j][4 * hf + 1] * inv * w.y;
          v[j][4 * hf + 2] += u[j][4 * hf + 2] * inv * w.z;
          v[j][4 * hf + 3] += u[j][4 * hf + 3] * inv * w.w;
          if (!rows)
            *reinterpret_cast<float4*>(x + i + 4 * hf) =
                make_float4(v[j][4 * hf], v[j][4 * hf + 1], v[j][4 * hf + 2], v[j][4 * hf + 3]);
        }
      }
    }
  }
  float mean = 0.f;
  if (kind2 == NK_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < NV; j++)
#pragma unroll
      for (int e = 0; e < 8; e++) s += v[j][e];
    mean = slot_sum(s, red[2]) * inv_h;
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; j++) {
    if ((j * NT + threadIdx.x) * 8 < H) {
#pragma unroll
      for (int e = 0; e < 8; e++) {
        v[j][e] -= mean;
        ss = fmaf(v[j][e], v[j][e], ss);
      }
    }
  }
  const float inv = 1.0f / sqrtf(slot_sum(ss, red[3]) * inv_h + eps2);
  __nv_bfloat16* o = out + (long long)r * H;
#pragma unroll
  for (int j = 0; j < NV; j++) {
    const int i = (j * NT + threadIdx.x) * 8;
    if (i < H) {
      const float4 wa = *reinterpret_cast<const float4*>(w2 + i), wb = *reinterpret_cast<const float4*>(w2 + i + 4);
      uint4 pk;
      __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&pk);
      p[0] = __floats2bfloat162_rn(v[j][0] * inv * wa.x, v[j][1] * inv * wa.y);
      p[1] = __floats2bfloat162_rn(v[j][2] * inv * wa.z, v[j][3] * inv * wa.w);
      p[2] = __floats2bfloat162_rn(v[j][4] * inv * wb.x, v[j][5] * inv * wb.y);
      p[3] = __floats2bfloat162_rn(v[j][6] * inv * wb.z, v[j][7] * inv * wb.w);
      *reinterpret_cast<uint4*>(o + i) = pk;
    }
  }
}

}  // namespace

// kind1 (0: y is added as it is, 1: RMS norm, 2: layer norm) with w1 and eps1 for y (may be null: nothing is
// added); kind2 (1 or 2) with w2 and eps2 for the norm of the stream.
MF_API int mf_post_norm(float* resid, const void* y, int y_dtype, const float* w1, int kind1, float eps1,
                        const float* w2, int kind2, float eps2, void* out, int out_dtype, const int* rows, int n_rows,
                        int H, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (H <= 0 || kind1 < NK_NONE || kind1 > NK_LAYER || kind2 < NK_RMS || kind2 > NK_LAYER || !w2) return MF_ERR_BAD_ARG;
  if (y && kind1 != NK_NONE && !w1) return MF_ERR_BAD_ARG;
  mf_count(MF_K_POST_NORM);
  if (out_dtype == MF_BF16 && (!y || y_dtype == MF_BF16) && H % 8 == 0 && H <= 8 * 256 * 4 &&
      (((uintptr_t)resid | (uintptr_t)y | (uintptr_t)w1 | (uintptr_t)w2 | (uintptr_t)out) & 15) == 0) {
#define PV(NT, NV)                                                                                                   \
  return (int)launch_dep(post_norm_bf16_vec_kernel<NT, NV>, dim3(n_rows), dim3(NT), 0, stream, resid,                 \
                         (const __nv_bfloat16*)y, w1, kind1, eps1, w2, kind2, eps2, (__nv_bfloat16*)out, rows, H)
    // many rows: few threads with many values each, as the four sums are what a row costs beside its bytes; few
    // rows: many threads, as nothing else hides how long a thread takes
    if (H <= 1024) PV(128, 1);
    if (H <= 2048 && n_rows >= 256) PV(128, 2);
    if (H <= 2048) PV(256, 1);
    if (H <= 4096) PV(256, 2);
    PV(256, 4);
#undef PV
  }
  const size_t smem = (size_t)H * sizeof(float);
  if (smem > 200 * 1024) return MF_ERR_BAD_ARG;
#define PG(TY, TO)                                                                                                   \
  do {                                                                                                               \
    if (smem > 40 * 1024) {                                                                                          \
      cudaError_t e = cudaFuncSetAttribute(post_norm_kernel<TY, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                           (int)smem);                                                               \
      if (e != cudaSuccess) return (int)e;                                                                           \
    }                                                                                                                \
    return (int)launch_dep(post_norm_kernel<TY, TO>, dim3(n_rows), dim3(256), smem, stream, resid, (const TY*)y, w1, \
                           kind1, eps1, w2, kind2, eps2, (TO*)out, rows, H);                                         \
  } while (0)
  if (y_dtype == MF_F32 && out_dtype == MF_F32) PG(float, float);
  if (y_dtype == MF_BF16 && out_dtype == MF_BF16) PG(__nv_bfloat16, __nv_bfloat16);
  if (y_dtype == MF_F32 && out_dtype == MF_BF16) PG(float, __nv_bfloat16);
  if (y_dtype == MF_BF16 && out_dtype == MF_F32) PG(__nv_bfloat16, float);
#undef PG
  return MF_ERR_BAD_DTYPE;
}
