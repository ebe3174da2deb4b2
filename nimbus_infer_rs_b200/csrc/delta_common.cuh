// What the delta-rule recurrences share: the last row pass over a head's outputs.
#pragma once

#include "common.cuh"

namespace {

// out[r, h, :] = o[r, h, :] / sqrt(mean(o[r, h, :]^2) + eps) * norm_w[h * norm_pitch + :] *
// sigmoid(gate[r][gate_col + h*d + :]).  A CTA per row, its warps over the heads of d numbers;
// norm_pitch = d: a weight per head, 0: one for all; padding rows give zeros.
template <typename TOut>
__global__ void __launch_bounds__(128)
delta_finish_kernel(const float* o_raw, const float* gate, int gate_stride, int gate_col,
                    const float* __restrict__ norm_w, int norm_pitch, float eps, const int* row_slot,
                    TOut* out, int n_heads, int d) {
  nb_grid_dependency_wait();
  nb_launch_dependents();
  const int r = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int hd = n_heads * d;
  const bool live = row_slot[r] >= 0;
  for (int h = warp; h < n_heads; h += 4) {
    TOut* dst = out + (size_t)r * hd + h * d;
    if (!live) {
      for (int j = lane; j < d; j += 32) dst[j] = nb_from_f32<TOut>(0.0f);
      continue;
    }
    const float* o = o_raw + (size_t)r * hd + h * d;
    const float* g = gate + (size_t)r * gate_stride + gate_col + h * d;
    float ss = 0.0f;
    for (int j = lane; j < d; j += 32) ss = fmaf(o[j], o[j], ss);
    ss = nb_warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)d + eps);
    for (int j = lane; j < d; j += 32)
      dst[j] = nb_from_f32<TOut>(o[j] * inv * norm_w[h * norm_pitch + j] * nb_sigmoid(g[j]));
  }
}

// The same with a warp per (row, head) and the head in registers, 16 bytes a load: heads of d numbers,
// d a multiple of 4 and at most 128 * NQ.
template <typename TOut, int NQ>
__global__ void __launch_bounds__(256)
delta_finish_quads_kernel(const float* o_raw, const float* gate, int gate_stride, int gate_col,
                          const float* __restrict__ norm_w, int norm_pitch, float eps,
                          const int* row_slot, TOut* out, int n_heads, int d, int n_pairs) {
  nb_grid_dependency_wait();
  nb_launch_dependents();
  const int pair = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (pair >= n_pairs) return;
  const int r = pair / n_heads, h = pair - r * n_heads;
  const bool live = row_slot[r] >= 0;
  const float* o = o_raw + (size_t)pair * d;
  const float* g = gate + (size_t)r * gate_stride + gate_col + (size_t)h * d;
  TOut* dst = out + (size_t)pair * d;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 x[NQ], z[NQ];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = (i * 32 + lane) * 4;
    const bool in = live && c < d;
    x[i] = in ? *reinterpret_cast<const float4*>(o + c) : zero;
    z[i] = in ? *reinterpret_cast<const float4*>(g + c) : zero;
    ss += (x[i].x * x[i].x + x[i].y * x[i].y) + (x[i].z * x[i].z + x[i].w * x[i].w);
  }
  const float inv = 1.0f / sqrtf(nb_warp_sum(ss) / (float)d + eps);
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = (i * 32 + lane) * 4;
    if (c >= d) continue;
    const float4 w = *reinterpret_cast<const float4*>(norm_w + h * norm_pitch + c);
    const float y[4] = {x[i].x * inv * w.x * nb_sigmoid(z[i].x), x[i].y * inv * w.y * nb_sigmoid(z[i].y),
                        x[i].z * inv * w.z * nb_sigmoid(z[i].z), x[i].w * inv * w.w * nb_sigmoid(z[i].w)};
    if constexpr (sizeof(TOut) == 4) {
      *reinterpret_cast<float4*>(dst + c) = make_float4(y[0], y[1], y[2], y[3]);
    } else {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[1]), hi = __floats2bfloat162_rn(y[2], y[3]);
      uint2 u;
      u.x = *reinterpret_cast<const uint32_t*>(&lo);
      u.y = *reinterpret_cast<const uint32_t*>(&hi);
      *reinterpret_cast<uint2*>(dst + c) = u;
    }
  }
}

inline int launch_delta_finish(const float* o_raw, const float* gate, int gate_stride, int gate_col,
                               const float* norm_w, int norm_pitch, float eps, const int* row_slot,
                               void* out, int out_dtype, int n_heads, int d, int n_rows,
                               cudaStream_t stream) {
  const int n_pairs = n_rows * n_heads;
  if (d % 4 == 0 && d <= 256 && gate_stride % 4 == 0 && gate_col % 4 == 0 &&
      ((uintptr_t)o_raw | (uintptr_t)gate | (uintptr_t)norm_w | (uintptr_t)out) % 16 == 0) {
#define NB_DF(T, NQ)                                                                              \
  NB_CUDA(nb_launch(delta_finish_quads_kernel<T, NQ>, dim3((n_pairs + 7) / 8), dim3(256), 0,      \
                    stream, o_raw, gate, gate_stride, gate_col, norm_w, norm_pitch, eps, row_slot, \
                    (T*)out, n_heads, d, n_pairs))
    if (out_dtype == NB_F32) {
      if (d <= 128) NB_DF(float, 1);
      else NB_DF(float, 2);
    } else {
      if (d <= 128) NB_DF(__nv_bfloat16, 1);
      else NB_DF(__nv_bfloat16, 2);
    }
#undef NB_DF
    NB_CHECK_LAUNCH("delta_finish");
    return 0;
  }
  if (out_dtype == NB_F32)
    NB_CUDA(nb_launch(delta_finish_kernel<float>, dim3(n_rows), dim3(128), 0, stream, o_raw, gate,
                      gate_stride, gate_col, norm_w, norm_pitch, eps, row_slot, (float*)out, n_heads, d));
  else
    NB_CUDA(nb_launch(delta_finish_kernel<__nv_bfloat16>, dim3(n_rows), dim3(128), 0, stream, o_raw,
                      gate, gate_stride, gate_col, norm_w, norm_pitch, eps, row_slot,
                      (__nv_bfloat16*)out, n_heads, d));
  NB_CHECK_LAUNCH("delta_finish");
  return 0;
}

}  // namespace
