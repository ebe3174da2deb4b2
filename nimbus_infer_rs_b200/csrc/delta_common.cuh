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

inline int launch_delta_finish(const float* o_raw, const float* gate, int gate_stride, int gate_col,
                               const float* norm_w, int norm_pitch, float eps, const int* row_slot,
                               void* out, int out_dtype, int n_heads, int d, int n_rows,
                               cudaStream_t stream) {
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
