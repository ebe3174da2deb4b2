// Several residual streams side by side (hyper-connections), fp32, row by row:
//
//   u_r   = sum_s in[s] x_r[s]                              what a sublayer reads (then normed)
//   x_r[t] <- sum_s mix[s][t] x_r[s] + gain[t] * ls * y_r    its result y written back (the right
//                                                           side holds the streams as they were)
//
// One kernel does the write-back of a sublayer and, in the same pass over the row, what the next
// reader of the streams wants: the RMS-normed sum u of the next sublayer (statistics in fp32 over
// the unrounded u), or the plain sum of the streams where the layers end.  With no result to
// write back it is the read alone.  Before the first write-back all streams equal the
// embedding's output, so they are read from its single row (`in_stream` = 0) and first
// materialised by that write-back.
//
// A CTA per row; a thread holds whole columns (all streams of 1 or 4 neighbouring columns) and
// keeps its part of u in registers between the sum and the norm.
#include "common.cuh"

namespace {

typedef __nv_bfloat16 bf16;
constexpr int MAX_S = 8;      // streams
constexpr int COLS = 8;       // column groups a thread holds

template <int V>
struct Group;
template <>
struct Group<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
};
template <>
struct Group<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  }
  __device__ __forceinline__ void store(float* p) const {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};

__device__ __forceinline__ void store_act(float* p, const float (&v)[1]) { p[0] = v[0]; }
__device__ __forceinline__ void store_act(bf16* p, const float (&v)[1]) { p[0] = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void store_act(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store_act(bf16* p, const float (&v)[4]) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&lo);
  u.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}

// x_in: row r at x_in + r * in_row, stream s at + s * in_stream.  y == nullptr: read alone.
// xs == nullptr (with y): the streams are not written (only their sum is wanted).
template <typename TOut, int S, int V>
__global__ void streams_kernel(const float* x_in, int in_row, int in_stream, int n_streams, float* xs,
                               const float* y, const float* __restrict__ scale_w,
                               const float* __restrict__ mix_w, const float* __restrict__ gain_w,
                               float* sum, const float* __restrict__ next_coef,
                               const float* __restrict__ next_gamma, float next_eps, TOut* out_next,
                               int d) {
  __shared__ float c_mix[S][S], c_gain[S], c_in[S], red[32];
  const int tid = threadIdx.x;
  // the coefficients are constants of the model: fetched before the wait
  for (int i = tid; i < S * S; i += blockDim.x) {
    const int s = i / S, t = i - s * S;
    c_mix[s][t] = (y != nullptr && s < n_streams && t < n_streams) ? mix_w[s * n_streams + t] : 0.0f;
  }
  if (tid < S) {
    c_gain[tid] = (y != nullptr && tid < n_streams) ? gain_w[tid] : 0.0f;
    c_in[tid] = (out_next != nullptr && tid < n_streams) ? next_coef[tid] : 0.0f;
  }
  nb_grid_dependency_wait();
  nb_launch_dependents();
  __syncthreads();
  const int r = blockIdx.x;
  const float* xr = x_in + (size_t)r * in_row;
  const float* yr = y != nullptr ? y + (size_t)r * d : nullptr;
  float* wr = xs != nullptr ? xs + (size_t)r * n_streams * d : nullptr;
  Group<V> u[COLS];
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < COLS; ++k) {
    const int c = (tid + k * (int)blockDim.x) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) u[k].v[e] = 0.0f;
    if (c >= d) continue;
    Group<V> x[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (s < n_streams) {
        x[s].load(xr + (size_t)s * in_stream + c);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) x[s].v[e] = 0.0f;
      }
    }
    if (yr != nullptr) {
      Group<V> yv, lv;
      yv.load(yr + c);
      lv.load(scale_w + c);
#pragma unroll
      for (int e = 0; e < V; ++e) yv.v[e] *= lv.v[e];
      Group<V> total;
#pragma unroll
      for (int e = 0; e < V; ++e) total.v[e] = 0.0f;
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t < n_streams) {
          Group<V> n;
#pragma unroll
          for (int e = 0; e < V; ++e) {
            float a = c_gain[t] * yv.v[e];
#pragma unroll
            for (int s = 0; s < S; ++s) a = fmaf(c_mix[s][t], x[s].v[e], a);
            n.v[e] = a;
            total.v[e] += a;
            u[k].v[e] = fmaf(c_in[t], a, u[k].v[e]);
          }
          if (wr != nullptr) n.store(wr + (size_t)t * d + c);
        }
      }
      if (sum != nullptr) total.store(sum + (size_t)r * d + c);
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int e = 0; e < V; ++e) u[k].v[e] = fmaf(c_in[s], x[s].v[e], u[k].v[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(u[k].v[e], u[k].v[e], ss);
  }
  if (out_next == nullptr) return;
  ss = nb_block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)d + next_eps);
#pragma unroll
  for (int k = 0; k < COLS; ++k) {
    const int c = (tid + k * (int)blockDim.x) * V;
    if (c >= d) continue;
    Group<V> g;
    g.load(next_gamma + c);
    float o[V];
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = u[k].v[e] * inv * g.v[e];
    store_act(out_next + (size_t)r * d + c, o);
  }
}

}  // namespace

// x_in: fp32 rows of in_row floats, stream s at in_stream * s (0: every stream is the same row);
// xs: fp32 [n_rows][n_streams][d], may be x_in itself, or null where only `sum` is wanted; y: fp32
// [n_rows][d] or null (read alone); ls: fp32 [d]; mix: fp32 [from][to]; gain: fp32 [n_streams]; sum:
// fp32 [n_rows][d] or null; next_coef [n_streams], next_gamma [d] and out_next [n_rows][d], or
// null.
NB_EXPORT int nb_streams(const float* x_in, int in_row, int in_stream, int n_streams, float* xs,
                         const float* y, const float* ls, const float* mix, const float* gain,
                         float* sum, const float* next_coef, const float* next_gamma, float next_eps,
                         void* out_next, int out_dtype, int n_rows, int d, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NB_REQUIRE(n_rows > 0 && d > 0 && n_streams >= 1 && n_streams <= MAX_S && in_stream >= 0 &&
                 in_row >= in_stream * (n_streams - 1) + d,
             NB_ERR_BAD_ARG, "streams: bad sizes rows=%d d=%d streams=%d", n_rows, d, n_streams);
  NB_REQUIRE(y == nullptr || (ls != nullptr && mix != nullptr && gain != nullptr && (xs || sum)),
             NB_ERR_BAD_ARG, "streams: a write-back needs its coefficients and a place");
  NB_REQUIRE(out_next == nullptr || (next_coef != nullptr && next_gamma != nullptr), NB_ERR_BAD_ARG,
             "streams: a read needs its coefficients and the norm's weight");
  const uintptr_t all = (uintptr_t)x_in | (uintptr_t)xs | (uintptr_t)y | (uintptr_t)ls | (uintptr_t)sum |
                        (uintptr_t)next_gamma | (uintptr_t)out_next;
  const bool vec = d % 4 == 0 && in_row % 4 == 0 && in_stream % 4 == 0 && (all & 15) == 0;
  const int groups = vec ? d / 4 : d;
  // few rows (a one-token step): one or two column groups a thread; many rows: more loads in
  // flight per thread
  int threads = 64;
  const int per = n_rows >= 148 * 4 ? 2 : 1;
  while (threads < 512 && threads * per < groups) threads *= 2;
  NB_REQUIRE(threads * COLS >= groups, NB_ERR_UNSUPPORTED, "streams: width %d is too large", d);
#define NB_ST(TO, S_, V_)                                                                         \
  NB_CUDA(nb_launch(streams_kernel<TO, S_, V_>, dim3(n_rows), dim3(threads), 0, stream, x_in, in_row, \
                    in_stream, n_streams, xs, y, ls, mix, gain, sum, next_coef, next_gamma,       \
                    next_eps, (TO*)out_next, d))
#define NB_ST_S(TO, V_)                                                                           \
  switch (n_streams) {                                                                            \
    case 1: NB_ST(TO, 1, V_); break;                                                              \
    case 2: NB_ST(TO, 2, V_); break;                                                              \
    case 3: NB_ST(TO, 3, V_); break;                                                              \
    case 4: NB_ST(TO, 4, V_); break;                                                              \
    default: NB_ST(TO, 8, V_); break;                                                             \
  }
  if (out_next == nullptr || out_dtype == NB_F32) {
    if (vec) { NB_ST_S(float, 4) } else { NB_ST_S(float, 1) }
  } else if (out_dtype == NB_BF16) {
    if (vec) { NB_ST_S(bf16, 4) } else { NB_ST_S(bf16, 1) }
  } else {
    NB_REQUIRE(false, NB_ERR_BAD_ARG, "streams: unknown output dtype %d", out_dtype);
  }
#undef NB_ST_S
#undef NB_ST
  NB_CHECK_LAUNCH("streams");
  return 0;
}

// ---------------------------------------------------------------------------------
// x <- cap * tanh(x / cap), in place (logits with a cap).
// ---------------------------------------------------------------------------------
namespace {
__global__ void softcap_rows_kernel(float* x, float cap, float inv_cap, size_t total) {
  nb_grid_dependency_wait();
  nb_launch_dependents();
  const size_t step = (size_t)gridDim.x * blockDim.x * 4;
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4; i < total; i += step) {
    if (i + 4 <= total) {
      float4 f = *reinterpret_cast<float4*>(x + i);
      f.x = cap * tanhf(f.x * inv_cap);
      f.y = cap * tanhf(f.y * inv_cap);
      f.z = cap * tanhf(f.z * inv_cap);
      f.w = cap * tanhf(f.w * inv_cap);
      *reinterpret_cast<float4*>(x + i) = f;
    } else {
      for (size_t k = i; k < total; ++k) x[k] = cap * tanhf(x[k] * inv_cap);
    }
  }
}
}  // namespace

NB_EXPORT int nb_softcap_rows(float* x, float cap, long long total, cudaStream_t stream) {
  if (total == 0) return 0;
  NB_REQUIRE(total > 0 && cap > 0.0f && (uintptr_t)x % 16 == 0, NB_ERR_BAD_ARG,
             "softcap_rows: bad arguments (cap %g)", (double)cap);
  const long long want = (total + 1023) / 1024;
  const int blocks = (int)(want < 148 * 8 ? want : 148 * 8);
  NB_CUDA(nb_launch(softcap_rows_kernel, dim3(blocks), dim3(256), 0, stream, x, cap, 1.0f / cap,
                    (size_t)total));
  NB_CHECK_LAUNCH("softcap_rows");
  return 0;
}
