// The gated delta rule: a linear recurrence over a sequence's tokens with a matrix state per head
// (key channels x value channels, fp32) and a decay per key channel.
//
//   S' = diag(g_t) S_(t-1),   u_t = beta_t (v_t - S'^T k_t),   S_t = S' + k_t u_t^T,   o_t = S_t^T q_t
//
// q and k are unit vectors per head (x / sqrt(sum x^2 + key_eps), q also times d^(-1/2)), beta =
// sigmoid(logit), g = exp(-exp(a_log_h) softplus(x + dt_bias)).  Afterwards each head's o is
// divided by its root mean square (eps inside the root), times a weight shared by the heads, times
// sigmoid(gate logits).  Everything is fp32.
//
// Prompts.  Eight tokens are taken at a time.  With E_(s..t) = the product of g over tokens s+1 .. t
// of the block (per key channel; from the block's start: E_t) and S the state at its start,
//
//   u_t = beta_t v_t - (beta_t E_t k_t)^T S - sum_(s<t) A_ts u_s,   A_ts = beta_t sum_i k_ti k_si E_(s..t)i
//   o_t = (E_t q_t)^T S + sum_(s<=t) B_ts u_s,                     B_ts = sum_i q_ti k_si E_(s..t)i
//   S  <- diag(E_7) S + sum_s (k_s E_(s..7)) u_s^T
//
// so the state is read twice and written once per eight tokens, the sixteen dot products of a column
// with it are independent of one another, and only the eight u_t (a few multiply-adds) follow one
// another.  Decays are multiplied up, never divided by, so nothing overflows however strong they are.
//   gated_delta_prepare  two warps per (block of eight tokens, head), four tokens each: the short
//                        convolution and silu of q, k and v (of projected rows, the inputs before
//                        the step from the state row), then a record: E_7, the eight (beta_t E_t
//                        k_t), (E_t q_t), (k_s E_(s..7)), the numbers A and B, and the eight beta_t
//                        v_t.  The first four tokens' part and the second's meet through shared
//                        memory.  A block's missing tokens (a sequence's last block) are tokens with
//                        k = q = v = 0, g = 1.
//   gated_delta_walk     a CTA takes COLS columns of one (sequence, head); the columns are
//                        independent.  A group of LPG lanes holds NC columns, CH key channels a
//                        lane, two neighbouring channels in a register pair (packed multiply-adds).
//                        The 16 NC partial sums of a block (eight tokens, NC columns, two products)
//                        are reduced over the lanes by halving: each lane ends with 16 NC / LPG of
//                        them.  Records come through two buffers of asynchronous copies.
//   delta_finish         norm, weight and gate (the norm needs all of a head's columns).
// A sequence may be cut into steps anywhere: where blocks begin only changes the rounding.
//
// One-token steps.  gated_delta_step: a CTA per (sequence, head, 32 columns), the CTAs of a head in a
// thread-block cluster that adds up the head's sum of squares through shared memory, or, where there
// are heads enough to fill the GPU, a CTA per 128 columns.  The state is fetched before the wait on
// the kernel in front (which never writes it), read and written once; both products with it are
// taken of the decayed state (S_t^T q = S'^T q + (k . q) u), so their sums meet in one exchange.
#include "delta_common.cuh"
#include "attention_common.cuh"

namespace {

constexpr int BLK = 8;         // tokens of a block
constexpr int HALF = 4;        // ... of a preparing warp
constexpr int MAX_DIM = 256;

__device__ __forceinline__ float gd_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// Sums of N values over L lanes by halving; the lanes are STEP apart and q is the lane's number among
// them.  Afterwards it holds the sums with indices q * (N / L) .. in v[0 ..] (N >= L), or, when N < L,
// index q / (L / N).
template <int N, int L, int STEP>
__device__ __forceinline__ void reduce_by_halving(float (&v)[N], int q) {
  int n = N;
#pragma unroll
  for (int m = L / 2; m >= 1; m >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = (q & m) != 0;
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        if (i < n) {
          const float send = up ? v[i] : v[i + n];
          const float keep = up ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, m * STEP);
        }
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], m * STEP);
    }
  }
}

struct Source {               // where a row's numbers lie
  const float* qkv;           // rows of qkv_stride: q heads, k heads, v heads from column qkv_col
  int qkv_stride, qkv_col;
  // taps > 0: those are projections, to be convolved (conv: [channels][taps]; inputs: a slot's last
  // taps - 1 rows of channels at inputs + slot * in_stride) and activated; 0: they are ready
  const float* conv;
  int taps;
  float* inputs;
  int in_stride, channels;
  const float* beta;          // [rows][beta_stride], head h's logit at column beta_col + h
  int beta_stride, beta_col;
  const float* low;           // [rows][low_stride]: decay logits at decay_col, gate logits at gate_col
  int low_stride, decay_col, gate_col;
  const float* a_log;         // [heads]
  const float* dt_bias;       // [heads * d]
};

// A record: E at place 0 (of DP floats), beta E k at 1 .., E q at 1 + BLK .., k E at 1 + 2 BLK .., then A
// and B (BLK x BLK each) and the values.
// floats of a record of padded key size DP; dvp: the value size rounded up to a multiple of 4
__host__ __device__ constexpr int record_head(int DP) { return (3 * BLK + 1) * DP + 2 * BLK * BLK; }
__host__ __device__ inline int record_floats(int DP, int dvp) { return record_head(DP) + BLK * dvp; }

constexpr int MAX_FUSED_TAPS = 4;

// Four neighbouring channels c .. c+3 (those below `end`) of HALF tokens: y[t] = the ready numbers or
// silu of the convolution.  base: the channels' first column in a row; ch0: their first channel.
// CONV: 0 ready, 1 convolved, 2 convolved with the hardware's exponential and reciprocal in the silu
// (a bfloat16 run, where projections and their activations are rounded anyway).
template <int CONV>
__device__ __forceinline__ void take_channels(const Source& src, const float* in_row, int row0, int row1,
                                              int first, int ch0, int c, int end, bool vec,
                                              float (&y)[HALF][4]) {
  auto load4 = [&](const float* p, float (&v)[4]) {
    if (vec && c < end) {
      const float4 f = *reinterpret_cast<const float4*>(p);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = c + e < end ? p[e] : 0.0f;
    }
  };
  const float* col = src.qkv + src.qkv_col + ch0 + c;
  if constexpr (CONV == 0) {
#pragma unroll
    for (int t = 0; t < HALF; ++t)
      load4(col + (size_t)(first + t < row1 ? first + t : row0) * src.qkv_stride, y[t]);
  } else {
    // inputs first - 3 .. first + 3; weights with zeros in front up to four taps
    float x[HALF + MAX_FUSED_TAPS - 1][4], w[MAX_FUSED_TAPS][4];
    const int taps = src.taps;
#pragma unroll
    for (int i = 0; i < HALF + MAX_FUSED_TAPS - 1; ++i) {
      const int r = first - (MAX_FUSED_TAPS - 1) + i;
      const int back = row0 - r;                 // rows before the step's first: 1 is the newest
      if (back <= 0) load4(col + (size_t)(r < row1 ? r : row0) * src.qkv_stride, x[i]);
      else if (back < taps) load4(in_row + (size_t)(taps - 1 - back) * src.channels + ch0 + c, x[i]);
      else x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.0f;
    }
    if (taps == MAX_FUSED_TAPS && vec && c < end) {          // (the weights of a channel: 16 bytes)
      const float4* wp = reinterpret_cast<const float4*>(src.conv) + ch0 + c;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 f = wp[e];
        w[0][e] = f.x; w[1][e] = f.y; w[2][e] = f.z; w[3][e] = f.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < MAX_FUSED_TAPS; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int tap = j - (MAX_FUSED_TAPS - taps);
          w[j][e] = (tap >= 0 && c + e < end) ? src.conv[(size_t)(ch0 + c + e) * taps + tap] : 0.0f;
        }
    }
#pragma unroll
    for (int t = 0; t < HALF; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = 0.0f;
#pragma unroll
        for (int j = 0; j < MAX_FUSED_TAPS; ++j) v = fmaf(w[j][e], x[t + j][e], v);
        y[t][e] = CONV == 2 ? nb_silu_fast(v) : nb_silu(v);
      }
  }
}

// A sequence's blocks start at record cu_rows[seq] / BLK + seq, so that no two sequences overlap.
template <int DP, int CONV>
__global__ void __launch_bounds__(128)
gated_delta_prepare_kernel(Source src, float key_eps, const int* cu_rows, const int* seq_slot,
                           float* records, int n_heads, int n_kv_heads, int d, int dv, int vec,
                           int vec_in, int vec_v) {
  nb_grid_dependency_wait();
  nb_launch_dependents();
  constexpr int KIT = (DP + 127) / 128;             // quads of channels a lane holds
  constexpr int N = KIT * 4;
  __shared__ __align__(16) float kh_s[2][HALF][DP], e_s[2][2][DP];
  const int seq = blockIdx.z, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int pair = warp >> 1, part = warp & 1;      // the CTA's block, and which of its halves
  const int blk = blockIdx.x * 2 + pair;
  const int row0 = cu_rows[seq], row1 = cu_rows[seq + 1], slot = seq_slot[seq];
  if (slot < 0 || row0 + (int)blockIdx.x * 2 * BLK >= row1) return;      // the whole CTA
  const bool there = row0 + blk * BLK < row1;
  const int first = row0 + blk * BLK + part * HALF; // of this warp's tokens
  const int g = h / (n_heads / n_kv_heads);
  const int dvp = (dv + 3) & ~3;
  float* rec = records + ((size_t)(row0 / BLK + seq + blk) * n_heads + h) * record_floats(DP, dvp);
  const float* in_row = CONV ? src.inputs + (size_t)slot * src.in_stride : nullptr;
  const float rate = expf(src.a_log[h]);
  const float q_scale = 1.0f / sqrtf((float)d);
  // 16-byte loads of the rows; near the step's start also of the state row
  const bool inner = !CONV || vec || blk > 0 || part > 0;
  const bool vec_q = vec_in && inner;
  auto place = [&](int p, int j) { return rec + p * DP + (j * 32 + lane) * 4; };
  auto has = [&](int j) { return (j * 32 + lane) * 4 < DP; };
  auto store = [&](int p, const float (&v)[N]) {
#pragma unroll
    for (int j = 0; j < KIT; ++j)
      if (has(j))
        *reinterpret_cast<float4*>(place(p, j)) = make_float4(v[j * 4], v[j * 4 + 1], v[j * 4 + 2], v[j * 4 + 3]);
  };
  auto put = [&](float* at, const float (&v)[N]) {        // into a row of shared memory
#pragma unroll
    for (int j = 0; j < KIT; ++j)
      if (has(j))
        *reinterpret_cast<float4*>(at + (j * 32 + lane) * 4) =
            make_float4(v[j * 4], v[j * 4 + 1], v[j * 4 + 2], v[j * 4 + 3]);
  };
  auto take = [&](const float* at, float (&v)[N]) {
#pragma unroll
    for (int j = 0; j < KIT; ++j) {
      const float4 f = has(j) ? *reinterpret_cast<const float4*>(at + (j * 32 + lane) * 4)
                              : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      v[j * 4] = f.x; v[j * 4 + 1] = f.y; v[j * 4 + 2] = f.z; v[j * 4 + 3] = f.w;
    }
  };

  float k[HALF][N], q[HALF][N], w[HALF][N], beta[HALF], ab[16];
  if (there) {
#pragma unroll
    for (int j = 0; j < KIT; ++j) {
      const int c = (j * 32 + lane) * 4;
      float y[HALF][4];
      take_channels<CONV>(src, in_row, row0, row1, first, g * d, c, d, vec_q, y);
#pragma unroll
      for (int t = 0; t < HALF; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) q[t][j * 4 + e] = y[t][e];
      take_channels<CONV>(src, in_row, row0, row1, first, (n_kv_heads + g) * d, c, d, vec_q, y);
#pragma unroll
      for (int t = 0; t < HALF; ++t) {
        const int r = first + t < row1 ? first + t : row0;
        const float* dl = src.low + (size_t)r * src.low_stride + src.decay_col + h * d + c;
#pragma unroll
        for (int e = 0; e < 4; ++e) k[t][j * 4 + e] = y[t][e];
        if (vec_in && c < d) {
          const float4 f = *reinterpret_cast<const float4*>(dl);
          w[t][j * 4] = f.x; w[t][j * 4 + 1] = f.y; w[t][j * 4 + 2] = f.z; w[t][j * 4 + 3] = f.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) w[t][j * 4 + e] = c + e < d ? dl[e] : 0.0f;
        }
      }
    }
#pragma unroll
    for (int t = 0; t < HALF; ++t)
      beta[t] = first + t < row1
                    ? nb_sigmoid(src.beta[(size_t)(first + t) * src.beta_stride + src.beta_col + h]) : 0.0f;
    // unit vectors and decays
    float ss[2 * HALF];
#pragma unroll
    for (int t = 0; t < HALF; ++t) {
      ss[t] = ss[HALF + t] = 0.0f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        ss[t] = fmaf(k[t][i], k[t][i], ss[t]);
        ss[HALF + t] = fmaf(q[t][i], q[t][i], ss[HALF + t]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2 * HALF; ++i) ss[i] = nb_warp_sum(ss[i]);
#pragma unroll
    for (int t = 0; t < HALF; ++t) {
      const bool live = first + t < row1;
      const float ik = live ? 1.0f / sqrtf(ss[t] + key_eps) : 0.0f;
      const float iq = live ? q_scale / sqrtf(ss[HALF + t] + key_eps) : 0.0f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = ((i >> 2) * 32 + lane) * 4 + (i & 3);
        k[t][i] *= ik;
        q[t][i] *= iq;
        w[t][i] = (live && c < d) ? expf(-rate * gd_softplus(w[t][i] + src.dt_bias[h * d + c])) : 1.0f;
      }
    }
    // A (six numbers) and B (ten) among this half's tokens, and k_s decayed to the half's end
#pragma unroll
    for (int s = 0; s < HALF; ++s) {
      float kd[N];
#pragma unroll
      for (int i = 0; i < N; ++i) kd[i] = k[s][i];
#pragma unroll
      for (int t = s; t < HALF; ++t) {
        float a = 0.0f, b = 0.0f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
          if (t > s) kd[i] *= w[t][i];
          a = fmaf(k[t][i], kd[i], a);
          b = fmaf(q[t][i], kd[i], b);
        }
        if (t > s) ab[t * (t - 1) / 2 + s] = a;
        ab[6 + t * (t + 1) / 2 + s] = b;
      }
      if (part == 0) put(kh_s[pair][s], kd);
      else store(1 + 2 * BLK + HALF + s, kd);
    }
    reduce_by_halving<16, 32, 1>(ab, lane);           // lane l holds number l / 2
    // beta_t E_t k_t and E_t q_t from the half's start
#pragma unroll
    for (int t = 0; t < HALF; ++t)
#pragma unroll
      for (int i = 0; i < N; ++i) {
        if (t > 0) w[t][i] *= w[t - 1][i];
        k[t][i] *= beta[t] * w[t][i];
        q[t][i] *= w[t][i];
      }
    put(e_s[pair][part], w[HALF - 1]);
  }
  __syncthreads();
  if (!there) return;
  // a row of A and of B: slot `lane` is row t of the half, column s of the block
  float across[32];
  if (part == 0) {
    float e2[N], e[N];
    take(e_s[pair][1], e2);
#pragma unroll
    for (int s = 0; s < HALF; ++s) {
      float kd[N];
      take(kh_s[pair][s], kd);
#pragma unroll
      for (int i = 0; i < N; ++i) kd[i] *= e2[i];
      store(1 + 2 * BLK + s, kd);
      store(1 + s, k[s]);
      store(1 + BLK + s, q[s]);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) e[i] = w[HALF - 1][i] * e2[i];
    store(0, e);
  } else {
    float e1[N];
    take(e_s[pair][0], e1);
#pragma unroll
    for (int s = 0; s < HALF; ++s) {
      float kd[N];
      take(kh_s[pair][s], kd);
#pragma unroll
      for (int t = 0; t < HALF; ++t) {
        float a = 0.0f, b = 0.0f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
          a = fmaf(k[t][i], kd[i], a);
          b = fmaf(q[t][i], kd[i], b);
        }
        across[t * HALF + s] = a;
        across[16 + t * HALF + s] = b;
      }
    }
    reduce_by_halving<32, 32, 1>(across, lane);      // lane l holds number l
#pragma unroll
    for (int t = 0; t < HALF; ++t) {
#pragma unroll
      for (int i = 0; i < N; ++i) {
        k[t][i] *= e1[i];
        q[t][i] *= e1[i];
      }
      store(1 + HALF + t, k[t]);
      store(1 + BLK + HALF + t, q[t]);
    }
  }
  {
    const int t = lane >> 3, col = lane & 7, s = col - part * HALF;     // s: within the half
    const float bt = t == 0 ? beta[0] : t == 1 ? beta[1] : t == 2 ? beta[2] : beta[3];
    const bool in_a = s >= 0 && s < t, in_b = s >= 0 && s <= t && s < HALF;
    float a = __shfl_sync(0xffffffffu, ab[0], in_a ? 2 * (t * (t - 1) / 2 + s) : 0) * bt;
    float b = __shfl_sync(0xffffffffu, ab[0], in_b ? 2 * (6 + t * (t + 1) / 2 + s) : 0);
    if (!in_a) a = 0.0f;
    if (!in_b) b = 0.0f;
    if (part == 1) {
      const float xa = __shfl_sync(0xffffffffu, across[0], col < HALF ? t * HALF + col : 0);
      const float xb = __shfl_sync(0xffffffffu, across[0], col < HALF ? 16 + t * HALF + col : 0);
      if (col < HALF) {
        a = xa;
        b = xb;
      }
    }
    float* at = rec + (3 * BLK + 1) * DP + (part * HALF + t) * BLK + col;
    at[0] = a;
    at[BLK * BLK] = b;
  }
  // beta_t v_t
  float* vd = rec + record_head(DP) + part * HALF * dvp;
  for (int c = lane * 4; c < dvp; c += 128) {
    float y[HALF][4];
    take_channels<CONV>(src, in_row, row0, row1, first, 2 * n_kv_heads * d + h * dv, c, dv,
                        vec_v && inner, y);
#pragma unroll
    for (int t = 0; t < HALF; ++t) {
      const float b = beta[t];                     // zero for a missing token
      *reinterpret_cast<float4*>(vd + t * dvp + c) =
          make_float4(b * y[t][0], b * y[t][1], b * y[t][2], b * y[t][3]);
    }
  }
}

// two fp32 numbers in a register pair
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pair_of(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};\n" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpair(f32x2 v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;\n" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// NC numbers that lie side by side
template <int NC>
__device__ __forceinline__ void load_cols(const float* p, float (&v)[NC]) {
  if constexpr (NC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
  }
}
template <int NC>
__device__ __forceinline__ void store_cols(float* p, const float (&v)[NC]) {
  if constexpr (NC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}

// CH: key channels a lane holds for each of its NC columns; LPG: lanes of a group; NW: warps.
template <int CH, int LPG, int NC, int NW>
struct Walk {
  static constexpr int DP = CH * LPG;
  static constexpr int GPW = 32 / LPG;                           // groups of a warp
  static constexpr int GROUPS = NW * GPW;
  static constexpr int COLS = NC * GROUPS;
  static constexpr int V = 2 * BLK * NC;                         // sums of a block and group
  static constexpr int SB = DP > 128 ? 1 : 2;                    // blocks a buffer holds
  static constexpr int BUF = SB * (record_head(DP) + BLK * COLS);  // floats of a buffer
  static constexpr int SMEM = (2 * BUF + 2 * GROUPS * V) * 4;
};

template <int CH, int LPG, int NC, int NW>
__global__ void __launch_bounds__(NW * 32)
gated_delta_walk_kernel(const float* records, const int* cu_rows, const int* seq_slot, float* state,
                        int state_stride, float* o_raw, int n_heads, int d, int dv, int vec) {
  using W = Walk<CH, LPG, NC, NW>;
  constexpr int DP = W::DP, COLS = W::COLS, SB = W::SB, THREADS = NW * 32, HEAD = record_head(DP);
  constexpr int GPW = W::GPW, V = W::V;
  static_assert(CH % 4 == 0 && COLS % 4 == 0 && LPG >= BLK && V >= LPG && (NC == 2 || NC == 4),
                "a lane takes its channels four at a time");
  nb_grid_dependency_wait();
  extern __shared__ __align__(16) float sm[];
  float* red = sm + 2 * W::BUF;                     // [2][groups][V]
  const int col0 = blockIdx.x * COLS, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int row0 = cu_rows[seq], row1 = cu_rows[seq + 1];
  const int slot = seq_slot[seq];
  if (slot < 0 || row1 <= row0) return;
  // the groups of a warp lie in turn over its lanes: neighbours read the same numbers of a record
  const int lane = tid & 31, group = (tid >> 5) * GPW + lane % GPW, q = lane / GPW;
  const int col = col0 + group * NC;                // this group's columns
  const int dvp = (dv + 3) & ~3, rec_floats = record_floats(DP, dvp);
  const int n_blocks = (row1 - row0 + BLK - 1) / BLK;
  const float* recs = records + ((size_t)(row0 / BLK + seq) * n_heads + h) * rec_floats;
  const size_t rec_step = (size_t)n_heads * rec_floats;
  float* st = state + (size_t)slot * state_stride + (size_t)h * d * dv;

  auto fetch = [&](int b0, int buf) {               // blocks b0 .. b0 + SB - 1 (those that exist)
    float* dst = sm + buf * W::BUF;
    const int nb = min(SB, n_blocks - b0);
    for (int b = 0; b < nb; ++b) {
      const float* rec = recs + (size_t)(b0 + b) * rec_step;
      for (int i = tid; i < HEAD / 4; i += THREADS) cp_async16(dst + b * HEAD + i * 4, rec + i * 4);
      for (int i = tid; i < BLK * COLS / 4; i += THREADS) {
        const int t = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
        if (col0 + c < dvp)
          cp_async16(dst + SB * HEAD + (b * BLK + t) * COLS + c, rec + HEAD + t * dvp + col0 + c);
      }
    }
    cp_async_commit();
  };
  fetch(0, 0);

  // key channels of pair number i of this lane: quads of channels, dealt out to the lanes in turn
  auto channel = [q](int i) { return (((i >> 1) * LPG + q) << 2) + 2 * (i & 1); };
  f32x2 S[CH / 2][NC];                              // [channel pair][column]
#pragma unroll
  for (int i = 0; i < CH / 2; ++i) {
    float v[2][NC];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = channel(i) + e;
#pragma unroll
      for (int j = 0; j < NC; ++j) v[e][j] = 0.0f;
      if (c < d && col < dv) {
        if (vec) {
          load_cols<NC>(st + (size_t)c * dv + col, v[e]);
        } else {
#pragma unroll
          for (int j = 0; j < NC; ++j)
            if (col + j < dv) v[e][j] = st[(size_t)c * dv + col + j];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NC; ++j) S[i][j] = pair_of(v[0][j], v[1][j]);
  }

  // this lane's output: token q of a block (the first BLK lanes of a group)
  float* o_at = o_raw + ((size_t)(row0 + q) * n_heads + h) * dv + col;
  const size_t o_step = (size_t)BLK * n_heads * dv;
  const int o_rows = q < BLK && col < dv ? row1 - row0 - q : 0;    // tokens there are for it
  int parity = 0, token = 0;
  for (int b0 = 0, buf = 0; b0 < n_blocks; b0 += SB, buf ^= 1) {
    cp_async_wait<0>();
    __syncthreads();                 // the buffer is in, and every thread has left the other one
    if (b0 + SB < n_blocks) fetch(b0 + SB, buf ^ 1);
    const float* head = sm + buf * W::BUF;
    const float* vals = head + SB * HEAD + group * NC;
    const int nb = min(SB, n_blocks - b0);
    for (int b = 0; b < nb; ++b, head += HEAD, vals += BLK * COLS) {
      // (beta E k)_t . S_c at t NC + c,  (E q)_t . S_c at V / 2 + t NC + c
      float p[V];
#pragma unroll
      for (int t = 0; t < 2 * BLK; ++t) {           // the places 1 .. 2 BLK of the record
        f32x2 acc[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) acc[c] = 0ull;
#pragma unroll
        for (int g = 0; g < CH / 4; ++g) {
          const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(head + (1 + t) * DP + (g * LPG + q) * 4);
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            acc[c] = fma2(x.x, S[2 * g][c], acc[c]);
            acc[c] = fma2(x.y, S[2 * g + 1][c], acc[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          const float2 f = unpair(acc[c]);
          p[t * NC + c] = f.x + f.y;
        }
      }
      reduce_by_halving<V, LPG, GPW>(p, q);
      float* mine = red + (parity * W::GROUPS + group) * V;
      parity ^= 1;
#pragma unroll
      for (int i = 0; i < V / LPG; ++i) mine[q * (V / LPG) + i] = p[i];
      __syncwarp();
      // the eight u
      float u[BLK][NC];
      const float* amat = head + (3 * BLK + 1) * DP;
#pragma unroll
      for (int t = 0; t < BLK; ++t) {
        float r[NC];
        load_cols<NC>(mine + t * NC, r);
        load_cols<NC>(vals + t * COLS, u[t]);
        float a[BLK];
#pragma unroll
        for (int s4 = 0; s4 < (t + 3) / 4; ++s4) {
          const float4 f = *reinterpret_cast<const float4*>(amat + t * BLK + s4 * 4);
          a[s4 * 4] = f.x; a[s4 * 4 + 1] = f.y; a[s4 * 4 + 2] = f.z; a[s4 * 4 + 3] = f.w;
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          u[t][c] -= r[c];
#pragma unroll
          for (int s2 = 0; s2 < t; ++s2) u[t][c] = fmaf(-a[s2], u[s2][c], u[t][c]);
        }
      }
      // the state
      f32x2 uu[BLK][NC];
#pragma unroll
      for (int t = 0; t < BLK; ++t)
#pragma unroll
        for (int c = 0; c < NC; ++c) uu[t][c] = pair_of(u[t][c], u[t][c]);
#pragma unroll
      for (int g = 0; g < CH / 4; ++g) {
        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(head + (g * LPG + q) * 4);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          S[2 * g][c] = mul2(w.x, S[2 * g][c]);
          S[2 * g + 1][c] = mul2(w.y, S[2 * g + 1][c]);
        }
#pragma unroll
        for (int t = 0; t < BLK; ++t) {
          const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(head + (1 + 2 * BLK + t) * DP + (g * LPG + q) * 4);
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            S[2 * g][c] = fma2(kk.x, uu[t][c], S[2 * g][c]);
            S[2 * g + 1][c] = fma2(kk.y, uu[t][c], S[2 * g + 1][c]);
          }
        }
      }
      // a token's outputs: lane t of the group has token t
      if (token < o_rows) {
        float o[NC];
        load_cols<NC>(mine + V / 2 + q * NC, o);
#pragma unroll
        for (int s4 = 0; s4 < BLK / 4; ++s4) {
          const float4 f = *reinterpret_cast<const float4*>(amat + BLK * BLK + q * BLK + s4 * 4);
#pragma unroll
          for (int c = 0; c < NC; ++c)
            o[c] = fmaf(f.x, u[s4 * 4][c], fmaf(f.y, u[s4 * 4 + 1][c],
                   fmaf(f.z, u[s4 * 4 + 2][c], fmaf(f.w, u[s4 * 4 + 3][c], o[c]))));
        }
        if (vec) {
          store_cols<NC>(o_at, o);
        } else {
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (col + c < dv) o_at[c] = o[c];
        }
      }
      token += BLK;
      o_at += o_step;
    }
  }
  nb_launch_dependents();
#pragma unroll
  for (int i = 0; i < CH / 2; ++i) {
    float v[2][NC];
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      const float2 f = unpair(S[i][j]);
      v[0][j] = f.x;
      v[1][j] = f.y;
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = channel(i) + e;
      if (c >= d || col >= dv) continue;
      if (vec) {
        store_cols<NC>(st + (size_t)c * dv + col, v[e]);
      } else {
#pragma unroll
        for (int j = 0; j < NC; ++j)
          if (col + j < dv) st[(size_t)c * dv + col + j] = v[e][j];
      }
    }
  }
}

// One token per sequence.  COLS columns a CTA; thread: four neighbouring ones (cq) of the key channels
// rg, rg + RG, ...
constexpr int ST_THREADS = 256;

template <int NV, int COLS, typename TOut>
__global__ void __launch_bounds__(ST_THREADS, COLS == 128 ? 2 : (NV > 4 ? 1 : 4))
gated_delta_step_kernel(Source src, float key_eps, const float* __restrict__ norm_w, float eps,
                        const int* cu_rows, const int* seq_slot, float* state, int state_stride,
                        TOut* out, int n_heads, int n_kv_heads, int d, int dv, int vec) {
  constexpr int CQ = COLS / 4, RG = ST_THREADS / CQ, NW = ST_THREADS / 32;
  static_assert(CQ == 8 || CQ == 32, "a warp covers whole rows of columns");
  __shared__ float k_s[NV * RG], q_s[NV * RG], w_s[NV * RG];
  __shared__ __align__(16) float part[2][NW][COLS];
  __shared__ float red[3][NW], square[8];
  const int split = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int lane = tid & 31, warp = tid >> 5;
  const int n_splits = gridDim.x;                   // the cluster
  const int r = cu_rows[seq], slot = cu_rows[seq + 1] > r ? seq_slot[seq] : -1;
  const int hv = n_heads * dv;
  if (slot < 0) {              // the whole cluster leaves
    nb_grid_dependency_wait();
    nb_launch_dependents();
    const int c = split * COLS + tid;
    if (cu_rows[seq + 1] > r && tid < COLS && c < dv)
      out[(size_t)r * hv + h * dv + c] = nb_from_f32<TOut>(0.0f);
    return;
  }
  const int cq = tid % CQ, rg = tid / CQ, col = split * COLS + cq * 4;
  const int g = h / (n_heads / n_kv_heads);
  float* st = state + (size_t)slot * state_stride + (size_t)h * d * dv;
  float S[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = rg + RG * i;
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.0f;
    if (k >= d || col >= dv) continue;
    if (vec) {
      const float4 f = *reinterpret_cast<const float4*>(st + (size_t)k * dv + col);
      S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < dv) S[i][j] = st[(size_t)k * dv + col + j];
    }
  }
  nb_grid_dependency_wait();
  // every CTA of the cluster says that it runs; the matching wait stands in front of the first
  // store into another CTA's shared memory
  if (n_splits > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;\n" ::: "memory");

  const float* row = src.qkv + (size_t)r * src.qkv_stride + src.qkv_col;
  const float* low = src.low + (size_t)r * src.low_stride;
  float v4[4], gate[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const bool in = col + j < dv;
    v4[j] = in ? row[2 * n_kv_heads * d + h * dv + col + j] : 0.0f;
    gate[j] = (in && tid < CQ) ? low[src.gate_col + h * dv + col + j] : 0.0f;
  }
  const float beta = nb_sigmoid(src.beta[(size_t)r * src.beta_stride + src.beta_col + h]);
  float kx = 0.0f, qx = 0.0f, wx = 0.0f;
  if (tid < d) {
    kx = row[(n_kv_heads + g) * d + tid];
    qx = row[g * d + tid];
    wx = expf(-expf(src.a_log[h]) * gd_softplus(low[src.decay_col + h * d + tid] + src.dt_bias[h * d + tid]));
  }
  const float sk = nb_warp_sum(kx * kx), sq = nb_warp_sum(qx * qx), skq = nb_warp_sum(kx * qx);
  if (lane == 0) {
    red[0][warp] = sk;
    red[1][warp] = sq;
    red[2][warp] = skq;
  }
  __syncthreads();
  float tk = 0.0f, tq = 0.0f, kq = 0.0f;
#pragma unroll
  for (int i = 0; i < NW; ++i) {
    tk += red[0][i];
    tq += red[1][i];
    kq += red[2][i];
  }
  const float ik = 1.0f / sqrtf(tk + key_eps), iq = 1.0f / (sqrtf(tq + key_eps) * sqrtf((float)d));
  kq *= ik * iq;
  if (tid < NV * RG) {
    k_s[tid] = kx * ik;
    q_s[tid] = qx * iq;
    w_s[tid] = wx;
  }
  __syncthreads();
  // a: S'^T k, o: S'^T q of four columns: the thread's key channels, its warp's, then all warps'
  float a[4] = {0.0f, 0.0f, 0.0f, 0.0f}, o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const float w = w_s[rg + RG * i], k = k_s[rg + RG * i], q = q_s[rg + RG * i];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      S[i][j] *= w;
      a[j] = fmaf(k, S[i][j], a[j]);
      o[j] = fmaf(q, S[i][j], o[j]);
    }
  }
#pragma unroll
  for (int m = CQ; m < 32; m <<= 1)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      a[j] += __shfl_xor_sync(0xffffffffu, a[j], m);
      o[j] += __shfl_xor_sync(0xffffffffu, o[j], m);
    }
  if (lane < CQ) {
    *reinterpret_cast<float4*>(&part[0][warp][cq * 4]) = make_float4(a[0], a[1], a[2], a[3]);
    *reinterpret_cast<float4*>(&part[1][warp][cq * 4]) = make_float4(o[0], o[1], o[2], o[3]);
  }
  __syncthreads();
  float u[4];
  a[0] = a[1] = a[2] = a[3] = 0.0f;
#pragma unroll
  for (int w = 0; w < NW; ++w) {
    const float4 f = *reinterpret_cast<const float4*>(&part[0][w][cq * 4]);
    a[0] += f.x; a[1] += f.y; a[2] += f.z; a[3] += f.w;
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) u[j] = beta * (v4[j] - a[j]);
  // warp 0 has the CTA's outputs: lane cq's four columns
  float ss = 0.0f;
  if (warp == 0) {
    o[0] = o[1] = o[2] = o[3] = 0.0f;
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      const float4 f = *reinterpret_cast<const float4*>(&part[1][w][cq * 4]);
      o[0] += f.x; o[1] += f.y; o[2] += f.z; o[3] += f.w;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      o[j] = fmaf(kq, u[j], o[j]);
      if (tid < CQ && col + j < dv) ss = fmaf(o[j], o[j], ss);
    }
    ss = nb_warp_sum(ss);
  }
  if (n_splits > 1) {          // the head's sum of squares, over the cluster
    asm volatile("barrier.cluster.wait.aligned;\n" ::: "memory");
    if (warp == 0 && lane < n_splits) {
      const unsigned local = (unsigned)__cvta_generic_to_shared(&square[split]);
      unsigned remote;
      asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(remote) : "r"(local), "r"(lane));
      asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(remote), "f"(ss) : "memory");
    }
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
  }
  nb_launch_dependents();
  // the state, while the squares travel
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = rg + RG * i;
    if (c >= d || col >= dv) continue;
    const float k = k_s[c];
#pragma unroll
    for (int j = 0; j < 4; ++j) S[i][j] = fmaf(k, u[j], S[i][j]);
    if (vec) {
      *reinterpret_cast<float4*>(st + (size_t)c * dv + col) =
          make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < dv) st[(size_t)c * dv + col + j] = S[i][j];
    }
  }
  if (n_splits > 1) {
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
    ss = 0.0f;
    for (int i = 0; i < n_splits; ++i) ss += square[i];
  }
  if (tid < CQ) {
    const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (col + j < dv)
        out[(size_t)r * hv + h * dv + col + j] =
            nb_from_f32<TOut>(o[j] * inv * norm_w[col + j] * nb_sigmoid(gate[j]));
  }
}

template <int CH, int LPG, int NC, int NW>
int launch_walk(cudaStream_t stream, const float* records, const int* cu_rows, const int* seq_slot,
                float* state, int state_stride, float* o_raw, int n_heads, int d, int dv, int vec,
                int n_seqs, bool long_walk) {
  using W = Walk<CH, LPG, NC, NW>;
  auto kern = gated_delta_walk_kernel<CH, LPG, NC, NW>;
  static bool configured = false;   // per instantiation
  if (!configured && W::SMEM > 48 * 1024) {
    NB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, W::SMEM));
    configured = true;
  }
  const dim3 grid((dv + W::COLS - 1) / W::COLS, n_heads, n_seqs);
  // a prompt's walk runs long on few CTAs: it never overlaps its predecessor (nb_launch_serial)
  if (long_walk)
    NB_CUDA(nb_launch_serial(kern, grid, dim3(NW * 32), (size_t)W::SMEM, stream, records, cu_rows,
                             seq_slot, state, state_stride, o_raw, n_heads, d, dv, vec));
  else
    NB_CUDA(nb_launch(kern, grid, dim3(NW * 32), (size_t)W::SMEM, stream, records, cu_rows, seq_slot,
                      state, state_stride, o_raw, n_heads, d, dv, vec));
  NB_CHECK_LAUNCH("gated_delta_walk");
  return 0;
}

int padded_key(int d) { return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256; }

int check_sizes(const char* what, int n_heads, int n_kv_heads, int d, int dv, int n_seqs, int out_dtype) {
  NB_REQUIRE(n_heads >= 1 && n_heads <= 65535 && n_kv_heads >= 1 && n_heads % n_kv_heads == 0 &&
                 n_seqs >= 1 && n_seqs <= 65535,
             NB_ERR_BAD_ARG, "%s: bad sizes heads=%d/%d seqs=%d", what, n_heads, n_kv_heads, n_seqs);
  NB_REQUIRE(d >= 1 && d <= MAX_DIM && dv >= 1 && dv <= MAX_DIM, NB_ERR_UNSUPPORTED,
             "%s: heads of %d / %d channels are outside 1..%d", what, d, dv, MAX_DIM);
  NB_REQUIRE(out_dtype == NB_F32 || out_dtype == NB_BF16, NB_ERR_BAD_ARG, "%s: unknown output dtype %d",
             what, out_dtype);
  return 0;
}

}  // namespace

// Floats of scratch that nb_gated_delta needs for n_rows rows of n_seqs sequences.
NB_EXPORT long long nb_gated_delta_scratch(int n_rows, int n_seqs, int n_heads, int d, int dv) {
  return (long long)(n_rows / BLK + n_seqs + 1) * n_heads * record_floats(padded_key(d), (dv + 3) & ~3);
}

// qkv: fp32 rows, q heads (n_kv_heads * d), k heads, v heads (n_heads * dv) from column qkv_col: with
// taps > 0 projections, which conv ([channels][taps]; inputs: fp32, a slot's last taps - 1 rows of
// channels at inputs + slot * in_stride, brought up to date by nb_conv_state_update afterwards)
// convolves and silu activates, else ready; beta: fp32 rows, head h's logit at column beta_col + h;
// low: fp32 rows with the decay logits (n_heads * d) at decay_col and the gate logits (n_heads * dv)
// at gate_col; a_log [n_heads], dt_bias [n_heads*d], norm_w [dv]; state: a slot's row at state + slot *
// state_stride holds [n_heads][d][dv] (key channel, value channel); records: scratch
// (nb_gated_delta_scratch); o_raw: fp32 scratch [n_rows][n_heads*dv]; out: [n_rows][n_heads*dv].
NB_EXPORT int nb_gated_delta(const float* qkv, int qkv_stride, int qkv_col, const float* conv, int taps,
                             float* inputs, int in_stride, const float* beta, int beta_stride,
                             int beta_col, const float* low, int low_stride, int decay_col,
                             int gate_col, const float* a_log, const float* dt_bias,
                             const float* norm_w, float eps, float key_eps, const int* cu_rows,
                             const int* seq_slot, const int* row_slot, float* state,
                             int state_stride, float* records, float* o_raw, void* out, int out_dtype,
                             int n_heads, int n_kv_heads, int d, int dv, int n_seqs, int max_q_len,
                             int n_rows, cudaStream_t stream) {
  if (n_rows == 0 || n_seqs == 0 || max_q_len == 0) return 0;
  int rc = check_sizes("gated_delta", n_heads, n_kv_heads, d, dv, n_seqs, out_dtype);
  if (rc) return rc;
  NB_REQUIRE((uintptr_t)records % 16 == 0 && taps >= 0 && taps <= MAX_FUSED_TAPS && qkv_col >= 0 &&
                 (taps == 0 || conv != nullptr) && (taps <= 1 || inputs != nullptr),
             NB_ERR_BAD_ARG, "gated_delta: unaligned scratch or bad taps=%d", taps);
  const int channels = 2 * n_kv_heads * d + n_heads * dv;
  const Source src{qkv, qkv_stride, qkv_col, conv, taps, inputs, in_stride, channels, beta, beta_stride,
                   beta_col, low, low_stride, decay_col, gate_col, a_log, dt_bias};
  const bool rows16 = qkv_stride % 4 == 0 && qkv_col % 4 == 0 && ((uintptr_t)qkv | (uintptr_t)conv) % 16 == 0;
  const int vec_in = rows16 && d % 4 == 0 && low_stride % 4 == 0 && decay_col % 4 == 0 && (uintptr_t)low % 16 == 0;
  const int vec_v = rows16 && dv % 4 == 0 && (2 * n_kv_heads * d) % 4 == 0;
  const int vec_st = in_stride % 4 == 0 && channels % 4 == 0 && (uintptr_t)inputs % 16 == 0;
  const int vec = dv % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state | (uintptr_t)o_raw) % 16 == 0;
  const int blocks = (max_q_len + BLK - 1) / BLK;
  const dim3 grid((blocks + 1) / 2, n_heads, n_seqs);
  const bool long_walk = n_rows > 4 * n_seqs;
#define NB_PREP(DP_, CONV_)                                                                       \
  NB_CUDA(nb_launch(gated_delta_prepare_kernel<DP_, CONV_>, grid, dim3(128), 0, stream, src,      \
                    key_eps, cu_rows, seq_slot, records, n_heads, n_kv_heads, d, dv, vec_st,      \
                    vec_in, vec_v))
#define NB_WALK(CH, LPG, NC, NW)                                                                  \
  rc = launch_walk<CH, LPG, NC, NW>(stream, records, cu_rows, seq_slot, state, state_stride, o_raw, \
                                    n_heads, d, dv, vec, n_seqs, long_walk)
#define NB_GD(DP_)                                                                                \
  do {                                                                                            \
    if (taps == 0) NB_PREP(DP_, 0);                                                               \
    else if (out_dtype == NB_F32) NB_PREP(DP_, 1);                                                \
    else NB_PREP(DP_, 2);                                                                         \
    NB_CHECK_LAUNCH("gated_delta_prepare");                                                       \
  } while (0)
  // As measured on prompts of 2 x 1,024 tokens: two columns a lane (a block's time is one warp's
  // instructions), four for heads of up to 64 where there are enough of them to fill the schedulers.
  const bool few = (long long)n_heads * n_seqs * ((dv + 31) / 32) <= 148;
  if (d <= 32) {
    NB_GD(32);
    NB_WALK(4, 8, 2, 4);
  } else if (d <= 64) {
    NB_GD(64);
    if (few) NB_WALK(4, 16, 2, 4);
    else NB_WALK(4, 16, 4, 4);
  } else if (d <= 128) {
    NB_GD(128);
    NB_WALK(8, 16, 2, 8);
  } else {
    NB_GD(256);
    NB_WALK(16, 16, 2, 8);
  }
#undef NB_GD
#undef NB_WALK
#undef NB_PREP
  if (rc) return rc;
  return launch_delta_finish(o_raw, low, low_stride, gate_col, norm_w, 0, eps, row_slot, out, out_dtype,
                             n_heads, dv, n_rows, stream);
}

// The same for a step of one token per sequence (row cu_rows[s] of sequence s), its rows ready (qkv from
// column 0).
NB_EXPORT int nb_gated_delta_step(const float* qkv, int qkv_stride, const float* beta, int beta_stride,
                                  int beta_col, const float* low, int low_stride, int decay_col,
                                  int gate_col, const float* a_log, const float* dt_bias,
                                  const float* norm_w, float eps, float key_eps, const int* cu_rows,
                                  const int* seq_slot, float* state, int state_stride, void* out,
                                  int out_dtype, int n_heads, int n_kv_heads, int d, int dv,
                                  int n_seqs, cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  const int rc = check_sizes("gated_delta_step", n_heads, n_kv_heads, d, dv, n_seqs, out_dtype);
  if (rc) return rc;
  const Source src{qkv, qkv_stride, 0, nullptr, 0, nullptr, 0, 2 * n_kv_heads * d + n_heads * dv, beta,
                   beta_stride, beta_col, low, low_stride, decay_col, gate_col, a_log, dt_bias};
  const int vec = dv % 4 == 0 && state_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  // a CTA per 128 columns where that fills the GPU (and the state of a head fits its registers);
  // measured at 64 sequences of 16 heads of 128: 48 us with the convolution, 66 with 32 columns a CTA
  const bool wide = d <= 128 && dv > 32 && (long long)n_heads * n_seqs * ((dv + 127) / 128) >= 2 * 148;
  const int cols = wide ? 128 : 32, splits = (dv + cols - 1) / cols;
  const dim3 grid(splits, n_heads, n_seqs);
#define NB_GS(NV, COLS, TO)                                                                       \
  NB_CUDA(nb_launch_clusters(gated_delta_step_kernel<NV, COLS, TO>, grid, dim3(ST_THREADS), 0,    \
                             stream, splits, src, key_eps, norm_w, eps, cu_rows, seq_slot, state, \
                             state_stride, (TO*)out, n_heads, n_kv_heads, d, dv, vec))
#define NB_GS_T(NV, COLS)                                                                         \
  do {                                                                                            \
    if (out_dtype == NB_F32) NB_GS(NV, COLS, float);                                              \
    else NB_GS(NV, COLS, __nv_bfloat16);                                                          \
  } while (0)
  if (wide) {
    if (d <= 32) NB_GS_T(4, 128);
    else if (d <= 64) NB_GS_T(8, 128);
    else NB_GS_T(16, 128);
  } else if (d <= 32) NB_GS_T(1, 32);
  else if (d <= 64) NB_GS_T(2, 32);
  else if (d <= 128) NB_GS_T(4, 32);
  else NB_GS_T(8, 32);
#undef NB_GS_T
#undef NB_GS
  NB_CHECK_LAUNCH("gated_delta_step");
  return 0;
}

// The longest convolution that nb_gated_delta takes in (a longer one runs before it).
NB_EXPORT int nb_gated_delta_max_taps() { return MAX_FUSED_TAPS; }
