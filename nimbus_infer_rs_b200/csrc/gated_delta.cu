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
// Prompts.  Four tokens are taken at a time.  With E_(s..t) = the product of g over tokens s+1 .. t
// of the block (per key channel; from the block's start: E_t) and S the state at its start,
//
//   u_t = beta_t v_t - (beta_t E_t k_t)^T S - sum_(s<t) A_ts u_s,   A_ts = beta_t sum_i k_ti k_si E_(s..t)i
//   o_t = (E_t q_t)^T S + sum_(s<=t) B_ts u_s,                     B_ts = sum_i q_ti k_si E_(s..t)i
//   S  <- diag(E_3) S + sum_s (k_s E_(s..3)) u_s^T
//
// so the state is read twice and written once per four tokens, the eight dot products of a column
// with it are independent of one another, and only the four u_t (a few multiply-adds) follow one
// another.  Decays are multiplied up, never divided by, so nothing overflows however strong they are.
//   gated_delta_prepare  a warp per (block of four tokens, head) computes a record: E_3, the four
//                        (beta_t E_t k_t), (E_t q_t), (k_s E_(s..3)), the numbers A and B, and the
//                        four beta_t v_t.  A block's missing tokens (a sequence's last block) are
//                        tokens with k = q = v = 0, g = 1.
//   gated_delta_walk     a CTA takes COLS columns of one (sequence, head); the columns are
//                        independent.  A group of LPG lanes holds four columns, CH key channels a
//                        lane, so a number of the record that was read from shared memory meets
//                        four columns.  The 32 partial sums of a block (four tokens, four columns,
//                        two products) are reduced over the lanes by halving: each lane ends with
//                        32 / LPG of them.  Records come through two buffers of asynchronous copies.
//   delta_finish         norm, weight and gate (the norm needs all of a head's columns).
// A sequence may be cut into steps anywhere: where blocks begin only changes the rounding.
//
// One-token steps.  gated_delta_step: a CTA per (sequence, head, 32 columns), the CTAs of a head in a
// thread-block cluster that adds up the head's sum of squares through shared memory; the state is
// fetched before the wait on the kernel in front (which never writes it), read and written once.
#include "delta_common.cuh"
#include "attention_common.cuh"

namespace {

constexpr int BLK = 4;         // tokens of a block
constexpr int MAX_DIM = 256;

__device__ __forceinline__ float gd_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// Sums of N values over L lanes by halving: afterwards the lane with number q in its group of L
// holds the sums with indices q * (N / L) .. in v[0 ..] (N >= L), or, when N < L, index q / (L / N).
template <int N, int L>
__device__ __forceinline__ void reduce_by_halving(float (&v)[N], int lane) {
  int n = N;
#pragma unroll
  for (int m = L / 2; m >= 1; m >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = (lane & m) != 0;
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        if (i < n) {
          const float send = up ? v[i] : v[i + n];
          const float keep = up ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], m);
    }
  }
}

struct Source {               // where a row's numbers lie
  const float* qkv;           // [rows][qkv_stride]: q heads, k heads, v heads (convolved, activated)
  int qkv_stride;
  const float* beta;          // [rows][beta_stride], head h's logit at column beta_col + h
  int beta_stride, beta_col;
  const float* low;           // [rows][low_stride]: decay logits at decay_col, gate logits at gate_col
  int low_stride, decay_col, gate_col;
  const float* a_log;         // [heads]
  const float* dt_bias;       // [heads * d]
};

// floats of a record of padded key size DP; dvp: the value size rounded up to a multiple of 4
__host__ __device__ constexpr int record_head(int DP) { return 13 * DP + 32; }
__host__ __device__ inline int record_floats(int DP, int dvp) { return record_head(DP) + BLK * dvp; }

// A sequence's blocks start at record cu_rows[seq] / 4 + seq, so that no two sequences overlap.
template <int DP>
__global__ void __launch_bounds__(128)
gated_delta_prepare_kernel(Source src, float key_eps, const int* cu_rows, const int* seq_slot,
                           float* records, int n_heads, int n_kv_heads, int d, int dv, int vec) {
  nb_grid_dependency_wait();
  nb_launch_dependents();
  constexpr int KIT = (DP + 127) / 128;             // quads of channels a lane holds
  const int seq = blockIdx.z, h = blockIdx.y, lane = threadIdx.x & 31;
  const int blk = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int row0 = cu_rows[seq], row1 = cu_rows[seq + 1];
  const int first = row0 + blk * BLK;
  if (seq_slot[seq] < 0 || first >= row1) return;
  const int g = h / (n_heads / n_kv_heads);
  const int dvp = (dv + 3) & ~3;
  float* rec = records + ((size_t)(row0 / BLK + seq + blk) * n_heads + h) * record_floats(DP, dvp);
  const float rate = expf(src.a_log[h]);
  const float q_scale = 1.0f / sqrtf((float)d);

  float k[BLK][KIT * 4], q[BLK][KIT * 4], w[BLK][KIT * 4], beta[BLK];
  auto load4 = [&](const float* p, int c, float (&v)[KIT * 4], int at) {
    if (vec && c < d) {
      const float4 f = *reinterpret_cast<const float4*>(p + c);
      v[at] = f.x; v[at + 1] = f.y; v[at + 2] = f.z; v[at + 3] = f.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) v[at + e] = c + e < d ? p[c + e] : 0.0f;
    }
  };
#pragma unroll
  for (int t = 0; t < BLK; ++t) {
    const int r = first + t;
    const bool live = r < row1;
    const float* row = src.qkv + (size_t)(live ? r : row0) * src.qkv_stride;
    const float* dl = src.low + (size_t)(live ? r : row0) * src.low_stride + src.decay_col + h * d;
#pragma unroll
    for (int j = 0; j < KIT; ++j) {
      const int c = (j * 32 + lane) * 4;
      load4(row + g * d, c, q[t], j * 4);
      load4(row + (n_kv_heads + g) * d, c, k[t], j * 4);
      load4(dl, c, w[t], j * 4);
    }
    beta[t] = live ? nb_sigmoid(src.beta[(size_t)r * src.beta_stride + src.beta_col + h]) : 0.0f;
  }
  // unit vectors and decays
  float ss[2 * BLK];
#pragma unroll
  for (int t = 0; t < BLK; ++t) {
    ss[t] = ss[BLK + t] = 0.0f;
#pragma unroll
    for (int i = 0; i < KIT * 4; ++i) {
      ss[t] = fmaf(k[t][i], k[t][i], ss[t]);
      ss[BLK + t] = fmaf(q[t][i], q[t][i], ss[BLK + t]);
    }
  }
#pragma unroll
  for (int i = 0; i < 2 * BLK; ++i) ss[i] = nb_warp_sum(ss[i]);
#pragma unroll
  for (int t = 0; t < BLK; ++t) {
    const bool live = first + t < row1;
    const float ik = live ? 1.0f / sqrtf(ss[t] + key_eps) : 0.0f;
    const float iq = live ? q_scale / sqrtf(ss[BLK + t] + key_eps) : 0.0f;
#pragma unroll
    for (int i = 0; i < KIT * 4; ++i) {
      const int c = ((i >> 2) * 32 + lane) * 4 + (i & 3);
      k[t][i] *= ik;
      q[t][i] *= iq;
      w[t][i] = (live && c < d) ? expf(-rate * gd_softplus(w[t][i] + src.dt_bias[h * d + c])) : 1.0f;
    }
  }
  auto store = [&](int place, const float (&v)[KIT * 4]) {
#pragma unroll
    for (int j = 0; j < KIT; ++j) {
      const int c = (j * 32 + lane) * 4;
      if (c < DP)
        *reinterpret_cast<float4*>(rec + place * DP + c) =
            make_float4(v[j * 4], v[j * 4 + 1], v[j * 4 + 2], v[j * 4 + 3]);
    }
  };
  // the numbers A (six of them) and B (ten), and k_s E_(s..3)
  float ab[16];
#pragma unroll
  for (int s = 0; s < BLK; ++s) {
    float kd[KIT * 4];
#pragma unroll
    for (int i = 0; i < KIT * 4; ++i) kd[i] = k[s][i];
#pragma unroll
    for (int t = s; t < BLK; ++t) {
      float a = 0.0f, b = 0.0f;
#pragma unroll
      for (int i = 0; i < KIT * 4; ++i) {
        if (t > s) kd[i] *= w[t][i];
        a = fmaf(k[t][i], kd[i], a);
        b = fmaf(q[t][i], kd[i], b);
      }
      if (t > s) ab[t * (t - 1) / 2 + s] = a;
      ab[6 + t * (t + 1) / 2 + s] = b;
    }
    store(9 + s, kd);
  }
  reduce_by_halving<16, 32>(ab, lane);           // lane l holds number l / 2
  {
    const int t = (lane & 15) >> 2, s = lane & 3;   // slot `lane`: A (0..15), B (16..31), row t, column s
    const bool is_b = lane >= 16, there = is_b ? s <= t : s < t;
    const int idx = is_b ? 6 + t * (t + 1) / 2 + s : t * (t - 1) / 2 + s;
    float v = __shfl_sync(0xffffffffu, ab[0], there ? 2 * idx : 0);
    const float bt = t == 0 ? beta[0] : t == 1 ? beta[1] : t == 2 ? beta[2] : beta[3];
    rec[13 * DP + lane] = there ? (is_b ? v : v * bt) : 0.0f;
  }
  // beta_t E_t k_t, E_t q_t, E_3
#pragma unroll
  for (int t = 0; t < BLK; ++t) {
    float kt[KIT * 4], qt[KIT * 4];
#pragma unroll
    for (int i = 0; i < KIT * 4; ++i) {
      if (t > 0) w[t][i] *= w[t - 1][i];
      kt[i] = beta[t] * k[t][i] * w[t][i];
      qt[i] = q[t][i] * w[t][i];
    }
    store(1 + t, kt);
    store(5 + t, qt);
  }
  store(0, w[BLK - 1]);
  // beta_t v_t
  float* vd = rec + record_head(DP);
#pragma unroll
  for (int t = 0; t < BLK; ++t) {
    const int r = first + t;
    const float* v = src.qkv + (size_t)(r < row1 ? r : row0) * src.qkv_stride + 2 * n_kv_heads * d + h * dv;
    for (int c = lane; c < dvp; c += 32)
      vd[t * dvp + c] = (r < row1 && c < dv) ? beta[t] * v[c] : 0.0f;
  }
}

// CH: key channels a lane holds for each of its four columns; LPG: lanes of a group; NW: warps.
template <int CH, int LPG, int NW>
struct Walk {
  static constexpr int DP = CH * LPG;
  static constexpr int GROUPS = NW * (32 / LPG);
  static constexpr int COLS = 4 * GROUPS;
  static constexpr int SB = DP > 128 ? 2 : 4;                    // blocks a buffer holds
  static constexpr int BUF = SB * (record_head(DP) + BLK * COLS);  // floats of a buffer
  static constexpr int SMEM = (2 * BUF + 2 * GROUPS * 32) * 4;
};

template <int CH, int LPG, int NW>
__global__ void __launch_bounds__(NW * 32)
gated_delta_walk_kernel(const float* records, const int* cu_rows, const int* seq_slot, float* state,
                        int state_stride, float* o_raw, int n_heads, int d, int dv, int vec) {
  using W = Walk<CH, LPG, NW>;
  constexpr int DP = W::DP, COLS = W::COLS, SB = W::SB, THREADS = NW * 32, HEAD = record_head(DP);
  static_assert(CH % 4 == 0, "a lane takes its channels four at a time");
  nb_grid_dependency_wait();
  extern __shared__ __align__(16) float sm[];
  float* red = sm + 2 * W::BUF;                     // [2][groups][32]
  const int col0 = blockIdx.x * COLS, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int row0 = cu_rows[seq], row1 = cu_rows[seq + 1];
  const int slot = seq_slot[seq];
  if (slot < 0 || row1 <= row0) return;
  const int lane = tid & 31, group = tid / LPG, q = tid % LPG;
  const int col = col0 + group * 4;                 // this group's four columns
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

  // key channel of state number i of this lane: groups of four, dealt out to the lanes in turn
  auto channel = [q](int i) { return (((i >> 2) * LPG + q) << 2) + (i & 3); };
  float S[CH][4];
#pragma unroll
  for (int i = 0; i < CH; ++i) {
    const int c = channel(i);
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.0f;
    if (c >= d || col >= dv) continue;
    if (vec) {
      const float4 f = *reinterpret_cast<const float4*>(st + (size_t)c * dv + col);
      S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < dv) S[i][j] = st[(size_t)c * dv + col + j];
    }
  }

  int parity = 0;
  for (int b0 = 0, buf = 0; b0 < n_blocks; b0 += SB, buf ^= 1) {
    cp_async_wait<0>();
    __syncthreads();                 // the buffer is in, and every thread has left the other one
    if (b0 + SB < n_blocks) fetch(b0 + SB, buf ^ 1);
    const float* head = sm + buf * W::BUF;
    const float* vals = head + SB * HEAD + group * 4;
    const int nb = min(SB, n_blocks - b0);
    for (int b = 0; b < nb; ++b, head += HEAD, vals += BLK * COLS) {
      // r[t][c] = (beta E k)_t . S_c at 4 t + c,  (E q)_t . S_c at 16 + 4 t + c
      float p[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) p[i] = 0.0f;
#pragma unroll
      for (int g = 0; g < CH / 4; ++g) {
#pragma unroll
        for (int t = 0; t < BLK; ++t) {
          const float4 kk = *reinterpret_cast<const float4*>(head + (1 + t) * DP + (g * LPG + q) * 4);
          const float4 qq = *reinterpret_cast<const float4*>(head + (5 + t) * DP + (g * LPG + q) * 4);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            p[4 * t + c] = fmaf(kk.x, S[4 * g][c], p[4 * t + c]);
            p[4 * t + c] = fmaf(kk.y, S[4 * g + 1][c], p[4 * t + c]);
            p[4 * t + c] = fmaf(kk.z, S[4 * g + 2][c], p[4 * t + c]);
            p[4 * t + c] = fmaf(kk.w, S[4 * g + 3][c], p[4 * t + c]);
            p[16 + 4 * t + c] = fmaf(qq.x, S[4 * g][c], p[16 + 4 * t + c]);
            p[16 + 4 * t + c] = fmaf(qq.y, S[4 * g + 1][c], p[16 + 4 * t + c]);
            p[16 + 4 * t + c] = fmaf(qq.z, S[4 * g + 2][c], p[16 + 4 * t + c]);
            p[16 + 4 * t + c] = fmaf(qq.w, S[4 * g + 3][c], p[16 + 4 * t + c]);
          }
        }
      }
      reduce_by_halving<32, LPG>(p, lane);
      float* mine = red + (parity * W::GROUPS + group) * 32;
      parity ^= 1;
#pragma unroll
      for (int i = 0; i < 32 / LPG; ++i) mine[q * (32 / LPG) + i] = p[i];
      __syncwarp();
      // the four u, then the state
      float u[BLK][4];
#pragma unroll
      for (int t = 0; t < BLK; ++t) {
        const float4 rr = *reinterpret_cast<const float4*>(mine + 4 * t);
        const float4 vv = *reinterpret_cast<const float4*>(vals + t * COLS);
        u[t][0] = vv.x - rr.x; u[t][1] = vv.y - rr.y; u[t][2] = vv.z - rr.z; u[t][3] = vv.w - rr.w;
        if (t == 0) continue;
        const float4 a = *reinterpret_cast<const float4*>(head + 13 * DP + 4 * t);
        const float at[3] = {a.x, a.y, a.z};
#pragma unroll
        for (int s = 0; s < t; ++s)
#pragma unroll
          for (int c = 0; c < 4; ++c) u[t][c] = fmaf(-at[s], u[s][c], u[t][c]);
      }
#pragma unroll
      for (int g = 0; g < CH / 4; ++g) {
        const float4 w = *reinterpret_cast<const float4*>(head + (g * LPG + q) * 4);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          S[4 * g][c] *= w.x;
          S[4 * g + 1][c] *= w.y;
          S[4 * g + 2][c] *= w.z;
          S[4 * g + 3][c] *= w.w;
        }
#pragma unroll
        for (int s = 0; s < BLK; ++s) {
          const float4 kk = *reinterpret_cast<const float4*>(head + (9 + s) * DP + (g * LPG + q) * 4);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            S[4 * g][c] = fmaf(kk.x, u[s][c], S[4 * g][c]);
            S[4 * g + 1][c] = fmaf(kk.y, u[s][c], S[4 * g + 1][c]);
            S[4 * g + 2][c] = fmaf(kk.z, u[s][c], S[4 * g + 2][c]);
            S[4 * g + 3][c] = fmaf(kk.w, u[s][c], S[4 * g + 3][c]);
          }
        }
      }
      // a token's four outputs: lane t of the group has token t
      if (q < BLK) {
        const float4 oo = *reinterpret_cast<const float4*>(mine + 16 + 4 * q);
        const float4 bb = *reinterpret_cast<const float4*>(head + 13 * DP + 16 + 4 * q);
        float o[4] = {oo.x, oo.y, oo.z, oo.w};
        const float bt[4] = {bb.x, bb.y, bb.z, bb.w};
#pragma unroll
        for (int s = 0; s < BLK; ++s)
#pragma unroll
          for (int c = 0; c < 4; ++c) o[c] = fmaf(bt[s], u[s][c], o[c]);
        const int r = row0 + (b0 + b) * BLK + q;
        if (r < row1) {
          float* dst = o_raw + ((size_t)r * n_heads + h) * dv + col;
          if (vec && col < dv) {
            *reinterpret_cast<float4*>(dst) = make_float4(o[0], o[1], o[2], o[3]);
          } else {
#pragma unroll
            for (int c = 0; c < 4; ++c)
              if (col + c < dv) dst[c] = o[c];
          }
        }
      }
    }
  }
  nb_launch_dependents();
#pragma unroll
  for (int i = 0; i < CH; ++i) {
    const int c = channel(i);
    if (c >= d || col >= dv) continue;
    if (vec) {
      *reinterpret_cast<float4*>(st + (size_t)c * dv + col) =
          make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < dv) st[(size_t)c * dv + col + j] = S[i][j];
    }
  }
}

// One token per sequence.  Thread: four neighbouring columns (cq) of the key channels rg, rg + 32, ...
constexpr int ST_THREADS = 256, ST_COLS = 32;

template <int NV, typename TOut>
__global__ void __launch_bounds__(ST_THREADS)
gated_delta_step_kernel(Source src, float key_eps, const float* __restrict__ norm_w, float eps,
                        const int* cu_rows, const int* seq_slot, float* state, int state_stride,
                        TOut* out, int n_heads, int n_kv_heads, int d, int dv, int vec) {
  __shared__ float k_s[NV * 32], q_s[NV * 32], w_s[NV * 32];
  __shared__ __align__(16) float part[ST_THREADS / 32][ST_COLS];
  __shared__ float red[2][8], square[8];
  const int split = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int lane = tid & 31, warp = tid >> 5;
  const int n_splits = gridDim.x;
  const int r = cu_rows[seq], slot = cu_rows[seq + 1] > r ? seq_slot[seq] : -1;
  const int hv = n_heads * dv;
  if (slot < 0) {              // the whole cluster leaves
    nb_grid_dependency_wait();
    nb_launch_dependents();
    const int c = split * ST_COLS + tid;
    if (cu_rows[seq + 1] > r && tid < ST_COLS && c < dv)
      out[(size_t)r * hv + h * dv + c] = nb_from_f32<TOut>(0.0f);
    return;
  }
  const int cq = tid & 7, rg = tid >> 3, col = split * ST_COLS + cq * 4;
  const int g = h / (n_heads / n_kv_heads);
  float* st = state + (size_t)slot * state_stride + (size_t)h * d * dv;
  float S[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = rg + 32 * i;
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
  asm volatile("barrier.cluster.arrive.relaxed.aligned;\n" ::: "memory");

  const float* row = src.qkv + (size_t)r * src.qkv_stride;
  float v4[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) v4[j] = col + j < dv ? row[2 * n_kv_heads * d + h * dv + col + j] : 0.0f;
  const float beta = nb_sigmoid(src.beta[(size_t)r * src.beta_stride + src.beta_col + h]);
  const float gate = (tid < ST_COLS && split * ST_COLS + tid < dv)
                         ? src.low[(size_t)r * src.low_stride + src.gate_col + h * dv + split * ST_COLS + tid]
                         : 0.0f;
  float kx = 0.0f, qx = 0.0f, wx = 0.0f;
  if (tid < d) {
    kx = row[(n_kv_heads + g) * d + tid];
    qx = row[g * d + tid];
    wx = expf(-expf(src.a_log[h]) *
              gd_softplus(src.low[(size_t)r * src.low_stride + src.decay_col + h * d + tid] +
                          src.dt_bias[h * d + tid]));
  }
  const float sk = nb_warp_sum(kx * kx), sq = nb_warp_sum(qx * qx);
  if (lane == 0) {
    red[0][warp] = sk;
    red[1][warp] = sq;
  }
  __syncthreads();
  float tk = 0.0f, tq = 0.0f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    tk += red[0][i];
    tq += red[1][i];
  }
  if (tid < NV * 32) {
    k_s[tid] = kx / sqrtf(tk + key_eps);
    q_s[tid] = qx / sqrtf(tq + key_eps) * (1.0f / sqrtf((float)d));
    w_s[tid] = wx;
  }
  __syncthreads();
  // sums over the key channels of four columns: the thread's, its warp's, then all warps'
  auto total = [&](float (&a)[4]) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      a[j] += __shfl_xor_sync(0xffffffffu, a[j], 8);
      a[j] += __shfl_xor_sync(0xffffffffu, a[j], 16);
    }
    if (lane < 8) *reinterpret_cast<float4*>(&part[warp][cq * 4]) = make_float4(a[0], a[1], a[2], a[3]);
    __syncthreads();
    a[0] = a[1] = a[2] = a[3] = 0.0f;
#pragma unroll
    for (int w = 0; w < ST_THREADS / 32; ++w) {
      const float4 f = *reinterpret_cast<const float4*>(&part[w][cq * 4]);
      a[0] += f.x; a[1] += f.y; a[2] += f.z; a[3] += f.w;
    }
  };
  float a[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const float w = w_s[rg + 32 * i], k = k_s[rg + 32 * i];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      S[i][j] *= w;
      a[j] = fmaf(k, S[i][j], a[j]);
    }
  }
  total(a);
  float u[4], o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int j = 0; j < 4; ++j) u[j] = beta * (v4[j] - a[j]);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const float k = k_s[rg + 32 * i], q = q_s[rg + 32 * i];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      S[i][j] = fmaf(k, u[j], S[i][j]);
      o[j] = fmaf(q, S[i][j], o[j]);
    }
    const int c = rg + 32 * i;
    if (c < d && col < dv) {
      if (vec) {
        *reinterpret_cast<float4*>(st + (size_t)c * dv + col) =
            make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (col + j < dv) st[(size_t)c * dv + col + j] = S[i][j];
      }
    }
  }
  nb_launch_dependents();
  __syncthreads();             // `part` is used again
  total(o);
  asm volatile("barrier.cluster.wait.aligned;\n" ::: "memory");
  // the head's sum of squares: warp 0 has this CTA's columns, the cluster the rest
  float mine = 0.0f;
  if (warp == 0) {
    // lane l takes column l: it sits in lane l / 4 (cq), number l % 4
    const float x0 = __shfl_sync(0xffffffffu, o[0], lane >> 2), x1 = __shfl_sync(0xffffffffu, o[1], lane >> 2);
    const float x2 = __shfl_sync(0xffffffffu, o[2], lane >> 2), x3 = __shfl_sync(0xffffffffu, o[3], lane >> 2);
    const int j = lane & 3;
    mine = j == 0 ? x0 : j == 1 ? x1 : j == 2 ? x2 : x3;
    if (split * ST_COLS + lane >= dv) mine = 0.0f;
    const float ss = nb_warp_sum(mine * mine);
    if (lane < n_splits) {
      const unsigned local = (unsigned)__cvta_generic_to_shared(&square[split]);
      unsigned remote;
      asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(remote) : "r"(local), "r"(lane));
      asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(remote), "f"(ss) : "memory");
    }
  }
  asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
  if (warp == 0 && split * ST_COLS + lane < dv) {
    float ss = 0.0f;
    for (int i = 0; i < n_splits; ++i) ss += square[i];
    const int c = split * ST_COLS + lane;
    out[(size_t)r * hv + h * dv + c] = nb_from_f32<TOut>(
        mine * (1.0f / sqrtf(ss / (float)dv + eps)) * norm_w[c] * nb_sigmoid(gate));
  }
}

template <int CH, int LPG, int NW>
int launch_walk(cudaStream_t stream, const float* records, const int* cu_rows, const int* seq_slot,
                float* state, int state_stride, float* o_raw, int n_heads, int d, int dv, int vec,
                int n_seqs, bool long_walk) {
  using W = Walk<CH, LPG, NW>;
  auto kern = gated_delta_walk_kernel<CH, LPG, NW>;
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

// qkv: fp32 [rows][qkv_stride], q heads (n_kv_heads * d), k heads, v heads (n_heads * dv), convolved
// and activated; beta: fp32 rows, head h's logit at column beta_col + h; low: fp32 rows with the
// decay logits (n_heads * d) at decay_col and the gate logits (n_heads * dv) at gate_col; a_log
// [n_heads], dt_bias [n_heads*d], norm_w [dv]; state: a slot's row at state + slot * state_stride
// holds [n_heads][d][dv] (key channel, value channel); records: scratch (nb_gated_delta_scratch);
// o_raw: fp32 scratch [n_rows][n_heads*dv]; out: [n_rows][n_heads*dv].
NB_EXPORT int nb_gated_delta(const float* qkv, int qkv_stride, const float* beta, int beta_stride,
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
  NB_REQUIRE((uintptr_t)records % 16 == 0, NB_ERR_BAD_ARG, "gated_delta: unaligned scratch");
  const Source src{qkv, qkv_stride, beta, beta_stride, beta_col, low, low_stride, decay_col, gate_col,
                   a_log, dt_bias};
  const int vec_in = d % 4 == 0 && qkv_stride % 4 == 0 && low_stride % 4 == 0 && decay_col % 4 == 0 &&
                     ((uintptr_t)qkv | (uintptr_t)low) % 16 == 0;
  const int vec = dv % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state | (uintptr_t)o_raw) % 16 == 0;
  const int blocks = (max_q_len + BLK - 1) / BLK;
  const dim3 grid((blocks + 3) / 4, n_heads, n_seqs);
  const bool long_walk = n_rows > 4 * n_seqs;
  const int few = n_heads * n_seqs * ((dv + 31) / 32) < 148;     // fewer columns a CTA fill the GPU
#define NB_GD(CH, LPG, NW)                                                                        \
  do {                                                                                            \
    NB_CUDA(nb_launch(gated_delta_prepare_kernel<CH * LPG>, grid, dim3(128), 0, stream, src,      \
                      key_eps, cu_rows, seq_slot, records, n_heads, n_kv_heads, d, dv, vec_in));  \
    NB_CHECK_LAUNCH("gated_delta_prepare");                                                       \
    rc = few ? launch_walk<CH, LPG, (NW + 1) / 2>(stream, records, cu_rows, seq_slot, state,      \
                                                  state_stride, o_raw, n_heads, d, dv, vec,       \
                                                  n_seqs, long_walk)                              \
             : launch_walk<CH, LPG, NW>(stream, records, cu_rows, seq_slot, state, state_stride,  \
                                        o_raw, n_heads, d, dv, vec, n_seqs, long_walk);           \
  } while (0)
  if (d <= 32) NB_GD(4, 8, 2);
  else if (d <= 64) NB_GD(4, 16, 4);
  else if (d <= 128) NB_GD(4, 32, 8);
  else NB_GD(8, 32, 8);
#undef NB_GD
  if (rc) return rc;
  return launch_delta_finish(o_raw, low, low_stride, gate_col, norm_w, 0, eps, row_slot, out, out_dtype,
                             n_heads, dv, n_rows, stream);
}

// The same for a step of one token per sequence (row cu_rows[s] of sequence s).
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
  const Source src{qkv, qkv_stride, beta, beta_stride, beta_col, low, low_stride, decay_col, gate_col,
                   a_log, dt_bias};
  const int vec = dv % 4 == 0 && state_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  const int splits = (dv + ST_COLS - 1) / ST_COLS;
  const dim3 grid(splits, n_heads, n_seqs);
#define NB_GS(NV, TO)                                                                             \
  NB_CUDA(nb_launch_clusters(gated_delta_step_kernel<NV, TO>, grid, dim3(ST_THREADS), 0, stream,  \
                             splits, src, key_eps, norm_w, eps, cu_rows, seq_slot, state,         \
                             state_stride, (TO*)out, n_heads, n_kv_heads, d, dv, vec))
#define NB_GS_T(NV)                                                                               \
  do {                                                                                            \
    if (out_dtype == NB_F32) NB_GS(NV, float);                                                    \
    else NB_GS(NV, __nv_bfloat16);                                                                \
  } while (0)
  if (d <= 32) NB_GS_T(1);
  else if (d <= 64) NB_GS_T(2);
  else if (d <= 128) NB_GS_T(4);
  else NB_GS_T(8);
#undef NB_GS_T
#undef NB_GS
  NB_CHECK_LAUNCH("gated_delta_step");
  return 0;
}
