// Differential attention: a head has two query maps and two key maps over ONE set of values.  Each
// map is a softmax attention of its own over what the row sees,
//
//   s_a(j) = scale * q_a . k_a(j),   A_a = sum_j softmax_j(s_a) v(j),   a = 1, 2
//   o = A_1 - lambda A_2,            o <- o / sqrt(mean(o^2) + eps) * factor     (over the head)
//
// with lambda, factor and eps constants of the layer.  Position i sees j <= i (window <= 0), or
// of those only i - j < window.
//
// Layouts: a query row holds head after head [map 1 | map 2] (2 d numbers a head); the key plane
// [page][kv_head][64][2 d] holds a key head's two maps side by side, the value plane
// [page][kv_head][64][dv] its values.  Both planes may belong to one paged store (dv = 2 d) or to
// two with block tables of their own.  Query head h reads key/value head h / group.
//
// Kernels here: fp32 on the CUDA cores, any sizes (the 32-bit path, and what the others leave), and
// bf16 on the tensor cores through mma.sync (sizes that are multiples of 8; tiles of 64 rows).
#include "attention_common.cuh"
#include "mma_common.cuh"

namespace {

typedef __nv_bfloat16 bf16;

constexpr int AD_THREADS = 128;
constexpr int AD_WARPS = AD_THREADS / 32;
constexpr int AD_CHUNK = 512;     // keys whose scores (of both maps) are in shared memory at a time
constexpr int AD_MAXD = 256;
constexpr int AD_DPL = AD_MAXD / 32;

// A CTA per (row, head): warps over keys, lanes over the head's numbers; every row is reduced in
// the same order whatever the step's cut or the batch.
template <typename TQ, typename TC, typename TOut>
__global__ void __launch_bounds__(AD_THREADS)
attention_differential_kernel(const TQ* q, const int* row_slot, const int* row_pos, const TC* kc,
                              const int* k_table, int k_max_pages, const TC* vc, const int* v_table,
                              int v_max_pages, int page, int n_heads, int n_kv_heads, int d, int dv,
                              TOut* out, float scale, int window, float lambda, float factor,
                              float eps) {
  nb_grid_dependency_wait();
  nb_launch_dependents();
  __shared__ float scores[2][AD_CHUNK];
  __shared__ float q_s[2 * AD_MAXD];
  __shared__ float part[AD_WARPS][2][AD_MAXD];
  __shared__ float red[32];
  const int r = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  TOut* o = out + ((size_t)r * n_heads + h) * dv;
  const int slot = row_slot[r];
  if (slot < 0) {
    for (int i = tid; i < dv; i += AD_THREADS) o[i] = nb_from_f32<TOut>(0.0f);
    return;
  }
  const int pos = row_pos[r];
  const int g = h / (n_heads / n_kv_heads);
  const int* kt = k_table + (size_t)slot * k_max_pages;
  const int* vt = v_table + (size_t)slot * v_max_pages;
  const TQ* qr = q + ((size_t)r * n_heads + h) * 2 * d;
  for (int i = tid; i < 2 * d; i += AD_THREADS) q_s[i] = nb_to_f32(qr[i]);
  __syncthreads();
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
  float acc[2][AD_DPL];
#pragma unroll
  for (int a = 0; a < AD_DPL; ++a) acc[0][a] = acc[1][a] = 0.0f;

  for (int c0 = lo; c0 <= pos; c0 += AD_CHUNK) {
    const int c1 = min(c0 + AD_CHUNK, pos + 1);
    float cmax[2] = {-INFINITY, -INFINITY};
    for (int j = c0 + warp; j < c1; j += AD_WARPS) {
      const TC* kr = kc + (((size_t)kt[j / page] * n_kv_heads + g) * page + (j % page)) * 2 * d;
      float d0 = 0.0f, d1 = 0.0f;
      for (int i = lane; i < d; i += 32) {
        d0 = fmaf(q_s[i], nb_to_f32(kr[i]), d0);
        d1 = fmaf(q_s[d + i], nb_to_f32(kr[d + i]), d1);
      }
      d0 = nb_warp_sum(d0) * scale;
      d1 = nb_warp_sum(d1) * scale;
      if (lane == 0) {
        scores[0][j - c0] = d0;
        scores[1][j - c0] = d1;
      }
      cmax[0] = fmaxf(cmax[0], d0);
      cmax[1] = fmaxf(cmax[1], d1);
    }
    float rescale[2];
#pragma unroll
    for (int a = 0; a < 2; ++a) {
      const float m_new = fmaxf(m_run[a], nb_block_max(cmax[a], red));
      float csum = 0.0f;
      for (int j = c0 + tid; j < c1; j += AD_THREADS) {
        const float p = expf(scores[a][j - c0] - m_new);
        scores[a][j - c0] = p;
        csum += p;
      }
      csum = nb_block_sum(csum, red);   // also orders the writes of `scores` before the reads below
      rescale[a] = (m_run[a] == -INFINITY) ? 0.0f : expf(m_run[a] - m_new);
      l_run[a] = l_run[a] * rescale[a] + csum;
      m_run[a] = m_new;
    }
#pragma unroll
    for (int i = 0; i < AD_DPL; ++i) {
      acc[0][i] *= rescale[0];
      acc[1][i] *= rescale[1];
    }
    for (int j = c0 + warp; j < c1; j += AD_WARPS) {
      const TC* vr = vc + (((size_t)vt[j / page] * n_kv_heads + g) * page + (j % page)) * dv;
      const float p0 = scores[0][j - c0], p1 = scores[1][j - c0];
#pragma unroll
      for (int a = 0; a < AD_DPL; ++a) {
        const int i = lane + 32 * a;
        if (i < dv) {
          const float v = nb_to_f32(vr[i]);
          acc[0][a] = fmaf(p0, v, acc[0][a]);
          acc[1][a] = fmaf(p1, v, acc[1][a]);
        }
      }
    }
    __syncthreads();   // `scores` is rewritten by the next chunk
  }
#pragma unroll
  for (int a = 0; a < AD_DPL; ++a) {
    const int i = lane + 32 * a;
    if (i < dv) {
      part[warp][0][i] = acc[0][a];
      part[warp][1][i] = acc[1][a];
    }
  }
  __syncthreads();
  const float i0 = l_run[0] > 0.0f ? 1.0f / l_run[0] : 0.0f;
  const float i1 = l_run[1] > 0.0f ? lambda / l_run[1] : 0.0f;
  float diff[AD_MAXD / AD_THREADS], ss = 0.0f;
#pragma unroll
  for (int k = 0; k < AD_MAXD / AD_THREADS; ++k) {
    const int i = tid + k * AD_THREADS;
    diff[k] = 0.0f;
    if (i < dv) {
      float v0 = 0.0f, v1 = 0.0f;
#pragma unroll
      for (int w = 0; w < AD_WARPS; ++w) {
        v0 += part[w][0][i];
        v1 += part[w][1][i];
      }
      diff[k] = v0 * i0 - v1 * i1;
    }
    ss = fmaf(diff[k], diff[k], ss);
  }
  ss = nb_block_sum(ss, red);
  const float f = factor / sqrtf(ss / (float)dv + eps);
#pragma unroll
  for (int k = 0; k < AD_MAXD / AD_THREADS; ++k) {
    const int i = tid + k * AD_THREADS;
    if (i < dv) o[i] = nb_from_f32<TOut>(diff[k] * f);
  }
}

// ---------------------------------------------------------------------------------------------
// bf16 on mma.sync: a CTA takes 64 query rows of one sequence and one head, a warp 16 of them.
// Key/value pages come in by 16-byte asynchronous copies, two in flight; a key page is staged as
// two tiles, one per map, padded with zeros to a multiple of 16 numbers.  Per page a warp forms
// both maps' scores and probabilities (fp32 softmax per row and map), then walks the values once:
// every value fragment read from shared memory feeds both maps' accumulators.  The difference,
// its norm over the head and the factor are taken on the fp32 accumulators at the end.
// ---------------------------------------------------------------------------------------------
constexpr int MD_THREADS = 128;
constexpr int MD_TILE = 64;
constexpr int MD_PAGE = 64;

template <int NTV>   // the value size rounded up to NTV * 16
__global__ void __launch_bounds__(MD_THREADS)
differential_mma_kernel(const bf16* q, int q_stride, const int* cu_rows, const int* seq_slot,
                        const int* seq_pos0, const bf16* kc, const int* k_table, int k_max_pages,
                        const bf16* vc, const int* v_table, int v_max_pages, int n_heads,
                        int n_kv_heads, int d, int dv, bf16* out, float scale_log2, int window,
                        float lambda, float factor, float eps) {
  using namespace nbmma;
  constexpr int DVP = NTV * 16, LDV = DVP + 8;
  nb_grid_dependency_wait();
  nb_launch_dependents();
  const int k_steps = (d + 15) / 16, LDK = k_steps * 16 + 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* Qs = reinterpret_cast<bf16*>(smem_raw);              // [2 maps][64][LDK]
  bf16* Ks = Qs + 2 * MD_TILE * LDK;                          // [2 stages][2 maps][64][LDK]
  bf16* Vs = Ks + 4 * MD_PAGE * LDK;                          // [2 stages][64][LDV]

  // long tiles (late rows see many keys) start first
  const int tile = (int)gridDim.x - 1 - (int)blockIdx.x, h = blockIdx.y, s = blockIdx.z;
  const int row0 = cu_rows[s], n_q = cu_rows[s + 1] - row0;
  const int q0 = tile * MD_TILE;
  if (q0 >= n_q) return;
  const int slot = seq_slot[s];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rows_here = min(MD_TILE, n_q - q0);
  if (slot < 0) {     // a sequence that has ended (a decode session keeps its row)
    for (int i = tid; i < rows_here * dv; i += MD_THREADS)
      out[((size_t)(row0 + q0 + i / dv) * n_heads + h) * dv + i % dv] = __float2bfloat16_rn(0.0f);
    return;
  }
  const int pos0 = seq_pos0[s];
  const int kvh = h / (n_heads / n_kv_heads);
  const int g = lane >> 2, t = lane & 3;
  const int last_pos = pos0 + q0 + rows_here - 1;
  const int first_key = window > 0 ? max(0, pos0 + q0 + 1 - window) : 0;
  const int p_begin = first_key / MD_PAGE, p_end = last_pos / MD_PAGE + 1;
  const int* kt = k_table + (size_t)slot * k_max_pages;
  const int* vt = v_table + (size_t)slot * v_max_pages;
  const int kch = d >> 3, vch = dv >> 3;      // 16-byte pieces of a map's key, of a value

  if (d != k_steps * 16 || dv != DVP) {       // the padding takes part in the products: zeros
    uint4* p = reinterpret_cast<uint4*>(smem_raw);
    const int n16 = ((2 * MD_TILE * LDK + 4 * MD_PAGE * LDK + 2 * MD_PAGE * LDV) * 2) >> 4;
    for (int i = tid; i < n16; i += MD_THREADS) p[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
  }
  auto issue = [&](int p, int stage) {
    const bf16* ksrc = kc + ((size_t)kt[p] * n_kv_heads + kvh) * MD_PAGE * 2 * d;
    bf16* kdst = Ks + (size_t)stage * 2 * MD_PAGE * LDK;
    for (int i = tid; i < MD_PAGE * 2 * kch; i += MD_THREADS) {
      const int row = i / (2 * kch), c = i - row * 2 * kch;
      const int map = c >= kch ? 1 : 0;
      cp_async16(kdst + (map * MD_PAGE + row) * LDK + (c - map * kch) * 8,
                 ksrc + (size_t)row * 2 * d + c * 8);
    }
    const bf16* vsrc = vc + ((size_t)vt[p] * n_kv_heads + kvh) * MD_PAGE * dv;
    bf16* vdst = Vs + (size_t)stage * MD_PAGE * LDV;
    for (int i = tid; i < MD_PAGE * vch; i += MD_THREADS) {
      const int row = i / vch, c = i - row * vch;
      cp_async16(vdst + row * LDV + c * 8, vsrc + (size_t)row * dv + c * 8);
    }
  };
  for (int i = tid; i < MD_TILE * 2 * kch; i += MD_THREADS) {
    const int row = i / (2 * kch), c = i - row * 2 * kch;
    const int map = c >= kch ? 1 : 0;
    const bool ok = row < rows_here;
    cp_async16_zfill(Qs + (map * MD_TILE + row) * LDK + (c - map * kch) * 8,
                     ok ? q + (size_t)(row0 + q0 + row) * q_stride + (size_t)h * 2 * d + c * 8 : q, ok);
  }
  issue(p_begin, 0);
  ::cp_async_commit();

  float o[2][2 * NTV][4];
#pragma unroll
  for (int a = 0; a < 2; ++a)
#pragma unroll
    for (int n = 0; n < 2 * NTV; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[a][n][j] = 0.0f;
  float m_run[2][2], l_run[2][2];
#pragma unroll
  for (int a = 0; a < 2; ++a) {
    m_run[a][0] = m_run[a][1] = -INFINITY;
    l_run[a][0] = l_run[a][1] = 0.0f;
  }
  const int qpos_a = pos0 + q0 + warp * 16 + g, qpos_b = qpos_a + 8;
  const bool warp_has_rows = warp * 16 < rows_here;

  for (int p = p_begin; p < p_end; ++p) {
    const int stage = (p - p_begin) & 1;
    if (p + 1 < p_end) issue(p + 1, stage ^ 1);
    ::cp_async_commit();
    ::cp_async_wait<1>();
    __syncthreads();
    const bf16* kp = Ks + (size_t)stage * 2 * MD_PAGE * LDK;
    bf16* vp = Vs + (size_t)stage * MD_PAGE * LDV;
    // Rows of the last page after the newest key hold whatever an earlier owner of the page left
    // there; their weights are zero, but zero times a non-finite value is not.
    const int tail_row = last_pos + 1 - p * MD_PAGE;
    if (tail_row < MD_PAGE) {
      for (int i = tid; i < (MD_PAGE - tail_row) * (LDV / 8); i += MD_THREADS) {
        const int row = tail_row + i / (LDV / 8), c = (i % (LDV / 8)) * 8;
        *reinterpret_cast<uint4*>(vp + row * LDV + c) = make_uint4(0u, 0u, 0u, 0u);
      }
      __syncthreads();
    }
    if (warp_has_rows) {
      const int j0 = p * MD_PAGE;
      const bool plain = window <= 0 && j0 + MD_PAGE - 1 <= pos0 + q0 + warp * 16;
      uint32_t pf[2][4][4];
#pragma unroll
      for (int a = 0; a < 2; ++a) {
        float sc[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
        const bf16* qa = Qs + (a * MD_TILE + warp * 16 + (lane & 15)) * LDK + (lane >> 4) * 8;
        const bf16* ka = kp + (a * MD_PAGE + (lane & 7) + (lane >> 4) * 8) * LDK + ((lane >> 3) & 1) * 8;
#pragma unroll 4
        for (int ks = 0; ks < k_steps; ++ks) {
          uint32_t qf[4];
          nbmma::ldmatrix_x4(qf, qa + ks * 16);
#pragma unroll
          for (int n2 = 0; n2 < 4; ++n2) {
            uint32_t kb[4];
            nbmma::ldmatrix_x4(kb, ka + n2 * 16 * LDK + ks * 16);
            nbmma::mma_bf16(sc[2 * n2], qf, kb[0], kb[1]);
            nbmma::mma_bf16(sc[2 * n2 + 1], qf, kb[2], kb[3]);
          }
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 8; ++n) {
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            float v = sc[n][j] * scale_log2;
            if (!plain) {
              const int key = j0 + n * 8 + t * 2 + (j & 1);
              const int qp = (j < 2) ? qpos_a : qpos_b;
              if (key > qp || (window > 0 && key <= qp - window)) v = -INFINITY;
            }
            sc[n][j] = v;
            mx[j >> 1] = fmaxf(mx[j >> 1], v);
          }
        }
        float m_use[2], resc[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
          mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
          const float m_new = fmaxf(m_run[a][r], mx[r]);
          m_use[r] = (m_new == -INFINITY) ? 0.0f : m_new;
          resc[r] = (m_run[a][r] == -INFINITY) ? 0.0f : nb_exp2(m_run[a][r] - m_use[r]);
          m_run[a][r] = m_new;
          l_run[a][r] *= resc[r];
        }
#pragma unroll
        for (int n = 0; n < 2 * NTV; ++n) {
          o[a][n][0] *= resc[0]; o[a][n][1] *= resc[0];
          o[a][n][2] *= resc[1]; o[a][n][3] *= resc[1];
        }
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          const float p0 = nb_exp2(sc[n][0] - m_use[0]), p1 = nb_exp2(sc[n][1] - m_use[0]);
          const float p2 = nb_exp2(sc[n][2] - m_use[1]), p3 = nb_exp2(sc[n][3] - m_use[1]);
          l_run[a][0] += p0 + p1;
          l_run[a][1] += p2 + p3;
          pf[a][n >> 1][(n & 1) * 2] = nbmma::pack_bf16(p0, p1);
          pf[a][n >> 1][(n & 1) * 2 + 1] = nbmma::pack_bf16(p2, p3);
        }
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
#pragma unroll
        for (int n2 = 0; n2 < NTV; ++n2) {
          uint32_t vb[4];
          nbmma::ldmatrix_x4_trans(vb, vp + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDV +
                                           n2 * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int a = 0; a < 2; ++a) {
            nbmma::mma_bf16(o[a][2 * n2], pf[a][kk], vb[0], vb[1]);
            nbmma::mma_bf16(o[a][2 * n2 + 1], pf[a][kk], vb[2], vb[3]);
          }
        }
      }
    }
    __syncthreads();   // the stage may be refilled
  }
  ::cp_async_wait<0>();
  if (!warp_has_rows) return;

  float inv[2][2];
#pragma unroll
  for (int a = 0; a < 2; ++a)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float l = l_run[a][r];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      inv[a][r] = l > 0.0f ? (a == 0 ? 1.0f : lambda) / l : 0.0f;
    }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float ss = 0.0f;
#pragma unroll
    for (int n = 0; n < 2 * NTV; ++n)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const float v = o[0][n][2 * r + c] * inv[0][r] - o[1][n][2 * r + c] * inv[1][r];
        o[0][n][2 * r + c] = v;
        ss = fmaf(v, v, ss);
      }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    const float f = factor / sqrtf(ss / (float)dv + eps);
    const int row = warp * 16 + g + 8 * r;
    if (row < rows_here) {
      bf16* dst = out + ((size_t)(row0 + q0 + row) * n_heads + h) * dv;
#pragma unroll
      for (int n = 0; n < 2 * NTV; ++n) {
        const int col = n * 8 + 2 * t;
        if (col < dv)
          *reinterpret_cast<uint32_t*>(dst + col) =
              nbmma::pack_bf16(o[0][n][2 * r] * f, o[0][n][2 * r + 1] * f);
      }
    }
  }
}

template <int NTV>
int launch_mma(const bf16* q, int q_stride, const int* cu_rows, const int* seq_slot, const int* seq_pos0,
               const bf16* kc, const int* k_table, int k_max_pages, const bf16* vc, const int* v_table,
               int v_max_pages, int n_heads, int n_kv_heads, int d, int dv, bf16* out, float scale,
               int window, float lambda, float factor, float eps, int n_seqs, int max_q_len,
               cudaStream_t stream) {
  const int ldk = (d + 15) / 16 * 16 + 8, ldv = NTV * 16 + 8;
  const size_t smem = (size_t)(2 * MD_TILE * ldk + 4 * MD_PAGE * ldk + 2 * MD_PAGE * ldv) * sizeof(bf16);
  static size_t configured = 48 * 1024;   // per instantiation: the largest size asked for
  if (smem > configured) {
    NB_CUDA(cudaFuncSetAttribute(differential_mma_kernel<NTV>,
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  const dim3 grid((max_q_len + MD_TILE - 1) / MD_TILE, n_heads, n_seqs);
  NB_CUDA(nb_launch(differential_mma_kernel<NTV>, grid, dim3(MD_THREADS), smem, stream, q, q_stride,
                    cu_rows, seq_slot, seq_pos0, kc, k_table, k_max_pages, vc, v_table, v_max_pages,
                    n_heads, n_kv_heads, d, dv, out, scale * 1.4426950408889634f, window, lambda,
                    factor, eps));
  return 0;
}

}  // namespace

// q: [n_rows][n_heads * 2 d]; kc: [n_pages][n_kv_heads][page][2 d]; vc: [n_pages][n_kv_heads][page][dv];
// out: [n_rows][n_heads * dv]; window <= 0: every earlier token.
NB_EXPORT int nb_attention_differential(const void* q, int q_dtype, const int* row_slot,
                                        const int* row_pos, const void* kc, const int* k_table,
                                        int k_max_pages, const void* vc, const int* v_table,
                                        int v_max_pages, int cache_dtype, int page, int n_heads,
                                        int n_kv_heads, int d, int dv, void* out, int out_dtype,
                                        float scale, int window, float lambda, float factor, float eps,
                                        int n_rows, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NB_REQUIRE(d >= 1 && d <= AD_MAXD && dv >= 1 && dv <= AD_MAXD, NB_ERR_UNSUPPORTED,
             "attention_differential: heads of %d / %d are outside 1..%d", d, dv, AD_MAXD);
  NB_REQUIRE(n_heads >= 1 && n_heads <= 65535 && n_kv_heads >= 1 && n_heads % n_kv_heads == 0 && page > 0,
             NB_ERR_BAD_ARG, "attention_differential: bad sizes heads=%d/%d page=%d", n_heads,
             n_kv_heads, page);
  const dim3 grid(n_rows, n_heads);
#define NB_AD(TQ, TC, TO)                                                                            \
  NB_CUDA(nb_launch(attention_differential_kernel<TQ, TC, TO>, grid, dim3(AD_THREADS), 0, stream,    \
                    (const TQ*)q, row_slot, row_pos, (const TC*)kc, k_table, k_max_pages,            \
                    (const TC*)vc, v_table, v_max_pages, page, n_heads, n_kv_heads, d, dv, (TO*)out, \
                    scale, window, lambda, factor, eps))
  switch (q_dtype * 4 + cache_dtype * 2 + out_dtype) {
    case 0: NB_AD(float, float, float); break;
    case 7: NB_AD(bf16, bf16, bf16); break;
    default:
      NB_REQUIRE(false, NB_ERR_UNSUPPORTED, "attention_differential: dtypes %d/%d/%d are not built",
                 q_dtype, cache_dtype, out_dtype);
  }
#undef NB_AD
  NB_CHECK_LAUNCH("attention_differential");
  return 0;
}

NB_EXPORT int nb_attention_differential_mma_supported(int dtype, int d, int dv, int page, int q_stride) {
  return dtype == NB_BF16 && page == MD_PAGE && d % 8 == 0 && d >= 8 && d <= 128 && dv % 8 == 0 &&
         dv >= 8 && dv <= 128 && q_stride % 8 == 0;
}

// bf16 throughout; rows of sequence s are cu_rows[s] .. cu_rows[s+1] at positions seq_pos0[s] .. of
// slot seq_slot[s], their keys and values already in the cache.
NB_EXPORT int nb_attention_differential_mma(const void* q, int q_stride, const int* cu_rows,
                                            const int* seq_slot, const int* seq_pos0, const void* kc,
                                            const int* k_table, int k_max_pages, const void* vc,
                                            const int* v_table, int v_max_pages, int page, int n_heads,
                                            int n_kv_heads, int d, int dv, void* out, float scale,
                                            int window, float lambda, float factor, float eps,
                                            int n_seqs, int max_q_len, cudaStream_t stream) {
  if (n_seqs == 0 || max_q_len == 0) return 0;
  NB_REQUIRE(nb_attention_differential_mma_supported(NB_BF16, d, dv, page, q_stride), NB_ERR_UNSUPPORTED,
             "attention_differential_mma: unsupported shape (%d / %d, page %d)", d, dv, page);
  NB_REQUIRE(n_kv_heads >= 1 && n_heads % n_kv_heads == 0 && n_seqs <= 65535 && n_heads <= 65535,
             NB_ERR_UNSUPPORTED, "attention_differential_mma: bad grid");
  NB_REQUIRE(((uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)out) % 16 == 0, NB_ERR_BAD_ARG,
             "attention_differential_mma: pointers must be 16-byte aligned");
  const int nt = (dv + 15) / 16;
  int rc;
#define NB_MD(N_)                                                                                     \
  rc = launch_mma<N_>((const bf16*)q, q_stride, cu_rows, seq_slot, seq_pos0, (const bf16*)kc, k_table, \
                      k_max_pages, (const bf16*)vc, v_table, v_max_pages, n_heads, n_kv_heads, d, dv,  \
                      (bf16*)out, scale, window, lambda, factor, eps, n_seqs, max_q_len, stream)
  if (nt <= 2) NB_MD(2);
  else if (nt <= 4) NB_MD(4);
  else if (nt <= 6) NB_MD(6);
  else NB_MD(8);
#undef NB_MD
  if (rc) return rc;
  NB_CHECK_LAUNCH("attention_differential_mma");
  return 0;
}
