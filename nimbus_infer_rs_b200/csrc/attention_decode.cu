// Decode attention: one query row per sequence over that sequence's paged keys and values.
//
// The work is reading the cache once, so the kernel is laid out for bandwidth: a CTA takes one
// (row, key/value head, split of the sequence's pages), streams whole pages (64 keys x head_dim,
// contiguous) into shared memory with 16-byte cp.async copies, two or four pages in flight (the
// first ones asked for before the kernel's wait on its predecessor), and all query heads that
// share the key/value head are served from the same staged page.  Scores, softmax and the
// weighted sum are fp32; every warp keeps a running (max, sum, accumulator) for its quarter of
// a page (the bfloat16 kernel has four warps on a page, or eight on two pages at a time), the
// warps are merged at the end of the split, and the splits are merged either inside a
// thread-block cluster (2 to 8 splits of the bfloat16 kernel: partial results into the first
// CTA's shared memory, one cluster barrier) or by whichever CTA of the (row, head) finishes
// last (a counter in scratch memory that it leaves at zero again).
//
// Scratch (caller-allocated): part_acc [rows][heads][splits][head_dim] fp32, part_ml
// [rows][heads][splits][2] fp32, counters [rows][kv_heads] int32, zero before the first use.
//
// Reference: src/model.rs:401-422 (scores = dot(q,k)*scale over keys 0..pos, softmax,
// weighted values), head h reads key/value head h / group (src/model.rs:390).
#include <mutex>

#include "common.cuh"
#include <atomic>

#include "attention_decode_mma.cuh"

namespace {

constexpr int THREADS = 128;
constexpr int WARPS = 4;

// G: query heads per key/value head served by one CTA (group <= G).
template <typename T, int HD, int G, typename TOut>
__global__ void __launch_bounds__(THREADS)
attention_decode_kernel(const T* q, int q_stride, int q_col,
                        const int* row_slot, const int* row_pos,
                        NbPagedKV kv, int group, TOut* out, int out_stride,
                        float scale, float softcap, const float* sink, NbAttnOpts opt, int n_splits, float* part_acc,
                        float* part_ml, int* counters, int append,
                        int k_col, int v_col) {
  constexpr int EPL = Lane16<T>::N;           // elements per lane
  constexpr int LPR = HD / EPL;               // lanes per key row
  constexpr int RPW = 32 / LPR;               // key rows per warp iteration
  constexpr int KEYS_PER_WARP = PAGE_TOKENS / WARPS;
  constexpr int ITERS = KEYS_PER_WARP / RPW;
  constexpr int TILE = PAGE_TOKENS * HD;      // elements of one page of one head
  static_assert(LPR >= 1 && LPR <= 32 && (LPR & (LPR - 1)) == 0, "head size not supported");
  static_assert(ITERS >= 1, "head size not supported");

  extern __shared__ __align__(16) unsigned char smem_raw[];
  T* tiles = reinterpret_cast<T*>(smem_raw);                       // [2 stages][K tile | V tile]
  float* q_s = reinterpret_cast<float*>(smem_raw + (size_t)4 * TILE * sizeof(T));  // [G][HD]
  float* w_acc = q_s + G * HD;                                     // [WARPS][G][HD]
  float* w_ml = w_acc + WARPS * G * HD;                            // [WARPS][G][2]
  __shared__ int s_last;

  nb_grid_dependency_wait();
  const int split = blockIdx.x, kvh = blockIdx.y, r = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int sub = lane / LPR, part = lane % LPR;
  const int n_heads = kv.n_kv_heads * group;
  const int slot = row_slot[r];
  if (slot < 0) {   // padding row: zeros, written by split 0
    if (split == 0)
      for (int i = tid; i < group * HD; i += THREADS)
        out[(size_t)r * out_stride + (size_t)kvh * group * HD + i] = nb_from_f32<TOut>(0.0f);
    return;
  }
  const int pos = row_pos[r];
  const int kv_len = pos + 1;
  const int j_begin = opt.first_key(pos);
  const int keep_first = opt.keeps() ? opt.keep_first : 0;
  const int first_page = j_begin / PAGE_TOKENS;
  const int n_pages = (kv_len + PAGE_TOKENS - 1) / PAGE_TOKENS - first_page;
  // with kept first tokens the last split is theirs: the pages before the window's first that
  // hold some of them (none when the window still reaches back to them)
  const int run_splits = opt.keeps() ? n_splits - 1 : n_splits;
  const int per_split = (n_pages + run_splits - 1) / run_splits;
  const bool head_split = opt.keeps() && split == n_splits - 1;
  const int p_begin = head_split ? 0 : first_page + split * per_split;
  const int p_end = head_split ? min((keep_first + PAGE_TOKENS - 1) / PAGE_TOKENS, first_page)
                               : min(first_page + n_pages, p_begin + per_split);

  // queries of the group, fp32
  for (int i = tid; i < G * HD; i += THREADS) {
    const int gh = i / HD, c = i - gh * HD;
    q_s[i] = (gh < group)
                 ? nb_to_f32(q[(size_t)r * q_stride + q_col + (size_t)(kvh * group + gh) * HD + c])
                 : 0.0f;
  }

  const int* table = kv.block_table + (size_t)slot * kv.max_pages;
  auto issue = [&](int page_idx, int stage) {
    const int page_id = table[page_idx];
    const T* ksrc = (const T*)kv.k + ((size_t)page_id * kv.n_kv_heads + kvh) * TILE;
    const T* vsrc = (const T*)kv.v + ((size_t)page_id * kv.n_kv_heads + kvh) * TILE;
    T* kdst = tiles + (size_t)stage * 2 * TILE;
    T* vdst = kdst + TILE;
    constexpr int VECS = TILE / EPL;   // 16-byte pieces per tile
    for (int i = tid; i < VECS; i += THREADS) {
      cp_async16(kdst + i * EPL, ksrc + i * EPL);
      cp_async16(vdst + i * EPL, vsrc + i * EPL);
    }
    cp_async_commit();
  };

  float m_run[G], l_run[G], acc[G][EPL];
#pragma unroll
  for (int gh = 0; gh < G; ++gh) {
    m_run[gh] = -INFINITY;
    l_run[gh] = 0.0f;
#pragma unroll
    for (int e = 0; e < EPL; ++e) acc[gh][e] = 0.0f;
  }

  if (p_begin < p_end) issue(p_begin, 0);
  __syncthreads();   // q_s is complete
  float qreg[G][EPL];
#pragma unroll
  for (int gh = 0; gh < G; ++gh)
#pragma unroll
    for (int e = 0; e < EPL; ++e) qreg[gh][e] = q_s[gh * HD + part * EPL + e];

  for (int p = p_begin; p < p_end; ++p) {
    const int stage = (p - p_begin) & 1;
    if (p + 1 < p_end) {
      issue(p + 1, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    T* kt = tiles + (size_t)stage * 2 * TILE;
    T* vt = kt + TILE;
    if (append > 0 && p == pos / PAGE_TOKENS) {
      // this step's own key and value (row r of the projection output) belong at token `pos`
      // of this page: put them into the staged tile and into the cache
      const int in_page = pos % PAGE_TOKENS;
      const int page_id = table[p];
      for (int i = tid; i < 2 * LPR; i += THREADS) {
        const bool is_v = i >= LPR;
        const int c = (is_v ? i - LPR : i) * EPL;
        const uint4 val = *reinterpret_cast<const uint4*>(
            q + (size_t)r * q_stride + (is_v ? v_col : k_col) + (size_t)kvh * HD + c);
        *reinterpret_cast<uint4*>((is_v ? vt : kt) + in_page * HD + c) = val;
        T* cache = (T*)(is_v ? kv.v : kv.k);
        *reinterpret_cast<uint4*>(cache + ((size_t)page_id * kv.n_kv_heads + kvh) * TILE +
                                  in_page * HD + c) = val;
      }
      __syncthreads();
    }
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int row = warp * KEYS_PER_WARP + it * RPW + sub;   // key within the page
      const int j = p * PAGE_TOKENS + row;
      const bool valid = (j >= j_begin || j < keep_first) && (j < kv_len);
      float kf[EPL], vf[EPL];
      Lane16<T>::load(kt + (size_t)row * HD + part * EPL, kf);
      Lane16<T>::load(vt + (size_t)row * HD + part * EPL, vf);
      if (!valid) {   // whatever an unused cache row holds must not reach the sum
#pragma unroll
        for (int e = 0; e < EPL; ++e) vf[e] = 0.0f;
      }
#pragma unroll
      for (int gh = 0; gh < G; ++gh) {
        float dot = 0.0f;
#pragma unroll
        for (int e = 0; e < EPL; ++e) dot = fmaf(qreg[gh][e], kf[e], dot);
#pragma unroll
        for (int o = LPR / 2; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
        float s = dot * scale;
        if (softcap > 0.0f) s = softcap * tanhf(s / softcap);
        if (!valid) s = -INFINITY;
        float mx = s;
#pragma unroll
        for (int o = LPR; o < 32; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m_run[gh], mx);
        if (m_new > -INFINITY) {   // warp-uniform
          const float rescale = (m_run[gh] == -INFINITY) ? 0.0f : expf(m_run[gh] - m_new);
          const float pr = valid ? expf(s - m_new) : 0.0f;
          l_run[gh] = l_run[gh] * rescale + pr;
#pragma unroll
          for (int e = 0; e < EPL; ++e) acc[gh][e] = fmaf(pr, vf[e], acc[gh][e] * rescale);
          m_run[gh] = m_new;
        }
      }
    }
    __syncthreads();   // the stage is free for the copy after next
  }

  nb_launch_dependents();   // the pages are read: the next kernel may be set up
  // merge the key rows a warp handled side by side (lanes with equal `part`)
#pragma unroll
  for (int gh = 0; gh < G; ++gh) {
    // l_run of a lane counts only its own rows; every lane of a row group holds the same value
#pragma unroll
    for (int o = LPR; o < 32; o <<= 1) {
      l_run[gh] += __shfl_xor_sync(0xffffffffu, l_run[gh], o);
#pragma unroll
      for (int e = 0; e < EPL; ++e) acc[gh][e] += __shfl_xor_sync(0xffffffffu, acc[gh][e], o);
    }
    if (sub == 0) {
#pragma unroll
      for (int e = 0; e < EPL; ++e) w_acc[(warp * G + gh) * HD + part * EPL + e] = acc[gh][e];
      if (part == 0) {
        w_ml[(warp * G + gh) * 2] = m_run[gh];
        w_ml[(warp * G + gh) * 2 + 1] = l_run[gh];
      }
    }
  }
  __syncthreads();
  // merge the warps -> partial result of this split
  for (int i = tid; i < group * HD; i += THREADS) {
    const int gh = i / HD, c = i - gh * HD;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) M = fmaxf(M, w_ml[(w * G + gh) * 2]);
    float a = 0.0f, l = 0.0f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float mw = w_ml[(w * G + gh) * 2];
      const float f = (mw == -INFINITY) ? 0.0f : expf(mw - M);
      a += f * w_acc[(w * G + gh) * HD + c];
      l += f * w_ml[(w * G + gh) * 2 + 1];
    }
    const int head = kvh * group + gh;
    if (n_splits == 1) {   // nothing to merge with: this is the result
      if (sink != nullptr) a *= nb_sink_fix(l, M, sink[head], false);
      a *= opt.gate_of(r, head);
      out[(size_t)r * out_stride + (size_t)head * HD + c] = nb_from_f32<TOut>(l > 0.0f ? a / l : a);
      continue;
    }
    const size_t pi = ((size_t)r * n_heads + head) * n_splits + split;
    part_acc[pi * HD + c] = a;
    if (c == 0) {
      part_ml[pi * 2] = M;
      part_ml[pi * 2 + 1] = l;
    }
  }
  if (n_splits == 1) return;
  // the CTA that finishes last for this (row, key/value head) merges the splits
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const int old = atomicAdd(&counters[r * kv.n_kv_heads + kvh], 1);
    s_last = (old == n_splits - 1);
    if (s_last) counters[r * kv.n_kv_heads + kvh] = 0;   // ready for the next launch
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int i = tid; i < group * HD; i += THREADS) {
    const int gh = i / HD, c = i - gh * HD;
    const int head = kvh * group + gh;
    const size_t base = ((size_t)r * n_heads + head) * n_splits;
    float M = -INFINITY;
    for (int s = 0; s < n_splits; ++s) M = fmaxf(M, __ldcg(&part_ml[(base + s) * 2]));
    float a = 0.0f, l = 0.0f;
    for (int s = 0; s < n_splits; ++s) {
      const float ms = __ldcg(&part_ml[(base + s) * 2]);
      const float f = (ms == -INFINITY) ? 0.0f : expf(ms - M);
      a += f * __ldcg(&part_acc[(base + s) * HD + c]);
      l += f * __ldcg(&part_ml[(base + s) * 2 + 1]);
    }
    if (sink != nullptr) a *= nb_sink_fix(l, M, sink[head], false);
    a *= opt.gate_of(r, head);
    out[(size_t)r * out_stride + (size_t)head * HD + c] = nb_from_f32<TOut>(l > 0.0f ? a / l : a);
  }
}

template <typename TOut>
int mma_by_head_dim(int hd, const void* q, int q_stride, int q_col, const int* row_slot,
                    const int* row_pos, const NbPagedKV& kv, int group, void* out, int out_stride,
                    float scale, float softcap, const float* sink, NbAttnOpts opt, int n_rows, int n_splits, float* pa, float* pm,
                    int* cn, int ap, int kc, int vc, bool clustered, cudaStream_t st) {
#define NB_ARGS q, q_stride, q_col, row_slot, row_pos, kv, group, out, out_stride, scale, softcap, sink, opt, n_rows, n_splits, pa, pm, cn, ap, kc, vc, clustered, st
  if constexpr (sizeof(TOut) == 2) {
    if (opt.maps) {
      switch (hd) {
        case 32: return launch_mma<32, TOut, true, false>(NB_ARGS);
        case 64: return launch_mma<64, TOut, true, false>(NB_ARGS);
        case 96: return launch_mma<96, TOut, true, false>(NB_ARGS);
        case 128: return launch_mma<128, TOut, true, false>(NB_ARGS);
      }
      return NB_ERR_UNSUPPORTED;
    }
  }
#define NB_HD(HD_) \
  case HD_: return launch_mma<HD_, TOut, false, false>(NB_ARGS)
  switch (hd) {
    NB_HD(16); NB_HD(32); NB_HD(48); NB_HD(64); NB_HD(80); NB_HD(96); NB_HD(112); NB_HD(128);
  }
#undef NB_HD
#undef NB_ARGS
  return NB_ERR_UNSUPPORTED;
}

template <typename T, int HD, int G, typename TOut>
int launch(const void* q, int q_stride, int q_col, const int* row_slot, const int* row_pos,
           const NbPagedKV& kv, int group, void* out, int out_stride, float scale, float softcap, const float* sink, NbAttnOpts opt,
           int n_rows, int n_splits, float* part_acc, float* part_ml, int* counters, int append,
           int k_col, int v_col, cudaStream_t stream) {
  const size_t smem = (size_t)4 * PAGE_TOKENS * HD * sizeof(T) +
                      (size_t)(G * HD + WARPS * G * HD + WARPS * G * 2) * sizeof(float);
  auto kern = attention_decode_kernel<T, HD, G, TOut>;
  if (smem > 48 * 1024)
    NB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  dim3 grid(n_splits, kv.n_kv_heads, n_rows);
  NB_CUDA(nb_launch(kern, grid, dim3(THREADS), smem, stream, (const T*)q, q_stride, q_col, row_slot,
                    row_pos, kv, group, (TOut*)out, out_stride, scale, softcap, sink, opt, n_splits, part_acc,
                    part_ml, counters, append, k_col, v_col));
  return 0;
}

template <typename T, int HD, typename TOut>
int by_group(int group, const void* q, int q_stride, int q_col, const int* row_slot,
             const int* row_pos, const NbPagedKV& kv, void* out, int out_stride, float scale, float softcap,
             const float* sink, NbAttnOpts opt, int n_rows, int n_splits, float* pa, float* pm, int* cn, int ap,
             int kc, int vc, cudaStream_t st) {
#define NB_G(G_) \
  return launch<T, HD, G_, TOut>(q, q_stride, q_col, row_slot, row_pos, kv, group, out, out_stride, scale, softcap, sink, opt, n_rows, n_splits, pa, pm, cn, ap, kc, vc, st)
  if (group == 1) NB_G(1);
  if (group == 2) NB_G(2);
  if (group <= 4) NB_G(4);
  NB_G(8);
#undef NB_G
}

template <typename T, typename TOut>
int by_head_dim(int hd, int group, const void* q, int q_stride, int q_col, const int* row_slot,
                const int* row_pos, const NbPagedKV& kv, void* out, int out_stride, float scale, float softcap,
                const float* sink, NbAttnOpts opt, int n_rows, int n_splits, float* pa, float* pm, int* cn, int ap,
                int kc, int vc, cudaStream_t st) {
#define NB_HD(HD_) \
  return by_group<T, HD_, TOut>(group, q, q_stride, q_col, row_slot, row_pos, kv, out, out_stride, scale, softcap, sink, opt, n_rows, n_splits, pa, pm, cn, ap, kc, vc, st)
  switch (hd) {
    case 16: NB_HD(16);
    case 32: NB_HD(32);
    case 64: NB_HD(64);
    case 128: NB_HD(128);
  }
#undef NB_HD
  return NB_ERR_UNSUPPORTED;
}

}  // namespace

// 1 if this kernel takes the shape (otherwise the caller uses the generic kernel).
NB_EXPORT int nb_attention_decode_supported(int dtype, int head_dim, int n_heads, int n_kv_heads,
                                            int page) {
  if (page != PAGE_TOKENS || n_kv_heads < 1 || n_heads % n_kv_heads != 0) return 0;
  if (n_heads / n_kv_heads > 8) return 0;
  if (dtype == NB_BF16) return head_dim % 16 == 0 && head_dim >= 16 && head_dim <= 128;
  if (dtype != NB_F32) return 0;
  return head_dim == 16 || head_dim == 32 || head_dim == 64 || head_dim == 128;
}

// Floats of part_acc, floats of part_ml and ints of counters that a launch needs.
NB_EXPORT void nb_attention_decode_scratch(int n_rows, int n_heads, int n_kv_heads, int head_dim,
                                           int n_splits, long long* acc_floats,
                                           long long* ml_floats, long long* counter_ints) {
  *acc_floats = (long long)n_rows * n_heads * n_splits * head_dim;
  *ml_floats = (long long)n_rows * n_heads * n_splits * 2;
  *counter_ints = (long long)n_rows * n_kv_heads;
}

// append != 0: row r of `q` also holds this step's key and value at columns k_col / v_col;
// the kernel writes them to the cache at token row_pos[r] and attends to them as well, so no
// separate append pass is needed.
namespace {
std::atomic<int> g_cluster_merge{1};

int attention_decode(const void* q, int dtype, int q_stride, int q_col, const int* row_slot,
                     const int* row_pos, const void* k_cache, const void* v_cache,
                     const int* block_table, int max_pages, int page, int n_heads, int n_kv_heads,
                     int head_dim, void* out, int out_dtype, int out_stride, float scale, float softcap, const float* sink, NbAttnOpts opt,
                     int n_rows, int n_splits, float* part_acc, float* part_ml, int* counters,
                     int append, int k_col, int v_col, int clusters_allowed, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NB_REQUIRE(nb_attention_decode_supported(dtype, head_dim, n_heads, n_kv_heads, page),
             NB_ERR_UNSUPPORTED,
             "attention_decode: unsupported shape (head size %d, %d/%d heads, page %d)", head_dim,
             n_heads, n_kv_heads, page);
  NB_REQUIRE(n_splits >= 1 && n_splits <= 65535 && n_rows <= 65535 && n_kv_heads <= 65535,
             NB_ERR_UNSUPPORTED, "attention_decode: grid too large");
  NB_REQUIRE(part_acc && part_ml && counters, NB_ERR_BAD_ARG, "attention_decode: scratch missing");
  if (append > 0) {
    const int epl = dtype == NB_F32 ? 4 : 8;
    NB_REQUIRE(q_stride % epl == 0 && k_col % epl == 0 && v_col % epl == 0 && (uintptr_t)q % 16 == 0,
               NB_ERR_UNSUPPORTED, "attention_decode: keys/values to append must be 16-byte aligned");
  }
  NbPagedKV kv{(void*)k_cache, (void*)v_cache, block_table, max_pages, page, n_kv_heads, head_dim};
  const int group = n_heads / n_kv_heads;
  typedef __nv_bfloat16 bf16;
  int rc;
#define NB_ARGS head_dim, group, q, q_stride, q_col, row_slot, row_pos, kv, out, out_stride, scale, softcap, sink, opt, n_rows, n_splits, part_acc, part_ml, counters, append, k_col, v_col, stream
  if (dtype == NB_F32) {
    rc = out_dtype == NB_F32 ? by_head_dim<float, float>(NB_ARGS) : by_head_dim<float, bf16>(NB_ARGS);
  } else {
    // bf16 cache: tensor cores (needs 16-byte aligned rows and 4-byte aligned query columns)
    NB_REQUIRE(q_stride % 8 == 0 && q_col % 2 == 0 && (uintptr_t)q % 16 == 0, NB_ERR_UNSUPPORTED,
               "attention_decode: query rows must be 16-byte aligned");
    // up to MAX_CLUSTER splits merge through the shared memory of a thread-block cluster, more
    // through the scratch arrays and a counter
    const bool clustered = clusters_allowed > 0 && n_splits >= 2 && n_splits <= MAX_CLUSTER;
    rc = out_dtype == NB_F32
             ? mma_by_head_dim<float>(head_dim, q, q_stride, q_col, row_slot, row_pos, kv, group, out, out_stride, scale, softcap, sink, opt, n_rows, n_splits, part_acc, part_ml, counters, append, k_col, v_col, clustered, stream)
             : mma_by_head_dim<bf16>(head_dim, q, q_stride, q_col, row_slot, row_pos, kv, group, out, out_stride, scale, softcap, sink, opt, n_rows, n_splits, part_acc, part_ml, counters, append, k_col, v_col, clustered, stream);
  }
#undef NB_ARGS
  if (rc) return rc;
  NB_CHECK_LAUNCH("attention_decode");
  return 0;
}
}  // namespace

NB_EXPORT int nb_attention_decode(const void* q, int dtype, int q_stride, int q_col,
                                  const int* row_slot, const int* row_pos, const void* k_cache,
                                  const void* v_cache, const int* block_table, int max_pages,
                                  int page, int n_heads, int n_kv_heads, int head_dim, void* out,
                                  int out_dtype, int out_stride, float scale, int window,
                                  int n_rows, int n_splits, float* part_acc, float* part_ml,
                                  int* counters, int append, int k_col, int v_col,
                                  cudaStream_t stream) {
  return attention_decode(q, dtype, q_stride, q_col, row_slot, row_pos, k_cache, v_cache, block_table,
                          max_pages, page, n_heads, n_kv_heads, head_dim, out, out_dtype, out_stride,
                          scale, 0.0f, nullptr, NbAttnOpts{window, 0, 0, nullptr, 0, 0}, n_rows, n_splits, part_acc, part_ml,
                          counters, append, k_col, v_col, g_cluster_merge.load(), stream);
}

// The same with capped scores (softcap > 0: a score becomes softcap * tanh(score / softcap)) and
// a sink (fp32 [n_heads] logits of one more term of the softmax's denominator, without key or
// value; null for none), and with the options of NbAttnOpts (a window that keeps the sequence's first
// tokens, which then take the last of the n_splits splits, or blocks of positions; a gate per
// head).  The step's keys and values are in the cache already, written by the
// kernel launched before this one: the pages are asked for only after that kernel is done.
NB_EXPORT int nb_attention_decode_capped(const void* q, int dtype, int q_stride, int q_col,
                                         const int* row_slot, const int* row_pos,
                                         const void* k_cache, const void* v_cache,
                                         const int* block_table, int max_pages, int page,
                                         int n_heads, int n_kv_heads, int head_dim, void* out,
                                         int out_dtype, int out_stride, float scale, float softcap,
                                         const float* sink, int window, int keep_first,
                                         int mask_block, const float* gate, int gate_stride,
                                         int gate_col, int n_rows, int n_splits,
                                         float* part_acc, float* part_ml, int* counters,
                                         cudaStream_t stream) {
  NB_REQUIRE(softcap >= 0.0f, NB_ERR_BAD_ARG, "attention_decode: a cap is positive, or 0 for none");
  NB_REQUIRE(window >= 0 && keep_first >= 0 && mask_block >= 0 && !(window > 0 && mask_block > 0),
             NB_ERR_BAD_ARG, "attention_decode: a mask is a window (with kept first tokens) or a block");
  const NbAttnOpts opt{window, keep_first, mask_block, gate, gate_stride, gate_col};
  NB_REQUIRE(!opt.keeps() || n_splits >= 2, NB_ERR_BAD_ARG,
             "attention_decode: kept first tokens take a split of their own");
  return attention_decode(q, dtype, q_stride, q_col, row_slot, row_pos, k_cache, v_cache, block_table,
                          max_pages, page, n_heads, n_kv_heads, head_dim, out, out_dtype, out_stride,
                          scale, softcap, sink, opt, n_rows, n_splits, part_acc, part_ml, counters,
                          /*append=*/-1, 0, 0, g_cluster_merge.load(), stream);
}

// Differential heads on the bfloat16 kernel (NbAttnOpts::maps): n_heads of them over n_kv_heads
// key/value heads of head_dim numbers, a key head's two maps side by side; q: head after head
// [map 1 | map 2].  The step's keys and values are in the cache already (as above).
NB_EXPORT int nb_attention_decode_maps_supported(int dtype, int head_dim, int n_heads, int n_kv_heads,
                                                 int page) {
  return dtype == NB_BF16 && head_dim % 32 == 0 &&
         nb_attention_decode_supported(dtype, head_dim, 2 * n_heads, n_kv_heads, page);
}

NB_EXPORT int nb_attention_decode_maps(const void* q, int q_stride, const int* row_slot,
                                       const int* row_pos, const void* k_cache, const void* v_cache,
                                       const int* block_table, int max_pages, int page, int n_heads,
                                       int n_kv_heads, int head_dim, void* out, int out_stride,
                                       float scale, int window, float lambda, float factor, float eps,
                                       int n_rows, int n_splits, float* part_acc, float* part_ml,
                                       int* counters, cudaStream_t stream) {
  NB_REQUIRE(nb_attention_decode_maps_supported(NB_BF16, head_dim, n_heads, n_kv_heads, page),
             NB_ERR_UNSUPPORTED, "attention_decode_maps: unsupported shape (head size %d, %d/%d heads)",
             head_dim, n_heads, n_kv_heads);
  NB_REQUIRE(window >= 0, NB_ERR_BAD_ARG, "attention_decode_maps: bad window %d", window);
  NbAttnOpts opt{window, 0, 0, nullptr, 0, 0};
  opt.maps = 1;
  opt.lambda = lambda;
  opt.factor = factor;
  opt.eps = eps;
  return attention_decode(q, NB_BF16, q_stride, 0, row_slot, row_pos, k_cache, v_cache, block_table,
                          max_pages, page, 2 * n_heads, n_kv_heads, head_dim, out, NB_BF16, out_stride,
                          scale, 0.0f, nullptr, opt, n_rows, n_splits, part_acc, part_ml, counters,
                          /*append=*/-1, 0, 0, g_cluster_merge.load(), stream);
}

// How the splits of the bfloat16 kernel merge: 0 always through the scratch arrays; otherwise
// (the default) through a cluster's shared memory where there are 2 to 8 of them.  Returns the
// earlier setting.
NB_EXPORT int nb_attention_decode_cluster_merge(int mode) {
  return g_cluster_merge.exchange(mode != 0 ? 1 : 0);
}

// Most splits that merge inside a cluster.
NB_EXPORT int nb_attention_decode_cluster_limit() { return MAX_CLUSTER; }

// ---------------------------------------------------------------------------------------
// The same kernel for callers that cannot allocate device memory (see no_alloc.h).
// Its scratch is this file-scope array: every GPU that loads the library holds these
// NB_STATIC_SCRATCH_BYTES until the process exits.
// ---------------------------------------------------------------------------------------
#include "no_alloc.h"

static __device__ __align__(256) unsigned char g_static_scratch[NB_STATIC_SCRATCH_BYTES];

namespace {
constexpr int MAX_DEVICES = 64;
std::mutex g_static_mutex;
void* g_static_ptr[MAX_DEVICES] = {nullptr};

// The array's device address on the current device.  In host code the name
// `g_static_scratch` is only a handle for the runtime, never an address a kernel may use.
int static_scratch_address(unsigned char** out, cudaStream_t stream) {
  int dev = -1;
  NB_CUDA(cudaGetDevice(&dev));
  NB_REQUIRE(dev >= 0 && dev < MAX_DEVICES, NB_ERR_UNSUPPORTED,
             "attention_decode_static: device index %d is beyond %d", dev, MAX_DEVICES);
  // the address below is the current device's copy of the array: a stream of another device
  // would run the kernel there, on memory it does not own
  int stream_dev = dev;
  if (stream != nullptr && cudaStreamGetDevice(stream, &stream_dev) != cudaSuccess) {
    (void)cudaGetLastError();
    stream_dev = dev;
  }
  NB_REQUIRE(stream_dev == dev, NB_ERR_BAD_ARG,
             "attention_decode_static: the stream belongs to device %d, the current device is %d",
             stream_dev, dev);
  std::lock_guard<std::mutex> lock(g_static_mutex);
  if (g_static_ptr[dev] == nullptr) {
    void* p = nullptr;
    NB_CUDA(cudaGetSymbolAddress(&p, g_static_scratch));
    NB_REQUIRE(p != nullptr, NB_ERR_UNSUPPORTED, "attention_decode_static: no symbol address");
    g_static_ptr[dev] = p;
  }
  *out = static_cast<unsigned char*>(g_static_ptr[dev]);
  return 0;
}
}  // namespace

NB_EXPORT long long nb_attention_decode_static_capacity() { return NB_STATIC_SCRATCH_BYTES; }

NB_EXPORT int nb_attention_decode_static(const void* q, int dtype, int q_stride, int q_col,
                                         const int* row_slot, const int* row_pos,
                                         const void* k_cache, const void* v_cache,
                                         const int* block_table, int max_pages, int page,
                                         int n_heads, int n_kv_heads, int head_dim, void* out,
                                         int out_dtype, int out_stride, float scale, int window,
                                         int n_rows, int n_splits, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NB_REQUIRE(n_rows > 0 && n_heads > 0 && n_kv_heads > 0 && head_dim > 0 && n_splits > 0,
             NB_ERR_BAD_ARG, "attention_decode_static: sizes must be positive");
  long long acc_f = 0, ml_f = 0, cnt_i = 0;
  nb_attention_decode_scratch(n_rows, n_heads, n_kv_heads, head_dim, n_splits, &acc_f, &ml_f, &cnt_i);
  // layout: [counters | (max,sum) pairs | partial sums], each part rounded up to 256 bytes
  auto up = [](long long b) { return (b + 255) / 256 * 256; };
  const long long cnt_b = up(cnt_i * 4), ml_b = up(ml_f * 4), acc_b = up(acc_f * 4);
  NB_REQUIRE(cnt_b + ml_b + acc_b <= (long long)NB_STATIC_SCRATCH_BYTES, NB_ERR_UNSUPPORTED,
             "attention_decode_static: %d rows x %d heads x %d splits x head size %d need %lld "
             "bytes of scratch, the built-in array holds %lld; use fewer splits or "
             "nb_attention_decode with scratch of your own",
             n_rows, n_heads, n_splits, head_dim, cnt_b + ml_b + acc_b,
             (long long)NB_STATIC_SCRATCH_BYTES);
  unsigned char* base = nullptr;
  const int rc = static_scratch_address(&base, stream);
  if (rc) return rc;
  // the array keeps what the last call left; the counters are the only part that must start
  // at zero (a launch that ran to its end leaves them so, an interrupted one may not)
  NB_CUDA(cudaMemsetAsync(base, 0, (size_t)cnt_b, stream));
  // always through the scratch arrays: this entry point exists for them
  return attention_decode(q, dtype, q_stride, q_col, row_slot, row_pos, k_cache, v_cache,
                          block_table, max_pages, page, n_heads, n_kv_heads, head_dim, out,
                          out_dtype, out_stride, scale, 0.0f, nullptr, NbAttnOpts{window, 0, 0, nullptr, 0, 0}, n_rows,
                          n_splits, reinterpret_cast<float*>(base + cnt_b + ml_b),
                          reinterpret_cast<float*>(base + cnt_b),
                          reinterpret_cast<int*>(base), /*append=*/0, 0, 0,
                          /*clusters_allowed=*/0, stream);
}
