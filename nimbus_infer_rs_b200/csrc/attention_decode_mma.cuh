// The tensor-core decode kernel over a bf16 cache and its launcher: one query row per sequence (see
// attention_decode.cu, whose work this is; attention_decode_mixed.cu holds the variant for keys and
// values of different sizes).
#pragma once

#include "attention_common.cuh"

namespace {

constexpr int PAGE_TOKENS = 64;
constexpr int MAX_CLUSTER = 8;   // most splits that one thread-block cluster merges (portable size)

// ---------------------------------------------------------------------------------------
// Decode attention on the tensor cores, for a bf16 cache.  The CUDA-core kernel spends its
// time on instructions (widening every key and value, shuffles, a running softmax per four
// keys); here a warp's 16 keys of a page are one mma.sync operand: scores = K (16 keys x
// head_dim) times Q^T (head_dim x 8 query heads of the group, unused columns zero), then the
// value product out^T (head_dim x 8 heads) += V^T (head_dim x 16 keys) times P (16 keys x 8
// heads).  Softmax statistics stay fp32 per head (in units of log2 e); probabilities are
// rounded to bf16 only as the operand of the value product, as in the prefill kernel.  Pages
// are staged with padded rows so that ldmatrix runs without bank conflicts.  Any head size
// that is a multiple of 16 up to 128; up to 8 query heads per key/value head at no extra cost.
// ---------------------------------------------------------------------------------------
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], const void* p) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0,
                                          uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
      "{%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2_bf16(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&h);
}

// MMA_STAGES: pages (keys and values) in flight per CTA; NW: warps.  Four warps share a page
// (16 keys each).  A page costs a warp about 1,400 clocks of dependent steps (loads from
// shared memory, two rounds of tensor-core instructions with the softmax between them), so
// when the CTAs of a launch fit on the GPU with four pages each, eight warps take two pages
// at a time; a large batch has four warps and two pages per CTA, for more CTAs per SM.
// MAPS: differential heads (NbAttnOpts::maps).
// MIXED: keys of kv.head_dim and values of kv.value_dim numbers (multiples of 8, at most HD), each
// plane with its own pitch in memory, both staged in rows of HD; no append.
template <int HD, typename TOut, int MMA_STAGES, bool CLUSTERED, int NW, bool MAPS, bool MIXED>
__global__ void __launch_bounds__(NW * 32)
attention_decode_mma_kernel(const __nv_bfloat16* q, int q_stride, int q_col,
                            const int* row_slot, const int* row_pos,
                            NbPagedKV kv, int group, TOut* out, int out_stride,
                            float scale, float softcap, const float* sink, NbAttnOpts opt, int n_splits, float* part_acc,
                            float* part_ml, int* counters, int append,
                            int k_col, int v_col) {
  typedef __nv_bfloat16 bf16;
  constexpr bool clustered = CLUSTERED;
  constexpr int ROW = HD + 8;          // padded row of a staged page (elements)
  constexpr int KS = HD / 16;          // k-steps of the score product = row tiles of the value product
  constexpr int GH = 8;                // query heads an MMA column block holds
  constexpr int NT = NW * 32;          // threads
  constexpr int PPI = NW / 4;          // pages per turn of the loop
  static_assert((NW == 4 || NW == 8) && MMA_STAGES % PPI == 0, "four or eight warps");
  const int dk = MIXED ? kv.head_dim : HD, dv = MIXED ? kv.value_dim : HD;
  const int KTILE = PAGE_TOKENS * dk, VTILE = PAGE_TOKENS * dv;    // elements of one page of one head
  constexpr int STILE = PAGE_TOKENS * ROW;
  static_assert(HD % 16 == 0 && HD >= 16 && HD <= 128, "head size not supported");

  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* tiles = reinterpret_cast<bf16*>(smem_raw);                   // [stages][K | V][64][ROW]
  // the warps' partial results, after the last page has been read: over the page tiles
  // (more CTAs fit on an SM that way)
  float* w_acc = reinterpret_cast<float*>(smem_raw);                 // [NW][GH][HD]
  float* w_ml = w_acc + NW * GH * HD;                                // [NW][GH][2]
  static_assert((size_t)(NW * GH * HD + NW * GH * 2) * sizeof(float) <=
                    (size_t)2 * MMA_STAGES * STILE * sizeof(bf16), "partial results must fit in the page tiles");
  __shared__ int s_last;
  // clustered: the splits of a row and key-value head are one thread-block cluster (split =
  // rank); they hand their partial results to split 0 through its shared memory, in a region
  // of its own behind the page tiles, instead of through global memory and a counter
  float* c_part = reinterpret_cast<float*>(smem_raw + (size_t)2 * MMA_STAGES * STILE * sizeof(bf16));

  // Before the wait: where the row's pages lie, and its first pages on their way.  The batch
  // layout, the block table and the pages were written at least two kernels ago (earlier
  // steps, host copies); the only thing the kernel in front of this one writes is the step's
  // own rows (queries, and the new key and value, which are patched into the staged page
  // after the wait).
  const int split = blockIdx.x, kvh = blockIdx.y, r = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int wq = warp & 3, po = warp >> 2;   // quarter of a page, page of a turn
  const int n_heads = kv.n_kv_heads * group;
  const int slot = row_slot[r];
  if (slot < 0) {   // padding row: zeros, written by split 0
    nb_grid_dependency_wait();
    nb_launch_dependents();
    const int width = (MAPS ? group / 2 : group) * dv;
    if (split == 0)
      for (int i = tid; i < width; i += NT)
        out[(size_t)r * out_stride + (size_t)kvh * width + i] = nb_from_f32<TOut>(0.0f);
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
  const int* table = kv.block_table + (size_t)slot * kv.max_pages;
  const bf16* qrow = q + (size_t)r * q_stride;

  auto issue = [&](int page_idx, int stage) {
    const int page_id = table[page_idx];
    const bf16* ksrc = (const bf16*)kv.k + ((size_t)page_id * kv.n_kv_heads + kvh) * KTILE;
    const bf16* vsrc = (const bf16*)kv.v + ((size_t)page_id * kv.n_kv_heads + kvh) * VTILE;
    bf16* kdst = tiles + (size_t)stage * 2 * STILE;
    bf16* vdst = kdst + STILE;
    constexpr int CPR = HD / 8;   // 16-byte pieces per row
    if constexpr (MIXED) {
      for (int i = tid; i < PAGE_TOKENS * CPR; i += NT) {
        const int row = i / CPR, c = (i - row * CPR) * 8;
        if (c < dk) cp_async16(kdst + row * ROW + c, ksrc + row * dk + c);
        if (c < dv) cp_async16(vdst + row * ROW + c, vsrc + row * dv + c);
      }
    } else {
      for (int i = tid; i < PAGE_TOKENS * CPR; i += NT) {
        const int row = i / CPR, c = i - row * CPR;
        cp_async16(kdst + row * ROW + c * 8, ksrc + row * HD + c * 8);
        cp_async16(vdst + row * ROW + c * 8, vsrc + row * HD + c * 8);
      }
    }
  };
  if (MIXED && dk % 16 != 0)      // what the last k-step reads beyond a key: zeros (nothing else writes there)
    for (int i = tid; i < MMA_STAGES * PAGE_TOKENS; i += NT)
      *reinterpret_cast<uint4*>(tiles + (size_t)(i / PAGE_TOKENS) * 2 * STILE + (i % PAGE_TOKENS) * ROW + dk) =
          make_uint4(0u, 0u, 0u, 0u);
  // append < 0: the kernel in front of this one wrote the step's key and value into the cache
  // itself; no page may be asked for before it is done.
  if (append < 0) nb_grid_dependency_wait();
  // one commit group per stage of the ring, also an empty one: the count of groups in flight
  // then says which page has landed
#pragma unroll
  for (int i = 0; i < MMA_STAGES; ++i) {
    if (p_begin + i < p_end) issue(p_begin + i, i);
    cp_async_commit();
  }

  nb_grid_dependency_wait();
  // Every CTA of a cluster says that it runs (a padding row's CTAs have all left above); the
  // matching wait stands in front of the first store into another CTA's shared memory.
  if constexpr (clustered) asm volatile("barrier.cluster.arrive.relaxed.aligned;\n" ::: "memory");

  // Q^T as the B operand of the score product: column g of the block is query head g of the
  // group (zero beyond the group); this thread holds rows 2t, 2t+1 and 2t+8, 2t+9 of each k-step
  uint32_t qb[KS][2];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    qb[ks][0] = qb[ks][1] = 0u;
    if (MIXED) {
      const bf16* p = qrow + q_col + (size_t)(kvh * group + g) * dk + ks * 16 + 2 * t;
      if (g < group && ks * 16 < dk) qb[ks][0] = *reinterpret_cast<const uint32_t*>(p);
      if (g < group && ks * 16 + 8 < dk) qb[ks][1] = *reinterpret_cast<const uint32_t*>(p + 8);
    } else if (!MAPS && g < group) {
      const bf16* p = qrow + q_col + (size_t)(kvh * group + g) * HD + ks * 16 + 2 * t;
      qb[ks][0] = *reinterpret_cast<const uint32_t*>(p);
      qb[ks][1] = *reinterpret_cast<const uint32_t*>(p + 8);
    } else if (MAPS && g < group && (ks * 16 >= HD / 2) == ((g & 1) != 0)) {
      // a map's query meets its half of the key only: zeros against the other half
      const bf16* p = qrow + q_col + (size_t)(kvh * group + g) * (HD / 2) + ks * 16 -
                      (g & 1) * (HD / 2) + 2 * t;
      qb[ks][0] = *reinterpret_cast<const uint32_t*>(p);
      qb[ks][1] = *reinterpret_cast<const uint32_t*>(p + 8);
    }
  }

  // this thread's share: heads 2t and 2t+1; keys g and g+8 of the warp's 16; rows g, g+8 of
  // every 16-row tile of the output
  float o[KS][4];
#pragma unroll
  for (int i = 0; i < KS; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[i][j] = 0.0f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
  const float sl2 = (softcap > 0.0f ? 1.0f : scale) * 1.4426950408889634f;
  const float cap_in = softcap > 0.0f ? scale / softcap : 0.0f;

  int stage = 0;
  for (int p0 = p_begin; p0 < p_end; p0 += PPI) {
    cp_async_wait<MMA_STAGES - PPI>();   // all but the newest groups: the turn's pages are in
    __syncthreads();
#pragma unroll
    for (int q2 = 0; q2 < PPI; ++q2) {
    const int p = p0 + q2;
    if (p >= p_end) break;
    bf16* kt = tiles + (size_t)(stage + q2) * 2 * STILE;
    bf16* vt = kt + STILE;
    const bool own_page = !MIXED && append > 0 && p == pos / PAGE_TOKENS;
    const int tail_row = kv_len - p * PAGE_TOKENS;   // first row of the page that holds no key yet
    if (own_page || tail_row < PAGE_TOKENS) {        // uniform over the CTA
      constexpr int CPR = HD / 8;
      if (own_page) {
        // this step's own key and value belong at token `pos` of this page: into the staged
        // tile and into the cache
        const int in_page = pos % PAGE_TOKENS;
        const int page_id = table[p];
        for (int i = tid; i < 2 * CPR; i += NT) {
          const bool is_v = i >= CPR;
          const int c = (is_v ? i - CPR : i) * 8;
          const uint4 val = *reinterpret_cast<const uint4*>(
              qrow + (is_v ? v_col : k_col) + (size_t)kvh * HD + c);
          *reinterpret_cast<uint4*>((is_v ? vt : kt) + in_page * ROW + c) = val;
          bf16* cache = (bf16*)(is_v ? kv.v : kv.k);
          *reinterpret_cast<uint4*>(cache + ((size_t)page_id * kv.n_kv_heads + kvh) * KTILE +
                                    in_page * HD + c) = val;
        }
      }
      // Rows of the page after the sequence's last key hold whatever an earlier owner of the
      // page left there.  Their probabilities are zero, but zero times a non-finite value is
      // not: the value rows are cleared in the staged copy (a masked score needs no such care,
      // it is replaced, not multiplied).
      for (int i = tid; i < (PAGE_TOKENS - tail_row) * CPR; i += NT) {
        const int row = tail_row + i / CPR, c = (i % CPR) * 8;
        *reinterpret_cast<uint4*>(vt + row * ROW + c) = make_uint4(0u, 0u, 0u, 0u);
      }
      __syncthreads();
    }
    }
    const int p = p0 + po;                            // this warp's page
    bf16* kt = tiles + (size_t)(stage + po) * 2 * STILE;
    bf16* vt = kt + STILE;
    const int key0 = p * PAGE_TOKENS + wq * 16;       // first key of this warp's 16
    if (p < p_end && key0 < kv_len && (key0 + 16 > j_begin || key0 < keep_first)) {   // warp-uniform: something to attend to
      // the k-steps of the score product in accumulators of their own, added up afterwards:
      // a tensor-core instruction takes long to hand its result to the next one
      float sck[KS < 4 ? KS : 4][4];
#pragma unroll
      for (int i = 0; i < (KS < 4 ? KS : 4); ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) sck[i][j] = 0.0f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        if (MIXED && ks * 16 >= dk) break;
        uint32_t ka[4];
        ldsm_x4(ka, kt + (wq * 16 + (lane & 15)) * ROW + ks * 16 + (lane >> 4) * 8);
        mma_16816(sck[ks & 3], ka, qb[ks][0], qb[ks][1]);
      }
      float sc[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float a = sck[0][j];
#pragma unroll
        for (int i = 1; i < (KS < 4 ? KS : 4); ++i) a += sck[i][j];
        sc[j] = a;
      }
      const int ja = key0 + g, jb = ja + 8;
      const bool va = (ja >= j_begin || ja < keep_first) && ja < kv_len,
                 vb = (jb >= j_begin || jb < keep_first) && jb < kv_len;
      if (softcap > 0.0f) {   // uniform: capped scores carry their scale already
#pragma unroll
        for (int j = 0; j < 4; ++j) sc[j] = nb_softcap(sc[j], cap_in, softcap);
      }
      const float s0 = va ? sc[0] * sl2 : -INFINITY, s1 = va ? sc[1] * sl2 : -INFINITY;
      const float s2 = vb ? sc[2] * sl2 : -INFINITY, s3 = vb ? sc[3] * sl2 : -INFINITY;
      float mx0 = fmaxf(s0, s2), mx1 = fmaxf(s1, s3);
#pragma unroll
      for (int off = 4; off < 32; off <<= 1) {
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, off));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, off));
      }
      const float mn0 = fmaxf(m_run[0], mx0), mn1 = fmaxf(m_run[1], mx1);   // finite: a key is valid
      const float r0 = (m_run[0] == -INFINITY) ? 0.0f : nb_exp2(m_run[0] - mn0);
      const float r1 = (m_run[1] == -INFINITY) ? 0.0f : nb_exp2(m_run[1] - mn1);
      m_run[0] = mn0;
      m_run[1] = mn1;
      const float p0 = nb_exp2(s0 - mn0), p1 = nb_exp2(s1 - mn1);
      const float p2 = nb_exp2(s2 - mn0), p3 = nb_exp2(s3 - mn1);
      l_run[0] = l_run[0] * r0 + p0 + p2;
      l_run[1] = l_run[1] * r1 + p1 + p3;
#pragma unroll
      for (int i = 0; i < KS; ++i) {
        o[i][0] *= r0; o[i][1] *= r1; o[i][2] *= r0; o[i][3] *= r1;
      }
      // P as the B operand of the value product: this thread needs keys 2t, 2t+1 (and +8) of
      // head g; they sit in lanes (g' = 2t, t' = g/2) and (g' = 2t+1, t' = g/2)
      const uint32_t pe = pack2_bf16(p0, p2);   // head 2t:   keys g, g+8
      const uint32_t po = pack2_bf16(p1, p3);   // head 2t+1: keys g, g+8
      const int src1 = (2 * t) * 4 + (g >> 1), src2 = src1 + 4;
      const uint32_t e1 = __shfl_sync(0xffffffffu, pe, src1), o1 = __shfl_sync(0xffffffffu, po, src1);
      const uint32_t e2 = __shfl_sync(0xffffffffu, pe, src2), o2 = __shfl_sync(0xffffffffu, po, src2);
      const uint32_t x1 = (g & 1) ? o1 : e1, x2 = (g & 1) ? o2 : e2;
      const uint32_t pb0 = __byte_perm(x1, x2, 0x5410);   // keys 2t, 2t+1
      const uint32_t pb1 = __byte_perm(x1, x2, 0x7632);   // keys 2t+8, 2t+9
#pragma unroll
      for (int i = 0; i < KS; ++i) {
        if (MIXED && i * 16 >= dv) break;
        uint32_t va4[4];
        ldsm_x4_trans(va4, vt + (wq * 16 + (lane & 7) + (lane >> 4) * 8) * ROW + i * 16 +
                               ((lane >> 3) & 1) * 8);
        mma_16816(o[i], va4, pb0, pb1);
      }
    }
    __syncthreads();   // the stages are free: the pages after the ones in flight go there
#pragma unroll
    for (int q2 = 0; q2 < PPI; ++q2) {
      if (p0 + q2 + MMA_STAGES < p_end) issue(p0 + q2 + MMA_STAGES, stage + q2);
      cp_async_commit();
    }
    stage += PPI;
    if (stage == MMA_STAGES) stage = 0;
  }
  cp_async_wait<0>();

  nb_launch_dependents();   // the pages are read: the next kernel may be set up
  // row sums over the lanes that share a head (different keys), then the warps
#pragma unroll
  for (int off = 4; off < 32; off <<= 1) {
    l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], off);
    l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], off);
  }
#pragma unroll
  for (int i = 0; i < KS; ++i) {
    float* base = w_acc + (size_t)warp * GH * HD;
    base[(2 * t) * HD + i * 16 + g] = o[i][0];
    base[(2 * t + 1) * HD + i * 16 + g] = o[i][1];
    base[(2 * t) * HD + i * 16 + g + 8] = o[i][2];
    base[(2 * t + 1) * HD + i * 16 + g + 8] = o[i][3];
  }
  if (g == 0) {
    w_ml[(warp * GH + 2 * t) * 2] = m_run[0];
    w_ml[(warp * GH + 2 * t) * 2 + 1] = l_run[0];
    w_ml[(warp * GH + 2 * t + 1) * 2] = m_run[1];
    w_ml[(warp * GH + 2 * t + 1) * 2 + 1] = l_run[1];
  }
  __syncthreads();
  // merge the warps -> partial result of this split (maxima in units of log2 e)
  // A finished number of a head's result: to its place in the output or, with two maps a head, to
  // shared memory, where `finish_maps` takes the heads' differences.  (A thread overwrites only
  // what it alone has read.)
  auto emit = [&](int gh, int c, float v) {
    if constexpr (MAPS)
      w_acc[gh * HD + c] = v;
    else
      out[(size_t)r * out_stride + (size_t)(kvh * group + gh) * dv + c] = nb_from_f32<TOut>(v);
  };
  auto finish_maps = [&]() {
    if constexpr (!MAPS) return;
    __syncthreads();
    for (int hh = warp; hh < group / 2; hh += NW) {
      const float* a1 = w_acc + (size_t)2 * hh * HD;
      float u[(HD + 31) / 32], ss = 0.0f;
#pragma unroll
      for (int k = 0; k < (HD + 31) / 32; ++k) {
        const int c = lane + 32 * k;
        u[k] = c < HD ? a1[c] - opt.lambda * a1[HD + c] : 0.0f;
        ss = fmaf(u[k], u[k], ss);
      }
      const float f = opt.factor / sqrtf(nb_warp_sum(ss) / (float)HD + opt.eps);
      TOut* dst = out + (size_t)r * out_stride + (size_t)(kvh * (group / 2) + hh) * HD;
#pragma unroll
      for (int k = 0; k < (HD + 31) / 32; ++k)
        if (lane + 32 * k < HD) dst[lane + 32 * k] = nb_from_f32<TOut>(u[k] * f);
    }
  };
  unsigned c_remote = 0;    // this split's place in split 0's shared memory
  if constexpr (clustered) {
    asm volatile("barrier.cluster.wait.aligned;\n" ::: "memory");
    const unsigned local = (unsigned)__cvta_generic_to_shared(c_part + (size_t)split * group * (HD + 2));
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(c_remote) : "r"(local), "r"(0));
  }
  for (int i = tid; i < group * HD; i += NT) {
    const int gh = i / HD, c = i - gh * HD;
    if (MIXED && c >= dv) continue;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < NW; ++w) M = fmaxf(M, w_ml[(w * GH + gh) * 2]);
    float a = 0.0f, l = 0.0f;
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      const float mw = w_ml[(w * GH + gh) * 2];
      const float f = (mw == -INFINITY) ? 0.0f : nb_exp2(mw - M);
      a += f * w_acc[(w * GH + gh) * HD + c];
      l += f * w_ml[(w * GH + gh) * 2 + 1];
    }
    const int head = kvh * group + gh;
    if (n_splits == 1) {
      if (sink != nullptr) a *= nb_sink_fix(l, M, sink[head], true);
      a *= opt.gate_of(r, head);
      emit(gh, c, l > 0.0f ? a / l : a);
      continue;
    }
    if constexpr (clustered) {
      const unsigned at = c_remote + (unsigned)(gh * (HD + 2)) * 4u;
      asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(at + (unsigned)c * 4u), "f"(a) : "memory");
      if (c == 0) {
        asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(at + (unsigned)HD * 4u), "f"(M) : "memory");
        asm volatile("st.shared::cluster.f32 [%0], %1;\n" ::"r"(at + (unsigned)(HD + 1) * 4u), "f"(l) : "memory");
      }
      continue;
    }
    const size_t pi = ((size_t)r * n_heads + head) * n_splits + split;
    part_acc[pi * HD + c] = a;
    if (c == 0) {
      part_ml[pi * 2] = M;
      part_ml[pi * 2 + 1] = l;
    }
  }
  if (n_splits == 1) {
    finish_maps();
    return;
  }
  if constexpr (clustered) {
    // the stores above are visible to split 0 once every CTA has arrived (release) and split 0
    // has waited (acquire); the other splits wait too, so that none leaves the cluster early
    asm volatile("barrier.cluster.arrive.release.aligned;\n" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
    if (split != 0) return;
    for (int i = tid; i < group * HD; i += NT) {
      const int gh = i / HD, c = i - gh * HD;
      if (MIXED && c >= dv) continue;
      const float* row = c_part + (size_t)gh * (HD + 2);
      const int step = group * (HD + 2);
      float M = -INFINITY;
      for (int s = 0; s < n_splits; ++s) M = fmaxf(M, row[s * step + HD]);
      float a = 0.0f, l = 0.0f;
      for (int s = 0; s < n_splits; ++s) {
        const float ms = row[s * step + HD];
        const float f = (ms == -INFINITY) ? 0.0f : nb_exp2(ms - M);
        a += f * row[s * step + c];
        l += f * row[s * step + HD + 1];
      }
      if (sink != nullptr) a *= nb_sink_fix(l, M, sink[kvh * group + gh], true);
      a *= opt.gate_of(r, kvh * group + gh);
      emit(gh, c, l > 0.0f ? a / l : a);
    }
    finish_maps();
    return;
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const int old = atomicAdd(&counters[r * kv.n_kv_heads + kvh], 1);
    s_last = (old == n_splits - 1);
    if (s_last) counters[r * kv.n_kv_heads + kvh] = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int i = tid; i < group * HD; i += NT) {
    const int gh = i / HD, c = i - gh * HD;
    if (MIXED && c >= dv) continue;
    const int head = kvh * group + gh;
    const size_t base = ((size_t)r * n_heads + head) * n_splits;
    // eight splits at a time, everything asked for before anything is used: one trip to L2
    // for the maxima, the sums and the partial results together
    float M = -INFINITY, a = 0.0f, l = 0.0f;
    for (int s0 = 0; s0 < n_splits; s0 += 8) {
      float2 ml8[8];
      float acc8[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const bool in = s0 + j < n_splits;
        ml8[j] = in ? __ldcg(reinterpret_cast<const float2*>(part_ml + (base + s0 + j) * 2))
                    : make_float2(-INFINITY, 0.0f);
        acc8[j] = in ? __ldcg(&part_acc[(base + s0 + j) * HD + c]) : 0.0f;
      }
      float Mn = M;
#pragma unroll
      for (int j = 0; j < 8; ++j) Mn = fmaxf(Mn, ml8[j].x);
      const float keep = (M == -INFINITY) ? 0.0f : nb_exp2(M - Mn);
      a *= keep;
      l *= keep;
#pragma unroll
      for (int j = 0; j < 8; ++j) {   // in split order
        const float f = (ml8[j].x == -INFINITY) ? 0.0f : nb_exp2(ml8[j].x - Mn);
        a += f * acc8[j];
        l += f * ml8[j].y;
      }
      M = Mn;
    }
    if (sink != nullptr) a *= nb_sink_fix(l, M, sink[head], true);
    a *= opt.gate_of(r, head);
    emit(gh, c, l > 0.0f ? a / l : a);
  }
  finish_maps();
}

template <int HD, typename TOut, int MMA_STAGES, int NW, bool MAPS, bool MIXED>
int launch_mma_s(const void* q, int q_stride, int q_col, const int* row_slot, const int* row_pos,
                 const NbPagedKV& kv, int group, void* out, int out_stride, float scale, float softcap, const float* sink, NbAttnOpts opt,
                 int n_rows, int n_splits, float* part_acc, float* part_ml, int* counters, int append,
                 int k_col, int v_col, bool clustered, cudaStream_t stream) {
  const size_t tiles = (size_t)2 * MMA_STAGES * PAGE_TOKENS * (HD + 8) * sizeof(__nv_bfloat16);
  // room for the splits' partial results in split 0's shared memory (see the kernel)
  const size_t most = tiles + (size_t)MAX_CLUSTER * 8 * (HD + 2) * sizeof(float);
  dim3 grid(n_splits, kv.n_kv_heads, n_rows);
  if (clustered) {
    auto kern = attention_decode_mma_kernel<HD, TOut, MMA_STAGES, true, NW, MAPS, MIXED>;
    static bool configured = false;   // per instantiation
    if (most > 48 * 1024 && !configured) {
      NB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most));
      configured = true;
    }
    const size_t smem = tiles + (size_t)n_splits * group * (HD + 2) * sizeof(float);
    NB_CUDA(nb_launch_clusters(kern, grid, dim3(NW * 32), smem, stream, n_splits,
                               (const __nv_bfloat16*)q, q_stride, q_col, row_slot, row_pos, kv, group,
                               (TOut*)out, out_stride, scale, softcap, sink, opt, n_splits, part_acc, part_ml,
                               counters, append, k_col, v_col));
    return 0;
  }
  auto kern = attention_decode_mma_kernel<HD, TOut, MMA_STAGES, false, NW, MAPS, MIXED>;
  static bool configured = false;   // per instantiation
  if (tiles > 48 * 1024 && !configured) {
    NB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tiles));
    configured = true;
  }
  NB_CUDA(nb_launch(kern, grid, dim3(NW * 32), tiles, stream, (const __nv_bfloat16*)q, q_stride, q_col,
                    row_slot, row_pos, kv, group, (TOut*)out, out_stride, scale, softcap, sink, opt, n_splits,
                    part_acc, part_ml, counters, append, k_col, v_col));
  return 0;
}

template <int HD, typename TOut, bool MAPS, bool MIXED>
int launch_mma(const void* q, int q_stride, int q_col, const int* row_slot, const int* row_pos,
               const NbPagedKV& kv, int group, void* out, int out_stride, float scale, float softcap, const float* sink, NbAttnOpts opt,
               int n_rows, int n_splits, float* part_acc, float* part_ml, int* counters, int append,
               int k_col, int v_col, bool clustered, cudaStream_t stream) {
  static int sms = 0;
  if (sms == 0) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess ||
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0)
      sms = 148;
  }
  // Eight warps and four pages in flight per CTA when the whole launch fits on the GPU that
  // way (an SM has 228 KB of shared memory, a CTA costs its own and 1 KB), else four warps and
  // two pages, for more CTAs per SM.
  const size_t smem4 = (size_t)8 * PAGE_TOKENS * (HD + 8) * sizeof(__nv_bfloat16) +
                       (clustered ? (size_t)n_splits * group * (HD + 2) * sizeof(float) : 0);
  const long long ctas = (long long)n_splits * kv.n_kv_heads * n_rows;
  long long per_sm = (long long)((228 * 1024) / (smem4 + 1024));
  if (per_sm > 8) per_sm = 8;   // 2,048 threads an SM
  if (ctas <= per_sm * sms)
    return launch_mma_s<HD, TOut, 4, 8, MAPS, MIXED>(q, q_stride, q_col, row_slot, row_pos, kv, group, out, out_stride,
                                        scale, softcap, sink, opt, n_rows, n_splits, part_acc, part_ml, counters,
                                        append, k_col, v_col, clustered, stream);
  return launch_mma_s<HD, TOut, 2, 4, MAPS, MIXED>(q, q_stride, q_col, row_slot, row_pos, kv, group, out, out_stride,
                                      scale, softcap, sink, opt, n_rows, n_splits, part_acc, part_ml, counters, append,
                                      k_col, v_col, clustered, stream);
}

}  // namespace
