// Differential attention of prompts on the 5th-generation tensor cores (sm_100a): heads whose two
// maps hold d = 32 or 64 numbers each over values of 2 d, bf16 operands, fp32 scores, softmax,
// difference and norm (see attention_differential.cu for the equations and the layouts).
//
// One CTA takes 128 consecutive query rows of one sequence and one head; a row of the tile is a
// lane of tensor memory.  Warp 0 is the producer: one thread brings the query tile and then the
// pages' keys (both maps side by side) and values, two pages (128 keys) at a time, into a ring of
// stages with TMA.  Warp 1 issues the products in turns: turn i = (page pair i / 2, map i % 2) is
// S_a = Q_a K_a^T (M=128, N=128, K=d: the map's own columns of the query and key tiles) into the
// map's score columns, and O_a += P_a V (M=128, N=2d, K=128), whose A operand is what the softmax
// wrote over the scores.  Both maps' turns read the same staged values.  The outputs of both maps
// stay in tensor memory for the whole walk (2 x 2d columns beside 2 x 128 score columns).
//
// Warps 2..9 are the softmax, two threads per row (one of the two pages of a turn each, and half
// of the head's columns at the end).  The reference that exponents are taken against is moved only
// when a row's maximum has grown by more than 2^REF_SLACK over it: then the eight warps' threads
// rescale their part of O_a in tensor memory before they hand over P_a.  No barrier guards that:
// the score product of a turn is issued behind the value product of the same map's turn before,
// and MMAs complete in order, so whoever has seen S_a complete finds O_a at rest until P_a is
// handed over.  While one map's turn is in the softmax the other map's products run.
//
// Every wait on an mbarrier is bounded by a clock budget; a wait that runs out raises an error
// word, and the CTA ends after its copies have landed and its tensor memory is freed.
#include "attention_common.cuh"
#include "tc05_common.cuh"

namespace {

typedef __nv_bfloat16 bf16;

constexpr int TILE_Q = 128;
constexpr int PAGE_TOKENS = 64;
constexpr int TC_THREADS = 320;      // producer, MMA issuer, eight softmax warps
constexpr float REF_SLACK = 8.0f;    // in log2: probabilities stay below 2^8

__host__ __device__ constexpr uint32_t instr_desc_bf16_b_mn(int m, int n) {
  return instr_desc_bf16(m, n) | (1u << 16);      // MN-major B operand
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(bar) : "memory");
}
// D (tensor memory) += A (tensor memory, bf16 packed two per column) * B (shared memory)
__device__ __forceinline__ void tc05_mma_bf16_a_tmem(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b,
                                                     uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %6, %7, %8}, p;\n\t}\n" ::"r"(tmem_d),
      "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u), "r"(0u), "r"(0u), "r"(0u)
      : "memory");
}
__device__ __forceinline__ void tc05_st_32x32b_x32(uint32_t taddr, const uint32_t (&v)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, %20, "
      "%21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};\n" ::"r"(taddr),
      "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]),
      "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]),
      "r"(v[16]), "r"(v[17]), "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]),
      "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
      : "memory");
}
__device__ __forceinline__ void tc05_wait_st() {
  asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
}

template <int HD>   // a key head: two maps of HD / 2; a value head: HD
struct DiffSmem {
  static constexpr int HB = HD / 64;                      // 64-column boxes per row of a head
  static constexpr int Q_BYTES = TILE_Q * 128 * HB;       // [HB][128 rows][128 B]
  static constexpr int PAGE_BOX = PAGE_TOKENS * 128;      // one page, 64 head columns: 8 KB
  static constexpr int K_BYTES = 2 * PAGE_BOX * HB;       // [HB][2 pages][64 keys][128 B]
  static constexpr int STAGE_BYTES = 2 * K_BYTES;         // keys, then values
  static constexpr int STAGES = HD == 64 ? 4 : 2;
  static constexpr int TILES_BYTES = Q_BYTES + STAGES * STAGE_BYTES;
  // q_full, kv_full[S], kv_empty[S], s_full[2], p_full[2], o_done
  static constexpr int N_BARRIERS = 2 * STAGES + 6;
  static constexpr int XCH_BYTES = 8 * TILE_Q * 4;        // row maxima and sums, per map and half
  static constexpr int TOTAL = TILES_BYTES + N_BARRIERS * 8 + 16 + XCH_BYTES + 1024 /* alignment slack */;
  // tensor memory columns: the maps' scores (the probabilities of a turn take the first 64 of
  // them), the maps' outputs
  static constexpr int S_COL = 0, O_COL = 256, TMEM_COLS = 512;
};

template <int HD>
__global__ void __launch_bounds__(TC_THREADS, 1)
differential_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                       const __grid_constant__ CUtensorMap map_k,
                       const __grid_constant__ CUtensorMap map_v, const int* cu_rows,
                       const int* seq_slot, const int* seq_pos0, const int* block_table, int max_pages,
                       int n_kv_heads, int group, bf16* out, int out_stride, float scale_log2,
                       int window, float lambda, float factor, float eps, int* err_word) {
  using L = DiffSmem<HD>;
  constexpr int HB = L::HB, KM = HD / 32;     // boxes of a head, k-steps of a map's score product
  extern __shared__ unsigned char smem_dyn[];
  const uint32_t raw = smem_u32(smem_dyn);
  const uint32_t base = (raw + 1023u) & ~1023u;
  unsigned char* gen = smem_dyn + (base - raw);
  const uint32_t q_smem = base, kv_smem = base + L::Q_BYTES, bars = base + L::TILES_BYTES;
  const uint32_t q_full = bars;
  auto kv_full = [&](int s) { return bars + 8u * (1 + s); };
  auto kv_empty = [&](int s) { return bars + 8u * (1 + L::STAGES + s); };
  auto s_full = [&](int a) { return bars + 8u * (1 + 2 * L::STAGES + a); };
  auto p_full = [&](int a) { return bars + 8u * (3 + 2 * L::STAGES + a); };
  const uint32_t o_done = bars + 8u * (5 + 2 * L::STAGES);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(gen + L::TILES_BYTES + L::N_BARRIERS * 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* xch = reinterpret_cast<float*>(tmem_slot + 4);   // [maxima, sums][2 maps][2 halves][128 rows]

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // the last tiles (which see most keys when there is no window) start first
  const int linear = (int)blockIdx.x + (int)gridDim.x * ((int)blockIdx.y + (int)gridDim.y * (int)blockIdx.z);
  const int per_tile = (int)gridDim.y * (int)gridDim.z;
  const int tile = (int)gridDim.x - 1 - linear / per_tile;
  const int h = (linear % per_tile) % (int)gridDim.y, s = (linear % per_tile) / (int)gridDim.y;
  const int row0 = cu_rows[s], n_q = cu_rows[s + 1] - row0;
  const int q0 = tile * TILE_Q;
  const int slot = seq_slot[s];
  // (a CTA that leaves waits for the kernel before this one all the same: a grid that ended
  // early would let the kernel after it overtake that one)
  if (q0 >= n_q || slot < 0) {                // the whole CTA leaves: nothing is allocated yet
    nb_grid_dependency_wait();
    return;
  }
  const int pos0 = seq_pos0[s];
  const int kvh = h / group;
  const int rows_here = min(TILE_Q, n_q - q0);
  const int last_pos = pos0 + q0 + rows_here - 1;                    // newest key any row sees
  const int first_key = window > 0 ? max(0, pos0 + q0 + 1 - window) : 0;
  const int p_begin = first_key / PAGE_TOKENS, p_end = last_pos / PAGE_TOKENS + 1;
  const int nb = (p_end - p_begin + 1) / 2;             // pairs of pages
  const int tail_row = last_pos % PAGE_TOKENS + 1;      // first row of the last page without a key
  auto two_pages = [&](int j) { return p_begin + 2 * j + 1 < p_end; };
  const int* table = block_table + (size_t)slot * max_pages;

  if (tid == 0) {
    prefetch_tensormap(&map_q);
    prefetch_tensormap(&map_k);
    prefetch_tensormap(&map_v);
    mbar_init(q_full, 1);
    for (int i = 0; i < L::STAGES; ++i) {
      mbar_init(kv_full(i), 1);
      mbar_init(kv_empty(i), 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(s_full(a), 1);
      mbar_init(p_full(a), 8);     // one arrival per softmax warp
    }
    mbar_init(o_done, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    fence_async_smem();
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(
                     smem_u32(tmem_slot)),
                 "r"((uint32_t)L::TMEM_COLS)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  tc05_fence_before();
  __syncthreads();
  tc05_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  // the batch layout and the block table are older than the kernel before this one, which wrote
  // the queries and the step's keys and values
  nb_grid_dependency_wait();

  if (warp == 0) {
    if (lane == 0) {   // ------------------------------------------------------ TMA producer
      mbar_expect_tx(q_full, L::Q_BYTES);
#pragma unroll
      for (int b = 0; b < HB; ++b)
        tma_load_2d(q_smem + b * (TILE_Q * 128), &map_q, h * HD + b * 64, row0 + q0, q_full);
      for (int j = 0; j < nb; ++j) {
        const int st = j % L::STAGES, pa = p_begin + 2 * j;
        const bool two = two_pages(j);
        const int row_a = (table[pa] * n_kv_heads + kvh) * PAGE_TOKENS;
        const int row_b = two ? (table[pa + 1] * n_kv_heads + kvh) * PAGE_TOKENS : 0;
        if (!mbar_wait(kv_empty(st), ((j / L::STAGES) & 1u) ^ 1u, abort_flag)) break;
        mbar_expect_tx(kv_full(st), two ? L::STAGE_BYTES : L::STAGE_BYTES / 2);
#pragma unroll
        for (int b = 0; b < HB; ++b) {
          const uint32_t kb = kv_smem + st * L::STAGE_BYTES + b * (2 * L::PAGE_BOX), vb = kb + L::K_BYTES;
          tma_load_2d(kb, &map_k, b * 64, row_a, kv_full(st));
          tma_load_2d(vb, &map_v, b * 64, row_a, kv_full(st));
          if (two) {
            tma_load_2d(kb + L::PAGE_BOX, &map_k, b * 64, row_b, kv_full(st));
            tma_load_2d(vb + L::PAGE_BOX, &map_v, b * 64, row_b, kv_full(st));
          }
        }
      }
      nb_launch_dependents();        // all loads are on their way: the next kernel may be set up
    }
  } else if (warp == 1) {
    if (lane == 0) {   // ------------------------------------------------------ MMA issuer
      constexpr uint32_t idesc_s2 = instr_desc_bf16(TILE_Q, 2 * PAGE_TOKENS);   // two pages of keys
      constexpr uint32_t idesc_s1 = instr_desc_bf16(TILE_Q, PAGE_TOKENS);       // one
      constexpr uint32_t idesc_o = instr_desc_bf16_b_mn(TILE_Q, HD);
      bool ok = mbar_wait(q_full, 0u, abort_flag);
      tc05_fence_after();
      auto value_product = [&](int i) -> bool {
        const int a = i & 1, j = i >> 1, st = j % L::STAGES;
        if (!mbar_wait(p_full(a), j & 1u, abort_flag)) return false;
        tc05_fence_after();
        const uint32_t v_addr = kv_smem + st * L::STAGE_BYTES + L::K_BYTES;
        const uint32_t a_tmem = tmem_base + L::S_COL + a * (2 * PAGE_TOKENS);
        const uint32_t d_tmem = tmem_base + L::O_COL + a * HD;
        const int k_steps = two_pages(j) ? 8 : 4;
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (k < k_steps) {
            const uint64_t db = smem_desc_sw128_mn(v_addr + (k >> 2) * L::PAGE_BOX + (k & 3) * 2048u,
                                                   2 * L::PAGE_BOX, 1024u);
            tc05_mma_bf16_a_tmem(d_tmem, a_tmem + k * 8, db, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
          }
        }
        if (a == 1) tc05_commit(kv_empty(st));     // both maps have read the stage
        return true;
      };
      for (int i = 0; i < 2 * nb && ok; ++i) {
        const int a = i & 1, j = i >> 1, st = j % L::STAGES;
        if (a == 0) {
          ok = mbar_wait(kv_full(st), (j / L::STAGES) & 1u, abort_flag);
          if (!ok) break;
          tc05_fence_after();
        }
        const uint32_t k_addr = kv_smem + st * L::STAGE_BYTES;
        const uint32_t d_tmem = tmem_base + L::S_COL + a * (2 * PAGE_TOKENS);
        const uint32_t idesc_s = two_pages(j) ? idesc_s2 : idesc_s1;
#pragma unroll
        for (int k = 0; k < KM; ++k) {
          // the map's columns: 16 per MMA, 32 bytes inside a 64-column box
          const uint32_t step = a * KM + k, box = step >> 2, in_box = (step & 3) * 2;
          const uint64_t da = smem_desc_sw128(q_smem + box * (TILE_Q * 128)) + in_box;
          const uint64_t db = smem_desc_sw128(k_addr + box * (2 * L::PAGE_BOX)) + in_box;
          tc05_mma_bf16(d_tmem, da, db, idesc_s, k > 0 ? 1u : 0u);
        }
        tc05_commit(s_full(a));
        if (i > 0) ok = value_product(i - 1);
      }
      if (ok && value_product(2 * nb - 1)) tc05_commit(o_done);
    }
  } else {             // ------------------------------------------------------ softmax
    // A thread that has seen a wait run out goes on through the loop without touching tensor
    // memory, so that its partner never waits for it at the barrier.
    const int quarter = warp & 3;              // the 32 tensor-memory lanes this warp may read
    const int half = (warp - 2) >> 2;
    const int r = quarter * 32 + lane;         // row of the tile
    const int qpos = pos0 + q0 + r;            // absolute position of this row's query
    const int row_first = window > 0 ? max(0, qpos + 1 - window) : 0;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(quarter * 32) << 16);
    constexpr int OC = HD / 2;                 // output columns of this thread
    float m_ref[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    bool ok = true;
    auto pair_barrier = [&]() {   // the two warps of a quarter; barrier numbers 1..4
      asm volatile("bar.sync %0, 64;\n" ::"r"(quarter + 1) : "memory");
    };
    auto warp_wait = [&](uint32_t bar, uint32_t parity) -> bool {   // one lane polls for the warp
      int got = 1;
      if (lane == 0) got = (int)mbar_wait(bar, parity, abort_flag);
      return __shfl_sync(0xffffffffu, got, 0) != 0;
    };

    for (int j = 0; j < nb; ++j) {
      const bool has_keys = half == 0 || two_pages(j);   // the last pair may be one page only
      // bit e of `vis`: key k0 + e counts for this row
      const int k0 = (p_begin + 2 * j + half) * PAGE_TOKENS;
      const bool all_visible = window <= 0 && two_pages(j) &&
                               (p_begin + 2 * j + 2) * PAGE_TOKENS - 1 <= pos0 + q0 + quarter * 32;
      unsigned long long vis = 0ull;
      if (has_keys) {
        const int hi = qpos - k0, lo = row_first - k0;
        const unsigned long long up = hi >= 63 ? ~0ull : (hi < 0 ? 0ull : ((2ull << hi) - 1ull));
        const unsigned long long dn = lo <= 0 ? ~0ull : (lo > 63 ? 0ull : (~0ull << lo));
        vis = up & dn;
      }
#pragma unroll
      for (int a = 0; a < 2; ++a) {
        const uint32_t s_addr = lane_addr + L::S_COL + a * (2 * PAGE_TOKENS);
        uint32_t v0[32], v1[32];
        if (ok) ok = warp_wait(s_full(a), j & 1u);
        if (ok && has_keys) {
          tc05_fence_after();
          tc05_ld_32x32b_x32(s_addr + half * PAGE_TOKENS, v0);
          tc05_ld_32x32b_x32(s_addr + half * PAGE_TOKENS + 32, v1);
          tc05_wait_ld();
        } else {
#pragma unroll
          for (int e = 0; e < 32; ++e) v0[e] = v1[e] = 0u;
        }
        // the scale is positive (the launcher sees to it): the maximum is taken over the raw
        // scores, and the scaling is folded into the exponent
        float x[64], mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        if (all_visible) {
#pragma unroll
          for (int e = 0; e < 64; ++e) {
            x[e] = __uint_as_float(e < 32 ? v0[e] : v1[e - 32]);
            mx4[e & 3] = fmaxf(mx4[e & 3], x[e]);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 64; ++e) {
            x[e] = ((vis >> e) & 1ull) ? __uint_as_float(e < 32 ? v0[e] : v1[e - 32]) : -INFINITY;
            mx4[e & 3] = fmaxf(mx4[e & 3], x[e]);
          }
        }
        float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
        xch[(a * 2 + half) * TILE_Q + r] = mx;
        pair_barrier();   // also: both halves have read their scores, which the probabilities overwrite
        mx = fmaxf(mx, xch[(a * 2 + (half ^ 1)) * TILE_Q + r]);
        // move the reference only when the maximum has outgrown it (never for a row that has
        // seen nothing yet: its sum and outputs are zero)
        const bool grown = m_ref[a] > -INFINITY && mx > m_ref[a] + REF_SLACK;
        const float f = grown ? nb_exp2(m_ref[a] - mx) : 1.0f;
        if (grown || m_ref[a] == -INFINITY) m_ref[a] = mx;
        l_run[a] *= f;
        if (__any_sync(0xffffffffu, grown) && ok && j > 0) {
#pragma unroll
          for (int c = 0; c < OC / 32; ++c) {
            const uint32_t o_addr = lane_addr + L::O_COL + a * HD + half * OC + c * 32;
            tc05_ld_32x32b_x32(o_addr, v0);
            tc05_wait_ld();
#pragma unroll
            for (int e = 0; e < 32; ++e) v0[e] = __float_as_uint(__uint_as_float(v0[e]) * f);
            tc05_st_32x32b_x32(o_addr, v0);
          }
          tc05_wait_st();
        }
        const float m_use = m_ref[a] == -INFINITY ? 0.0f : m_ref[a];
        float sum4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        uint32_t pk[32];
#pragma unroll
        for (int e = 0; e < 32; ++e) {
          const float p0 = nb_exp2(fmaf(x[2 * e], scale_log2, -m_use));
          const float p1 = nb_exp2(fmaf(x[2 * e + 1], scale_log2, -m_use));
          sum4[e & 3] += p0 + p1;
          const __nv_bfloat162 hh = __floats2bfloat162_rn(p0, p1);
          pk[e] = *reinterpret_cast<const uint32_t*>(&hh);
        }
        l_run[a] += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
        if (ok) {
          if (has_keys) {   // this thread's probabilities: 64 bf16 = 32 columns, over the scores
            tc05_st_32x32b_x32(s_addr + half * 32, pk);
            tc05_wait_st();
          }
          if (a == 0 && j == nb - 1 && tail_row < PAGE_TOKENS) {
            // Rows of the sequence's last page after its newest key hold whatever an earlier owner
            // of the page left there.  Their probabilities are zero, but zero times a non-finite
            // value is not: the softmax warps clear those value rows in the staged page before
            // the first value product that reads them may start.  A row is 128 bytes inside each
            // 64-column box, whatever the swizzle does within it.
            unsigned char* vpage = gen + L::Q_BYTES + (j % L::STAGES) * L::STAGE_BYTES + L::K_BYTES +
                                   ((p_end - 1) - (p_begin + 2 * j)) * L::PAGE_BOX;
            const int per_box = (PAGE_TOKENS - tail_row) * 8;
            for (int i = (warp - 2) * 32 + lane; i < per_box * HB; i += 256) {
              const int box = i / per_box, rem = i % per_box;
              *reinterpret_cast<uint4*>(vpage + box * (2 * L::PAGE_BOX) + (tail_row + rem / 8) * 128 +
                                        (rem % 8) * 16) = make_uint4(0u, 0u, 0u, 0u);
            }
            fence_async_smem();
          }
          tc05_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(p_full(a));
        }
      }
    }

    // the rows' sums (both halves), then the difference of the maps, its norm and the factor
#pragma unroll
    for (int a = 0; a < 2; ++a) xch[(4 + a * 2 + half) * TILE_Q + r] = l_run[a];
    pair_barrier();
#pragma unroll
    for (int a = 0; a < 2; ++a) l_run[a] += xch[(4 + a * 2 + (half ^ 1)) * TILE_Q + r];
    const float i1 = l_run[0] > 0.0f ? 1.0f / l_run[0] : 0.0f;
    const float i2 = l_run[1] > 0.0f ? lambda / l_run[1] : 0.0f;
    if (ok) ok = warp_wait(o_done, 0u);
    float u[OC], ss = 0.0f;
    if (ok) {
      tc05_fence_after();
#pragma unroll
      for (int c = 0; c < OC / 32; ++c) {
        uint32_t o1[32], o2[32];
        tc05_ld_32x32b_x32(lane_addr + L::O_COL + half * OC + c * 32, o1);
        tc05_ld_32x32b_x32(lane_addr + L::O_COL + HD + half * OC + c * 32, o2);
        tc05_wait_ld();
#pragma unroll
        for (int e = 0; e < 32; ++e) {
          const float v = __uint_as_float(o1[e]) * i1 - __uint_as_float(o2[e]) * i2;
          u[c * 32 + e] = v;
          ss = fmaf(v, v, ss);
        }
      }
    } else {
#pragma unroll
      for (int e = 0; e < OC; ++e) u[e] = 0.0f;
    }
    xch[half * TILE_Q + r] = ss;
    pair_barrier();
    ss += xch[(half ^ 1) * TILE_Q + r];
    if (ok && r < rows_here) {
      const float f = factor / sqrtf(ss / (float)HD + eps);
      bf16* dst = out + (size_t)(row0 + q0 + r) * out_stride + (size_t)h * HD + half * OC;
#pragma unroll
      for (int c = 0; c < OC / 8; ++c) {
        uint4 w;
        __nv_bfloat162* hh = reinterpret_cast<__nv_bfloat162*>(&w);
#pragma unroll
        for (int e = 0; e < 4; ++e)
          hh[e] = __floats2bfloat162_rn(u[c * 8 + 2 * e] * f, u[c * 8 + 2 * e + 1] * f);
        *reinterpret_cast<uint4*>(dst + c * 8) = w;
      }
    }
  }

  tc05_fence_before();
  __syncthreads();
  if (*abort_flag) {
    if (tid == 0) {
      nb_report_timeout(err_word);
      // let TMA copies that are still in flight land before the shared memory goes away
      const long long t0 = clock64();
      while (clock64() - t0 < 4000000LL) {
      }
    }
    __syncthreads();
  }
  if (warp == 1) {
    tc05_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base),
                 "r"((uint32_t)L::TMEM_COLS)
                 : "memory");
  }
}

template <int HD>
int launch_tc(const void* q, int q_stride, int n_rows, const int* cu_rows, const int* seq_slot,
              const int* seq_pos0, const void* k_cache, const void* v_cache, long long n_pages,
              const int* block_table, int max_pages, int n_heads, int n_kv_heads, void* out,
              int out_stride, float scale, int window, float lambda, float factor, float eps,
              int n_seqs, int max_q_len, cudaStream_t stream) {
  using L = DiffSmem<HD>;
  CUtensorMap mq, mk, mv;
  int rc = make_map(&mq, q, n_rows, q_stride, TILE_Q, 64, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2);
  if (rc) return rc;
  const long long kv_rows = n_pages * n_kv_heads * PAGE_TOKENS;
  rc = make_map(&mk, k_cache, kv_rows, HD, PAGE_TOKENS, 64, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2);
  if (rc) return rc;
  rc = make_map(&mv, v_cache, kv_rows, HD, PAGE_TOKENS, 64, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2);
  if (rc) return rc;
  auto kern = differential_tc_kernel<HD>;
  static bool configured = false;   // per instantiation
  if (!configured) {
    NB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
    configured = true;
  }
  int* word = nb_error_words();
  const dim3 grid((max_q_len + TILE_Q - 1) / TILE_Q, n_heads, n_seqs);
  NB_CUDA(nb_launch(kern, grid, dim3(TC_THREADS), (size_t)L::TOTAL, stream, mq, mk, mv, cu_rows,
                    seq_slot, seq_pos0, block_table, max_pages, n_kv_heads, n_heads / n_kv_heads,
                    (bf16*)out, out_stride, scale * 1.4426950408889634f, window, lambda, factor, eps,
                    word ? word + NB_ERRW_DIFFERENTIAL_TC : nullptr));
  return 0;
}

}  // namespace

// Whether the kernel takes this shape: bf16, values of two maps' size in the keys' store, head_dim
// = 2 d = 64 or 128.
NB_EXPORT int nb_attention_differential_tc_supported(int dtype, int head_dim, int n_heads,
                                                     int n_kv_heads, int page) {
  return dtype == NB_BF16 && page == PAGE_TOKENS && n_kv_heads >= 1 && n_heads % n_kv_heads == 0 &&
         (head_dim == 64 || head_dim == 128);
}

// Clock cycles a wait of this kernel may take before it gives up (default 4e9).
NB_EXPORT int nb_attention_differential_tc_set_wait_budget(long long cycles) {
  NB_REQUIRE(cycles >= 0, NB_ERR_BAD_ARG, "wait budget must not be negative");
  return set_wait_budget(cycles);
}

// q: [n_rows][n_heads * head_dim]; k_cache / v_cache: [n_pages][n_kv_heads][64][head_dim], keys and
// values of the step's rows among them; out: [n_rows][out_stride].
NB_EXPORT int nb_attention_differential_tc(const void* q, int n_rows, const int* cu_rows,
                                           const int* seq_slot, const int* seq_pos0,
                                           const void* k_cache, const void* v_cache, int n_pages,
                                           const int* block_table, int max_pages, int page, int n_heads,
                                           int n_kv_heads, int head_dim, void* out, int out_stride,
                                           float scale, int window, float lambda, float factor,
                                           float eps, int n_seqs, int max_q_len, cudaStream_t stream) {
  if (n_seqs == 0 || max_q_len == 0) return 0;
  NB_REQUIRE(nb_attention_differential_tc_supported(NB_BF16, head_dim, n_heads, n_kv_heads, page),
             NB_ERR_UNSUPPORTED, "attention_differential_tc: unsupported shape (head size %d, %d/%d heads)",
             head_dim, n_heads, n_kv_heads);
  NB_REQUIRE(n_seqs <= 65535 && n_heads <= 65535 && n_rows > 0 && n_pages > 0 && out_stride % 8 == 0,
             NB_ERR_UNSUPPORTED, "attention_differential_tc: bad sizes");
  NB_REQUIRE(scale > 0.0f && window >= 0, NB_ERR_UNSUPPORTED,
             "attention_differential_tc: takes a positive scale and no negative window");
  NB_REQUIRE(((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)out) % 16 == 0,
             NB_ERR_UNSUPPORTED, "attention_differential_tc: operands must be 16-byte aligned");
#define NB_ARGS q, n_heads * head_dim, n_rows, cu_rows, seq_slot, seq_pos0, k_cache, v_cache, (long long)n_pages, block_table, max_pages, n_heads, n_kv_heads, out, out_stride, scale, window, lambda, factor, eps, n_seqs, max_q_len, stream
  const int rc = head_dim == 64 ? launch_tc<64>(NB_ARGS) : launch_tc<128>(NB_ARGS);
#undef NB_ARGS
  if (rc) return rc;
  NB_CHECK_LAUNCH("attention_differential_tc");
  return 0;
}
