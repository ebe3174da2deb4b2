// Decode attention over keys and values of different head sizes: the tensor-core kernel of
// attention_decode_mma.cuh with a plane of its own pitch for each (a store of two planes and one
// block table), staged in rows of the larger size rounded up to 32, 64 or 128.
#include "attention_decode_mma.cuh"

// 1 if this kernel takes the shape: bf16, sizes that are multiples of 8 up to 128.
NB_EXPORT int nb_attention_decode_mixed_supported(int dtype, int d, int dv, int n_heads, int n_kv_heads,
                                                  int page) {
  if (dtype != NB_BF16 || page != PAGE_TOKENS || n_kv_heads < 1 || n_heads % n_kv_heads != 0) return 0;
  return n_heads / n_kv_heads <= 8 && d % 8 == 0 && dv % 8 == 0 && d >= 8 && dv >= 8 && d <= 128 && dv <= 128;
}

// The row a key and a value are staged in: what the scratch of the splits is counted by.
NB_EXPORT int nb_attention_decode_mixed_row(int d, int dv) {
  const int most = d > dv ? d : dv;
  return most <= 32 ? 32 : most <= 64 ? 64 : 128;
}

// q: bf16 rows with head h's query at column h * d; k_cache: [n_pages][n_kv_heads][page][d], v_cache:
// [n_pages][n_kv_heads][page][dv], their pages listed in one block table; out: bf16 rows, head h at
// column h * dv.  Masks, sink, gate and splits as in nb_attention_decode_capped.  The step's keys and
// values are in the cache already.
NB_EXPORT int nb_attention_decode_mixed(const void* q, int q_stride, const int* row_slot,
                                        const int* row_pos, const void* k_cache, const void* v_cache,
                                        const int* block_table, int max_pages, int page, int n_heads,
                                        int n_kv_heads, int d, int dv, void* out, int out_stride,
                                        float scale, float softcap, const float* sink, int window,
                                        int keep_first, int mask_block, const float* gate,
                                        int gate_stride, int gate_col, int n_rows, int n_splits,
                                        float* part_acc, float* part_ml, int* counters,
                                        int clusters_allowed, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  NB_REQUIRE(nb_attention_decode_mixed_supported(NB_BF16, d, dv, n_heads, n_kv_heads, page),
             NB_ERR_UNSUPPORTED, "attention_decode_mixed: unsupported shape (head sizes %d/%d, %d/%d heads)",
             d, dv, n_heads, n_kv_heads);
  NB_REQUIRE(n_splits >= 1 && n_splits <= 65535 && n_rows <= 65535 && n_kv_heads <= 65535,
             NB_ERR_UNSUPPORTED, "attention_decode_mixed: grid too large");
  NB_REQUIRE(part_acc && part_ml && counters, NB_ERR_BAD_ARG, "attention_decode_mixed: scratch missing");
  NB_REQUIRE(q_stride % 8 == 0 && ((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16 == 0,
             NB_ERR_UNSUPPORTED, "attention_decode_mixed: rows must be 16-byte aligned");
  NB_REQUIRE(softcap >= 0.0f && window >= 0 && keep_first >= 0 && mask_block >= 0 &&
                 !(window > 0 && mask_block > 0),
             NB_ERR_BAD_ARG, "attention_decode_mixed: a bad mask or cap");
  const NbAttnOpts opt{window, keep_first, mask_block, gate, gate_stride, gate_col};
  NB_REQUIRE(!opt.keeps() || n_splits >= 2, NB_ERR_BAD_ARG,
             "attention_decode_mixed: kept first tokens take a split of their own");
  const NbPagedKV kv{(void*)k_cache, (void*)v_cache, block_table, max_pages, page, n_kv_heads, d, dv};
  const bool clustered = clusters_allowed > 0 && n_splits >= 2 && n_splits <= MAX_CLUSTER;
  int rc = 0;
#define NB_MIX(HD_)                                                                              \
  rc = launch_mma<HD_, __nv_bfloat16, false, true>(q, q_stride, 0, row_slot, row_pos, kv,        \
                                                   n_heads / n_kv_heads, out, out_stride, scale, \
                                                   softcap, sink, opt, n_rows, n_splits,         \
                                                   part_acc, part_ml, counters, /*append=*/-1, 0, 0, \
                                                   clustered, stream)
  switch (nb_attention_decode_mixed_row(d, dv)) {
    case 32: NB_MIX(32); break;
    case 64: NB_MIX(64); break;
    default: NB_MIX(128); break;
  }
#undef NB_MIX
  if (rc) return rc;
  NB_CHECK_LAUNCH("attention_decode_mixed");
  return 0;
}
