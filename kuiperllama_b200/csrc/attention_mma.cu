// Entry points of the mma.sync attention kernel (attention_mma.cuh) with values of the keys' size: prefill, decode in its
// plain and fused forms, and the options of `AttentionExtra` up to pooled rows.
#include "attention_mma.cuh"

using namespace kl;

// Attention of a ragged batch: sequence b brings seq_new[b] tokens (rows cu_tokens[b] ... of q
// and out) that start at position seq_starts[b] of slot seq_slots[b]; its keys and values are
// already in the cache.  max_new is the largest seq_new (host copy, sizes the grid); n_rows the
// number of packed rows.  few_rows != 0 picks the layout for decode (one token per sequence:
// the warps of a CTA split the keys).  Head sizes 64 and 128; others KL_ERR_BAD_SIZE.
static int attention_mma_dispatch(const void* q, int q_stride, void* out, const void* k_cache, const void* v_cache,
                            const int* block_table, int blocks_per_seq, const int* cu_tokens, const int* seq_slots,
                            const int* seq_starts, const int* seq_new, float* part_o, float* part_ml, int n_seqs,
                            int max_new, int n_rows, int H, int KV, int hd, float scale, int window, int splits,
                            int few_rows, const DecodeFuse& fuse, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return KL_OK;
    if (KV <= 0 || H % KV || splits < 1) return KL_ERR_BAD_SIZE;
    if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return KL_ERR_BAD_SIZE;
    if (q_stride % 2 || ((uintptr_t)q & 3)) return KL_ERR_BAD_ALIGN;
#define KL_MMA(HD, WM, WN, NS)                                                                                        \
    return launch_mma<HD, WM, WN, NS>((const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_cache, (const bf16*)v_cache,     \
                                  block_table, blocks_per_seq, cu_tokens, seq_slots, seq_starts, seq_new, part_o,      \
                                  part_ml, n_seqs, max_new, n_rows, H, KV, scale, window, splits, fuse, stream)
#define KL_MMA5(HD, WM, WN, NS, SK)                                                                                   \
    return launch_mma<HD, WM, WN, NS, SK>((const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_cache, (const bf16*)v_cache, \
                                  block_table, blocks_per_seq, cu_tokens, seq_slots, seq_starts, seq_new, part_o,      \
                                  part_ml, n_seqs, max_new, n_rows, H, KV, scale, window, splits, fuse, stream)
    // Decode: three CTAs of two stages fit an SM, or two CTAs of three stages.  A CTA's time is set by
    // its chain of pages either way, so what counts is how many rounds of CTAs the grid needs: three
    // stages where they do not add a round (64 sequences of 8 kv heads: 2 rounds both ways, 47 against 53 us).
    const int sms = kl::sm_count();
    if (sms <= 0) return KL_ERR_SETUP;
    if (hd == 128 && few_rows) {
        const long long ctas = (long long)n_seqs * KV * splits;
        const long long rounds2 = (ctas + 3 * sms - 1) / (3 * sms), rounds3 = (ctas + 2 * sms - 1) / (2 * sms);
        // More CTAs than three per SM: light CTAs (two warps, half pages, three stages), four to an SM.
        static const int light = getenv("KL_ATTN_LIGHT") ? atoi(getenv("KL_ATTN_LIGHT")) : 1;
        // Light CTAs of two stages (32 KB, 168 registers) fit six to an SM: taken where that saves rounds
        // over four of three stages (each of its rounds moves fewer bytes at a time; measured on the 8B
        // shape: one round against two and two against three are faster, three against four is not).
        const long long rounds4 = (ctas + 4 * sms - 1) / (4 * sms), rounds6 = (ctas + 6 * sms - 1) / (6 * sms);
        if (rounds2 > 1 && light && rounds6 * 7 < rounds4 * 5) KL_MMA5(128, 1, 2, 2, 32);
        if (rounds2 > 1 && light) KL_MMA5(128, 1, 2, 3, 32);
        if (rounds2 > 1 && rounds3 <= rounds2) KL_MMA(128, 1, 4, 3);
    }
    if (hd == 128) { if (few_rows) KL_MMA(128, 1, 4, 2); else KL_MMA(128, 4, 1, 2); }
    if (hd == 64) { if (few_rows) KL_MMA(64, 1, 4, 2); else KL_MMA(64, 4, 1, 2); }
#undef KL_MMA
#undef KL_MMA5
    return KL_ERR_BAD_SIZE;
}

KL_API int kl_attention_mma(const void* q, int q_stride, void* out, const void* k_cache, const void* v_cache,
                            const int* block_table, int blocks_per_seq, const int* cu_tokens, const int* seq_slots,
                            const int* seq_starts, const int* seq_new, float* part_o, float* part_ml, int n_seqs,
                            int max_new, int n_rows, int H, int KV, int hd, float scale, int window, int splits,
                            int few_rows, cudaStream_t stream) {
    DecodeFuse none;
    memset(&none, 0, sizeof(none));
    return attention_mma_dispatch(q, q_stride, out, k_cache, v_cache, block_table, blocks_per_seq, cu_tokens, seq_slots,
                                  seq_starts, seq_new, part_o, part_ml, n_seqs, max_new, n_rows, H, KV, hd, scale, window,
                                  splits, few_rows, none, stream);
}

// The same with the options of `AttentionExtra`: a sink per head (weights 0), sigmoid weights with a number per head (weights 1),
// pooled rows (pool > 0: caches of block means [pages][KV][PAGE][hd] with a block table of their own, a window is needed).
// Prefill layout, or with few_rows the four-warp decode layout on whole pages.
KL_API int kl_attention_mma_extra(const void* q, int q_stride, void* out, const void* k_cache, const void* v_cache,
                                  const int* block_table, int blocks_per_seq, const int* cu_tokens, const int* seq_slots,
                                  const int* seq_starts, const int* seq_new, float* part_o, float* part_ml, int n_seqs,
                                  int max_new, int n_rows, int H, int KV, int hd, float scale, int window, int splits,
                                  int few_rows, const float* sink, const float* head_bias, int weights, const void* pool_k,
                                  const void* pool_v, const int* pool_table, int pool_blocks_per_seq, int pool, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return KL_OK;
    if (KV <= 0 || H % KV || splits < 1 || (weights != 0 && weights != 1)) return KL_ERR_BAD_SIZE;
    if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return KL_ERR_BAD_SIZE;
    if (q_stride % 2 || ((uintptr_t)q & 3)) return KL_ERR_BAD_ALIGN;
    if (pool > 0 && (window <= 0 || pool_k == nullptr || pool_v == nullptr || pool_table == nullptr)) return KL_ERR_BAD_SIZE;
    if (weights == 1 && sink != nullptr) return KL_ERR_BAD_SIZE;
    DecodeFuse none;
    memset(&none, 0, sizeof(none));
    AttentionExtra ex;
    ex.sink = sink; ex.head_bias = head_bias; ex.pool_k = (const bf16*)pool_k; ex.pool_v = (const bf16*)pool_v;
    ex.pool_table = pool_table; ex.pool_blocks_per_seq = pool_blocks_per_seq; ex.pool = pool > 0 ? pool : 0;
#define KL_MMAX(HD, WM, WN, W)                                                                                                   \
    return launch_mma<HD, WM, WN, 2, PAGE, W>((const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_cache, (const bf16*)v_cache,  \
                                              block_table, blocks_per_seq, cu_tokens, seq_slots, seq_starts, seq_new, part_o,   \
                                              part_ml, n_seqs, max_new, n_rows, H, KV, scale, window, splits, none, stream, ex)
    ex.chunk = 0; ex.rel = nullptr; ex.rel_n = 0;
    // template parameter: 1 = sigmoid weights, 2 = softmax with the options compiled in
    if (hd == 128 && weights == 0) { if (few_rows) KL_MMAX(128, 1, 4, 2); else KL_MMAX(128, 4, 1, 2); }
    if (hd == 128 && weights == 1) { if (few_rows) KL_MMAX(128, 1, 4, 1); else KL_MMAX(128, 4, 1, 1); }
    if (hd == 64 && weights == 0) { if (few_rows) KL_MMAX(64, 1, 4, 2); else KL_MMAX(64, 4, 1, 2); }
    if (hd == 64 && weights == 1) { if (few_rows) KL_MMAX(64, 1, 4, 1); else KL_MMAX(64, 4, 1, 1); }
#undef KL_MMAX
    return KL_ERR_BAD_SIZE;
}

// A whole decode step's attention in one kernel: one token per sequence, rows in sequence
// order.  The q/k/v projections come as `qkv` (bfloat16 [rows, (H + 2 KV) * hd]) or as
// float32 pieces `partials` [n_partials, rows, width]; the kernel rotates q and k (full
// rotation, inv_freq [hd / 2]), writes the token's key and value into the cache, attends, and
// merges the splits itself (`counters`: int32 [rows * KV], zero, left zero).
KL_API int kl_attention_decode_fused(const void* qkv, const float* partials, int n_partials, long long partial_stride,
                                     const float* inv_freq, void* out, void* k_cache, void* v_cache,
                                     const int* block_table, int blocks_per_seq, const int* cu_tokens,
                                     const int* seq_slots, const int* seq_starts, const int* seq_new, float* part_o,
                                     float* part_ml, int* counters, int n_seqs, int H, int KV, int hd, float scale,
                                     int window, int splits, cudaStream_t stream) {
    if (n_seqs <= 0) return KL_OK;
    if (inv_freq == nullptr || counters == nullptr || (n_partials == 0 && qkv == nullptr)) return KL_ERR_BAD_SIZE;
    DecodeFuse fuse;
    fuse.enabled = 1;
    fuse.partials = partials;
    fuse.n_partials = n_partials;
    fuse.partial_stride = (size_t)partial_stride;
    fuse.qkv = (const bf16*)qkv;
    fuse.inv_freq = inv_freq;
    fuse.k_cache_w = (bf16*)k_cache;
    fuse.v_cache_w = (bf16*)v_cache;
    fuse.counters = counters;
    return attention_mma_dispatch(out /* unused as q */, 8, out, k_cache, v_cache, block_table, blocks_per_seq, cu_tokens,
                                  seq_slots, seq_starts, seq_new, part_o, part_ml, n_seqs, 1, n_seqs, H, KV, hd, scale,
                                  window, splits, 1, fuse, stream);
}
