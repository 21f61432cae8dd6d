// Entry point of the mma.sync attention kernel (attention_mma.cuh) with values of a size of their own: windows, chunks, a bias by
// distance and a sink.
#include "attention_mma.cuh"

using namespace kl;

// Arguments as for kl_attention_mma; chunks of `chunk` positions (0: none), a bias by distance (rel: float32 [H, rel_n], or null), a sink
// (float32 [H]: exp(sink[h]) joins the denominator, or null) and values of size vd in a cache of their own row size; key and
// value sizes of 32, 64, 96 and 128.
KL_API int kl_attention_mma_chunked(const void* q, int q_stride, void* out, const void* k_cache, const void* v_cache,
                                    const int* block_table, int blocks_per_seq, const int* cu_tokens, const int* seq_slots,
                                    const int* seq_starts, const int* seq_new, float* part_o, float* part_ml, int n_seqs,
                                    int max_new, int n_rows, int H, int KV, int hd, int vd, float scale, int window, int splits,
                                    int few_rows, int chunk, const float* rel, int rel_n, const float* sink, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return KL_OK;
    if (KV <= 0 || H % KV || splits < 1 || chunk < 0 || (rel != nullptr && rel_n < 1)) return KL_ERR_BAD_SIZE;
    if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return KL_ERR_BAD_SIZE;
    if (q_stride % 2 || ((uintptr_t)q & 3)) return KL_ERR_BAD_ALIGN;
    DecodeFuse none;
    memset(&none, 0, sizeof(none));
    AttentionExtra ex;
    memset(&ex, 0, sizeof(ex));
    ex.chunk = chunk; ex.rel = rel; ex.rel_n = rel_n; ex.sink = sink;
#define KL_MMAC(HD, VD, WM, WN)                                                                                                     \
    return launch_mma<HD, WM, WN, 2, PAGE, 3, VD>((const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_cache, (const bf16*)v_cache, \
                                                  block_table, blocks_per_seq, cu_tokens, seq_slots, seq_starts, seq_new, part_o,  \
                                                  part_ml, n_seqs, max_new, n_rows, H, KV, scale, window, splits, none, stream, ex)
#define KL_MMAC_VD(HD)                                                                                     \
    do {                                                                                                   \
        if (vd == 32) { if (few_rows) KL_MMAC(HD, 32, 1, 4); else KL_MMAC(HD, 32, 4, 1); }                 \
        if (vd == 64) { if (few_rows) KL_MMAC(HD, 64, 1, 4); else KL_MMAC(HD, 64, 4, 1); }                 \
        if (vd == 96) { if (few_rows) KL_MMAC(HD, 96, 1, 4); else KL_MMAC(HD, 96, 4, 1); }                 \
        if (vd == 128) { if (few_rows) KL_MMAC(HD, 128, 1, 4); else KL_MMAC(HD, 128, 4, 1); }              \
    } while (0)
    if (hd == 32) KL_MMAC_VD(32);
    if (hd == 64) KL_MMAC_VD(64);
    if (hd == 96) KL_MMAC_VD(96);
    if (hd == 128) KL_MMAC_VD(128);
#undef KL_MMAC_VD
#undef KL_MMAC
    return KL_ERR_BAD_SIZE;
}
