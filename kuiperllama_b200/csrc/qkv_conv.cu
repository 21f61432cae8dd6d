// What attention behind short convolutions needs between its input product and the scores, in one kernel:
//
//   u_t      the token's projected q | k | v (one row of the product)
//   y_t      = sum_j w[:, j] u_(t - taps + 1 + j)         a causal filter per channel; nothing before the sequence's start
//   q, k     the first `rot` elements of every head of y turn by the position, times `magnitude`, in pairs
//            (i, i + rot / 2) or, interleaved, (2i, 2i + 1)
//   v        y, or (1 - lambda) y + lambda v_first; y itself also to v_keep where one is given
//
// q goes to q_out, k and v into the token's rows of the paged cache.  Without weights (w null) y = u.  Inputs before the step's
// first token of a sequence come from the slot's state, float32 [taps - 1][ld] (oldest first, zero in a fresh slot): whole
// product rows, so that one layout serves q, k and v.  Sums, angles and rotation are 32-bit; the filter's sum runs in the order
// j = 0 .. taps - 1 whatever the cut of the prompt.
//
//   qkv_conv_kernel<T, V, TAPS, SINGLE>   a thread owns an item of up to 2 V channels of one head (V pairs of the turned part, or
//       2 V channels of the rest) and walks a tile of tokens of one sequence with the last taps - 1 inputs in registers (TAPS
//       2, 3, 4; TAPS 0 reads them again).  SINGLE: one token per sequence; the row may come as float32 pieces of a product
//       whose k range was cut (added in ascending order), and the thread moves the state of its own channels on.
//
// The state after a step of several tokens is a second launch (short_conv.cu: the convolution's CTAs read the old one).
// ExiledOfCode/KuiperLLama projects and rotates q and k without convolutions (kuiper/source/model/llama3.cpp:610-639).
#include "common.cuh"

namespace kl {

constexpr int QC_MAX_TAPS = 16;
constexpr int QC_TILE = 16;            // tokens per CTA
constexpr int QC_THREADS = 128;

struct QkvConv {
    const void* rows; const float* pieces; int n_pieces; long long piece_stride; long long ld;
    int q_col, k_col, v_col;
    const float* w;                    // [taps][ld], or null
    int taps;
    float* state; long long state_ld;
    const float* inv_freq; int rot; int interleaved; float magnitude;
    void* q_out; long long q_ld;
    void* k_cache; void* v_cache; const int* block_table; int blocks_per_seq;
    const void* v_first; long long v_first_ld; const float* lambda; void* v_keep;
    const int* cu_tokens; const int* seq_slots; const int* seq_starts;
    int H, KV, hd, vd, items_hd, items_vd;
};

template <typename T, int V> __device__ __forceinline__ void qc_load(const T* p, float (&x)[V]) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        x[0] = a.x; x[1] = a.y; x[2] = b.x; x[3] = b.y;
    } else if constexpr (V == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = to_f32(p[e]);
    }
}
template <typename T, int V> __device__ __forceinline__ void qc_store(T* p, const float (&x)[V]) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        __nv_bfloat162 a = __floats2bfloat162_rn(x[0], x[1]), b = __floats2bfloat162_rn(x[2], x[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&a);
        raw.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    } else if constexpr (V == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) p[e] = from_f32<T>(x[e]);
    }
}
// The token row's values of one chunk of V channels: from the product's rows, or the sum of its pieces (four on their way at a time).
template <typename T, int V>
__device__ __forceinline__ void qc_input(const QkvConv& A, size_t at, float (&x)[V]) {
    if (A.pieces == nullptr) { qc_load<T, V>((const T*)A.rows + at, x); return; }
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = 0.f;
    for (int z0 = 0; z0 < A.n_pieces; z0 += 4) {
        float p[4][V];
#pragma unroll
        for (int z = 0; z < 4; ++z) {
            if (z0 + z < A.n_pieces) qc_load<float, V>(A.pieces + (size_t)(z0 + z) * A.piece_stride + at, p[z]);
            else {
#pragma unroll
                for (int e = 0; e < V; ++e) p[z][e] = 0.f;
            }
        }
#pragma unroll
        for (int z = 0; z < 4; ++z)
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] += p[z][e];
    }
}

template <typename T, int V, int TAPS, bool SINGLE>
__global__ void __launch_bounds__(QC_THREADS)
qkv_conv_kernel(const QkvConv A) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float cs[];          // [tokens of the tile][rot / 2][2]: cos and sin times the magnitude
    const int item = blockIdx.z * QC_THREADS + threadIdx.x;
    const int q_items = A.H * A.items_hd, k_items = A.KV * A.items_hd, v_items = A.KV * A.items_vd;
    const bool live = item < q_items + k_items + v_items;
    const int role = !live ? 3 : (item < q_items ? 0 : (item < q_items + k_items ? 1 : 2));
    const int half = A.rot / 2;
    // which channels: chunk a at ea, chunk b at eb of head g (b may be absent); turned: the two chunks hold V pairs
    int g = 0, ea = 0, eb = 0, pair0 = 0, base_col = 0, width = A.hd;
    bool has_b = true, turned = false;
    if (role < 2) {
        const int it = role == 0 ? item : item - q_items;
        g = it / A.items_hd;
        const int i = it - g * A.items_hd;
        const int turn_items = half / V;
        turned = i < turn_items;
        if (turned) {
            pair0 = i * V;
            ea = A.interleaved ? 2 * i * V : i * V;
            eb = A.interleaved ? ea + V : ea + half;
        } else {
            ea = A.rot + (i - turn_items) * 2 * V;
            eb = ea + V;
            has_b = eb < A.hd;
        }
        base_col = (role == 0 ? A.q_col : A.k_col) + g * A.hd;
    } else if (role == 2) {
        const int it = item - q_items - k_items;
        g = it / A.items_vd;
        ea = (it - g * A.items_vd) * 2 * V;
        eb = ea + V;
        width = A.vd;
        has_b = eb < A.vd;
        base_col = A.v_col + g * A.vd;
    }
    const int ca = base_col + ea, cb = base_col + (has_b ? eb : ea);
    constexpr int NW = TAPS > 0 ? TAPS : 1;
    float wa[NW][V], wb[NW][V];
    if constexpr (TAPS > 0) {                             // weights are written by no kernel
        if (live) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) { qc_load<float, V>(A.w + (size_t)j * A.ld + ca, wa[j]); qc_load<float, V>(A.w + (size_t)j * A.ld + cb, wb[j]); }
        }
    }
    pdl_wait();
    const int s = blockIdx.y;
    const int row0 = A.cu_tokens[s], n_new = A.cu_tokens[s + 1] - row0;
    const int first = SINGLE ? 0 : (int)blockIdx.x * QC_TILE;
    if (first >= n_new) return;
    const int count = SINGLE ? 1 : min(QC_TILE, n_new - first);
    const int slot = A.seq_slots[s], start = A.seq_starts[s];
    for (int i = threadIdx.x; i < count * half; i += QC_THREADS) {
        const int t = i / half, f = i - t * half;
        float sn, c;
        sincosf((float)(start + first + t) * A.inv_freq[f], &sn, &c);
        cs[2 * i] = c * A.magnitude;
        cs[2 * i + 1] = sn * A.magnitude;
    }
    __syncthreads();
    if (!live) return;
    const bool write = A.k_cache != nullptr;
    if (role > 0 && !write && !(role == 2 && A.v_keep != nullptr) && !(SINGLE && A.state != nullptr)) return;
    const int keep = A.taps - 1;
    const float* st = A.state != nullptr ? A.state + (size_t)slot * A.state_ld : nullptr;
    // inputs before the tile's first token, oldest first
    float ha[NW][V], hb[NW][V];
    if constexpr (TAPS > 1) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int li = first - (TAPS - 1) + j;
            if (li >= 0) { qc_input<T, V>(A, (size_t)(row0 + li) * A.ld + ca, ha[j]); qc_input<T, V>(A, (size_t)(row0 + li) * A.ld + cb, hb[j]); }
            else { qc_load<float, V>(st + (size_t)(TAPS - 1 + li) * A.ld + ca, ha[j]); qc_load<float, V>(st + (size_t)(TAPS - 1 + li) * A.ld + cb, hb[j]); }
        }
    }
    const float lam = (role == 2 && A.v_first != nullptr) ? A.lambda[0] : 0.f;
    float na[V], nb[V];                                   // the next token's inputs are on their way while this one's are used
    qc_input<T, V>(A, (size_t)(row0 + first) * A.ld + ca, na);
    qc_input<T, V>(A, (size_t)(row0 + first) * A.ld + cb, nb);
    for (int t = 0; t < count; ++t) {
        float xa[V], xb[V], ya[V], yb[V];
#pragma unroll
        for (int e = 0; e < V; ++e) { xa[e] = na[e]; xb[e] = nb[e]; }
        const size_t row = (size_t)(row0 + first + t);
        if (!SINGLE && t + 1 < count) { qc_input<T, V>(A, (row + 1) * A.ld + ca, na); qc_input<T, V>(A, (row + 1) * A.ld + cb, nb); }
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int e = 0; e < V; ++e) {
                float a = 0.f, b = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) { a = fmaf(wa[j][e], ha[j][e], a); b = fmaf(wb[j][e], hb[j][e], b); }
                ya[e] = fmaf(wa[TAPS - 1][e], xa[e], a);
                yb[e] = fmaf(wb[TAPS - 1][e], xb[e], b);
            }
            if constexpr (SINGLE) {
                if (A.state != nullptr) {                     // this thread's channels of the slot's state move on
                    float* sw = A.state + (size_t)slot * A.state_ld;
#pragma unroll
                    for (int j = 0; j < TAPS - 1; ++j) {
                        qc_store<float, V>(sw + (size_t)j * A.ld + ca, j < TAPS - 2 ? ha[j + 1 < NW ? j + 1 : j] : xa);
                        if (has_b) qc_store<float, V>(sw + (size_t)j * A.ld + cb, j < TAPS - 2 ? hb[j + 1 < NW ? j + 1 : j] : xb);
                    }
                }
            } else {
#pragma unroll
                for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
                    for (int e = 0; e < V; ++e) { ha[j][e] = ha[j + 1][e]; hb[j][e] = hb[j + 1][e]; }
                if constexpr (TAPS > 1) {
#pragma unroll
                    for (int e = 0; e < V; ++e) { ha[TAPS - 2][e] = xa[e]; hb[TAPS - 2][e] = xb[e]; }
                }
            }
        } else if (A.w != nullptr) {
            // any number of taps: earlier inputs are read again
#pragma unroll
            for (int e = 0; e < V; ++e) ya[e] = yb[e] = 0.f;
            for (int j = 0; j < A.taps; ++j) {
                float va[V], vb[V], ja[V], jb[V];
                const int li = first + t - keep + j;
                if (j == keep) {
#pragma unroll
                    for (int e = 0; e < V; ++e) { va[e] = xa[e]; vb[e] = xb[e]; }
                } else if (li >= 0) {
                    qc_input<T, V>(A, (size_t)(row0 + li) * A.ld + ca, va);
                    qc_input<T, V>(A, (size_t)(row0 + li) * A.ld + cb, vb);
                } else {
                    qc_load<float, V>(st + (size_t)(keep + li) * A.ld + ca, va);
                    qc_load<float, V>(st + (size_t)(keep + li) * A.ld + cb, vb);
                }
                qc_load<float, V>(A.w + (size_t)j * A.ld + ca, ja);
                qc_load<float, V>(A.w + (size_t)j * A.ld + cb, jb);
#pragma unroll
                for (int e = 0; e < V; ++e) { ya[e] = fmaf(ja[e], va[e], ya[e]); yb[e] = fmaf(jb[e], vb[e], yb[e]); }
            }
            if constexpr (SINGLE) {
                if (A.state != nullptr) {
                    float* sw = A.state + (size_t)slot * A.state_ld;
                    for (int j = 0; j < keep; ++j) {
                        float va[V], vb[V];
                        if (j + 1 < keep) { qc_load<float, V>(sw + (size_t)(j + 1) * A.ld + ca, va); qc_load<float, V>(sw + (size_t)(j + 1) * A.ld + cb, vb); }
                        else {
#pragma unroll
                            for (int e = 0; e < V; ++e) { va[e] = xa[e]; vb[e] = xb[e]; }
                        }
                        qc_store<float, V>(sw + (size_t)j * A.ld + ca, va);
                        if (has_b) qc_store<float, V>(sw + (size_t)j * A.ld + cb, vb);
                    }
                }
            }
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) { ya[e] = xa[e]; yb[e] = xb[e]; }
        }
        const int pos = start + first + t;
        if (role == 2) {
            if (A.v_keep != nullptr) {
                T* dst = (T*)A.v_keep + row * (size_t)(A.KV * A.vd) + (size_t)g * A.vd;
                qc_store<T, V>(dst + ea, ya);
                if (has_b) qc_store<T, V>(dst + eb, yb);
            }
            if (!write) continue;
            if (A.v_first != nullptr) {
                const T* f = (const T*)A.v_first + row * (size_t)A.v_first_ld + (size_t)g * A.vd;
                float fa[V], fb[V];
                qc_load<T, V>(f + ea, fa);
                qc_load<T, V>(f + (has_b ? eb : ea), fb);
#pragma unroll
                for (int e = 0; e < V; ++e) { ya[e] = (1.0f - lam) * ya[e] + lam * fa[e]; yb[e] = (1.0f - lam) * yb[e] + lam * fb[e]; }
            }
            T* dst = (T*)A.v_cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, pos, g, A.KV, width);
            qc_store<T, V>(dst + ea, ya);
            if (has_b) qc_store<T, V>(dst + eb, yb);
            continue;
        }
        if (turned) {
            const float* c = cs + (size_t)t * A.rot + 2 * pair0;
            if (A.interleaved) {
                if constexpr (V == 1) {
                    const float u = ya[0], v = yb[0];
                    ya[0] = u * c[0] - v * c[1];
                    yb[0] = v * c[0] + u * c[1];
                } else {
#pragma unroll
                    for (int e = 0; e < V / 2; ++e) {
                        const float u = ya[2 * e], v = ya[2 * e + 1];
                        ya[2 * e] = u * c[2 * e] - v * c[2 * e + 1];
                        ya[2 * e + 1] = v * c[2 * e] + u * c[2 * e + 1];
                        const float u2 = yb[2 * e], v2 = yb[2 * e + 1];
                        yb[2 * e] = u2 * c[V + 2 * e] - v2 * c[V + 2 * e + 1];
                        yb[2 * e + 1] = v2 * c[V + 2 * e] + u2 * c[V + 2 * e + 1];
                    }
                }
            } else {
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    const float u = ya[e], v = yb[e];
                    ya[e] = u * c[2 * e] - v * c[2 * e + 1];
                    yb[e] = v * c[2 * e] + u * c[2 * e + 1];
                }
            }
        }
        if (role == 1 && !write) continue;
        T* dst = role == 0 ? (T*)A.q_out + row * (size_t)A.q_ld + (size_t)g * A.hd
                           : (T*)A.k_cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, pos, g, A.KV, A.hd);
        qc_store<T, V>(dst + ea, ya);
        if (has_b) qc_store<T, V>(dst + eb, yb);
    }
}

}  // namespace kl

using namespace kl;

// rows (compute dtype, `ld` elements apart) or pieces (float32 [n_pieces][..][ld], piece_stride apart; single steps alone).  w: float32
// [taps][ld] or null (then taps is 1).  state: float32, the slot's row at state + slot * state_ld holds [taps - 1][ld] (null where
// taps is 1, or for `single`, where the caller wants no convolution); `single`: every sequence brings one token, and the state moves
// on in this kernel.  q_out is not the rows themselves.  v_first (compute dtype) with lambda (one number on the device) or null;
// v_keep [n_tokens, KV * vd] or null; caches both null: q (and v_keep) alone.
KL_API int kl_qkv_conv(const void* rows, const float* pieces, int n_pieces, long long piece_stride, long long ld, int q_col, int k_col,
                       int v_col, const float* w, int taps, float* state, long long state_ld, const float* inv_freq, int rot,
                       int interleaved, float magnitude, void* q_out, long long q_ld, void* k_cache, void* v_cache,
                       const int* block_table, int blocks_per_seq, const void* v_first, long long v_first_ld, const float* lambda,
                       void* v_keep, const int* cu_tokens, const int* seq_slots, const int* seq_starts, int n_seqs, int max_new, int single,
                       int H, int KV, int hd, int vd, int dtype, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return KL_OK;
    if (H <= 0 || KV <= 0 || hd <= 0 || vd <= 0 || rot < 0 || rot % 2 || rot > hd || (rot > 0 && inv_freq == nullptr)) return KL_ERR_BAD_SIZE;
    if ((rows == nullptr) == (pieces == nullptr) || (pieces != nullptr && (n_pieces < 1 || !single)) || (single && max_new != 1)) return KL_ERR_BAD_SIZE;
    if (taps < 1 || taps > QC_MAX_TAPS || (w == nullptr && taps != 1) || (taps > 1 && state == nullptr)) return KL_ERR_BAD_SIZE;
    if ((k_cache == nullptr) != (v_cache == nullptr) || (v_first != nullptr && lambda == nullptr) || q_out == nullptr || q_out == rows) return KL_ERR_BAD_SIZE;
    if (n_seqs > 65535) return KL_ERR_BAD_SIZE;
    if (dtype != KL_F32 && dtype != KL_BF16) return KL_ERR_BAD_DTYPE;
    QkvConv A{rows, pieces, n_pieces, piece_stride, ld, q_col, k_col, v_col, w, taps, taps > 1 ? state : nullptr, state_ld, inv_freq, rot, interleaved,
              magnitude, q_out, q_ld, k_cache, v_cache, block_table, blocks_per_seq, v_first, v_first_ld, lambda, v_keep, cu_tokens,
              seq_slots, seq_starts, H, KV, hd, vd, 0, 0};
    const uintptr_t m = dtype == KL_BF16 ? 7 : 15;
    const bool four = hd % 4 == 0 && vd % 4 == 0 && rot % 8 == 0 && ld % 4 == 0 && q_col % 4 == 0 && k_col % 4 == 0 && v_col % 4 == 0 && q_ld % 4 == 0 &&
                      v_first_ld % 4 == 0 && piece_stride % 4 == 0 && state_ld % 4 == 0 &&
                      (((uintptr_t)rows | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)v_first | (uintptr_t)v_keep) & m) == 0 &&
                      (((uintptr_t)pieces | (uintptr_t)w | (uintptr_t)A.state) & 15) == 0;
    const int V = four ? 4 : 1;
    A.items_hd = rot / 2 / V + (hd - rot + 2 * V - 1) / (2 * V);
    A.items_vd = (vd + 2 * V - 1) / (2 * V);
    const long long items = (long long)(H + KV) * A.items_hd + (long long)KV * A.items_vd;
    const long long zb = (items + QC_THREADS - 1) / QC_THREADS;
    if (zb > 65535) return KL_ERR_BAD_SIZE;
    const dim3 grid(single ? 1 : (max_new + QC_TILE - 1) / QC_TILE, n_seqs, (unsigned)zb);
    const size_t smem = (size_t)(single ? 1 : QC_TILE) * rot * sizeof(float);
    if (smem > 48 * 1024) return KL_ERR_BAD_SIZE;
#define KL_QC(T, VV, TAPS)                                                                                              \
    do {                                                                                                                \
        if (single) launch_kernel(qkv_conv_kernel<T, VV, TAPS, true>, grid, QC_THREADS, smem, stream, A);               \
        else launch_kernel(qkv_conv_kernel<T, VV, TAPS, false>, grid, QC_THREADS, smem, stream, A);                     \
    } while (0)
#define KL_QC_T(T)                                                                                                      \
    do {                                                                                                                \
        if (four && taps == 4) KL_QC(T, 4, 4); else if (four && taps == 3) KL_QC(T, 4, 3); else if (four && taps == 2) KL_QC(T, 4, 2); \
        else if (four) KL_QC(T, 4, 0); else KL_QC(T, 1, 0);                                                             \
    } while (0)
    if (dtype == KL_F32) KL_QC_T(float); else KL_QC_T(bf16);
#undef KL_QC_T
#undef KL_QC
    KL_LAUNCH_CHECK();
    return KL_OK;
}
