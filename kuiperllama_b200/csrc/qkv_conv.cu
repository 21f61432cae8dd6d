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
//       2 V channels of the rest or of a value head) and walks a tile of tokens of one sequence with the last taps - 1 inputs in registers (TAPS
//       2, 3, 4; TAPS 0 reads them again).  SINGLE: one token per sequence; the row may come as float32 pieces of a product
//       whose k range was cut (added in ascending order), and the thread moves the state of its own channels on.
//
// The state after a step of several tokens is a second launch (short_conv.cu: the convolution's CTAs read the old one).
// ExiledOfCode/KuiperLLama projects and rotates q and k without convolutions (kuiper/source/model/llama3.cpp:610-639).
#include "common.cuh"

namespace kl {

constexpr int QC_MAX_TAPS = 16;
constexpr int QC_TILE = 4;             // tokens per CTA
constexpr int QC_AHEAD = 4;            // tokens whose inputs are requested together
constexpr int QC_VECTOR = 2;           // elements an access
constexpr int QC_THREADS = 128;
constexpr int QC_CTAS = 6;             // per multiprocessor

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
    int H, KV, hd, vd, items_hd, items_vd, qk_blocks;
};

// V elements as they lie in memory: what is held while a load is on its way.
template <typename T, int V> struct QcRaw { T v[V]; };
template <> struct QcRaw<bf16, 4> { uint2 v; };
template <> struct QcRaw<bf16, 2> { uint32_t v; };
template <> struct QcRaw<float, 4> { float4 v; };
template <> struct QcRaw<float, 2> { float2 v; };
template <typename T, int V> __device__ __forceinline__ QcRaw<T, V> qc_fetch(const T* p) { return *reinterpret_cast<const QcRaw<T, V>*>(p); }
template <typename T, int V> __device__ __forceinline__ void qc_unpack(const QcRaw<T, V>& raw, float (&x)[V]) {
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] = to_f32(e[i]);
}
template <typename T, int V> __device__ __forceinline__ void qc_load(const T* p, float (&x)[V]) { qc_unpack<T, V>(qc_fetch<T, V>(p), x); }
template <typename T, int V> __device__ __forceinline__ void qc_store(T* p, const float (&x)[V]) {
    QcRaw<T, V> raw;
    T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) e[i] = from_f32<T>(x[i]);
    *reinterpret_cast<QcRaw<T, V>*>(p) = raw;
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

// One item over a tile of tokens: `count` tokens from the sequence's token `first` of this step (position `start` + first).  VALUES: a
// value head's channels (no rotation, mixing); else a query's or key's.  cs: cos and sin of the tile's positions.
template <typename T, int V, int TAPS, bool SINGLE, bool VALUES>
__device__ __forceinline__ void qc_item(const QkvConv& A, bool live, const float* cs, int row0, int first, int count, int start,
                                        int slot, const float (&wa)[TAPS > 0 ? TAPS : 1][V], const float (&wb)[TAPS > 0 ? TAPS : 1][V],
                                        int g, int ea, int eb, bool has_b, bool turned, bool is_q, int pair0, int ca, int cb) {
    if (!live) return;
    const bool write = A.k_cache != nullptr;
    const bool keeps = VALUES && A.v_keep != nullptr;
    if (!is_q && !write && !keeps && !(SINGLE && A.state != nullptr)) return;
    constexpr int NW = TAPS > 0 ? TAPS : 1;
    const int keep = A.taps - 1;
    const float* st = A.state != nullptr ? A.state + (size_t)slot * A.state_ld : nullptr;
    const int width = VALUES ? A.vd : A.hd;
    const size_t row_first = (size_t)(row0 + first);
    // inputs on their way: the next tokens' (and what is mixed into their values) while one is worked on
    constexpr int AHEAD = SINGLE ? 1 : QC_AHEAD;
    constexpr int FA = VALUES ? AHEAD : 1;
    QcRaw<T, V> na[AHEAD], nb[AHEAD], fa[FA], fb[FA];
    const T* pa = (const T*)A.rows + row_first * A.ld + ca;
    const T* pb = (const T*)A.rows + row_first * A.ld + cb;
    const bool mixes = VALUES && A.v_first != nullptr && write;
    const T* pf = mixes ? (const T*)A.v_first + row_first * (size_t)A.v_first_ld + (size_t)g * A.vd + ea : nullptr;
    const int fb_off = has_b ? eb - ea : 0;
    if constexpr (!SINGLE) {
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (i < count) { na[i] = qc_fetch<T, V>(pa + (size_t)i * A.ld); nb[i] = qc_fetch<T, V>(pb + (size_t)i * A.ld); }
    }
    if constexpr (VALUES) {
        if (mixes) {
#pragma unroll
            for (int i = 0; i < AHEAD; ++i)
                if (i < count) { fa[i] = qc_fetch<T, V>(pf + (size_t)i * A.v_first_ld); fb[i] = qc_fetch<T, V>(pf + (size_t)i * A.v_first_ld + fb_off); }
        }
    }
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
    const float lam = mixes ? A.lambda[0] : 0.f;
    // where the token's row goes: q by rows, k and v along their page
    T* dst = is_q ? (T*)A.q_out + row_first * (size_t)A.q_ld + (size_t)g * A.hd + ea : nullptr;
    T* const cache = VALUES ? (T*)A.v_cache : (T*)A.k_cache;
    if (!is_q && write) dst = cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, start + first, g, A.KV, width) + ea;
    const size_t advance = is_q ? (size_t)A.q_ld : (size_t)width;
    const int b_off = eb - ea;
    T* kept = keeps ? (T*)A.v_keep + row_first * (size_t)(A.KV * A.vd) + (size_t)g * A.vd + ea : nullptr;
    const float* c = cs + 2 * pair0;
    for (int t0 = 0; t0 < count; t0 += AHEAD)
#pragma unroll
    for (int ti = 0; ti < AHEAD; ++ti) {
        const int t = t0 + ti;
        if (t >= count) break;
        float xa[V], xb[V], ya[V], yb[V];
        if constexpr (SINGLE) {
            qc_input<T, V>(A, row_first * A.ld + ca, xa);
            qc_input<T, V>(A, row_first * A.ld + cb, xb);
        } else {
            qc_unpack<T, V>(na[ti], xa);
            qc_unpack<T, V>(nb[ti], xb);
            pa += A.ld;
            pb += A.ld;
            if (t + AHEAD < count) { na[ti] = qc_fetch<T, V>(pa + (size_t)(AHEAD - 1) * A.ld); nb[ti] = qc_fetch<T, V>(pb + (size_t)(AHEAD - 1) * A.ld); }
        }
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
        if constexpr (VALUES) {
            if (keeps) {
                qc_store<T, V>(kept, ya);
                if (has_b) qc_store<T, V>(kept + b_off, yb);
                kept += A.KV * A.vd;
            }
            if (mixes) {
                float xf[V], yf[V];
                qc_unpack<T, V>(fa[ti], xf);
                qc_unpack<T, V>(fb[ti], yf);
                pf += A.v_first_ld;
                if (!SINGLE && t + AHEAD < count) {
                    fa[ti] = qc_fetch<T, V>(pf + (size_t)(AHEAD - 1) * A.v_first_ld);
                    fb[ti] = qc_fetch<T, V>(pf + (size_t)(AHEAD - 1) * A.v_first_ld + fb_off);
                }
#pragma unroll
                for (int e = 0; e < V; ++e) { ya[e] = (1.0f - lam) * ya[e] + lam * xf[e]; yb[e] = (1.0f - lam) * yb[e] + lam * yf[e]; }
            }
        } else if (turned) {
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
        c += A.rot;
        if (dst != nullptr) {
            qc_store<T, V>(dst, ya);
            if (has_b) qc_store<T, V>(dst + b_off, yb);
            dst += advance;
            const int next = start + first + t + 1;
            if (!SINGLE && !is_q && next % PAGE == 0 && t + 1 < count)       // a new page
                dst = cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, next, g, A.KV, width) + ea;
        }
    }
}

template <typename T, int V, int TAPS, bool SINGLE>
__global__ void __launch_bounds__(QC_THREADS, QC_CTAS)
qkv_conv_kernel(const QkvConv A) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float cs[];          // [tokens of the tile][rot / 2][2]: cos and sin times the magnitude
    // the first `qk_blocks` CTAs along z hold the items of q and k, the others those of v
    const bool values = (int)blockIdx.z >= A.qk_blocks;
    const int item = ((int)blockIdx.z - (values ? A.qk_blocks : 0)) * QC_THREADS + threadIdx.x;
    const int q_items = A.H * A.items_hd;
    const bool live = item < (values ? A.KV * A.items_vd : q_items + A.KV * A.items_hd);
    const bool is_q = !values && item < q_items;
    const int half = A.rot / 2;
    // which channels: chunk a at ea, chunk b at eb of head g (b may be absent); turned: the two chunks hold V pairs
    int g = 0, ea = 0, eb = V, pair0 = 0, base_col = 0;
    bool has_b = false, turned = false;
    if (live && !values) {
        const int it = is_q ? item : item - q_items;
        g = it / A.items_hd;
        const int i = it - g * A.items_hd;
        const int turn_items = half / V;
        turned = i < turn_items;
        if (turned) {
            pair0 = i * V;
            ea = A.interleaved ? 2 * i * V : i * V;
            eb = A.interleaved ? ea + V : ea + half;
            has_b = true;
        } else {
            ea = A.rot + (i - turn_items) * 2 * V;
            eb = ea + V;
            has_b = eb < A.hd;
        }
        base_col = (is_q ? A.q_col : A.k_col) + g * A.hd;
    } else if (live) {
        g = item / A.items_vd;
        ea = (item - g * A.items_vd) * 2 * V;
        eb = ea + V;
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
    const int slot = A.seq_slots[s], start = A.seq_starts[s];
    const int first = SINGLE ? 0 : (int)blockIdx.x * QC_TILE;
    if (first >= n_new) return;
    const int count = SINGLE ? 1 : min(QC_TILE, n_new - first);
    if (values) {
        qc_item<T, V, TAPS, SINGLE, true>(A, live, cs, row0, first, count, start, slot, wa, wb, g, ea, eb, has_b, false, false, 0, ca, cb);
        return;
    }
    for (int i = threadIdx.x; i < count * half; i += QC_THREADS) {
        const int t = i / half, f = i - t * half;
        float sn, c;
        sincosf((float)(start + first + t) * A.inv_freq[f], &sn, &c);
        cs[2 * i] = c * A.magnitude;
        cs[2 * i + 1] = sn * A.magnitude;
    }
    __syncthreads();
    qc_item<T, V, TAPS, SINGLE, false>(A, live, cs, row0, first, count, start, slot, wa, wb, g, ea, eb, has_b, turned, is_q, pair0, ca, cb);
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
              seq_slots, seq_starts, H, KV, hd, vd, 0, 0, 0};
    constexpr int VEC = QC_VECTOR;
    const uintptr_t m = VEC * (dtype == KL_BF16 ? 2 : 4) - 1;
    const bool vec = hd % VEC == 0 && vd % VEC == 0 && rot % (2 * VEC) == 0 && ld % VEC == 0 && q_col % VEC == 0 && k_col % VEC == 0 && v_col % VEC == 0 &&
                     q_ld % VEC == 0 && v_first_ld % VEC == 0 && piece_stride % VEC == 0 && state_ld % VEC == 0 &&
                     (((uintptr_t)rows | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)v_first | (uintptr_t)v_keep) & m) == 0 &&
                     (((uintptr_t)pieces | (uintptr_t)w | (uintptr_t)A.state) & (VEC * 4 - 1)) == 0;
    const int V = vec ? VEC : 1;
    A.items_hd = rot / 2 / V + (hd - rot + 2 * V - 1) / (2 * V);
    A.items_vd = (vd + 2 * V - 1) / (2 * V);
    const long long qk_blocks = ((long long)(H + KV) * A.items_hd + QC_THREADS - 1) / QC_THREADS;
    const long long zb = qk_blocks + ((long long)KV * A.items_vd + QC_THREADS - 1) / QC_THREADS;
    if (zb > 65535) return KL_ERR_BAD_SIZE;
    A.qk_blocks = (int)qk_blocks;
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
        if (vec && taps == 4) KL_QC(T, VEC, 4); else if (vec && taps == 3) KL_QC(T, VEC, 3); else if (vec && taps == 2) KL_QC(T, VEC, 2);  \
        else if (vec) KL_QC(T, VEC, 0); else KL_QC(T, 1, 0);                                                            \
    } while (0)
    if (dtype == KL_F32) KL_QC_T(float); else KL_QC_T(bf16);
#undef KL_QC_T
#undef KL_QC
    KL_LAUNCH_CHECK();
    return KL_OK;
}
