// A matrix memory with exponential gates over whole prompts, in chunks of 64 tokens on the tensor cores (bfloat16 q, k and v).
//
//   S_t = a_t S_(t-1) + c_t k_t v_t^T,   z_t likewise with k_t alone,   y_t = S_t^T q_t,   den_t = max(|z_t . q_t|, exp(-m_t)) + eps
//
// With f, i the log gates, m the running maximum (mlstm.cu) and F the sum of f from a chunk's first token, a token t of a chunk
// that starts from S_in, z_in and m_in has
//
//   y_t = exp(F_t + m_in - m_t) S_in^T q_t + sum over s <= t of exp(F_t - F_s + i_s - m_t) (q_t . k_s) v_s
//
// and the chunk leaves  S_out = exp(F_C + m_in - m_C) S_in + sum over s of exp(F_C - F_s + i_s - m_C) k_s v_s^T.  No exponent is
// above zero.  Two launches:
//
//   mlstm_intra_kernel    a CTA per (chunk, head, sequence): the weighted products p[t, s] of the chunk (float32), and the
//                         factors of the chunk's tokens and of the chunk.
//   mlstm_walk_kernel     a CTA per (DVS columns of S, head, sequence) walks the sequence's chunks: S lies in float32 accumulators
//                         (rows over the warps); per chunk y = dq (Q S) + p V, then S = alpha S + K^T (w V).  One more CTA per
//                         (head, sequence) does the same with z in S's place and a column of ones in V's, and makes den.
//
// The state, the gates and every factor are 32-bit.  q, k and v enter as they are (bfloat16, exact).  What is a 32-bit number and
// enters a product (S, p, w v) enters as the sum of two bfloat16 numbers, high + rest: 16 bits of mantissa, two products.
// ExiledOfCode/KuiperLLama has no recurrent mixer (its mixer is mha_kernel.cu:61,74-106).
#include "common.cuh"

namespace kl {

constexpr int MC = 64;                 // tokens per chunk
constexpr int MC_PS = MC + 4;          // row stride of p in shared memory (floats)

struct ChunkedArgs {
    const bf16* q; long long ld_q; const bf16* k; long long ld_k; const bf16* v; long long ld_v;   // head h at column h * dim (h * vdim)
    const float* lf; const float* li; const float* mb; const float* m;    // [rows, heads]: log gates, the maximum before and after a token
    float* p;                           // [rows, heads, MC]
    float* dq; float* w;                // [rows, heads]
    float* alpha;                       // [sequences, max_chunks, heads]
    float* state; long long ld_state;   // S at state + slot * ld_state, [heads, dim, vdim]; z at z_off, [heads, dim]
    long long z_off;
    float* y; float* den;               // [rows, heads * vdim], [rows, heads]
    const int* cu_tokens; const int* seq_slots;
    int heads, dim, vdim, max_chunks, slices;
    float q_scale, den_eps;
};

__device__ __forceinline__ uint32_t mc_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mc_copy16(void* dst, const void* src, bool live) {       // not live: the piece becomes zero, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mc_smem(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void mc_copy4(void* dst, const void* src, bool live) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(mc_smem(dst)), "l"(src), "r"(live ? 4 : 0) : "memory");
}
__device__ __forceinline__ void mc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void mc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void mc_ldm4(uint32_t a, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mc_ldm4t(uint32_t a, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two float32 numbers as packed bfloat16: the nearest ones, and what they leave over
__device__ __forceinline__ void mc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
// the place of 16-byte piece c of row r in a tile of rows of W elements, in elements; neighbouring rows' pieces fall on different banks
template <int W> __device__ __forceinline__ int mc_at(int r, int c) {
    constexpr int P = W / 8;
    if constexpr (P >= 8) return r * W + ((c ^ (r & 7)) << 3);
    else return r * W + ((c ^ ((r / (8 / P)) & (P - 1))) << 3);
}
// a chunk's rows (column block of `width` elements, zero beyond it and beyond the live rows) into a tile of rows of W elements
template <int W, int THREADS>
__device__ __forceinline__ void mc_load(bf16* tile, const bf16* src, long long ld, int live, int width) {
    constexpr int P = W / 8;
    for (int idx = threadIdx.x; idx < MC * P; idx += THREADS) {
        const int r = idx / P, c = idx - r * P;
        const bool in = r < live && c * 8 < width;
        mc_copy16(tile + mc_at<W>(r, c), in ? (const void*)(src + (size_t)r * ld + c * 8) : (const void*)src, in);
    }
}

template <int DK>
__global__ void __launch_bounds__(128)
mlstm_intra_kernel(const ChunkedArgs A) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(128) unsigned char mc_raw[];
    bf16* Qt = reinterpret_cast<bf16*>(mc_raw);            // [MC][DK]
    bf16* Kt = Qt + MC * DK;
    __shared__ float F[MC], G[MC], M[MC];                  // sums of f, i - F, m
    const int s = blockIdx.z, h = blockIdx.y, c = blockIdx.x;
    const int row0 = A.cu_tokens[s] + c * MC, live = min(MC, A.cu_tokens[s + 1] - row0);
    if (live <= 0) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    mc_load<DK, 128>(Qt, A.q + (size_t)row0 * A.ld_q + (size_t)h * A.dim, A.ld_q, live, A.dim);
    mc_load<DK, 128>(Kt, A.k + (size_t)row0 * A.ld_k + (size_t)h * A.dim, A.ld_k, live, A.dim);
    mc_commit();
    if (warp == 0) {                                       // two tokens a lane
        const int t = 2 * lane;
        auto at = [&](int j) { return (size_t)(row0 + j) * A.heads + h; };
        const float f0 = t < live ? A.lf[at(t)] : 0.f, f1 = t + 1 < live ? A.lf[at(t + 1)] : 0.f;
        float sum = f0 + f1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += up;
        }
        F[t + 1] = sum; F[t] = sum - f1;
        __syncwarp();
        const float F_end = F[live - 1], m_in = A.mb[at(0)], m_end = A.m[at(live - 1)];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int j = t + e;
            G[j] = 0.f; M[j] = 0.f;
            if (j < live) {
                const float g = A.li[at(j)] - F[j], m = A.m[at(j)];
                G[j] = g; M[j] = m;
                A.dq[at(j)] = A.q_scale * expf(F[j] + m_in - m);
                A.w[at(j)] = expf(F_end + g - m_end);
            }
        }
        if (lane == 0) A.alpha[((size_t)s * A.max_chunks + c) * A.heads + h] = expf(F_end + m_in - m_end);
    }
    mc_wait<0>();
    __syncthreads();
    // 16 tokens a warp, the keys up to the last of them
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }
    const int n_pairs = warp + 1;                          // pairs of n tiles (16 keys) that reach the diagonal
#pragma unroll 4
    for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t a[4];
        mc_ldm4(mc_smem(Qt + mc_at<DK>(warp * 16 + (lane & 15), ks * 2 + (lane >> 4))), a);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
            if (n2 < n_pairs) {
                uint32_t b[4];
                mc_ldm4(mc_smem(Kt + mc_at<DK>(n2 * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1))), b);
                mc_mma(acc[2 * n2], a, b[0], b[1]);
                mc_mma(acc[2 * n2 + 1], a, b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int t = warp * 16 + (lane >> 2) + 8 * i;
        const bool in = t < live;
        float* row = A.p + ((size_t)(row0 + t) * A.heads + h) * MC;
        const float Ft = F[t] - M[t];
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            const int j = n * 8 + 2 * (lane & 3);
            float2 o;
            o.x = j <= t ? acc[n][2 * i] * A.q_scale * expf(Ft + G[j]) : 0.f;
            o.y = j + 1 <= t ? acc[n][2 * i + 1] * A.q_scale * expf(Ft + G[j + 1]) : 0.f;
            if (in) *reinterpret_cast<float2*>(row + j) = o;
        }
    }
}

// Warps: DK / 32 of them, at least 4; a warp holds MT tiles of 16 rows of S (all DVS columns) in accumulators.  In y a warp takes
// 16 tokens (warp % 4) and DVS / (warps / 4) columns.
template <int DK, int DVS>
__global__ void __launch_bounds__(DK >= 128 ? 256 : 128)
mlstm_walk_kernel(const ChunkedArgs A) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int WARPS = DK >= 128 ? 8 : 4, THREADS = WARPS * 32;
    constexpr int MT = DK / (16 * WARPS), NT = DVS / 8;
    constexpr int YT = NT / (WARPS / 4);                   // n tiles of y per warp
    extern __shared__ __align__(128) unsigned char mc_raw[];
    bf16* Qt = reinterpret_cast<bf16*>(mc_raw);            // [2][MC][DK]
    bf16* Kt = Qt + 2 * MC * DK;                           // [2][MC][DK]
    bf16* Vt = Kt + 2 * MC * DK;                           // [2][MC][DVS]
    bf16* Vh = Vt + 2 * MC * DVS;                          // [MC][DVS]: w v, high
    bf16* Vl = Vh + MC * DVS;                              //            and the rest
    bf16* Sh = Vl + MC * DVS;                              // [DK][DVS]: S at the chunk's start, high
    bf16* Sl = Sh + DK * DVS;
    float* Pt = reinterpret_cast<float*>(Sl + DK * DVS);   // [2][MC][MC_PS]
    float* wt = Pt + 2 * MC * MC_PS;                       // [2][MC]
    float* dt = wt + 2 * MC;                               // [2][MC]
    const int s = blockIdx.z, h = blockIdx.y, slice = blockIdx.x;
    const int first = A.cu_tokens[s], n_new = A.cu_tokens[s + 1] - first;
    if (n_new <= 0) return;
    const int chunks = (n_new + MC - 1) / MC;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int H = A.heads, dk = A.dim, dv = A.vdim;
    float* slot = A.state + (size_t)A.seq_slots[s] * A.ld_state;
    const bool carries_z = slice == A.slices;              // the CTA of the normaliser
    const int col0 = carries_z ? 0 : slice * DVS, cols = carries_z ? 1 : min(DVS, dv - col0);

    auto request = [&](int c, int buf) {
        const int row0 = first + c * MC, live = min(MC, n_new - c * MC);
        mc_load<DK, THREADS>(Qt + buf * MC * DK, A.q + (size_t)row0 * A.ld_q + (size_t)h * dk, A.ld_q, live, dk);
        mc_load<DK, THREADS>(Kt + buf * MC * DK, A.k + (size_t)row0 * A.ld_k + (size_t)h * dk, A.ld_k, live, dk);
        for (int t = threadIdx.x; t < 2 * MC; t += THREADS) {
            const int j = t % MC;
            const float* src = (t < MC ? A.w : A.dq) + (size_t)(row0 + min(j, live - 1)) * H + h;
            mc_copy4((t < MC ? wt : dt) + buf * MC + j, src, j < live);
        }
        if (!carries_z)
            mc_load<DVS, THREADS>(Vt + buf * MC * DVS, A.v + (size_t)row0 * A.ld_v + (size_t)h * dv + col0, A.ld_v, live, cols);
        for (int idx = threadIdx.x; idx < MC * (MC / 4); idx += THREADS) {
            const int r = idx / (MC / 4), e = (idx - r * (MC / 4)) * 4;
            mc_copy16(Pt + (buf * MC + r) * MC_PS + e, A.p + ((size_t)(row0 + min(r, live - 1)) * H + h) * MC + e, r < live);
        }
        mc_commit();
    };
    request(0, 0);

    // S: this CTA's columns of the slot's [dim, vdim] matrix, or z as a matrix of one column
    const int width = carries_z ? 1 : dv;
    float* S_slot = carries_z ? slot + A.z_off + (size_t)h * dk : slot + (size_t)h * dk * dv + col0;
    if (carries_z)
        for (int idx = threadIdx.x; idx < 2 * MC * DVS; idx += THREADS) {
            const int t = (idx / DVS) % MC, j = idx % DVS;
            Vt[(idx / (MC * DVS)) * MC * DVS + mc_at<DVS>(t, j >> 3) + (j & 7)] = __float2bfloat16_rn(j == 0 ? 1.f : 0.f);
        }

    float S[MT][NT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = (warp * MT + mt) * 16 + (lane >> 2) + 8 * (e >> 1), col = n * 8 + 2 * (lane & 3) + (e & 1);
                S[mt][n][e] = (r < dk && col < cols) ? S_slot[(size_t)r * width + col] : 0.f;
            }

    const int yt = warp & 3, yn = (warp >> 2) * YT;        // this warp's 16 tokens and first n tile of y
    for (int c = 0; c < chunks; ++c) {
        const int buf = c & 1, row0 = first + c * MC, live = min(MC, n_new - c * MC);
        const float alpha = A.alpha[((size_t)s * A.max_chunks + c) * H + h];
        mc_wait<0>();
        __syncthreads();                                   // this chunk is here; the chunk before is done with every buffer
        if (c + 1 < chunks) request(c + 1, buf ^ 1);
        float floor_at[2] = {0.f, 0.f};                    // exp(-m) of this thread's two tokens of y
        if (carries_z) {
#pragma unroll
            for (int i = 0; i < 2; ++i) floor_at[i] = expf(-A.m[(size_t)(row0 + min(yt * 16 + (lane >> 2) + 8 * i, live - 1)) * H + h]);
        }
        // S at the chunk's start as high + rest, then its decay
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int r = (warp * MT + mt) * 16 + (lane >> 2) + 8 * i;
                    uint32_t hi, lo;
                    mc_split(S[mt][n][2 * i], S[mt][n][2 * i + 1], hi, lo);
                    const int at = mc_at<DVS>(r, n) + 2 * (lane & 3);
                    *reinterpret_cast<uint32_t*>(Sh + at) = hi;
                    *reinterpret_cast<uint32_t*>(Sl + at) = lo;
                    S[mt][n][2 * i] *= alpha;
                    S[mt][n][2 * i + 1] *= alpha;
                }
        const bf16* V = Vt + buf * MC * DVS;
        for (int idx = threadIdx.x; idx < MC * DVS / 2; idx += THREADS) {
            const int t = idx / (DVS / 2), j = (idx - t * (DVS / 2)) * 2;
            const int at = mc_at<DVS>(t, j >> 3) + (j & 7);
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(V + at));
            const float wv = wt[buf * MC + t];
            uint32_t hi, lo;
            mc_split(wv * f.x, wv * f.y, hi, lo);
            *reinterpret_cast<uint32_t*>(Vh + at) = hi;
            *reinterpret_cast<uint32_t*>(Vl + at) = lo;
        }
        __syncthreads();
        const bf16* Q = Qt + buf * MC * DK;
        const bf16* K = Kt + buf * MC * DK;
        // y = dq (Q S): tokens yt * 16 .., columns yn * 8 ..
        float y[YT][4];
#pragma unroll
        for (int n = 0; n < YT; ++n) { y[n][0] = y[n][1] = y[n][2] = y[n][3] = 0.f; }
#pragma unroll 4
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t a[4];
            mc_ldm4(mc_smem(Q + mc_at<DK>(yt * 16 + (lane & 15), ks * 2 + (lane >> 4))), a);
            if constexpr (YT == 1) {
                uint32_t b[4];                             // high rows ks * 16 .. + 15, then the rest's
                mc_ldm4t(mc_smem((lane < 16 ? Sh : Sl) + mc_at<DVS>(ks * 16 + (lane & 15), yn)), b);
                mc_mma(y[0], a, b[0], b[1]);
                mc_mma(y[0], a, b[2], b[3]);
            } else {
#pragma unroll
                for (int n = 0; n < YT; n += 2) {
                    uint32_t b[4];
                    const int at = mc_at<DVS>(ks * 16 + (lane & 15), yn + n + (lane >> 4));
                    mc_ldm4t(mc_smem(Sh + at), b);
                    mc_mma(y[n], a, b[0], b[1]);
                    mc_mma(y[n + 1], a, b[2], b[3]);
                    mc_ldm4t(mc_smem(Sl + at), b);
                    mc_mma(y[n], a, b[0], b[1]);
                    mc_mma(y[n + 1], a, b[2], b[3]);
                }
            }
        }
        {
            const int t = yt * 16 + (lane >> 2);
            const float d0 = dt[buf * MC + t], d1 = dt[buf * MC + t + 8];
#pragma unroll
            for (int n = 0; n < YT; ++n) { y[n][0] *= d0; y[n][1] *= d0; y[n][2] *= d1; y[n][3] *= d1; }
        }
        // + p V: the keys up to the tile of the diagonal
#pragma unroll
        for (int ks = 0; ks < MC / 16; ++ks) {
            if (ks <= yt) {
                const float* P = Pt + (size_t)(buf * MC + yt * 16 + (lane >> 2)) * MC_PS + ks * 16 + 2 * (lane & 3);
                const float2 p0 = *reinterpret_cast<const float2*>(P), p1 = *reinterpret_cast<const float2*>(P + 8 * MC_PS);
                const float2 p2 = *reinterpret_cast<const float2*>(P + 8), p3 = *reinterpret_cast<const float2*>(P + 8 * MC_PS + 8);
                uint32_t ah[4], al[4];
                mc_split(p0.x, p0.y, ah[0], al[0]); mc_split(p1.x, p1.y, ah[1], al[1]);
                mc_split(p2.x, p2.y, ah[2], al[2]); mc_split(p3.x, p3.y, ah[3], al[3]);
#pragma unroll
                for (int n = 0; n < YT; n += 2) {
                    uint32_t b[4];
                    mc_ldm4t(mc_smem(V + mc_at<DVS>(ks * 16 + (lane & 15), yn + n + (YT == 1 ? 0 : (lane >> 4)))), b);
                    mc_mma(y[n], ah, b[0], b[1]);
                    mc_mma(y[n], al, b[0], b[1]);
                    if constexpr (YT > 1) {
                        mc_mma(y[n + 1], ah, b[2], b[3]);
                        mc_mma(y[n + 1], al, b[2], b[3]);
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int t = yt * 16 + (lane >> 2) + 8 * i;
            if (carries_z) {
                const size_t at = (size_t)(row0 + t) * H + h;
                if (t < live && yn == 0 && (lane & 3) == 0) A.den[at] = fmaxf(fabsf(y[0][2 * i]), floor_at[i]) + A.den_eps;
            } else if (t < live) {
                float* o = A.y + (size_t)(row0 + t) * H * dv + (size_t)h * dv + col0;
#pragma unroll
                for (int n = 0; n < YT; ++n) {
                    const int col = (yn + n) * 8 + 2 * (lane & 3);
                    if (col < cols) *reinterpret_cast<float2*>(o + col) = make_float2(y[n][2 * i], y[n][2 * i + 1]);      // vdim is a multiple of 8
                }
            }
        }
        // S += K^T (w V): the warp's rows of S are columns of K
#pragma unroll
        for (int ks = 0; ks < MC / 16; ++ks) {
            uint32_t bh[NT][2], bl[NT][2];
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                uint32_t b[4];
                const int at = mc_at<DVS>(ks * 16 + (lane & 15), n + (lane >> 4));
                mc_ldm4t(mc_smem(Vh + at), b);
                bh[n][0] = b[0]; bh[n][1] = b[1]; bh[n + 1][0] = b[2]; bh[n + 1][1] = b[3];
                mc_ldm4t(mc_smem(Vl + at), b);
                bl[n][0] = b[0]; bl[n][1] = b[1]; bl[n + 1][0] = b[2]; bl[n + 1][1] = b[3];
            }
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                uint32_t a[4];
                mc_ldm4t(mc_smem(K + mc_at<DK>(ks * 16 + (lane & 7) + ((lane >> 4) << 3), (warp * MT + mt) * 2 + ((lane >> 3) & 1))), a);
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    mc_mma(S[mt][n], a, bh[n][0], bh[n][1]);
                    mc_mma(S[mt][n], a, bl[n][0], bl[n][1]);
                }
            }
        }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = (warp * MT + mt) * 16 + (lane >> 2) + 8 * (e >> 1), col = n * 8 + 2 * (lane & 3) + (e & 1);
                if (r < dk && col < cols) S_slot[(size_t)r * width + col] = S[mt][n][e];
            }
}

template <int DK, int DVS>
static int launch_walk(const ChunkedArgs& A, int n_seqs, cudaStream_t stream) {
    constexpr size_t smem = (size_t)(4 * MC * DK + 2 * MC * DVS + 2 * MC * DVS + 2 * DK * DVS) * sizeof(bf16) + (size_t)(2 * MC * MC_PS + 4 * MC) * sizeof(float);
    static_assert(smem <= 227 * 1024, "mlstm_walk_kernel: shared memory");
    KL_CUDA(cudaFuncSetAttribute(mlstm_walk_kernel<DK, DVS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_kernel(mlstm_walk_kernel<DK, DVS>, dim3(A.slices + 1, A.heads, n_seqs), DK >= 128 ? 256 : 128, smem, stream, A);
    KL_LAUNCH_CHECK();
    return KL_OK;
}
template <int DK>
static int launch_chunked(ChunkedArgs& A, int n_seqs, cudaStream_t stream) {
    constexpr size_t smem = (size_t)2 * MC * DK * sizeof(bf16);
    KL_CUDA(cudaFuncSetAttribute(mlstm_intra_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_kernel(mlstm_intra_kernel<DK>, dim3(A.max_chunks, A.heads, n_seqs), 128, smem, stream, A);
    KL_LAUNCH_CHECK();
    // narrow slices of S while the wide ones would leave SMs without work
    const int wide = (A.vdim + 31) / 32;
    if ((long long)wide * A.heads * n_seqs * 4 >= 3LL * kl::sm_count()) { A.slices = wide; return launch_walk<DK, 32>(A, n_seqs, stream); }
    A.slices = (A.vdim + 15) / 16;
    return launch_walk<DK, 16>(A, n_seqs, stream);
}

}  // namespace kl

using namespace kl;

// q, k: bfloat16 [rows, heads * dim], v: [rows, heads * vdim], rows on 16-byte boundaries (column slices allowed); dim and vdim
// multiples of 8, dim at most 256.  logs: float32 [4, rows, heads] as kl_mlstm_gates leaves them (log f, log i, the maximum before
// and after the token).  scratch: float32 [rows * heads * 66 + n_seqs * ceil(max_new / 64) * heads].  state: S [heads, dim, vdim]
// per slot, z [heads, dim] z_off elements behind it.  y [rows, heads * vdim], den [rows, heads]: float32.
KL_API int kl_mlstm_chunked(const void* q, long long ld_q, const void* k, long long ld_k, const void* v, long long ld_v, const float* logs,
                            float* scratch, float* state, long long ld_state, long long z_off, float* y, float* den, const int* cu_tokens,
                            const int* seq_slots, int rows, int n_seqs, int max_new, int heads, int dim, int vdim, float q_scale,
                            float den_eps, cudaStream_t stream) {
    if (rows <= 0 || n_seqs <= 0 || max_new <= 0) return KL_OK;
    if (heads <= 0 || heads > 65535 || n_seqs > 65535 || dim <= 0 || dim > 256 || dim % 8 || vdim <= 0 || vdim % 8) return KL_ERR_BAD_SIZE;
    if ((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)scratch) & 15) || ((uintptr_t)y & 7) || ld_q % 8 || ld_k % 8 || ld_v % 8) return KL_ERR_BAD_ALIGN;
    if (kl::sm_count() <= 0) return KL_ERR_SETUP;
    const size_t rh = (size_t)rows * heads;
    ChunkedArgs A;
    A.q = (const bf16*)q; A.ld_q = ld_q; A.k = (const bf16*)k; A.ld_k = ld_k; A.v = (const bf16*)v; A.ld_v = ld_v;
    A.lf = logs; A.li = logs + rh; A.mb = logs + 2 * rh; A.m = logs + 3 * rh;
    A.p = scratch; A.dq = scratch + rh * MC; A.w = A.dq + rh; A.alpha = A.w + rh;
    A.state = state; A.ld_state = ld_state; A.z_off = z_off; A.y = y; A.den = den; A.cu_tokens = cu_tokens; A.seq_slots = seq_slots;
    A.heads = heads; A.dim = dim; A.vdim = vdim; A.max_chunks = (max_new + MC - 1) / MC; A.slices = 0; A.q_scale = q_scale; A.den_eps = den_eps;
    if (dim <= 64) return launch_chunked<64>(A, n_seqs, stream);
    if (dim <= 128) return launch_chunked<128>(A, n_seqs, stream);
    return launch_chunked<256>(A, n_seqs, stream);
}
