// The gates of a matrix memory with exponential gating (mLSTM), everything in 32 bits.  Per (token, head), with the log
// gates made from a pre-activation pair (zi, zf) plus a bias each:
//
//   soft(z) = cap * tanh(z / cap);     i = soft(zi + bi);     f = logsigmoid(soft(zf + bf))
//   m_t = max(f_t + m_(t-1), i_t)                     (a running maximum from the slot's state, zero in a fresh slot)
//   a_t = exp(f_t + m_(t-1) - m_t);   c_t = exp(i_t - m_t);   floor_t = exp(-m_t)
//
// so that S_t = a_t S_(t-1) + c_t k_t v_t^T never overflows (outer_recurrence.cu takes a, c and floor).
//
//   mlstm_gates_kernel          a CTA per (sequence, head): the maximum is a scan over the tokens under
//                               (F1, M1) o (F2, M2) = (F1 + F2, max(M1 + F2, M2)), a thread per token, tile after tile.
//   mlstm_gate_project_kernel   the pre-activations themselves, z = W h in 32 bits (W: 2 * heads rows); in a step of single tokens
//                               it makes a, c and floor at once.
//
// ExiledOfCode/KuiperLLama has no recurrent mixer (its mixer is mha_kernel.cu:61,74-106).
#include "common.cuh"

namespace kl {

struct MlstmGates {
    const float* bias;                        // [2 * heads]: the input gate's, then the forget gate's
    float* state; long long ld_state;         // the slot's m at state + slot * ld_state, [heads]
    float* a; float* c; float* floor;         // [rows, heads]
    float* logs; long long logs_stride;       // or, where given, [4][rows, heads]: f, i, m before the token and m after it
    const int* cu_tokens; const int* seq_slots;
    int heads;
    float cap;
};

__device__ __forceinline__ float ml_soft(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// What one token does to the running maximum, and the three factors that come of it (or the numbers they are made of).
__device__ __forceinline__ void ml_factors(const MlstmGates& G, size_t row, int h, float f, float i, float m_before, float m) {
    const size_t at = row * G.heads + h;
    if (G.logs != nullptr) {
        G.logs[at] = f; G.logs[G.logs_stride + at] = i; G.logs[2 * G.logs_stride + at] = m_before; G.logs[3 * G.logs_stride + at] = m;
        return;
    }
    G.a[at] = expf(f + m_before - m);
    G.c[at] = expf(i - m);
    G.floor[at] = expf(-m);
}

constexpr int ML_SCAN_THREADS = 512;

// z: float32 [rows, 2 * heads], the pre-activations without bias.
__global__ void __launch_bounds__(ML_SCAN_THREADS)
mlstm_gates_kernel(const MlstmGates G, const float* __restrict__ z, long long ld_z) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float warp_F[32], warp_M[32], last_m[33];
    const int s = blockIdx.x, h = blockIdx.y;
    const int row0 = G.cu_tokens[s], n_new = G.cu_tokens[s + 1] - row0;
    if (n_new <= 0) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    float* m_slot = G.state + (size_t)G.seq_slots[s] * G.ld_state + h;
    const float bi = G.bias[h], bf = G.bias[G.heads + h];
    float carry = *m_slot;
    for (int t0 = 0; t0 < n_new; t0 += blockDim.x) {
        const int t = t0 + threadIdx.x;
        float F = 0.f, M = -INFINITY, f = 0.f, i = 0.f;          // past the end: the scan's neutral element
        if (t < n_new) {
            const float* zr = z + (size_t)(row0 + t) * ld_z;
            i = ml_soft(zr[h] + bi, G.cap);
            f = ml_logsigmoid(ml_soft(zr[G.heads + h] + bf, G.cap));
            F = f; M = i;
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fl = __shfl_up_sync(0xffffffffu, F, o), Ml = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) { M = fmaxf(Ml + F, M); F = Fl + F; }
        }
        if (lane == 31) { warp_F[warp] = F; warp_M[warp] = M; }
        __syncthreads();
        float m_in = carry;                                      // the maximum before this warp's first token
        for (int w = 0; w < warp; ++w) m_in = fmaxf(warp_F[w] + m_in, warp_M[w]);
        const float m = fmaxf(F + m_in, M);
        float m_before = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) m_before = m_in;
        if (t < n_new) ml_factors(G, (size_t)(row0 + t), h, f, i, m_before, m);
        if (warp == nwarps - 1 && lane == 31) last_m[0] = m;     // tokens past the end leave it alone: F adds 0, M is -inf
        __syncthreads();
        carry = last_m[0];
    }
    if (threadIdx.x == 0) *m_slot = carry;
}

// W: [2 * heads, width] in the compute dtype; x rows of the compute dtype.  A CTA takes TT tokens and ML_HG heads (2 ML_HG rows of
// W), its warps cut the width between them in pieces of 16 bytes a lane, and the warps' sums meet in shared memory.  With
// `gates` (every sequence brings one token, row = sequence) a thread per (token, head) finishes its head; else z float32
// [rows, 2 * heads].
constexpr int ML_WARPS = 8, ML_HG = 4;
template <typename T, int TT>
__global__ void __launch_bounds__(ML_WARPS * 32)
mlstm_gate_project_kernel(const T* __restrict__ x, long long ld_x, const T* __restrict__ W, int width, int rows, int n_seqs, int gates,
                          float* __restrict__ z, const MlstmGates G) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float part[ML_WARPS][2 * ML_HG * TT];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t0 = blockIdx.x * TT, h0 = blockIdx.y * ML_HG;
    float acc[2 * ML_HG][TT];
#pragma unroll
    for (int g = 0; g < 2 * ML_HG; ++g)
#pragma unroll
        for (int t = 0; t < TT; ++t) acc[g][t] = 0.f;
    // rows past the end read the last one (their sums are not used), and so do heads past the end
    const T* xr[TT];
#pragma unroll
    for (int t = 0; t < TT; ++t) xr[t] = x + (size_t)min(t0 + t, rows - 1) * ld_x;
    auto w_row = [&](int g) { return W + (size_t)((g < ML_HG ? 0 : G.heads) + min(h0 + g % ML_HG, G.heads - 1)) * width; };
    constexpr int V = 16 / sizeof(T);
    if (width % V == 0 && ld_x % V == 0 && ((((uintptr_t)x) | ((uintptr_t)W)) & 15) == 0) {
        for (int c = (warp * 32 + lane) * V; c < width; c += ML_WARPS * 32 * V) {
            uint4 rx[TT], rw[2 * ML_HG];
#pragma unroll
            for (int t = 0; t < TT; ++t) rx[t] = *reinterpret_cast<const uint4*>(xr[t] + c);
#pragma unroll
            for (int g = 0; g < 2 * ML_HG; ++g) rw[g] = *reinterpret_cast<const uint4*>(w_row(g) + c);
#pragma unroll
            for (int g = 0; g < 2 * ML_HG; ++g) {
                const T* pw = reinterpret_cast<const T*>(&rw[g]);
#pragma unroll
                for (int t = 0; t < TT; ++t) {
                    const T* px = reinterpret_cast<const T*>(&rx[t]);
#pragma unroll
                    for (int e = 0; e < V; ++e) acc[g][t] = fmaf(to_f32(pw[e]), to_f32(px[e]), acc[g][t]);
                }
            }
        }
    } else {
        for (int c = warp * 32 + lane; c < width; c += ML_WARPS * 32) {
#pragma unroll
            for (int g = 0; g < 2 * ML_HG; ++g) {
                const float wv = to_f32(w_row(g)[c]);
#pragma unroll
                for (int t = 0; t < TT; ++t) acc[g][t] = fmaf(wv, to_f32(xr[t][c]), acc[g][t]);
            }
        }
    }
#pragma unroll
    for (int g = 0; g < 2 * ML_HG; ++g)
#pragma unroll
        for (int t = 0; t < TT; ++t) {
            const float v = warp_sum(acc[g][t]);
            if (lane == 0) part[warp][g * TT + t] = v;
        }
    __syncthreads();
    const int t = threadIdx.x / ML_HG, hg = threadIdx.x % ML_HG, row = t0 + t, h = h0 + hg;
    if (t >= TT || row >= rows || h >= G.heads) return;
    float zi = 0.f, zf = 0.f;
#pragma unroll
    for (int w = 0; w < ML_WARPS; ++w) { zi += part[w][hg * TT + t]; zf += part[w][(ML_HG + hg) * TT + t]; }
    if (!gates) {
        z[(size_t)row * 2 * G.heads + h] = zi;
        z[(size_t)row * 2 * G.heads + G.heads + h] = zf;
    } else if (row < n_seqs) {
        float* m_slot = G.state + (size_t)G.seq_slots[row] * G.ld_state + h;
        const float i = ml_soft(zi + G.bias[h], G.cap), f = ml_logsigmoid(ml_soft(zf + G.bias[G.heads + h], G.cap));
        const float before = *m_slot, m = fmaxf(f + before, i);
        ml_factors(G, (size_t)row, h, f, i, before, m);
        *m_slot = m;
    }
}

}  // namespace kl

using namespace kl;

// x: [rows, width] in the compute dtype; W [2 * heads, width] (the input gates' rows, then the forget gates'); bias float32
// [2 * heads]; state: the slots' running maxima; a, c, floor: float32 [rows, heads], or logs: float32 [4, rows, heads] in their
// place (see MlstmGates); z: float32 [rows, 2 * heads] scratch (null where single != 0: every sequence brings one token and rows
// are in the order of the sequences).
KL_API int kl_mlstm_gates(const void* x, long long ld_x, const void* W, int width, const float* bias, float cap, float* state,
                          long long ld_state, float* z, float* a, float* c, float* floor, float* logs, const int* cu_tokens, const int* seq_slots,
                          int rows, int n_seqs, int max_new, int heads, int single, int dtype, cudaStream_t stream) {
    if (rows <= 0 || n_seqs <= 0) return KL_OK;
    if (heads <= 0 || width <= 0 || !(cap > 0.f) || n_seqs > 65535 || heads > 65535 || (!single && z == nullptr)) return KL_ERR_BAD_SIZE;
    if (dtype != KL_F32 && dtype != KL_BF16) return KL_ERR_BAD_DTYPE;
    const MlstmGates G{bias, state, ld_state, a, c, floor, logs, (long long)rows * heads, cu_tokens, seq_slots, heads, cap};
    const int tt = rows <= 256 ? 1 : 4;
    const dim3 grid((rows + tt - 1) / tt, (heads + ML_HG - 1) / ML_HG);
#define KL_GP(T, TT) launch_kernel(mlstm_gate_project_kernel<T, TT>, grid, ML_WARPS * 32, 0, stream, (const T*)x, ld_x, (const T*)W, width, rows, n_seqs, single, z, G)
    if (dtype == KL_F32) { if (tt == 1) KL_GP(float, 1); else KL_GP(float, 4); }
    else { if (tt == 1) KL_GP(bf16, 1); else KL_GP(bf16, 4); }
#undef KL_GP
    KL_LAUNCH_CHECK();
    if (single) return KL_OK;
    int threads = 32;
    while (threads < ML_SCAN_THREADS && threads < max_new) threads <<= 1;
    launch_kernel(mlstm_gates_kernel, dim3(n_seqs, heads), threads, 0, stream, G, (const float*)z, (long long)2 * heads);
    KL_LAUNCH_CHECK();
    return KL_OK;
}
