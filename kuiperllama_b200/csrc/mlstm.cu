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
//   mlstm_gate_project_kernel   the pre-activations themselves, z = W h in 32 bits (W: 2 * heads rows): a warp per head and tile of
//                               tokens; in a step of single tokens it makes a, c and floor at once.
//
// ExiledOfCode/KuiperLLama has no recurrent mixer (its mixer is mha_kernel.cu:61,74-106).
#include "common.cuh"

namespace kl {

struct MlstmGates {
    const float* bias;                        // [2 * heads]: the input gate's, then the forget gate's
    float* state; long long ld_state;         // the slot's m at state + slot * ld_state, [heads]
    float* a; float* c; float* floor;         // [rows, heads]
    const int* cu_tokens; const int* seq_slots;
    int heads;
    float cap;
};

__device__ __forceinline__ float ml_soft(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// What one token does to the running maximum, and the three factors that come of it.
__device__ __forceinline__ void ml_factors(const MlstmGates& G, size_t row, int h, float f, float i, float m_before, float m) {
    const size_t at = row * G.heads + h;
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

// W: [2 * heads, width] in the compute dtype; x rows of the compute dtype.  Grid (tiles of TT tokens, heads / warps).  With
// `gates` (every sequence brings one token, row = sequence) the warp finishes its head; else z float32 [rows, 2 * heads].
template <typename T, int TT>
__global__ void __launch_bounds__(128)
mlstm_gate_project_kernel(const T* __restrict__ x, long long ld_x, const T* __restrict__ W, int width, int rows, int n_seqs, int gates,
                          float* __restrict__ z, const MlstmGates G) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, h = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (h >= G.heads) return;
    const int t0 = blockIdx.x * TT;
    const T* wi = W + (size_t)h * width;
    const T* wf = W + (size_t)(G.heads + h) * width;
    float ai[TT], af[TT];
#pragma unroll
    for (int t = 0; t < TT; ++t) { ai[t] = 0.f; af[t] = 0.f; }
    constexpr int V = 16 / sizeof(T);
    const bool vec = width % V == 0 && ld_x % V == 0 && ((((uintptr_t)x) | ((uintptr_t)W)) & 15) == 0;
    if (vec) {
#pragma unroll 2
        for (int c = lane * V; c < width; c += 32 * V) {
            const uint4 ri = *reinterpret_cast<const uint4*>(wi + c), rf = *reinterpret_cast<const uint4*>(wf + c);
            const T* pi = reinterpret_cast<const T*>(&ri); const T* pf = reinterpret_cast<const T*>(&rf);
#pragma unroll
            for (int t = 0; t < TT; ++t) {
                if (t0 + t >= rows) break;
                const uint4 rx = *reinterpret_cast<const uint4*>(x + (size_t)(t0 + t) * ld_x + c);
                const T* px = reinterpret_cast<const T*>(&rx);
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    const float xv = to_f32(px[e]);
                    ai[t] = fmaf(to_f32(pi[e]), xv, ai[t]);
                    af[t] = fmaf(to_f32(pf[e]), xv, af[t]);
                }
            }
        }
    } else {
        for (int c = lane; c < width; c += 32) {
            const float vi = to_f32(wi[c]), vf = to_f32(wf[c]);
#pragma unroll
            for (int t = 0; t < TT; ++t) {
                if (t0 + t >= rows) break;
                const float xv = to_f32(x[(size_t)(t0 + t) * ld_x + c]);
                ai[t] = fmaf(vi, xv, ai[t]);
                af[t] = fmaf(vf, xv, af[t]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < TT; ++t) {
        const int row = t0 + t;
        if (row >= rows) break;
        const float zi = warp_sum(ai[t]), zf = warp_sum(af[t]);
        if (lane != 0) continue;
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
}

}  // namespace kl

using namespace kl;

// x: [rows, width] in the compute dtype; W [2 * heads, width] (the input gates' rows, then the forget gates'); bias float32
// [2 * heads]; state: the slots' running maxima; a, c, floor: float32 [rows, heads]; z: float32 [rows, 2 * heads] scratch (null
// where single != 0: every sequence brings one token and rows are in the order of the sequences).
KL_API int kl_mlstm_gates(const void* x, long long ld_x, const void* W, int width, const float* bias, float cap, float* state,
                          long long ld_state, float* z, float* a, float* c, float* floor, const int* cu_tokens, const int* seq_slots,
                          int rows, int n_seqs, int max_new, int heads, int single, int dtype, cudaStream_t stream) {
    if (rows <= 0 || n_seqs <= 0) return KL_OK;
    if (heads <= 0 || width <= 0 || !(cap > 0.f) || n_seqs > 65535 || heads > 65535 || (!single && z == nullptr)) return KL_ERR_BAD_SIZE;
    if (dtype != KL_F32 && dtype != KL_BF16) return KL_ERR_BAD_DTYPE;
    const MlstmGates G{bias, state, ld_state, a, c, floor, cu_tokens, seq_slots, heads, cap};
    const int tt = rows <= 256 ? 1 : 8;
    const dim3 grid((rows + tt - 1) / tt, (heads + 3) / 4);
#define KL_GP(T, TT) launch_kernel(mlstm_gate_project_kernel<T, TT>, grid, 128, 0, stream, (const T*)x, ld_x, (const T*)W, width, rows, n_seqs, single, z, G)
    if (dtype == KL_F32) { if (tt == 1) KL_GP(float, 1); else KL_GP(float, 8); }
    else { if (tt == 1) KL_GP(bf16, 1); else KL_GP(bf16, 8); }
#undef KL_GP
    KL_LAUNCH_CHECK();
    if (single) return KL_OK;
    int threads = 32;
    while (threads < ML_SCAN_THREADS && threads < max_new) threads <<= 1;
    launch_kernel(mlstm_gates_kernel, dim3(n_seqs, heads), threads, 0, stream, G, (const float*)z, (long long)2 * heads);
    KL_LAUNCH_CHECK();
    return KL_OK;
}
