// Causal grouped-query attention over the paged cache, plain SIMT arithmetic in 32 bits.
//
// This is the kernel of the true 32-bit path (prefill and decode) and the fallback of the
// bfloat16 path for sizes and options that the tensor-core kernels refuse (a window, a
// head size that is not on their list; any key size and value sizes up to 512 run here).  One CTA of four warps per
// (token, query head).  Query token t of slot s at position p reads keys lo..p of that
// slot, lo = max(0, p - window + 1) with a window, else 0.  Head h reads kv head
// h / (H / KV); score = (q . k) * scale; softmax with the maximum subtracted; o = sum p v
// (ExiledOfCode/KuiperLLama mha_kernel.cu:61,74-106; there one CTA per head loops over one
// sequence and the scores pass through global memory).
//
// Keys are cut into chunks of 32 by absolute position and the chunks are dealt to the warps
// round-robin, so the order of every sum depends only on the token's own position: the
// result does not change with the way tokens are cut into steps or batched.
//
// Options beyond KuiperLLama's attention: values of another size than the keys (`vd` columns of rows
// that are `v_ld` apart; with v_cache == k_cache and v_ld == hd the values are the leading columns of
// the keys, which is what attention over a shared latent reads), and a sink: a learned number per
// head that joins the softmax's denominator as exp(sink) and has no value; chunks: a token reads the keys of its own chunk
// of `chunk` positions, counted from position 0; and a learned bias by distance: rel[h, min(pos - key, rel_n - 1)] is
// added to the scaled score.
#include "common.cuh"

namespace kl {

constexpr int ATT_WARPS = 4;
constexpr int ATT_MAX_VALUE_DIM = 512;   // value columns per head (32 lanes x PL, PL = 8 or 16)

template <typename T>
__device__ __forceinline__ float dot_row(const T* __restrict__ k, const float* __restrict__ q, int hd);

// Head sizes whose rows do not start on 16-byte boundaries take the element-by-element form.
template <typename T>
__device__ __forceinline__ float dot_row_scalar(const T* __restrict__ k, const float* __restrict__ q, int hd) {
    float s = 0.f;
    for (int i = 0; i < hd; ++i) s += to_f32(k[i]) * q[i];
    return s;
}

template <>
__device__ __forceinline__ float dot_row<float>(const float* __restrict__ k, const float* __restrict__ q, int hd) {
    if (hd & 3) return dot_row_scalar(k, q, hd);
    float s = 0.f;
    for (int i = 0; i < hd; i += 4) {
        const float4 kv = *reinterpret_cast<const float4*>(k + i);
        s += kv.x * q[i] + kv.y * q[i + 1] + kv.z * q[i + 2] + kv.w * q[i + 3];
    }
    return s;
}
template <>
__device__ __forceinline__ float dot_row<bf16>(const bf16* __restrict__ k, const float* __restrict__ q, int hd) {
    if (hd & 7) return dot_row_scalar(k, q, hd);
    float s = 0.f;
    for (int i = 0; i < hd; i += 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(k + i);
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 f = __bfloat1622float2(p[j]);
            s += f.x * q[i + 2 * j] + f.y * q[i + 2 * j + 1];
        }
    }
    return s;
}

template <typename T, int PL>
__global__ void __launch_bounds__(ATT_WARPS * 32)
attention_simt_kernel(const T* __restrict__ q, int q_stride, T* __restrict__ out,
                      const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                      const int* __restrict__ block_table, int blocks_per_seq,
                      const int* __restrict__ positions, const int* __restrict__ token_slot,
                      int H, int KV, int hd, float scale, int window, int vd, int v_ld, const float* __restrict__ sink, int chunk,
                      const float* __restrict__ rel, int rel_n) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float smem[];
    float* q_s = smem;                               // [hd]
    float* m_s = q_s + hd;                           // [ATT_WARPS]
    float* l_s = m_s + ATT_WARPS;                    // [ATT_WARPS]
    float* acc_s = l_s + ATT_WARPS;                  // [ATT_WARPS][vd]

    const int t = blockIdx.x, h = blockIdx.y;
    const int slot = token_slot[t];
    if (slot < 0) return;                            // a padding row: nothing is written
    const int pos = positions[t];
    const int g = h / (H / KV);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;

    const T* qrow = q + (size_t)t * q_stride + (size_t)h * hd;
    for (int i = threadIdx.x; i < hd; i += blockDim.x) q_s[i] = to_f32(qrow[i]);
    __syncthreads();

    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    float m = -INFINITY, l = 0.f;
    float acc[PL];
#pragma unroll
    for (int i = 0; i < PL; ++i) acc[i] = 0.f;

    const int* table = block_table + (size_t)slot * blocks_per_seq;
    for (int c = lo / 32 + warp; c * 32 <= pos; c += ATT_WARPS) {
        const int base = c * 32;                                     // 32 keys inside one page
        const int page = table[base / PAGE];
        const size_t page_off = (((size_t)page * KV + g) * PAGE + (base % PAGE)) * (size_t)hd;
        const int key = base + lane;
        const bool valid = key >= lo && key <= pos;
        float s = -INFINITY;
        if (valid) {
            s = dot_row<T>(k_cache + page_off + (size_t)lane * hd, q_s, hd) * scale;
            if (rel != nullptr) s += rel[(size_t)h * rel_n + min(pos - key, rel_n - 1)];
        }
        const float m_new = fmaxf(m, warp_max(s));                   // finite: the chunk holds a valid key
        const float corr = expf(m - m_new);                          // exp(-inf) = 0 at the first chunk
        const float p = valid ? expf(s - m_new) : 0.f;
        l = l * corr + warp_sum(p);
        m = m_new;
#pragma unroll
        for (int i = 0; i < PL; ++i) acc[i] *= corr;
        const int j_lo = max(lo - base, 0), j_hi = min(pos - base, 31);
        const T* vbase = v_cache + (((size_t)page * KV + g) * PAGE + (base % PAGE)) * (size_t)v_ld;
        for (int j = j_lo; j <= j_hi; ++j) {
            const float pj = __shfl_sync(0xffffffffu, p, j);
            const T* vrow = vbase + (size_t)j * v_ld;
#pragma unroll
            for (int i = 0; i < PL; ++i) {
                const int d = lane + 32 * i;
                if (d < vd) acc[i] += pj * to_f32(vrow[d]);
            }
        }
    }
    if (lane == 0) { m_s[warp] = m; l_s[warp] = l; }
#pragma unroll
    for (int i = 0; i < PL; ++i) {
        const int d = lane + 32 * i;
        if (d < vd) acc_s[warp * vd + d] = acc[i];
    }
    __syncthreads();
    float M = m_s[0];
#pragma unroll
    for (int w = 1; w < ATT_WARPS; ++w) M = fmaxf(M, m_s[w]);
    const float snk = sink ? sink[h] : -INFINITY;
    M = fmaxf(M, snk);
    float L = sink ? expf(snk - M) : 0.f;
    float wgt[ATT_WARPS];
#pragma unroll
    for (int w = 0; w < ATT_WARPS; ++w) {
        wgt[w] = m_s[w] == -INFINITY ? 0.f : expf(m_s[w] - M);
        L += l_s[w] * wgt[w];
    }
    T* orow = out + ((size_t)t * H + h) * vd;
    for (int d = threadIdx.x; d < vd; d += blockDim.x) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < ATT_WARPS; ++w) o += acc_s[w * vd + d] * wgt[w];
        orow[d] = from_f32<T>(o / L);
    }
}

}  // namespace kl

using namespace kl;

// q: rows of q_stride elements, head h at column h * hd.  out: [tokens, H * vd].  vd <= 0 means values like
// keys (vd = v_ld = hd).  sink: float32 [H] or null.  chunk: positions per chunk (0: none).  rel: float32 [H, rel_n] or null.
KL_API int kl_attention_simt(const void* q, int q_stride, void* out, const void* k_cache, const void* v_cache,
                             const int* block_table, int blocks_per_seq, const int* positions,
                             const int* token_slot, int n_tokens, int H, int KV, int hd, float scale, int window,
                             int vd, int v_ld, const float* sink, int chunk, const float* rel, int rel_n, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return KL_OK;
    if (vd <= 0) { vd = hd; v_ld = hd; }
    if (vd > ATT_MAX_VALUE_DIM || hd <= 0 || v_ld < vd || KV <= 0 || H % KV) return KL_ERR_BAD_SIZE;
    if (H > 65535 || chunk < 0 || (rel != nullptr && rel_n < 1)) return KL_ERR_BAD_SIZE;
    const dim3 grid(n_tokens, H);
    const size_t smem = (size_t)(hd + 2 * ATT_WARPS + ATT_WARPS * vd) * sizeof(float);
    if (smem > 200 * 1024) return KL_ERR_BAD_SIZE;
#define KL_ATT(T, PL)                                                                                                         \
    do {                                                                                                                      \
        if (smem > 48 * 1024) KL_CUDA(cudaFuncSetAttribute(attention_simt_kernel<T, PL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        launch_kernel(attention_simt_kernel<T, PL>, grid, ATT_WARPS * 32, smem, stream, (const T*)q, q_stride, (T*)out,       \
                      (const T*)k_cache, (const T*)v_cache, block_table, blocks_per_seq, positions, token_slot, H, KV, hd,    \
                      scale, window, vd, v_ld, sink, chunk, rel, rel_n);                                                                         \
    } while (0)
    if (dtype == KL_F32) { if (vd <= 256) KL_ATT(float, 8); else KL_ATT(float, 16); }
    else if (dtype == KL_BF16) { if (vd <= 256) KL_ATT(bf16, 8); else KL_ATT(bf16, 16); }
    else return KL_ERR_BAD_DTYPE;
#undef KL_ATT
    KL_LAUNCH_CHECK();
    return KL_OK;
}
