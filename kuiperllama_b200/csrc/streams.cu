// Several residual streams side by side (hyper-connections): one kernel between two sublayers.
//
// A token has S streams x_1 .. x_S (float32 [tokens, S, hidden]) instead of one.  The sublayer before left its result y
// (`delta`: rows in the compute dtype, or float32 pieces of a product, added in ascending order), the sublayer after reads a
// normed combination of the new streams:
//
//   x'_t = sum_s mix[s, t] x_s + out_w[t] y            (every t from the old streams; no mix: the streams stay, y is ignored)
//   u    = sum_t in_w[t] x'_t                          (no in_w: the plain sum)
//   out  = u / sqrt(mean(u^2) + eps) * w
//
// All of it in 32 bits; the new streams are written to `dst` (null: not written), which may be `src`.  With a stream stride
// of zero all S old streams are one row (a model's first sublayers, where every stream is the embedding's row).
//
//   stream_norm_vec_kernel   S of 1, 2, 3, 4; four floats an access; the row's u in registers between the two passes.
//   stream_norm_kernel       up to 16 streams, any width; u passes through shared memory.
//
// ExiledOfCode/KuiperLLama has one residual stream (kuiper/source/model/llama3.cpp:155-164).
#include "common.cuh"

namespace kl {

constexpr int ST_MAX_STREAMS = 16;

struct StreamNorm {
    const float* src; long long src_stream, src_row;       // strides in elements
    float* dst;                                            // [rows][S][hidden] or null
    const void* delta; long long delta_ld;                 // rows in the compute dtype, or null
    const float* pieces; int n_pieces; long long piece_stride;   // float32 [n_pieces][rows][hidden], or null
    const float* mix; const float* out_w; const float* in_w;
    const float* w; float eps;
    void* out;                                             // compute dtype [rows][hidden], or null (the streams alone)
    const int* rows;                                       // row r of `out` reads source row rows[r] (null: r)
    int streams, hidden;
};

template <typename T> struct Quad;
template <> struct Quad<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Quad<bf16> {
    static __device__ __forceinline__ float4 load(const bf16* p) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(bf16* p, float4 v) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&a);
        raw.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    }
};
__device__ __forceinline__ float4 axpy4(float a, float4 x, float4 y) {
    return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}
__device__ __forceinline__ float4 scale4(float a, float4 x) { return make_float4(a * x.x, a * x.y, a * x.z, a * x.w); }

template <typename T, int S, int THREADS, int VPT>
__global__ void __launch_bounds__(THREADS)
stream_norm_vec_kernel(const StreamNorm A) {
    pdl_launch_dependents();
    // the weights are written by no kernel
    float mix[S][S], ow[S], iw[S];
    const bool update = A.mix != nullptr;
#pragma unroll
    for (int s = 0; s < S; ++s) {
        ow[s] = update ? A.out_w[s] : 0.f;
        iw[s] = A.in_w != nullptr ? A.in_w[s] : 1.f;
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s][t] = update ? A.mix[s * S + t] : 0.f;
    }
    pdl_wait();
    __shared__ float scratch[33];
    const int hidden = A.hidden, n4 = hidden >> 2;
    const int r = blockIdx.x;
    const int row = A.rows ? A.rows[r] : r;
    const float* src = A.src + (size_t)row * A.src_row;
    float* dst = A.dst ? A.dst + (size_t)row * S * hidden : nullptr;
    const T* d = A.delta ? (const T*)A.delta + (size_t)row * A.delta_ld : nullptr;
    const float* p = A.n_pieces > 0 ? A.pieces + (size_t)row * hidden : nullptr;
    float4 u[VPT];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i4 = threadIdx.x + j * THREADS;
        u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i4 >= n4) continue;
        float4 x[S];
#pragma unroll
        for (int s = 0; s < S; ++s) x[s] = *reinterpret_cast<const float4*>(src + (size_t)s * A.src_stream + 4 * i4);
        if (update) {
            float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
            if (d != nullptr) y = Quad<T>::load(d + 4 * i4);
            // four pieces (eight in the form for few rows) are requested at a time and added in ascending order
            constexpr int ZB = THREADS == 512 && VPT == 1 ? 8 : 4;
            for (int z0 = 0; z0 < A.n_pieces; z0 += ZB) {
                float4 b[ZB];
#pragma unroll
                for (int z = 0; z < ZB; ++z)
                    b[z] = z0 + z < A.n_pieces ? *reinterpret_cast<const float4*>(p + (size_t)(z0 + z) * A.piece_stride + 4 * i4)
                                               : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int z = 0; z < ZB; ++z) { y.x += b[z].x; y.y += b[z].y; y.z += b[z].z; y.w += b[z].w; }
            }
            float4 n[S];
#pragma unroll
            for (int t = 0; t < S; ++t) {
                n[t] = scale4(mix[0][t], x[0]);
#pragma unroll
                for (int s = 1; s < S; ++s) n[t] = axpy4(mix[s][t], x[s], n[t]);
                n[t] = axpy4(ow[t], y, n[t]);
                if (dst != nullptr) *reinterpret_cast<float4*>(dst + (size_t)t * hidden + 4 * i4) = n[t];
            }
#pragma unroll
            for (int t = 0; t < S; ++t) x[t] = n[t];
        } else if (dst != nullptr) {
#pragma unroll
            for (int t = 0; t < S; ++t) *reinterpret_cast<float4*>(dst + (size_t)t * hidden + 4 * i4) = x[t];
        }
        u[j] = scale4(iw[0], x[0]);
#pragma unroll
        for (int t = 1; t < S; ++t) u[j] = axpy4(iw[t], x[t], u[j]);
        ss += (u[j].x * u[j].x + u[j].y * u[j].y) + (u[j].z * u[j].z + u[j].w * u[j].w);
    }
    if (A.out == nullptr) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + A.eps);
    T* o = (T*)A.out + (size_t)r * hidden;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i4 = threadIdx.x + j * THREADS;
        if (i4 >= n4) continue;
        const float4 w = *reinterpret_cast<const float4*>(A.w + 4 * i4);
        Quad<T>::store(o + 4 * i4, make_float4(u[j].x * inv * w.x, u[j].y * inv * w.y, u[j].z * inv * w.z, u[j].w * inv * w.w));
    }
}

template <typename T>
__global__ void __launch_bounds__(256)
stream_norm_kernel(const StreamNorm A) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float us[];                          // [hidden]: a thread reads back its own elements only
    __shared__ float scratch[33];
    const int hidden = A.hidden, S = A.streams;
    const int r = blockIdx.x;
    const int row = A.rows ? A.rows[r] : r;
    const float* src = A.src + (size_t)row * A.src_row;
    float* dst = A.dst ? A.dst + (size_t)row * S * hidden : nullptr;
    const T* d = A.delta ? (const T*)A.delta + (size_t)row * A.delta_ld : nullptr;
    float ss = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float x[ST_MAX_STREAMS];
        for (int s = 0; s < S; ++s) x[s] = src[(size_t)s * A.src_stream + i];
        float y = d != nullptr ? to_f32(d[i]) : 0.f;
        for (int z = 0; z < A.n_pieces; ++z) y += A.pieces[(size_t)z * A.piece_stride + (size_t)row * hidden + i];
        float u = 0.f;
        for (int t = 0; t < S; ++t) {
            float n = x[t];
            if (A.mix != nullptr) {
                n = A.mix[t] * x[0];
                for (int s = 1; s < S; ++s) n = fmaf(A.mix[s * S + t], x[s], n);
                n = fmaf(A.out_w[t], y, n);
            }
            if (dst != nullptr) dst[(size_t)t * hidden + i] = n;
            const float a = A.in_w != nullptr ? A.in_w[t] : 1.f;
            u = t == 0 ? a * n : fmaf(a, n, u);
        }
        us[i] = u;
        ss += u * u;
    }
    if (A.out == nullptr) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + A.eps);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) ((T*)A.out)[(size_t)r * hidden + i] = from_f32<T>(us[i] * inv * A.w[i]);
}

}  // namespace kl

using namespace kl;

// delta (compute dtype, rows delta_ld apart) and pieces exclude each other; both null with mix: y = 0.  out null: w may be null too.
KL_API int kl_stream_norm(const float* src, long long src_stream, long long src_row, float* dst, const void* delta, long long delta_ld,
                          const float* pieces, int n_pieces, long long piece_stride, const float* mix, const float* out_w,
                          const float* in_w, const float* w, float eps, void* out, const int* rows, int n_rows, int streams, int hidden,
                          int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return KL_OK;
    if (streams < 1 || streams > ST_MAX_STREAMS || hidden <= 0 || hidden > 48 * 1024) return KL_ERR_BAD_SIZE;
    if ((out != nullptr && w == nullptr) || (mix != nullptr && out_w == nullptr) || n_pieces < 0 || (n_pieces > 0 && pieces == nullptr) ||
        (delta != nullptr && n_pieces > 0)) return KL_ERR_BAD_SIZE;
    if (dst != nullptr && rows != nullptr) return KL_ERR_BAD_SIZE;      // rows may name a row twice
    if (dtype != KL_F32 && dtype != KL_BF16) return KL_ERR_BAD_DTYPE;
    StreamNorm A{src, src_stream, src_row, dst, delta, delta_ld, pieces, n_pieces, piece_stride, mix, out_w, in_w, w, eps, out, rows, streams, hidden};
    const uintptr_t m = dtype == KL_BF16 ? 7 : 15;
    const int n4 = hidden / 4;
    const bool aligned = hidden % 4 == 0 && src_stream % 4 == 0 && src_row % 4 == 0 && delta_ld % 4 == 0 && piece_stride % 4 == 0 &&
                         (((uintptr_t)src | (uintptr_t)dst | (uintptr_t)pieces | (uintptr_t)w) & 15) == 0 && (((uintptr_t)delta | (uintptr_t)out) & m) == 0;
    if (aligned && streams <= 4 && n4 <= 2048) {
#define KL_SV(T, S, THREADS, VPT) launch_kernel(stream_norm_vec_kernel<T, S, THREADS, VPT>, n_rows, THREADS, 0, stream, A)
#define KL_SV_BY(T, S)                                                                                                                   \
    do {                                                                                                                                  \
        /* few rows of a wide model (decode): a row over 512 or 1,024 threads, so that one round of loads fetches it */                   \
        if (n_rows <= 256 && n4 > 256) { if (n4 <= 512) KL_SV(T, S, 512, 1); else if (n4 <= 1024) KL_SV(T, S, 1024, 1); else KL_SV(T, S, 1024, 2); } \
        else if (n4 <= 64) KL_SV(T, S, 64, 1); else if (n4 <= 128) KL_SV(T, S, 128, 1); else if (n4 <= 256) KL_SV(T, S, 256, 1);         \
        else if (n4 <= 512) KL_SV(T, S, 256, 2); else if (n4 <= 1024) KL_SV(T, S, 512, 2); else KL_SV(T, S, 512, 4);                     \
    } while (0)
#define KL_SV_S(T)                                                                                       \
    do {                                                                                                 \
        if (streams == 1) KL_SV_BY(T, 1); else if (streams == 2) KL_SV_BY(T, 2);                         \
        else if (streams == 3) KL_SV_BY(T, 3); else KL_SV_BY(T, 4);                                      \
    } while (0)
        if (dtype == KL_BF16) KL_SV_S(bf16); else KL_SV_S(float);
#undef KL_SV_S
#undef KL_SV_BY
#undef KL_SV
        KL_LAUNCH_CHECK();
        return KL_OK;
    }
    const size_t smem = (size_t)hidden * sizeof(float);
    if (dtype == KL_F32) {
        if (smem > 48 * 1024) KL_CUDA(cudaFuncSetAttribute(stream_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        launch_kernel(stream_norm_kernel<float>, n_rows, 256, smem, stream, A);
    } else {
        if (smem > 48 * 1024) KL_CUDA(cudaFuncSetAttribute(stream_norm_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        launch_kernel(stream_norm_kernel<bf16>, n_rows, 256, smem, stream, A);
    }
    KL_LAUNCH_CHECK();
    return KL_OK;
}
