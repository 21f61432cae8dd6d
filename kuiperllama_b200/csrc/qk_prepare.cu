// What grouped-query attention needs between its input product and the scores, as one kernel per step with
// every step optional: for every token
//
//   * a bias is added to the projected q, k and v (float32 vectors),
//   * the first `rot` elements of every q and k head turn by the token's position, in pairs (2i, 2i + 1)
//     (interleaved) or (i, i + rot / 2); angle = position * inv_freq[i] in 32 bits with sincosf,
//   * every q and k head is divided by its root mean square over the head (eps inside the root) and
//     multiplied by a weight per element (one vector for the q heads, one for the k heads) where one is given,
//   * q is written back where it came from, k into the token's row of the paged cache, and v (as projected,
//     with its bias) into the value cache, whose rows may have another size than the keys'; with v_col < 0
//     there is no value projection and the key heads as projected (with bias, before rotation and norm)
//     are stored as values.
//
// A token's heads are dealt to the CTAs of its grid row, a warp per head, and the head passes through a row of
// shared memory, so the order of a head's sum of squares depends on the head size only.  ExiledOfCode/KuiperLLama
// rotates whole heads from tables and has neither biases nor norms on q and k (rope_kernel.cu:5-49,
// kuiper/source/model/llama3.cpp:610-639).
#include "common.cuh"

namespace kl {

constexpr int QKP_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(QKP_WARPS * 32)
qk_prepare_kernel(T* __restrict__ proj, long long ld, int q_col, int k_col, int v_col,
                  const float* __restrict__ q_bias, const float* __restrict__ k_bias, const float* __restrict__ v_bias,
                  const float* __restrict__ inv_freq, int rot, int interleaved,
                  int head_norm, float eps, const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w,
                  const int* __restrict__ positions, const int* __restrict__ token_slot,
                  const int* __restrict__ block_table, int blocks_per_seq,
                  T* __restrict__ k_cache, T* __restrict__ v_cache, int H, int KV, int hd, int vd) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float smem[];
    float* cs = smem;                                   // [rot]: cos, sin of every pair
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    if (slot < 0) return;                               // a padding row
    const int pos = positions[t];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* buf = smem + rot + (size_t)warp * hd;        // [hd] per warp
    for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
        float s, c;
        sincosf((float)pos * inv_freq[i], &s, &c);
        cs[2 * i] = c;
        cs[2 * i + 1] = s;
    }
    __syncthreads();
    T* row = proj + (size_t)t * ld;
    const bool write = k_cache != nullptr;
    const int half = rot / 2;
    for (int head = blockIdx.y * QKP_WARPS + warp; head < H + KV; head += gridDim.y * QKP_WARPS) {
        const bool is_q = head < H;
        if (!is_q && !write) continue;
        const int g = is_q ? head : head - H;
        T* src = row + (is_q ? q_col + (size_t)g * hd : k_col + (size_t)g * hd);
        const float* bias = is_q ? q_bias : k_bias;
        T* vdst = (!is_q && v_col < 0) ? v_cache + cache_row_offset(block_table, blocks_per_seq, slot, pos, g, KV, vd) : nullptr;
        for (int i = lane; i < hd; i += 32) {
            const float x = to_f32(src[i]) + (bias ? bias[(size_t)g * hd + i] : 0.f);
            buf[i] = x;
            if (vdst != nullptr) vdst[i] = from_f32<T>(x);          // the values are the keys as projected
        }
        __syncwarp();
        for (int i = lane; i < half; i += 32) {
            const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + half;
            const float u = buf[a], v = buf[b], c = cs[2 * i], s = cs[2 * i + 1];
            buf[a] = u * c - v * s;
            buf[b] = v * c + u * s;
        }
        __syncwarp();
        float inv = 1.f;
        if (head_norm) {
            float ss = 0.f;
            for (int i = lane; i < hd; i += 32) ss += buf[i] * buf[i];
            ss = warp_sum(ss);
            inv = 1.0f / sqrtf(ss / (float)hd + eps);
        }
        const float* w = is_q ? q_norm_w : k_norm_w;
        T* dst = is_q ? src : k_cache + cache_row_offset(block_table, blocks_per_seq, slot, pos, g, KV, hd);
        for (int i = lane; i < hd; i += 32) dst[i] = from_f32<T>(w ? buf[i] * inv * w[i] : buf[i] * inv);
        __syncwarp();
    }
    if (write && v_col >= 0) {
        for (int idx = blockIdx.y * blockDim.x + threadIdx.x; idx < KV * vd; idx += gridDim.y * blockDim.x) {
            const int g = idx / vd, e = idx - g * vd;
            T* dst = v_cache + cache_row_offset(block_table, blocks_per_seq, slot, pos, g, KV, vd);
            dst[e] = from_f32<T>(to_f32(row[(size_t)v_col + idx]) + (v_bias ? v_bias[idx] : 0.f));
        }
    }
}

// The same for bfloat16 rows on 16-byte boundaries and head sizes of 8 L with L a power of two up to 32: a lane holds eight
// neighbouring elements of a head (one 16-byte access each way), L lanes a head, so a warp carries 512 bytes a load instead
// of 64 and a tenth as many warps move the same rows.  Interleaved pairs lie inside a lane's eight elements; a pair
// (i, i + rot / 2) has its partner rot / 16 lanes away (rot a multiple of 16) and comes by shuffle.  The head's sum of squares
// is added over the lane's elements in order, then over the L lanes by shuffles.
template <int L>
__global__ void __launch_bounds__(256)
qk_prepare_vec_kernel(bf16* __restrict__ proj, long long ld, int q_col, int k_col, int v_col,
                      const float* __restrict__ q_bias, const float* __restrict__ k_bias, const float* __restrict__ v_bias,
                      const float* __restrict__ inv_freq, int rot, int interleaved,
                      int head_norm, float eps, const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w,
                      const int* __restrict__ positions, const int* __restrict__ token_slot,
                      const int* __restrict__ block_table, int blocks_per_seq,
                      bf16* __restrict__ k_cache, bf16* __restrict__ v_cache, int H, int KV, int vd) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int hd = 8 * L;
    extern __shared__ float smem[];
    float* cs = smem;                                   // [rot]: cos, sin of every pair
    const int t = blockIdx.x;
    const int slot = token_slot[t];
    if (slot < 0) return;                               // a padding row
    const int pos = positions[t];
    for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
        float sn, c;
        sincosf((float)pos * inv_freq[i], &sn, &c);
        cs[2 * i] = c;
        cs[2 * i + 1] = sn;
    }
    __syncthreads();
    bf16* row = proj + (size_t)t * ld;
    const bool write = k_cache != nullptr;
    const int half = rot / 2;
    const int part = threadIdx.x % L;                   // which eight elements of the head
    const int e0 = part * 8;
    // every thread of the warp walks the same number of turns, so the shuffles below are whole
    const int per_turn = gridDim.y * (blockDim.x / L);
    for (int base = blockIdx.y * (blockDim.x / L); base < H + KV; base += per_turn) {
        const int head = base + threadIdx.x / L;
        const bool live = head < H + KV && (head < H || write);
        const bool is_q = head < H;
        const int g = is_q ? head : head - H;
        float x[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = 0.f;
        bf16* src = row + (is_q ? q_col + (size_t)g * hd : k_col + (size_t)g * hd) + e0;
        if (live) {
            const uint4 raw = *reinterpret_cast<const uint4*>(src);
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
            for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(p[e]); x[2 * e] = f.x; x[2 * e + 1] = f.y; }
            const float* bias = is_q ? q_bias : k_bias;
            if (bias != nullptr) {
                const float4 b0 = *reinterpret_cast<const float4*>(bias + (size_t)g * hd + e0), b1 = *reinterpret_cast<const float4*>(bias + (size_t)g * hd + e0 + 4);
                x[0] += b0.x; x[1] += b0.y; x[2] += b0.z; x[3] += b0.w; x[4] += b1.x; x[5] += b1.y; x[6] += b1.z; x[7] += b1.w;
            }
            if (!is_q && v_col < 0) {                   // the values are the keys as projected
                uint4 out;
                __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
                for (int e = 0; e < 4; ++e) o[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
                *reinterpret_cast<uint4*>(v_cache + cache_row_offset(block_table, blocks_per_seq, slot, pos, g, KV, vd) + e0) = out;
            }
        }
        if (rot > 0) {
            if (interleaved) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = (e0 >> 1) + e;        // the pair's index in the head
                    if (i < half) {
                        const float u = x[2 * e], v = x[2 * e + 1], c = cs[2 * i], sn = cs[2 * i + 1];
                        x[2 * e] = u * c - v * sn;
                        x[2 * e + 1] = v * c + u * sn;
                    }
                }
            } else {
                // the partner of element a < rot / 2 is a + rot / 2, rot / 16 lanes up; of a in [rot / 2, rot) it is rot / 16 lanes down
                const int away = half >> 3;
                const bool low = e0 < half, in = e0 < rot;
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const float up = __shfl_down_sync(0xffffffffu, x[e], away), down = __shfl_up_sync(0xffffffffu, x[e], away);
                    if (in) {
                        const int i = (low ? e0 : e0 - half) + e;
                        const float c = cs[2 * i], sn = cs[2 * i + 1];
                        x[e] = low ? x[e] * c - up * sn : x[e] * c + down * sn;
                    }
                }
            }
        }
        float inv = 1.f;
        if (head_norm) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
#pragma unroll
            for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            inv = 1.0f / sqrtf(ss / (float)hd + eps);
        }
        if (!live) continue;
        const float* w = is_q ? q_norm_w : k_norm_w;
        if (w != nullptr) {
            const float4 w0 = *reinterpret_cast<const float4*>(w + e0), w1 = *reinterpret_cast<const float4*>(w + e0 + 4);
            x[0] *= w0.x; x[1] *= w0.y; x[2] *= w0.z; x[3] *= w0.w; x[4] *= w1.x; x[5] *= w1.y; x[6] *= w1.z; x[7] *= w1.w;
        }
        uint4 out;
        __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = __floats2bfloat162_rn(x[2 * e] * inv, x[2 * e + 1] * inv);
        bf16* dst = is_q ? src : k_cache + cache_row_offset(block_table, blocks_per_seq, slot, pos, g, KV, hd) + e0;
        *reinterpret_cast<uint4*>(dst) = out;
    }
    if (write && v_col >= 0) {
        for (int idx = (blockIdx.y * blockDim.x + threadIdx.x) * 8; idx < KV * vd; idx += gridDim.y * blockDim.x * 8) {
            const int g = idx / vd, e = idx - g * vd;
            const uint4 raw = *reinterpret_cast<const uint4*>(row + (size_t)v_col + idx);
            uint4 out = raw;
            if (v_bias != nullptr) {
                const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
                __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float2 f = __bfloat1622float2(p[j]);
                    o[j] = __floats2bfloat162_rn(f.x + v_bias[idx + 2 * j], f.y + v_bias[idx + 2 * j + 1]);
                }
            }
            *reinterpret_cast<uint4*>(v_cache + cache_row_offset(block_table, blocks_per_seq, slot, pos, g, KV, vd) + e) = out;
        }
    }
}

// The preparation for attention whose q and k are normed over the WHOLE projection (all heads at once) and whose values
// may be mixed with those of another layer; no rotation.  A CTA per (token, role):
//
//   role 0   q / sqrt(mean(q^2) + eps) * q_w  -> q_out
//   role 1   k likewise                       -> the token's row of the key cache
//   role 2   v, or (1 - lambda) v + lambda v_first -> the value cache; v as projected also -> v_keep where one is given
//
// The projections are rows in the compute dtype or float32 pieces [n_pieces][rows][ld] of a product whose K range was cut
// (added in ascending order).  V: elements an access (8 where rows, heads and pointers allow 16-byte accesses, else 1).
struct RowPrepare {
    const void* rows; const float* pieces; int n_pieces; long long piece_stride; long long ld;
    int q_col, k_col, v_col;
    const float* q_w; const float* k_w; float eps; int norm;
    void* q_out; long long q_ld;
    void* k_cache; void* v_cache; const int* block_table; int blocks_per_seq;
    const void* v_first; long long v_first_ld; const float* lambda; void* v_keep;
    const int* positions; const int* token_slot;
    int H, KV, hd, vd;
};
template <typename T, int V>
__device__ __forceinline__ void rp_load(const RowPrepare& A, size_t at, float (&x)[V]) {
    if (A.pieces != nullptr) {
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = 0.f;
        for (int z = 0; z < A.n_pieces; ++z) {
            const float* p = A.pieces + (size_t)z * A.piece_stride + at;
            if constexpr (V == 8) {
                const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
                x[0] += a.x; x[1] += a.y; x[2] += a.z; x[3] += a.w; x[4] += b.x; x[5] += b.y; x[6] += b.z; x[7] += b.w;
            } else x[0] += p[0];
        }
        return;
    }
    const T* p = (const T*)A.rows + at;
    if constexpr (V == 8 && sizeof(T) == 2) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(b[e]); x[2 * e] = f.x; x[2 * e + 1] = f.y; }
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = to_f32(p[e]);
    }
}
template <typename T, int V>
__device__ __forceinline__ void rp_store(T* p, const float (&x)[V]) {
    if constexpr (V == 8 && sizeof(T) == 2) {
        uint4 out;
        __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
        *reinterpret_cast<uint4*>(p) = out;
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) p[e] = from_f32<T>(x[e]);
    }
}
template <typename T, int V>
__global__ void __launch_bounds__(256)
qk_row_prepare_kernel(const RowPrepare A) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float smem[];       // [width]: a thread reads back its own elements only
    __shared__ float scratch[33];
    const int t = blockIdx.x, role = blockIdx.y;
    const int slot = A.token_slot[t];
    if (slot < 0) return;                               // a padding row
    const int pos = A.positions[t];
    if (role > 0 && A.k_cache == nullptr && !(role == 2 && A.v_keep != nullptr)) return;
    const int width = role == 0 ? A.H * A.hd : (role == 1 ? A.KV * A.hd : A.KV * A.vd);
    const size_t at = (size_t)t * A.ld + (role == 0 ? A.q_col : (role == 1 ? A.k_col : A.v_col));
    if (role == 2) {
        const float lam = A.v_first != nullptr ? A.lambda[0] : 0.f;
        for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
            float x[V];
            rp_load<T, V>(A, at + i, x);
            if (A.v_keep != nullptr) rp_store<T, V>((T*)A.v_keep + (size_t)t * width + i, x);
            if (A.k_cache == nullptr) continue;
            if (A.v_first != nullptr) {
                const T* f = (const T*)A.v_first + (size_t)t * A.v_first_ld + i;
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] = (1.0f - lam) * x[e] + lam * to_f32(f[e]);
            }
            const int g = i / A.vd, e0 = i - g * A.vd;
            rp_store<T, V>((T*)A.v_cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, pos, g, A.KV, A.vd) + e0, x);
        }
        return;
    }
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float x[V];
        rp_load<T, V>(A, at + i, x);
#pragma unroll
        for (int e = 0; e < V; ++e) { ss += x[e] * x[e]; smem[i + e] = x[e]; }
    }
    float inv = 1.f;
    if (A.norm) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + A.eps);
    const float* w = role == 0 ? A.q_w : A.k_w;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float x[V];
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = smem[i + e] * inv * (w != nullptr ? w[i + e] : 1.f);
        if (role == 0) {
            rp_store<T, V>((T*)A.q_out + (size_t)t * A.q_ld + i, x);
        } else {
            const int g = i / A.hd, e0 = i - g * A.hd;
            rp_store<T, V>((T*)A.k_cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, pos, g, A.KV, A.hd) + e0, x);
        }
    }
}

// The same with one CTA per token: the token's q | k | v are cut into pieces of eight elements (bfloat16, 16-byte accesses), VPT
// pieces a thread in registers, and one meeting of the warps adds both sums of squares.
template <int VPT>
__global__ void __launch_bounds__(512)
qk_row_prepare_vec_kernel(const RowPrepare A) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float part[2][16];
    const int t = blockIdx.x;
    const int slot = A.token_slot[t];
    if (slot < 0) return;                               // a padding row
    const int pos = A.positions[t];
    const int nq = A.H * A.hd / 8, nk = A.KV * A.hd / 8, nv = A.KV * A.vd / 8;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
    float x[VPT][8];
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i >= nq + nk + nv) continue;
        const int col = i < nq ? A.q_col + i * 8 : (i < nq + nk ? A.k_col + (i - nq) * 8 : A.v_col + (i - nq - nk) * 8);
        rp_load<bf16, 8>(A, (size_t)t * A.ld + col, x[j]);
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += x[j][e] * x[j][e];
        if (i < nq) sq += ss;
        else if (i < nq + nk) sk += ss;
    }
    float inv_q = 1.f, inv_k = 1.f;
    if (A.norm) {
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) { part[0][warp] = sq; part[1][warp] = sk; }
        __syncthreads();
        sq = warp_sum(lane < nwarps ? part[0][lane] : 0.f);
        sk = warp_sum(lane < nwarps ? part[1][lane] : 0.f);
        inv_q = 1.0f / sqrtf(sq / (float)(nq * 8) + A.eps);
        inv_k = 1.0f / sqrtf(sk / (float)(nk * 8) + A.eps);
    }
    const bool write = A.k_cache != nullptr;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i >= nq + nk + nv) continue;
        const bool is_q = i < nq, is_k = !is_q && i < nq + nk;
        const int at = (is_q ? i : (is_k ? i - nq : i - nq - nk)) * 8;
        if (is_q || is_k) {
            const float* w = is_q ? A.q_w : A.k_w;
            const float inv = is_q ? inv_q : inv_k;
            if (w != nullptr) {
                const float4 w0 = *reinterpret_cast<const float4*>(w + at), w1 = *reinterpret_cast<const float4*>(w + at + 4);
                x[j][0] *= w0.x; x[j][1] *= w0.y; x[j][2] *= w0.z; x[j][3] *= w0.w; x[j][4] *= w1.x; x[j][5] *= w1.y; x[j][6] *= w1.z; x[j][7] *= w1.w;
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) x[j][e] *= inv;
            if (is_q) rp_store<bf16, 8>((bf16*)A.q_out + (size_t)t * A.q_ld + at, x[j]);
            else if (write) rp_store<bf16, 8>((bf16*)A.k_cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, pos, at / A.hd, A.KV, A.hd) + at % A.hd, x[j]);
        } else {
            if (A.v_keep != nullptr) rp_store<bf16, 8>((bf16*)A.v_keep + (size_t)t * nv * 8 + at, x[j]);
            if (!write) continue;
            if (A.v_first != nullptr) {
                const float lam = A.lambda[0];
                const uint4 raw = *reinterpret_cast<const uint4*>((const bf16*)A.v_first + (size_t)t * A.v_first_ld + at);
                const bf16* f = reinterpret_cast<const bf16*>(&raw);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[j][e] = (1.0f - lam) * x[j][e] + lam * to_f32(f[e]);
            }
            rp_store<bf16, 8>((bf16*)A.v_cache + cache_row_offset(A.block_table, A.blocks_per_seq, slot, pos, at / A.vd, A.KV, A.vd) + at % A.vd, x[j]);
        }
    }
}

}  // namespace kl

using namespace kl;

// rows (compute dtype, `ld` elements apart; q_out may be their q columns) or pieces (float32 [n_pieces][..][ld], piece_stride
// elements apart): q heads from column q_col, k heads from k_col, v heads from v_col.  v_first (compute dtype) with lambda
// (float32, one number on the device) or null; v_keep [n_tokens, KV * vd] or null; caches both null: q (and v_keep) alone.
KL_API int kl_qk_row_prepare(const void* rows, const float* pieces, int n_pieces, long long piece_stride, long long ld, int q_col,
                             int k_col, int v_col, int norm, float eps, const float* q_w, const float* k_w, void* q_out,
                             long long q_ld, void* k_cache, void* v_cache, const int* block_table, int blocks_per_seq,
                             const void* v_first, long long v_first_ld, const float* lambda, void* v_keep, const int* positions,
                             const int* token_slot, int n_tokens, int H, int KV, int hd, int vd, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return KL_OK;
    if (H <= 0 || KV <= 0 || hd <= 0 || vd <= 0 || (rows == nullptr) == (pieces == nullptr) || (pieces != nullptr && n_pieces < 1)) return KL_ERR_BAD_SIZE;
    if ((k_cache == nullptr) != (v_cache == nullptr) || (v_first != nullptr && lambda == nullptr) || q_out == nullptr) return KL_ERR_BAD_SIZE;
    if (dtype != KL_F32 && dtype != KL_BF16) return KL_ERR_BAD_DTYPE;
    RowPrepare A{rows, pieces, n_pieces, piece_stride, ld, q_col, k_col, v_col, q_w, k_w, eps, norm, q_out, q_ld, k_cache, v_cache,
                 block_table, blocks_per_seq, v_first, v_first_ld, lambda, v_keep, positions, token_slot, H, KV, hd, vd};
    const size_t smem = (size_t)(H > KV ? H : KV) * hd * sizeof(float);
    if (smem > 200 * 1024) return KL_ERR_BAD_SIZE;
    const uintptr_t ptrs = (uintptr_t)rows | (uintptr_t)pieces | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)v_first |
                           (uintptr_t)v_keep;
    const bool wide = dtype == KL_BF16 && hd % 8 == 0 && vd % 8 == 0 && ld % 8 == 0 && q_ld % 8 == 0 && v_first_ld % 8 == 0 && q_col % 8 == 0 &&
                      k_col % 8 == 0 && v_col % 8 == 0 && piece_stride % 8 == 0 && (ptrs & 15) == 0;
    const int pieces8 = wide ? (H * hd + KV * hd + KV * vd) / 8 : 0;
    if (wide && pieces8 <= 4 * 512 && (((uintptr_t)q_w | (uintptr_t)k_w) & 15) == 0) {
        const int vpt = pieces8 <= 512 ? 1 : (pieces8 <= 1024 ? 2 : 4);
        const int threads = ((pieces8 + vpt - 1) / vpt + 31) / 32 * 32;
        if (vpt == 1) launch_kernel(qk_row_prepare_vec_kernel<1>, n_tokens, threads, 0, stream, A);
        else if (vpt == 2) launch_kernel(qk_row_prepare_vec_kernel<2>, n_tokens, threads, 0, stream, A);
        else launch_kernel(qk_row_prepare_vec_kernel<4>, n_tokens, threads, 0, stream, A);
        KL_LAUNCH_CHECK();
        return KL_OK;
    }
    const dim3 grid(n_tokens, 3);
#define KL_RP(T, V)                                                                                                                \
    do {                                                                                                                           \
        if (smem > 40 * 1024) KL_CUDA(cudaFuncSetAttribute(qk_row_prepare_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        launch_kernel(qk_row_prepare_kernel<T, V>, grid, 256, smem, stream, A);                                                    \
    } while (0)
    if (dtype == KL_F32) KL_RP(float, 1);
    else if (wide) KL_RP(bf16, 8);
    else KL_RP(bf16, 1);
#undef KL_RP
    KL_LAUNCH_CHECK();
    return KL_OK;
}

// proj: rows of `ld` elements; q heads from column q_col, k heads from k_col, v heads from v_col (< 0: none).
// Caches: [pages, KV, PAGE, hd] and [pages, KV, PAGE, vd]; both null: a layer that only reads a cache.
KL_API int kl_qk_prepare(void* proj, long long ld, int q_col, int k_col, int v_col, const float* q_bias, const float* k_bias,
                         const float* v_bias, const float* inv_freq, int rot, int interleaved, int head_norm, float eps,
                         const float* q_norm_w, const float* k_norm_w, const int* positions, const int* token_slot,
                         const int* block_table, int blocks_per_seq, void* k_cache, void* v_cache, int n_tokens, int H, int KV,
                         int hd, int vd, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return KL_OK;
    if (rot % 2 || rot < 0 || rot > hd || H <= 0 || KV <= 0 || hd <= 0 || vd <= 0) return KL_ERR_BAD_SIZE;
    if (rot > 0 && inv_freq == nullptr) return KL_ERR_BAD_SIZE;
    if ((k_cache == nullptr) != (v_cache == nullptr)) return KL_ERR_BAD_SIZE;
    if (v_col < 0 && vd != hd) return KL_ERR_BAD_SIZE;
    // bfloat16 rows on 16-byte boundaries, head sizes 8 L with L a power of two: the form with eight elements a lane
    const int L = hd / 8;
    const bool pairs_ok = rot == 0 || interleaved || rot % 16 == 0;
    if (dtype == KL_BF16 && hd % 8 == 0 && L <= 32 && (L & (L - 1)) == 0 && vd % 8 == 0 && ld % 8 == 0 && q_col % 8 == 0 && k_col % 8 == 0 &&
        (v_col < 0 || v_col % 8 == 0) && pairs_ok && (((uintptr_t)proj | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0 &&
        (((uintptr_t)q_bias | (uintptr_t)k_bias | (uintptr_t)q_norm_w | (uintptr_t)k_norm_w) & 15) == 0) {
        const int heads_per_cta = 256 / L;
        const dim3 grid(n_tokens, (H + KV + heads_per_cta - 1) / heads_per_cta);
        const size_t table = (size_t)rot * sizeof(float);
#define KL_QKV(LL)                                                                                                                 \
    launch_kernel(qk_prepare_vec_kernel<LL>, grid, 256, table, stream, (bf16*)proj, ld, q_col, k_col, v_col, q_bias, k_bias, v_bias, \
                  inv_freq, rot, interleaved, head_norm, eps, q_norm_w, k_norm_w, positions, token_slot, block_table, blocks_per_seq, \
                  (bf16*)k_cache, (bf16*)v_cache, H, KV, vd)
        switch (L) {
            case 1: KL_QKV(1); break;
            case 2: KL_QKV(2); break;
            case 4: KL_QKV(4); break;
            case 8: KL_QKV(8); break;
            case 16: KL_QKV(16); break;
            default: KL_QKV(32); break;
        }
#undef KL_QKV
        KL_LAUNCH_CHECK();
        return KL_OK;
    }
    const size_t smem = (size_t)(rot + QKP_WARPS * hd) * sizeof(float);
    if (smem > 48 * 1024 || (H + KV + QKP_WARPS - 1) / QKP_WARPS > 65535) return KL_ERR_BAD_SIZE;
#define KL_QKP(T)                                                                                                                  \
    launch_kernel(qk_prepare_kernel<T>, dim3(n_tokens, (H + KV + QKP_WARPS - 1) / QKP_WARPS), QKP_WARPS * 32, smem, stream, (T*)proj, ld, q_col, k_col, v_col, q_bias, k_bias, \
                  v_bias, inv_freq, rot, interleaved, head_norm, eps, q_norm_w, k_norm_w, positions, token_slot, block_table,      \
                  blocks_per_seq, (T*)k_cache, (T*)v_cache, H, KV, hd, vd)
    if (dtype == KL_F32) KL_QKP(float);
    else if (dtype == KL_BF16) KL_QKP(bf16);
    else return KL_ERR_BAD_DTYPE;
#undef KL_QKP
    KL_LAUNCH_CHECK();
    return KL_OK;
}
