// Routing for a mixture of experts: who goes where, and the weighted sum at the end.
//
//   moe_route_kernel    a warp per token: s = softmax(z) over all experts in 32 bits (z plus a bias per expert
//                       where one is given), the `top` largest (the lower index among equals), their scores
//                       as weights (divided by their sum if asked, which is the softmax over the chosen
//                       logits alone).  Or s = sigmoid(z).  With either a correction per expert may join the scores
//                       for the choice but not for the weights; weights times a scale.
//   moe_plan_kernel     one CTA: counts per expert, a list of (token, choice) pairs sorted by expert in
//                       which every expert's run is padded to whole tiles, the expert of every tile, and
//                       each pair's place in the list (-1: the row belongs to no sequence, -2: the choice is
//                       an identity expert, one whose number is not below `experts`, which has no product).
//                       Everything stays on the device, so a step with experts needs no answer from the host
//                       and can be captured in a graph.
//   moe_combine_kernel  out[t] = sum over the token's choices, in the order of the choices, of
//                       weight * (the expert's result at the pair's place, or for an identity expert the
//                       layer's input row), in 32 bits; optionally plus the result of an expert that every
//                       token takes (rows, or float32 pieces of a product), times sigmoid(a number per token)
//                       where one is given.
//
// The order of the pairs inside an expert's run is whatever the counters gave; no result depends on it,
// because the grouped product computes every row by itself.  ExiledOfCode/KuiperLLama has dense
// feed-forwards alone (kuiper/source/model/llama3.cpp:692-718).
#include "common.cuh"

namespace kl {

constexpr int MOE_MAX_PER_LANE = 8;      // experts <= 256
constexpr int MOE_PLAN_THREADS = 1024;
constexpr int MOE_MAX_EXPERTS = 32 * MOE_MAX_PER_LANE;

struct RouteArgs {
    const float* logits; long long ld;
    const float* bias;              // [experts], joins the logits, or null
    const float* correction;        // [experts], joins the scores for the choice alone, or null
    int tokens, experts, top, renormalise, groups, keep_groups, sigmoid, group_top;    // group_top: a group's score is the sum of its so many best
    float renorm_eps, scale;
    int* choice; float* weight;
};

__global__ void __launch_bounds__(128)
moe_route_kernel(const RouteArgs A) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float group_best[4][MOE_MAX_EXPERTS];
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (t >= A.tokens) return;
    const int experts = A.experts, top = A.top, groups = A.groups;
    const float* z = A.logits + (size_t)t * A.ld;
    float s[MOE_MAX_PER_LANE], w[MOE_MAX_PER_LANE];          // choice scores (taken and absent experts hold -inf) and weights
    float m = -INFINITY;
#pragma unroll
    for (int i = 0; i < MOE_MAX_PER_LANE; ++i) {
        const int e = lane + 32 * i;
        s[i] = e < experts ? (A.bias ? z[e] + A.bias[e] : z[e]) : -INFINITY;
        m = fmaxf(m, s[i]);
    }
    m = warp_max(m);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < MOE_MAX_PER_LANE; ++i) {
        const int e = lane + 32 * i;
        w[i] = 0.f;
        if (e < experts) {
            w[i] = A.sigmoid ? 1.0f / (1.0f + expf(-s[i])) : expf(s[i] - m);
            s[i] = w[i];
            sum += w[i];
        }
    }
    sum = A.sigmoid ? 1.f : warp_sum(sum);                   // softmax: scores are w / sum
    if (A.correction != nullptr) {
#pragma unroll
        for (int i = 0; i < MOE_MAX_PER_LANE; ++i) {
            const int e = lane + 32 * i;
            if (e < experts) s[i] = w[i] / sum + A.correction[e];
        }
    }
    float* weight = A.weight + (size_t)t * top;
    if (groups > 1 && A.keep_groups < groups) {
        // Experts form `groups` equal groups of neighbours; a group's score is its largest choice score, or the sum of its
        // `group_top` largest, and only the experts of the `keep_groups` best groups (the lower index among equals) stay.
        float* gb = group_best[threadIdx.x >> 5];
        const int per = experts / groups;
        for (int g = 0; g < groups; ++g) {
            float total = 0.f, below = INFINITY;             // the largest not above `below`, each expert once
            int after = -1;
            for (int k = 0; k < min(A.group_top, per); ++k) {
                float b = -INFINITY;
                int be = 0x7fffffff;
#pragma unroll
                for (int i = 0; i < MOE_MAX_PER_LANE; ++i) {
                    const int e = lane + 32 * i;
                    if (e < experts && e / per == g && (s[i] < below || (s[i] == below && e > after)) && (s[i] > b || (s[i] == b && e < be))) { b = s[i]; be = e; }
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    const float ob = __shfl_xor_sync(0xffffffffu, b, o);
                    const int oe = __shfl_xor_sync(0xffffffffu, be, o);
                    if (ob > b || (ob == b && oe < be)) { b = ob; be = oe; }
                }
                total += b;
                below = b;
                after = be;
            }
            if (lane == 0) gb[g] = total;
        }
        __syncwarp();
        // rank of every group: how many groups come before it (a larger score, or an equal one with a lower index)
#pragma unroll
        for (int i = 0; i < MOE_MAX_PER_LANE; ++i) {
            const int e = lane + 32 * i;
            if (e < experts) {
                const int g = e / per;
                const float mine_b = gb[g];
                int before = 0;
                for (int o = 0; o < groups; ++o) before += (gb[o] > mine_b || (gb[o] == mine_b && o < g)) ? 1 : 0;
                if (before >= A.keep_groups) s[i] = -INFINITY;
            }
        }
    }
    float chosen_sum = 0.f, mine = 0.f;
    int mine_e = 0;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int best_e = 0x7fffffff;
#pragma unroll
        for (int i = 0; i < MOE_MAX_PER_LANE; ++i)
            if (s[i] > best) { best = s[i]; best_e = lane + 32 * i; }    // ascending e inside a lane: the lower index wins
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oe = __shfl_xor_sync(0xffffffffu, best_e, o);
            if (ob > best || (ob == best && oe < best_e)) { best = ob; best_e = oe; }
        }
        if (best_e >= experts) best_e = k;                   // no comparable score is left (logits that are not numbers): any expert, in bounds
        float chosen_w = 0.f;
#pragma unroll
        for (int i = 0; i < MOE_MAX_PER_LANE; ++i)
            if (lane + 32 * i == best_e) { chosen_w = w[i]; s[i] = -INFINITY; }
        chosen_w = __shfl_sync(0xffffffffu, chosen_w, best_e & 31);
        chosen_sum += chosen_w;
        if (lane == k % 32) { mine = chosen_w; mine_e = best_e; }
        if (k % 32 == 31 || k == top - 1) {
            const int kk = (k / 32) * 32 + lane;
            if (kk <= k) { A.choice[(size_t)t * top + kk] = mine_e; weight[kk] = mine; }
        }
    }
    // weights: the scores, or those divided by the chosen ones' sum, times the scale
    __syncwarp();
    const float denom = A.renormalise ? chosen_sum + A.renorm_eps * sum : sum;      // softmax scores are w / sum: s_k / (sum of chosen s + eps)
    for (int kk = lane; kk < top; kk += 32) weight[kk] = weight[kk] / denom * A.scale;
}

__global__ void __launch_bounds__(MOE_PLAN_THREADS)
moe_plan_kernel(const int* __restrict__ choice, const int* __restrict__ token_slot, int tokens, int top, int experts, int tile_rows,
                int cap, int tiles, int* __restrict__ rank, int* __restrict__ pair_pos, int* __restrict__ list_rows,
                int* __restrict__ tile_group) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ int count[MOE_MAX_EXPERTS];
    __shared__ int first[MOE_MAX_EXPERTS + 1];
    const int pairs = tokens * top;
    for (int e = threadIdx.x; e < experts; e += blockDim.x) count[e] = 0;
    for (int i = threadIdx.x; i < cap; i += blockDim.x) list_rows[i] = -1;
    for (int i = threadIdx.x; i < tiles; i += blockDim.x) tile_group[i] = -1;
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int t = p / top;
        const bool live = token_slot == nullptr || token_slot[t] >= 0;
        rank[p] = !live ? -1 : (choice[p] >= experts ? -2 : atomicAdd(&count[choice[p]], 1));
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int at = 0;
        for (int e = 0; e < experts; ++e) {
            first[e] = at;
            at += (count[e] + tile_rows - 1) / tile_rows * tile_rows;
        }
        first[experts] = at;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < experts; e += blockDim.x)
        for (int tile = first[e] / tile_rows; tile < first[e + 1] / tile_rows; ++tile) tile_group[tile] = e;
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int r = rank[p];
        const int pos = r < 0 ? r : first[choice[p]] + r;
        pair_pos[p] = pos;
        if (pos >= 0) list_rows[pos] = p / top;
    }
}

struct CombineArgs {
    const void* results; long long ld;             // the list's rows, compute dtype
    const int* pair_pos; const float* weight;
    const void* x; long long x_ld;                 // the layer's input rows, compute dtype (identity experts), or null
    const void* shared; long long shared_ld;       // the expert every token takes: rows in the compute dtype, or null
    const float* pieces; int n_pieces; long long piece_stride;   // or float32 [n_pieces][tokens][hidden]
    const float* gate; long long gate_ld;          // its factor is sigmoid(gate[t * gate_ld]); null: 1
    int tokens, top, hidden;
    float* out;
};

// V elements of a row a thread (16 bytes of results an access where rows allow it; with PIECES, few rows, 4 elements, so that
// more threads share them; else 1), a token's results on their way four at a time, pieces eight at a time and ahead of them.
template <typename T, int V> struct McRaw { T v[V]; };       // a piece of a row as it lies in memory, held while it is on its way
template <> struct McRaw<bf16, 8> { uint4 v; };
template <> struct McRaw<bf16, 4> { uint2 v; };
template <> struct McRaw<float, 4> { uint4 v; };
template <typename T, int V> __device__ __forceinline__ McRaw<T, V> mc_fetch(const T* p) { return *reinterpret_cast<const McRaw<T, V>*>(p); }
template <typename T, int V> __device__ __forceinline__ void mc_axpy(float a, const McRaw<T, V>& raw, float (&acc)[V]) {
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = fmaf(a, to_f32(e[i]), acc[i]);
}
template <typename T, int V, bool PIECES>
__global__ void __launch_bounds__(256)
moe_combine_kernel(const CombineArgs A) {
    pdl_launch_dependents();
    pdl_wait();
    const int per = A.hidden / V, top = A.top;
    const size_t total = (size_t)A.tokens * per;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t t = idx / per;
        const int c = (int)(idx - t * per) * V;
        float acc[V], y[V];
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = y[e] = 0.f;
        // the expert every token takes: its result is asked for first and joins the sum last
        McRaw<T, V> every;
        if (!PIECES && A.shared != nullptr) every = mc_fetch<T, V>((const T*)A.shared + t * A.shared_ld + c);
        const float z_gate = A.gate != nullptr ? A.gate[t * A.gate_ld] : 0.f;
        if constexpr (PIECES) {
            const float* p = A.pieces + t * A.hidden + c;
            for (int z0 = 0; z0 < A.n_pieces; z0 += 8) {                 // pieces are added in ascending order
                McRaw<float, V> q[8];
#pragma unroll
                for (int z = 0; z < 8; ++z)
                    if (z0 + z < A.n_pieces) q[z] = mc_fetch<float, V>(p + (size_t)(z0 + z) * A.piece_stride);
#pragma unroll
                for (int z = 0; z < 8; ++z)
                    if (z0 + z < A.n_pieces) mc_axpy<float, V>(1.0f, q[z], y);
            }
        }
        for (int k0 = 0; k0 < top; k0 += 4) {
            McRaw<T, V> r[4];
            float wt[4];
            bool any[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int pos = k0 + k < top ? A.pair_pos[t * top + k0 + k] : -1;
                const T* src = pos >= 0 ? (const T*)A.results + (size_t)pos * A.ld + c
                                        : (pos == -2 && A.x != nullptr ? (const T*)A.x + t * A.x_ld + c : nullptr);
                any[k] = src != nullptr;
                wt[k] = any[k] ? A.weight[t * top + k0 + k] : 0.f;
                if (any[k]) r[k] = mc_fetch<T, V>(src);
            }
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (any[k]) mc_axpy<T, V>(wt[k], r[k], acc);
        }
        if (PIECES || A.shared != nullptr) {
            const float f = A.gate != nullptr ? 1.0f / (1.0f + expf(-z_gate)) : 1.0f;
            if constexpr (PIECES) {
#pragma unroll
                for (int e = 0; e < V; ++e) acc[e] = fmaf(f, y[e], acc[e]);
            } else mc_axpy<T, V>(f, every, acc);
        }
        float* o = A.out + t * A.hidden + c;
        if constexpr (V % 4 == 0) {
#pragma unroll
            for (int e = 0; e < V; e += 4) *reinterpret_cast<float4*>(o + e) = make_float4(acc[e], acc[e + 1], acc[e + 2], acc[e + 3]);
        } else o[0] = acc[0];
    }
}

// rows[p] = x[list_rows[p]] for every place of the list, zeros at padding places: the operand of a product
// whose loader reads whole tiles of consecutive rows.
template <typename T>
__global__ void __launch_bounds__(256)
moe_gather_kernel(const T* __restrict__ x, long long ld, const int* __restrict__ list_rows, int cap, int width, T* __restrict__ rows) {
    pdl_launch_dependents();
    pdl_wait();
    const int per = width / 8;                                  // 16-byte pieces per row
    const size_t total = (size_t)cap * per;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t p = idx / per;
        const int c = (int)(idx - p * per) * 8;
        const int src = list_rows[p];
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (src >= 0) v = *reinterpret_cast<const uint4*>(x + (size_t)src * ld + c);
        *reinterpret_cast<uint4*>(rows + p * width + c) = v;
    }
}

}  // namespace kl

using namespace kl;

// bfloat16 rows of width % 8 == 0 on 16-byte boundaries.
KL_API int kl_moe_gather(const void* x, long long ld, const int* list_rows, int cap, int width, void* rows, cudaStream_t stream) {
    if (cap <= 0) return KL_OK;
    if (width <= 0 || width % 8 || ld % 8 || (((uintptr_t)x | (uintptr_t)rows) & 15)) return KL_ERR_BAD_ALIGN;
    const int blocks = kl::strided_grid((size_t)cap * (width / 8), 256, 16);
    launch_kernel(moe_gather_kernel<bf16>, blocks, 256, 0, stream, (const bf16*)x, ld, list_rows, cap, width, (bf16*)rows);
    KL_LAUNCH_CHECK();
    return KL_OK;
}

// scores: 0 softmax over the experts, 1 sigmoid; correction: float32 [experts] or null; group_top: see RouteArgs.
KL_API int kl_moe_route(const float* logits, long long ld, const float* bias, int tokens, int experts, int top, int renormalise, int groups,
                        int keep_groups, float renorm_eps, int scores, const float* correction, int group_top, float scale,
                        int* choice, float* weight, cudaStream_t stream) {
    if (tokens <= 0) return KL_OK;
    if (experts <= 0 || experts > MOE_MAX_EXPERTS || top <= 0 || top > experts) return KL_ERR_BAD_SIZE;
    if (groups < 1 || experts % groups || keep_groups < 1 || keep_groups > groups || top > keep_groups * (experts / groups)) return KL_ERR_BAD_SIZE;
    if ((scores != 0 && scores != 1) || group_top < 1) return KL_ERR_BAD_SIZE;
    const RouteArgs A{logits, ld, bias, correction, tokens, experts, top, renormalise, groups, keep_groups, scores, group_top, renorm_eps, scale,
                      choice, weight};
    launch_kernel(moe_route_kernel, (tokens + 3) / 4, 128, 0, stream, A);
    KL_LAUNCH_CHECK();
    return KL_OK;
}

// cap: length of the padded list (at least tokens * top + experts * (tile_rows - 1), a multiple of tile_rows);
// tiles = cap / tile_rows.
KL_API int kl_moe_plan(const int* choice, const int* token_slot, int tokens, int top, int experts, int tile_rows, int cap, int tiles,
                       int* rank, int* pair_pos, int* list_rows, int* tile_group, cudaStream_t stream) {
    if (tokens <= 0) return KL_OK;
    if (experts <= 0 || experts > MOE_MAX_EXPERTS || tile_rows <= 0 || cap % tile_rows || tiles * tile_rows != cap) return KL_ERR_BAD_SIZE;
    if ((long long)cap < (long long)tokens * top + (long long)experts * (tile_rows - 1)) return KL_ERR_BAD_SIZE;
    launch_kernel(moe_plan_kernel, 1, MOE_PLAN_THREADS, 0, stream, choice, token_slot, tokens, top, experts, tile_rows, cap, tiles,
                  rank, pair_pos, list_rows, tile_group);
    KL_LAUNCH_CHECK();
    return KL_OK;
}

// x: the layer's input rows (compute dtype; needed where pair_pos has identity experts) or null.  The expert every token takes: rows
// `shared` (compute dtype) or float32 pieces [n_pieces][tokens][hidden], or neither; gate: float32, the token's number at t * gate_ld, or null.
KL_API int kl_moe_combine(const void* results, long long ld, const int* pair_pos, const float* weight, const void* x, long long x_ld,
                          const void* shared, long long shared_ld, const float* pieces, int n_pieces, long long piece_stride,
                          const float* gate, long long gate_ld, int tokens, int top, int hidden, float* out, int dtype, cudaStream_t stream) {
    if (tokens <= 0 || hidden <= 0) return KL_OK;
    if (dtype != KL_F32 && dtype != KL_BF16) return KL_ERR_BAD_DTYPE;
    if (n_pieces < 0 || (n_pieces > 0 && (pieces == nullptr || shared != nullptr))) return KL_ERR_BAD_SIZE;
    const CombineArgs A{results, ld, pair_pos, weight, x, x_ld, shared, shared_ld, pieces, n_pieces, piece_stride, gate, gate_ld, tokens, top, hidden, out};
    const int v = (dtype == KL_F32 || n_pieces > 0) ? 4 : 8;
    const bool wide = hidden % v == 0 && ld % v == 0 && x_ld % v == 0 && shared_ld % v == 0 && piece_stride % v == 0 &&
                      (((uintptr_t)results | (uintptr_t)out | (uintptr_t)x | (uintptr_t)shared | (uintptr_t)pieces) & 15) == 0;
    const int threads = n_pieces > 0 ? 128 : 256;
    const int grid = kl::strided_grid((size_t)tokens * (wide ? hidden / v : hidden), threads, 16);
#define KL_MC(T, V, P) launch_kernel(moe_combine_kernel<T, V, P>, grid, threads, 0, stream, A)
    if (dtype == KL_F32) {
        if (n_pieces > 0) { if (wide) KL_MC(float, 4, true); else KL_MC(float, 1, true); }
        else { if (wide) KL_MC(float, 4, false); else KL_MC(float, 1, false); }
    } else {
        if (n_pieces > 0) { if (wide) KL_MC(bf16, 4, true); else KL_MC(bf16, 1, true); }
        else { if (wide) KL_MC(bf16, 8, false); else KL_MC(bf16, 1, false); }
    }
#undef KL_MC
    KL_LAUNCH_CHECK();
    return KL_OK;
}
