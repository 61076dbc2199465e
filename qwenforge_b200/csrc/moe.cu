// Routing of a mixture-of-experts feed-forward, on the device from start to end (no count ever reaches the host, so a
// step with routed experts replays from a captured graph like any other).
//
//   plan     from the router's float32 logits [tokens][experts]: per token the `top` experts with the largest
//            score, the score being sigmoid(logit) or, with `softmax_scores`, the softmax over the experts; the weights
//            are the chosen scores, divided by their sum when `renormalize` is set. The (token, expert) pairs are
//            sorted by expert: rows offsets[e] .. offsets[e+1]-1 of the sorted order belong to expert e, and every
//            expert's rows are cut into tiles of `tile_rows` rows for the grouped product (csrc/grouped_gemm.cu).
//            For a step of few tokens the plan can make the logits itself from the tokens' rows and the router's
//            weights (float32 sums of the products, a warp per logit), which saves a launch where launches are the cost.
//   gather   x_sorted[r] = x[token of r] (* weight of r, when the weight multiplies the expert's input)
//   combine  out[t] = sum over the token's pairs, in the order of its choice, of y_sorted[row of the pair]
//            (* weight, when the weight multiplies the expert's output), summed in float32
//
// One block makes the plan: the work is a few values per token. The order of an expert's rows among themselves is
// whatever the block's atomics gave; no result depends on it, since a row of a product is computed alone.
#include <float.h>

#include "mma.cuh"

#define MOE_PLAN_THREADS 1024
// Whether the plan's block makes the router's logits on the tensor cores: few tokens and experts, rows in whole steps of K.
__host__ __device__ inline bool plan_on_tiles(int n_tokens, int n_experts, int width) { return n_tokens <= 32 && n_experts <= 32 && width % 16 == 0; }
#define PLAN_HELD 512     // pairs that the plan keeps in shared memory
#define MOE_MAX_TOP 16

// One token's choice: the `top` experts with the largest scores (the larger logit is the larger score; ties go to the
// lower index) and their weights.
// `bias` (float32 per expert, or null) is added to the logits before anything else looks at them.
__device__ __forceinline__ void moe_choose(const float* z_raw, const float* bias, int n_experts, int top, int softmax_scores,
                                           int renormalize, int* chosen, float* weight) {
    auto z = [&](int e) { return bias ? z_raw[e] + bias[e] : z_raw[e]; };
    float top_z = -FLT_MAX, denom = 1.f;
    if (softmax_scores) {
        for (int e = 0; e < n_experts; ++e) top_z = fmaxf(top_z, z(e));
        denom = 0.f;
        for (int e = 0; e < n_experts; ++e) denom += expf(z(e) - top_z);
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        int best = -1;
        float best_z = -FLT_MAX;
        for (int e = 0; e < n_experts; ++e) {
            bool taken = false;
            for (int j = 0; j < k; ++j) taken |= chosen[j] == e;
            if (!taken && (best < 0 || z(e) > best_z)) {
                best = e;
                best_z = z(e);
            }
        }
        chosen[k] = best;
        weight[k] = softmax_scores ? expf(best_z - top_z) / denom : 1.0f / (1.0f + expf(-best_z));
        total += weight[k];
    }
    if (renormalize)
        for (int k = 0; k < top; ++k) weight[k] /= total;
}

// The choice among groups of neighbouring experts, with a correction that steers the choice and not the weights:
//   s_e = sigmoid(z_e), or with `softmax_scores` the softmax over all experts;  c_e = s_e + correction_e (the choice score);  the
//   experts form `count` equal groups of neighbours, a group's score is the sum of its `best` largest c (1 or 2; of its one, in
//   groups of one);  only experts of the `keep` groups with the largest scores can be chosen;  among them the `top` largest c;
//   weights s_e, divided by their sum with `renormalize`.  Ties go to the lower index.  (count 1: no groups.)
// Softmax scores rise with their logits: where no correction and no sum of two enters, the choice compares the logits.
struct MoeGroups {
    const float* correction;   // float32 [experts] or null
    int count, keep, best;
};
#define MOE_MAX_GROUPS 64

__device__ __forceinline__ void moe_choose_grouped(const float* z_raw, const float* bias, int n_experts, int top, int softmax_scores,
                                                   int renormalize, MoeGroups groups, int* chosen, float* weight) {
    auto z = [&](int e) { return bias ? z_raw[e] + bias[e] : z_raw[e]; };
    float top_z = -FLT_MAX, denom = 1.f;
    if (softmax_scores) {
        for (int e = 0; e < n_experts; ++e) top_z = fmaxf(top_z, z(e));
        denom = 0.f;
        for (int e = 0; e < n_experts; ++e) denom += expf(z(e) - top_z);
    }
    const bool by_logit = softmax_scores && !groups.correction && groups.best == 1;
    auto score = [&](int e) { return softmax_scores ? expf(z(e) - top_z) / denom : 1.0f / (1.0f + expf(-z(e))); };
    auto choice = [&](int e) { return by_logit ? z(e) : groups.correction ? score(e) + groups.correction[e] : score(e); };
    unsigned long long kept = ~0ull;
    const int size = n_experts / groups.count;
    if (groups.count > 1 && groups.keep < groups.count) {
        float group_score[MOE_MAX_GROUPS];
        for (int g = 0; g < groups.count; ++g) {
            float first = -FLT_MAX, second = -FLT_MAX;
            for (int e = g * size; e < (g + 1) * size; ++e) {
                const float c = choice(e);
                if (c > first) {
                    second = first;
                    first = c;
                } else if (c > second) {
                    second = c;
                }
            }
            group_score[g] = size > 1 && groups.best > 1 ? first + second : first;
        }
        kept = 0ull;
        for (int k = 0; k < groups.keep; ++k) {
            int best = -1;
            for (int g = 0; g < groups.count; ++g)
                if (!((kept >> g) & 1ull) && (best < 0 || group_score[g] > group_score[best])) best = g;
            kept |= 1ull << best;
        }
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        int best = -1;
        float best_c = -FLT_MAX;
        for (int e = 0; e < n_experts; ++e) {
            if (groups.count > 1 && !((kept >> (e / size)) & 1ull)) continue;
            bool taken = false;
            for (int j = 0; j < k; ++j) taken |= chosen[j] == e;
            if (taken) continue;
            const float c = choice(e);
            if (best < 0 || c > best_c) {
                best = e;
                best_c = c;
            }
        }
        chosen[k] = best;
        weight[k] = score(best);
        total += weight[k];
    }
    if (renormalize)
        for (int k = 0; k < top; ++k) weight[k] /= total;
}

// The same choice by a warp, a lane per expert (up to 32 of them): every lane learns its expert's place in the token's choice (0 the
// best; -1: not chosen) and its weight. Ranks are counted by comparing with every other lane, so there is no chain of choices.
// groups.count 0: the plain choice, by the logits.
__device__ __forceinline__ int moe_choose_warp(float z, int n_experts, int top, int softmax_scores, int renormalize, MoeGroups groups,
                                               float& weight) {
    const int lane = threadIdx.x & 31;
    const bool real = lane < n_experts;
    float s;
    if (softmax_scores) {
        const float top_z = warp_max(real ? z : -FLT_MAX);
        const float e = real ? expf(z - top_z) : 0.f;
        s = e / warp_sum(e);
    } else {
        s = 1.0f / (1.0f + expf(-z));
    }
    float c = z;   // the choice score
    if (groups.count > 0 && !(softmax_scores && !groups.correction && groups.best == 1))
        c = groups.correction ? s + (real ? groups.correction[lane] : 0.f) : s;
    bool allowed = real;
    if (groups.count > 1 && groups.keep < groups.count) {
        const int size = n_experts / groups.count, g = lane / size;
        float first = -FLT_MAX, second = -FLT_MAX;
        for (int i = 0; i < size; ++i) {
            const float x = __shfl_sync(0xffffffffu, c, (g * size + i) & 31);
            second = fmaxf(second, fminf(first, x));
            first = fmaxf(first, x);
        }
        const float score = size > 1 && groups.best > 1 ? first + second : first;
        int better = 0;
        for (int o = 0; o < groups.count; ++o) {
            const float x = __shfl_sync(0xffffffffu, score, o * size);
            better += x > score || (x == score && o < g);
        }
        allowed = real && better < groups.keep;
    }
    const unsigned open = __ballot_sync(0xffffffffu, allowed);
    int rank = 0;
    for (int j = 0; j < n_experts; ++j) {
        const float x = __shfl_sync(0xffffffffu, c, j);
        rank += ((open >> j) & 1u) && (x > c || (x == c && j < lane));
    }
    const bool chosen = allowed && rank < top;
    weight = renormalize ? s / warp_sum(chosen ? s : 0.f) : s;
    return chosen ? rank : -1;
}

// Rows and tiles of up to 32 experts from their row counts: lane e gets its expert's first row and first tile; the totals in every lane.
__device__ __forceinline__ void moe_scan_warp(int count, int tile_rows, int& row, int& tile, int& rows, int& tiles) {
    const int lane = threadIdx.x & 31, t = (count + tile_rows - 1) / tile_rows;
    int r_sum = count, t_sum = t;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, r_sum, o), b = __shfl_up_sync(0xffffffffu, t_sum, o);
        if (lane >= o) {
            r_sum += a;
            t_sum += b;
        }
    }
    row = r_sum - count;
    tile = t_sum - t;
    rows = __shfl_sync(0xffffffffu, r_sum, 31);
    tiles = __shfl_sync(0xffffffffu, t_sum, 31);
}

// Scratch in pair order (pair = token * top + k): pair_expert, pair_weight. Results: dest [pairs] (the row of every pair),
// and in row order sorted_token [pairs], sorted_weight float32 [pairs]; offsets [experts + 1]; tile_group, tile_row0
// [max_tiles]; n_tiles [1].
__global__ void __launch_bounds__(MOE_PLAN_THREADS)
moe_plan_kernel(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                int* pair_expert, float* pair_weight, int* __restrict__ sorted_token,
                float* __restrict__ sorted_weight, int* dest, int* __restrict__ offsets,
                int* __restrict__ tile_group, int* __restrict__ tile_row0, int* __restrict__ n_tiles, int max_tiles,
                int tile_rows, const void* __restrict__ x, const void* __restrict__ router, int width, int x_is_bf16,
                const float* __restrict__ bias, MoeGroups groups) {
    grid_launch_dependents();
    extern __shared__ int shared[];
    int* counts = shared;                   // [experts]: rows per expert, then every expert's first row
    int* first_tile = shared + n_experts;   // [experts + 1]
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x) counts[e] = 0;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const bool wide = x && x_is_bf16 && width % 8 == 0 && (((uintptr_t)x | (uintptr_t)router) & 15) == 0;
    if (x) {  // the router's product first: z[t][e] = sum_c x[t][c] * router[e][c], kept in shared memory
        float* logits_out = reinterpret_cast<float*>(shared + (2 * n_experts + 1 + 3) / 4 * 4);
        if (wide && plan_on_tiles(n_tokens, n_experts, width)) {
            // Tiles of 16 tokens x 8 experts on the tensor cores (float32 sums), the block's warps dealing out K in steps of 16 columns;
            // their partial sums are added in the warps' order. One SM fetches every row once: that is what a logit per warp lacked.
            // The router's weights, which no kernel before this one writes, are asked for before the wait for it.
            float* part = logits_out + (n_tokens * n_experts + 3) / 4 * 4;   // [n_warps][128]
            const int steps = width / 16, g = lane >> 2, q = 2 * (lane & 3);
            constexpr int AHEAD = 4;
            uint32_t b[AHEAD][2];
            auto router_steps = [&](int e0, int s0) {
                const bf16* rr = (const bf16*)router + (size_t)min(e0 + g, n_experts - 1) * width + q;
#pragma unroll
                for (int u = 0; u < AHEAD; ++u) {
                    const int s = s0 + u * n_warps;
                    b[u][0] = s < steps ? *reinterpret_cast<const uint32_t*>(rr + 16 * s) : 0u;
                    b[u][1] = s < steps ? *reinterpret_cast<const uint32_t*>(rr + 16 * s + 8) : 0u;
                }
            };
            router_steps(0, warp);
            grid_dependency_wait();
            for (int t0 = 0; t0 < n_tokens; t0 += 16)
                for (int e0 = 0; e0 < n_experts; e0 += 8) {
                    const bf16* x0 = (const bf16*)x + (size_t)min(t0 + g, n_tokens - 1) * width + q;
                    const bf16* x1 = (const bf16*)x + (size_t)min(t0 + g + 8, n_tokens - 1) * width + q;
                    float acc[4] = {0.f, 0.f, 0.f, 0.f};
                    for (int s0 = warp; s0 < steps; s0 += AHEAD * n_warps) {
                        if (t0 + e0 > 0 || s0 != warp) router_steps(e0, s0);
                        uint32_t a[AHEAD][4];
#pragma unroll
                        for (int u = 0; u < AHEAD; ++u) {
                            const int s = s0 + u * n_warps;
                            const bool ok = s < steps;
                            a[u][0] = ok ? *reinterpret_cast<const uint32_t*>(x0 + 16 * s) : 0u;
                            a[u][1] = ok ? *reinterpret_cast<const uint32_t*>(x1 + 16 * s) : 0u;
                            a[u][2] = ok ? *reinterpret_cast<const uint32_t*>(x0 + 16 * s + 8) : 0u;
                            a[u][3] = ok ? *reinterpret_cast<const uint32_t*>(x1 + 16 * s + 8) : 0u;
                        }
#pragma unroll
                        for (int u = 0; u < AHEAD; ++u) mma_bf16_16816(acc, a[u], b[u][0], b[u][1]);
                    }
                    __syncthreads();   // the tile before has been added up
                    *reinterpret_cast<float4*>(part + warp * 128 + 4 * lane) = make_float4(acc[0], acc[1], acc[2], acc[3]);
                    __syncthreads();
                    // eight threads per logit, each a run of warps
                    const int i = threadIdx.x >> 3, each = n_warps / 8, from = (threadIdx.x & 7) * each;
                    float z = 0.f;
                    for (int w = from; w < from + each; ++w) z += part[w * 128 + i];
#pragma unroll
                    for (int o = 1; o < 8; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
                    const int t = t0 + (i >> 4) + 8 * ((i >> 1) & 1), e = e0 + 2 * ((i >> 2) & 3) + (i & 1);
                    if ((threadIdx.x & 7) == 0 && t < n_tokens && e < n_experts) logits_out[t * n_experts + e] = bias ? z + bias[e] : z;
                }
        } else if (wide) {
            grid_dependency_wait();
            for (int i = warp; i < n_tokens * n_experts; i += n_warps) {   // a warp per logit, eight elements per load, four loads ahead
                const uint4* xv = reinterpret_cast<const uint4*>((const bf16*)x + (size_t)(i / n_experts) * width);
                const uint4* rv = reinterpret_cast<const uint4*>((const bf16*)router + (size_t)(i % n_experts) * width);
                float sum = 0.f;
                for (int c0 = lane; c0 < width / 8; c0 += 4 * 32) {
                    uint4 a[4], b[4];
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const int c = c0 + 32 * u;
                        a[u] = b[u] = make_uint4(0u, 0u, 0u, 0u);   // (zeros beyond the row's end add nothing)
                        if (c < width / 8) {
                            a[u] = xv[c];
                            b[u] = rv[c];
                        }
                    }
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const __nv_bfloat162* a2 = reinterpret_cast<const __nv_bfloat162*>(&a[u]);
                        const __nv_bfloat162* b2 = reinterpret_cast<const __nv_bfloat162*>(&b[u]);
#pragma unroll
                        for (int j = 0; j < 4; ++j) {
                            const float2 af = __bfloat1622float2(a2[j]), bf = __bfloat1622float2(b2[j]);
                            sum = fmaf(af.x, bf.x, sum);
                            sum = fmaf(af.y, bf.y, sum);
                        }
                    }
                }
                sum = warp_sum(sum);
                if (lane == 0) logits_out[i] = bias ? sum + bias[i % n_experts] : sum;
            }
        } else {
            grid_dependency_wait();
            for (int i = warp; i < n_tokens * n_experts; i += n_warps) {   // a warp per logit
                const int t = i / n_experts, e = i % n_experts;
                float sum = 0.f;
                if (x_is_bf16) {
                    const bf16* xr = (const bf16*)x + (size_t)t * width;
                    const bf16* rr = (const bf16*)router + (size_t)e * width;
                    for (int c = lane; c < width; c += 32) sum = fmaf(__bfloat162float(xr[c]), __bfloat162float(rr[c]), sum);
                } else {
                    const float* xr = (const float*)x + (size_t)t * width;
                    const float* rr = (const float*)router + (size_t)e * width;
                    for (int c = lane; c < width; c += 32) sum = fmaf(xr[c], rr[c], sum);
                }
                sum = warp_sum(sum);
                if (lane == 0) logits_out[i] = bias ? sum + bias[e] : sum;
            }
        }
        logits = logits_out;
        bias = nullptr;
    } else {
        grid_dependency_wait();
    }
    __syncthreads();
    // pass 1: choose, and take a rank among the expert's rows; few pairs stay in shared memory on their way to the second pass
    __shared__ int held_expert[PLAN_HELD], held_rank[PLAN_HELD];
    __shared__ float held_weight[PLAN_HELD];
    int* experts_out = n_tokens * top <= PLAN_HELD ? pair_expert : nullptr;
    if (n_tokens * top <= PLAN_HELD) {
        pair_expert = held_expert;
        pair_weight = held_weight;
    }
    int* rank_of = n_tokens * top <= PLAN_HELD ? held_rank : dest;
    if (n_experts <= 32) {   // a warp per token
        for (int t = threadIdx.x >> 5; t < n_tokens; t += blockDim.x >> 5) {
            const float z = lane < n_experts ? logits[(size_t)t * n_experts + lane] + (bias ? bias[lane] : 0.f) : 0.f;
            float weight;
            const int k = moe_choose_warp(z, n_experts, top, softmax_scores, renormalize, groups, weight);
            if (k >= 0) {
                const int pair = t * top + k;
                pair_expert[pair] = lane;
                rank_of[pair] = atomicAdd(&counts[lane], 1);     // the pair's rank among its expert's rows
                pair_weight[pair] = weight;
            }
        }
    } else {
        for (int t = threadIdx.x; t < n_tokens; t += blockDim.x) {
            int chosen[MOE_MAX_TOP];
            float weight[MOE_MAX_TOP];
            if (groups.count > 0) moe_choose_grouped(logits + (size_t)t * n_experts, bias, n_experts, top, softmax_scores, renormalize, groups, chosen, weight);
            else moe_choose(logits + (size_t)t * n_experts, bias, n_experts, top, softmax_scores, renormalize, chosen, weight);
            for (int k = 0; k < top; ++k) {
                const int pair = t * top + k;
                pair_expert[pair] = chosen[k];
                rank_of[pair] = atomicAdd(&counts[chosen[k]], 1);
                pair_weight[pair] = weight[k];
            }
        }
    }
    __syncthreads();
    if (n_experts <= 32) {
        if (threadIdx.x < 32) {
            int row, tile, rows, tiles;
            moe_scan_warp(lane < n_experts ? counts[lane] : 0, tile_rows, row, tile, rows, tiles);
            if (lane < n_experts) {
                offsets[lane] = row;
                counts[lane] = row;
                first_tile[lane] = tile;
            }
            if (lane == 0) {
                offsets[n_experts] = rows;
                first_tile[n_experts] = tiles;
                n_tiles[0] = tiles < max_tiles ? tiles : max_tiles;
            }
        }
    } else if (threadIdx.x == 0) {
        int row = 0, tile = 0;
        for (int e = 0; e < n_experts; ++e) {
            const int n = counts[e];
            offsets[e] = row;
            counts[e] = row;
            first_tile[e] = tile;
            row += n;
            tile += (n + tile_rows - 1) / tile_rows;
        }
        offsets[n_experts] = row;
        first_tile[n_experts] = tile;
        n_tiles[0] = tile < max_tiles ? tile : max_tiles;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x) {
        const int row0 = counts[e];
        for (int i = first_tile[e]; i < first_tile[e + 1] && i < max_tiles; ++i) {
            tile_group[i] = e;
            tile_row0[i] = row0 + (i - first_tile[e]) * tile_rows;
        }
    }
    // pass 2: every pair's row
    for (int pair = threadIdx.x; pair < n_tokens * top; pair += blockDim.x) {
        const int row = counts[pair_expert[pair]] + rank_of[pair];
        if (experts_out) experts_out[pair] = pair_expert[pair];
        dest[pair] = row;
        sorted_token[row] = pair / top;
        sorted_weight[row] = pair_weight[pair];
    }
}

// The same plan for a long step, where one block would be what the step waits for: (1) blocks of 256 tokens choose and count
// in shared memory, then reserve their rows of every expert with ONE atomic per block and expert on `expert_rows` (zero
// before the launch); (2) one block turns the experts' row counts into offsets and tiles; (3) every pair goes to its row.
__global__ void __launch_bounds__(256)
moe_route_kernel(const float* __restrict__ logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                 int* __restrict__ pair_expert, float* __restrict__ pair_weight, int* __restrict__ dest,
                 int* __restrict__ expert_rows, const float* __restrict__ bias, MoeGroups groups) {
    grid_chain_entry();
    extern __shared__ int shared[];
    int* counts = shared;               // [experts] pairs of this block
    int* base = shared + n_experts;     // [experts] where this block's pairs start among the expert's rows
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x) counts[e] = 0;
    __syncthreads();
    const int t = blockIdx.x * blockDim.x + threadIdx.x;
    int chosen[MOE_MAX_TOP], rank[MOE_MAX_TOP];
    float weight[MOE_MAX_TOP];
    if (t < n_tokens) {
        if (groups.count > 0) moe_choose_grouped(logits + (size_t)t * n_experts, bias, n_experts, top, softmax_scores, renormalize, groups, chosen, weight);
        else moe_choose(logits + (size_t)t * n_experts, bias, n_experts, top, softmax_scores, renormalize, chosen, weight);
        for (int k = 0; k < top; ++k) rank[k] = atomicAdd(&counts[chosen[k]], 1);
    }
    __syncthreads();
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x) base[e] = counts[e] > 0 ? atomicAdd(&expert_rows[e], counts[e]) : 0;
    __syncthreads();
    if (t < n_tokens)
        for (int k = 0; k < top; ++k) {
            const int pair = t * top + k;
            pair_expert[pair] = chosen[k];
            dest[pair] = base[chosen[k]] + rank[k];
            pair_weight[pair] = weight[k];
        }
}

// (1) by a warp per token, up to 32 experts; a block takes ROUTE_TOKENS tokens.
#define ROUTE_TOKENS 16
__global__ void __launch_bounds__(256)
moe_route_warp_kernel(const float* __restrict__ logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                      int* __restrict__ pair_expert, float* __restrict__ pair_weight, int* __restrict__ dest,
                      int* __restrict__ expert_rows, const float* __restrict__ bias, MoeGroups groups) {
    grid_chain_entry();
    __shared__ int counts[32], base[32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (threadIdx.x < 32) counts[threadIdx.x] = 0;
    __syncthreads();
    constexpr int EACH = ROUTE_TOKENS / 8;
    int place[EACH], rank[EACH];
    float z[EACH], weight[EACH];
#pragma unroll
    for (int u = 0; u < EACH; ++u) {
        const int t = blockIdx.x * ROUTE_TOKENS + warp * EACH + u;
        z[u] = t < n_tokens && lane < n_experts ? logits[(size_t)t * n_experts + lane] + (bias ? bias[lane] : 0.f) : 0.f;
    }
#pragma unroll
    for (int u = 0; u < EACH; ++u) {
        place[u] = moe_choose_warp(z[u], n_experts, top, softmax_scores, renormalize, groups, weight[u]);
        if (blockIdx.x * ROUTE_TOKENS + warp * EACH + u >= n_tokens) place[u] = -1;
        rank[u] = place[u] >= 0 ? atomicAdd(&counts[lane], 1) : 0;
    }
    __syncthreads();
    if (threadIdx.x < n_experts) base[threadIdx.x] = counts[threadIdx.x] > 0 ? atomicAdd(&expert_rows[threadIdx.x], counts[threadIdx.x]) : 0;
    __syncthreads();
#pragma unroll
    for (int u = 0; u < EACH; ++u) {
        if (place[u] < 0) continue;
        const int pair = (blockIdx.x * ROUTE_TOKENS + warp * EACH + u) * top + place[u];
        pair_expert[pair] = lane;
        dest[pair] = base[lane] + rank[u];
        pair_weight[pair] = weight[u];
    }
}

// (2) and (3) in one launch for up to 32 experts: every block works the experts' first rows out for itself, the first one also writes
// the offsets and the tiles.
__global__ void __launch_bounds__(256)
moe_place_warp_kernel(const int* __restrict__ pair_expert, const float* __restrict__ pair_weight, const int* __restrict__ expert_rows,
                      int n_experts, int* __restrict__ offsets, int* __restrict__ tile_group, int* __restrict__ tile_row0,
                      int* __restrict__ n_tiles, int max_tiles, int tile_rows, int* __restrict__ dest, int* __restrict__ sorted_token,
                      float* __restrict__ sorted_weight, int pairs, int top) {
    grid_chain_entry();
    __shared__ int first[32];
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x, n = lane < n_experts ? expert_rows[lane] : 0;
        int row, tile, rows, tiles;
        moe_scan_warp(n, tile_rows, row, tile, rows, tiles);
        first[lane] = row;
        if (blockIdx.x == 0) {
            if (lane < n_experts) {
                offsets[lane] = row;
                for (int i = 0; i * tile_rows < n && tile + i < max_tiles; ++i) {
                    tile_group[tile + i] = lane;
                    tile_row0[tile + i] = row + i * tile_rows;
                }
            }
            if (lane == 0) {
                offsets[n_experts] = rows;
                n_tiles[0] = tiles < max_tiles ? tiles : max_tiles;
            }
        }
    }
    __syncthreads();
    const int pair = blockIdx.x * blockDim.x + threadIdx.x;
    if (pair >= pairs) return;
    const int row = first[pair_expert[pair]] + dest[pair];
    dest[pair] = row;
    sorted_token[row] = pair / top;
    sorted_weight[row] = pair_weight[pair];
}

__global__ void __launch_bounds__(256)
moe_offsets_kernel(const int* __restrict__ expert_rows, int n_experts, int* __restrict__ offsets, int* __restrict__ tile_group,
                   int* __restrict__ tile_row0, int* __restrict__ n_tiles, int max_tiles, int tile_rows) {
    grid_chain_entry();
    extern __shared__ int shared[];
    int* first_row = shared;                 // [experts]
    int* first_tile = shared + n_experts;    // [experts + 1]
    if (threadIdx.x == 0) {
        int row = 0, tile = 0;
        for (int e = 0; e < n_experts; ++e) {
            const int n = expert_rows[e];
            offsets[e] = row;
            first_row[e] = row;
            first_tile[e] = tile;
            row += n;
            tile += (n + tile_rows - 1) / tile_rows;
        }
        offsets[n_experts] = row;
        first_tile[n_experts] = tile;
        n_tiles[0] = tile < max_tiles ? tile : max_tiles;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x)
        for (int i = first_tile[e]; i < first_tile[e + 1] && i < max_tiles; ++i) {
            tile_group[i] = e;
            tile_row0[i] = first_row[e] + (i - first_tile[e]) * tile_rows;
        }
}

__global__ void __launch_bounds__(256)
moe_place_kernel(const int* __restrict__ pair_expert, const float* __restrict__ pair_weight, const int* __restrict__ offsets,
                 int* __restrict__ dest, int* __restrict__ sorted_token, float* __restrict__ sorted_weight, int pairs, int top) {
    grid_chain_entry();
    const int pair = blockIdx.x * blockDim.x + threadIdx.x;
    if (pair >= pairs) return;
    const int row = offsets[pair_expert[pair]] + dest[pair];
    dest[pair] = row;
    sorted_token[row] = pair / top;
    sorted_weight[row] = pair_weight[pair];
}

template <typename T>
__global__ void __launch_bounds__(128)
moe_gather_kernel(const T* __restrict__ x, const int* __restrict__ sorted_token, const float* __restrict__ sorted_weight,
                  T* __restrict__ out, int n_rows, int width, int scale_input) {
    grid_chain_entry();
    const int r = blockIdx.x;
    if (r >= n_rows) return;
    const T* src = x + (size_t)sorted_token[r] * width;
    const float w = scale_input ? sorted_weight[r] : 1.f;
    T* dst = out + (size_t)r * width;
    if (!scale_input && ((size_t)width * sizeof(T)) % 16 == 0 && (((uintptr_t)x | (uintptr_t)out) & 15) == 0) {
        const uint4* s4 = reinterpret_cast<const uint4*>(src);   // a plain copy of the row, 16 bytes at a time
        uint4* d4 = reinterpret_cast<uint4*>(dst);
        for (int c = threadIdx.x; c < (int)((size_t)width * sizeof(T) / 16); c += blockDim.x) d4[c] = s4[c];
        return;
    }
    for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = Num<T>::from_f(Num<T>::to_f(src[c]) * w);
}

template <typename T>
__global__ void __launch_bounds__(128)
moe_combine_kernel(const T* __restrict__ y, const int* __restrict__ dest, const float* __restrict__ sorted_weight,
                   T* __restrict__ out, int n_tokens, int top, int width, int scale_output, const T* __restrict__ extra,
                   const float* __restrict__ extra_gate, const T* __restrict__ gate_input, const T* __restrict__ gate_weight,
                   int gate_k) {
    grid_chain_entry();
    __shared__ float scratch[33];
    const int t = blockIdx.x;
    if (t >= n_tokens) return;
    // an output that every token gets beside its chosen ones (`extra`), under a sigmoid gate of one logit per token: given,
    // or formed here as the token's row times the gate's weights (float32 sums in a fixed order)
    constexpr int V = 16 / (int)sizeof(T);
    // the rows of the token's pairs and their weights are asked for first: two loads that hang on each other, on their way
    // while the gate's logit is formed
    const bool wide = width % V == 0 && top <= MOE_MAX_TOP && (((uintptr_t)y | (uintptr_t)out | (uintptr_t)extra) & 15) == 0;
    int row[MOE_MAX_TOP];
    float rw[MOE_MAX_TOP];
    if (wide) {
#pragma unroll
        for (int k = 0; k < MOE_MAX_TOP; ++k)
            if (k < top) {
                row[k] = dest[t * top + k];
                rw[k] = scale_output ? sorted_weight[row[k]] : 1.f;
            }
    }
    float share = extra ? 1.f : 0.f;
    if (extra && extra_gate) share = 1.f / (1.f + expf(-extra_gate[t]));
    if (extra && gate_weight) {
        float sum = 0.f;
        if (gate_k % V == 0 && (((uintptr_t)gate_input | (uintptr_t)gate_weight) & 15) == 0) {
            for (int c = threadIdx.x * V; c < gate_k; c += blockDim.x * V) {   // 16 bytes of the row and of the weights at a time
                T a[V], b[V];
                *reinterpret_cast<uint4*>(a) = *reinterpret_cast<const uint4*>(gate_input + (size_t)t * gate_k + c);
                *reinterpret_cast<uint4*>(b) = *reinterpret_cast<const uint4*>(gate_weight + c);
#pragma unroll
                for (int v = 0; v < V; ++v) sum = fmaf(Num<T>::to_f(a[v]), Num<T>::to_f(b[v]), sum);
            }
        } else {
            for (int c = threadIdx.x; c < gate_k; c += blockDim.x)
                sum = fmaf(Num<T>::to_f(gate_input[(size_t)t * gate_k + c]), Num<T>::to_f(gate_weight[c]), sum);
        }
        share = 1.f / (1.f + expf(-block_sum(sum, scratch)));
    }
    if (wide) {
        // the same sums, 16 bytes of every row at a time
        for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
            float sum[V];
#pragma unroll
            for (int v = 0; v < V; ++v) sum[v] = 0.f;
#pragma unroll
            for (int k = 0; k < MOE_MAX_TOP; ++k)
                if (k < top) {
                    T in[V];
                    *reinterpret_cast<uint4*>(in) = *reinterpret_cast<const uint4*>(y + (size_t)row[k] * width + c);
#pragma unroll
                    for (int v = 0; v < V; ++v) sum[v] += scale_output ? Num<T>::to_f(in[v]) * rw[k] : Num<T>::to_f(in[v]);
                }
            T res[V];
            if (extra) {
                T in[V];
                *reinterpret_cast<uint4*>(in) = *reinterpret_cast<const uint4*>(extra + (size_t)t * width + c);
#pragma unroll
                for (int v = 0; v < V; ++v) sum[v] = fmaf(share, Num<T>::to_f(in[v]), sum[v]);
            }
#pragma unroll
            for (int v = 0; v < V; ++v) res[v] = Num<T>::from_f(sum[v]);
            *reinterpret_cast<uint4*>(out + (size_t)t * width + c) = *reinterpret_cast<const uint4*>(res);
        }
        return;
    }
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float sum = 0.f;
        for (int k = 0; k < top; ++k) {
            const int row = dest[t * top + k];
            const float v = Num<T>::to_f(y[(size_t)row * width + c]);
            sum += scale_output ? v * sorted_weight[row] : v;
        }
        if (extra) sum = fmaf(share, Num<T>::to_f(extra[(size_t)t * width + c]), sum);
        out[(size_t)t * width + c] = Num<T>::from_f(sum);
    }
}

// pairs = n_tokens * top: pair_expert, pair_weight (scratch), sorted_token, sorted_weight and dest have that many elements;
// tile_group and tile_row0 max_tiles >= ceil(pairs / tile_rows) + n_experts. Either `logits` float32 [n_tokens][n_experts]
// is given, or x [n_tokens][width] and router [n_experts][width] (both bfloat16 or both float32), from which the kernel makes
// the logits itself in shared memory (n_tokens * n_experts <= 8192).
// bias: float32 [n_experts] added to the logits, or null.
// correction (float32 [n_experts] or null), group_count, group_keep, group_best: the choice among groups of neighbouring experts
// (`moe_choose_grouped`); group_count 0: the plain choice.
QF_EXPORT int qf_moe_plan_grouped(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                                  int* pair_expert, float* pair_weight, int* sorted_token, float* sorted_weight, int* dest,
                                  int* offsets, int* tile_group, int* tile_row0, int* n_tiles, int max_tiles, int tile_rows,
                                  const void* x, const void* router, int width, int x_is_bf16, const float* bias,
                                  const float* correction, int group_count, int group_keep, int group_best, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (group_count < 0 || group_count > MOE_MAX_GROUPS || (group_count > 0 && (n_experts % group_count || group_keep < 1 ||
        group_keep > group_count || (long long)group_keep * (n_experts / group_count) < top || group_best < 1 || group_best > 2)))
        return (int)cudaErrorInvalidValue;
    const MoeGroups groups = {correction, group_count, group_keep, group_best};
    if (top < 1 || top > MOE_MAX_TOP || top > n_experts || n_experts > 8192 || tile_rows <= 0) return (int)cudaErrorInvalidValue;
    if (!logits && !(x && router && (long long)n_tokens * n_experts <= 8192)) return (int)cudaErrorInvalidValue;
    const size_t logits_floats = (size_t)((long long)n_tokens * n_experts + 3) / 4 * 4;
    const size_t smem = (size_t)((2 * n_experts + 1 + 3) / 4 * 4) * sizeof(int) +
                        (logits ? 0 : logits_floats * sizeof(float) + (plan_on_tiles(n_tokens, n_experts, width) ? MOE_PLAN_THREADS / 32 * 128 * sizeof(float) : 0));
    if (smem > 40 * 1024) {   // (the kernel has six KB of its own beside it)
        cudaError_t e = cudaFuncSetAttribute(moe_plan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(moe_plan_kernel, dim3(1), dim3(MOE_PLAN_THREADS), smem, stream, logits, n_tokens, n_experts, top,
                           softmax_scores, renormalize, pair_expert, pair_weight, sorted_token, sorted_weight, dest, offsets,
                           tile_group, tile_row0, n_tiles, max_tiles, tile_rows, logits ? nullptr : x, router, width, x_is_bf16, bias,
                           groups);
}

QF_EXPORT int qf_moe_plan_biased(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                                 int* pair_expert, float* pair_weight, int* sorted_token, float* sorted_weight, int* dest,
                                 int* offsets, int* tile_group, int* tile_row0, int* n_tiles, int max_tiles, int tile_rows,
                                 const void* x, const void* router, int width, int x_is_bf16, const float* bias,
                                 cudaStream_t stream) {
    return qf_moe_plan_grouped(logits, n_tokens, n_experts, top, softmax_scores, renormalize, pair_expert, pair_weight, sorted_token,
                               sorted_weight, dest, offsets, tile_group, tile_row0, n_tiles, max_tiles, tile_rows, x, router, width,
                               x_is_bf16, bias, nullptr, 0, 0, 2, stream);
}

QF_EXPORT int qf_moe_plan(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                          int* pair_expert, float* pair_weight, int* sorted_token, float* sorted_weight, int* dest,
                          int* offsets, int* tile_group, int* tile_row0, int* n_tiles, int max_tiles, int tile_rows,
                          const void* x, const void* router, int width, int x_is_bf16, cudaStream_t stream) {
    return qf_moe_plan_biased(logits, n_tokens, n_experts, top, softmax_scores, renormalize, pair_expert, pair_weight, sorted_token,
                              sorted_weight, dest, offsets, tile_group, tile_row0, n_tiles, max_tiles, tile_rows, x, router, width,
                              x_is_bf16, nullptr, stream);
}

QF_EXPORT int qf_moe_gather(int is_bf16, const void* x, const int* sorted_token, const float* sorted_weight, void* out,
                            int n_rows, int width, int scale_input, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (is_bf16)
        return (int)launch_pdl(moe_gather_kernel<bf16>, dim3(n_rows), dim3(128), 0, stream, (const bf16*)x, sorted_token,
                               sorted_weight, (bf16*)out, n_rows, width, scale_input);
    return (int)launch_pdl(moe_gather_kernel<float>, dim3(n_rows), dim3(128), 0, stream, (const float*)x, sorted_token,
                           sorted_weight, (float*)out, n_rows, width, scale_input);
}

// extra: [n_tokens][width] added to every token's sum (or null), times sigmoid(extra_gate[t]) where extra_gate (float32
// [n_tokens]) is given, or times sigmoid(gate_input[t] . gate_weight) where gate_weight [gate_k] and gate_input
// [n_tokens][gate_k] are.
QF_EXPORT int qf_moe_combine_shared(int is_bf16, const void* y, const int* dest, const float* sorted_weight, void* out, int n_tokens,
                                    int top, int width, int scale_output, const void* extra, const float* extra_gate,
                                    const void* gate_input, const void* gate_weight, int gate_k, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (is_bf16)
        return (int)launch_pdl(moe_combine_kernel<bf16>, dim3(n_tokens), dim3(128), 0, stream, (const bf16*)y, dest, sorted_weight,
                               (bf16*)out, n_tokens, top, width, scale_output, (const bf16*)extra, extra_gate,
                               (const bf16*)gate_input, (const bf16*)gate_weight, gate_k);
    return (int)launch_pdl(moe_combine_kernel<float>, dim3(n_tokens), dim3(128), 0, stream, (const float*)y, dest, sorted_weight,
                           (float*)out, n_tokens, top, width, scale_output, (const float*)extra, extra_gate,
                           (const float*)gate_input, (const float*)gate_weight, gate_k);
}

QF_EXPORT int qf_moe_combine(int is_bf16, const void* y, const int* dest, const float* sorted_weight, void* out, int n_tokens,
                             int top, int width, int scale_output, cudaStream_t stream) {
    return qf_moe_combine_shared(is_bf16, y, dest, sorted_weight, out, n_tokens, top, width, scale_output, nullptr, nullptr, nullptr,
                                 nullptr, 0, stream);
}

// The plan of a long step by three launches (see moe_route_kernel), or two for up to 32 experts. expert_rows: int32 [n_experts], zero before the call.
QF_EXPORT int qf_moe_plan_long_grouped(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores,
                                       int renormalize, int* pair_expert, float* pair_weight, int* sorted_token,
                                       float* sorted_weight, int* dest, int* offsets, int* tile_group, int* tile_row0, int* n_tiles,
                                       int max_tiles, int tile_rows, int* expert_rows, const float* bias, const float* correction,
                                       int group_count, int group_keep, int group_best, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (group_count < 0 || group_count > MOE_MAX_GROUPS || (group_count > 0 && (n_experts % group_count || group_keep < 1 ||
        group_keep > group_count || (long long)group_keep * (n_experts / group_count) < top || group_best < 1 || group_best > 2)))
        return (int)cudaErrorInvalidValue;
    const MoeGroups groups = {correction, group_count, group_keep, group_best};
    if (top < 1 || top > MOE_MAX_TOP || top > n_experts || n_experts > 4096 || tile_rows <= 0 || !logits || !expert_rows)
        return (int)cudaErrorInvalidValue;
    const int pairs = n_tokens * top;
    if (n_experts <= 32) {
        int code = (int)launch_pdl(moe_route_warp_kernel, dim3((n_tokens + ROUTE_TOKENS - 1) / ROUTE_TOKENS), dim3(256), 0, stream, logits, n_tokens,
                                   n_experts, top, softmax_scores, renormalize, pair_expert, pair_weight, dest, expert_rows, bias, groups);
        if (code) return code;
        return (int)launch_pdl(moe_place_warp_kernel, dim3((pairs + 255) / 256), dim3(256), 0, stream, (const int*)pair_expert,
                               (const float*)pair_weight, (const int*)expert_rows, n_experts, offsets, tile_group, tile_row0, n_tiles, max_tiles,
                               tile_rows, dest, sorted_token, sorted_weight, pairs, top);
    }
    const size_t smem = (size_t)(2 * n_experts + 1) * sizeof(int);
    int code = (int)launch_pdl(moe_route_kernel, dim3((n_tokens + 255) / 256), dim3(256), smem, stream, logits, n_tokens, n_experts,
                               top, softmax_scores, renormalize, pair_expert, pair_weight, dest, expert_rows, bias, groups);
    if (code) return code;
    code = (int)launch_pdl(moe_offsets_kernel, dim3(1), dim3(256), smem, stream, (const int*)expert_rows, n_experts, offsets,
                           tile_group, tile_row0, n_tiles, max_tiles, tile_rows);
    if (code) return code;
    return (int)launch_pdl(moe_place_kernel, dim3((pairs + 255) / 256), dim3(256), 0, stream, (const int*)pair_expert,
                           (const float*)pair_weight, (const int*)offsets, dest, sorted_token, sorted_weight, pairs, top);
}

QF_EXPORT int qf_moe_plan_long_biased(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores,
                                      int renormalize, int* pair_expert, float* pair_weight, int* sorted_token,
                                      float* sorted_weight, int* dest, int* offsets, int* tile_group, int* tile_row0, int* n_tiles,
                                      int max_tiles, int tile_rows, int* expert_rows, const float* bias, cudaStream_t stream) {
    return qf_moe_plan_long_grouped(logits, n_tokens, n_experts, top, softmax_scores, renormalize, pair_expert, pair_weight,
                                    sorted_token, sorted_weight, dest, offsets, tile_group, tile_row0, n_tiles, max_tiles, tile_rows,
                                    expert_rows, bias, nullptr, 0, 0, 2, stream);
}

QF_EXPORT int qf_moe_plan_long(const float* logits, int n_tokens, int n_experts, int top, int softmax_scores, int renormalize,
                               int* pair_expert, float* pair_weight, int* sorted_token, float* sorted_weight, int* dest,
                               int* offsets, int* tile_group, int* tile_row0, int* n_tiles, int max_tiles, int tile_rows,
                               int* expert_rows, cudaStream_t stream) {
    return qf_moe_plan_long_biased(logits, n_tokens, n_experts, top, softmax_scores, renormalize, pair_expert, pair_weight,
                                   sorted_token, sorted_weight, dest, offsets, tile_group, tile_row0, n_tiles, max_tiles, tile_rows,
                                   expert_rows, nullptr, stream);
}
