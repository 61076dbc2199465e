// Causal grouped-query flash attention for spans of new tokens over the paged cache (bf16): whole prompts of
// unequal lengths, and continuations whose earlier keys already lie in the cache. The span's own keys were
// written to the cache before this kernel runs, so all keys come from one place.
//
// A block serves 64 consecutive query tokens of one (sequence, query head) with G groups of 4 warps; in a group each
// warp owns 16 rows. Key/value pages (64 positions) of the head's kv head stream through shared memory with
// double-buffered cp.async, G pages per turn, from the first page that any row's window reaches to the page of the
// last row's own position; group g takes every G-th page, so a tile's chain of pages is 1 / G as long (a single
// prompt's last tile walks all of its pages while the SMs have room for more warps). At the end the groups' running
// maxima, sums and outputs of the same rows are merged through shared memory, lane by lane.
// S = Q K^T and O += P V run on the tensor cores (m16n8k16, bf16 in, float32 accumulate); the online softmax
// is float32 with base-2 exponentials (the scale folded in). A query at position p sees keys j with
// max(0, p - window + 1) <= j <= p.
// `sinks` (float32 per query head, or null): a logit that joins the softmax's denominator once, unscaled, with no key and
// no value. `shared_values`: the values are the keys themselves (pages of one plane, as a latent attention keeps them):
// a page is fetched once and read as both.
// `pool` > 0 (with a window): beside the window's keys a query at p sees one key and value for every block of `pool`
// positions that lies wholly before its window (blocks b with b * pool + pool - 1 <= p - window). Those rows live in a
// second cache of the same head shape, one row per block (`blocks`); its pages are walked first, by the same loop and the
// same buffers, masked by how many blocks each row sees, and share the softmax with the window's keys.
// `bias_scale`, `bias_rate` (float32 per query head, or null): after the cap a score of key j under query i loses
// bias_scale[h] * ln(1 + bias_rate[h] * (i - j)), with the hardware's base-2 logarithm on the float32 argument; compiled as a
// variant of its own.
#include "mma.cuh"

#define PF_WARPS 4
#define PF_THREADS (PF_WARPS * 32)
#define PF_BM 64

__device__ __forceinline__ float fast_tanh(float x) {
    float y;
    asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int D, int G, bool POOLED, bool BIASED>
__global__ void __launch_bounds__(PF_THREADS * G, (D <= 64 ? 4 : 2) / G)
prefill_flash_kernel(const bf16* __restrict__ q, bf16* __restrict__ out, const int* __restrict__ cu_q,
                     const int* __restrict__ tok_pos, const int* __restrict__ slots, KvSite<bf16> site, int n_heads,
                     int n_seqs, int n_tiles, int wave, float scale_log2, int window, int* err,
                     const float* __restrict__ sinks, int shared_values, int mask_block, float cap_in, float cap_out,
                     KvSite<bf16> blocks, int pool, const float* __restrict__ bias_scale, const float* __restrict__ bias_rate) {
    grid_chain_entry();
    auto seen_of = [&](int pos) -> int {   // blocks of `pool` positions wholly before the window of a query at `pos`
        const int past = pos - window + 1;
        return POOLED && pool > 0 && window > 0 && past >= pool ? past / pool : 0;
    };
    // capped scores: s <- cap * tanh(s * scale / cap) in base-2 units, cap_in = scale / cap, cap_out = cap * log2(e); the
    // capped score then needs no further scale
    const float sl2 = cap_out > 0.f || BIASED ? 1.f : scale_log2;
    auto lo_of = [&](int pos) -> int {   // lowest position a query at `pos` sees: its window and its block of the mask
        int lo = window > 0 ? max(0, pos - window + 1) : 0;
        if (mask_block > 0) lo = max(lo, pos / mask_block * mask_block);
        return lo;
    };
    constexpr int LD = D + 8;
    constexpr int KS = D / 16;
    constexpr int NT = D / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* k_s = reinterpret_cast<bf16*>(smem_raw);  // [2][G][64][LD]
    bf16* v_s = shared_values ? k_s : k_s + 2 * G * QF_PAGE * LD;  // [2][G][64][LD]; the keys' own buffer when they are the values

    // Which (tile, head, sequence) this block serves. Tiles further down a prompt walk more pages, and the SMs hold
    // several blocks each, so what counts is that the blocks that share an SM have about the same work together:
    // blocks are taken in waves of `wave` (one block per SM), the first wave gets the longest tiles in falling order,
    // the second the next longest in rising order, and so on, so that the block that follows a long tile onto the same
    // SM is a short one.
    const int total = (int)gridDim.x, w = blockIdx.x / wave, j = blockIdx.x % wave;
    const int in_wave = min(wave, total - w * wave);
    const int item = w * wave + ((w & 1) ? in_wave - 1 - j : j);
    const int per_tile = n_heads * n_seqs;
    const int tile = n_tiles - 1 - item / per_tile, head = (item % per_tile) % n_heads, seq = (item % per_tile) / n_heads;
    const int q_begin = cu_q[seq], q_len = cu_q[seq + 1] - q_begin;
    const int row0 = tile * PF_BM;
    if (row0 >= q_len) return;
    const int n_rows = min(PF_BM, q_len - row0);
    const int slot = slots[seq];
    const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) % PF_WARPS, group = (threadIdx.x >> 5) / PF_WARPS;
    const int q_width = n_heads * D;
    const int kvh = head / (n_heads / site.kv_heads);

    if (slot < 0) {
        for (int i = threadIdx.x; i < n_rows * D; i += PF_THREADS * G)
            out[(size_t)(q_begin + row0 + i / D) * q_width + (size_t)head * D + i % D] = __float2bfloat16_rn(0.f);
        return;
    }
    const int pos0 = tok_pos[q_begin + row0];             // position of the tile's first row
    const int last_pos = pos0 + n_rows - 1;
    const int lo_min = lo_of(pos0);
    const int p_begin = lo_min / QF_PAGE, p_end = last_pos / QF_PAGE + 1;
    // the walk: n_pool pages of block rows first (walk index v < n_pool is page v of `blocks`), then pages p_begin .. p_end - 1
    // of the positions (walk index v is page p_begin + v - n_pool)
    const int n_pool = POOLED ? (seen_of(last_pos) + QF_PAGE - 1) / QF_PAGE : 0;
    const int v_end = n_pool + p_end - p_begin;

    // this thread's two rows
    const int r[2] = {16 * warp + (lane >> 2), 16 * warp + (lane >> 2) + 8};
    const bool row_ok[2] = {r[0] < n_rows, r[1] < n_rows};
    const int row_pos[2] = {pos0 + r[0], pos0 + r[1]};
    const int row_lo[2] = {lo_of(row_pos[0]), lo_of(row_pos[1])};
    const int row_seen[2] = {seen_of(row_pos[0]), seen_of(row_pos[1])};
    // the warp's rows span positions [warp_first, warp_last]
    const int warp_first = pos0 + 16 * warp, warp_last = min(pos0 + 16 * warp + 15, last_pos);
    const int warp_lo = lo_of(warp_first);
    const bool warp_active = 16 * warp < n_rows;

    uint32_t qa[KS][4];
    {
        const int c = 2 * (lane & 3);
        const bf16* q0 = q + (size_t)(q_begin + row0 + r[0]) * q_width + (size_t)head * D;
        const bf16* q1 = q + (size_t)(q_begin + row0 + r[1]) * q_width + (size_t)head * D;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            qa[ks][0] = row_ok[0] ? *reinterpret_cast<const uint32_t*>(q0 + 16 * ks + c) : 0u;
            qa[ks][1] = row_ok[1] ? *reinterpret_cast<const uint32_t*>(q1 + 16 * ks + c) : 0u;
            qa[ks][2] = row_ok[0] ? *reinterpret_cast<const uint32_t*>(q0 + 16 * ks + 8 + c) : 0u;
            qa[ks][3] = row_ok[1] ? *reinterpret_cast<const uint32_t*>(q1 + 16 * ks + 8 + c) : 0u;
        }
    }
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m_run[2] = {QF_NEG_BIG, QF_NEG_BIG}, l_run[2] = {0.f, 0.f};

    const int* table_row = site.table + (long long)slot * site.table_stride;
    const int* blocks_row = n_pool > 0 ? blocks.table + (long long)slot * blocks.table_stride : nullptr;
    // the pages of one turn: walk index first + g goes to group g's buffer; every thread helps to fetch all of them
    auto load_pages = [&](int first, int buf) {
        for (int gi = 0; gi < G; ++gi) {
            const int v = first + gi;
            if (v >= v_end) break;
            const bool rows = POOLED && v < n_pool;
            const KvSite<bf16>& from = rows ? blocks : site;
            const int page = rows ? blocks_row[v] : table_row[p_begin + v - n_pool];
            const bool held = page >= 0;
            if (!held && threadIdx.x == 0) atomicOr(err, QF_ERR_NO_PAGE);
            const bf16* kp = from.base + (long long)(held ? page : 0) * from.page_elems + (long long)kvh * QF_PAGE * D;
            const bf16* vp = kp + (long long)from.kv_heads * QF_PAGE * D;
            constexpr int CH = D / 8;
            for (int i = threadIdx.x; i < QF_PAGE * CH; i += PF_THREADS * G) {
                const int rr = i / CH, c = (i % CH) * 8;
                cp_async_16(k_s + (((size_t)buf * G + gi) * QF_PAGE + rr) * LD + c, kp + rr * D + c, held);
                if (!shared_values) cp_async_16(v_s + (((size_t)buf * G + gi) * QF_PAGE + rr) * LD + c, vp + rr * D + c, held);
            }
        }
    };

    load_pages(0, 0);
    cp_async_commit();
    for (int first = 0, turn = 0; first < v_end; first += G, ++turn) {
        const int buf = turn & 1;
        if (first + G < v_end) load_pages(first + G, buf ^ 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const int v = first + group;
        const bool rows = POOLED && v < n_pool;   // a page of block rows: its "positions" are block indices, seen from 0 up to a count
        const bf16* kb = k_s + ((size_t)buf * G + group) * QF_PAGE * LD;
        const bf16* vb = v_s + ((size_t)buf * G + group) * QF_PAGE * LD;
        const int key0 = (rows ? v : p_begin + v - n_pool) * QF_PAGE;
        const int span_last = rows ? seen_of(warp_last) - 1 : warp_last, span_lo = rows ? 0 : warp_lo;
        if (v < v_end && warp_active && key0 <= span_last && key0 + QF_PAGE > span_lo) {
            float s[8][4];
#pragma unroll
            for (int t = 0; t < 8; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
                for (int t2 = 0; t2 < 4; ++t2) {  // 16 keys per ldmatrix.x4
                    uint32_t kf[4];
                    ldmatrix_x4(kf, kb + (size_t)(16 * t2 + (lane >> 4) * 8 + (lane & 7)) * LD + 16 * ks + ((lane >> 3) & 1) * 8);
                    mma_bf16_16816(s[2 * t2], qa[ks], kf[0], kf[1]);
                    mma_bf16_16816(s[2 * t2 + 1], qa[ks], kf[2], kf[3]);
                }
            }
            // a page that every row of the warp sees whole needs no mask
            if (cap_out > 0.f) {
#pragma unroll
                for (int t = 0; t < 8; ++t)
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[t][e] = cap_out * fast_tanh(s[t][e] * cap_in);
            }
            if (BIASED) {   // in base-2 units: the factor log2(e) turns the natural logarithm into the base-2 one
                const float by = bias_scale[head], rate = bias_rate[head], raw = cap_out > 0.f ? 1.f : scale_log2;
#pragma unroll
                for (int t = 0; t < 8; ++t)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float far = (float)(row_pos[e >> 1] - (key0 + 8 * t + 2 * (lane & 3) + (e & 1)));
                        s[t][e] = fmaf(-by, __log2f(fmaf(rate, fmaxf(far, 0.f), 1.f)), s[t][e] * raw);
                    }
            }
            const bool full = rows ? key0 + QF_PAGE <= seen_of(warp_first)
                                   : key0 + QF_PAGE - 1 <= warp_first && key0 >= lo_of(warp_last);
            float corr[2], sum[2] = {0.f, 0.f};
            if (full) {
                // the common case (every page left of the diagonal): no comparisons, one fused multiply-add and one
                // hardware exponential per score
                float mx[2] = {s[0][0], s[0][2]};
#pragma unroll
                for (int t = 0; t < 8; ++t) {
                    mx[0] = fmaxf(mx[0], fmaxf(s[t][0], s[t][1]));
                    mx[1] = fmaxf(mx[1], fmaxf(s[t][2], s[t][3]));
                }
                float neg_m[2];
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
                    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
                    const float m_new = fmaxf(m_run[i], mx[i] * sl2);
                    corr[i] = fast_exp2(m_run[i] - m_new);
                    m_run[i] = m_new;
                    neg_m[i] = -m_new;
                }
#pragma unroll
                for (int t = 0; t < 8; ++t) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        s[t][e] = fast_exp2(fmaf(s[t][e], sl2, neg_m[0]));
                        s[t][2 + e] = fast_exp2(fmaf(s[t][2 + e], sl2, neg_m[1]));
                        sum[0] += s[t][e];
                        sum[1] += s[t][2 + e];
                    }
                }
            } else {
                float mx[2] = {QF_NEG_BIG, QF_NEG_BIG};
#pragma unroll
                for (int t = 0; t < 8; ++t) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int kj = key0 + 8 * t + 2 * (lane & 3) + e;
                        const bool ok0 = rows ? kj < row_seen[0] : kj <= row_pos[0] && kj >= row_lo[0];
                        const bool ok1 = rows ? kj < row_seen[1] : kj <= row_pos[1] && kj >= row_lo[1];
                        s[t][e] = ok0 ? s[t][e] * sl2 : QF_NEG_BIG;
                        s[t][2 + e] = ok1 ? s[t][2 + e] * sl2 : QF_NEG_BIG;
                        mx[0] = fmaxf(mx[0], s[t][e]);
                        mx[1] = fmaxf(mx[1], s[t][2 + e]);
                    }
                }
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
                    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
                    const float m_new = fmaxf(m_run[i], mx[i]);
                    corr[i] = fast_exp2(m_run[i] - m_new);
                    m_run[i] = m_new;
                }
#pragma unroll
                for (int t = 0; t < 8; ++t) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        // a masked score is QF_NEG_BIG: its exponential is 0 unless the whole row is masked so far,
                        // in which case the maximum is QF_NEG_BIG too and the difference would be 0
                        s[t][e] = s[t][e] > 0.5f * QF_NEG_BIG ? fast_exp2(s[t][e] - m_run[0]) : 0.f;
                        s[t][2 + e] = s[t][2 + e] > 0.5f * QF_NEG_BIG ? fast_exp2(s[t][2 + e] - m_run[1]) : 0.f;
                        sum[0] += s[t][e];
                        sum[1] += s[t][2 + e];
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
                sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
                l_run[i] = l_run[i] * corr[i] + sum[i];
            }
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
                o[nt][0] *= corr[0];
                o[nt][1] *= corr[0];
                o[nt][2] *= corr[1];
                o[nt][3] *= corr[1];
            }
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {  // 16 keys per step
                uint32_t pa[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                  pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
                for (int nt = 0; nt < NT; nt += 2) {
                    uint32_t vf[4];
                    ldmatrix_x4_trans(vf, vb + (size_t)(16 * kk + ((lane >> 3) & 1) * 8 + (lane & 7)) * LD + 8 * nt + (lane >> 4) * 8);
                    mma_bf16_16816(o[nt], pa, vf[0], vf[1]);
                    mma_bf16_16816(o[nt + 1], pa, vf[2], vf[3]);
                }
            }
        }
        __syncthreads();
    }
    cp_async_wait<0>();
    if (G > 1) {
        // ---- merge the groups: a lane of group g > 0 leaves its maxima, sums and outputs where the lane of group 0 with
        // the same rows finds them (the page buffers are free: the loop ended with a block-wide barrier)
        constexpr int PER_LANE = NT * 4 + 4;
        float* merge = reinterpret_cast<float*>(smem_raw);  // [G - 1][PF_WARPS][PER_LANE][32]
        if (group > 0) {
            float* mine = merge + ((size_t)(group - 1) * PF_WARPS + warp) * PER_LANE * 32 + lane;
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) mine[(nt * 4 + e) * 32] = o[nt][e];
            mine[(NT * 4 + 0) * 32] = m_run[0];
            mine[(NT * 4 + 1) * 32] = m_run[1];
            mine[(NT * 4 + 2) * 32] = l_run[0];
            mine[(NT * 4 + 3) * 32] = l_run[1];
        }
        __syncthreads();
        if (group > 0) return;
        for (int g = 1; g < G; ++g) {
            const float* theirs = merge + ((size_t)(g - 1) * PF_WARPS + warp) * PER_LANE * 32 + lane;
            float f_mine[2], f_theirs[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float m_other = theirs[(NT * 4 + i) * 32], l_other = theirs[(NT * 4 + 2 + i) * 32];
                const float m_new = fmaxf(m_run[i], m_other);
                f_mine[i] = fast_exp2(m_run[i] - m_new);     // both maxima QF_NEG_BIG (nothing seen): 2^0, sums stay 0
                f_theirs[i] = fast_exp2(m_other - m_new);
                m_run[i] = m_new;
                l_run[i] = l_run[i] * f_mine[i] + l_other * f_theirs[i];
            }
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[nt][e] = o[nt][e] * f_mine[e >> 1] + theirs[(nt * 4 + e) * 32] * f_theirs[e >> 1];
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        if (!row_ok[i]) continue;
        float den = l_run[i], keep = 1.f;
        if (sinks) {  // the sink's term, in base-2 units like the scores, on a common maximum
            const float s2 = sinks[head] * 1.4426950408889634f, m_new = fmaxf(m_run[i], s2);
            keep = exp2f(m_run[i] - m_new);
            den = l_run[i] * keep + exp2f(s2 - m_new);
        }
        const float inv = den > 0.f ? keep / den : 0.f;
        bf16* dst = out + (size_t)(q_begin + row0 + r[i]) * q_width + (size_t)head * D + 2 * (lane & 3);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
            *reinterpret_cast<uint32_t*>(dst + 8 * nt) = pack_bf16(o[nt][2 * i] * inv, o[nt][2 * i + 1] * inv);
    }
}

template <int D, int G, bool POOLED, bool BIASED>
static int launch_groups(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots, KvSite<bf16> site,
                         int n_heads, int n_seqs, int max_q_len, float scale, int window, int* err, const float* sinks,
                         int shared_values, int mask_block, float softcap, KvSite<bf16> block_rows, int pool,
                         const float* bias_scale, const float* bias_rate, cudaStream_t stream) {
    size_t smem = (size_t)4 * G * QF_PAGE * (D + 8) * sizeof(bf16);
    const size_t merge = (size_t)(G - 1) * PF_WARPS * (D / 8 * 4 + 4) * 32 * sizeof(float);
    if (smem < merge) smem = merge;
    cudaError_t e = cudaFuncSetAttribute(prefill_flash_kernel<D, G, POOLED, BIASED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    const int n_tiles = (max_q_len + PF_BM - 1) / PF_BM;
    const long long blocks = (long long)n_tiles * n_heads * n_seqs;
    if (blocks > 0x7fffffffll) return (int)cudaErrorInvalidValue;
    return (int)launch_pdl(prefill_flash_kernel<D, G, POOLED, BIASED>, dim3((unsigned)blocks), dim3(PF_THREADS * G), smem, stream, (const bf16*)q,
                           (bf16*)out, cu_q, tok_pos, slots, site, n_heads, n_seqs, n_tiles, qf_sm_count(),
                           scale * 1.4426950408889634f, window, err, sinks, shared_values, mask_block,
                           softcap > 0.f ? scale / softcap : 0.f, softcap > 0.f ? softcap * 1.4426950408889634f : 0.f, block_rows, pool,
                           bias_scale, bias_rate);
}

template <int D>
static int launch(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots, void* base,
                  const int* table, long long page_elems, int table_stride, int kv_heads, int n_heads, int n_seqs,
                  int n_tokens, int max_q_len, int max_kv_len, float scale, int window, int* err, const float* sinks,
                  int shared_values, int mask_block, float softcap, void* blocks_base, const int* blocks_table,
                  long long blocks_page_elems, int blocks_table_stride, int pool, const float* bias_scale,
                  const float* bias_rate, cudaStream_t stream) {
    KvSite<bf16> site{(bf16*)base, table, page_elems, table_stride, kv_heads, D};
    KvSite<bf16> blocks{(bf16*)blocks_base, blocks_table, blocks_page_elems, blocks_table_stride, kv_heads, D};
    // Two groups of warps per tile when tiles walk many pages and all tiles find room on the SMs at once (a short
    // continuation over a long cache, one prompt of a few thousand tokens): what bounds the kernel then is the longest
    // tile's chain of pages, which two groups halve. With more tiles than room, the SMs are busy anyway and one group
    // per tile wastes nothing. Measured on one prompt of 2,048 tokens, 14 heads of 64 (448 tiles, room for 592): 55.5
    // microseconds with one group, 41.6 with two; 16 heads of 128 (512 tiles, room for 296): 73 against 94.
    // (tiles that hold rows: the grid also has blocks for the rows that shorter sequences lack, which end at once)
    const long long tiles = (long long)min((max_q_len + PF_BM - 1) / PF_BM * n_seqs, n_tokens / PF_BM + n_seqs) * n_heads;
    int span = window > 0 && window + PF_BM < max_kv_len ? window + PF_BM : max_kv_len;
    if (mask_block > 0 && mask_block < span) span = mask_block;   // no tile walks more than its rows' block of the mask
    if (pool > 0) span += max_kv_len / pool;                      // the rows of the blocks before the window
    const bool split = span >= 8 * QF_PAGE && tiles < (long long)qf_sm_count() * (D <= 64 ? 4 : 2);
#define QF_GROUPS_ARGS q, out, cu_q, tok_pos, slots, site, n_heads, n_seqs, max_q_len, scale, window, err, sinks, shared_values, mask_block, \
                       softcap, blocks, pool, bias_scale, bias_rate, stream
    if (pool > 0) return split ? launch_groups<D, 2, true, false>(QF_GROUPS_ARGS) : launch_groups<D, 1, true, false>(QF_GROUPS_ARGS);
    if (bias_scale) return split ? launch_groups<D, 2, false, true>(QF_GROUPS_ARGS) : launch_groups<D, 1, false, true>(QF_GROUPS_ARGS);
    return split ? launch_groups<D, 2, false, false>(QF_GROUPS_ARGS) : launch_groups<D, 1, false, false>(QF_GROUPS_ARGS);
#undef QF_GROUPS_ARGS
}

// The arguments of the generic attention kernel, `n_tokens` (the rows of q: all sequences' new tokens) and `max_kv_len`,
// an upper bound of any sequence's length after this step (both only steer how a tile's pages are shared among warps);
// bf16 only. cudaErrorInvalidValue for a head size without an
// instantiation (the caller then uses the generic kernel).
// mask_block > 0: a query sees only the keys of its own block of that many positions; softcap > 0: a score s (after the
// scale) becomes softcap * tanh(s / softcap), with the hardware's approximate tanh.
// pool > 0: the rows of whole blocks of `pool` positions, kept in a second cache of the same head shape (blocks_*), join
// the window's keys (see the top of the file).
// bias_scale, bias_rate: the distance bias, float32 [n_heads] each, both or neither (not with rows of whole blocks).
QF_EXPORT int qf_attention_prefill_biased(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots,
                                          void* base, const int* table, long long page_elems, int table_stride, int kv_heads,
                                          int head_dim, int n_heads, int n_seqs, int n_tokens, int max_q_len, int max_kv_len,
                                          float scale, int window, int* err, const float* sinks, int shared_values,
                                          int mask_block, float softcap, void* blocks_base, const int* blocks_table,
                                          long long blocks_page_elems, int blocks_table_stride, int pool, const float* bias_scale,
                                          const float* bias_rate, cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return 0;
    if (!bias_scale != !bias_rate || (pool > 0 && bias_scale)) return (int)cudaErrorInvalidValue;
    if (kv_heads <= 0 || n_heads % kv_heads) return (int)cudaErrorInvalidValue;
    if (pool > 0 && (!blocks_base || !blocks_table || window <= 0 || shared_values)) return (int)cudaErrorInvalidValue;
#define QF_CASE(DIM)                                                                                                 \
    case DIM:                                                                                                        \
        return launch<DIM>(q, out, cu_q, tok_pos, slots, base, table, page_elems, table_stride, kv_heads, n_heads,  \
                           n_seqs, n_tokens, max_q_len, max_kv_len, scale, window, err, sinks, shared_values, mask_block, softcap, \
                           blocks_base, blocks_table, blocks_page_elems, blocks_table_stride, pool, bias_scale, bias_rate, stream);
    switch (head_dim) {
        QF_CASE(32)
        QF_CASE(64)
        QF_CASE(96)
        QF_CASE(128)
        default:
            return (int)cudaErrorInvalidValue;
    }
#undef QF_CASE
}

QF_EXPORT int qf_attention_prefill_pooled(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots,
                                          void* base, const int* table, long long page_elems, int table_stride, int kv_heads,
                                          int head_dim, int n_heads, int n_seqs, int n_tokens, int max_q_len, int max_kv_len,
                                          float scale, int window, int* err, const float* sinks, int shared_values,
                                          int mask_block, float softcap, void* blocks_base, const int* blocks_table,
                                          long long blocks_page_elems, int blocks_table_stride, int pool, cudaStream_t stream) {
    return qf_attention_prefill_biased(q, out, cu_q, tok_pos, slots, base, table, page_elems, table_stride, kv_heads, head_dim,
                                       n_heads, n_seqs, n_tokens, max_q_len, max_kv_len, scale, window, err, sinks, shared_values,
                                       mask_block, softcap, blocks_base, blocks_table, blocks_page_elems, blocks_table_stride, pool,
                                       nullptr, nullptr, stream);
}

QF_EXPORT int qf_attention_prefill_masked(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots,
                                          void* base, const int* table, long long page_elems, int table_stride, int kv_heads,
                                          int head_dim, int n_heads, int n_seqs, int n_tokens, int max_q_len, int max_kv_len,
                                          float scale, int window, int* err, const float* sinks, int shared_values,
                                          int mask_block, float softcap, cudaStream_t stream) {
    return qf_attention_prefill_pooled(q, out, cu_q, tok_pos, slots, base, table, page_elems, table_stride, kv_heads, head_dim,
                                       n_heads, n_seqs, n_tokens, max_q_len, max_kv_len, scale, window, err, sinks, shared_values,
                                       mask_block, softcap, nullptr, nullptr, 0, 0, 0, stream);
}

QF_EXPORT int qf_attention_prefill_ex(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots,
                                      void* base, const int* table, long long page_elems, int table_stride, int kv_heads,
                                      int head_dim, int n_heads, int n_seqs, int n_tokens, int max_q_len, int max_kv_len,
                                      float scale, int window, int* err, const float* sinks, int shared_values,
                                      cudaStream_t stream) {
    return qf_attention_prefill_masked(q, out, cu_q, tok_pos, slots, base, table, page_elems, table_stride, kv_heads, head_dim,
                                       n_heads, n_seqs, n_tokens, max_q_len, max_kv_len, scale, window, err, sinks, shared_values,
                                       0, 0.f, stream);
}

QF_EXPORT int qf_attention_prefill(const void* q, void* out, const int* cu_q, const int* tok_pos, const int* slots,
                                   void* base, const int* table, long long page_elems, int table_stride, int kv_heads,
                                   int head_dim, int n_heads, int n_seqs, int n_tokens, int max_q_len, int max_kv_len,
                                   float scale, int window, int* err, cudaStream_t stream) {
    return qf_attention_prefill_ex(q, out, cu_q, tok_pos, slots, base, table, page_elems, table_stride, kv_heads, head_dim,
                                   n_heads, n_seqs, n_tokens, max_q_len, max_kv_len, scale, window, err, nullptr, 0, stream);
}
