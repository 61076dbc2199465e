// The gated delta rule with a decay per head and key channel: per head a float32 matrix S (dim x vdim), kept per sequence,
//
//   S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   y_t = S^T q_t
//
// with q, k unit vectors per head (q also times q_scale), g = exp(-exp(rate) softplus(z + b)), beta = sigmoid(logit). A head reads the
// q and k of head / (heads / groups). Everything from q, k, v (activation dtype) on is float32. A sequence whose slot is -1 (a
// padding entry) runs from a zero state and stores nothing.
//
// Steps of many tokens take two kernels. Token by token, every token's u would wait for a sum over the whole column of S
// before the next token's could begin. So four tokens go together: with S the state before the four, G_i = g_1 .. g_i and
// G_(i,j) = g_(j+1) .. g_i (products of numbers between 0 and 1, no quotients),
//
//   u_i = beta_i (v_i - S^T (G_i k_i) - sum_(j<i) c_ij u_j),   c_ij = k_i . G_(i,j) k_j
//   y_i = S^T (G_i q_i) + sum_(j<=i) d_ij u_j,                 d_ij = q_i . G_(i,j) k_j
//   S  <- diag(G_4) S + sum_j (G_(4,j) k_j) u_j^T
//
// which is the same recurrence, written out. `delta_prepare` works out all that does not depend on the state, a warp per
// (head, four tokens): the unit vectors, the decays and their products, c, d and beta, packed as one record. `delta_scan` walks
// every sequence's records in order. LANES lanes share EACH columns of S, the rows dealt out in fours; a lane's part of S stays in
// registers, two rows to a register pair and one instruction, from the sequence's first token of the step to its last. A
// column's eight sums (four for u, four for y) are formed together and reduced together, each lane ending up with one of them.
// What bounds the kernel is a warp's chain from one four to the next, so a lane has few rows (four or eight), and the rows of the
// next four are asked for before the sums of this one are; two columns per lane where S is tall, because a block is then
// bound by what it reads from shared memory. Records are staged through shared memory 16 or 32 tokens at a time by bulk copies, the next
// ones under way while these are worked on. Fours are counted from a sequence's first token of the step; the last one is
// filled up with tokens that do nothing (g = 1, k = q = 0).
//
// Steps of one token per sequence take one kernel, `delta_token`: a block per (sequence, head, up to 128 columns) that does all of
// it: unit vectors, decays, both products with the old state in one pass over S (y = (g S)^T q + (k . q) u), the update, and,
// if asked, the RMS norm per head, its weight and the sigmoid gate that follow.
#include "mma.cuh"

#define DELTA_LENGTH_EPS 1e-6f               // under the root of the unit vectors' length

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float channel_decay_of(float z, float rate_exp) { return expf(-rate_exp * softplus(z)); }

// Two float32 in one register pair, worked on by one instruction, each half rounded as by fmaf and __fmul_rn.
__device__ __forceinline__ unsigned long long pair_of(float lo, float hi) {
    unsigned long long p;
    asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(lo), "f"(hi));
    return p;
}
__device__ __forceinline__ float2 unpair(unsigned long long p) {
    float2 v;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(p));
    return v;
}
__device__ __forceinline__ float sum_of_pair(unsigned long long p) {
    const float2 v = unpair(p);
    return v.x + v.y;
}
__device__ __forceinline__ unsigned long long fma_pair(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ unsigned long long mul_pair(unsigned long long a, unsigned long long b) {
    unsigned long long d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// A record of four tokens: [Gk 4][Gq 4][Gk' 4][G] rows of `padded` floats (zeros beyond dim; the four in this order: G_i k_i, G_i q_i,
// G_(4,j) k_j and G_4), then c (8: c_21, c_31, c_32, c_41, c_42, c_43, two unused), d (16: row i, column j), beta (4), four unused.
#define DS_GROUP 4
#define DS_ROWS 13
#define DS_SCALARS 32
__host__ __device__ constexpr long long record_floats(int padded) { return (long long)DS_ROWS * padded + DS_SCALARS; }
// The record of a sequence's first four tokens of the step (records of sequences do not overlap: see ops.delta_scan).
__device__ __forceinline__ int first_record(int begin, int seq) { return begin / DS_GROUP + seq; }

template <typename T, int NI>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k, int k_stride, const float* __restrict__ z,
                     int z_stride, const float* __restrict__ bias, const float* __restrict__ rate_log, const float* __restrict__ logit,
                     int logit_stride, const int* __restrict__ cu_q, int n_records, int heads, int groups, int dim, float q_scale,
                     float* __restrict__ packed) {
    grid_chain_entry();
    constexpr int P = 32 * NI;
    const int lane = threadIdx.x & 31, item = blockIdx.x * 4 + (threadIdx.x >> 5), seq = blockIdx.y;
    const int head = item % heads, four = item / heads, group = head / (heads / groups);
    const int begin = cu_q[seq], len = cu_q[seq + 1] - begin, t0 = four * DS_GROUP;
    if (t0 >= len) return;
    float qv[4][NI], kv[4][NI], g[4][NI];
    const float rate = expf(rate_log[head]);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const bool there = t0 + j < len;
        const size_t t = begin + t0 + j;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = lane + 32 * i;
            const bool in = there && d < dim;
            qv[j][i] = in ? Num<T>::to_f(q[t * q_stride + group * dim + d]) : 0.f;
            kv[j][i] = in ? Num<T>::to_f(k[t * k_stride + group * dim + d]) : 0.f;
            g[j][i] = in ? z[t * z_stride + (size_t)head * dim + d] : 0.f;
        }
    }
    float raw_beta = 0.f;
    if (lane < 4 && t0 + lane < len) raw_beta = logit[(size_t)(begin + t0 + lane) * logit_stride + head];
    float b[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) b[i] = lane + 32 * i < dim ? bias[(size_t)head * dim + lane + 32 * i] : 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        float qs = 0.f, ks = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            qs = fmaf(qv[j][i], qv[j][i], qs);
            ks = fmaf(kv[j][i], kv[j][i], ks);
        }
        const float q_inv = q_scale / sqrtf(warp_sum(qs) + DELTA_LENGTH_EPS), k_inv = 1.f / sqrtf(warp_sum(ks) + DELTA_LENGTH_EPS);
        const bool there = t0 + j < len;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            qv[j][i] *= q_inv;
            kv[j][i] *= k_inv;
            g[j][i] = there ? channel_decay_of(g[j][i] + b[i], rate) : 1.f;
        }
    }
    float* rec = packed + ((size_t)head * n_records + first_record(begin, seq) + four) * record_floats(P);
    float sums[16];   // c and d, this lane's parts: d_jj, then for i > j c_ij and d_ij
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int d = lane + 32 * i;
        float run = 1.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            run *= g[j][i];
            rec[j * P + d] = run * kv[j][i];
            rec[(4 + j) * P + d] = run * qv[j][i];
        }
        rec[12 * P + d] = d < dim ? run : 0.f;
    }
    int at = 0;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        float w[NI], part = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            w[i] = kv[j][i];
            part = fmaf(qv[j][i], w[i], part);
        }
        sums[at++] = part;
#pragma unroll
        for (int m = j + 1; m < 4; ++m) {
            float pc = 0.f, pd = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                w[i] *= g[m][i];
                pc = fmaf(kv[m][i], w[i], pc);
                pd = fmaf(qv[m][i], w[i], pd);
            }
            sums[at++] = pc;
            sums[at++] = pd;
        }
#pragma unroll
        for (int i = 0; i < NI; ++i) rec[(8 + j) * P + lane + 32 * i] = w[i];
    }
    // sixteen sums over the warp, halving the sums with the lanes: lane l ends with sum l / 2
#pragma unroll
    for (int o = 16, n = 8; n > 0; o >>= 1, n >>= 1) {
        const bool upper = lane & o;
#pragma unroll
        for (int j = 0; j < n; ++j) {
            const float mine = upper ? sums[j + n] : sums[j], theirs = upper ? sums[j] : sums[j + n];
            sums[j] = mine + __shfl_xor_sync(0xffffffffu, theirs, o);
        }
    }
    const float total = sums[0] + __shfl_xor_sync(0xffffffffu, sums[0], 1);
    float* tail = rec + DS_ROWS * P;
    if (!(lane & 1)) {
        // order of the sums: d00 c10 d10 c20 d20 c30 d30 | d11 c21 d21 c31 d31 | d22 c32 d32 | d33
        constexpr signed char place[16] = {8 + 0, 0, 8 + 4, 1, 8 + 8, 3, 8 + 12, 8 + 5, 2, 8 + 9, 4, 8 + 13, 8 + 10, 5, 8 + 14, 8 + 15};
        int to = 0;
#pragma unroll
        for (int x = 0; x < 16; ++x) to = x == lane / 2 ? place[x] : to;
        tail[to] = total;
    } else if (lane < 12) {   // the upper triangle of d
        constexpr signed char zero[6] = {8 + 1, 8 + 2, 8 + 3, 8 + 6, 8 + 7, 8 + 11};
        int to = 0;
#pragma unroll
        for (int x = 0; x < 6; ++x) to = x == lane / 2 ? zero[x] : to;
        tail[to] = 0.f;
    }
    if (lane < 4) tail[24 + lane] = t0 + lane < len ? 1.f / (1.f + expf(-raw_beta)) : 0.f;
}

// A load that stays where it is written (see the scan of csrc/recurrent.cu).
__device__ __forceinline__ float load_value(const float* p) {
    float x;
    asm volatile("ld.global.nc.f32 %0, [%1];" : "=f"(x) : "l"(p));
    return x;
}
__device__ __forceinline__ float load_value(const bf16* p) {
    unsigned short raw;
    asm volatile("ld.global.nc.u16 %0, [%1];" : "=h"(raw) : "l"(p));
    return __uint_as_float((unsigned)raw << 16);
}

// R rows of S per lane (a multiple of 4), padded = LANES * R. Lane l of a column has rows 4 * (l + LANES * i) .. + 3. A warp has
// 32 / LANES * EACH columns, a block of WARPS warps COLS of them.
template <typename T, int LANES, int EACH, int R, int WARPS, int TOKENS>
__global__ void __launch_bounds__(WARPS * 32)
delta_scan_kernel(const float* __restrict__ packed, const T* __restrict__ v, int v_stride, const int* __restrict__ cu_q,
                  const int* __restrict__ slots, float* __restrict__ state, long long slot_stride, long long s_offset, int n_records,
                  int heads, int dim, int vdim, float* __restrict__ y, int* err) {
    constexpr int P = LANES * R, Q4 = R / 4, THREADS = WARPS * 32, FOURS = TOKENS / DS_GROUP, COLS = WARPS * 32 / LANES * EACH;
    constexpr int REC = (int)record_floats(P), SUMS = 8 * EACH;
    constexpr int SH = LANES / SUMS == 1 ? 0 : LANES / SUMS == 2 ? 1 : 2;   // after the reduction a lane has sum `part >> SH`
    static_assert(LANES % SUMS == 0 && LANES / SUMS <= 4, "a sum per lane");
    extern __shared__ __align__(16) float ds_smem[];
    float* rec_s = ds_smem;                                // [2][FOURS][REC]
    float* v_s = rec_s + 2 * FOURS * REC;                  // [2][TOKENS][COLS]
    float* y_s = v_s + 2 * TOKENS * COLS;                  // [2][TOKENS][COLS]
    __shared__ __align__(8) uint64_t arrived[2];           // a tile's records are complete
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.y, seq = blockIdx.z;
    const int part = lane & (LANES - 1), col_in = (warp * (32 / LANES) + lane / LANES) * EACH, col = blockIdx.x * COLS + col_in;
    const int begin = cu_q[seq], len = cu_q[seq + 1] - begin, slot = slots[seq];
    if (len <= 0) return;
    float* column = slot >= 0 ? state + slot * slot_stride + s_offset + (long long)head * dim * vdim + col : nullptr;
    unsigned long long s[EACH][R / 2];   // rows in pairs
#pragma unroll
    for (int c = 0; c < EACH; ++c)
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
            const int d = 4 * (part + LANES * (i / 2)) + 2 * (i % 2);
            const bool there = column && col + c < vdim;
            s[c][i] = pair_of(there && d < dim ? column[(size_t)d * vdim + c] : 0.f, there && d + 1 < dim ? column[(size_t)(d + 1) * vdim + c] : 0.f);
        }
    if (threadIdx.x == 0) {
        mbar_init(&arrived[0], 1);
        mbar_init(&arrived[1], 1);
    }
    __syncthreads();
    // a thread's values of a tile (and outputs): tokens token0, token0 + STEP, .. of column c_own
    constexpr int STEP = THREADS / COLS, EACH_THREAD = TOKENS / STEP;
    static_assert(THREADS % COLS == 0 && TOKENS % STEP == 0, "a tile's values in whole rounds");
    const int token0 = threadIdx.x / COLS, c_own = threadIdx.x % COLS;
    const bool column_there = blockIdx.x * COLS + c_own < vdim;
    const T* v_own = v + (size_t)(begin + token0) * v_stride + (size_t)head * vdim + blockIdx.x * COLS + c_own;
    float* y_own = y + (size_t)(begin + token0) * ((size_t)heads * vdim) + (size_t)head * vdim + blockIdx.x * COLS + c_own;
    const size_t v_step = (size_t)STEP * v_stride, y_step = (size_t)STEP * heads * vdim;
    float v_next[EACH_THREAD];
    const float* records = packed + ((size_t)head * n_records + first_record(begin, seq)) * REC;
    auto fetch = [&](int t0, int buf) {   // the records by one bulk copy to shared memory, the values through registers
        if (threadIdx.x == 0) {
            const uint32_t bytes = (uint32_t)(min(FOURS, (len - t0 + DS_GROUP - 1) / DS_GROUP) * REC * sizeof(float));
            mbar_expect_tx(&arrived[buf], bytes);
            bulk_copy_g2s(rec_s + buf * FOURS * REC, records + (size_t)(t0 / DS_GROUP) * REC, bytes, &arrived[buf]);
        }
        const T* from = v_own + (size_t)t0 * v_stride;
#pragma unroll
        for (int u = 0; u < EACH_THREAD; ++u) {
            v_next[u] = 0.f;
            if (column_there && t0 + token0 + u * STEP < len) v_next[u] = load_value(from + u * v_step);
        }
    };
    auto stash = [&](int buf) {
#pragma unroll
        for (int u = 0; u < EACH_THREAD; ++u) v_s[buf * TOKENS * COLS + threadIdx.x + u * THREADS] = v_next[u];
    };
    auto flush = [&](int t0, int buf) {   // a finished tile's outputs
        float* to = y_own + (size_t)t0 * heads * vdim;
#pragma unroll
        for (int u = 0; u < EACH_THREAD; ++u)
            if (column_there && t0 + token0 + u * STEP < len) to[u * y_step] = y_s[buf * TOKENS * COLS + threadIdx.x + u * THREADS];
    };
    fetch(0, 0);
    stash(0);
    int t_last = 0, buf_last = 0;
    for (int t0 = 0, turn = 0; t0 < len; t0 += TOKENS, ++turn) {
        const int buf = turn & 1, fours = min(FOURS, (len - t0 + DS_GROUP - 1) / DS_GROUP);
        // these records have arrived for everyone, and everyone is done with the tile before
        if (!__syncthreads_and(mbar_wait(&arrived[buf], (turn >> 1) & 1))) {
            mbar_wait(&arrived[buf], (turn >> 1) & 1);   // (bounded too: nothing of this block's may still be under way when it ends)
            if (threadIdx.x == 0) atomicOr(err, QF_ERR_COPY_TIMEOUT);
            return;
        }
        const bool more = t0 + TOKENS < len;
        if (more) fetch(t0 + TOKENS, buf ^ 1);
        if (turn > 0) flush(t0 - TOKENS, buf ^ 1);
        t_last = t0;
        buf_last = buf;
        const float* vs = v_s + buf * TOKENS * COLS + col_in;
        float* ys = y_s + buf * TOKENS * COLS + col_in;
        auto rows_of = [&](int f) { return reinterpret_cast<const ulonglong2*>(rec_s + (buf * FOURS + f) * REC) + part; };
        ulonglong2 ahead[8][Q4];   // the rows of the eight sums: row x, its quarter i
        {
            const ulonglong2* rows = rows_of(0);
#pragma unroll
            for (int x = 0; x < 8; ++x)
#pragma unroll
                for (int i = 0; i < Q4; ++i) ahead[x][i] = rows[x * (P / 4) + LANES * i];
        }
        for (int f = 0; f < fours; ++f) {
            const float* rec = rec_s + (buf * FOURS + f) * REC;
            const ulonglong2* rows = rows_of(f);
            float sums[SUMS];
#pragma unroll
            for (int x = 0; x < 8; ++x)
#pragma unroll
                for (int c = 0; c < EACH; ++c) {
                    unsigned long long acc = mul_pair(s[c][0], ahead[x][0].x);
                    acc = fma_pair(s[c][1], ahead[x][0].y, acc);
#pragma unroll
                    for (int i = 1; i < Q4; ++i) {
                        acc = fma_pair(s[c][2 * i], ahead[x][i].x, acc);
                        acc = fma_pair(s[c][2 * i + 1], ahead[x][i].y, acc);
                    }
                    sums[8 * c + x] = sum_of_pair(acc);
                }
            // what the second half needs, and the next four's rows, are on their way under the reduction
            ulonglong2 g[Q4], k[4][Q4];
#pragma unroll
            for (int i = 0; i < Q4; ++i) {
                g[i] = rows[12 * (P / 4) + LANES * i];
#pragma unroll
                for (int j = 0; j < 4; ++j) k[j][i] = rows[(8 + j) * (P / 4) + LANES * i];
            }
            const float4 c0 = *reinterpret_cast<const float4*>(rec + DS_ROWS * P), c1 = *reinterpret_cast<const float4*>(rec + DS_ROWS * P + 4);
            const float4 beta = *reinterpret_cast<const float4*>(rec + DS_ROWS * P + 24);
            const float4 d = *reinterpret_cast<const float4*>(rec + DS_ROWS * P + 8 + 4 * ((part >> SH) & 3));   // this lane's token's row
            float value[4][EACH];
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int c = 0; c < EACH; ++c) value[j][c] = vs[(4 * f + j) * COLS + c];
            {
                const ulonglong2* next = rows_of(f + 1 < fours ? f + 1 : f);
#pragma unroll
                for (int x = 0; x < 8; ++x)
#pragma unroll
                    for (int i = 0; i < Q4; ++i) ahead[x][i] = next[x * (P / 4) + LANES * i];
            }
            // the sums over the lanes, halving the sums with the lanes while there is more than one
#pragma unroll
            for (int o = LANES / 2, n = SUMS / 2; o > 0; o >>= 1, n >>= 1) {
                if (n > 0) {
                    const bool upper = part & o;
#pragma unroll
                    for (int j = 0; j < n; ++j) {
                        const float mine = upper ? sums[j + n] : sums[j], theirs = upper ? sums[j] : sums[j + n];
                        sums[j] = mine + __shfl_xor_sync(0xffffffffu, theirs, o);
                    }
                } else {
                    sums[0] += __shfl_xor_sync(0xffffffffu, sums[0], o);
                }
            }
            float u[EACH][4];
#pragma unroll
            for (int c = 0; c < EACH; ++c) {
                float left[4];   // v_i - S^T G_i k_i
#pragma unroll
                for (int j = 0; j < 4; ++j) left[j] = value[j][c] - __shfl_sync(0xffffffffu, sums[0], (8 * c + j) << SH, LANES);
                u[c][0] = beta.x * left[0];
                u[c][1] = beta.y * fmaf(-c0.x, u[c][0], left[1]);
                u[c][2] = beta.z * fmaf(-c0.z, u[c][1], fmaf(-c0.y, u[c][0], left[2]));
                u[c][3] = beta.w * fmaf(-c1.y, u[c][2], fmaf(-c1.x, u[c][1], fmaf(-c0.w, u[c][0], left[3])));
            }
#pragma unroll
            for (int c = 0; c < EACH; ++c)
#pragma unroll
                for (int i = 0; i < Q4; ++i) {
                    s[c][2 * i] = mul_pair(g[i].x, s[c][2 * i]);
                    s[c][2 * i + 1] = mul_pair(g[i].y, s[c][2 * i + 1]);
                }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int c = 0; c < EACH; ++c) {
                    const unsigned long long uu = pair_of(u[c][j], u[c][j]);
#pragma unroll
                    for (int i = 0; i < Q4; ++i) {
                        s[c][2 * i] = fma_pair(k[j][i].x, uu, s[c][2 * i]);
                        s[c][2 * i + 1] = fma_pair(k[j][i].y, uu, s[c][2 * i + 1]);
                    }
                }
            const int sum = part >> SH, mine = sum >> 3;   // mine: the column of this lane's sum
            float out = sums[0];
            const float dj[4] = {d.x, d.y, d.z, d.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) out = fmaf(dj[j], EACH > 1 && mine ? u[EACH - 1][j] : u[0][j], out);
            if ((sum & 4) && !(part & ((1 << SH) - 1))) ys[(4 * f + (sum & 3)) * COLS + mine] = out;
        }
        if (more) stash(buf ^ 1);
    }
    __syncthreads();
    flush(t_last, buf_last);
    if (column) {
#pragma unroll
        for (int c = 0; c < EACH; ++c)
#pragma unroll
            for (int i = 0; i < R / 2; ++i) {
                const int d = 4 * (part + LANES * (i / 2)) + 2 * (i % 2);
                const float2 both = unpair(s[c][i]);
                if (col + c < vdim && d < dim) column[(size_t)d * vdim + c] = both.x;
                if (col + c < vdim && d + 1 < dim) column[(size_t)(d + 1) * vdim + c] = both.y;
            }
    }
}

template <typename T, int LANES, int EACH, int R, int WARPS, int TOKENS>
static int launch_scan(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* z, int z_stride,
                       const float* bias, const float* rate_log, const float* logit, int logit_stride, const int* cu_q, const int* slots,
                       int n_seqs, int max_q_len, float* state, long long slot_stride, long long s_offset, int n_tokens, int heads, int groups,
                       int dim, int vdim, float q_scale, float* packed, float* y, int* err, cudaStream_t stream) {
    constexpr int COLS = WARPS * 32 / LANES * EACH;
    const int n_records = n_tokens / DS_GROUP + n_seqs;
    const long long items = (long long)((max_q_len + DS_GROUP - 1) / DS_GROUP) * heads;
    cudaError_t e = launch_pdl(delta_prepare_kernel<T, LANES * R / 32>, dim3((unsigned)((items + 3) / 4), n_seqs), dim3(128), 0, stream,
                               (const T*)q, q_stride, (const T*)k, k_stride, z, z_stride, bias, rate_log, logit, logit_stride, cu_q, n_records,
                               heads, groups, dim, q_scale, packed);
    if (e != cudaSuccess) return (int)e;
    const size_t smem = (size_t)2 * (TOKENS / DS_GROUP * record_floats(LANES * R) + 2 * TOKENS * COLS) * sizeof(float);
    e = cudaFuncSetAttribute(delta_scan_kernel<T, LANES, EACH, R, WARPS, TOKENS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    // launched the ordinary way: blocks that started under the first kernel's tail would crowd onto the SMs it leaves first,
    // and this kernel's few blocks are as fast as the SM they have to themselves
    delta_scan_kernel<T, LANES, EACH, R, WARPS, TOKENS><<<dim3((vdim + COLS - 1) / COLS, heads, n_seqs), dim3(WARPS * 32), smem, stream>>>(
        packed, (const T*)v, v_stride, cu_q, slots, state, slot_stride, s_offset, n_records, heads, dim, vdim, y, err);
    return (int)cudaGetLastError();
}

// Floats of a record of four tokens for a state of `dim` rows (0: not supported).
static int padded_dim(int dim) { return dim <= 0 || dim > 256 ? 0 : dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
QF_EXPORT int qf_delta_record(int dim) { return padded_dim(dim) ? (int)record_floats(padded_dim(dim)) : 0; }

// q, k: [T][groups * dim], v: [T][heads * vdim], activation dtype with row strides; z (the decays' pre-activations): float32
// [T][heads * dim], logit (beta's): float32 [T][heads], with row strides; bias float32 [heads * dim], rate_log float32 [heads];
// packed: scratch of heads * (n_tokens / 4 + n_seqs) records; y: float32 [T][heads * vdim]; S in the slots' rows at s_offset.
QF_EXPORT int qf_delta_scan(int is_bf16, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                            const float* z, int z_stride, const float* bias, const float* rate_log, const float* logit,
                            int logit_stride, const int* cu_q, const int* slots, int n_seqs, int max_q_len, float* state,
                            long long slot_stride, long long s_offset, int n_tokens, int heads, int groups, int dim, int vdim, float q_scale,
                            float* packed, float* y, int* err, cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (padded_dim(dim) == 0 || vdim <= 0 || groups <= 0 || heads % groups || n_seqs > 65535 || max_q_len <= 0 || heads > 65535 ||
        ((uintptr_t)packed & 15))
        return (int)cudaErrorInvalidValue;
#define QF_DELTA_SCAN(...) (is_bf16 ? launch_scan<bf16, __VA_ARGS__>(QF_DELTA_ARGS) : launch_scan<float, __VA_ARGS__>(QF_DELTA_ARGS))
#define QF_DELTA_ARGS q, q_stride, k, k_stride, v, v_stride, z, z_stride, bias, rate_log, logit, logit_stride, cu_q, slots, n_seqs, max_q_len, \
                      state, slot_stride, s_offset, n_tokens, heads, groups, dim, vdim, q_scale, packed, y, err, stream
    switch (padded_dim(dim)) {
        case 32: return QF_DELTA_SCAN(8, 1, 4, 4, 32);
        case 64: return QF_DELTA_SCAN(16, 1, 4, 2, 32);
        case 128: return QF_DELTA_SCAN(32, 2, 4, 4, 32);
        default: return QF_DELTA_SCAN(32, 2, 8, 8, 16);
    }
#undef QF_DELTA_ARGS
#undef QF_DELTA_SCAN
}

// ------------------------------------------------------------------------------------------------------------------
// One token per sequence. Sixteen warps: warp w has rows w, w + 16, ... of S, a lane the columns lane, lane + 32, ... of the
// block's (up to 32 * CJ). RI rows per warp stay in registers between the pass that reads S and the one that writes it.
#define DT_WARPS 16

template <typename T, int RI, int CJ>
__global__ void __launch_bounds__(DT_WARPS * 32)
delta_token_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k, int k_stride, const T* __restrict__ v, int v_stride,
                   const float* __restrict__ z, int z_stride, const float* __restrict__ bias, const float* __restrict__ rate_log,
                   const float* __restrict__ logit, int logit_stride, const int* __restrict__ cu_q, const int* __restrict__ slots,
                   float* __restrict__ state, long long slot_stride, long long s_offset, int heads, int groups, int dim, int vdim,
                   float q_scale, float* __restrict__ y, const T* __restrict__ norm, float eps, const T* __restrict__ gate,
                   int gate_stride, T* __restrict__ out) {
    grid_launch_dependents();
    constexpr int COLS = 32 * CJ;
    __shared__ float g_s[256], k_s[256], q_s[256], seen_s[DT_WARPS][COLS], read_s[DT_WARPS][COLS], scratch[33], sums_s[3];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.y, seq = blockIdx.z, group = head / (heads / groups);
    const int c0 = blockIdx.x * COLS;
    // weights come before the wait for the kernel before this one
    const float b = threadIdx.x < dim ? bias[(size_t)head * dim + threadIdx.x] : 0.f, rate = expf(rate_log[head]);
    grid_dependency_wait();
    const int slot = slots[seq], t = cu_q[seq];
    if (cu_q[seq + 1] <= t) return;
    float* S = slot >= 0 ? state + slot * slot_stride + s_offset + (long long)head * dim * vdim + c0 : nullptr;
    float s[RI][CJ];
#pragma unroll
    for (int i = 0; i < RI; ++i)
#pragma unroll
        for (int j = 0; j < CJ; ++j) {
            const int d = warp + DT_WARPS * i, c = lane + 32 * j;
            s[i][j] = (S && d < dim && c0 + c < vdim) ? S[(size_t)d * vdim + c] : 0.f;
        }
    if (threadIdx.x < 256) {
        const int d = threadIdx.x;
        q_s[d] = d < dim ? Num<T>::to_f(q[(size_t)t * q_stride + group * dim + d]) : 0.f;
        k_s[d] = d < dim ? Num<T>::to_f(k[(size_t)t * k_stride + group * dim + d]) : 0.f;
        g_s[d] = d < dim ? channel_decay_of(z[(size_t)t * z_stride + (size_t)head * dim + d] + b, rate) : 0.f;
    }
    __syncthreads();
    if (warp < 3) {   // q . q, k . k and k . q, a warp each
        const float* left = warp == 0 ? q_s : k_s;
        const float* right = warp == 1 ? k_s : q_s;
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) sum = fmaf(left[lane + 32 * i], right[lane + 32 * i], sum);
        sum = warp_sum(sum);
        if (lane == 0) sums_s[warp] = sum;
    }
    float seen[CJ], read[CJ];
#pragma unroll
    for (int j = 0; j < CJ; ++j) seen[j] = read[j] = 0.f;
    __syncthreads();
    const float q_inv = q_scale / sqrtf(sums_s[0] + DELTA_LENGTH_EPS), k_inv = 1.f / sqrtf(sums_s[1] + DELTA_LENGTH_EPS);
    const float kq = sums_s[2] * k_inv * q_inv;
#pragma unroll
    for (int i = 0; i < RI; ++i) {
        const int d = warp + DT_WARPS * i;
        if (d >= dim) break;
        const float gd = g_s[d], kd = k_s[d] * k_inv, qd = q_s[d] * q_inv;
#pragma unroll
        for (int j = 0; j < CJ; ++j) {
            s[i][j] *= gd;
            seen[j] = fmaf(s[i][j], kd, seen[j]);
            read[j] = fmaf(s[i][j], qd, read[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < CJ; ++j) {
        seen_s[warp][lane + 32 * j] = seen[j];
        read_s[warp][lane + 32 * j] = read[j];
    }
    __syncthreads();
    float* u_s = g_s;   // (the decays are used up once every warp has passed the barrier)
    float value = 0.f;
    if (threadIdx.x < COLS) {
        const int c = c0 + threadIdx.x;
        float total = 0.f, old = 0.f;
#pragma unroll
        for (int w = 0; w < DT_WARPS; ++w) {
            total += seen_s[w][threadIdx.x];
            old += read_s[w][threadIdx.x];
        }
        float u = 0.f;
        if (c < vdim) {
            const float beta = 1.f / (1.f + expf(-logit[(size_t)t * logit_stride + head]));
            u = beta * (Num<T>::to_f(v[(size_t)t * v_stride + (size_t)head * vdim + c]) - total);
            value = fmaf(kq, u, old);
            if (y) y[(size_t)t * ((size_t)heads * vdim) + (size_t)head * vdim + c] = value;
        }
        u_s[threadIdx.x] = u;
    }
    __syncthreads();
    if (S) {
#pragma unroll
        for (int i = 0; i < RI; ++i) {
            const int d = warp + DT_WARPS * i;
            if (d >= dim) break;
            const float kd = k_s[d] * k_inv;
#pragma unroll
            for (int j = 0; j < CJ; ++j) {
                const int c = lane + 32 * j;
                if (c0 + c < vdim) S[(size_t)d * vdim + c] = fmaf(kd, u_s[c], s[i][j]);
            }
        }
    }
    if (out) {   // the whole head is in this block (vdim <= COLS): its norm, the weight and the gate
        const float inv = rsqrtf(block_sum(value * value, scratch) / (float)vdim + eps);
        if (threadIdx.x < vdim) {
            const size_t at = (size_t)head * vdim + threadIdx.x;
            const float raw = Num<T>::to_f(gate[(size_t)t * gate_stride + at]);
            out[(size_t)t * ((size_t)heads * vdim) + at] = Num<T>::from_f(value * inv * Num<T>::to_f(norm[threadIdx.x]) / (1.f + expf(-raw)));
        }
    }
}

template <typename T, int RI, int CJ>
static int launch_token(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* z, int z_stride,
                        const float* bias, const float* rate_log, const float* logit, int logit_stride, const int* cu_q, const int* slots,
                        int n_seqs, float* state, long long slot_stride, long long s_offset, int heads, int groups, int dim, int vdim,
                        float q_scale, float* y, const void* norm, float eps, const void* gate, int gate_stride, void* out,
                        cudaStream_t stream) {
    return (int)launch_pdl(delta_token_kernel<T, RI, CJ>, dim3((vdim + 32 * CJ - 1) / (32 * CJ), heads, n_seqs), dim3(DT_WARPS * 32), 0, stream,
                           (const T*)q, q_stride, (const T*)k, k_stride, (const T*)v, v_stride, z, z_stride, bias, rate_log, logit,
                           logit_stride, cu_q, slots, state, slot_stride, s_offset, heads, groups, dim, vdim, q_scale, y, (const T*)norm, eps,
                           (const T*)gate, gate_stride, (T*)out);
}

template <typename T, int RI>
static int token_columns(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* z, int z_stride,
                         const float* bias, const float* rate_log, const float* logit, int logit_stride, const int* cu_q, const int* slots,
                         int n_seqs, float* state, long long slot_stride, long long s_offset, int heads, int groups, int dim, int vdim,
                         float q_scale, float* y, const void* norm, float eps, const void* gate, int gate_stride, void* out,
                         cudaStream_t stream) {
#define QF_TOKEN_ARGS q, q_stride, k, k_stride, v, v_stride, z, z_stride, bias, rate_log, logit, logit_stride, cu_q, slots, n_seqs, state, \
                      slot_stride, s_offset, heads, groups, dim, vdim, q_scale, y, norm, eps, gate, gate_stride, out, stream
    if (vdim <= 32) return launch_token<T, RI, 1>(QF_TOKEN_ARGS);
    if (vdim <= 64) return launch_token<T, RI, 2>(QF_TOKEN_ARGS);
    return launch_token<T, RI, 4>(QF_TOKEN_ARGS);
}

// The same for a step of ONE token per sequence. y (float32, as above) or, for vdim <= 128, out [T][heads * vdim] in the activation
// dtype: y / rms(y) per head (eps inside the root) * norm [vdim] * sigmoid(gate [T][heads * vdim], row stride). Either may be null.
QF_EXPORT int qf_delta_token(int is_bf16, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                             const float* z, int z_stride, const float* bias, const float* rate_log, const float* logit,
                             int logit_stride, const int* cu_q, const int* slots, int n_seqs, float* state, long long slot_stride,
                             long long s_offset, int heads, int groups, int dim, int vdim, float q_scale, float* y, const void* norm,
                             float eps, const void* gate, int gate_stride, void* out, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (padded_dim(dim) == 0 || vdim <= 0 || groups <= 0 || heads % groups || n_seqs > 65535 || (out && (vdim > 128 || !norm || !gate)))
        return (int)cudaErrorInvalidValue;
    if (dim <= 64) return is_bf16 ? token_columns<bf16, 4>(QF_TOKEN_ARGS) : token_columns<float, 4>(QF_TOKEN_ARGS);
    if (dim <= 128) return is_bf16 ? token_columns<bf16, 8>(QF_TOKEN_ARGS) : token_columns<float, 8>(QF_TOKEN_ARGS);
    return is_bf16 ? token_columns<bf16, 16>(QF_TOKEN_ARGS) : token_columns<float, 16>(QF_TOKEN_ARGS);
#undef QF_TOKEN_ARGS
}
