// The gated delta rule with a decay per head and key channel: per head a float32 matrix S (dim x vdim), kept per sequence,
//
//   S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   y_t = S^T q_t
//
// with q, k unit vectors per head (q also times q_scale), g = exp(-exp(rate) softplus(z + b)), beta = sigmoid(logit). A head reads the
// q and k of head / (heads / groups). Everything from q, k, v (activation dtype) on is float32. A sequence whose slot is -1 (a
// padding entry) runs from a zero state and stores nothing.
//
// Steps of many tokens take two kernels. `delta_prepare` works out, a warp per (token, head), what does not depend on the state:
// the unit vectors, the decays and beta, packed for the scan as rows [g | k | q] of `padded` floats each. `delta_scan` then walks
// every sequence's tokens in order. Eight lanes share a column of S, the rows dealt out in fours, so a warp has four columns
// and a block of four warps sixteen; a lane's part of S stays in registers from the sequence's first token of the step to its
// last. A token costs a lane four multiply-adds per row of its part (decay, S^T k, update, S^T q) and three shuffles
// whose latency the chain waits for (u_t needs the whole column's S^T k); the shuffles of S^T q are put off and shared by
// eight tokens, one lane ending up with one token's sum. Tokens are staged through shared memory DS_TOKENS at a time by
// asynchronous copies, the next tile under way while one is worked on. The order of operations per token does not depend on
// the cut of the sequence.
//
// Steps of one token per sequence take one kernel, `delta_token`: a block per (sequence, head, up to 128 columns) that does all of
// it: unit vectors, decays, both products with the old state in one pass over S (y = (g S)^T q + (k . q) u), the update, and,
// if asked, the RMS norm per head, its weight and the sigmoid gate that follow.
#include "mma.cuh"

#define DS_LANES 8
#define DS_WARPS 4
#define DS_COLS (DS_WARPS * 32 / DS_LANES)   // columns of S per block
#define DELTA_LENGTH_EPS 1e-6f               // under the root of the unit vectors' length

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float channel_decay_of(float z, float rate_exp) { return expf(-rate_exp * softplus(z)); }

// packed: [heads][n_tokens][3][padded] (g, k, q; zeros beyond dim); beta: [heads][n_tokens]
template <typename T>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k, int k_stride, const float* __restrict__ z,
                     int z_stride, const float* __restrict__ bias, const float* __restrict__ rate_log, const float* __restrict__ logit,
                     int logit_stride, int n_tokens, int heads, int groups, int dim, int padded, float q_scale,
                     float* __restrict__ packed, float* __restrict__ beta) {
    grid_chain_entry();
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= (long long)n_tokens * heads) return;
    const int lane = threadIdx.x & 31, t = (int)(item / heads), head = (int)(item % heads), group = head / (heads / groups);
    const T* qt = q + (size_t)t * q_stride + group * dim;
    const T* kt = k + (size_t)t * k_stride + group * dim;
    const float* zt = z + (size_t)t * z_stride + (size_t)head * dim;
    float qv[8], kv[8], zv[8], qs = 0.f, ks = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {   // dim <= 256
        const int d = lane + 32 * i;
        qv[i] = d < dim ? Num<T>::to_f(qt[d]) : 0.f;
        kv[i] = d < dim ? Num<T>::to_f(kt[d]) : 0.f;
        zv[i] = d < dim ? zt[d] + bias[(size_t)head * dim + d] : 0.f;
        qs = fmaf(qv[i], qv[i], qs);
        ks = fmaf(kv[i], kv[i], ks);
    }
    const float q_inv = q_scale / sqrtf(warp_sum(qs) + DELTA_LENGTH_EPS), k_inv = 1.f / sqrtf(warp_sum(ks) + DELTA_LENGTH_EPS);
    const float rate = expf(rate_log[head]);
    float* row = packed + ((size_t)head * n_tokens + t) * 3 * padded;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = lane + 32 * i;
        if (d >= padded) break;
        row[d] = d < dim ? channel_decay_of(zv[i], rate) : 0.f;
        row[padded + d] = kv[i] * k_inv;
        row[2 * padded + d] = qv[i] * q_inv;
    }
    if (lane == 0) beta[(size_t)head * n_tokens + t] = 1.f / (1.f + expf(-logit[(size_t)t * logit_stride + head]));
}

// R rows of S per lane (a multiple of 4): padded = 8 * R. Lane l of a column has rows 4 * (l + 8 * i) .. + 3.
template <typename T, int R, int TOKENS>
__global__ void __launch_bounds__(DS_WARPS * 32)
delta_scan_kernel(const float* __restrict__ packed, const float* __restrict__ beta, const T* __restrict__ v, int v_stride,
                  const int* __restrict__ cu_q, const int* __restrict__ slots, float* __restrict__ state, long long slot_stride,
                  long long s_offset, int n_tokens, int heads, int dim, int vdim, float* __restrict__ y) {
    grid_chain_entry();
    constexpr int P = DS_LANES * R, ROW = 3 * P, Q4 = R / 4, THREADS = DS_WARPS * 32;
    extern __shared__ __align__(16) float ds_smem[];
    float* rows_s = ds_smem;                               // [2][TOKENS][ROW]
    float* v_s = rows_s + 2 * TOKENS * ROW;                // [2][TOKENS][DS_COLS]
    float* beta_s = v_s + 2 * TOKENS * DS_COLS;            // [2][TOKENS]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.y, seq = blockIdx.z;
    const int part = lane & (DS_LANES - 1), col_in = warp * (32 / DS_LANES) + lane / DS_LANES, col = blockIdx.x * DS_COLS + col_in;
    const int begin = cu_q[seq], end = cu_q[seq + 1], slot = slots[seq];
    if (begin >= end) return;
    float* column = (slot >= 0 && col < vdim) ? state + slot * slot_stride + s_offset + (long long)head * dim * vdim + col : nullptr;
    float s[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = 4 * (part + DS_LANES * (i / 4)) + i % 4;
        s[i] = (column && d < dim) ? column[(size_t)d * vdim] : 0.f;
    }
    constexpr int V_EACH = (TOKENS * DS_COLS + THREADS - 1) / THREADS;
    float v_next[V_EACH], beta_next = 0.f;
    // a tile's rows go straight to shared memory; its values and betas pass through registers
    auto fetch = [&](int t0, int buf) {
        const int n_here = min(TOKENS, end - t0);
        const float* from = packed + ((size_t)head * n_tokens + t0) * ROW;
        float* to = rows_s + buf * TOKENS * ROW;
        for (int i = threadIdx.x; i < n_here * (ROW / 4); i += THREADS) cp_async_16(to + 4 * i, from + 4 * i, true);
        cp_async_commit();
#pragma unroll
        for (int u = 0; u < V_EACH; ++u) {
            const int i = threadIdx.x + u * THREADS, j = i / DS_COLS, c = blockIdx.x * DS_COLS + i % DS_COLS;
            v_next[u] = (j < n_here && c < vdim) ? Num<T>::to_f(v[(size_t)(t0 + j) * v_stride + (size_t)head * vdim + c]) : 0.f;
        }
        if (threadIdx.x < n_here) beta_next = beta[(size_t)head * n_tokens + t0 + threadIdx.x];
    };
    auto stash = [&](int buf) {
#pragma unroll
        for (int u = 0; u < V_EACH; ++u) {
            const int i = threadIdx.x + u * THREADS;
            if (i < TOKENS * DS_COLS) v_s[buf * TOKENS * DS_COLS + i] = v_next[u];
        }
        if (threadIdx.x < TOKENS) beta_s[buf * TOKENS + threadIdx.x] = beta_next;
    };
    fetch(begin, 0);
    stash(0);
    for (int t0 = begin, turn = 0; t0 < end; t0 += TOKENS, ++turn) {
        const int buf = turn & 1, n_here = min(TOKENS, end - t0);
        cp_async_wait<0>();
        __syncthreads();   // this tile has arrived for everyone, and everyone is done with the other buffer
        const bool more = t0 + TOKENS < end;
        if (more) fetch(t0 + TOKENS, buf ^ 1);
        const float* rows = rows_s + buf * TOKENS * ROW;
        const float* vs = v_s + buf * TOKENS * DS_COLS + col_in;
        const float* bs = beta_s + buf * TOKENS;
        auto token = [&](int j) -> float {   // this lane's part of y
            const float4* g4 = reinterpret_cast<const float4*>(rows + j * ROW) + part;
            const float4* k4 = reinterpret_cast<const float4*>(rows + j * ROW + P) + part;
            const float4* q4 = reinterpret_cast<const float4*>(rows + j * ROW + 2 * P) + part;
            float k[R], a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < Q4; ++i) {
                const float4 gg = g4[DS_LANES * i], kk = k4[DS_LANES * i];
                const float ge[4] = {gg.x, gg.y, gg.z, gg.w}, ke[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    k[4 * i + e] = ke[e];
                    s[4 * i + e] *= ge[e];
                    a[e] = fmaf(s[4 * i + e], ke[e], a[e]);
                }
            }
            float seen = (a[0] + a[1]) + (a[2] + a[3]);
#pragma unroll
            for (int o = 1; o < DS_LANES; o <<= 1) seen += __shfl_xor_sync(0xffffffffu, seen, o);
            const float u = bs[j] * (vs[j * DS_COLS] - seen);
            float b[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < Q4; ++i) {
                const float4 qq = q4[DS_LANES * i];
                const float qe[4] = {qq.x, qq.y, qq.z, qq.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s[4 * i + e] = fmaf(k[4 * i + e], u, s[4 * i + e]);
                    b[e] = fmaf(s[4 * i + e], qe[e], b[e]);
                }
            }
            return (b[0] + b[1]) + (b[2] + b[3]);
        };
        for (int j0 = 0; j0 < n_here; j0 += DS_LANES) {
            float y8[DS_LANES];
            if (j0 + DS_LANES <= n_here) {
#pragma unroll
                for (int j = 0; j < DS_LANES; ++j) y8[j] = token(j0 + j);
            } else {
#pragma unroll
                for (int j = 0; j < DS_LANES; ++j) y8[j] = j0 + j < n_here ? token(j0 + j) : 0.f;
            }
            // eight sums over eight lanes, halving: lane `part` ends with token j0 + part's
#pragma unroll
            for (int o = DS_LANES / 2; o > 0; o >>= 1) {
                const bool upper = part & o;
#pragma unroll
                for (int j = 0; j < o; ++j) {
                    const float mine = upper ? y8[j + o] : y8[j], theirs = upper ? y8[j] : y8[j + o];
                    y8[j] = mine + __shfl_xor_sync(0xffffffffu, theirs, o);
                }
            }
            if (j0 + part < n_here && col < vdim) y[(size_t)(t0 + j0 + part) * ((size_t)heads * vdim) + (size_t)head * vdim + col] = y8[0];
        }
        if (more) stash(buf ^ 1);
    }
    if (column) {
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int d = 4 * (part + DS_LANES * (i / 4)) + i % 4;
            if (d < dim) column[(size_t)d * vdim] = s[i];
        }
    }
}

template <typename T, int R, int TOKENS>
static int launch_scan(const float* packed, const float* beta, const void* v, int v_stride, const int* cu_q, const int* slots, int n_seqs,
                       float* state, long long slot_stride, long long s_offset, int n_tokens, int heads, int dim, int vdim, float* y,
                       cudaStream_t stream) {
    const size_t smem = (size_t)2 * TOKENS * (3 * DS_LANES * R + DS_COLS + 1) * sizeof(float);
    cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<T, R, TOKENS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    return (int)launch_pdl(delta_scan_kernel<T, R, TOKENS>, dim3((vdim + DS_COLS - 1) / DS_COLS, heads, n_seqs), dim3(DS_WARPS * 32), smem,
                           stream, packed, beta, (const T*)v, v_stride, cu_q, slots, state, slot_stride, s_offset, n_tokens, heads, dim, vdim, y);
}

// Floats per row of the packed form for a state of `dim` rows (0: not supported).
QF_EXPORT int qf_delta_padded(int dim) { return dim <= 0 || dim > 256 ? 0 : dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

// q, k: [T][groups * dim], v: [T][heads * vdim], activation dtype with row strides; z (the decays' pre-activations): float32
// [T][heads * dim], logit (beta's): float32 [T][heads], with row strides; bias float32 [heads * dim], rate_log float32 [heads];
// packed: float32 [heads][T][3][padded] and beta [heads][T], scratch; y: float32 [T][heads * vdim]; S in the slots' rows at s_offset.
QF_EXPORT int qf_delta_scan(int is_bf16, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                            const float* z, int z_stride, const float* bias, const float* rate_log, const float* logit,
                            int logit_stride, const int* cu_q, const int* slots, int n_seqs, float* state, long long slot_stride,
                            long long s_offset, int n_tokens, int heads, int groups, int dim, int vdim, float q_scale, float* packed,
                            float* beta, float* y, cudaStream_t stream) {
    const int padded = qf_delta_padded(dim);
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (padded == 0 || vdim <= 0 || groups <= 0 || heads % groups || n_seqs > 65535) return (int)cudaErrorInvalidValue;
    const unsigned blocks = (unsigned)(((long long)n_tokens * heads + 7) / 8);
    cudaError_t e;
    if (is_bf16)
        e = launch_pdl(delta_prepare_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16*)q, q_stride, (const bf16*)k, k_stride, z,
                       z_stride, bias, rate_log, logit, logit_stride, n_tokens, heads, groups, dim, padded, q_scale, packed, beta);
    else
        e = launch_pdl(delta_prepare_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)q, q_stride, (const float*)k, k_stride,
                       z, z_stride, bias, rate_log, logit, logit_stride, n_tokens, heads, groups, dim, padded, q_scale, packed, beta);
    if (e != cudaSuccess) return (int)e;
#define QF_DELTA_SCAN(R, TOKENS) (is_bf16 ? launch_scan<bf16, R, TOKENS>(QF_DELTA_ARGS) : launch_scan<float, R, TOKENS>(QF_DELTA_ARGS))
#define QF_DELTA_ARGS packed, beta, v, v_stride, cu_q, slots, n_seqs, state, slot_stride, s_offset, n_tokens, heads, dim, vdim, y, stream
    if (padded == 32) return QF_DELTA_SCAN(4, 32);
    if (padded == 64) return QF_DELTA_SCAN(8, 32);
    if (padded == 128) return QF_DELTA_SCAN(16, 32);
    return QF_DELTA_SCAN(32, 16);
#undef QF_DELTA_ARGS
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
    if (qf_delta_padded(dim) == 0 || vdim <= 0 || groups <= 0 || heads % groups || n_seqs > 65535 || (out && (vdim > 128 || !norm || !gate)))
        return (int)cudaErrorInvalidValue;
    if (dim <= 64) return is_bf16 ? token_columns<bf16, 4>(QF_TOKEN_ARGS) : token_columns<float, 4>(QF_TOKEN_ARGS);
    if (dim <= 128) return is_bf16 ? token_columns<bf16, 8>(QF_TOKEN_ARGS) : token_columns<float, 8>(QF_TOKEN_ARGS);
    return is_bf16 ? token_columns<bf16, 16>(QF_TOKEN_ARGS) : token_columns<float, 16>(QF_TOKEN_ARGS);
#undef QF_TOKEN_ARGS
}
