// Retention: linear attention with a fixed decay per head, without a softmax or a denominator.
//
//   S <- decay_h S + k_t v_t^T,   o_t = S^T q_t      per head; S is dim x vdim, float32, kept per sequence
//   out_t = o_t / sqrt(mean(o_t^2) + eps) * silu(gate_t)     per head (the norm over the head's vdim components)
//
// with q and k turned by their token's position (split halves, the first rot_dim components) and k times k_scale on the way in.
// The projections q, k, v and the gate carry the activation dtype; the rotation, k_scale, the powers of the decay, every product,
// S and the norm are float32. `angles` [tokens][rot_dim / 2] holds (cos, sin) of the step's tokens, made once per step.
//
// A step of one token per sequence is one kernel: a block per sequence and head moves S once in and once out.
//
// Longer steps are cut into chunks of RT_CHUNK tokens, counted from a sequence's first token of the step, and the recurrence is
// written out over a chunk (i, j: tokens of the chunk from 0, n of them, S0 the state before it):
//   o_i = decay^(i+1) S0^T q_i + sum_{j <= i} decay^(i-j) (q_i . k_j) v_j
//   S_n = decay^n S0 + sum_j decay^(n-1-j) k_j v_j^T
// in three launches: (1) every chunk's own part of S_n, all chunks at once; (2) the states before every chunk, a short chain of
// one multiply-add per chunk and element of S; (3) every chunk's outputs, norm and gate, all chunks at once. No power of the decay
// exceeds 1, so nothing has to be rescaled. The products run on the tensor cores as tf32 with float32 sums, every float32 operand
// taken as the sum of two tf32 numbers (x = hi + lo to about 2^-21; hi hi + hi lo + lo hi), so they are float32 products to
// rounding; the values are bfloat16 numbers and need one.
#include <type_traits>

#include "mma.cuh"

#define RT_CHUNK 64
#define RT_THREADS 256
#define RT_MAX_DIM 128
#define RT_MAX_VDIM 128

struct Split {
    uint32_t hi, lo;
};
// The leading eleven bits of x's significand, and the next eleven (both by cutting off: two logical operations and a subtraction).
__device__ __forceinline__ Split split_tf32(float x) {
    Split s;
    s.hi = __float_as_uint(x) & 0xffffe000u;
    s.lo = __float_as_uint(x - __uint_as_float(s.hi)) & 0xffffe000u;
    return s;
}
// D[16x8] += A[16x8] * B[8x8], tf32 operands, float32 accumulation.
__device__ __forceinline__ void mma_tf32(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// float32 x float32, both split; the small products first
__device__ __forceinline__ void mma_split(float (&d)[4], const Split (&a)[4], Split b0, Split b1) {
    mma_tf32(d, a[0].lo, a[1].lo, a[2].lo, a[3].lo, b0.hi, b1.hi);
    mma_tf32(d, a[0].hi, a[1].hi, a[2].hi, a[3].hi, b0.lo, b1.lo);
    mma_tf32(d, a[0].hi, a[1].hi, a[2].hi, a[3].hi, b0.hi, b1.hi);
}
// float32 x numbers that are tf32 as they stand (bfloat16 values)
__device__ __forceinline__ void mma_half_split(float (&d)[4], const Split (&a)[4], float b0, float b1) {
    const uint32_t x0 = __float_as_uint(b0), x1 = __float_as_uint(b1);
    mma_tf32(d, a[0].lo, a[1].lo, a[2].lo, a[3].lo, x0, x1);
    mma_tf32(d, a[0].hi, a[1].hi, a[2].hi, a[3].hi, x0, x1);
}

__device__ __forceinline__ void load8(const bf16* p, float (&v)[8]) {   // (through the read-only path: may run ahead of stores)
    const uint4 raw = __ldg(reinterpret_cast<const uint4*>(p));
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h[e]);
        v[2 * e] = f.x;
        v[2 * e + 1] = f.y;
    }
}
__device__ __forceinline__ void put8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

// Rows t0 .. t0 + n - 1 of q or k of one head, turned, times `scale` (and times row_power[n - 1 - row] where given), to
// dst[row][0 .. padded), zeros in rows from n to RT_CHUNK and in columns from dim to padded. Sizes in whole eights.
__device__ __forceinline__ void stage_turned(float* dst, int stride, int padded, const bf16* src, int src_stride, int n, int dim, int rot_dim,
                                             const float2* angles, float scale, const float* row_power) {
    const int half = rot_dim / 2, per_row = padded / 8;
#pragma unroll 2
    for (int i = threadIdx.x; i < RT_CHUNK * per_row; i += RT_THREADS) {
        const int row = i / per_row, c = (i % per_row) * 8;
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
        if (row < n && c < dim) {
            const bf16* p = src + (size_t)row * src_stride;
            load8(p + c, v);
            if (c < rot_dim) {
                const bool first = c < half;
                const int j = first ? c : c - half;
                float other[8];
                load8(p + (first ? c + half : c - half), other);
                const float4* cs = reinterpret_cast<const float4*>(angles + (size_t)row * half + j);   // two pairs (cos, sin) each
                const float sign = first ? -1.f : 1.f;
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float4 a = __ldg(cs + e);
                    v[2 * e] = fmaf(sign * other[2 * e], a.y, v[2 * e] * a.x);
                    v[2 * e + 1] = fmaf(sign * other[2 * e + 1], a.w, v[2 * e + 1] * a.z);
                }
            }
            const float f = row_power ? scale * row_power[n - 1 - row] : scale;
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] *= f;
        }
        put8(dst + (size_t)row * stride + c, v);
    }
}
__device__ __forceinline__ void stage_values(float* dst, int stride, const bf16* src, int src_stride, int n, int vdim) {
    const int per_row = vdim / 8;
#pragma unroll 4
    for (int i = threadIdx.x; i < RT_CHUNK * per_row; i += RT_THREADS) {
        const int row = i / per_row, c = (i % per_row) * 8;
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
        if (row < n) load8(src + (size_t)row * src_stride + c, v);
        put8(dst + (size_t)row * stride + c, v);
    }
}

// Row strides of the staged tiles, in floats: 4 or 8 modulo 32, so that the eight rows or four rows that a fragment load touches
// lie in banks of their own.
__host__ __device__ inline int rt_padded(int dim) { return (dim + 15) / 16 * 16; }
__host__ __device__ inline int rt_stride(int width, int rest) { return (width + 31 - rest) / 32 * 32 + rest; }

// The first chunk record of a sequence: sequence s owns records cu_q[s] / RT_CHUNK + s onwards, as many as its chunks at most.
__device__ __forceinline__ long long rt_record(const int* cu_q, int seq, int chunk, int n_heads, int head) {
    return ((long long)(cu_q[seq] / RT_CHUNK + seq + chunk)) * n_heads + head;
}

// (1) A chunk's own part of the state after it: sum_j decay^(n-1-j) k_j v_j^T, float32 [dim][vdim] per (chunk, head).
__global__ void __launch_bounds__(RT_THREADS)
retention_local_kernel(const bf16* __restrict__ k, int k_stride, const bf16* __restrict__ v, int v_stride, const float2* __restrict__ angles,
                       int rot_dim, const float* __restrict__ powers, float k_scale, const int* __restrict__ cu_q, int n_heads, int dim,
                       int vdim, float* __restrict__ parts) {
    grid_chain_entry();
    extern __shared__ __align__(16) float rt_smem[];
    const int head = blockIdx.y, seq = blockIdx.z;
    const int begin = cu_q[seq] + blockIdx.x * RT_CHUNK, end = cu_q[seq + 1];
    if (begin >= end) return;
    const int n = min(RT_CHUNK, end - begin), dp = rt_padded(dim);
    const int ks = rt_stride(dp, 8), vs = rt_stride(vdim, 8);
    float* k_s = rt_smem;                     // [RT_CHUNK][ks]
    float* v_s = k_s + RT_CHUNK * ks;         // [RT_CHUNK][vs]
    float* pow_s = v_s + RT_CHUNK * vs;       // [RT_CHUNK + 1]
    for (int i = threadIdx.x; i <= RT_CHUNK; i += RT_THREADS) pow_s[i] = powers[(size_t)head * (RT_CHUNK + 1) + i];
    __syncthreads();
    stage_turned(k_s, ks, dp, k + (size_t)begin * k_stride + (size_t)head * dim, k_stride, n, dim, rot_dim,
                 angles + (size_t)begin * (rot_dim / 2), k_scale, pow_s);
    stage_values(v_s, vs, v + (size_t)begin * v_stride + (size_t)head * vdim, v_stride, n, vdim);
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, r = lane >> 2, q = lane & 3;
    const int col_blocks = (vdim + 31) / 32, items = dp / 16 * col_blocks;
    float* out = parts + rt_record(cu_q, seq, blockIdx.x, n_heads, head) * dim * vdim;
    for (int item = warp; item < items; item += RT_THREADS / 32) {
        const int d0 = item / col_blocks * 16, c0 = item % col_blocks * 32;
        float acc[4][4];
#pragma unroll
        for (int t = 0; t < 4; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
        for (int j0 = 0; j0 < n; j0 += 8) {   // (rows from n on are zeros)
            const float* ka = k_s + (size_t)(j0 + q) * ks + d0 + r;
            const Split a[4] = {split_tf32(ka[0]), split_tf32(ka[8]), split_tf32(ka[4 * ks]), split_tf32(ka[4 * ks + 8])};
            const float* vb = v_s + (size_t)(j0 + q) * vs + c0 + r;
#pragma unroll
            for (int t = 0; t < 4; ++t)
                if (c0 + 8 * t < vdim) mma_half_split(acc[t], a, vb[8 * t], vb[4 * vs + 8 * t]);
        }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const int c = c0 + 8 * t + 2 * q;
            if (c0 + 8 * t >= vdim) continue;
            if (d0 + r < dim) *reinterpret_cast<float2*>(out + (size_t)(d0 + r) * vdim + c) = make_float2(acc[t][0], acc[t][1]);
            if (d0 + r + 8 < dim) *reinterpret_cast<float2*>(out + (size_t)(d0 + r + 8) * vdim + c) = make_float2(acc[t][2], acc[t][3]);
        }
    }
}

// (2) The chain over a sequence's chunks: every chunk's record becomes the state BEFORE it, and the state after the last one goes
// to the sequence's row. Two elements of S per thread; the records are read sixteen ahead.
#define RT_CARRY_THREADS 128
__global__ void __launch_bounds__(RT_CARRY_THREADS)
retention_carry_kernel(float* __restrict__ parts, const float* __restrict__ powers, const int* __restrict__ cu_q, const int* __restrict__ slots,
                       float* __restrict__ state, long long slot_stride, long long s_offset, int n_heads, int dim, int vdim) {
    grid_chain_entry();
    const int head = blockIdx.y, seq = blockIdx.z, size = dim * vdim;
    const int at = (blockIdx.x * RT_CARRY_THREADS + threadIdx.x) * 2;
    const int len = cu_q[seq + 1] - cu_q[seq], slot = slots[seq];
    if (at >= size || len <= 0) return;
    const int chunks = (len + RT_CHUNK - 1) / RT_CHUNK;
    float* row = slot >= 0 ? state + slot * slot_stride + s_offset + (long long)head * size + at : nullptr;
    float2 s = row ? *reinterpret_cast<const float2*>(row) : make_float2(0.f, 0.f);
    float* rec = parts + rt_record(cu_q, seq, 0, n_heads, head) * size + at;
    const long long pitch = (long long)n_heads * size;
    const float whole = powers[(size_t)head * (RT_CHUNK + 1) + RT_CHUNK];
    const float last = powers[(size_t)head * (RT_CHUNK + 1) + len - (chunks - 1) * RT_CHUNK];
    constexpr int AHEAD = 16;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float2 own[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            own[u] = c0 + u < chunks ? *reinterpret_cast<const float2*>(rec + (c0 + u) * pitch) : make_float2(0.f, 0.f);
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            if (c0 + u >= chunks) break;
            *reinterpret_cast<float2*>(rec + (c0 + u) * pitch) = s;
            const float f = c0 + u == chunks - 1 ? last : whole;
            s = make_float2(fmaf(f, s.x, own[u].x), fmaf(f, s.y, own[u].y));
        }
    }
    if (row) *reinterpret_cast<float2*>(row) = s;
}

// (3) A chunk's outputs: the part of the state before it, Q S0 under the decay's powers, and the scores Q K^T under the decay and the
// causal mask times the values; then the norm over a token's vdim components, the gate and the store. Warp w owns the 16 tokens
// 16 (w % 4) onwards and one half (w / 4) of the value columns, whose sums stay in its registers; of the scores it makes every second
// tile of eight keys, and the halves meet in shared memory, where S0 has been read by then. NV: eight-column tiles of the values
// that a warp's registers hold; FULL: both halves have all of them, so that no test stands between their loads and products.
#define RT_PS (RT_CHUNK + 4)   // row stride of the scores in shared memory
__host__ __device__ inline int rt_front(int dp, int vdim) {   // floats of the piece that holds S0 and then the scores
    const int s0 = dp * rt_stride(vdim, 8);
    return s0 > RT_CHUNK * RT_PS ? s0 : RT_CHUNK * RT_PS;
}
template <int NV, bool FULL>
__global__ void __launch_bounds__(RT_THREADS, 2)
retention_out_kernel(const bf16* __restrict__ q, int q_stride, const bf16* __restrict__ k, int k_stride, const bf16* __restrict__ v, int v_stride,
                     const bf16* __restrict__ gate, int gate_stride, const float2* __restrict__ angles, int rot_dim,
                     const float* __restrict__ powers, float k_scale, float eps, const int* __restrict__ cu_q, int n_heads, int dim, int vdim,
                     const float* __restrict__ parts, bf16* __restrict__ out) {
    grid_chain_entry();
    extern __shared__ __align__(16) float rt_smem[];
    __shared__ float norm_s[2][RT_CHUNK];
    const int head = blockIdx.y, seq = blockIdx.z;
    const int begin = cu_q[seq] + blockIdx.x * RT_CHUNK, end = cu_q[seq + 1];
    if (begin >= end) return;
    const int n = min(RT_CHUNK, end - begin), dp = rt_padded(dim);
    const int qs = rt_stride(dp, 4), ss = rt_stride(vdim, 8);
    float* s_s = rt_smem;                     // [dp][ss], then the scores [RT_CHUNK][RT_PS]
    float* q_s = s_s + rt_front(dp, vdim);    // [RT_CHUNK][qs]
    float* k_s = q_s + RT_CHUNK * qs;         // [RT_CHUNK][qs]
    float* v_s = k_s + RT_CHUNK * qs;         // [RT_CHUNK][ss]
    float* pow_s = v_s + RT_CHUNK * ss;       // [RT_CHUNK + 1]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, r = lane >> 2, c4 = lane & 3;
    for (int i = threadIdx.x; i <= RT_CHUNK; i += RT_THREADS) pow_s[i] = powers[(size_t)head * (RT_CHUNK + 1) + i];
    {
        const float* s0 = parts + rt_record(cu_q, seq, blockIdx.x, n_heads, head) * dim * vdim;
        const int per_row = vdim / 4;
        for (int i = threadIdx.x; i < dp * per_row; i += RT_THREADS) {
            const int d = i / per_row, c = (i % per_row) * 4;
            cp_async_16(s_s + (size_t)d * ss + c, s0 + (d < dim ? (size_t)d * vdim + c : 0), d < dim);
        }
        cp_async_commit();
    }
    const float2* turn = angles + (size_t)begin * (rot_dim / 2);
    stage_turned(q_s, qs, dp, q + (size_t)begin * q_stride + (size_t)head * dim, q_stride, n, dim, rot_dim, turn, 1.f, nullptr);
    stage_turned(k_s, qs, dp, k + (size_t)begin * k_stride + (size_t)head * dim, k_stride, n, dim, rot_dim, turn, k_scale, nullptr);
    stage_values(v_s, ss, v + (size_t)begin * v_stride + (size_t)head * vdim, v_stride, n, vdim);
    cp_async_wait<0>();
    __syncthreads();
    const int rows = warp & 3, half = warp >> 2;       // 16 tokens, and a half of the columns
    const int row0 = 16 * rows + r, row1 = row0 + 8;   // this lane's two tokens
    const int tiles = vdim / 8, first = half * ((tiles + 1) / 2), mine = half ? tiles - first : (tiles + 1) / 2, col0 = 8 * first;
    const bool busy = 16 * rows < n;
    float o[NV][4], s[4][4];
#pragma unroll
    for (int t = 0; t < NV; ++t) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.f;
#pragma unroll
    for (int t = 0; t < 4; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.f;
    auto left = [&](int d0, Split (&a)[4]) {
        const float* qa = q_s + (size_t)row0 * qs + d0 + c4;
        a[0] = split_tf32(qa[0]);
        a[1] = split_tf32(qa[8 * qs]);
        a[2] = split_tf32(qa[4]);
        a[3] = split_tf32(qa[8 * qs + 4]);
    };
    // keys 16 t + 8 half onwards, t up to this warp's own tokens
    auto scores = [&](auto count) {
        for (int d0 = 0; d0 < dp; d0 += 8) {
            Split a[4];
            left(d0, a);
            const float* kb = k_s + (size_t)(8 * half + r) * qs + d0 + c4;
#pragma unroll
            for (int t = 0; t < decltype(count)::value; ++t)
                mma_split(s[t], a, split_tf32(kb[(size_t)16 * t * qs]), split_tf32(kb[(size_t)16 * t * qs + 4]));
        }
    };
    if (busy) {
        if (rows == 0) scores(std::integral_constant<int, 1>());
        else if (rows == 1) scores(std::integral_constant<int, 2>());
        else if (rows == 2) scores(std::integral_constant<int, 3>());
        else scores(std::integral_constant<int, 4>());
#pragma unroll 2
        for (int d0 = 0; d0 < dp; d0 += 8) {
            Split a[4];
            left(d0, a);
            const float* sb = s_s + (size_t)(d0 + c4) * ss + col0 + r;
#pragma unroll
            for (int t = 0; t < NV; ++t)
                if (FULL || t < mine) mma_split(o[t], a, split_tf32(sb[8 * t]), split_tf32(sb[4 * ss + 8 * t]));
        }
        const float f0 = pow_s[row0 + 1], f1 = pow_s[row1 + 1];
#pragma unroll
        for (int t = 0; t < NV; ++t) {
            o[t][0] *= f0;
            o[t][1] *= f0;
            o[t][2] *= f1;
            o[t][3] *= f1;
        }
    }
    __syncthreads();   // everyone has read S0: the scores take its place
    float* p_s = s_s;
    if (busy) {
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            if (t > rows) continue;
            const int j = 16 * t + 8 * half + 2 * c4;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int back = (e < 2 ? row0 : row1) - j - (e & 1);
                s[t][e] = back >= 0 ? s[t][e] * pow_s[back >= 0 ? back : 0] : 0.f;
            }
            *reinterpret_cast<float2*>(p_s + row0 * RT_PS + j) = make_float2(s[t][0], s[t][1]);
            *reinterpret_cast<float2*>(p_s + row1 * RT_PS + j) = make_float2(s[t][2], s[t][3]);
        }
    }
    __syncthreads();
    float sum[2] = {0.f, 0.f};
    if (busy) {
        for (int t = 0; t <= 2 * rows + 1; ++t) {
            const float* pa = p_s + row0 * RT_PS + 8 * t + c4;
            const Split a[4] = {split_tf32(pa[0]), split_tf32(pa[8 * RT_PS]), split_tf32(pa[4]), split_tf32(pa[8 * RT_PS + 4])};
            const float* vb = v_s + (size_t)(8 * t + c4) * ss + col0 + r;
#pragma unroll
            for (int u = 0; u < NV; ++u)
                if (FULL || u < mine) mma_half_split(o[u], a, vb[8 * u], vb[4 * ss + 8 * u]);
        }
#pragma unroll
        for (int t = 0; t < NV; ++t) {
            sum[0] = fmaf(o[t][0], o[t][0], fmaf(o[t][1], o[t][1], sum[0]));
            sum[1] = fmaf(o[t][2], o[t][2], fmaf(o[t][3], o[t][3], sum[1]));
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    }
    if (c4 == 0) {
        norm_s[half][row0] = sum[0];
        norm_s[half][row1] = sum[1];
    }
    uint32_t z_raw[2][NV];   // the gate's logits, on their way across the barrier
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int row = i ? row1 : row0;
        const bf16* g = gate + (size_t)(begin + min(row, n - 1)) * gate_stride + (size_t)head * vdim + col0 + 2 * c4;
#pragma unroll
        for (int t = 0; t < NV; ++t) z_raw[i][t] = FULL || t < mine ? __ldg(reinterpret_cast<const unsigned*>(g + 8 * t)) : 0u;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int row = i ? row1 : row0;
        if (row >= n) continue;
        const float inv = 1.0f / sqrtf((norm_s[0][row] + norm_s[1][row]) / (float)vdim + eps);
        bf16* dst = out + (size_t)(begin + row) * n_heads * vdim + (size_t)head * vdim + col0 + 2 * c4;
#pragma unroll
        for (int t = 0; t < NV; ++t) {
            if (!FULL && t >= mine) continue;
            const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&z_raw[i][t]));
            const float y0 = o[t][2 * i] * inv * __fdividef(z.x, 1.f + expf(-z.x)), y1 = o[t][2 * i + 1] * inv * __fdividef(z.y, 1.f + expf(-z.y));
            *reinterpret_cast<__nv_bfloat162*>(dst + 8 * t) = __floats2bfloat162_rn(y0, y1);
        }
    }
}

// Whether the chunked kernels take these sizes (bfloat16 rows that 16-byte accesses can address).
QF_EXPORT int qf_retention_chunks_take(int dim, int vdim, int rot_dim) {
    return dim > 0 && dim <= RT_MAX_DIM && vdim > 0 && vdim <= RT_MAX_VDIM && dim % 8 == 0 && vdim % 8 == 0 && rot_dim % 16 == 0 && rot_dim <= dim;
}
QF_EXPORT int qf_retention_chunk(void) { return RT_CHUNK; }

// q, k: [T][heads * dim], v, gate: [T][heads * vdim] with row strides (whole eights), out [T][heads * vdim]; angles float32
// [T][rot_dim / 2][2]; powers float32 [heads][RT_CHUNK + 1], the decays' powers from 0; parts: float32 scratch of
// (T / RT_CHUNK + n_seqs) * heads * dim * vdim; S [heads][dim][vdim] at s_offset of a slot's row (slot_stride and s_offset in
// whole fours). max_q_len: the most tokens any sequence brings.
QF_EXPORT int qf_retention_chunks(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const void* gate,
                                  int gate_stride, const void* angles, int rot_dim, const float* powers, float k_scale, float eps,
                                  const int* cu_q, const int* slots, int n_seqs, int max_q_len, float* state, long long slot_stride,
                                  long long s_offset, int n_heads, int dim, int vdim, float* parts, void* out, cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0 || n_heads <= 0) return 0;
    if (!qf_retention_chunks_take(dim, vdim, rot_dim) || q_stride % 8 || k_stride % 8 || v_stride % 8 || gate_stride % 2 || slot_stride % 4 ||
        s_offset % 4 || ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)parts | (uintptr_t)state) % 16 ||
        ((uintptr_t)gate | (uintptr_t)out) % 4)
        return (int)cudaErrorInvalidValue;
    const int chunks = (max_q_len + RT_CHUNK - 1) / RT_CHUNK, dp = rt_padded(dim);
    const dim3 grid(chunks, n_heads, n_seqs), block(RT_THREADS);
    const size_t local_smem = (size_t)(RT_CHUNK * (rt_stride(dp, 8) + rt_stride(vdim, 8)) + RT_CHUNK + 1) * sizeof(float);
    cudaError_t e = cudaFuncSetAttribute(retention_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local_smem);
    if (e != cudaSuccess) return (int)e;
    e = launch_pdl(retention_local_kernel, grid, block, local_smem, stream, (const bf16*)k, k_stride, (const bf16*)v, v_stride,
                   (const float2*)angles, rot_dim, powers, k_scale, cu_q, n_heads, dim, vdim, parts);
    if (e != cudaSuccess) return (int)e;
    const int pairs = dim * vdim / 2;
    e = launch_pdl(retention_carry_kernel, dim3((pairs + RT_CARRY_THREADS - 1) / RT_CARRY_THREADS, n_heads, n_seqs), dim3(RT_CARRY_THREADS), 0, stream, parts, powers, cu_q, slots,
                   state, slot_stride, s_offset, n_heads, dim, vdim);
    if (e != cudaSuccess) return (int)e;
    const size_t out_smem = (size_t)(rt_front(dp, vdim) + RT_CHUNK * (2 * rt_stride(dp, 4) + rt_stride(vdim, 8)) + RT_CHUNK + 1) * sizeof(float);
#define QF_RETENTION(NV)                                                                                                              \
    {                                                                                                                                 \
        auto kernel = vdim == 16 * NV ? retention_out_kernel<NV, true> : retention_out_kernel<NV, false>;                            \
        e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem);                                 \
        if (e != cudaSuccess) return (int)e;                                                                                          \
        return (int)launch_pdl(kernel, grid, block, out_smem, stream, (const bf16*)q, q_stride, (const bf16*)k, k_stride, \
                               (const bf16*)v, v_stride, (const bf16*)gate, gate_stride, (const float2*)angles, rot_dim, powers, k_scale, eps, \
                               cu_q, n_heads, dim, vdim, (const float*)parts, (bf16*)out);                                            \
    }
    if (vdim <= 32) QF_RETENTION(2)
    if (vdim <= 64) QF_RETENTION(4)
    QF_RETENTION(8)
#undef QF_RETENTION
}

// ------------------------------------------------------------------------------------------------------------------
// One token per sequence, any sizes: S <- decay S + k v^T, o = S^T q, the norm and the gate. A block per (sequence, head); a thread
// owns COLS neighbouring columns and every RB-th row of S, the row groups' parts of o are added in their order.
#define RK_THREADS 256
template <typename T, int COLS>
__global__ void __launch_bounds__(RK_THREADS)
retention_token_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k, int k_stride, const T* __restrict__ v, int v_stride,
                       const T* __restrict__ gate, int gate_stride, const int* __restrict__ tok_pos, const float* __restrict__ inv_freq,
                       int rot_dim, float amplitude, const float* __restrict__ decay, float k_scale, float eps, const int* __restrict__ cu_q,
                       const int* __restrict__ slots, float* __restrict__ state, long long slot_stride, long long s_offset, int n_heads,
                       int dim, int vdim, T* __restrict__ out) {
    grid_chain_entry();
    extern __shared__ __align__(16) float rk_smem[];
    __shared__ float scratch[33];
    const int head = blockIdx.x, seq = blockIdx.y, t = cu_q[seq], slot = slots[seq];
    if (cu_q[seq + 1] <= t) return;
    const int groups = (vdim + COLS - 1) / COLS, rb = max(1, min(dim, RK_THREADS / groups));
    float* q_s = rk_smem;                     // [dim]
    float* k_s = q_s + dim;                   // [dim]
    float* part_s = k_s + dim;                // [rb][vdim]
    const int half = rot_dim / 2;
    const T* qh = q + (size_t)t * q_stride + (size_t)head * dim;
    const T* kh = k + (size_t)t * k_stride + (size_t)head * dim;
    const int group = threadIdx.x % groups, r0 = threadIdx.x / groups;
    float* S = slot >= 0 ? state + slot * slot_stride + s_offset + (long long)head * dim * vdim : nullptr;
    constexpr int AHEAD = 8;
    float s[AHEAD][COLS];   // rows d0, d0 + rb, ... of this thread's columns
    auto load_rows = [&](int d0, int c) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int d = d0 + u * rb;
#pragma unroll
            for (int e = 0; e < COLS; ++e) s[u][e] = 0.f;
            if (S && d < dim) {
                if constexpr (COLS == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(S + (size_t)d * vdim + c);
                    s[u][0] = x.x;
                    s[u][1] = x.y;
                    s[u][2] = x.z;
                    s[u][3] = x.w;
                } else {
                    s[u][0] = S[(size_t)d * vdim + c];
                }
            }
        }
    };
    if (r0 < rb) load_rows(r0, group * COLS);   // the state's first rows are on their way while q and k are turned
    const float pos = (float)tok_pos[t], keep = decay[head];
    for (int i = threadIdx.x; i < dim; i += RK_THREADS) {
        float a = Num<T>::to_f(qh[i]), b = Num<T>::to_f(kh[i]);
        if (i < rot_dim) {
            const bool first = i < half;
            const int j = first ? i : i - half, other = first ? i + half : i - half;
            float sn, c;
            sincosf(pos * inv_freq[j], &sn, &c);
            sn *= first ? -amplitude : amplitude;
            c *= amplitude;
            a = a * c + Num<T>::to_f(qh[other]) * sn;
            b = b * c + Num<T>::to_f(kh[other]) * sn;
        }
        q_s[i] = a;
        k_s[i] = b * k_scale;
    }
    __syncthreads();
    // (more column groups than threads: a thread takes several, one row group)
    for (int g = group; g < groups && r0 < rb; g += RK_THREADS) {
        const int c = g * COLS;
        float val[COLS], acc[COLS];
#pragma unroll
        for (int e = 0; e < COLS; ++e) {
            val[e] = Num<T>::to_f(v[(size_t)t * v_stride + (size_t)head * vdim + c + e]);
            acc[e] = 0.f;
        }
        for (int d0 = r0; d0 < dim; d0 += rb * AHEAD) {
            if (g != group || d0 != r0) load_rows(d0, c);
#pragma unroll
            for (int u = 0; u < AHEAD; ++u) {
                const int d = d0 + u * rb;
                if (d >= dim) break;
                const float kd = k_s[d], qd = q_s[d];
#pragma unroll
                for (int e = 0; e < COLS; ++e) {
                    s[u][e] = fmaf(kd, val[e], s[u][e] * keep);
                    acc[e] = fmaf(s[u][e], qd, acc[e]);
                }
                if (S) {
                    if constexpr (COLS == 4) *reinterpret_cast<float4*>(S + (size_t)d * vdim + c) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
                    else S[(size_t)d * vdim + c] = s[u][0];
                }
            }
        }
#pragma unroll
        for (int e = 0; e < COLS; ++e) part_s[(size_t)r0 * vdim + c + e] = acc[e];
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < vdim; c += RK_THREADS) {
        float sum = 0.f;
        for (int r = 0; r < rb; ++r) sum += part_s[(size_t)r * vdim + c];
        part_s[c] = sum;
        ss = fmaf(sum, sum, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)vdim + eps);
    for (int c = threadIdx.x; c < vdim; c += RK_THREADS) {   // each thread re-reads the columns it summed itself
        const float z = Num<T>::to_f(gate[(size_t)t * gate_stride + (size_t)head * vdim + c]);
        out[(size_t)t * n_heads * vdim + (size_t)head * vdim + c] = Num<T>::from_f(part_s[c] * inv * (z / (1.f + expf(-z))));
    }
}

QF_EXPORT int qf_retention_token(int is_bf16, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                                 const void* gate, int gate_stride, const int* tok_pos, const float* inv_freq, int rot_dim, float amplitude,
                                 const float* decay, float k_scale, float eps, const int* cu_q, const int* slots, int n_seqs, float* state,
                                 long long slot_stride, long long s_offset, int n_heads, int dim, int vdim, void* out, cudaStream_t stream) {
    if (n_seqs <= 0 || n_heads <= 0) return 0;
    if (dim <= 0 || vdim <= 0 || rot_dim < 0 || rot_dim > dim || (rot_dim & 1) || (rot_dim && !inv_freq)) return (int)cudaErrorInvalidValue;
    const bool four = vdim % 4 == 0 && slot_stride % 4 == 0 && s_offset % 4 == 0 && (uintptr_t)state % 16 == 0;
    const int groups = four ? vdim / 4 : vdim;
    int rb = RK_THREADS / groups;
    rb = rb < 1 ? 1 : rb > dim ? dim : rb;
    const size_t smem = (size_t)(2 * dim + rb * vdim) * sizeof(float);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(n_heads, n_seqs), block(RK_THREADS);
#define QF_TOKEN(T, COLS)                                                                                                                  \
    return (int)launch_pdl(retention_token_kernel<T, COLS>, grid, block, smem, stream, (const T*)q, q_stride, (const T*)k, k_stride,      \
                           (const T*)v, v_stride, (const T*)gate, gate_stride, tok_pos, inv_freq, rot_dim, amplitude, decay, k_scale, eps, \
                           cu_q, slots, state, slot_stride, s_offset, n_heads, dim, vdim, (T*)out)
    if (is_bf16) {
        if (four) QF_TOKEN(bf16, 4);
        QF_TOKEN(bf16, 1);
    }
    if (four) QF_TOKEN(float, 4);
    QF_TOKEN(float, 1);
#undef QF_TOKEN
}

// ------------------------------------------------------------------------------------------------------------------
// What the scan of csrc/recurrent.cu reads where the chunked kernels do not run (true float32 steps, sizes in no whole eights): q
// and k turned, k times k_scale, and v, as float32 rows [q | k | v].
template <typename T>
__global__ void __launch_bounds__(256)
retention_rows_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k, int k_stride, const T* __restrict__ v, int v_stride,
                      const float2* __restrict__ angles, int rot_dim, float k_scale, int n_heads, int dim, int vdim, float* __restrict__ rows) {
    grid_chain_entry();
    const int t = blockIdx.x, half = rot_dim / 2, qk = n_heads * dim, vw = n_heads * vdim;
    float* dst = rows + (size_t)t * (2 * qk + vw);
    const float2* cs = angles + (size_t)t * half;
    for (int i = threadIdx.x; i < 2 * qk; i += blockDim.x) {
        const bool is_k = i >= qk;
        const int col = is_k ? i - qk : i, d = col % dim;
        const T* src = is_k ? k + (size_t)t * k_stride : q + (size_t)t * q_stride;
        float x = Num<T>::to_f(src[col]);
        if (d < rot_dim) {
            const bool first = d < half;
            const float other = Num<T>::to_f(src[first ? col + half : col - half]);
            const float2 a = cs[first ? d : d - half];
            x = first ? x * a.x - other * a.y : x * a.x + other * a.y;
        }
        dst[i] = is_k ? x * k_scale : x;
    }
    for (int i = threadIdx.x; i < vw; i += blockDim.x) dst[2 * qk + i] = Num<T>::to_f(v[(size_t)t * v_stride + i]);
}

QF_EXPORT int qf_retention_rows(int is_bf16, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                                const void* angles, int rot_dim, float k_scale, int n_tokens, int n_heads, int dim, int vdim, float* rows,
                                cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (dim <= 0 || vdim <= 0 || rot_dim < 0 || rot_dim > dim || (rot_dim & 1) || (rot_dim && !angles)) return (int)cudaErrorInvalidValue;
    if (is_bf16)
        return (int)launch_pdl(retention_rows_kernel<bf16>, dim3(n_tokens), dim3(256), 0, stream, (const bf16*)q, q_stride, (const bf16*)k, k_stride,
                               (const bf16*)v, v_stride, (const float2*)angles, rot_dim, k_scale, n_heads, dim, vdim, rows);
    return (int)launch_pdl(retention_rows_kernel<float>, dim3(n_tokens), dim3(256), 0, stream, (const float*)q, q_stride, (const float*)k, k_stride,
                           (const float*)v, v_stride, (const float2*)angles, rot_dim, k_scale, n_heads, dim, vdim, rows);
}
