// The two latents of a latent-attention mixer, from their fused down-projection:
//   down[t] = [ Dq h_t | Dkv h_t ]  (float32, q_rank + kv_rank columns)
//   a_t = down[t][:q_rank]  * rsqrt(mean(.^2) + eps) * q_norm      -> q_latent[t]    (what the query up-projection reads)
//   c_t = down[t][q_rank:]  * rsqrt(mean(.^2) + eps) * kv_norm     -> the cache row of the token's own position
// Both sums of squares and roots are float32. The key/value latent is the only thing the mixer keeps per position: it is
// written as the single "head" of a cache whose pages hold one plane, [pages][1][1][QF_PAGE][kv_rank]. With q_rank = 0
// there is no query latent and only the cache row is made. A padding entry (slot -1) writes no cache row; `latent_out`,
// if given, also receives c_t in token order (for whoever wants the step's latents without reading the cache).
// With `rot_dim` > 0 the down-projection has rot_dim columns more, [ .. | e_t ]: one key part that all heads share. Its
// neighbours (2i, 2i + 1) are turned by the token's position, angle = position * inv_freq[i], cosine and sine times
// `amplitude`, and it is kept behind the latent in the same cache row, which then has site.head_dim >= kv_rank + rot_dim
// elements (what lies beyond is never written and stays zero).
// `rotate_heads_kernel` does the same to the queries: per head it takes rot_dim columns of an input row, turns them, and
// writes them to their place in an output row (zeros from there to the end of the head's row).
#include "common.cuh"

__device__ __forceinline__ void turn_pair(float& a, float& b, int pos, float freq, float amplitude) {
    float sn, cs;
    sincosf((float)pos * freq, &sn, &cs);
    sn *= amplitude;
    cs *= amplitude;
    const float x = a, y = b;
    a = x * cs - y * sn;
    b = y * cs + x * sn;
}

template <typename T>
__global__ void __launch_bounds__(128)
latent_norm_cache_kernel(const float* __restrict__ down, int ld, int q_rank, int kv_rank, const T* __restrict__ q_norm,
                         const T* __restrict__ kv_norm, float eps, const int* __restrict__ tok_seq, const int* __restrict__ tok_pos,
                         const int* __restrict__ slots, T* __restrict__ q_latent, T* __restrict__ latent_out, KvSite<T> site,
                         int write_cache, int* err, int rot_dim, const float* __restrict__ inv_freq, float amplitude) {
    // the norm weights are nobody's output: a thread's first few are fetched before the wait for the kernel before this one
    grid_launch_dependents();
    constexpr int AHEAD = 4;
    float qw[AHEAD], kw[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
        const int c = threadIdx.x + u * 128;
        qw[u] = c < q_rank ? Num<T>::to_f(q_norm[c]) : 0.f;
        kw[u] = c < kv_rank ? Num<T>::to_f(kv_norm[c]) : 0.f;
    }
    grid_dependency_wait();
    __shared__ float scratch[33];
    const int t = blockIdx.x;
    const float* row = down + (size_t)t * ld;
    // where the latent goes: a chain of three dependent loads, started before the sums so that it runs under them
    T* cache_row = nullptr;
    const int slot = slots[tok_seq[t]];
    bool no_page = false;
    if (write_cache && slot >= 0) {
        cache_row = kv_row(site, slot, tok_pos[t], 0, 0);
        no_page = cache_row == nullptr;
    }
    if (q_rank > 0) {
        float ss = 0.f;
        for (int c = threadIdx.x; c < q_rank; c += blockDim.x) ss += row[c] * row[c];
        const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)q_rank + eps);
        T* dst = q_latent + (size_t)t * q_rank;
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int c = threadIdx.x + u * 128;
            if (c < q_rank) dst[c] = Num<T>::from_f(row[c] * inv * qw[u]);
        }
        for (int c = threadIdx.x + AHEAD * 128; c < q_rank; c += 128) dst[c] = Num<T>::from_f(row[c] * inv * Num<T>::to_f(q_norm[c]));
    }
    const float* kv = row + q_rank;
    if (cache_row) {   // the shared rotated key part, by the block's last warps first: the norms below start with the first
        const int pos = tok_pos[t];
        for (int i = (int)blockDim.x - 1 - (int)threadIdx.x; i < rot_dim / 2; i += blockDim.x) {
            float a = kv[kv_rank + 2 * i], b = kv[kv_rank + 2 * i + 1];
            turn_pair(a, b, pos, inv_freq[i], amplitude);
            cache_row[kv_rank + 2 * i] = Num<T>::from_f(a);
            cache_row[kv_rank + 2 * i + 1] = Num<T>::from_f(b);
        }
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < kv_rank; c += blockDim.x) ss += kv[c] * kv[c];
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)kv_rank + eps);
    if (no_page && threadIdx.x == 0) atomicOr(err, QF_ERR_NO_PAGE);
    T* plain = latent_out ? latent_out + (size_t)t * kv_rank : nullptr;
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
        const int c = threadIdx.x + u * 128;
        if (c < kv_rank) {
            const T v = Num<T>::from_f(kv[c] * inv * kw[u]);
            if (cache_row) cache_row[c] = v;
            if (plain) plain[c] = v;
        }
    }
    for (int c = threadIdx.x + AHEAD * 128; c < kv_rank; c += 128) {
        const T v = Num<T>::from_f(kv[c] * inv * Num<T>::to_f(kv_norm[c]));
        if (cache_row) cache_row[c] = v;
        if (plain) plain[c] = v;
    }
}

template <typename T>
static int launch(const float* down, int ld, int q_rank, int kv_rank, const void* q_norm, const void* kv_norm, float eps,
                  const int* tok_seq, const int* tok_pos, const int* slots, void* q_latent, void* latent_out, void* base,
                  const int* table, long long page_elems, int table_stride, int write_cache, int n_tokens, int* err,
                  int row_dim, int rot_dim, const float* inv_freq, float amplitude, cudaStream_t stream) {
    KvSite<T> site{(T*)base, table, page_elems, table_stride, 1, row_dim};
    return (int)launch_pdl(latent_norm_cache_kernel<T>, dim3(n_tokens), dim3(128), 0, stream, down, ld, q_rank, kv_rank,
                           (const T*)q_norm, (const T*)kv_norm, eps, tok_seq, tok_pos, slots, (T*)q_latent, (T*)latent_out, site,
                           write_cache, err, rot_dim, inv_freq, amplitude);
}

// down float32 [n_tokens][ld] (ld >= q_rank + kv_rank); the norm weights, q_latent [n_tokens][q_rank], latent_out
// [n_tokens][kv_rank] (may be null) and the cache share the activation dtype.
// row_dim: elements of a cache row, at least kv_rank + rot_dim; rot_dim even, 0 for a latent without a rotated part.
QF_EXPORT int qf_latent_norm_cache_turned(int is_bf16, const float* down, int ld, int q_rank, int kv_rank, const void* q_norm,
                                          const void* kv_norm, float eps, const int* tok_seq, const int* tok_pos, const int* slots,
                                          void* q_latent, void* latent_out, void* base, const int* table, long long page_elems,
                                          int table_stride, int write_cache, int n_tokens, int* err, int row_dim, int rot_dim,
                                          const float* inv_freq, float amplitude, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (kv_rank <= 0 || q_rank < 0 || rot_dim < 0 || rot_dim % 2 || ld < q_rank + kv_rank + rot_dim || row_dim < kv_rank + rot_dim ||
        (rot_dim > 0 && !inv_freq))
        return (int)cudaErrorInvalidValue;
    return is_bf16 ? launch<bf16>(down, ld, q_rank, kv_rank, q_norm, kv_norm, eps, tok_seq, tok_pos, slots, q_latent, latent_out,
                                  base, table, page_elems, table_stride, write_cache, n_tokens, err, row_dim, rot_dim, inv_freq,
                                  amplitude, stream)
                   : launch<float>(down, ld, q_rank, kv_rank, q_norm, kv_norm, eps, tok_seq, tok_pos, slots, q_latent, latent_out,
                                   base, table, page_elems, table_stride, write_cache, n_tokens, err, row_dim, rot_dim, inv_freq,
                                   amplitude, stream);
}

QF_EXPORT int qf_latent_norm_cache(int is_bf16, const float* down, int ld, int q_rank, int kv_rank, const void* q_norm,
                                   const void* kv_norm, float eps, const int* tok_seq, const int* tok_pos, const int* slots,
                                   void* q_latent, void* latent_out, void* base, const int* table, long long page_elems,
                                   int table_stride, int write_cache, int n_tokens, int* err, cudaStream_t stream) {
    return qf_latent_norm_cache_turned(is_bf16, down, ld, q_rank, kv_rank, q_norm, kv_norm, eps, tok_seq, tok_pos, slots, q_latent,
                                       latent_out, base, table, page_elems, table_stride, write_cache, n_tokens, err, kv_rank, 0, nullptr,
                                       1.f, stream);
}

// A thread per (token, head, pair of the rotated part or pair of the padding behind it).
template <typename T>
__global__ void __launch_bounds__(256)
rotate_heads_kernel(const T* __restrict__ x, long long ldx, int x_pitch, int x_first, T* __restrict__ out, long long ldo, int out_pitch,
                    int out_first, int rot_dim, const float* __restrict__ inv_freq, float amplitude, const int* __restrict__ tok_pos,
                    int heads, size_t total) {
    grid_chain_entry();
    const int tail = out_pitch - out_first, each = (tail + 1) / 2;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int p = (int)(i % each), h = (int)(i / each % heads);
        const size_t t = i / each / heads;
        float a = 0.f, b = 0.f;
        if (2 * p < rot_dim) {
            const T* src = x + t * ldx + (size_t)h * x_pitch + x_first + 2 * p;
            a = Num<T>::to_f(src[0]);
            b = Num<T>::to_f(src[1]);
            turn_pair(a, b, tok_pos[t], inv_freq[p], amplitude);
        }
        T* dst = out + t * ldo + (size_t)h * out_pitch + out_first + 2 * p;
        dst[0] = Num<T>::from_f(a);
        if (2 * p + 1 < tail) dst[1] = Num<T>::from_f(b);
    }
}

// x: rows of `heads` pieces of x_pitch columns whose rot_dim columns from x_first on are turned; out: rows of pieces of out_pitch
// columns that receive them from out_first on, zeros behind them.
QF_EXPORT int qf_rotate_heads(int is_bf16, const void* x, long long ldx, int x_pitch, int x_first, void* out, long long ldo, int out_pitch,
                              int out_first, int rot_dim, const float* inv_freq, float amplitude, const int* tok_pos, int heads,
                              int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0 || heads <= 0) return 0;
    if (rot_dim <= 0 || rot_dim % 2 || x_first < 0 || x_first + rot_dim > x_pitch || out_first < 0 || out_first + rot_dim > out_pitch)
        return (int)cudaErrorInvalidValue;
    const size_t total = (size_t)n_tokens * heads * ((out_pitch - out_first + 1) / 2);
    const size_t most = (size_t)(qf_sm_count() > 0 ? qf_sm_count() : 1) * 16, want = (total + 255) / 256;
    const dim3 grid((unsigned)(want < most ? want : most));
    if (is_bf16)
        return (int)launch_pdl(rotate_heads_kernel<bf16>, grid, dim3(256), 0, stream, (const bf16*)x, ldx, x_pitch, x_first, (bf16*)out, ldo,
                               out_pitch, out_first, rot_dim, inv_freq, amplitude, tok_pos, heads, total);
    return (int)launch_pdl(rotate_heads_kernel<float>, grid, dim3(256), 0, stream, (const float*)x, ldx, x_pitch, x_first, (float*)out, ldo,
                           out_pitch, out_first, rot_dim, inv_freq, amplitude, tok_pos, heads, total);
}
