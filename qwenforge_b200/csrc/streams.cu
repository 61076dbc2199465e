// Several residual streams side by side (hyper-connections): a token carries X[0..n-1], n float32 rows of `width`, instead of
// one. What stands between one sublayer and the next is ONE kernel here:
//
//   Y[r]  = sum_s mix[s][r] X[s] + out[r] y        the sublayer before enters the streams (all r from the old X)
//   u     = sum_r in[r] Y[r]                       what the next sublayer is to read
//   h     = tanh(alpha u) w + b                    its norm (a Dynamic Tanh: element by element, so no row has to be summed)
//   z_t   = h_t + sum_j f[j] h_(t - taps + 1 + j)  and a causal convolution over time per channel in front of it
//
// Everything is float32 until z is stored in the activation type; h is never stored. Every step may be absent: without y the
// streams pass as they are; without a destination they are not stored; without w the row u itself is stored (float32);
// without taps z = h; with `rows` only the named tokens are worked on (what an output head reads).
// At a sequence's start all streams are the embedding's row: `src_stream = 0` reads one row as every stream.
// y is a row per token, or (dest, top) the sum of the `top` rows y[dest[t * top + k]], each times row_weight[that row] if given
// (a feed-forward of routed experts leaves its chosen rows unsummed).
//
// A block takes a tile of tokens of one sequence and some of the channels, a thread one token's V neighbouring channels. The h of
// the tokens before the tile are worked out again from their streams (the old and the new streams are different buffers, so
// whoever owns those tokens has not changed them); what lies before the step's first token comes from the sequence's state,
// float32 [taps - 1][width], zeros at a sequence's start. The tile's h meet in shared memory, where the convolution reads them.
// Only a sequence's FIRST tile reads the state, and the same block replaces it, having read it, by the sequence's last taps - 1
// values of h: no second kernel, and no order between blocks. A row's arithmetic is the same chain of operations whatever
// the cut, the batch and the tile.
#include "common.cuh"

#define ST_THREADS 256

template <typename T> struct StreamsArgs {
    const float* src;           // old streams: element (t, s, c) at t * src_row + s * src_stream + c
    long long src_row, src_stream;
    float* dst;                 // new streams [tokens][n][width], or null
    const T* y;                 // null: nothing is pending
    const int* dest;
    int top;
    const float* row_weight;
    const float* mix;           // [n][n] (from, to); with y only
    const float* out_w;         // [n]; with y only
    const float* in_w;          // [n]; null: ones
    const T* weight;            // null: u itself goes to u_out
    const T* bias;
    float alpha;
    T* z;                       // [rows][width]
    float* u_out;               // [rows][width] float32
    const int* rows;            // null: every token of the step
    int n_rows, n_tokens;       // rows: how many are named; tokens that exist
    const float* taps;          // [width][n_taps], null: no convolution
    int n_taps;
    const int* cu_q;
    const int* slots;
    float* state;
    long long slot_stride, offset;
    int n, width;
    int* err;
};

template <typename T, int V> struct Channels;
template <typename T> struct Channels<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float* v) { v[0] = Num<T>::to_f(*p); }
    static __device__ __forceinline__ void store(T* p, const float* v) { *p = Num<T>::from_f(v[0]); }
};
template <> struct Channels<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float* v) {
        const float4 r = *reinterpret_cast<const float4*>(p);
        v[0] = r.x, v[1] = r.y, v[2] = r.z, v[3] = r.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* v) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <> struct Channels<bf16, 4> {
    static __device__ __forceinline__ void load(const bf16* p, float* v) {
        const uint2 r = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
        v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
    }
    static __device__ __forceinline__ void store(bf16* p, const float* v) {
        uint2 r;
        *reinterpret_cast<__nv_bfloat162*>(&r.x) = __floats2bfloat162_rn(v[0], v[1]);
        *reinterpret_cast<__nv_bfloat162*>(&r.y) = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = r;
    }
};

// NS: the most streams (a.n <= NS); HIST: the most inputs a convolution keeps (a.n_taps - 1 <= HIST), 0 without one; ROWS: tokens
// of a tile, the HIST before it included.
template <typename T, int V, int NS, int HIST, int ROWS>
__global__ void __launch_bounds__(ST_THREADS, NS <= 4 ? 4 : 2)
streams_kernel(const StreamsArgs<T> a) {
    grid_launch_dependents();
    constexpr int GROUPS = ST_THREADS / ROWS, OWN = ROWS - HIST;
    __shared__ float mix_s[NS * NS], out_s[NS], in_s[NS];
    __shared__ __align__(16) float h_s[2][HIST > 0 ? ROWS : 1][HIST > 0 ? GROUPS * V : 1];   // two tiles in turn
    // the coefficients are weights: fetched before the wait for the kernel before this one
    for (int i = threadIdx.x; i < NS * NS; i += ST_THREADS) {
        const int s = i / NS, r = i % NS;
        mix_s[i] = (a.mix && s < a.n && r < a.n) ? a.mix[s * a.n + r] : 0.f;
    }
    if (threadIdx.x < NS) {
        out_s[threadIdx.x] = (a.out_w && threadIdx.x < a.n) ? a.out_w[threadIdx.x] : 0.f;
        in_s[threadIdx.x] = threadIdx.x < a.n ? (a.in_w ? a.in_w[threadIdx.x] : 1.f) : 0.f;
    }
    const int group = threadIdx.x % GROUPS, row = threadIdx.x / GROUPS;
    const int c0 = (blockIdx.x * GROUPS + group) * V;
    const bool in = c0 < a.width;
    __shared__ __align__(16) float f_s[HIST + 1][HIST > 0 ? GROUPS * V : 1];   // the filter, a column per channel
    float w[V], b[V];
#pragma unroll
    for (int v = 0; v < V; ++v) w[v] = b[v] = 0.f;
    if (a.weight && in) {
        Channels<T, V>::load(a.weight + c0, w);
        Channels<T, V>::load(a.bias + c0, b);
    }
    if constexpr (HIST > 0) {
        for (int i = threadIdx.x; i < (HIST + 1) * GROUPS * V; i += ST_THREADS) {   // the oldest places of a shorter filter hold zeros
            const int c = i / (HIST + 1), j = i % (HIST + 1), channel = blockIdx.x * GROUPS * V + c, at = j - (HIST + 1 - a.n_taps);
            f_s[j][c] = (channel < a.width && at >= 0) ? a.taps[(size_t)channel * a.n_taps + at] : 0.f;
        }
    }
    __syncthreads();
    grid_dependency_wait();

    // h of token t (or u, without a norm); the new streams are stored on the way if asked
    auto value = [&](int t, bool keep, float (&h)[V]) {
        float x[NS][V], y[V];
        const float* xs = a.src + t * a.src_row + c0;
#pragma unroll
        for (int s = 0; s < NS; ++s) {
#pragma unroll
            for (int v = 0; v < V; ++v) x[s][v] = 0.f;
            if (s < a.n) Channels<float, V>::load(xs + s * a.src_stream, x[s]);
        }
        if (a.y) {
            if (a.dest) {
#pragma unroll
                for (int v = 0; v < V; ++v) y[v] = 0.f;
                for (int k = 0; k < a.top; k += 2) {   // two rows asked for together
                    const int r0 = a.dest[(size_t)t * a.top + k], r1 = k + 1 < a.top ? a.dest[(size_t)t * a.top + k + 1] : r0;
                    float p0[V], p1[V];
                    Channels<T, V>::load(a.y + (size_t)r0 * a.width + c0, p0);
                    Channels<T, V>::load(a.y + (size_t)r1 * a.width + c0, p1);
                    const float by0 = a.row_weight ? a.row_weight[r0] : 1.f;
                    const float by1 = k + 1 < a.top ? (a.row_weight ? a.row_weight[r1] : 1.f) : 0.f;
#pragma unroll
                    for (int v = 0; v < V; ++v) y[v] = fmaf(by1, p1[v], fmaf(by0, p0[v], y[v]));
                }
            } else {
                Channels<T, V>::load(a.y + (size_t)t * a.width + c0, y);
            }
        }
#pragma unroll
        for (int v = 0; v < V; ++v) h[v] = 0.f;
#pragma unroll
        for (int r = 0; r < NS; ++r) {
            if (r >= a.n) break;
            float to[V];
#pragma unroll
            for (int v = 0; v < V; ++v) to[v] = x[r][v];
            if (a.y) {
#pragma unroll
                for (int v = 0; v < V; ++v) to[v] = out_s[r] * y[v];
#pragma unroll
                for (int s = 0; s < NS; ++s)
#pragma unroll
                    for (int v = 0; v < V; ++v) to[v] = fmaf(mix_s[s * NS + r], x[s][v], to[v]);
            }
            if (keep && a.dst) Channels<float, V>::store(a.dst + ((size_t)t * a.n + r) * a.width + c0, to);
#pragma unroll
            for (int v = 0; v < V; ++v) h[v] = fmaf(in_s[r], to[v], h[v]);
        }
        if (a.weight) {
#pragma unroll
            for (int v = 0; v < V; ++v) h[v] = fmaf(tanhf(a.alpha * h[v]), w[v], b[v]);
        }
    };

    if constexpr (HIST == 0) {
        const int i = blockIdx.y * ROWS + row;
        if (!in || i >= (a.rows ? a.n_rows : a.n_tokens)) return;
        int t = i;
        if (a.rows) {
            t = a.rows[i];
            if (t < 0 || t >= a.n_tokens) {
                if (c0 == 0) atomicOr(a.err, QF_ERR_ROW_RANGE);
                t = 0;
            }
        }
        float h[V];
        value(t, !a.rows, h);
        if (a.weight) Channels<T, V>::store(a.z + (size_t)i * a.width + c0, h);
        else Channels<float, V>::store(a.u_out + (size_t)i * a.width + c0, h);
    } else {
        const int begin = a.cu_q[blockIdx.z], len = a.cu_q[blockIdx.z + 1] - begin, slot = a.slots[blockIdx.z];
        const int kept = a.n_taps - 1;
        float* rows = (slot >= 0 && in) ? a.state + slot * a.slot_stride + a.offset + c0 : nullptr;
        for (int first = blockIdx.y * OWN, buf = 0; first < len; first += gridDim.y * OWN, buf ^= 1) {   // (the same for the whole block)
            const int at = first - HIST + row;   // this thread's token, counted from the sequence's first of the step
            float h[V];
#pragma unroll
            for (int v = 0; v < V; ++v) h[v] = 0.f;
            if (in && at < len) {
                if (at >= 0 && row >= HIST - kept) {
                    value(begin + at, row >= HIST, h);
                } else if (at < 0 && rows && kept + at >= 0) {   // (before the step: the state's row, the newest last)
                    Channels<float, V>::load(rows + (size_t)(kept + at) * a.width, h);
                }
            }
            Channels<float, V>::store(&h_s[buf][row][group * V], h);
            __syncthreads();   // the tile's h are there; and nobody still reads the tile before the last
            if (row >= HIST && in && at < len) {
                float z[V];
#pragma unroll
                for (int v = 0; v < V; ++v) z[v] = 0.f;
#pragma unroll
                for (int j = 0; j < HIST; ++j) {
                    float before[V], f[V];
                    Channels<float, V>::load(&h_s[buf][row - HIST + j][group * V], before);
                    Channels<float, V>::load(&f_s[j][group * V], f);
#pragma unroll
                    for (int v = 0; v < V; ++v) z[v] = fmaf(f[v], before[v], z[v]);
                }
                float f[V];
                Channels<float, V>::load(&f_s[HIST][group * V], f);
#pragma unroll
                for (int v = 0; v < V; ++v) z[v] = h[v] + fmaf(f[v], h[v], z[v]);
                Channels<T, V>::store(a.z + (size_t)(begin + at) * a.width + c0, z);
            }
            if (first == 0 && rows && row < kept) {
                // the sequence's last `kept` values: in shared memory if it ends in this tile, else worked out again
                const int back = len - kept + row;
                float last[V];
                if (len <= OWN) Channels<float, V>::load(&h_s[buf][HIST + back][group * V], last);
                else value(begin + back, false, last);
                Channels<float, V>::store(rows + (size_t)row * a.width, last);
            }
        }
    }
}

template <typename T, int V, int NS, int HIST, int ROWS>
static int launch_streams(const StreamsArgs<T>& a, int n_seqs, int max_q_len, cudaStream_t stream) {
    constexpr int OWN = ROWS - HIST, CHANNELS = ST_THREADS / ROWS * V;
    const long long longest = HIST > 0 ? max_q_len : (a.rows ? a.n_rows : a.n_tokens);
    const long long tiles = (longest + OWN - 1) / OWN;
    const int columns = (a.width + CHANNELS - 1) / CHANNELS;
    long long down = tiles;
    if (HIST > 0) {   // a block walks several tiles when there are more than the SMs hold at once: its coefficients stay
        const long long held = (NS <= 4 ? 4ll : 2ll) * qf_sm_count() / ((long long)columns * n_seqs);
        if (held >= 1 && down > held) down = (down + (down + held - 1) / held - 1) / ((down + held - 1) / held);
        else if (held < 1) down = 1;
    }
    const dim3 grid(columns, (unsigned)down, HIST > 0 ? n_seqs : 1);
    if (down > 65535 || grid.z > 65535) return (int)cudaErrorInvalidValue;
    return (int)launch_pdl(streams_kernel<T, V, NS, HIST, ROWS>, grid, dim3(ST_THREADS), 0, stream, a);
}

template <typename T, int V, int NS>
static int launch_taps(const StreamsArgs<T>& a, int n_seqs, int max_q_len, cudaStream_t stream) {
    if (!a.taps) return launch_streams<T, V, NS, 0, 4>(a, n_seqs, max_q_len, stream);
    // one token per sequence: the three before it and itself, each a thread's
    if (max_q_len == 1) return launch_streams<T, V, NS, 3, 4>(a, n_seqs, max_q_len, stream);
    return launch_streams<T, V, NS, 3, 32>(a, n_seqs, max_q_len, stream);
}

template <typename T>
static int launch(const StreamsArgs<T>& a, int n_seqs, int max_q_len, cudaStream_t stream) {
    const uintptr_t all = (uintptr_t)a.src | (uintptr_t)a.dst | (uintptr_t)a.y | (uintptr_t)a.weight | (uintptr_t)a.bias | (uintptr_t)a.z |
                          (uintptr_t)a.u_out | (uintptr_t)a.state;
    const bool wide = a.width % 4 == 0 && all % 16 == 0 && (a.src_row | a.src_stream | a.slot_stride | a.offset) % 4 == 0;
    if (a.taps && a.n_taps > 4) return launch_streams<T, 1, 8, 15, 32>(a, n_seqs, max_q_len, stream);   // long filters: one form for all
#define QF_STREAMS(NS) return wide ? launch_taps<T, 4, NS>(a, n_seqs, max_q_len, stream) : launch_taps<T, 1, NS>(a, n_seqs, max_q_len, stream)
    if (a.n <= 2) QF_STREAMS(2);
    if (a.n <= 4) QF_STREAMS(4);
    QF_STREAMS(8);
#undef QF_STREAMS
}

template <typename T>
static int dispatch(const float* src, long long src_row, long long src_stream, float* dst, const void* y, const int* dest, int top,
                    const float* row_weight, const float* mix, const float* out_w, const float* in_w, const void* weight,
                    const void* bias, float alpha, void* z, float* u_out, const int* rows, int n_rows, int n_tokens, const float* taps,
                    int n_taps, const int* cu_q, const int* slots, int n_seqs, int max_q_len, float* state, long long slot_stride,
                    long long offset, int n, int width, int* err, cudaStream_t stream) {
    return launch<T>(StreamsArgs<T>{src, src_row, src_stream, dst, (const T*)y, dest, top, row_weight, mix, out_w, in_w, (const T*)weight,
                                    (const T*)bias, alpha, (T*)z, u_out, rows, n_rows, n_tokens, taps, n_taps, cu_q, slots, state,
                                    slot_stride, offset, n, width, err},
                     n_seqs, max_q_len, stream);
}

// See the top of the file and `ops.streams_norm`. n: 1 to 8 streams; n_taps: 1 to 16, a filter of one tap keeps nothing.
QF_EXPORT int qf_streams_norm(int is_bf16, const float* src, long long src_row, long long src_stream, float* dst, const void* y,
                              const int* dest, int top, const float* row_weight, const float* mix, const float* out_w,
                              const float* in_w, const void* weight, const void* bias, float alpha, void* z, float* u_out,
                              const int* rows, int n_rows, int n_tokens, const float* taps, int n_taps, const int* cu_q,
                              const int* slots, int n_seqs, int max_q_len, float* state, long long slot_stride, long long offset,
                              int n, int width, int* err, cudaStream_t stream) {
    if (n_tokens <= 0 || width <= 0 || (rows && n_rows <= 0)) return 0;
    if (n < 1 || n > 8 || (y && (!mix || !out_w)) || (weight ? (!bias || !z) : (!u_out || taps != nullptr)) ||
        (taps && (n_taps < 1 || n_taps > 16 || rows || n_seqs <= 0 || max_q_len <= 0 || (n_taps > 1 && !state))) || (dst && rows) ||
        (const float*)dst == src)
        return (int)cudaErrorInvalidValue;
    return is_bf16 ? dispatch<bf16>(src, src_row, src_stream, dst, y, dest, top, row_weight, mix, out_w, in_w, weight, bias, alpha, z,
                                    u_out, rows, n_rows, n_tokens, taps, n_taps, cu_q, slots, n_seqs, max_q_len, state, slot_stride,
                                    offset, n, width, err, stream)
                   : dispatch<float>(src, src_row, src_stream, dst, y, dest, top, row_weight, mix, out_w, in_w, weight, bias, alpha, z,
                                     u_out, rows, n_rows, n_tokens, taps, n_taps, cu_q, slots, n_seqs, max_q_len, state, slot_stride,
                                     offset, n, width, err, stream);
}
