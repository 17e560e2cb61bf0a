// A short causal convolution over time on each channel of a projection, y_t = sum_j w[:, j] u_(t - n + 1 + j) with n taps per
// channel, and what a mixer does with its result right away.  The n - 1 inputs before a step's first row come from the sequence's
// state (32-bit, zeros at a sequence's start), which keeps the step's last n - 1 inputs.
//
//   heads     u holds query, key and value heads: after the convolution the first `rot` numbers of a query or key head turn by
//             position (pairs (2i, 2i + 1), angle fp32(pos) * freq[i]; optional), and the head is divided by its root mean square
//             (optional; in this order).  Queries go to rows of their own, keys and values to the cache.  A warp owns a head and walks up to eight rows with
//             their inputs in registers, so a row is read once for all its taps; the rows' cosines and sines are made once per
//             block and shared by its heads.
//   rows      silu(conv + bias) as rows of their own; a thread owns two neighbouring channels and walks up to sixteen rows.
//   history   the state takes the last n - 1 inputs of every sequence (after the kernels above have read it).  In a step that brings
//             one token per sequence they move it on themselves: the thread that convolves a channel is the only one to touch it.
//
// All arithmetic is fp32; inputs are read, and results stored, in the dtypes of the rows.
#include <math.h>

#include "common.cuh"

FR_EXPORT const char* short_conv_last_error() { return fr_error_text; }

typedef __nv_bfloat16 bf16;

namespace {

constexpr int PAGE_ROWS = 64;

struct ConvArgs {
    const void* x;           // [rows][ld]: the channels at `off`, one after another
    FrVec taps_w;            // [channels][taps]
    float* state;            // [slots][state_stride], history [taps - 1][channels] at hist_off
    long long state_stride, hist_off;
    const int* row_seq;
    const int* seq_start;
    const int* seq_qlen;
    const int* seq_slots;
    int ld, off, channels, taps, rows;
    int shift;               // 1: every sequence brings one row, and its history moves on here
    int pairs;               // rows are read, and written, two channels at a time
    // heads
    const int* row_pos;
    const float* freq;       // [rot / 2]; null: no rotation
    void* q_out;             // [rows][heads * dim]
    void* k_pool;
    void* v_pool;
    const int* block_table;
    int table_width, heads, kv_heads, dim, vdim, rot, norm;
    float eps;
    // rows
    FrVec bias;              // [channels]; p null: none
    void* out;               // [rows][channels]
};

template <typename T> struct Two;
template <> struct Two<float> { typedef float2 type; };
template <> struct Two<bf16> { typedef uint32_t type; };
__device__ __forceinline__ float2 unpack(float2 v) { return v; }
__device__ __forceinline__ float2 unpack(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }
__device__ __forceinline__ void pack(float a, float b, float2& v) { v = make_float2(a, b); }
__device__ __forceinline__ void pack(float a, float b, uint32_t& v) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    v = *(const uint32_t*)&h;
}
// two neighbouring channels (the second only if `two`)
template <typename T>
__device__ __forceinline__ typename Two<T>::type load_two(const T* p, bool two, int whole) {
    if (whole) return *(const typename Two<T>::type*)p;
    typename Two<T>::type v;
    pack(fr_load(p), two ? fr_load(p + 1) : 0.f, v);
    return v;
}
template <typename T>
__device__ __forceinline__ void store_two(T* p, float a, float b, bool two, int whole) {
    if (whole) {
        typename Two<T>::type v;
        pack(a, b, v);
        *(typename Two<T>::type*)p = v;
        return;
    }
    fr_store(p, a);
    if (two) fr_store(p + 1, b);
}

// Taps of two neighbouring channels, the last one the present row's.  TAPS 4 serves up to four taps (missing ones count zero).
template <int TAPS>
struct Weights {
    float a[TAPS], b[TAPS];
    __device__ __forceinline__ void load(const ConvArgs& p, int c, bool two) {
        if constexpr (TAPS == 4) {
            if (p.taps == 4 && two) {
                p.taps_w.four(c * 4, a);
                p.taps_w.four(c * 4 + 4, b);
                return;
            }
        }
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const int at = j - (TAPS - p.taps);
            a[j] = at >= 0 ? p.taps_w.at(c * p.taps + at) : 0.f;
            b[j] = at >= 0 && two ? p.taps_w.at((c + 1) * p.taps + at) : 0.f;
        }
    }
};

// The convolution of channels c, c + 1 at a row whose inputs are in `raw` (raw[TAPS - 1] the row's own), where `known` rows before it belong
// to its sequence's part of this step; older ones are in the history.
template <typename T, int TAPS>
__device__ __forceinline__ float2 convolve(const ConvArgs& p, const typename Two<T>::type (&raw)[TAPS], const Weights<TAPS>& w, int known, const float* hist, int c, bool two) {
    float2 acc = make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        const int back = TAPS - 1 - j;
        if (back >= p.taps) continue;
        float2 u;
        if (back <= known) u = unpack(raw[j]);
        else {
            const float* at = hist + (size_t)(p.taps - 1 + known - back) * p.channels + c;
            u = make_float2(at[0], two ? at[1] : 0.f);
        }
        acc.x = fmaf(w.a[j], u.x, acc.x);
        acc.y = fmaf(w.b[j], u.y, acc.y);
    }
    return acc;
}

// any number of taps, nothing kept in registers
template <typename T>
__device__ __forceinline__ float2 convolve_any(const ConvArgs& p, const T* x, int row, int known, const float* hist, int c, bool two) {
    float2 acc = make_float2(0.f, 0.f);
    for (int j = 0; j < p.taps; ++j) {
        const int back = p.taps - 1 - j;
        float2 u;
        if (back <= known) {
            const T* at = x + (size_t)(row - back) * p.ld + p.off + c;
            u = make_float2(fr_load(at), two ? fr_load(at + 1) : 0.f);
        } else {
            const float* at = hist + (size_t)(p.taps - 1 + known - back) * p.channels + c;
            u = make_float2(at[0], two ? at[1] : 0.f);
        }
        acc.x = fmaf(p.taps_w.at(c * p.taps + j), u.x, acc.x);
        if (two) acc.y = fmaf(p.taps_w.at((c + 1) * p.taps + j), u.y, acc.y);
    }
    return acc;
}

// one row per sequence: the history of channels c, c + 1 drops its oldest input and takes the present one
__device__ __forceinline__ void move_on(const ConvArgs& p, float* hist, int c, bool two, float2 u) {
    for (int j = 0; j + 1 < p.taps; ++j) {
        float* at = hist + (size_t)j * p.channels + c;
        const bool last = j + 2 >= p.taps;
        at[0] = last ? u.x : at[p.channels];
        if (two) at[1] = last ? u.y : at[p.channels + 1];
    }
}

// ------------------------------------------------------------------ heads
constexpr int HEAD_WARPS = 8;

// PAIRS: pairs of channels per lane; TAPS 0: convolve_any; R rows per tile
template <typename T, int PAIRS, int TAPS, int R>
__global__ void __launch_bounds__(HEAD_WARPS * 32) conv_heads_kernel(ConvArgs p) {
    constexpr int K = TAPS > 0 ? TAPS : 1;
    __shared__ float2 turn[R][128];          // cosine and sine of every row's angles
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row0 = blockIdx.x * R, n = min(R, p.rows - row0);
    const int item = blockIdx.y * HEAD_WARPS + warp;
    const int half = p.freq != nullptr ? p.rot / 2 : 0;
    fr_pdl_wait();
    fr_pdl_launch();
    if (half > 0 && (int)blockIdx.y * HEAD_WARPS < p.heads + p.kv_heads) {
        for (int idx = threadIdx.x; idx < n * half; idx += HEAD_WARPS * 32) {
            const int r = idx / half, i = idx - r * half;
            float s, c;
            sincosf((float)p.row_pos[row0 + r] * p.freq[i], &s, &c);
            turn[r][i] = make_float2(c, s);
        }
        __syncthreads();
    }
    if (item >= p.heads + 2 * p.kv_heads) return;
    const bool is_q = item < p.heads, is_v = item >= p.heads + p.kv_heads;
    const int g = is_q ? item : is_v ? item - p.heads - p.kv_heads : item - p.heads;
    const int width = is_v ? p.vdim : p.dim;
    const int c0 = is_v ? (p.heads + p.kv_heads) * p.dim + g * p.vdim : item * p.dim;       // queries, then keys, then values
    const T* x = (const T*)p.x;
    typedef typename Two<T>::type two_t;
    two_t raw[PAIRS][R + K - 1];
    Weights<K> w[PAIRS];
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
        const int d = 2 * (lane + 32 * i);
        if constexpr (TAPS > 0) {
            if (d >= width) continue;
#pragma unroll
            for (int k = 0; k < R + K - 1; ++k) {
                const int row = row0 + k - (K - 1);
                if (row >= 0 && row < p.rows && k < n + K - 1) raw[i][k] = load_two(x + (size_t)row * p.ld + p.off + c0 + d, d + 1 < width, p.pairs);
                else pack(0.f, 0.f, raw[i][k]);
            }
            w[i].load(p, c0 + d, d + 1 < width);
        }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= n) break;
        const int row = row0 + r, seq = p.row_seq[row];
        if (seq < 0) continue;
        const int known = row - p.seq_start[seq], pos = p.row_pos[row];
        float* hist = p.state + (size_t)p.seq_slots[seq] * p.state_stride + p.hist_off;
        float2 v[PAIRS];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            const int pair = lane + 32 * i, d = 2 * pair;
            v[i] = make_float2(0.f, 0.f);
            if (d >= width) continue;
            const bool two = d + 1 < width;
            float2 own;
            if constexpr (TAPS > 0) {
                two_t at[K];
#pragma unroll
                for (int k = 0; k < K; ++k) at[k] = raw[i][r + k];
                v[i] = convolve<T, K>(p, at, w[i], known, hist, c0 + d, two);
                own = unpack(at[K - 1]);
            } else {
                v[i] = convolve_any(p, x, row, known, hist, c0 + d, two);
                own = unpack(load_two(x + (size_t)row * p.ld + p.off + c0 + d, two, p.pairs));
            }
            if (p.shift) move_on(p, hist, c0 + d, two, own);
            if (!is_v && pair < half) {
                const float2 t = turn[r][pair];
                const float a = v[i].x, b = v[i].y;
                fr_rotate(a, b, t.x, t.y, v[i].x, v[i].y);
            }
            ss = fmaf(v[i].x, v[i].x, ss);
            ss = fmaf(v[i].y, v[i].y, ss);
        }
        float inv = 1.f;
        if (!is_v && p.norm) inv = 1.0f / sqrtf(fr_warp_sum(ss) / (float)p.dim + p.eps);
        T* dst;
        if (is_q) dst = (T*)p.q_out + (size_t)row * p.heads * p.dim + (size_t)g * p.dim;
        else {
            const size_t at = (size_t)p.block_table[(size_t)seq * p.table_width + pos / PAGE_ROWS] * PAGE_ROWS + pos % PAGE_ROWS;
            dst = (is_v ? (T*)p.v_pool : (T*)p.k_pool) + (at * p.kv_heads + g) * width;
        }
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            const int d = 2 * (lane + 32 * i);
            if (d < width) store_two(dst + d, v[i].x * inv, v[i].y * inv, d + 1 < width, p.pairs);
        }
    }
}

template <typename T, int PAIRS>
int launch_heads(const ConvArgs& p, cudaStream_t stream) {
    const int items = p.heads + 2 * p.kv_heads;
    // few rows: one per tile, so that the heads of every row have warps of their own
    const bool single = p.shift || (long long)p.rows * items < (long long)fr_sm_count() * 64;
    const dim3 grid(single ? p.rows : (p.rows + 7) / 8, (items + HEAD_WARPS - 1) / HEAD_WARPS), block(HEAD_WARPS * 32);
    if (p.taps > 4) FR_CUDA(fr_launch(conv_heads_kernel<T, PAIRS, 0, 1>, dim3(p.rows, grid.y), block, 0, stream, p));
    else if (single) FR_CUDA(fr_launch(conv_heads_kernel<T, PAIRS, 4, 1>, grid, block, 0, stream, p));
    else FR_CUDA(fr_launch(conv_heads_kernel<T, PAIRS, 4, 8>, grid, block, 0, stream, p));
    FR_CHECK_LAUNCH("short_conv heads");
    return FR_OK;
}

// ------------------------------------------------------------------ rows
constexpr int ROW_THREADS = 128;

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

template <typename TI, typename TO, int TAPS, int R>
__global__ void __launch_bounds__(ROW_THREADS) conv_rows_kernel(ConvArgs p) {
    constexpr int K = TAPS > 0 ? TAPS : 1;
    const int c = 2 * (blockIdx.y * ROW_THREADS + threadIdx.x);
    const int row0 = blockIdx.x * R, n = min(R, p.rows - row0);
    fr_pdl_wait();
    fr_pdl_launch();
    if (c >= p.channels) return;
    const bool two = c + 1 < p.channels;
    const TI* x = (const TI*)p.x;
    typedef typename Two<TI>::type two_t;
    two_t raw[R + K - 1];
    Weights<K> w;
    if constexpr (TAPS > 0) {
#pragma unroll
        for (int k = 0; k < R + K - 1; ++k) {
            const int row = row0 + k - (K - 1);
            if (row >= 0 && row < p.rows && k < n + K - 1) raw[k] = load_two(x + (size_t)row * p.ld + p.off + c, two, p.pairs);
            else pack(0.f, 0.f, raw[k]);
        }
        w.load(p, c, two);
    }
    const float b0 = p.bias.p != nullptr ? p.bias.at(c) : 0.f, b1 = p.bias.p != nullptr && two ? p.bias.at(c + 1) : 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= n) break;
        const int row = row0 + r, seq = p.row_seq[row];
        if (seq < 0) continue;
        const int known = row - p.seq_start[seq];
        float* hist = p.state + (size_t)p.seq_slots[seq] * p.state_stride + p.hist_off;
        float2 v, own;
        if constexpr (TAPS > 0) {
            two_t at[K];
#pragma unroll
            for (int k = 0; k < K; ++k) at[k] = raw[r + k];
            v = convolve<TI, K>(p, at, w, known, hist, c, two);
            own = unpack(at[K - 1]);
        } else {
            v = convolve_any(p, x, row, known, hist, c, two);
            own = unpack(load_two(x + (size_t)row * p.ld + p.off + c, two, p.pairs));
        }
        if (p.shift) move_on(p, hist, c, two, own);
        store_two((TO*)p.out + (size_t)row * p.channels + c, silu_f(v.x + b0), silu_f(v.y + b1), two, p.pairs);
    }
}

template <typename TI, typename TO>
int launch_rows(const ConvArgs& p, cudaStream_t stream) {
    const int blocks = (p.channels / 2 + ROW_THREADS) / ROW_THREADS;
    const bool single = p.shift || (long long)p.rows * blocks < (long long)fr_sm_count() * 16;
    if (p.taps > 4) FR_CUDA(fr_launch(conv_rows_kernel<TI, TO, 0, 1>, dim3(p.rows, blocks), dim3(ROW_THREADS), 0, stream, p));
    else if (single) FR_CUDA(fr_launch(conv_rows_kernel<TI, TO, 4, 1>, dim3(p.rows, blocks), dim3(ROW_THREADS), 0, stream, p));
    else FR_CUDA(fr_launch(conv_rows_kernel<TI, TO, 4, 16>, dim3((p.rows + 15) / 16, blocks), dim3(ROW_THREADS), 0, stream, p));
    FR_CHECK_LAUNCH("short_conv rows");
    return FR_OK;
}

// ------------------------------------------------------------------ eight channels per thread
// The usual shapes (up to four taps, rows in whole 16-byte pieces; heads of a power of two): a thread owns eight channels of a run of
// rows, asks for all of its rows at once and keeps the last three inputs in registers, so an input is read, and widened, once for all
// its taps.
template <typename T> struct Eight;
template <> struct Eight<float> { float4 a, b; };
template <> struct Eight<bf16> { uint4 a; };
__device__ __forceinline__ void load_eight(const float* p, Eight<float>& v) { v.a = *(const float4*)p; v.b = *(const float4*)(p + 4); }
__device__ __forceinline__ void load_eight(const bf16* p, Eight<bf16>& v) { v.a = *(const uint4*)p; }
__device__ __forceinline__ void widen(const Eight<float>& v, float (&f)[8]) {
    f[0] = v.a.x; f[1] = v.a.y; f[2] = v.a.z; f[3] = v.a.w; f[4] = v.b.x; f[5] = v.b.y; f[6] = v.b.z; f[7] = v.b.w;
}
__device__ __forceinline__ void widen(const Eight<bf16>& v, float (&f)[8]) {
    const uint32_t w[4] = {v.a.x, v.a.y, v.a.z, v.a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void store_eight(float* p, const float (&f)[8]) {
    *(float4*)p = make_float4(f[0], f[1], f[2], f[3]);
    *(float4*)(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void store_eight(bf16* p, const float (&f)[8]) {
    uint4 r;
    pack(f[0], f[1], r.x);
    pack(f[2], f[3], r.y);
    pack(f[4], f[5], r.z);
    pack(f[6], f[7], r.w);
    *(uint4*)p = r;
}

// What a row means to the kernels below: rows of its sequence before it in this step (-1: a dead row), its slot, and where its key and
// value lie in the cache.  A block makes it once for each of its rows, ahead of the wait for the kernel before (the step's geometry is
// final by then).
struct RowPlace {
    int known, slot, to;
};
__device__ __forceinline__ RowPlace place_of(const ConvArgs& p, int row) {
    RowPlace r;
    const int seq = p.row_seq[row];
    r.known = seq >= 0 ? row - p.seq_start[seq] : -1;
    r.slot = seq >= 0 ? p.seq_slots[seq] : 0;
    r.to = 0;
    if (seq >= 0 && p.block_table != nullptr) {
        const int pos = p.row_pos[row];
        r.to = p.block_table[(size_t)seq * p.table_width + pos / PAGE_ROWS] * PAGE_ROWS + pos % PAGE_ROWS;
    }
    return r;
}
// 1 / sqrt(mean square + eps): exact for 32-bit rows, the hardware's reciprocal square root (its error is far below the rounding that
// follows) for rows in bf16
template <typename T> __device__ __forceinline__ float inverse_rms(float mean_square_eps);
template <> __device__ __forceinline__ float inverse_rms<float>(float v) { return 1.0f / sqrtf(v); }
template <> __device__ __forceinline__ float inverse_rms<bf16>(float v) { return rsqrtf(v); }

template <typename T>
struct Walk {
    float w[4][8];                   // taps, the last one the present row's; missing ones count zero
    float back[3][8];                // the inputs three, two and one row before the present one
    __device__ __forceinline__ void load_taps(const ConvArgs& p, int c) {
        if (p.taps == 4) {
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                float v[4];
                p.taps_w.four((c + i) * 4, v);
#pragma unroll
                for (int j = 0; j < 4; ++j) w[j][i] = v[j];
            }
            return;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int i = 0; i < 8; ++i) w[j][i] = j >= 4 - p.taps ? p.taps_w.at((c + i) * p.taps + j - (4 - p.taps)) : 0.f;
    }
    // the inputs before `row`: rows of this step as far as its sequence has them, then the sequence's history
    __device__ __forceinline__ void begin(const ConvArgs& p, const T* x, int row, int known, const float* hist, int c) {
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            const int b = 3 - k;
            if (b <= known) {
                Eight<T> v;
                load_eight(x + (size_t)(row - b) * p.ld + p.off + c, v);
                widen(v, back[k]);
            } else if (b <= p.taps - 1 + known && b < p.taps) {
                Eight<float> v;
                load_eight(hist + (size_t)(p.taps - 1 + known - b) * p.channels + c, v);
                widen(v, back[k]);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) back[k][i] = 0.f;
            }
        }
    }
    // the convolution at a row whose input is `u`
    __device__ __forceinline__ void step(const float (&u)[8], float (&y)[8]) const {
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(w[3][i], u[i], fmaf(w[2][i], back[2][i], fmaf(w[1][i], back[1][i], w[0][i] * back[0][i])));
    }
    __device__ __forceinline__ void take(const float (&u)[8]) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            back[0][i] = back[1][i];
            back[1][i] = back[2][i];
            back[2][i] = u[i];
        }
    }
    // after take(): the last taps - 1 inputs are the sequence's history
    __device__ __forceinline__ void leave(const ConvArgs& p, float* hist, int c) const {
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            const int j = k - (3 - (p.taps - 1));
            if (j >= 0) store_eight(hist + (size_t)j * p.channels + c, back[k]);
        }
    }
};

constexpr int VEC_THREADS = 128;

// LANES: threads of a head (its channels / 8)
template <typename T, int LANES, int R>
__global__ void __launch_bounds__(VEC_THREADS) conv_heads_vec_kernel(ConvArgs p) {
    __shared__ float2 turn[R][128];          // cosine and sine of every row's angles
    __shared__ RowPlace place[R];
    const int row0 = blockIdx.x * R, n = min(R, p.rows - row0);
    const int c = 8 * (blockIdx.y * VEC_THREADS + threadIdx.x);
    const int half = p.freq != nullptr ? p.rot / 2 : 0, nq = p.heads * p.dim, nk = p.kv_heads * p.dim, nv = p.kv_heads * p.vdim;
    const bool live = c < nq + nk + nv, is_q = c < nq, is_v = c >= nq + nk;
    Walk<T> walk;
    if ((int)threadIdx.x < n) place[threadIdx.x] = place_of(p, row0 + threadIdx.x);
    if (live) walk.load_taps(p, c);
    if (half > 0 && 8 * (int)blockIdx.y * VEC_THREADS < nq + nk) {
        for (int idx = threadIdx.x; idx < n * half; idx += VEC_THREADS) {
            const int r = idx / half, i = idx - r * half;
            float s, co;
            sincosf((float)p.row_pos[row0 + r] * p.freq[i], &s, &co);
            turn[r][i] = make_float2(co, s);
        }
    }
    fr_pdl_wait();
    fr_pdl_launch();
    __syncthreads();
    if (!live) return;                       // whole heads: a head's lanes are all live or none
    const T* x = (const T*)p.x;
    Eight<T> raw[R];
#pragma unroll
    for (int r = 0; r < R; ++r)
        if (r < n) load_eight(x + (size_t)(row0 + r) * p.ld + p.off + c, raw[r]);
    const int d = is_v ? 0 : c % p.dim;
    const float inv_dim = 1.0f / (float)p.dim;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= n) break;
        const int row = row0 + r;
        const RowPlace at = place[r];
        if (at.known < 0) continue;          // (a dead row: the walk begins anew at the next sequence's first row)
        float* hist = p.state + (size_t)at.slot * p.state_stride + p.hist_off;
        if (r == 0 || at.known == 0) walk.begin(p, x, row, at.known, hist, c);
        float u[8], y[8];
        widen(raw[r], u);
        walk.step(u, y);
        walk.take(u);
        if (p.shift) walk.leave(p, hist, c);
        if (!is_v) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (d / 2 + i < half) {
                    const float2 t = turn[r][d / 2 + i];
                    const float a = y[2 * i], b = y[2 * i + 1];
                    fr_rotate(a, b, t.x, t.y, y[2 * i], y[2 * i + 1]);
                }
            }
            if (p.norm) {
                float ss = 0.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) ss = fmaf(y[i], y[i], ss);
                const unsigned lanes = LANES == 32 ? 0xffffffffu : ((1u << LANES) - 1u) << ((threadIdx.x & 31) / LANES * LANES);
#pragma unroll
                for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(lanes, ss, o);
                const float inv = inverse_rms<T>(fmaf(ss, inv_dim, p.eps));
#pragma unroll
                for (int i = 0; i < 8; ++i) y[i] *= inv;
            }
        }
        if (is_q) {
            store_eight((T*)p.q_out + (size_t)row * nq + c, y);
        } else {
            if (is_v) store_eight((T*)p.v_pool + (size_t)at.to * nv + (c - nq - nk), y);
            else store_eight((T*)p.k_pool + (size_t)at.to * nk + (c - nq), y);
        }
    }
}

template <typename T, int LANES>
int launch_heads_vec(const ConvArgs& p, cudaStream_t stream) {
    const int blocks = (p.channels / 8 + VEC_THREADS - 1) / VEC_THREADS;
    const bool single = p.shift || (long long)p.rows * blocks < (long long)fr_sm_count() * 8;
    if (single) FR_CUDA(fr_launch(conv_heads_vec_kernel<T, LANES, 1>, dim3(p.rows, blocks), dim3(VEC_THREADS), 0, stream, p));
    else FR_CUDA(fr_launch(conv_heads_vec_kernel<T, LANES, 8>, dim3((p.rows + 7) / 8, blocks), dim3(VEC_THREADS), 0, stream, p));
    FR_CHECK_LAUNCH("short_conv heads");
    return FR_OK;
}

// silu: exact for 32-bit rows; for rows about to be rounded to bf16 with the hardware's exponential and reciprocal
template <typename T> __device__ __forceinline__ float silu_to(float z);
template <> __device__ __forceinline__ float silu_to<float>(float z) { return z / (1.0f + expf(-z)); }
template <> __device__ __forceinline__ float silu_to<bf16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

template <typename TI, typename TO, int R>
__global__ void __launch_bounds__(VEC_THREADS) conv_rows_vec_kernel(ConvArgs p) {
    const int row0 = blockIdx.x * R, n = min(R, p.rows - row0);
    const int c = 8 * (blockIdx.y * VEC_THREADS + threadIdx.x);
    const bool live = c < p.channels;
    __shared__ RowPlace place[R];
    Walk<TI> walk;
    if ((int)threadIdx.x < n) place[threadIdx.x] = place_of(p, row0 + threadIdx.x);
    float bias[8];
    if (live) {
        walk.load_taps(p, c);
#pragma unroll
        for (int i = 0; i < 8; ++i) bias[i] = p.bias.p != nullptr ? p.bias.at(c + i) : 0.f;
    }
    fr_pdl_wait();
    fr_pdl_launch();
    __syncthreads();
    if (!live) return;
    const TI* x = (const TI*)p.x;
    Eight<TI> raw[R];
#pragma unroll
    for (int r = 0; r < R; ++r)
        if (r < n) load_eight(x + (size_t)(row0 + r) * p.ld + p.off + c, raw[r]);
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= n) break;
        const int row = row0 + r;
        const RowPlace at = place[r];
        if (at.known < 0) continue;
        float* hist = p.state + (size_t)at.slot * p.state_stride + p.hist_off;
        if (r == 0 || at.known == 0) walk.begin(p, x, row, at.known, hist, c);
        float u[8], y[8];
        widen(raw[r], u);
        walk.step(u, y);
        walk.take(u);
        if (p.shift) walk.leave(p, hist, c);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = silu_to<TO>(y[i] + bias[i]);
        store_eight((TO*)p.out + (size_t)row * p.channels + c, y);
    }
}

template <typename TI, typename TO>
int launch_rows_vec(const ConvArgs& p, cudaStream_t stream) {
    const int blocks = (p.channels / 8 + VEC_THREADS - 1) / VEC_THREADS;
    const bool single = p.shift || (long long)p.rows * blocks < (long long)fr_sm_count() * 8;
    if (single) FR_CUDA(fr_launch(conv_rows_vec_kernel<TI, TO, 1>, dim3(p.rows, blocks), dim3(VEC_THREADS), 0, stream, p));
    else FR_CUDA(fr_launch(conv_rows_vec_kernel<TI, TO, 8>, dim3((p.rows + 7) / 8, blocks), dim3(VEC_THREADS), 0, stream, p));
    FR_CHECK_LAUNCH("short_conv rows");
    return FR_OK;
}

// ------------------------------------------------------------------ history
template <typename T>
__global__ void __launch_bounds__(256) conv_history_kernel(ConvArgs p) {
    const int seq = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    const int r0 = p.seq_start[seq], n = p.seq_qlen[seq], keep = p.taps - 1;
    fr_pdl_wait();
    fr_pdl_launch();
    if (n <= 0 || c >= p.channels || p.row_seq[r0] < 0) return;
    float* hist = p.state + (size_t)p.seq_slots[seq] * p.state_stride + p.hist_off + c;
    const T* x = (const T*)p.x + p.off + c;
    for (int j = 0; j < keep; ++j) {                  // in this order no input is overwritten before it has moved
        const int idx = n - keep + j;                 // row of the step, counted from the sequence's first
        hist[(size_t)j * p.channels] = idx >= 0 ? fr_load(x + (size_t)(r0 + idx) * p.ld) : hist[(size_t)(j + n) * p.channels];
    }
}

int check(const ConvArgs& p, int n_seqs) {
    if (p.taps < 1 || p.channels < 1 || p.off < 0 || p.off + p.channels > p.ld) FR_REFUSE("short_conv: %d taps, channels %d .. %d of rows of %d", p.taps, p.off, p.off + p.channels, p.ld);
    if (p.state == nullptr || p.hist_off < 0 || p.hist_off + (long long)(p.taps - 1) * p.channels > p.state_stride)
        FR_REFUSE("short_conv: the state does not hold %d inputs of %d channels", p.taps - 1, p.channels);
    if (n_seqs > 65535) FR_REFUSE("short_conv: %d sequences", n_seqs);
    return FR_OK;
}

int history(const ConvArgs& p, int n_seqs, int dtype, cudaStream_t stream) {
    if (p.shift || p.taps < 2 || n_seqs <= 0) return FR_OK;
    const dim3 grid((p.channels + 255) / 256, n_seqs);
    if (dtype == FR_F32) FR_CUDA(fr_launch(conv_history_kernel<float>, grid, dim3(256), 0, stream, p));
    else FR_CUDA(fr_launch(conv_history_kernel<bf16>, grid, dim3(256), 0, stream, p));
    FR_CHECK_LAUNCH("short_conv history");
    return FR_OK;
}

}  // namespace

// x [rows][ld] of `dtype`: query heads, key heads and value heads one after another from column `off` on; taps [channels][taps] of
// w_dtype; freq [rot / 2] (null: no rotation); norm 1: every query and key head divided by sqrt(mean square + eps).  q_out [rows][heads * dim],
// pools of pages of 64 positions, all of `dtype`.  state [slots][state_stride] fp32, the history [taps - 1][channels] at hist_off.
// one_token 1: every sequence brings one row.
FR_EXPORT int short_conv_heads(const void* x, int ld, int off, const void* taps_w, int w_dtype, int taps, const float* freq, int rot, int norm, float eps,
                               void* q_out, void* k_pool, void* v_pool, const int* block_table, int table_width, int page, float* state,
                               long long state_stride, long long hist_off, const int* row_seq, const int* row_pos, const int* seq_start, const int* seq_qlen,
                               const int* seq_slots, int n_seqs, int rows, int heads, int kv_heads, int dim, int vdim, int one_token, int dtype,
                               cudaStream_t stream) {
    if (rows <= 0) return FR_OK;
    if (page != PAGE_ROWS) FR_REFUSE("short_conv: pages of %d positions (64)", page);
    if (heads <= 0 || kv_heads <= 0 || dim <= 0 || dim > 256 || vdim <= 0 || vdim > 256) FR_REFUSE("short_conv: %d and %d heads of %d and %d channels (1 to 256)", heads, kv_heads, dim, vdim);
    if (freq != nullptr && (rot <= 0 || rot % 2 || rot > dim)) FR_REFUSE("short_conv: %d rotated numbers in heads of %d", rot, dim);
    if (heads + 2 * kv_heads > 65535 * HEAD_WARPS) FR_REFUSE("short_conv: %d heads", heads);
    ConvArgs p{};
    p.x = x; p.taps_w = FrVec{taps_w, w_dtype}; p.state = state; p.state_stride = state_stride; p.hist_off = hist_off; p.row_seq = row_seq;
    p.seq_start = seq_start; p.seq_qlen = seq_qlen; p.seq_slots = seq_slots; p.ld = ld; p.off = off; p.channels = (heads + kv_heads) * dim + kv_heads * vdim;
    p.taps = taps; p.rows = rows; p.shift = one_token; p.row_pos = row_pos; p.freq = freq; p.q_out = q_out; p.k_pool = k_pool; p.v_pool = v_pool;
    p.block_table = block_table; p.table_width = table_width; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.rot = rot;
    p.norm = norm; p.eps = eps;
    const int rc = check(p, n_seqs);
    if (rc != FR_OK) return rc;
    const uintptr_t at = (uintptr_t)x | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool;
    p.pairs = ((ld | off | dim | vdim) & 1) == 0 && (at & 7) == 0;
    const int big = dim > vdim ? dim : vdim;
    int done;
    const bool eights = taps <= 4 && ((ld | off | vdim) & 7) == 0 && ((at | (uintptr_t)state) & 15) == 0 && ((state_stride | hist_off | p.channels) & 3) == 0 &&
                        (rot <= 256 || freq == nullptr);
    if (eights && (dim == 32 || dim == 64 || dim == 128 || dim == 256) && (dtype == FR_F32 || dtype == FR_BF16)) {
        const bool wide = dtype == FR_F32;
        if (dim == 32) done = wide ? launch_heads_vec<float, 4>(p, stream) : launch_heads_vec<bf16, 4>(p, stream);
        else if (dim == 64) done = wide ? launch_heads_vec<float, 8>(p, stream) : launch_heads_vec<bf16, 8>(p, stream);
        else if (dim == 128) done = wide ? launch_heads_vec<float, 16>(p, stream) : launch_heads_vec<bf16, 16>(p, stream);
        else done = wide ? launch_heads_vec<float, 32>(p, stream) : launch_heads_vec<bf16, 32>(p, stream);
        return done != FR_OK ? done : history(p, n_seqs, dtype, stream);
    }
    if (dtype == FR_F32) done = big <= 64 ? launch_heads<float, 1>(p, stream) : big <= 128 ? launch_heads<float, 2>(p, stream) : launch_heads<float, 4>(p, stream);
    else if (dtype == FR_BF16) done = big <= 64 ? launch_heads<bf16, 1>(p, stream) : big <= 128 ? launch_heads<bf16, 2>(p, stream) : launch_heads<bf16, 4>(p, stream);
    else FR_REFUSE("short_conv: unknown dtype %d", dtype);
    return done != FR_OK ? done : history(p, n_seqs, dtype, stream);
}

// x [rows][ld] of in_dtype, its channels from column `off` on; bias [channels] of b_dtype (null: none); out [rows][channels] of out_dtype =
// silu(conv + bias).  The rest as above.
FR_EXPORT int short_conv_rows(const void* x, int ld, int off, int channels, const void* taps_w, int w_dtype, int taps, const void* bias, int b_dtype,
                              void* out, float* state, long long state_stride, long long hist_off, const int* row_seq, const int* seq_start,
                              const int* seq_qlen, const int* seq_slots, int n_seqs, int rows, int one_token, int in_dtype, int out_dtype, cudaStream_t stream) {
    if (rows <= 0) return FR_OK;
    ConvArgs p{};
    p.x = x; p.taps_w = FrVec{taps_w, w_dtype}; p.state = state; p.state_stride = state_stride; p.hist_off = hist_off; p.row_seq = row_seq;
    p.seq_start = seq_start; p.seq_qlen = seq_qlen; p.seq_slots = seq_slots; p.ld = ld; p.off = off; p.channels = channels; p.taps = taps;
    p.rows = rows; p.shift = one_token; p.bias = FrVec{bias, b_dtype}; p.out = out;
    const int rc = check(p, n_seqs);
    if (rc != FR_OK) return rc;
    if (channels > 65535 * ROW_THREADS) FR_REFUSE("short_conv: %d channels", channels);
    p.pairs = ((ld | off | channels) & 1) == 0 && (((uintptr_t)x | (uintptr_t)out) & 7) == 0;
    int done;
    if (taps <= 4 && ((ld | off | channels) & 7) == 0 && (((uintptr_t)x | (uintptr_t)out | (uintptr_t)state) & 15) == 0 && ((state_stride | hist_off) & 3) == 0) {
        if (in_dtype == FR_F32 && out_dtype == FR_F32) done = launch_rows_vec<float, float>(p, stream);
        else if (in_dtype == FR_F32 && out_dtype == FR_BF16) done = launch_rows_vec<float, bf16>(p, stream);
        else if (in_dtype == FR_BF16 && out_dtype == FR_BF16) done = launch_rows_vec<bf16, bf16>(p, stream);
        else FR_REFUSE("short_conv: rows of dtype %d from inputs of dtype %d", out_dtype, in_dtype);
        return done != FR_OK ? done : history(p, n_seqs, in_dtype, stream);
    }
    if (in_dtype == FR_F32 && out_dtype == FR_F32) done = launch_rows<float, float>(p, stream);
    else if (in_dtype == FR_F32 && out_dtype == FR_BF16) done = launch_rows<float, bf16>(p, stream);
    else if (in_dtype == FR_BF16 && out_dtype == FR_BF16) done = launch_rows<bf16, bf16>(p, stream);
    else FR_REFUSE("short_conv: rows of dtype %d from inputs of dtype %d", out_dtype, in_dtype);
    return done != FR_OK ? done : history(p, n_seqs, in_dtype, stream);
}
