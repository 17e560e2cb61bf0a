// The state space duality recurrence: a matrix state S [N][dv] per head that every token decays by one number, adds to and reads,
//
//     S_t = exp(-exp(A_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T,    y_t = S_t^T C_t + D_h x_t,    dt_t = softplus(raw_t + dt_bias_h)
//
// with x per head and B, C shared by the heads of a group (head h reads group h / (heads / groups)).  The state, the step sizes,
// the decays with their logarithms and everything that is added to the state are fp32; x, B and C are rows of an earlier kernel (after
// their convolution), read in its dtype.
//
//   scan           any size and dtype; one-token steps, float32, prompts of a few tokens.  A block owns one head of one sequence
//                  and 32 value channels: lanes are value channels, the warps share the N rows of S (a thread keeps its part of a
//                  column in registers); tokens are staged eight at a time, the warps' parts of the read-outs meet in shared
//                  memory.  A one-token step is the same kernel: all of a block's state is requested at once.
//   chunk_states   bf16 prompts, on the tensor cores (mma.sync.m16n8k16, fp32 sums): a prompt is cut into chunks of 128 tokens; with
//                  c_t the sum of the decays' logarithms up to token t of its chunk, a chunk adds U = sum_t e^(c_last - c_t) dt_t B_t x_t^T
//                  to e^(c_last) times the state before it.  The scaled x enter the product as two bf16 numbers each (head and
//                  remainder), which keeps them 32-bit in effect.
//   chunk_chain    walks a sequence's chunks in order, fp32: leaves every chunk's starting state where its U was and the last
//                  state with the sequence.
//   chunk_outputs  y_t = e^(c_t) S^T C_t + sum_(s <= t) e^(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t for a chunk's tokens and its starting state S; S and
//                  the decayed scores enter their products as head and remainder, too.
//   gate_group_norm   y silu(z), each of `parts` equal runs of the row divided by its own root mean square, times a weight
#include <math.h>

#include "common.cuh"
#include "mma_sync.cuh"

FR_EXPORT const char* ssd_last_error() { return fr_error_text; }

namespace {

constexpr int CH = 128;             // tokens per chunk
constexpr int PAD = 8;              // bf16 numbers between rows of a staged tile: rows fall into different banks
constexpr float LOG2E = 1.4426950408889634f;

struct SsdArgs {
    const void* xbc;                // [rows][ld]: x heads at x_off (dv each), B groups at b_off, C groups at c_off (n each)
    const float* dt;                // [rows][dt_ld]: raw step sizes, a column per head
    FrVec dt_bias, a_log, skip;     // [heads]
    float* out;                     // [rows][heads * dv]
    float* state;                   // [slots][state_stride]: S of head h at s_off + h * n * dv, laid out [n][dv]
    float* chunk;                   // [n_seqs][max_chunks][heads][n][dv]: U of each chunk, then its starting state
    float* chunk_decay;             // [n_seqs][max_chunks][heads]: e^(c_last)
    const int* row_seq;
    const int* seq_start;
    const int* seq_qlen;
    const int* seq_slots;
    long long state_stride, s_off;
    int ld, x_off, b_off, c_off, dt_ld, heads, groups, n, dv, max_chunks;
};

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// a token's step size
__device__ __forceinline__ float step_of(const SsdArgs& p, int row, int head) { return softplus_f(p.dt[(size_t)row * p.dt_ld + head] + p.dt_bias.at(head)); }

// ------------------------------------------------------------------ scan
constexpr int STAGE = 8;            // tokens staged at a time

template <typename T, int KPT>
__global__ void __launch_bounds__(256) scan_kernel(SsdArgs p) {
    constexpr int N = 8 * KPT;
    __shared__ __align__(16) float sc[STAGE][N], sb[STAGE][N];
    __shared__ float sx[STAGE][32], part[STAGE][8][33], decay[STAGE], step[STAGE];
    const int seq = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31, group = threadIdx.x >> 5;
    const int col = blockIdx.z * 32 + lane;
    const int r0 = p.seq_start[seq], n = p.seq_qlen[seq];
    const bool live = col < p.dv;
    fr_pdl_wait();
    fr_pdl_launch();
    if (n <= 0 || p.row_seq[r0] < 0) return;
    float* S = p.state + (size_t)p.seq_slots[seq] * p.state_stride + p.s_off + (size_t)head * p.n * p.dv;
    const int bg = head / (p.heads / p.groups);
    const float rate = expf(p.a_log.at(head)), skip = p.skip.at(head);
    float s[KPT];
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
        const int k = group * KPT + i;
        s[i] = live && k < p.n ? S[(size_t)k * p.dv + col] : 0.f;
    }
    for (int t0 = 0; t0 < n; t0 += STAGE) {
        const int nt = min(STAGE, n - t0);
        for (int idx = threadIdx.x; idx < nt * N; idx += 256) {
            const int t = idx / N, k = idx - t * N;
            const T* row = (const T*)p.xbc + (size_t)(r0 + t0 + t) * p.ld;
            sc[t][k] = k < p.n ? fr_load(row + p.c_off + bg * p.n + k) : 0.f;
            sb[t][k] = k < p.n ? fr_load(row + p.b_off + bg * p.n + k) : 0.f;
        }
        if (group < nt) sx[group][lane] = live ? fr_load((const T*)p.xbc + (size_t)(r0 + t0 + group) * p.ld + p.x_off + head * p.dv + col) : 0.f;
        if ((int)threadIdx.x < nt) {
            const float dt = step_of(p, r0 + t0 + threadIdx.x, head);
            step[threadIdx.x] = dt;
            decay[threadIdx.x] = expf(-rate * dt);
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float v = step[t] * sx[t][lane], d = decay[t];
            float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                s[i] = fmaf(d, s[i], sb[t][group * KPT + i] * v);
                o[i & 3] = fmaf(sc[t][group * KPT + i], s[i], o[i & 3]);
            }
            part[t][group][lane] = (o[0] + o[1]) + (o[2] + o[3]);
        }
        __syncthreads();
        if (group < nt && live) {
            float o = skip * sx[group][lane];
#pragma unroll
            for (int g = 0; g < 8; ++g) o += part[group][g][lane];
            p.out[(size_t)(r0 + t0 + group) * ((size_t)p.heads * p.dv) + head * p.dv + col] = o;
        }
        __syncthreads();                       // sx is read above; the next round's staging writes it
    }
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
        const int k = group * KPT + i;
        if (live && k < p.n) S[(size_t)k * p.dv + col] = s[i];
    }
}

// ------------------------------------------------------------------ chunks on the tensor cores
constexpr int THR = 256;            // threads of a chunk's block
constexpr int WARPS = THR / 32;
static_assert(WARPS * 16 == CH, "a warp owns sixteen of a chunk's tokens");

// The step sizes of a chunk's tokens, and the running sums of the decays' logarithms (in units of log2), the last of them at [CH]; a thread
// per token, then a barrier
__device__ __forceinline__ void chunk_steps(const SsdArgs& p, int r0, int n, int head, float* step, float* cum) {
    __shared__ float sums[CH / 32];
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    float dt = 0.f, sum = 0.f;
    if (t < CH) {
        dt = t < n ? step_of(p, r0 + t, head) : 0.f;
        sum = -LOG2E * expf(p.a_log.at(head)) * dt;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += v;
        }
        if (lane == 31) sums[warp] = sum;
        step[t] = dt;
    }
    __syncthreads();
    if (t < CH) {
#pragma unroll
        for (int w = 0; w < CH / 32; ++w)
            if (w < warp) sum += sums[w];
        cum[t] = sum;
        if (t == CH - 1) cum[CH] = sum;
    }
    __syncthreads();
}

// A thread's share of the rows r0 .. r0 + n - 1 of `width` channels: all loads first (`fetch`), stored to a tile [CH][D + PAD] later
template <int D> constexpr int pieces_of() { return CH * (D / 8) / THR; }
template <int D>
__device__ __forceinline__ void fetch_rows(const SsdArgs& p, int off, int width, int r0, int n, uint4 (&raw)[pieces_of<D>()]) {
#pragma unroll
    for (int i = 0; i < pieces_of<D>(); ++i) {
        const int idx = threadIdx.x + i * THR, t = idx / (D / 8), c = (idx % (D / 8)) * 8;
        raw[i] = make_uint4(0, 0, 0, 0);
        if (t < n) raw[i] = raw8((const bf16*)p.xbc + (size_t)(r0 + t) * p.ld + off, c, width);
    }
}
template <int D>
__device__ __forceinline__ void put_rows(const uint4 (&raw)[pieces_of<D>()], bf16* tile) {
#pragma unroll
    for (int i = 0; i < pieces_of<D>(); ++i) {
        const int idx = threadIdx.x + i * THR, t = idx / (D / 8), c = (idx % (D / 8)) * 8;
        *(uint4*)(tile + t * (D + PAD) + c) = raw[i];
    }
}

template <int DK, int DV>
__global__ void __launch_bounds__(THR) chunk_states_kernel(SsdArgs p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* sb = (bf16*)smem_raw;                           // [CH][DK + PAD]
    bf16* sxh = sb + CH * (DK + PAD);                     // [CH][DV + PAD] scaled x, head
    bf16* sxl = sxh + CH * (DV + PAD);                    // and remainder
    __shared__ __align__(8) float step[CH], cum[CH + 2];
    // warps share the tiles of 16 rows of the state; where there are fewer tiles than warps, the value channels as well
    constexpr int MT = DK / 16, COLS = WARPS / MT, DVW = DV / COLS < 16 ? 16 : DV / COLS;
    static_assert(MT <= WARPS, "at most eight tiles of the state's rows");
    const int c = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int qlen = p.seq_qlen[seq];
    if (c * CH >= qlen) return;
    const int r0 = p.seq_start[seq] + c * CH, n = min(CH, qlen - c * CH);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    fr_pdl_wait();
    fr_pdl_launch();
    if (p.row_seq[r0] < 0) return;
    const int bg = head / (p.heads / p.groups);
    uint4 br[pieces_of<DK>()], xr[pieces_of<DV>()];
    fetch_rows<DV>(p, p.x_off + head * p.dv, p.dv, r0, n, xr);
    fetch_rows<DK>(p, p.b_off + bg * p.n, p.n, r0, n, br);
    chunk_steps(p, r0, n, head, step, cum);
    if (threadIdx.x == 0) p.chunk_decay[((size_t)seq * p.max_chunks + c) * p.heads + head] = exp2f(cum[CH]);
#pragma unroll
    for (int i = 0; i < pieces_of<DV>(); ++i) {
        const int idx = threadIdx.x + i * THR, t = idx / (DV / 8), k = (idx % (DV / 8)) * 8;
        const float f = exp2f(cum[CH] - cum[t]) * step[t];          // zero beyond the last token
        const uint32_t w[4] = {xr[i].x, xr[i].y, xr[i].z, xr[i].w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split2(__uint_as_float(w[e] << 16) * f, __uint_as_float(w[e] & 0xffff0000u) * f, hi[e], lo[e]);
        *(uint4*)(sxh + t * (DV + PAD) + k) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *(uint4*)(sxl + t * (DV + PAD) + k) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    put_rows<DK>(br, sb);
    __syncthreads();
    const int m0 = warp % MT, v0 = (warp / MT) * DVW;
    if (v0 >= DV) return;
    float acc[DVW / 8][4];
#pragma unroll
    for (int j = 0; j < DVW / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const int a_row = (lane & 7) + ((lane >> 4) & 1) * 8, a_col = ((lane >> 3) & 1) * 8;      // A is stored [token][row of the state]
#pragma unroll
    for (int ks = 0; ks < CH / 16; ++ks) {
        if (ks * 16 >= n) break;
        uint32_t a[4];
        ldsm4t(a, sb + (ks * 16 + a_row) * (DK + PAD) + m0 * 16 + a_col);
#pragma unroll
        for (int j = 0; j < DVW / 16; ++j) {
            uint32_t bh[4], bl[4];
            const int at = (ks * 16 + (lane & 15)) * (DV + PAD) + v0 + j * 16 + (lane >> 4) * 8;
            ldsm4t(bh, sxh + at);
            ldsm4t(bl, sxl + at);
            mma_16816(acc[2 * j], a, bh[0], bh[1]);
            mma_16816(acc[2 * j + 1], a, bh[2], bh[3]);
            mma_16816(acc[2 * j], a, bl[0], bl[1]);
            mma_16816(acc[2 * j + 1], a, bl[2], bl[3]);
        }
    }
    float* U = p.chunk + (((size_t)seq * p.max_chunks + c) * p.heads + head) * p.n * p.dv;
    const bool pairs = p.dv % 2 == 0;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int k = m0 * 16 + g + 8 * half;
        if (k >= p.n) continue;
#pragma unroll
        for (int j = 0; j < DVW / 8; ++j) {
            const int col = v0 + j * 8 + 2 * t4;
            float* dst = U + (size_t)k * p.dv + col;
            if (pairs && col + 1 < p.dv) *(float2*)dst = make_float2(acc[j][2 * half], acc[j][2 * half + 1]);
            else {
                if (col < p.dv) dst[0] = acc[j][2 * half];
                if (col + 1 < p.dv) dst[1] = acc[j][2 * half + 1];
            }
        }
    }
}

// One thread per element (or four neighbouring ones) of a head's matrix
template <typename V>
__global__ void __launch_bounds__(256) chunk_chain_kernel(SsdArgs p) {
    constexpr int NV = sizeof(V) / 4;
    const int seq = blockIdx.x, head = blockIdx.y;
    const int r0 = p.seq_start[seq], n = p.seq_qlen[seq];
    fr_pdl_wait();
    fr_pdl_launch();
    if (n <= 0 || p.row_seq[r0] < 0) return;
    const int chunks = (n + CH - 1) / CH, per = p.n * p.dv;
    float* S = p.state + (size_t)p.seq_slots[seq] * p.state_stride + p.s_off + (size_t)head * per;
    const int e = (blockIdx.z * 256 + threadIdx.x) * NV;
    if (e >= per) return;
    float* u0 = p.chunk + ((size_t)seq * p.max_chunks * p.heads + head) * per + e;
    const float* d0 = p.chunk_decay + (size_t)seq * p.max_chunks * p.heads + head;
    const size_t stride = (size_t)p.heads * per;
    V r = *(V*)(S + e);
    float* rf = (float*)&r;
    for (int c0 = 0; c0 < chunks; c0 += 8) {                // eight chunks' numbers are loaded together, then chained
        V u[8];
        float d[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const int c = min(c0 + k, chunks - 1);
            u[k] = *(const V*)(u0 + (size_t)c * stride);
            d[k] = d0[(size_t)c * p.heads];
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            if (c0 + k < chunks) {
                *(V*)(u0 + (size_t)(c0 + k) * stride) = r;
                const float* uf = (const float*)&u[k];
#pragma unroll
                for (int i = 0; i < NV; ++i) rf[i] = fmaf(d[k], rf[i], uf[i]);
            }
        }
    }
    *(V*)(S + e) = r;
}

template <int DK, int DV>
constexpr int outputs_smem() {
    constexpr int states = 2 * DK * (DV + PAD), rows = CH * (DK + PAD) + CH * (DV + PAD);
    return (CH * (DK + PAD) + (states > rows ? states : rows)) * 2;
}

template <int DK, int DV>
__global__ void __launch_bounds__(THR) chunk_outputs_kernel(SsdArgs p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* sc = (bf16*)smem_raw;                           // [CH][DK + PAD]
    bf16* sh = sc + CH * (DK + PAD);                      // [DK][DV + PAD] the chunk's starting state, head
    bf16* sl = sh + DK * (DV + PAD);                      // and remainder; once they are used, in their place:
    bf16* sb = sh;                                        // [CH][DK + PAD]
    bf16* sx = sb + CH * (DK + PAD);                      // [CH][DV + PAD]
    __shared__ __align__(8) float step[CH], cum[CH + 2];
    const int c = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int qlen = p.seq_qlen[seq];
    if (c * CH >= qlen) return;
    const int r0 = p.seq_start[seq] + c * CH, n = min(CH, qlen - c * CH);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int w_row = warp * 16;
    fr_pdl_wait();
    fr_pdl_launch();
    if (p.row_seq[r0] < 0) return;
    const int bg = head / (p.heads / p.groups);
    {
        uint4 cr[pieces_of<DK>()];
        fetch_rows<DK>(p, p.c_off + bg * p.n, p.n, r0, n, cr);
        chunk_steps(p, r0, n, head, step, cum);
        const float* S = p.chunk + (((size_t)seq * p.max_chunks + c) * p.heads + head) * p.n * p.dv;
        const bool fours = p.dv % 4 == 0;
        constexpr int ITEMS = DK * (DV / 4) / THR, BATCH = ITEMS < 8 ? ITEMS : 8;       // pieces of four numbers; loads in flight
#pragma unroll 1
        for (int i0 = 0; i0 < ITEMS; i0 += BATCH) {
            float4 x[BATCH];
#pragma unroll
            for (int i = 0; i < BATCH; ++i) {
                const int idx = threadIdx.x + (i0 + i) * THR, k = idx / (DV / 4), v = (idx % (DV / 4)) * 4;
                x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (k >= p.n || v >= p.dv) continue;
                const float* src = S + (size_t)k * p.dv + v;
                if (fours) x[i] = *(const float4*)src;
                else {
                    x[i].x = src[0];
                    if (v + 1 < p.dv) x[i].y = src[1];
                    if (v + 2 < p.dv) x[i].z = src[2];
                    if (v + 3 < p.dv) x[i].w = src[3];
                }
            }
#pragma unroll
            for (int i = 0; i < BATCH; ++i) {
                const int idx = threadIdx.x + (i0 + i) * THR, k = idx / (DV / 4), v = (idx % (DV / 4)) * 4;
                uint2 hi, lo;
                split2(x[i].x, x[i].y, hi.x, lo.x);
                split2(x[i].z, x[i].w, hi.y, lo.y);
                *(uint2*)(sh + k * (DV + PAD) + v) = hi;
                *(uint2*)(sl + k * (DV + PAD) + v) = lo;
            }
        }
        put_rows<DK>(cr, sc);
    }
    __syncthreads();
    // the chunk's B and x are on their way while the state is read
    uint4 br[pieces_of<DK>()], xr[pieces_of<DV>()];
    fetch_rows<DK>(p, p.b_off + bg * p.n, p.n, r0, n, br);
    fetch_rows<DV>(p, p.x_off + head * p.dv, p.dv, r0, n, xr);
    // what the state before the chunk gives its rows
    float o[DV / 8][4];
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    const bf16* c_at = sc + (w_row + (lane & 15)) * (DK + PAD) + (lane >> 4) * 8;
    const bool mine = w_row < n;                          // the same for a whole warp
    if (mine) {
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t ca[4];
            ldsm4(ca, c_at + ks * 16);
#pragma unroll
            for (int j = 0; j < DV / 16; ++j) {
                uint32_t bh[4], bl[4];
                ldsm4t(bh, sh + (ks * 16 + (lane & 15)) * (DV + PAD) + j * 16 + (lane >> 4) * 8);
                ldsm4t(bl, sl + (ks * 16 + (lane & 15)) * (DV + PAD) + j * 16 + (lane >> 4) * 8);
                mma_16816(o[2 * j], ca, bh[0], bh[1]);
                mma_16816(o[2 * j + 1], ca, bh[2], bh[3]);
                mma_16816(o[2 * j], ca, bl[0], bl[1]);
                mma_16816(o[2 * j + 1], ca, bl[2], bl[3]);
            }
        }
    }
    const int row[2] = {w_row + g, w_row + g + 8};
    const float at[2] = {cum[row[0]], cum[row[1]]};
    const float f0 = exp2f(at[0]), f1 = exp2f(at[1]);
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) {
        o[j][0] *= f0;
        o[j][1] *= f0;
        o[j][2] *= f1;
        o[j][3] *= f1;
    }
    __syncthreads();
    put_rows<DK>(br, sb);
    put_rows<DV>(xr, sx);
    __syncthreads();
    if (!mine) return;
    // and the chunk's own tokens, those up to each row (a warp's rows see no token beyond its last row), 32 at a time: four sums run side
    // by side
#pragma unroll 1
    for (int kk = 0; kk <= warp; kk += 2) {
        float s[4][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
        const bf16* b_at = sb + (kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * (DK + PAD) + ((lane >> 3) & 1) * 8;      // stored [token][channel]
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t ca[4], b0[4], b1[4];
            ldsm4(ca, c_at + ks * 16);
            ldsm4(b0, b_at + ks * 16);
            ldsm4(b1, b_at + 16 * (DK + PAD) + ks * 16);
            mma_16816(s[0], ca, b0[0], b0[1]);
            mma_16816(s[1], ca, b0[2], b0[3]);
            mma_16816(s[2], ca, b1[0], b1[1]);
            mma_16816(s[3], ca, b1[2], b1[3]);
        }
        uint32_t hi[2][4], lo[2][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            const int t = kk * 16 + nt * 8 + 2 * t4;
            const float2 ct = *(const float2*)(cum + t), st = *(const float2*)(step + t);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int half = e >> 1;
                const float f = exp2f(at[half] - (e & 1 ? ct.y : ct.x)) * (e & 1 ? st.y : st.x);
                s[nt][e] = t + (e & 1) <= row[half] ? s[nt][e] * f : 0.f;
            }
            split2(s[nt][0], s[nt][1], hi[nt >> 1][2 * (nt & 1)], lo[nt >> 1][2 * (nt & 1)]);
            split2(s[nt][2], s[nt][3], hi[nt >> 1][2 * (nt & 1) + 1], lo[nt >> 1][2 * (nt & 1) + 1]);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int j = 0; j < DV / 16; ++j) {
                uint32_t b[4];
                ldsm4t(b, sx + ((kk + u) * 16 + (lane & 15)) * (DV + PAD) + j * 16 + (lane >> 4) * 8);
                mma_16816(o[2 * j], hi[u], b[0], b[1]);
                mma_16816(o[2 * j + 1], hi[u], b[2], b[3]);
                mma_16816(o[2 * j], lo[u], b[0], b[1]);
                mma_16816(o[2 * j + 1], lo[u], b[2], b[3]);
            }
    }
    const bool pairs = p.dv % 2 == 0;
    const float skip = p.skip.at(head);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        if (row[half] >= n) continue;
        float* dst = p.out + (size_t)(r0 + row[half]) * ((size_t)p.heads * p.dv) + (size_t)head * p.dv;
#pragma unroll
        for (int j = 0; j < DV / 8; ++j) {
            const int col = j * 8 + 2 * t4;
            const uint32_t own = *(const uint32_t*)(sx + row[half] * (DV + PAD) + col);
            const float a = fmaf(skip, __uint_as_float(own << 16), o[j][2 * half]), b = fmaf(skip, __uint_as_float(own & 0xffff0000u), o[j][2 * half + 1]);
            if (pairs && col + 1 < p.dv) *(float2*)(dst + col) = make_float2(a, b);
            else {
                if (col < p.dv) dst[col] = a;
                if (col + 1 < p.dv) dst[col + 1] = b;
            }
        }
    }
}

template <int DK, int DV>
int launch_chunks(const SsdArgs& p, int n_seqs, cudaStream_t stream) {
    constexpr int smem_a = (CH * (DK + PAD) + 2 * CH * (DV + PAD)) * 2, smem_c = outputs_smem<DK, DV>();
    static bool set = false;
    if (!set) {
        FR_CUDA(cudaFuncSetAttribute(chunk_states_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_a));
        FR_CUDA(cudaFuncSetAttribute(chunk_outputs_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_c));
        set = true;
    }
    const dim3 grid(p.max_chunks, p.heads, n_seqs);
    FR_CUDA(fr_launch(chunk_states_kernel<DK, DV>, grid, dim3(THR), smem_a, stream, p));
    const int per = p.n * p.dv;
    if (per % 4 == 0 && p.state_stride % 4 == 0 && p.s_off % 4 == 0 && ((((uintptr_t)p.state) | ((uintptr_t)p.chunk)) & 15) == 0)
        FR_CUDA(fr_launch(chunk_chain_kernel<float4>, dim3(n_seqs, p.heads, (per / 4 + 255) / 256), dim3(256), 0, stream, p));
    else
        FR_CUDA(fr_launch(chunk_chain_kernel<float>, dim3(n_seqs, p.heads, (per + 255) / 256), dim3(256), 0, stream, p));
    FR_CUDA(fr_launch(chunk_outputs_kernel<DK, DV>, grid, dim3(THR), smem_c, stream, p));
    FR_CHECK_LAUNCH("ssd chunks");
    return FR_OK;
}

template <int DK>
int chunks_by_value_size(const SsdArgs& p, int n_seqs, cudaStream_t stream) {
    if (p.dv <= 32) return launch_chunks<DK, 32>(p, n_seqs, stream);
    if (p.dv <= 64) return launch_chunks<DK, 64>(p, n_seqs, stream);
    return launch_chunks<DK, 128>(p, n_seqs, stream);
}

template <typename T>
int launch_scan(const SsdArgs& p, int n_seqs, cudaStream_t stream) {
    const dim3 grid(n_seqs, p.heads, (p.dv + 31) / 32);
    if (p.n <= 32) FR_CUDA(fr_launch(scan_kernel<T, 4>, grid, dim3(256), 0, stream, p));
    else if (p.n <= 64) FR_CUDA(fr_launch(scan_kernel<T, 8>, grid, dim3(256), 0, stream, p));
    else if (p.n <= 128) FR_CUDA(fr_launch(scan_kernel<T, 16>, grid, dim3(256), 0, stream, p));
    else if (p.n <= 256) FR_CUDA(fr_launch(scan_kernel<T, 32>, grid, dim3(256), 0, stream, p));
    else FR_CUDA(fr_launch(scan_kernel<T, 64>, grid, dim3(256), 0, stream, p));
    FR_CHECK_LAUNCH("ssd scan");
    return FR_OK;
}

bool chunks_fit(int max_q_len, int n, int dv, int dtype) { return dtype == FR_BF16 && max_q_len >= 32 && n <= 128 && dv <= 128; }

// ------------------------------------------------------------------ gate and norm
// A block per run of a row.  TZ: dtype of the gates, T: of the result.
template <typename TZ, typename T>
__global__ void __launch_bounds__(256) gate_group_norm_kernel(const float* __restrict__ y, const TZ* __restrict__ z, int z_ld, T* __restrict__ out, FrVec w,
                                                              int per, int parts, float eps, int by_four) {
    __shared__ float partial[8];
    fr_pdl_wait();
    fr_pdl_launch();
    const size_t row = blockIdx.x;
    const int c0 = blockIdx.y * per;
    const float* yr = y + row * ((size_t)per * parts) + c0;
    const TZ* zr = z + row * z_ld + c0;
    T* o = out + row * ((size_t)per * parts) + c0;
    constexpr int KEEP = 4;                           // pieces of four numbers that a thread keeps between its two passes
    float held[KEEP][4], ss = 0.f;
    const int threads = blockDim.x;
    auto gated = [&](int c, float (&v)[4]) {
        const float4 a = *(const float4*)(yr + c);
        float g[4];
        FrVec{zr, sizeof(TZ) == 2 ? FR_BF16 : FR_F32}.four(c, g);
        const float as[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = as[i] * g[i] / (1.0f + expf(-g[i]));
    };
    auto one = [&](int c) {
        const float g = fr_load(zr + c);
        return yr[c] * g / (1.0f + expf(-g));
    };
    if (by_four) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            const int c = (threadIdx.x + k * threads) * 4;
            if (c >= per) break;
            gated(c, held[k]);
#pragma unroll
            for (int i = 0; i < 4; ++i) ss = fmaf(held[k][i], held[k][i], ss);
        }
        for (int c = (threadIdx.x + KEEP * threads) * 4; c < per; c += threads * 4) {
            float v[4];
            gated(c, v);
#pragma unroll
            for (int i = 0; i < 4; ++i) ss = fmaf(v[i], v[i], ss);
        }
    } else {
        for (int c = threadIdx.x; c < per; c += threads) {
            const float v = one(c);
            ss = fmaf(v, v, ss);
        }
    }
    ss = fr_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int k = 0; k < threads / 32; ++k) ss += partial[k];
    const float inv = 1.0f / sqrtf(ss / (float)per + eps);
    if (by_four) {
        auto put = [&](int c, const float (&v)[4]) {
            float ws[4];
            w.four(c0 + c, ws);
            if constexpr (sizeof(T) == 2) *(uint2*)(o + c) = make_uint2(pack2(v[0] * inv * ws[0], v[1] * inv * ws[1]), pack2(v[2] * inv * ws[2], v[3] * inv * ws[3]));
            else *(float4*)(o + c) = make_float4(v[0] * inv * ws[0], v[1] * inv * ws[1], v[2] * inv * ws[2], v[3] * inv * ws[3]);
        };
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            const int c = (threadIdx.x + k * threads) * 4;
            if (c >= per) break;
            put(c, held[k]);
        }
        for (int c = (threadIdx.x + KEEP * threads) * 4; c < per; c += threads * 4) {
            float v[4];
            gated(c, v);
            put(c, v);
        }
    } else {
        for (int c = threadIdx.x; c < per; c += threads) fr_store(o + c, one(c) * inv * w.at(c0 + c));
    }
}

template <typename TZ, typename T>
int launch_gate_norm(const float* y, const void* z, int z_ld, void* out, FrVec w, int rows, int per, int parts, float eps, int by_four, cudaStream_t stream) {
    const int want = (by_four ? per / 4 : per), threads = want >= 256 ? 256 : (want + 31) / 32 * 32;
    FR_CUDA(fr_launch(gate_group_norm_kernel<TZ, T>, dim3(rows, parts), dim3(threads), 0, stream, y, (const TZ*)z, z_ld, (T*)out, w, per, parts, eps, by_four));
    FR_CHECK_LAUNCH("gate_group_norm");
    return FR_OK;
}

}  // namespace

// Floats of scratch that ssd_run wants for a step (0: none; the chunked form does not take it).
FR_EXPORT long long ssd_scratch_floats(int n_seqs, int max_q_len, int heads, int n, int dv, int dtype) {
    if (!chunks_fit(max_q_len, n, dv, dtype)) return 0;
    return (long long)n_seqs * ((max_q_len + CH - 1) / CH) * heads * ((long long)n * dv + 1);
}

// xbc [rows][ld] of `dtype`: x [heads][dv] at x_off, B and C [groups][n] at b_off and c_off; dt [rows][dt_ld] fp32, a raw step size per head;
// dt_bias, a_log, skip [heads] of vec_dtype.  out [rows][heads * dv] fp32; state [slots][state_stride] fp32, the heads' matrices at s_off.
// scratch (may be null): the chunked form runs if it is given and takes the step.
FR_EXPORT int ssd_run(const void* xbc, int ld, int x_off, int b_off, int c_off, const float* dt, int dt_ld, const void* dt_bias, const void* a_log,
                      const void* skip, int vec_dtype, float* out, float* state, long long state_stride, long long s_off, const int* row_seq,
                      const int* seq_start, const int* seq_qlen, const int* seq_slots, int n_seqs, int max_q_len, int heads, int groups, int n, int dv,
                      float* scratch, int dtype, cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return FR_OK;
    if (heads <= 0 || heads > 65535 || groups <= 0 || heads % groups) FR_REFUSE("ssd: %d heads cannot share %d groups", heads, groups);
    if (n <= 0 || n > 512 || dv <= 0 || dv > 65535) FR_REFUSE("ssd: a state of %d x %d per head (1 to 512 rows)", n, dv);
    if (s_off < 0 || s_off + (long long)heads * n * dv > state_stride) FR_REFUSE("ssd: the state is smaller than the heads' matrices");
    SsdArgs p;
    p.xbc = xbc; p.dt = dt; p.dt_bias = FrVec{dt_bias, vec_dtype}; p.a_log = FrVec{a_log, vec_dtype}; p.skip = FrVec{skip, vec_dtype};
    p.out = out; p.state = state; p.chunk = scratch; p.row_seq = row_seq; p.seq_start = seq_start; p.seq_qlen = seq_qlen; p.seq_slots = seq_slots;
    p.state_stride = state_stride; p.s_off = s_off; p.ld = ld; p.x_off = x_off; p.b_off = b_off; p.c_off = c_off; p.dt_ld = dt_ld;
    p.heads = heads; p.groups = groups; p.n = n; p.dv = dv; p.max_chunks = (max_q_len + CH - 1) / CH;
    p.chunk_decay = scratch != nullptr ? scratch + (size_t)n_seqs * p.max_chunks * heads * n * dv : nullptr;
    if (scratch != nullptr && chunks_fit(max_q_len, n, dv, dtype) && n_seqs <= 65535) {
        if (n <= 32) return chunks_by_value_size<32>(p, n_seqs, stream);
        if (n <= 64) return chunks_by_value_size<64>(p, n_seqs, stream);
        return chunks_by_value_size<128>(p, n_seqs, stream);
    }
    if (dtype == FR_F32) return launch_scan<float>(p, n_seqs, stream);
    if (dtype == FR_BF16) return launch_scan<bf16>(p, n_seqs, stream);
    FR_REFUSE("ssd: unknown dtype %d", dtype);
}

// y [rows][n] fp32, z (z_ld apart) of z_dtype, out [rows][n] of `dtype`, weight [n] of w_dtype: y silu(z), every one of `parts` equal runs of a
// row divided by sqrt(its mean square + eps), times the weight
FR_EXPORT int ssd_gate_group_norm(const float* y, const void* z, int z_ld, int z_dtype, void* out, const void* weight, int w_dtype, int rows, int n,
                                  int parts, float eps, int dtype, cudaStream_t stream) {
    if (rows <= 0 || n <= 0) return FR_OK;
    if (parts < 1 || n % parts || parts > 65535) FR_REFUSE("gate_group_norm: %d channels in %d equal parts", n, parts);
    const FrVec w{weight, w_dtype};
    const int per = n / parts;
    const int by_four = per % 4 == 0 && z_ld % 4 == 0 && ((((uintptr_t)y) | ((uintptr_t)out) | ((uintptr_t)z)) & 15) == 0;
    if (z_dtype == FR_F32 && dtype == FR_F32) return launch_gate_norm<float, float>(y, z, z_ld, out, w, rows, per, parts, eps, by_four, stream);
    if (z_dtype == FR_F32 && dtype == FR_BF16) return launch_gate_norm<float, bf16>(y, z, z_ld, out, w, rows, per, parts, eps, by_four, stream);
    if (z_dtype == FR_BF16 && dtype == FR_BF16) return launch_gate_norm<bf16, bf16>(y, z, z_ld, out, w, rows, per, parts, eps, by_four, stream);
    FR_REFUSE("gate_group_norm: rows of dtype %d with gates of dtype %d", dtype, z_dtype);
}
