// Linear attention with a constant decay per head: S_t = d_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, where q, k and v are silu of
// columns of a stacked projection.  The state S [dk][dv] of every head and sequence, everything that is added to it and the
// read-outs are fp32; silu is fp32 and its results are rounded to the projection's dtype, in every kernel alike, so that a
// token means the same numbers in a prompt and alone.
//
//   scan           any size and dtype; one-token steps, float32, prompts of a few tokens.  A block owns one head of one sequence
//                  and 32 value channels: lanes are value channels, the warps share the key channels (a thread keeps its part
//                  of a column of S in registers); tokens are staged eight at a time, the warps' parts of the read-outs meet in
//                  shared memory.  A one-token step is the same kernel: all of a block's state is requested at once.
//   chunk_states   bf16 prompts, on the tensor cores (mma.sync.m16n8k16, fp32 sums): a prompt is cut into chunks of 64 tokens;
//                  a chunk of n tokens adds U = sum_t d^(n - 1 - t) k_t v_t^T to d^n times the state before it.  The scaled
//                  keys enter the product as two bf16 numbers each (head and remainder), which keeps them 32-bit in effect.
//   chunk_chain    walks a sequence's chunks in order, fp32: leaves every chunk's starting state where its U was and the last
//                  state with the sequence.
//   chunk_outputs  o_t = d^(t + 1) S^T q_t + sum_(s <= t) d^(t - s) (q_t . k_s) v_s for a chunk's tokens (t from 0) and its starting
//                  state S; S and the decayed scores enter their products as head and remainder, too.
//   row_norm_gate  o / sqrt(mean(o^2) + eps) * weight * sigmoid(gate): one norm over all heads of a row
#include <math.h>

#include "common.cuh"
#include "mma_sync.cuh"

FR_EXPORT const char* linear_decay_last_error() { return fr_error_text; }

namespace {

constexpr int CH = 64;              // tokens per chunk
constexpr int PAD = 8;              // bf16 numbers between rows of a staged tile: rows fall into different banks

struct DecayArgs {
    const void* proj;               // [rows][ld]: q heads at q_off, k heads at k_off (dk each), v heads at v_off (dv each)
    const float* decay;             // [heads]
    float* out;                     // [rows][heads * dv]
    float* state;                   // [slots][state_stride]: S of head h at h * dk * dv, laid out [dk][dv]
    float* chunk;                   // [n_seqs][max_chunks][heads][dk][dv]: U of each chunk, then its starting state
    const int* row_seq;
    const int* seq_start;
    const int* seq_qlen;
    const int* seq_slots;
    long long state_stride;
    int ld, q_off, k_off, v_off, heads, dk, dv, max_chunks;
};

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// silu, rounded to the dtype of the rows
template <typename T> __device__ __forceinline__ float silu_as(float z);
template <> __device__ __forceinline__ float silu_as<float>(float z) { return silu_f(z); }
template <> __device__ __forceinline__ float silu_as<bf16>(float z) { return __bfloat162float(__float2bfloat16_rn(silu_f(z))); }

// ------------------------------------------------------------------ scan
constexpr int STAGE = 8;            // tokens staged at a time

template <typename T, int KPT>
__global__ void __launch_bounds__(256) scan_kernel(DecayArgs p) {
    constexpr int DK = 8 * KPT;
    __shared__ __align__(16) float sq[STAGE][DK], sk[STAGE][DK];
    __shared__ float sv[STAGE][32], part[STAGE][8][33];
    const int seq = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31, group = threadIdx.x >> 5;
    const int col = blockIdx.z * 32 + lane;
    const int r0 = p.seq_start[seq], n = p.seq_qlen[seq];
    fr_pdl_wait();
    fr_pdl_launch();
    if (n <= 0 || p.row_seq[r0] < 0) return;
    const float d = p.decay[head];
    float* S = p.state + (size_t)p.seq_slots[seq] * p.state_stride + (size_t)head * p.dk * p.dv;
    const bool live = col < p.dv;
    float s[KPT];
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
        const int k = group * KPT + i;
        s[i] = live && k < p.dk ? S[(size_t)k * p.dv + col] : 0.f;
    }
    for (int t0 = 0; t0 < n; t0 += STAGE) {
        const int nt = min(STAGE, n - t0);
        for (int idx = threadIdx.x; idx < nt * DK; idx += 256) {
            const int t = idx / DK, k = idx - t * DK;
            const T* row = (const T*)p.proj + (size_t)(r0 + t0 + t) * p.ld;
            sq[t][k] = k < p.dk ? silu_as<T>(fr_load(row + p.q_off + head * p.dk + k)) : 0.f;
            sk[t][k] = k < p.dk ? silu_as<T>(fr_load(row + p.k_off + head * p.dk + k)) : 0.f;
        }
        if (group < nt)
            sv[group][lane] = live ? silu_as<T>(fr_load((const T*)p.proj + (size_t)(r0 + t0 + group) * p.ld + p.v_off + head * p.dv + col)) : 0.f;
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float v = sv[t][lane];
            float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                s[i] = fmaf(d, s[i], sk[t][group * KPT + i] * v);
                o[i & 3] = fmaf(sq[t][group * KPT + i], s[i], o[i & 3]);
            }
            part[t][group][lane] = (o[0] + o[1]) + (o[2] + o[3]);
        }
        __syncthreads();
        if (group < nt && live) {
            float o = 0.f;
#pragma unroll
            for (int g = 0; g < 8; ++g) o += part[group][g][lane];
            p.out[(size_t)(r0 + t0 + group) * ((size_t)p.heads * p.dv) + head * p.dv + col] = o;
        }
        // the next round's staging writes sq, sk and sv, which nobody reads any more; its parts are written after a barrier
    }
#pragma unroll
    for (int i = 0; i < KPT; ++i) {
        const int k = group * KPT + i;
        if (live && k < p.dk) S[(size_t)k * p.dv + col] = s[i];
    }
}

// ------------------------------------------------------------------ chunks on the tensor cores
constexpr int THR = 256;             // threads of a chunk's block

// the silu of eight channels, fp32 values that bf16 holds exactly
__device__ __forceinline__ void silu8(const uint4& r, float (&v)[8]) {
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = silu_as<bf16>(__uint_as_float(w[i] << 16));
        v[2 * i + 1] = silu_as<bf16>(__uint_as_float(w[i] & 0xffff0000u));
    }
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) { return make_uint4(pack2(v[0], v[1]), pack2(v[2], v[3]), pack2(v[4], v[5]), pack2(v[6], v[7])); }

// A thread's share of the rows r0 .. r0 + n - 1 of a head's channels: all loads first (`fetch`), used later
template <int D> constexpr int pieces_of() { return (CH * (D / 8) + THR - 1) / THR; }
template <int D>
__device__ __forceinline__ void fetch_rows(const DecayArgs& p, int off, int width, int r0, int n, uint4 (&raw)[pieces_of<D>()]) {
#pragma unroll
    for (int i = 0; i < pieces_of<D>(); ++i) {
        const int idx = threadIdx.x + i * THR, t = idx / (D / 8), c = (idx % (D / 8)) * 8;
        raw[i] = make_uint4(0, 0, 0, 0);
        if (t < n) raw[i] = raw8((const bf16*)p.proj + (size_t)(r0 + t) * p.ld + off, c, width);
    }
}
// into a tile [CH][D + PAD], silu applied (zero stays zero)
template <int D>
__device__ __forceinline__ void put_rows(const uint4 (&raw)[pieces_of<D>()], bf16* tile) {
#pragma unroll
    for (int i = 0; i < pieces_of<D>(); ++i) {
        const int idx = threadIdx.x + i * THR, t = idx / (D / 8), c = (idx % (D / 8)) * 8;
        if (t >= CH) break;
        float v[8];
        silu8(raw[i], v);
        *(uint4*)(tile + t * (D + PAD) + c) = pack8(v);
    }
}

template <int DK, int DV>
__global__ void __launch_bounds__(THR) chunk_states_kernel(DecayArgs p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* skh = (bf16*)smem_raw;                          // [CH][DK + PAD] scaled keys, head
    bf16* skl = skh + CH * (DK + PAD);                    // and remainder
    bf16* sv = skl + CH * (DK + PAD);                     // [CH][DV + PAD]
    __shared__ float pw[CH];
    // warps share the tiles of 16 key channels; where there are fewer tiles than warps, the value channels as well
    constexpr int MT = DK / 16, PER = (MT + 7) / 8, COLS = MT >= 8 ? 1 : 8 / MT, DVW = DV / COLS < 16 ? 16 : DV / COLS;
    const int c = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int qlen = p.seq_qlen[seq];
    if (c * CH >= qlen) return;
    const int r0 = p.seq_start[seq] + c * CH, n = min(CH, qlen - c * CH);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    fr_pdl_wait();
    fr_pdl_launch();
    if (p.row_seq[r0] < 0) return;
    uint4 kr[pieces_of<DK>()], vr[pieces_of<DV>()];
    fetch_rows<DK>(p, p.k_off + head * p.dk, p.dk, r0, n, kr);
    fetch_rows<DV>(p, p.v_off + head * p.dv, p.dv, r0, n, vr);
    if (threadIdx.x < CH) pw[threadIdx.x] = powf(p.decay[head], (float)threadIdx.x);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < pieces_of<DK>(); ++i) {
        const int idx = threadIdx.x + i * THR, t = idx / (DK / 8), k = (idx % (DK / 8)) * 8;
        if (t >= CH) break;
        float v[8];
        silu8(kr[i], v);
        const float f = t < n ? pw[n - 1 - t] : 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= f;
        uint4 hi, lo;
        split2(v[0], v[1], hi.x, lo.x); split2(v[2], v[3], hi.y, lo.y); split2(v[4], v[5], hi.z, lo.z); split2(v[6], v[7], hi.w, lo.w);
        *(uint4*)(skh + t * (DK + PAD) + k) = hi;
        *(uint4*)(skl + t * (DK + PAD) + k) = lo;
    }
    put_rows<DV>(vr, sv);
    __syncthreads();
    const int m0 = COLS == 1 ? warp : warp % MT, v0 = COLS == 1 ? 0 : (warp / MT) * DVW;
    if (v0 >= DV) return;
    float acc[PER][DVW / 8][4];
#pragma unroll
    for (int m = 0; m < PER; ++m)
#pragma unroll
        for (int j = 0; j < DVW / 8; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f;
    const int a_row = (lane & 7) + ((lane >> 4) & 1) * 8, a_col = ((lane >> 3) & 1) * 8;      // A is stored [token][key channel]
#pragma unroll
    for (int ks = 0; ks < CH / 16; ++ks) {
        uint32_t ah[PER][4], al[PER][4];
#pragma unroll
        for (int m = 0; m < PER; ++m) {
            const int tile = m0 + 8 * m;
            if (tile < MT) {
                ldsm4t(ah[m], skh + (ks * 16 + a_row) * (DK + PAD) + tile * 16 + a_col);
                ldsm4t(al[m], skl + (ks * 16 + a_row) * (DK + PAD) + tile * 16 + a_col);
            }
        }
#pragma unroll
        for (int j = 0; j < DVW / 16; ++j) {
            uint32_t b[4];
            ldsm4t(b, sv + (ks * 16 + (lane & 15)) * (DV + PAD) + v0 + j * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int m = 0; m < PER; ++m) {
                if (m0 + 8 * m < MT) {
                    mma_16816(acc[m][2 * j], ah[m], b[0], b[1]);
                    mma_16816(acc[m][2 * j], al[m], b[0], b[1]);
                    mma_16816(acc[m][2 * j + 1], ah[m], b[2], b[3]);
                    mma_16816(acc[m][2 * j + 1], al[m], b[2], b[3]);
                }
            }
        }
    }
    float* U = p.chunk + (((size_t)seq * p.max_chunks + c) * p.heads + head) * p.dk * p.dv;
    const bool pairs = p.dv % 2 == 0;
#pragma unroll
    for (int m = 0; m < PER; ++m) {
        const int tile = m0 + 8 * m;
        if (tile >= MT) continue;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int k = tile * 16 + g + 8 * half;
            if (k >= p.dk) continue;
#pragma unroll
            for (int j = 0; j < DVW / 8; ++j) {
                const int col = v0 + j * 8 + 2 * t4;
                float* dst = U + (size_t)k * p.dv + col;
                if (pairs && col + 1 < p.dv) *(float2*)dst = make_float2(acc[m][j][2 * half], acc[m][j][2 * half + 1]);
                else {
                    if (col < p.dv) dst[0] = acc[m][j][2 * half];
                    if (col + 1 < p.dv) dst[1] = acc[m][j][2 * half + 1];
                }
            }
        }
    }
}

// One thread per element (or four neighbouring ones) of a head's matrix
template <typename V>
__global__ void __launch_bounds__(256) chunk_chain_kernel(DecayArgs p) {
    constexpr int N = sizeof(V) / 4;
    const int seq = blockIdx.x, head = blockIdx.y;
    const int r0 = p.seq_start[seq], n = p.seq_qlen[seq];
    fr_pdl_wait();
    fr_pdl_launch();
    if (n <= 0 || p.row_seq[r0] < 0) return;
    const int chunks = (n + CH - 1) / CH, per = p.dk * p.dv;
    const float d = p.decay[head], whole = powf(d, (float)CH), last = powf(d, (float)(n - (chunks - 1) * CH));
    float* S = p.state + (size_t)p.seq_slots[seq] * p.state_stride + (size_t)head * per;
    const int e = (blockIdx.z * 256 + threadIdx.x) * N;
    if (e >= per) return;
    float* u0 = p.chunk + ((size_t)seq * p.max_chunks * p.heads + head) * per + e;
    const size_t step = (size_t)p.heads * per;
    V r = *(V*)(S + e);
    float* rf = (float*)&r;
    for (int c0 = 0; c0 < chunks; c0 += 8) {                // eight chunks' numbers are loaded together, then chained
        V u[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) u[k] = *(const V*)(u0 + (size_t)min(c0 + k, chunks - 1) * step);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            if (c0 + k < chunks) {
                *(V*)(u0 + (size_t)(c0 + k) * step) = r;
                const float f = c0 + k + 1 < chunks ? whole : last;
                const float* uf = (const float*)&u[k];
#pragma unroll
                for (int i = 0; i < N; ++i) rf[i] = fmaf(f, rf[i], uf[i]);
            }
        }
    }
    *(V*)(S + e) = r;
}

template <int DK, int DV>
constexpr int outputs_smem() {
    constexpr int states = 2 * DK * (DV + PAD), rows = CH * (DK + PAD) + CH * (DV + PAD);
    return (CH * (DK + PAD) + (states > rows ? states : rows)) * 2 + (CH + 1) * 4;
}

template <int DK, int DV>
__global__ void __launch_bounds__(THR) chunk_outputs_kernel(DecayArgs p) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    constexpr int states = 2 * DK * (DV + PAD), rows = CH * (DK + PAD) + CH * (DV + PAD);
    constexpr int DH = DV / 2;                            // value channels of a warp: two warps share 16 rows
    bf16* sq = (bf16*)smem_raw;                           // [CH][DK + PAD]
    bf16* sh = sq + CH * (DK + PAD);                      // [DK][DV + PAD] the chunk's starting state, head
    bf16* sl = sh + DK * (DV + PAD);                      // and remainder; once they are used, in their place:
    bf16* sk = sh;                                        // [CH][DK + PAD]
    bf16* sv = sk + CH * (DK + PAD);                      // [CH][DV + PAD]
    float* pw = (float*)(sq + CH * (DK + PAD) + (states > rows ? states : rows));      // powers of the decay, 0 .. CH
    const int c = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int qlen = p.seq_qlen[seq];
    if (c * CH >= qlen) return;
    const int r0 = p.seq_start[seq] + c * CH, n = min(CH, qlen - c * CH);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int w_row = (warp & 3) * 16, v0 = (warp >> 2) * DH;
    fr_pdl_wait();
    fr_pdl_launch();
    if (p.row_seq[r0] < 0) return;
    uint4 qr[pieces_of<DK>()];
    fetch_rows<DK>(p, p.q_off + head * p.dk, p.dk, r0, n, qr);
    if (threadIdx.x <= CH) pw[threadIdx.x] = powf(p.decay[head], (float)threadIdx.x);
    const float* S = p.chunk + (((size_t)seq * p.max_chunks + c) * p.heads + head) * p.dk * p.dv;
    const bool fours = p.dv % 4 == 0;
    constexpr int ITEMS = DK * (DV / 4) / THR, BATCH = ITEMS < 8 ? ITEMS : 8;       // pieces of four numbers; loads in flight
#pragma unroll 1
    for (int i0 = 0; i0 < ITEMS; i0 += BATCH) {
        float4 x[BATCH];
#pragma unroll
        for (int i = 0; i < BATCH; ++i) {
            const int idx = threadIdx.x + (i0 + i) * THR, k = idx / (DV / 4), v = (idx % (DV / 4)) * 4;
            x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (k >= p.dk || v >= p.dv) continue;
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
    put_rows<DK>(qr, sq);
    __syncthreads();
    // the chunk's keys and values are on their way while the state is read
    uint4 kr[pieces_of<DK>()], vr[pieces_of<DV>()];
    fetch_rows<DK>(p, p.k_off + head * p.dk, p.dk, r0, n, kr);
    fetch_rows<DV>(p, p.v_off + head * p.dv, p.dv, r0, n, vr);
    // what the state before the chunk gives its rows
    float o[DH / 8][4];
#pragma unroll
    for (int j = 0; j < DH / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    const bf16* q_at = sq + (w_row + (lane & 15)) * (DK + PAD) + (lane >> 4) * 8;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t qa[4];
        ldsm4(qa, q_at + ks * 16);
#pragma unroll
        for (int j = 0; j < DH / 16; ++j) {
            uint32_t bh[4], bl[4];
            ldsm4t(bh, sh + (ks * 16 + (lane & 15)) * (DV + PAD) + v0 + j * 16 + (lane >> 4) * 8);
            ldsm4t(bl, sl + (ks * 16 + (lane & 15)) * (DV + PAD) + v0 + j * 16 + (lane >> 4) * 8);
            mma_16816(o[2 * j], qa, bh[0], bh[1]);
            mma_16816(o[2 * j], qa, bl[0], bl[1]);
            mma_16816(o[2 * j + 1], qa, bh[2], bh[3]);
            mma_16816(o[2 * j + 1], qa, bl[2], bl[3]);
        }
    }
    const int row[2] = {w_row + g, w_row + g + 8};
    const float f0 = pw[row[0] + 1], f1 = pw[row[1] + 1];
#pragma unroll
    for (int j = 0; j < DH / 8; ++j) {
        o[j][0] *= f0;
        o[j][1] *= f0;
        o[j][2] *= f1;
        o[j][3] *= f1;
    }
    __syncthreads();
    put_rows<DK>(kr, sk);
    put_rows<DV>(vr, sv);
    __syncthreads();
    // and the chunk's own tokens, those up to each row (a warp's rows see no token beyond its last row)
#pragma unroll
    for (int kk = 0; kk < CH / 16; ++kk) {
        if (kk > (warp & 3)) break;
        float s[2][4];
#pragma unroll
        for (int e = 0; e < 4; ++e) s[0][e] = s[1][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t qa[4], b[4];                         // keys kk * 16 .. + 15: B is stored [token][key channel]
            ldsm4(qa, q_at + ks * 16);
            ldsm4(b, sk + (kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * (DK + PAD) + ks * 16 + ((lane >> 3) & 1) * 8);
            mma_16816(s[0], qa, b[0], b[1]);
            mma_16816(s[1], qa, b[2], b[3]);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int back = row[e >> 1] - (kk * 16 + nt * 8 + 2 * t4 + (e & 1));
                s[nt][e] = back >= 0 ? s[nt][e] * pw[back] : 0.f;
            }
        uint32_t hi[4], lo[4];
        split2(s[0][0], s[0][1], hi[0], lo[0]);
        split2(s[0][2], s[0][3], hi[1], lo[1]);
        split2(s[1][0], s[1][1], hi[2], lo[2]);
        split2(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
        for (int j = 0; j < DH / 16; ++j) {
            uint32_t b[4];
            ldsm4t(b, sv + (kk * 16 + (lane & 15)) * (DV + PAD) + v0 + j * 16 + (lane >> 4) * 8);
            mma_16816(o[2 * j], hi, b[0], b[1]);
            mma_16816(o[2 * j], lo, b[0], b[1]);
            mma_16816(o[2 * j + 1], hi, b[2], b[3]);
            mma_16816(o[2 * j + 1], lo, b[2], b[3]);
        }
    }
    const bool pairs = p.dv % 2 == 0;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        if (row[half] >= n) continue;
        float* dst = p.out + (size_t)(r0 + row[half]) * ((size_t)p.heads * p.dv) + (size_t)head * p.dv;
#pragma unroll
        for (int j = 0; j < DH / 8; ++j) {
            const int col = v0 + j * 8 + 2 * t4;
            if (pairs && col + 1 < p.dv) *(float2*)(dst + col) = make_float2(o[j][2 * half], o[j][2 * half + 1]);
            else {
                if (col < p.dv) dst[col] = o[j][2 * half];
                if (col + 1 < p.dv) dst[col + 1] = o[j][2 * half + 1];
            }
        }
    }
}

template <int DK, int DV>
int launch_chunks(const DecayArgs& p, int n_seqs, cudaStream_t stream) {
    constexpr int smem_a = (2 * CH * (DK + PAD) + CH * (DV + PAD)) * 2, smem_c = outputs_smem<DK, DV>();
    static bool set = false;
    if (!set) {
        FR_CUDA(cudaFuncSetAttribute(chunk_states_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_a));
        FR_CUDA(cudaFuncSetAttribute(chunk_outputs_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_c));
        set = true;
    }
    const dim3 grid(p.max_chunks, p.heads, n_seqs);
    FR_CUDA(fr_launch(chunk_states_kernel<DK, DV>, grid, dim3(THR), smem_a, stream, p));
    const int per = p.dk * p.dv;
    if (per % 4 == 0 && p.state_stride % 4 == 0 && ((((uintptr_t)p.state) | ((uintptr_t)p.chunk)) & 15) == 0)
        FR_CUDA(fr_launch(chunk_chain_kernel<float4>, dim3(n_seqs, p.heads, (per / 4 + 255) / 256), dim3(256), 0, stream, p));
    else
        FR_CUDA(fr_launch(chunk_chain_kernel<float>, dim3(n_seqs, p.heads, (per + 255) / 256), dim3(256), 0, stream, p));
    FR_CUDA(fr_launch(chunk_outputs_kernel<DK, DV>, grid, dim3(THR), smem_c, stream, p));
    FR_CHECK_LAUNCH("linear_decay chunks");
    return FR_OK;
}

template <int DK>
int chunks_by_value_size(const DecayArgs& p, int n_seqs, cudaStream_t stream) {
    if (p.dv <= 32) return launch_chunks<DK, 32>(p, n_seqs, stream);
    if (p.dv <= 64) return launch_chunks<DK, 64>(p, n_seqs, stream);
    return launch_chunks<DK, 128>(p, n_seqs, stream);
}

template <typename T>
int launch_scan(const DecayArgs& p, int n_seqs, cudaStream_t stream) {
    const dim3 grid(n_seqs, p.heads, (p.dv + 31) / 32);
    if (p.dk <= 32) FR_CUDA(fr_launch(scan_kernel<T, 4>, grid, dim3(256), 0, stream, p));
    else if (p.dk <= 64) FR_CUDA(fr_launch(scan_kernel<T, 8>, grid, dim3(256), 0, stream, p));
    else if (p.dk <= 128) FR_CUDA(fr_launch(scan_kernel<T, 16>, grid, dim3(256), 0, stream, p));
    else FR_CUDA(fr_launch(scan_kernel<T, 32>, grid, dim3(256), 0, stream, p));
    FR_CHECK_LAUNCH("linear_decay scan");
    return FR_OK;
}

// ------------------------------------------------------------------ norm over the heads side by side, and the gate
__device__ __forceinline__ float row_sum(float v, float* partial) {
    v = fr_warp_sum(v);
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = v;
    __syncthreads();
    v = 0.f;
    for (int w = 0; w < (int)blockDim.x / 32; ++w) v += partial[w];
    return v;
}

template <typename T>
__global__ void __launch_bounds__(256) row_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, int gate_ld, T* __restrict__ out,
                                                            FrVec w, int n, float eps, int by_four) {
    __shared__ float partial[8];
    fr_pdl_wait();
    fr_pdl_launch();
    const float* x = o + (size_t)blockIdx.x * n;
    const T* g = gate + (size_t)blockIdx.x * gate_ld;
    T* y = out + (size_t)blockIdx.x * n;
    float ss = 0.f;
    if (by_four) {
        for (int c = threadIdx.x * 4; c < n; c += 1024) {
            const float4 v = *(const float4*)(x + c);
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
        }
    } else {
        for (int c = threadIdx.x; c < n; c += 256) ss = fmaf(x[c], x[c], ss);
    }
    const float inv = 1.0f / sqrtf(row_sum(ss, partial) / (float)n + eps);
    if (by_four) {
        for (int c = threadIdx.x * 4; c < n; c += 1024) {
            const float4 v = *(const float4*)(x + c);
            const float xs[4] = {v.x, v.y, v.z, v.w};
            float r[4], ws[4], gs[4];
            w.four(c, ws);
            FrVec{g, sizeof(T) == 2 ? FR_BF16 : FR_F32}.four(c, gs);
#pragma unroll
            for (int i = 0; i < 4; ++i) r[i] = xs[i] * inv * ws[i] / (1.0f + expf(-gs[i]));
            if constexpr (sizeof(T) == 2) *(uint2*)(y + c) = make_uint2(pack2(r[0], r[1]), pack2(r[2], r[3]));
            else *(float4*)(y + c) = make_float4(r[0], r[1], r[2], r[3]);
        }
    } else {
        for (int c = threadIdx.x; c < n; c += 256) fr_store(y + c, x[c] * inv * w.at(c) / (1.0f + expf(-fr_load(g + c))));
    }
}

bool chunks_fit(int max_q_len, int dk, int dv, int dtype) { return dtype == FR_BF16 && max_q_len >= 32 && dk <= 128 && dv <= 128; }

}  // namespace

// Floats of scratch that linear_decay_run wants for a step (0: none; the chunked form does not take it).
FR_EXPORT long long linear_decay_scratch_floats(int n_seqs, int max_q_len, int heads, int dk, int dv, int dtype) {
    if (!chunks_fit(max_q_len, dk, dv, dtype)) return 0;
    return (long long)n_seqs * ((max_q_len + CH - 1) / CH) * heads * dk * dv;
}

// proj [rows][ld] of `dtype`; out [rows][heads * dv] fp32; state [slots][state_stride] fp32.  scratch (may be null): the chunked
// form runs if it is given and takes the step.
FR_EXPORT int linear_decay_run(const void* proj, int ld, int q_off, int k_off, int v_off, const float* decay, float* out, float* state,
                               long long state_stride, const int* row_seq, const int* seq_start, const int* seq_qlen, const int* seq_slots,
                               int n_seqs, int max_q_len, int heads, int dk, int dv, float* scratch, int dtype, cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return FR_OK;
    if (heads <= 0 || heads > 65535 || dk <= 0 || dk > 256 || dv <= 0) FR_REFUSE("linear_decay: %d heads, sizes %d and %d (keys of 1 to 256)", heads, dk, dv);
    if (state_stride < (long long)heads * dk * dv) FR_REFUSE("linear_decay: the state is smaller than the heads' matrices");
    DecayArgs p;
    p.proj = proj; p.decay = decay; p.out = out; p.state = state; p.chunk = scratch; p.row_seq = row_seq; p.seq_start = seq_start;
    p.seq_qlen = seq_qlen; p.seq_slots = seq_slots; p.state_stride = state_stride; p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
    p.heads = heads; p.dk = dk; p.dv = dv; p.max_chunks = (max_q_len + CH - 1) / CH;
    if (scratch != nullptr && chunks_fit(max_q_len, dk, dv, dtype) && n_seqs <= 65535) {
        if (dk <= 32) return chunks_by_value_size<32>(p, n_seqs, stream);
        if (dk <= 64) return chunks_by_value_size<64>(p, n_seqs, stream);
        return chunks_by_value_size<128>(p, n_seqs, stream);
    }
    if (dtype == FR_F32) return launch_scan<float>(p, n_seqs, stream);
    if (dtype == FR_BF16) return launch_scan<bf16>(p, n_seqs, stream);
    FR_REFUSE("linear_decay: unknown dtype %d", dtype);
}

// o [rows][n] fp32, gate (gate_ld apart) and out [rows][n] of `dtype`, weight [n] of w_dtype
FR_EXPORT int linear_decay_row_norm_gate(const float* o, const void* gate, int gate_ld, void* out, const void* weight, int w_dtype, int rows, int n,
                                         float eps, int dtype, cudaStream_t stream) {
    if (rows <= 0 || n <= 0) return FR_OK;
    const FrVec w{weight, w_dtype};
    const int by_four = n % 4 == 0 && ((((uintptr_t)o) | ((uintptr_t)out)) & 15) == 0;
    if (dtype == FR_F32) FR_CUDA(fr_launch(row_norm_gate_kernel<float>, dim3(rows), dim3(256), 0, stream, o, (const float*)gate, gate_ld, (float*)out, w, n, eps, by_four));
    else if (dtype == FR_BF16) FR_CUDA(fr_launch(row_norm_gate_kernel<bf16>, dim3(rows), dim3(256), 0, stream, o, (const bf16*)gate, gate_ld, (bf16*)out, w, n, eps, by_four));
    else FR_REFUSE("row_norm_gate: unknown dtype %d", dtype);
    FR_CHECK_LAUNCH("row_norm_gate");
    return FR_OK;
}
