// The state-space recurrence of state_space.cu over portions of prompts in bfloat16, chunk by chunk on the tensor cores.
//
// With l_t = -exp(A_log) d_t, L_t the sum of l over a chunk's tokens up to t, and S_0 the state before the chunk:
//   y_t  = exp(L_t) S_0^T C_t + sum_{s <= t} (C_t . B_s) exp(L_t - L_s) d_s x_s + D x_t
//   S'   = exp(L_last) S_0 + sum_s exp(L_last - L_s) d_s B_s x_s^T
// Two kernels.  The walk goes along a sequence's chunks (a CTA a (sequence, head, 32 columns), the state in the accumulators of
// its products) and leaves the state before every chunk; the outputs of all chunks are then formed side by side.
// In 32-bit: step sizes, their logarithms, sums and exponentials, the state, every sum.  B, C and x are the convolution's bfloat16
// results; what stands beside them in a product and is 32-bit (the weighted x of the state's update, the state itself) goes in as
// two bfloat16 numbers, the value and what its rounding left, so that it counts with 16 bits of mantissa; the weights within a
// chunk are rounded once, like an attention's.
#include "attention_mma.cuh"
#include "common.cuh"
#include "kernels.h"
#include "launch.cuh"

namespace vtb {

namespace {

constexpr int kChunk = 64;           // tokens of a chunk
constexpr int kCols = 64;            // columns of the state (values of a head) a CTA owns
constexpr int kPad = 8;              // 16-bit numbers between rows in shared memory
constexpr int kLC = kCols + kPad;
constexpr int kWalkCols = 32;        // ... in the walk, whose time is the length of its chain: more CTAs, each with less to do
constexpr int kWalkThreads = 256;
constexpr int kOutThreads = 256;

struct ChunkArgs {
    const __nv_bfloat16* u;          // [tokens, u_stride]: x at 0, B at heads * v_dim, C behind it
    int u_stride;
    const __nv_bfloat16* y;          // the raw step sizes at dt_col + h
    int stride, dt_col;
    const float *a_log, *dt_bias, *d;
    float* state;                    // [state_rows, heads, dim, v_dim]
    int state_rows;
    const int* cu_q;
    const int* rows;
    int n_seqs;
    const int2* walks;               // [grid.x of the walk]: (sequence, its first chunk)
    const int2* chunks;              // [chunks]: (sequence, first of its new tokens)
    float* starts;                   // [chunks, heads, dim, v_dim]: the state before every chunk
    float* out;                      // [tokens, heads * v_dim]
    int heads, groups, dim, v_dim;
    int* status;
};

__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float warp_running_sum(float v) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += u;
    }
    return v;
}

// v as two bfloat16 numbers: hi + lo is v to 16 bits of mantissa.
__device__ __forceinline__ void split_pair(float v0, float v1, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat16 h0 = __float2bfloat16_rn(v0), h1 = __float2bfloat16_rn(v1);
    hi = pack_bf16(v0, v1);
    lo = pack_bf16(v0 - __bfloat162float(h0), v1 - __bfloat162float(h1));
}

}  // namespace

// ------------------------------------------------------------------------- the walk along a sequence's chunks

// Warps: 8 / WN along the state's rows (MT tiles of 16 rows each), WN along the CTA's 32 columns.  A chunk's step sizes and weights
// are formed by the first warp, two tokens a lane, while the products of the chunk before run.
template <int MT, int WN>
__global__ void __launch_bounds__(kWalkThreads)
state_space_walk_kernel(const ChunkArgs a) {
    constexpr int WM = 8 / WN, NP = WM * MT * 16, LN = NP + kPad, NT = kWalkCols / 8 / WN, LC = kWalkCols + kPad;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* bs = reinterpret_cast<__nv_bfloat16*>(smem_raw);          // [2][chunk][LN]
    __nv_bfloat16* xs = bs + 2 * kChunk * LN;                                // [2][chunk][LC]
    __nv_bfloat16* hi = xs + 2 * kChunk * LC;                                // [chunk][LC]: weighted x
    __nv_bfloat16* lo = hi + kChunk * LC;                                    // [chunk][LC]: what its rounding left
    float* ws = reinterpret_cast<float*>(lo + kChunk * LC);                  // [2][chunk]: weights
    float* all = ws + 2 * kChunk;                                            // [2]: the chunk's whole decay
    pdl_launch();
    const int2 walk = a.walks[blockIdx.x];
    const int seq = walk.x, h = blockIdx.y, col0 = blockIdx.z * kWalkCols;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int wm = warp / WN, wn = warp % WN;
    const int dim = a.dim, v_dim = a.v_dim;
    const float rate = expf(a.a_log[h]), bias = a.dt_bias[h];
    const bool seq_ok = seq >= 0 && seq < a.n_seqs;
    const int t0 = seq_ok ? a.cu_q[seq] : 0, t1 = seq_ok ? a.cu_q[seq + 1] : 0;
    const int row = seq_ok ? a.rows[seq] : 0;
    pdl_wait();
    if (t1 <= t0) return;
    if (row < 0 || row >= a.state_rows) {
        if (tid == 0) set_status(a.status, kStatusBadRow, row);
        return;
    }
    const int inner = a.heads * v_dim, b_col = inner + (h / (a.heads / a.groups)) * dim;
    auto load = [&](int tb, int stage) {
        const int n = min(kChunk, t1 - tb);
        __nv_bfloat16* b = bs + stage * kChunk * LN;
        __nv_bfloat16* x = xs + stage * kChunk * LC;
        for (int c = tid; c < kChunk * (NP / 8); c += kWalkThreads) {
            const int r = c / (NP / 8), i = (c % (NP / 8)) * 8;
            const bool ok = r < n && i < dim;
            cp_async16(b + r * LN + i, a.u + (ok ? (size_t)(tb + r) * a.u_stride + b_col + i : 0), ok);
        }
        for (int c = tid; c < kChunk * (kWalkCols / 8); c += kWalkThreads) {
            const int r = c / (kWalkCols / 8), i = (c % (kWalkCols / 8)) * 8;
            const bool ok = r < n && col0 + i < v_dim;
            cp_async16(x + r * LC + i, a.u + (ok ? (size_t)(tb + r) * a.u_stride + (size_t)h * v_dim + col0 + i : 0), ok);
        }
        cp_async_commit();
    };
    // raw step sizes of tokens 2 lane and 2 lane + 1 of a chunk, fetched a chunk before they are used
    float raw[2] = {0.f, 0.f};
    auto fetch = [&](int tb) {
#pragma unroll
        for (int k = 0; k < 2; ++k) raw[k] = __bfloat162float(a.y[(size_t)min(tb + 2 * lane + k, t1 - 1) * a.stride + a.dt_col + h]);
    };
    auto weigh = [&](int tb, int buf) {
        float step[2], L[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) step[k] = tb + 2 * lane + k < t1 ? softplus_of(raw[k] + bias) : 0.f;
        const float mine = -rate * step[0] - rate * step[1], sum = warp_running_sum(mine);
        L[1] = sum;
        L[0] = sum + rate * step[1];
        const float last = __shfl_sync(0xffffffffu, sum, 31);
#pragma unroll
        for (int k = 0; k < 2; ++k) ws[buf * kChunk + 2 * lane + k] = expf(last - L[k]) * step[k];
        if (lane == 0) all[buf] = expf(last);
    };
    load(t0, 0);
    if (warp == 0) fetch(t0);
    // the state: row (wm MT + m) 16 + gq + 8 i, columns (wn NT + n) 8 + 2 tq and the one behind it
    float* sp = a.state + ((size_t)row * a.heads + h) * dim * v_dim;
    float acc[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int r = (wm * MT + m) * 16 + gq + 8 * i, c = col0 + (wn * NT + n) * 8 + 2 * tq;
                float2 v = make_float2(0.f, 0.f);
                if (r < dim && c < v_dim) v = *reinterpret_cast<const float2*>(sp + (size_t)r * v_dim + c);
                acc[m][n][2 * i] = v.x;
                acc[m][n][2 * i + 1] = v.y;
            }
    auto keep = [&](float* to) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int r = (wm * MT + m) * 16 + gq + 8 * i, c = col0 + (wn * NT + n) * 8 + 2 * tq;
                    if (r < dim && c < v_dim)
                        *reinterpret_cast<float2*>(to + (size_t)r * v_dim + c) = make_float2(acc[m][n][2 * i], acc[m][n][2 * i + 1]);
                }
    };
    if (warp == 0) {
        weigh(t0, 0);
        fetch(min(t0 + kChunk, t1 - 1));
    }
    const int mat = lane >> 3, r8 = lane & 7;
    int chunk = walk.y, stage = 0;
    for (int tb = t0; tb < t1; tb += kChunk, ++chunk, stage ^= 1) {
        cp_async_wait<0>();
        __syncthreads();                 // the chunk's rows and weights are there; the products of the chunk before are done
        if (tb + kChunk < t1) load(tb + kChunk, stage ^ 1);
        keep(a.starts + ((size_t)chunk * a.heads + h) * dim * v_dim);
        const __nv_bfloat16* x = xs + stage * kChunk * LC;
        const float* w = ws + stage * kChunk;
#pragma unroll
        for (int e = tid; e < kChunk * (kWalkCols / 2); e += kWalkThreads) {
            const int r = e / (kWalkCols / 2), i = (e % (kWalkCols / 2)) * 2;
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x + r * LC + i));
            uint32_t vh, vl;
            split_pair(v.x * w[r], v.y * w[r], vh, vl);
            *reinterpret_cast<uint32_t*>(hi + r * LC + i) = vh;
            *reinterpret_cast<uint32_t*>(lo + r * LC + i) = vl;
        }
        const float decay = all[stage];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[m][n][e] *= decay;
        __syncthreads();
        if (warp == 0 && tb + kChunk < t1) {
            weigh(tb + kChunk, stage ^ 1);
            fetch(min(tb + 2 * kChunk, t1 - 1));
        }
        const __nv_bfloat16* b = bs + stage * kChunk * LN;
#pragma unroll
        for (int k = 0; k < kChunk / 16; ++k) {
            // the operand's rows are the state's (B's columns): read transposed from [token][row]
            uint32_t af[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
                ldmatrix_x4_trans(af[m], b + (size_t)(k * 16 + (mat >> 1) * 8 + r8) * LN + (wm * MT + m) * 16 + (mat & 1) * 8);
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                uint32_t vh[4], vl[4];
                const size_t at = (size_t)(k * 16 + (mat & 1) * 8 + r8) * LC + (wn * NT + n) * 8 + (mat >> 1) * 8;
                ldmatrix_x4_trans(vh, hi + at);
                ldmatrix_x4_trans(vl, lo + at);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma_bf16(acc[m][n], af[m], vl[0], vl[1]);
                    mma_bf16(acc[m][n + 1], af[m], vl[2], vl[3]);
                    mma_bf16(acc[m][n], af[m], vh[0], vh[1]);
                    mma_bf16(acc[m][n + 1], af[m], vh[2], vh[3]);
                }
            }
        }
    }
    keep(sp);
}

// ------------------------------------------------------------------------- the outputs of every chunk

// A CTA: a chunk, a head, 64 columns; its eight warps 16 tokens and one half of the columns each (the two warps of the same tokens
// both form their weights).  NP: the state's rows, padded.
template <int NP>
__global__ void __launch_bounds__(kOutThreads)
state_space_out_kernel(const ChunkArgs a) {
    constexpr int LN = NP + kPad;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* cs = reinterpret_cast<__nv_bfloat16*>(smem_raw);          // [chunk][LN]
    __nv_bfloat16* bs = cs + kChunk * LN;                                    // [chunk][LN]
    __nv_bfloat16* xs = bs + kChunk * LN;                                    // [chunk][kLC]
    __nv_bfloat16* sh = xs + kChunk * kLC;                                   // [NP][kLC]: the state before the chunk
    __nv_bfloat16* sl = sh + NP * kLC;                                       // [NP][kLC]: what its rounding left
    float* Ls = reinterpret_cast<float*>(sl + NP * kLC);                     // [chunk]: sums of logarithms
    float* ds = Ls + kChunk;                                                 // [chunk]: step sizes; [64]: the first warp's sum
    pdl_launch();
    const int2 ch = a.chunks[blockIdx.x];
    const int seq = ch.x, h = blockIdx.y, col0 = blockIdx.z * kCols;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int dim = a.dim, v_dim = a.v_dim;
    const float rate = expf(a.a_log[h]), bias = a.dt_bias[h], skip = a.d[h];
    const bool seq_ok = seq >= 0 && seq < a.n_seqs;
    const int tb = seq_ok ? a.cu_q[seq] + ch.y : 0, t1 = seq_ok ? a.cu_q[seq + 1] : 0;
    pdl_wait();
    const int n = min(kChunk, t1 - tb);
    if (n <= 0) return;
    const int inner = a.heads * v_dim, g = h / (a.heads / a.groups);
    for (int c = tid; c < kChunk * (NP / 8); c += kOutThreads) {
        const int r = c / (NP / 8), i = (c % (NP / 8)) * 8;
        const bool ok = r < n && i < dim;
        const __nv_bfloat16* ur = a.u + (ok ? (size_t)(tb + r) * a.u_stride + inner + (size_t)g * dim + i : 0);
        cp_async16(bs + r * LN + i, ur, ok);
        cp_async16(cs + r * LN + i, ok ? ur + (size_t)a.groups * dim : ur, ok);
    }
    for (int c = tid; c < kChunk * (kCols / 8); c += kOutThreads) {
        const int r = c / (kCols / 8), i = (c % (kCols / 8)) * 8;
        const bool ok = r < n && col0 + i < v_dim;
        cp_async16(xs + r * kLC + i, a.u + (ok ? (size_t)(tb + r) * a.u_stride + (size_t)h * v_dim + col0 + i : 0), ok);
    }
    cp_async_commit();
    float L = 0.f;
    if (tid < kChunk) {
        const float step = tid < n ? softplus_of(__bfloat162float(a.y[(size_t)(tb + tid) * a.stride + a.dt_col + h]) + bias) : 0.f;
        L = warp_running_sum(-rate * step);
        ds[tid] = step;
        if (tid == 31) ds[kChunk] = L;
    }
    // the state: all of a thread's quads on their way together (the products' registers are free yet)
    const float* S = a.starts + ((size_t)blockIdx.x * a.heads + h) * dim * v_dim;
    constexpr int kQuads = NP * (kCols / 4);
    constexpr int kMine = kQuads / kOutThreads, kAtOnce = kMine < 16 ? kMine : 16;
    static_assert(kQuads % (kOutThreads * kAtOnce) == 0, "quads of the state a thread");
#pragma unroll 1
    for (int c0 = tid; c0 < kQuads; c0 += kOutThreads * kAtOnce) {
        float4 v[kAtOnce];
#pragma unroll
        for (int k = 0; k < kAtOnce; ++k) {
            const int c = c0 + k * kOutThreads, r = c / (kCols / 4), i = (c % (kCols / 4)) * 4;
            v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < dim && col0 + i < v_dim) v[k] = *reinterpret_cast<const float4*>(S + (size_t)r * v_dim + col0 + i);
        }
#pragma unroll
        for (int k = 0; k < kAtOnce; ++k) {
            const int c = c0 + k * kOutThreads, r = c / (kCols / 4), i = (c % (kCols / 4)) * 4;
            uint2 vh, vl;
            split_pair(v[k].x, v[k].y, vh.x, vl.x);
            split_pair(v[k].z, v[k].w, vh.y, vl.y);
            *reinterpret_cast<uint2*>(sh + r * kLC + i) = vh;
            *reinterpret_cast<uint2*>(sl + r * kLC + i) = vl;
        }
    }
    __syncthreads();
    if (tid < kChunk) Ls[tid] = tid >= 32 ? L + ds[kChunk] : L;
    cp_async_wait<0>();
    __syncthreads();

    const int mat = lane >> 3, r8 = lane & 7, row0 = (warp & 3) * 16, half0 = (warp >> 2) * (kCols / 2);
    if (row0 >= n) return;
    // C's fragments serve both products: with the state and with B
    constexpr int kTiles = kCols / 16;                  // of eight columns
    float o[kTiles][4], s[kChunk / 8][4];
#pragma unroll
    for (int j = 0; j < kTiles; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < kChunk / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll 2
    for (int k = 0; k < NP / 16; ++k) {
        uint32_t cf[4];
        ldmatrix_x4(cf, cs + (size_t)(row0 + (lane & 7) + ((lane >> 3) & 1) * 8) * LN + k * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int j = 0; j < kTiles; j += 2) {
            uint32_t vh[4], vl[4];
            const size_t at = (size_t)(k * 16 + (mat & 1) * 8 + r8) * kLC + half0 + j * 8 + (mat >> 1) * 8;
            ldmatrix_x4_trans(vh, sh + at);
            ldmatrix_x4_trans(vl, sl + at);
            mma_bf16(o[j], cf, vl[0], vl[1]);
            mma_bf16(o[j + 1], cf, vl[2], vl[3]);
            mma_bf16(o[j], cf, vh[0], vh[1]);
            mma_bf16(o[j + 1], cf, vh[2], vh[3]);
        }
#pragma unroll
        for (int j = 0; j < kChunk / 8; j += 2) {
            if (j * 8 > row0 + 15) continue;         // tokens behind all of the warp's
            uint32_t bf[4];
            ldmatrix_x4(bf, bs + (size_t)((j + (mat >> 1)) * 8 + r8) * LN + k * 16 + (mat & 1) * 8);
            mma_bf16(s[j], cf, bf[0], bf[1]);
            mma_bf16(s[j + 1], cf, bf[2], bf[3]);
        }
    }
    const int row[2] = {row0 + gq, row0 + gq + 8};
    const float Lr[2] = {Ls[row[0]], Ls[row[1]]};
    const float from[2] = {expf(Lr[0]), expf(Lr[1])};
#pragma unroll
    for (int j = 0; j < kTiles; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] *= from[e >> 1];
#pragma unroll
    for (int j = 0; j < kChunk / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = j * 8 + 2 * tq + (e & 1);
            s[j][e] = c <= row[e >> 1] ? s[j][e] * expf(Lr[e >> 1] - Ls[c]) * ds[c] : 0.f;
        }
#pragma unroll
    for (int k = 0; k < kChunk / 16; ++k) {
        if (k * 16 > row0 + 15) continue;
        uint32_t pf[4];
        pf[0] = pack_bf16(s[2 * k][0], s[2 * k][1]);
        pf[1] = pack_bf16(s[2 * k][2], s[2 * k][3]);
        pf[2] = pack_bf16(s[2 * k + 1][0], s[2 * k + 1][1]);
        pf[3] = pack_bf16(s[2 * k + 1][2], s[2 * k + 1][3]);
#pragma unroll
        for (int j = 0; j < kTiles; j += 2) {
            uint32_t vf[4];
            ldmatrix_x4_trans(vf, xs + (size_t)(k * 16 + (mat & 1) * 8 + r8) * kLC + half0 + j * 8 + (mat >> 1) * 8);
            mma_bf16(o[j], pf, vf[0], vf[1]);
            mma_bf16(o[j + 1], pf, vf[2], vf[3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        if (row[i] >= n) continue;
        float* op = a.out + (size_t)(tb + row[i]) * inner + (size_t)h * v_dim + col0;
#pragma unroll
        for (int j = 0; j < kTiles; ++j) {
            const int c = half0 + j * 8 + 2 * tq;
            if (col0 + c >= v_dim) continue;
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(xs + row[i] * kLC + c));
            *reinterpret_cast<float2*>(op + c) = make_float2(fmaf(skip, x.x, o[j][2 * i]), fmaf(skip, x.y, o[j][2 * i + 1]));
        }
    }
}

// ------------------------------------------------------------------------- launches

namespace {
constexpr int kMostBytes = 200 * 1024;

template <int MT, int WN>
cudaError_t launch_walk(const ChunkArgs& a, int n, cudaStream_t stream) {
    constexpr int NP = 8 / WN * MT * 16;
    constexpr int bytes = (2 * kChunk * (NP + kPad) + 4 * kChunk * (kWalkCols + kPad)) * 2 + (2 * kChunk + 4) * 4;
    static std::atomic<unsigned long long> done{0};
    if (cudaError_t e = allow_dynamic_smem(state_space_walk_kernel<MT, WN>, bytes, done); e != cudaSuccess) return e;
    return launch(state_space_walk_kernel<MT, WN>, dim3(n, a.heads, (a.v_dim + kWalkCols - 1) / kWalkCols), dim3(kWalkThreads), bytes, stream, a);
}

template <int NP>
cudaError_t launch_out(const ChunkArgs& a, int n, cudaStream_t stream) {
    constexpr int bytes = (2 * kChunk * (NP + kPad) + kChunk * kLC + 2 * NP * kLC) * 2 + (2 * kChunk + 4) * 4;
    static_assert(bytes <= kMostBytes, "shared memory");
    static std::atomic<unsigned long long> done{0};
    if (cudaError_t e = allow_dynamic_smem(state_space_out_kernel<NP>, bytes, done); e != cudaSuccess) return e;
    return launch(state_space_out_kernel<NP>, dim3(n, a.heads, (a.v_dim + kCols - 1) / kCols), dim3(kOutThreads), bytes, stream, a);
}
}  // namespace

bool state_space_chunks_supports(int heads, int groups, int dim, int v_dim) {
    return dim >= 8 && dim <= 256 && dim % 8 == 0 && v_dim % 8 == 0 && groups >= 1 && heads % groups == 0;
}

cudaError_t launch_state_space_chunks(const void* u, int u_stride, const void* y, int stride, int dt_col, const float* a_log, const float* dt_bias,
                                      const float* d, float* state, int state_rows, const int* cu_q, const int* rows, int n_seqs,
                                      const int* walks, int n_walks, const int* chunks, int n_chunks, float* starts, float* out, int heads,
                                      int groups, int dim, int v_dim, int* status, cudaStream_t stream) {
    if (n_walks == 0 || n_chunks == 0) return cudaSuccess;
    if (!state_space_chunks_supports(heads, groups, dim, v_dim) || u_stride % 8 || ((uintptr_t)u & 15) || ((uintptr_t)state & 15) ||
        ((uintptr_t)starts & 15))
        return cudaErrorInvalidValue;
    ChunkArgs a = {(const __nv_bfloat16*)u, u_stride, (const __nv_bfloat16*)y, stride, dt_col, a_log, dt_bias, d, state, state_rows, cu_q, rows,
                   n_seqs, reinterpret_cast<const int2*>(walks), reinterpret_cast<const int2*>(chunks), starts, out, heads, groups, dim, v_dim,
                   status};
    cudaError_t e = dim <= 64 ? launch_walk<1, 2>(a, n_walks, stream)
                    : dim <= 128 ? launch_walk<1, 1>(a, n_walks, stream)
                                 : launch_walk<2, 1>(a, n_walks, stream);
    if (e != cudaSuccess) return e;
    return dim <= 32 ? launch_out<32>(a, n_chunks, stream)
           : dim <= 64 ? launch_out<64>(a, n_chunks, stream)
           : dim <= 128 ? launch_out<128>(a, n_chunks, stream)
                        : launch_out<256>(a, n_chunks, stream);
}

}  // namespace vtb
