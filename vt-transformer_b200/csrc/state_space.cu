// State-space mixers: a recurrence with one decay a (token, head), whose keys and queries are shared by groups of heads.
//
// For one head with state S [dim, v_dim] in 32-bit, d_t = softplus(raw step + bias) and a = exp(A_log):
//   S <- exp(-a d_t) S + d_t B_t x_t^T,   y_t = S^T C_t + D x_t
// x (a head's own), B and C (a group's) are the outputs of one causal convolution over time.
//
// Kernels here:
//   causal_conv      the convolution with its bias and silu over the step's tokens, its last inputs kept for each request
//   state_space_scan the recurrence token by token: a CTA a (sequence, head, block of columns), the state in registers
#include "attention_mma.cuh"
#include "common.cuh"
#include "kernels.h"
#include "launch.cuh"

namespace vtb {

namespace {

// softplus without a threshold: max(z, 0) + log(1 + exp(-|z|))
__device__ __forceinline__ float softplus_all(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_of(float z) { return z / (1.f + expf(-z)); }

__device__ __forceinline__ float silu_fast(float z) {
    // the power of two and the reciprocal by the hardware's approximations, for a result that is rounded to 16 bits
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(z * -1.4426950408889634f));
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(r) : "f"(1.f + e));
    return z * r;
}

// VEC consecutive values as they lie, fetched ahead of their use.
template <typename T, int VEC> struct Fetched {
    T v[VEC];
    __device__ __forceinline__ void load(const T* p) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = p[i];
    }
    __device__ __forceinline__ float get(int i) const { return to_float(v[i]); }
};
template <> struct Fetched<__nv_bfloat16, 4> {
    uint2 q;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { q = *reinterpret_cast<const uint2*>(p); }
    __device__ __forceinline__ float get(int i) const {
        const uint32_t w = i < 2 ? q.x : q.y;
        return __uint_as_float((i & 1) ? (w & 0xffff0000u) : (w << 16));
    }
};
template <> struct Fetched<float, 4> {
    float4 q;
    __device__ __forceinline__ void load(const float* p) { q = *reinterpret_cast<const float4*>(p); }
    __device__ __forceinline__ float get(int i) const { return i == 0 ? q.x : (i == 1 ? q.y : (i == 2 ? q.z : q.w)); }
};

// VEC consecutive values as floats, and back.
template <typename T, int VEC> __device__ __forceinline__ void load_values(const T* p, float (&f)[VEC]) {
    Fetched<T, VEC> v;
    v.load(p);
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = v.get(i);
}
template <typename T, int VEC> __device__ __forceinline__ void store_values(T* p, const float (&f)[VEC]) {
    if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
    else if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) p[i] = from_float<T>(f[i]);
    }
}

}  // namespace

// ------------------------------------------------------------------------- causal convolution over a step's tokens

// A CTA: a tile of up to `per_tile` tokens of one sequence, threadIdx.x * VEC channels on; a thread walks the tile's tokens
// with the last MAXT - 1 inputs of its channels in registers.  out[t, c] = act(bias[c] + sum_j w[j, c] in[t - taps + 1 + j, c])
// with in[t, c] = y[t, col + c], the taps added oldest first.  The rows before a sequence's first token of the step come from
// tail [rows, taps - 1, channels] (oldest first).  A tile has at least taps - 1 tokens unless it is its sequence's last, so
// only a sequence's first tile reads the tail, and its threads renew it (each its own channels).
// With fewer than MAXT taps the missing ones (the oldest) have weight zero.
template <typename T, int VEC, int MAXT>      // MAXT at least 2
__global__ void __launch_bounds__(128)
causal_conv_kernel(const T* __restrict__ y, int stride, int col, int channels, const float* __restrict__ w, int taps,
                   const float* __restrict__ bias, int act, float* __restrict__ tail, int state_rows, const int* __restrict__ cu_q,
                   const int* __restrict__ seq_rows, int n_seqs, const int2* __restrict__ tiles, int per_tile, T* __restrict__ out,
                   int* status) {
    pdl_launch();
    const int c0 = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    const bool live = c0 < channels;
    float wt[MAXT][VEC], b[VEC];
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
        const int tap = j - (MAXT - taps);
#pragma unroll
        for (int v = 0; v < VEC; ++v) wt[j][v] = 0.f;
        if (live && tap >= 0) load_values<float, VEC>(w + (size_t)tap * channels + c0, wt[j]);
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) b[v] = 0.f;
    if (live && bias != nullptr) load_values<float, VEC>(bias + c0, b);
    const int seq = tiles ? tiles[blockIdx.x].x : blockIdx.x;
    const int first = tiles ? tiles[blockIdx.x].y : 0;
    const bool seq_ok = seq >= 0 && seq < n_seqs;
    const int t0 = seq_ok ? cu_q[seq] : 0, t1 = seq_ok ? cu_q[seq + 1] : 0;
    const int row = seq_ok ? seq_rows[seq] : 0;
    pdl_wait();
    if (!seq_ok) {
        if (threadIdx.x == 0) set_status(status, kStatusBadSequence, seq);
        return;
    }
    const int a = t0 + first, e = min(t1, a + per_tile);
    if (a >= e || !live) return;
    const int kept = taps - 1;
    if (kept > 0 && (row < 0 || row >= state_rows)) {
        if (threadIdx.x == 0) set_status(status, kStatusBadRow, row);
        return;
    }
    const T* in = y + col + c0;
    constexpr int PAST = MAXT - 1, AHEAD = 4;
    float win[PAST + AHEAD][VEC];     // the PAST inputs in front of the present four, and these
#pragma unroll
    for (int j = 0; j < PAST; ++j) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) win[j][v] = 0.f;
        const int back = PAST - j, s = a - back;
        if (back <= kept) {
            if (s >= t0) load_values<T, VEC>(in + (size_t)s * stride, win[j]);
            else load_values<float, VEC>(tail + ((size_t)row * kept + kept - (t0 - s)) * channels + c0, win[j]);
        }
    }
    // four tokens' inputs are fetched while the four before them are worked on
    Fetched<T, VEC> next[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) next[k].load(in + (size_t)min(a + k, e - 1) * stride);
    if (first == 0 && kept > 0) {
        // the kept inputs after the step: its last tokens and, where it brings fewer, what was kept before (a thread reads slot
        // i + n after it has written the slots below i only, so the shift is safe in place)
        const int n = t1 - t0;
        float* tr = tail + (size_t)row * kept * channels + c0;
        for (int i = 0; i < kept; ++i) {
            const int s = t1 - kept + i;
            float v[VEC];
            if (s >= t0) load_values<T, VEC>(in + (size_t)s * stride, v);
            else load_values<float, VEC>(tr + (size_t)(i + n) * channels, v);
            store_values<float, VEC>(tr + (size_t)i * channels, v);
        }
    }
    for (int t = a; t < e; t += AHEAD) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k)
#pragma unroll
            for (int v = 0; v < VEC; ++v) win[PAST + k][v] = next[k].get(v);
        if (t + AHEAD < e) {
#pragma unroll
            for (int k = 0; k < AHEAD; ++k) next[k].load(in + (size_t)min(t + AHEAD + k, e - 1) * stride);
        }
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            if (t + k >= e) break;
            float o[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                float s = b[v];
#pragma unroll
                for (int j = 0; j < MAXT; ++j) s = fmaf(wt[j][v], win[k + j][v], s);
                o[v] = !act ? s : (sizeof(T) == 2 ? silu_fast(s) : silu_of(s));
            }
            store_values<T, VEC>(out + (size_t)(t + k) * channels + c0, o);
        }
#pragma unroll
        for (int j = 0; j < PAST; ++j)
#pragma unroll
            for (int v = 0; v < VEC; ++v) win[j][v] = win[AHEAD + j][v];
    }
}

template <typename T>
static cudaError_t launch_causal_conv_t(const void* y, int stride, int col, int channels, const float* w, int taps, const float* bias, int act,
                                        float* tail, int state_rows, const int* cu_q, const int* seq_rows, int n_seqs, const int* tiles,
                                        int n_tiles, int per_tile, void* out, int* status, cudaStream_t stream) {
    const bool vec = stride % 4 == 0 && col % 4 == 0 && channels % 4 == 0 && ((uintptr_t)y & 15) == 0 && ((uintptr_t)out & 15) == 0 &&
                     ((uintptr_t)w & 15) == 0 && ((uintptr_t)bias & 15) == 0 && ((uintptr_t)tail & 15) == 0 && taps <= 4;
    const int per_cta = 128 * (vec ? 4 : 1);
    const dim3 grid(n_tiles, (channels + per_cta - 1) / per_cta);
    auto kernel = vec ? causal_conv_kernel<T, 4, 4> : (taps <= 4 ? causal_conv_kernel<T, 1, 4> : causal_conv_kernel<T, 1, 16>);
    return launch(kernel, grid, dim3(128), 0, stream, (const T*)y, stride, col, channels, w, taps, bias, act, tail, state_rows, cu_q, seq_rows,
                  n_seqs, reinterpret_cast<const int2*>(tiles), per_tile, (T*)out, status);
}

cudaError_t launch_causal_conv(int dtype, const void* y, int stride, int col, int channels, const float* w, int taps, const float* bias, int act,
                               float* tail, int state_rows, const int* cu_q, const int* seq_rows, int n_seqs, const int* tiles, int n_tiles,
                               int per_tile, void* out, int* status, cudaStream_t stream) {
    if (n_tiles == 0 || channels == 0) return cudaSuccess;
    if (taps < 1 || taps > 16 || per_tile < max(1, taps - 1)) return cudaErrorInvalidValue;
    if (dtype == kBF16)
        return launch_causal_conv_t<__nv_bfloat16>(y, stride, col, channels, w, taps, bias, act, tail, state_rows, cu_q, seq_rows, n_seqs, tiles,
                                                   n_tiles, per_tile, out, status, stream);
    return launch_causal_conv_t<float>(y, stride, col, channels, w, taps, bias, act, tail, state_rows, cu_q, seq_rows, n_seqs, tiles, n_tiles,
                                       per_tile, out, status, stream);
}

// ------------------------------------------------------------------------- the recurrence, token by token

namespace {
constexpr int kScanQuads = 16;       // quads of columns that a CTA owns: 64 columns
constexpr int kScanGroups = 16;      // groups of rows: row r of the state belongs to group r % 16
constexpr int kScanBatch = 8;        // tokens staged in shared memory at once
}

struct SpaceArgs {
    const void* u;                   // [tokens, u_stride]: x at 0, B at heads * v_dim, C behind it
    int u_stride;
    const void* y;                   // [tokens, stride]: the raw step sizes at dt_col + h
    int stride, dt_col;
    const float *a_log, *dt_bias, *d;   // [heads] each
    float* state;                    // [state_rows, heads, dim, v_dim]
    int state_rows;
    const int* cu_q;
    const int* rows;
    const int* seqs;                 // [grid.x]: which sequences of the step run here; null: all
    int n_seqs;
    float* out;                      // [tokens, heads * v_dim]
    int heads, groups, dim, v_dim;
    int* status;
};

// Thread (quad, group) keeps rows group, group + 16, ... (KD of them) of the four columns 4 quad .. 4 quad + 3 of its CTA's 64.
// A token's sum over the rows: each thread its own rows in rising order, the two groups of a warp, then the eight warps in their
// order: fixed by the sizes, never by how the tokens were cut into steps.
template <typename T, int KD, bool QUADS>
__global__ void __launch_bounds__(256)
state_space_scan_kernel(const SpaceArgs a) {
    extern __shared__ __align__(16) float smem[];
    pdl_launch();
    const int seq = a.seqs ? a.seqs[blockIdx.x] : blockIdx.x, h = blockIdx.y;
    const int quad = threadIdx.x & (kScanQuads - 1), grp = threadIdx.x / kScanQuads;
    const int col0 = blockIdx.z * 4 * kScanQuads, j0 = col0 + quad * 4;
    const int dim = a.dim, v_dim = a.v_dim;
    const int dim_p = KD * kScanGroups;
    const int g = h / (a.heads / a.groups);
    float* bs = smem;                                   // [batch, dim_p]
    float* cs = bs + kScanBatch * dim_p;                // [batch, dim_p]
    float* xs = cs + kScanBatch * dim_p;                // [batch, 64]
    float* sc = xs + kScanBatch * 64;                   // [batch, 2]: decay, step size
    float* part = sc + kScanBatch * 2;                  // [batch, 8 warps, 64]
    const float rate = expf(a.a_log[h]), bias = a.dt_bias[h], skip = a.d[h];
    const bool seq_ok = seq >= 0 && seq < a.n_seqs;
    const int t0 = seq_ok ? a.cu_q[seq] : 0, t1 = seq_ok ? a.cu_q[seq + 1] : 0;
    const int row = seq_ok ? a.rows[seq] : 0;
    pdl_wait();
    if (t1 <= t0) return;                               // a sequence without tokens in this step (padding): its state stays
    if (row < 0 || row >= a.state_rows) {
        if (threadIdx.x == 0) set_status(a.status, kStatusBadRow, row);
        return;
    }
    float* sp = a.state + ((size_t)row * a.heads + h) * dim * v_dim;
    float S[KD][4];
#pragma unroll
    for (int i = 0; i < KD; ++i) {
        const int r = grp + i * kScanGroups;
#pragma unroll
        for (int k = 0; k < 4; ++k) S[i][k] = 0.f;
        if (r < dim) {
            if (QUADS) {
                if (j0 < v_dim) *reinterpret_cast<float4*>(S[i]) = *reinterpret_cast<const float4*>(sp + (size_t)r * v_dim + j0);
            } else {
#pragma unroll
                for (int k = 0; k < 4; ++k) if (j0 + k < v_dim) S[i][k] = sp[(size_t)r * v_dim + j0 + k];
            }
        }
    }
    const T* u = reinterpret_cast<const T*>(a.u);
    const T* y = reinterpret_cast<const T*>(a.y);
    const int inner = a.heads * v_dim, b_col = inner + g * dim, c_col = inner + (a.groups + g) * dim;
    for (int tb0 = t0; tb0 < t1; tb0 += kScanBatch) {
        const int n = min(kScanBatch, t1 - tb0);
        __syncthreads();
        for (int e = threadIdx.x; e < n * dim_p; e += 256) {
            const int tb = e / dim_p, i = e % dim_p;
            const T* ur = u + (size_t)(tb0 + tb) * a.u_stride;
            bs[e] = i < dim ? to_float(ur[b_col + i]) : 0.f;
            cs[e] = i < dim ? to_float(ur[c_col + i]) : 0.f;
        }
        for (int e = threadIdx.x; e < n * 64; e += 256) {
            const int tb = e / 64, i = col0 + e % 64;
            xs[e] = i < v_dim ? to_float(u[(size_t)(tb0 + tb) * a.u_stride + h * v_dim + i]) : 0.f;
        }
        if (threadIdx.x < n) {
            const float step = softplus_all(to_float(y[(size_t)(tb0 + threadIdx.x) * a.stride + a.dt_col + h]) + bias);
            sc[2 * threadIdx.x] = expf(-rate * step);
            sc[2 * threadIdx.x + 1] = step;
        }
        __syncthreads();
        for (int tb = 0; tb < n; ++tb) {
            const float decay = sc[2 * tb], step = sc[2 * tb + 1];
            const float4 x = *reinterpret_cast<const float4*>(xs + tb * 64 + quad * 4);
            const float xv[4] = {step * x.x, step * x.y, step * x.z, step * x.w};
            float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < KD; ++i) {
                const float b = bs[tb * dim_p + grp + i * kScanGroups], c = cs[tb * dim_p + grp + i * kScanGroups];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    S[i][k] = fmaf(decay, S[i][k], b * xv[k]);
                    o[k] = fmaf(S[i][k], c, o[k]);
                }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) o[k] += __shfl_xor_sync(0xffffffffu, o[k], 16);
            if ((threadIdx.x & 31) < 16)
                *reinterpret_cast<float4*>(part + (tb * 8 + (threadIdx.x >> 5)) * 64 + quad * 4) = make_float4(o[0], o[1], o[2], o[3]);
        }
        __syncthreads();
        for (int e = threadIdx.x; e < n * 64; e += 256) {
            const int tb = e / 64, i = e % 64;
            if (col0 + i >= v_dim) continue;
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) o += part[(tb * 8 + w) * 64 + i];
            a.out[(size_t)(tb0 + tb) * inner + (size_t)h * v_dim + col0 + i] = fmaf(skip, xs[e], o);
        }
    }
#pragma unroll
    for (int i = 0; i < KD; ++i) {
        const int r = grp + i * kScanGroups;
        if (r < dim) {
            if (QUADS) {
                if (j0 < v_dim) *reinterpret_cast<float4*>(sp + (size_t)r * v_dim + j0) = *reinterpret_cast<const float4*>(S[i]);
            } else {
#pragma unroll
                for (int k = 0; k < 4; ++k) if (j0 + k < v_dim) sp[(size_t)r * v_dim + j0 + k] = S[i][k];
            }
        }
    }
}

template <typename T, int KD>
static cudaError_t launch_space_scan_kd(const SpaceArgs& a, int n, cudaStream_t stream) {
    const bool quads = a.v_dim % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const size_t bytes = sizeof(float) * ((size_t)kScanBatch * (2 * KD * kScanGroups + 64 + 2 + 8 * 64));
    const dim3 grid(n, a.heads, (a.v_dim + 63) / 64);
    auto kernel = quads ? state_space_scan_kernel<T, KD, true> : state_space_scan_kernel<T, KD, false>;
    if (bytes > 48 * 1024) {
        static std::atomic<unsigned long long> done[2] = {{0}, {0}};
        if (cudaError_t e = allow_dynamic_smem(kernel, 64 * 1024, done[quads ? 1 : 0]); e != cudaSuccess) return e;
    }
    return launch(kernel, grid, dim3(256), bytes, stream, a);
}

template <typename T>
static cudaError_t launch_space_scan_t(const SpaceArgs& a, int n, cudaStream_t stream) {
    if (a.dim <= 4 * kScanGroups) return launch_space_scan_kd<T, 4>(a, n, stream);
    if (a.dim <= 8 * kScanGroups) return launch_space_scan_kd<T, 8>(a, n, stream);
    if (a.dim <= 16 * kScanGroups) return launch_space_scan_kd<T, 16>(a, n, stream);
    return launch_space_scan_kd<T, 32>(a, n, stream);
}

cudaError_t launch_state_space_scan(int dtype, const void* u, int u_stride, const void* y, int stride, int dt_col, const float* a_log,
                                    const float* dt_bias, const float* d, float* state, int state_rows, const int* cu_q, const int* rows,
                                    int n_seqs, const int* seqs, int n_listed, float* out, int heads, int groups, int dim, int v_dim, int* status,
                                    cudaStream_t stream) {
    const int n = seqs ? n_listed : n_seqs;
    if (n == 0) return cudaSuccess;
    if (dim < 1 || dim > 32 * kScanGroups || groups < 1 || heads % groups) return cudaErrorInvalidValue;
    SpaceArgs a = {u, u_stride, y, stride, dt_col, a_log, dt_bias, d, state, state_rows, cu_q, rows, seqs, n_seqs, out, heads, groups, dim,
                   v_dim, status};
    return dtype == kBF16 ? launch_space_scan_t<__nv_bfloat16>(a, n, stream) : launch_space_scan_t<float>(a, n, stream);
}

}  // namespace vtb
