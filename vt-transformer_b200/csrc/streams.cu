// Kernels of models whose residual is several streams side by side, and of what stands before their sublayers: the
// embedding with a second table looked up by pairs of tokens, the step from one sublayer to the next (streams mixed and
// added to, read as one vector, normed), and the short causal convolution over what a sublayer reads.
//
// x [tokens, S, width] holds a token's S streams one behind the other (32-bit).  A sublayer reads u = sum_s in[s] x_s,
// normed; its result y changes all streams at once: x_t <- sum_s mix[s, t] x_s + out[t] y.  The kernel that prepares the
// next sublayer's input applies the change of the sublayer before it while it has the token's streams in its registers, so
// that they are read and written once a sublayer.
#include "common.cuh"
#include "kernels.h"
#include "launch.cuh"

namespace vtb {

namespace {

// four consecutive values as floats
template <typename T> struct Vec4;
template <> struct Vec4<float> {
    static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&f)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    }
};
template <> struct Vec4<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[4]) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
        const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[4]) {
        uint2 u;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
        h[0] = __floats2bfloat162_rn(f[0], f[1]);
        h[1] = __floats2bfloat162_rn(f[2], f[3]);
        *reinterpret_cast<uint2*>(p) = u;
    }
};

constexpr int kMaxStreams = 16;
constexpr int kMaxTaps = 16;
constexpr int kStreamThreads = 512;
constexpr int kMaxWidth = 12288;       // two rows of a token's values in 32-bit lie in shared memory where the block is narrower

}  // namespace

// ------------------------------------------------------------------------- embedding by token and by pair of tokens

// One block a token: v = table[id] + second[row] with row = (id before * mul_prev + id * mul_cur) mod buckets, row number
// `buckets` for a sequence's first token; with `weight`, v is divided by its root mean square and multiplied by the
// weight; every one of the `streams` rows of x[t] takes the result.  The token in front of a sequence's first token of
// the step is what the sequence's state holds; the block of that first token leaves the step's last token there (no
// other block touches the state).
template <typename T>
__global__ void embedding_pair_kernel(const T* __restrict__ table, const T* __restrict__ second, const int* __restrict__ ids,
                                      const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ cu_q,
                                      const int* __restrict__ rows, int n_seqs, int* __restrict__ state, int state_rows,
                                      const float* __restrict__ weight, float eps, float* __restrict__ x, int streams, int width, int vocab,
                                      long long buckets, long long mul_prev, long long mul_cur, int* status) {
    __shared__ float scratch[32];
    __shared__ long long row_of;
    extern __shared__ __align__(16) float vs[];
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t], seq = token_seq[t];
    float* xt = x + (size_t)t * streams * width;
    const bool live = seq >= 0 && seq < n_seqs && id >= 0 && id < vocab;
    if (threadIdx.x == 0) {
        row_of = -1;
        if (seq >= n_seqs) set_status(status, kStatusBadSequence, seq);
        if (seq >= 0 && seq < n_seqs) {
            const int first = cu_q[seq], last = cu_q[seq + 1] - 1, row = rows[seq];
            const bool row_ok = row >= 0 && row < state_rows;
            if (!row_ok) set_status(status, kStatusBadRow, row);
            long long r = buckets;
            if (positions[t] > 0 && (t > first || row_ok)) {
                const long long before = t > first ? ids[t - 1] : state[row];
                r = (before * mul_prev + (long long)id * mul_cur) % buckets;
                if (r < 0) r += buckets;
            }
            if (t == first && row_ok && last >= first) state[row] = ids[last];
            row_of = r;
        }
        if (id >= vocab) set_status(status, kStatusBadTokenId, id);
    }
    __syncthreads();
    if (!live) {            // padding, or an id that no table holds: rows of zeros
        for (int i = threadIdx.x; i < streams * width; i += blockDim.x) xt[i] = 0.f;
        return;
    }
    const T* a = table + (size_t)id * width;
    const T* b = second + (size_t)row_of * width;
    float ss = 0.f;
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
        float v[4], w[4];
        Vec4<T>::load(a + i, v);
        Vec4<T>::load(b + i, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            v[j] += w[j];
            ss = fmaf(v[j], v[j], ss);
        }
        Vec4<float>::store(vs + i, v);
    }
    const float rs = weight ? rsqrtf(block_sum(ss, scratch) / (float)width + eps) : 1.f;
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
        float v[4], w[4] = {1.f, 1.f, 1.f, 1.f};
        Vec4<float>::load(vs + i, v);                   // this thread's own values
        if (weight) Vec4<float>::load(weight + i, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = v[j] * rs * w[j];
        for (int s = 0; s < streams; ++s) Vec4<float>::store(xt + (size_t)s * width + i, v);
    }
}

cudaError_t launch_embedding_pair(int dtype, const void* table, const void* second, const int* ids, const int* positions,
                                  const int* token_seq, const int* cu_q, const int* rows, int n_seqs, int* state, int state_rows,
                                  const float* weight, float eps, float* x, int streams, int n_tokens, int width, int vocab,
                                  long long buckets, long long mul_prev, long long mul_cur, int* status, cudaStream_t stream) {
    if (n_tokens == 0) return cudaSuccess;
    if (width % 8 || width > kMaxWidth || streams < 1 || buckets < 1) return cudaErrorInvalidValue;
    const int threads = min(kStreamThreads, max(32, ((width / 4 + 31) / 32) * 32));
    const size_t bytes = (size_t)width * sizeof(float);
    if (dtype == kBF16)
        return launch(embedding_pair_kernel<__nv_bfloat16>, n_tokens, threads, bytes, stream, (const __nv_bfloat16*)table,
                      (const __nv_bfloat16*)second, ids, positions, token_seq, cu_q, rows, n_seqs, state, state_rows, weight, eps, x,
                      streams, width, vocab, buckets, mul_prev, mul_cur, status);
    return launch(embedding_pair_kernel<float>, n_tokens, threads, bytes, stream, (const float*)table, (const float*)second, ids, positions,
                  token_seq, cu_q, rows, n_seqs, state, state_rows, weight, eps, x, streams, width, vocab, buckets, mul_prev, mul_cur,
                  status);
}

// ------------------------------------------------------------------------- from one sublayer to the next

struct StreamsParams {
    float* x;                        // [n_tokens, S, width]
    const float* parts;              // the result of the sublayer before as n_parts unadded shares [n_parts, n_tokens, width]
    int n_parts;
    const float* mix;                // [S, S] (from, to) and out [S] of the sublayer before (null: nothing to apply)
    const float* w_out;
    const float* w_in;               // [S]
    const float* weight;             // the norm's [width]
    float eps;
    float* out32;                    // the normed rows in 32-bit instead of `out` (for a convolution over the step's tokens)
    const int* rows;                 // the tokens to do (null: all), packed in that order
    int n_tokens, width, S;
    int store;                       // 1: the changed streams go back to x
    // the convolution, for steps in which every sequence brings one token (or taps == 1): conv [taps, width], the last tap the
    // present row's, and tail [state_rows, taps - 1, width], the sequence's rows before, oldest first
    const float* conv;
    int taps;
    float* tail;
    int state_rows;
    const int* token_seq;
    const int* seq_rows;
    int n_seqs;
    int* status;
};

// One block a token, four columns a thread at a time.  CONV: h becomes h + conv(h) here (see StreamsParams::conv) and the
// tail moves on by one row.  SC: the number of streams where it is known when compiled (0: p.S).  The sum of squares has an
// order that depends on the width alone.
template <typename T, int SC, bool CONV>
__global__ void __launch_bounds__(kStreamThreads, CONV || SC == 0 ? 1 : 2)
streams_norm_kernel(const StreamsParams p, const T* __restrict__ delta, T* __restrict__ out) {
    constexpr int SM = SC > 0 ? SC : kMaxStreams;
    constexpr int kNear = 3;             // rows before that are fetched ahead (more, with more taps, one after the other)
    __shared__ float scratch[32];
    __shared__ float mix_s[SM * SM], out_s[SM], in_s[SM];
    extern __shared__ __align__(16) float us[];           // [width] u, [width] the tail's part of the convolution
    pdl_launch();
    const int S = SC > 0 ? SC : p.S, width = p.width;
    const bool change = p.mix != nullptr;
    // weights and the step's own description: written by no kernel of the step, read before the wait
    if (change) {
        for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix_s[i] = p.mix[i];
        if ((int)threadIdx.x < S) out_s[threadIdx.x] = p.w_out[threadIdx.x];
    }
    if ((int)threadIdx.x < S) in_s[threadIdx.x] = p.w_in[threadIdx.x];
    const int r = blockIdx.x;
    const int t = p.rows ? p.rows[r] : r;
    const bool t_ok = t >= 0 && t < p.n_tokens;
    float* tail = nullptr;
    if (CONV && p.taps > 1 && t_ok) {
        const int seq = p.token_seq[t];
        const int row = seq >= 0 && seq < p.n_seqs ? p.seq_rows[seq] : -1;
        if (row >= 0 && row < p.state_rows) tail = p.tail + (size_t)row * (p.taps - 1) * width;
        else if (seq >= 0 && threadIdx.x == 0) set_status(p.status, kStatusBadRow, row);
    }
    __syncthreads();
    pdl_wait();
    if (!t_ok) {
        if (threadIdx.x == 0) set_status(p.status, kStatusBadRow, t);
        return;
    }
    float* xt = p.x + (size_t)t * S * width;
    const size_t stride = (size_t)p.n_tokens * width;
    float ss = 0.f;
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
        // everything that is read comes before anything is written, so that the loads are in flight together
        float v[SM][4], u[4] = {0.f, 0.f, 0.f, 0.f}, d[4] = {0.f, 0.f, 0.f, 0.f}, before[kNear][4];
#pragma unroll
        for (int s = 0; s < SM; ++s)
            if (s < S) Vec4<float>::load(xt + (size_t)s * width + i, v[s]);
        if (CONV && tail != nullptr) {
#pragma unroll
            for (int k = 0; k < kNear; ++k)
                if (k < p.taps - 1) Vec4<float>::load(tail + (size_t)k * width + i, before[k]);
        }
        if (change) {
            if (delta != nullptr) {
                Vec4<T>::load(delta + (size_t)t * width + i, d);
            } else {
                for (int q0 = 0; q0 < p.n_parts; q0 += 4) {
                    float e[4][4];
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        if (q0 + q < p.n_parts) {
                            Vec4<float>::load(p.parts + (size_t)t * width + i + (q0 + q) * stride, e[q]);
                        } else {
                            e[q][0] = e[q][1] = e[q][2] = e[q][3] = 0.f;
                        }
                    }
#pragma unroll
                    for (int q = 0; q < 4; ++q)
#pragma unroll
                        for (int j = 0; j < 4; ++j) d[j] += e[q][j];
                }
            }
#pragma unroll
            for (int to = 0; to < SM; ++to) {
                if (to < S) {
                    float n[4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) n[j] = out_s[to] * d[j];
#pragma unroll
                    for (int s = 0; s < SM; ++s) {
                        if (s < S) {
                            const float m = mix_s[s * S + to];
#pragma unroll
                            for (int j = 0; j < 4; ++j) n[j] = fmaf(m, v[s][j], n[j]);
                        }
                    }
                    const float w = in_s[to];
#pragma unroll
                    for (int j = 0; j < 4; ++j) u[j] = fmaf(w, n[j], u[j]);
                    if (p.store) Vec4<float>::store(xt + (size_t)to * width + i, n);
                }
            }
        } else {
#pragma unroll
            for (int s = 0; s < SM; ++s)
                if (s < S) {
                    const float w = in_s[s];
#pragma unroll
                    for (int j = 0; j < 4; ++j) u[j] = fmaf(w, v[s][j], u[j]);
                }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) ss = fmaf(u[j], u[j], ss);
        Vec4<float>::store(us + i, u);
        if (CONV) {
            // what the rows before add, and the tail one row on (its last row follows below)
            float c[4] = {0.f, 0.f, 0.f, 0.f};
            if (tail != nullptr) {
#pragma unroll
                for (int k = 0; k < kNear; ++k) {
                    if (k < p.taps - 1) {
                        float w[4];
                        Vec4<float>::load(p.conv + (size_t)k * width + i, w);
#pragma unroll
                        for (int j = 0; j < 4; ++j) c[j] = fmaf(w[j], before[k][j], c[j]);
                        if (k > 0) Vec4<float>::store(tail + (size_t)(k - 1) * width + i, before[k]);
                    }
                }
                for (int k = kNear; k < p.taps - 1; ++k) {
                    float h[4], w[4];
                    Vec4<float>::load(tail + (size_t)k * width + i, h);
                    Vec4<float>::load(p.conv + (size_t)k * width + i, w);
#pragma unroll
                    for (int j = 0; j < 4; ++j) c[j] = fmaf(w[j], h[j], c[j]);
                    Vec4<float>::store(tail + (size_t)(k - 1) * width + i, h);
                }
            }
            Vec4<float>::store(us + width + i, c);
        }
    }
    const float rs = rsqrtf(block_sum(ss, scratch) / (float)width + p.eps);
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
        float u[4], w[4], h[4];
        Vec4<float>::load(us + i, u);                    // this thread's own values
        Vec4<float>::load(p.weight + i, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) h[j] = u[j] * rs * w[j];
        if (CONV) {
            float c[4], wl[4];
            Vec4<float>::load(us + width + i, c);
            Vec4<float>::load(p.conv + (size_t)(p.taps - 1) * width + i, wl);
            if (tail != nullptr) Vec4<float>::store(tail + (size_t)(p.taps - 2) * width + i, h);
#pragma unroll
            for (int j = 0; j < 4; ++j) h[j] += fmaf(wl[j], h[j], c[j]);
        }
        if (p.out32 != nullptr) Vec4<float>::store(p.out32 + (size_t)r * width + i, h);
        else Vec4<T>::store(out + (size_t)r * width + i, h);
    }
}

namespace {

template <typename T, bool CONV>
cudaError_t launch_streams_as(const StreamsParams& p, const void* delta, void* out, int n_rows, int threads, size_t bytes,
                              cudaStream_t stream) {
    switch (p.S) {
        case 1: return launch(streams_norm_kernel<T, 1, CONV>, n_rows, threads, bytes, stream, p, (const T*)delta, (T*)out);
        case 2: return launch(streams_norm_kernel<T, 2, CONV>, n_rows, threads, bytes, stream, p, (const T*)delta, (T*)out);
        case 3: return launch(streams_norm_kernel<T, 3, CONV>, n_rows, threads, bytes, stream, p, (const T*)delta, (T*)out);
        case 4: return launch(streams_norm_kernel<T, 4, CONV>, n_rows, threads, bytes, stream, p, (const T*)delta, (T*)out);
        default: return launch(streams_norm_kernel<T, 0, CONV>, n_rows, threads, bytes, stream, p, (const T*)delta, (T*)out);
    }
}

}  // namespace

cudaError_t launch_streams_norm(int out_dtype, float* x, int n_tokens, int streams, int width, const void* delta, const float* parts,
                                int n_parts, const float* mix, const float* w_out, const float* w_in, const float* weight, float eps,
                                void* out, float* out32, const int* rows, int n_rows, int store, const float* conv, int taps, float* tail,
                                int state_rows, const int* token_seq, const int* seq_rows, int n_seqs, int* status, cudaStream_t stream) {
    if (n_rows == 0) return cudaSuccess;
    if (width % 8 || width > kMaxWidth || streams < 1 || streams > kMaxStreams) return cudaErrorInvalidValue;
    if ((delta != nullptr && parts != nullptr) || (mix != nullptr) != (delta != nullptr || parts != nullptr)) return cudaErrorInvalidValue;
    if ((mix != nullptr) != (w_out != nullptr)) return cudaErrorInvalidValue;
    if ((out != nullptr) == (out32 != nullptr)) return cudaErrorInvalidValue;
    if (conv != nullptr && (taps < 1 || taps > kMaxTaps || (taps > 1 && (tail == nullptr || token_seq == nullptr || seq_rows == nullptr))))
        return cudaErrorInvalidValue;
    const StreamsParams p = {x, parts, n_parts, mix, w_out, w_in, weight, eps, out32, rows, n_tokens, width, streams, store, conv, taps, tail,
                             state_rows, token_seq, seq_rows, n_seqs, status};
    const int threads = min(kStreamThreads, max(32, ((width / 4 + 31) / 32) * 32));
    const size_t bytes = (size_t)width * sizeof(float) * (conv != nullptr ? 2 : 1);
    if (bytes > 48 * 1024) return cudaErrorInvalidValue;
    if (out_dtype == kBF16)
        return conv != nullptr ? launch_streams_as<__nv_bfloat16, true>(p, delta, out, n_rows, threads, bytes, stream)
                               : launch_streams_as<__nv_bfloat16, false>(p, delta, out, n_rows, threads, bytes, stream);
    return conv != nullptr ? launch_streams_as<float, true>(p, delta, out, n_rows, threads, bytes, stream)
                           : launch_streams_as<float, false>(p, delta, out, n_rows, threads, bytes, stream);
}

// ------------------------------------------------------------------------- a convolution over the rows of a step

// out[t] = h[t] + sum_j w[j] h[t - taps + 1 + j], the rows in front of a sequence's first row of the step from its tail
// [taps - 1, width] (oldest first).  A block: a tile (sequence, first of its new tokens) of up to `per_tile` >= taps - 1
// tokens and 4 columns a thread.  So only a sequence's first tile reads the tail, and the same threads leave the
// sequence's last taps - 1 rows there when they are done.  TC: taps where it is known when compiled (0: p_taps); the rows
// before then stay in registers while the tile is walked.
template <typename T, int TC>
__global__ void __launch_bounds__(128)
conv_rows_kernel(const float* __restrict__ h, const float* __restrict__ w, int p_taps, float* __restrict__ tail, int state_rows,
                 const int* __restrict__ cu_q, const int* __restrict__ seq_rows, const int2* __restrict__ tiles, int per_tile,
                 T* __restrict__ out, int width, int* status) {
    constexpr int KM = TC > 0 ? TC - 1 : kMaxTaps - 1;        // rows before
    const int kept = (TC > 0 ? TC : p_taps) - 1;
    pdl_launch();
    const int2 tile = tiles[blockIdx.x];
    const int t0 = cu_q[tile.x], t1 = cu_q[tile.x + 1];
    const int row = seq_rows[tile.x];
    const int i = (blockIdx.y * 128 + threadIdx.x) * 4;
    float wk[KM + 1][4];
    if (i < width) {
#pragma unroll
        for (int k = 0; k <= KM; ++k)
            if (k <= kept) Vec4<float>::load(w + (size_t)k * width + i, wk[k]);
    }
    pdl_wait();
    const int a = t0 + tile.y, b = min(t1, a + per_tile);
    if (i >= width || a >= b) return;
    if (row < 0 || row >= state_rows) {
        if (threadIdx.x == 0 && blockIdx.y == 0) set_status(status, kStatusBadRow, row);
        return;
    }
    float* tr = tail + (size_t)row * kept * width + i;
    // the rows before the tile, oldest first
    float before[KM][4];
#pragma unroll
    for (int k = 0; k < KM; ++k) {
        if (k < kept) {
            const int s = a - kept + k;
            if (s >= t0) Vec4<float>::load(h + (size_t)s * width + i, before[k]);
            else Vec4<float>::load(tr + (size_t)(s - t0 + kept) * width, before[k]);
        }
    }
    if (tile.y == 0) {
        // a short sequence keeps rows of its old tail: they move up before the new ones take their places
        const int n = t1 - t0;
#pragma unroll
        for (int k = 0; k < KM; ++k)
            if (k >= n && k < kept) Vec4<float>::store(tr + (size_t)(k - n) * width, before[k]);
        for (int k = max(0, kept - n); k < kept; ++k) {
            float v[4];
            Vec4<float>::load(h + (size_t)(t1 - kept + k) * width + i, v);
            Vec4<float>::store(tr + (size_t)k * width, v);
        }
    }
    for (int t = a; t < b; ++t) {
        float v[4], c[4] = {0.f, 0.f, 0.f, 0.f};
        Vec4<float>::load(h + (size_t)t * width + i, v);
#pragma unroll
        for (int k = 0; k < KM; ++k)
            if (k < kept) {
#pragma unroll
                for (int j = 0; j < 4; ++j) c[j] = fmaf(wk[k][j], before[k][j], c[j]);
            }
        float y[4];
        // (the last tap's index is a constant where the taps are known; the row itself is added last)
        if (TC > 0) {
#pragma unroll
            for (int j = 0; j < 4; ++j) y[j] = v[j] + fmaf(wk[KM][j], v[j], c[j]);
        } else {
            float wl[4];
            Vec4<float>::load(w + (size_t)kept * width + i, wl);
#pragma unroll
            for (int j = 0; j < 4; ++j) y[j] = v[j] + fmaf(wl[j], v[j], c[j]);
        }
        Vec4<T>::store(out + (size_t)t * width + i, y);
#pragma unroll
        for (int k = 0; k < KM; ++k) {
            if (k < kept) {
                const bool newest = k == kept - 1;
#pragma unroll
                for (int j = 0; j < 4; ++j) before[k][j] = newest ? v[j] : before[k + 1 < KM ? k + 1 : k][j];
            }
        }
    }
}

namespace {

template <typename T>
cudaError_t launch_conv_rows_as(const float* h, const float* w, int taps, float* tail, int state_rows, const int* cu_q, const int* seq_rows,
                                const int* tiles, int n_tiles, int per_tile, void* out, int width, int* status, cudaStream_t stream) {
    const dim3 grid(n_tiles, (width / 4 + 127) / 128);
    const int2* tl = reinterpret_cast<const int2*>(tiles);
    switch (taps) {
        case 2: return launch(conv_rows_kernel<T, 2>, grid, 128, 0, stream, h, w, taps, tail, state_rows, cu_q, seq_rows, tl, per_tile, (T*)out, width, status);
        case 3: return launch(conv_rows_kernel<T, 3>, grid, 128, 0, stream, h, w, taps, tail, state_rows, cu_q, seq_rows, tl, per_tile, (T*)out, width, status);
        case 4: return launch(conv_rows_kernel<T, 4>, grid, 128, 0, stream, h, w, taps, tail, state_rows, cu_q, seq_rows, tl, per_tile, (T*)out, width, status);
        default: return launch(conv_rows_kernel<T, 0>, grid, 128, 0, stream, h, w, taps, tail, state_rows, cu_q, seq_rows, tl, per_tile, (T*)out, width, status);
    }
}

}  // namespace

cudaError_t launch_conv_rows(int out_dtype, const float* h, const float* w, int taps, float* tail, int state_rows, const int* cu_q,
                             const int* seq_rows, const int* tiles, int n_tiles, int per_tile, void* out, int width, int* status,
                             cudaStream_t stream) {
    if (n_tiles == 0) return cudaSuccess;
    if (width % 8 || taps < 2 || taps > kMaxTaps || per_tile < taps - 1) return cudaErrorInvalidValue;
    if (out_dtype == kBF16)
        return launch_conv_rows_as<__nv_bfloat16>(h, w, taps, tail, state_rows, cu_q, seq_rows, tiles, n_tiles, per_tile, out, width, status, stream);
    return launch_conv_rows_as<float>(h, w, taps, tail, state_rows, cu_q, seq_rows, tiles, n_tiles, per_tile, out, width, status, stream);
}

// ------------------------------------------------------------------------- the square of relu

template <typename T>
__global__ void relu_square_kernel(const T* __restrict__ z, T* __restrict__ out, long long n) {
    pdl_launch();
    pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const float v = fmaxf(to_float(z[i]), 0.f);
        out[i] = from_float<T>(v * v);
    }
}

cudaError_t launch_relu_square(int dtype, const void* z, void* out, long long n, cudaStream_t stream) {
    if (n == 0) return cudaSuccess;
    const int blocks = (int)min((n + 255) / 256, (long long)148 * 16);
    if (dtype == kBF16)
        return launch(relu_square_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (const __nv_bfloat16*)z, (__nv_bfloat16*)out, n);
    return launch(relu_square_kernel<float>, blocks, 256, 0, stream, (const float*)z, (float*)out, n);
}

}  // namespace vtb
