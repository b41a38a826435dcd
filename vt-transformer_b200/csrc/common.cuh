// Shared device helpers of the sm_100a kernels.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace vtb {

// Codes a kernel leaves in the status word when it meets an index it must not follow.
// The kernel skips the access and goes on; the host reads the word after the step.
enum StatusCode : int {
    kStatusOk = 0,
    kStatusBadTokenId = 1,     // token id outside the embedding table
    kStatusBadPosition = 2,    // position outside the rotation table
    kStatusBadPage = 3,        // block table entry outside the page pool
    kStatusBadSequence = 4,    // token's sequence index outside the step
    kStatusBadRow = 5,         // row index outside the tensor
    kStatusWaitTimeout = 6,    // a bounded wait on a barrier ran out
};

__device__ __forceinline__ void set_status(int* status, int code, int detail) {
    if (status != nullptr && atomicCAS(status, 0, code) == 0) {
        status[1] = detail;
    }
}

// Programmatic dependent launch: every kernel of this library is launched so that it may start
// while the kernel before it in the stream is still running.  `pdl_launch` lets the next kernel's
// CTAs be scheduled as soon as there is room; `pdl_wait` returns when the kernels before have
// completed and their writes are visible.  A kernel calls both at its top, before it reads or
// writes global memory, so only set-up that touches no global data overlaps.
__device__ __forceinline__ void pdl_launch() { asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }

template <typename T> __device__ __forceinline__ float to_float(T v);
template <> __device__ __forceinline__ float to_float<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_float<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// The first key that a token at position `pos` sees: key 0; with a window, the first of the last `window` keys; with
// chunks, the first of its own chunk of `chunk` positions (chunks are counted from position 0 of the sequence); the
// later of the two where both are given.  It never falls as the position grows.
__device__ __forceinline__ int first_visible_key(int pos, int window, int chunk) {
    int lo = (window > 0) ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    return lo;
}

// tanh(x) for a score that is capped, given x2 = 2 x log2(e): 1 - 2 / (1 + e^(2x)), the power of two and the reciprocal by the hardware's
// approximations.  The absolute error stays within a few 2^-22 (near zero the difference cancels, which a cap's absolute scale
// allows); both ends come out as -1 and 1.
__device__ __forceinline__ float cap_tanh(float x2) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(x2));
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(r) : "f"(1.f + e));
    return fmaf(-2.f, r, 1.f);
}

// The clamped gate of a feed-forward: g = min(gate, limit), u = clamp(up, -limit, limit), g * sigmoid(alpha g) * (u + 1).
__device__ __forceinline__ float gate_clamp(float g, float u, float alpha, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  `scratch` holds
// 32 floats of shared memory.  The order of the additions depends on the block size only.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    const int nwarps = (blockDim.x + 31) >> 5;
    float r = (lane < nwarps) ? scratch[lane] : 0.f;
    r = warp_sum(r);
    return r;
}

// Eight consecutive elements as floats (16-byte load for bfloat16, two for float).
template <typename T> struct Vec8;
template <> struct Vec8<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[8]) {
        uint4 u = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float2 t = __bfloat1622float2(h[i]);
            f[2 * i] = t.x;
            f[2 * i + 1] = t.y;
        }
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[8]) {
        uint4 u;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = u;
    }
};
template <> struct Vec8<float> {
    static __device__ __forceinline__ void load(const float* p, float (&f)[8]) {
        float4 a = *reinterpret_cast<const float4*>(p);
        float4 b = *reinterpret_cast<const float4*>(p + 4);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
        f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&f)[8]) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
    }
};

}  // namespace vtb
