// Shared helpers of libtiny_llm_b200_blocks.so (see include/tiny_llm_b200_blocks.h).
#pragma once

#include "../common.cuh"
#include "../../../include/tiny_llm_b200_blocks.h"

namespace tlb {

using tl::as_stream;
using tl::ceil_div;
using tl::from_f;
using tl::to_f;
using tl::warp_max;
using tl::warp_sum;

typedef __nv_bfloat16 bf16;

// Sum over a CTA of `blockDim.x` threads (a multiple of 32, at most 1024); every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float *scratch /* [33] */) {
    v = warp_sum(v);
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < (int)(blockDim.x >> 5) ? scratch[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// cos / sin of position * base^(-2 i / dims), evaluated in double so that the angle is exact at any position.
__device__ __forceinline__ void rope_angle(int pos, int i, int dims, double log2_base, float &c, float &s) {
    double freq = exp2(-2.0 * (double)i / (double)dims * log2_base);
    double sn, cs;
    sincos((double)pos * freq, &sn, &cs);
    c = (float)cs;
    s = (float)sn;
}

__device__ __forceinline__ float sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float act_apply(float z, int act) {
    if (act == 0) return z / (1.0f + expf(-z));
    float inner = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return 0.5f * z * (1.0f + tanhf(inner));
}

// The inside of a gated feed-forward: act(g) * u, or (act 3) the clamped form, the gate bounded from above and the other half on
// both sides: g sigmoid(slope g) (u + 1).
__device__ __forceinline__ float gated_pair(float g, float u, int act, float limit, float slope) {
    if (act == 3) {
        g = fminf(g, limit), u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-slope * g)) * (u + 1.0f);
    }
    return act_apply(g, act) * u;
}

// 4 consecutive elements of a row as floats (one 8- or 16-byte access)
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const bf16 *p) {
    uint2 u = *reinterpret_cast<const uint2 *>(p);
    float2 a = tl::unpack2<bf16>(u.x), b = tl::unpack2<bf16>(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(bf16 *p, float4 v) {
    *reinterpret_cast<uint2 *>(p) = make_uint2(tl::pack2<bf16>(v.x, v.y), tl::pack2<bf16>(v.z, v.w));
}

}  // namespace tlb

#define TLB_DISPATCH(dtype, name, ...)                                               \
    do {                                                                             \
        if ((dtype) == TL_F32) { using T = float; __VA_ARGS__; }                     \
        else if ((dtype) == TL_BF16) { using T = ::tlb::bf16; __VA_ARGS__; }         \
        else return ::tl::fail(TL_EDTYPE, "%s: dtype must be float32 or bfloat16", name); \
    } while (0)
