// Shared pieces of the recurrence scans: packed fp32 pairs, rows into shared memory.
#pragma once

#include "hybrid.cuh"
#include "../pipeline.cuh"

namespace b200 {
namespace hybrid {

// Two fp32 values in one register pair: packed multiply-adds, each half rounded as a single one.
__device__ __forceinline__ unsigned long long pack2(float a, float b) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack2(unsigned long long v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
// One row of `n` elements to shared memory by a warp: 16-byte asynchronous copies where the row allows them.
template <typename E>
__device__ __forceinline__ void fetch_row(E* dst, const E* src, int n, bool wide, int lane) {
    constexpr int VE = 16 / (int)sizeof(E);
    if (wide)
        for (int c = lane * VE; c < n; c += 32 * VE) cp_async16(smem_u32(dst + c), src + c);
    else
        for (int c = lane; c < n; c += 32) dst[c] = src[c];
}

}  // namespace hybrid
}  // namespace b200
