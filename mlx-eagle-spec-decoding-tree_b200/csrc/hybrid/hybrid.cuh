// Shared pieces of the layer-list ("hybrid") decoder kernels: activation types, the epilogues of the matrix products
// and the launch functions the pass driver calls.
#pragma once

#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "b200_hybrid.h"
#include "../common.cuh"

namespace b200 {
namespace hybrid {

// (Kernel parameters carry no __restrict__: the compiler would take what earlier kernels wrote for constant and could move
// its loads across the grid-dependency wait.)

using bf16 = __nv_bfloat16;

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

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
// Sum over the CTA (blockDim.x a multiple of 32, at most 1024); every thread gets it.  `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nw ? red[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) red[32] = t;
    }
    __syncthreads();
    return red[32];
}

// The sums of three values over the CTA at once.  `red` holds 99 floats.
__device__ __forceinline__ float3 block_sum3(float3 v, float* red) {
    v.x = warp_sum(v.x); v.y = warp_sum(v.y); v.z = warp_sum(v.z);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    __syncthreads();
    if (lane == 0) { red[warp] = v.x; red[33 + warp] = v.y; red[66 + warp] = v.z; }
    __syncthreads();
    if (warp < 3) {
        float t = lane < nw ? red[33 * warp + lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) red[33 * warp + 32] = t;
    }
    __syncthreads();
    return make_float3(red[32], red[65], red[98]);
}

__host__ __device__ constexpr int round_up(int v, int m) { return (v + m - 1) / m * m; }

// ---------------------------------------------------------------- epilogues of the matrix products
// A product's output columns are cut into segments; each has an operation on the fp32 accumulator and a destination.
enum : int {
    kOpNone = 0,        // acc
    kOpSilu = 1,        // silu(acc)
    kOpSigmoid = 2,     // sigmoid(acc)
    kOpForget = 3,      // 1 - f with f = l + (1 - l) sigmoid(acc + b):  (1 - l) sigmoid(-(acc + b))
    kOpResidual = 4,    // dst += mult * acc (+ add)
    kOpSoftcap = 5      // cap * tanh(acc / cap), cap <= 0: acc
};

struct Seg {
    int n0, n1;             // columns
    int op;
    int f32;                // destination is fp32 (else the activation type)
    void* dst;
    long long row_stride;   // elements between rows
    // column c of the segment: element (c / unit / maps) * group_stride + (c / unit % maps) * unit_pitch + c % unit of a row
    int unit, maps, unit_pitch;
    int at_cache_row;       // row m goes to row prefix[0] + write_off + m
    long long group_stride;
    const float* p0;        // kOpForget: bias and lower bound per column
    const float* p1;
};

struct Epi {
    int nseg, M;
    Seg seg[4];
    const int* prefix;
    int write_off;
    float mult;             // kOpResidual
    const float* add;       // kOpResidual: added too, laid out like dst (or null)
    float cap;              // kOpSoftcap
    __half* half_copy;      // kOpSoftcap: fp16 copy of the result, laid out like dst (or null)
};

inline Seg plain_seg(int n0, int n1, int op, int f32, void* dst, long long row_stride) {
    Seg s{};
    s.n0 = n0; s.n1 = n1; s.op = op; s.f32 = f32; s.dst = dst; s.row_stride = row_stride;
    s.unit = n1 - n0 > 0 ? n1 - n0 : 1; s.maps = 1; s.unit_pitch = 0; s.group_stride = 0;
    return s;
}

// One output column: where it goes and what is done to it.
template <typename T>
struct ColumnOut {
    int op, f32;
    char* base;             // null: not a column of the product
    long long stride;       // bytes between rows
    float p0, p1;
    __half* half_base;
    const char* add_base;

    __device__ __forceinline__ void init(const Epi& e, int n) {
        op = kOpNone; f32 = 1; base = nullptr; stride = 0; p0 = p1 = 0.f; half_base = nullptr; add_base = nullptr;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            if (i < e.nseg && n >= e.seg[i].n0 && n < e.seg[i].n1) {
                const Seg& s = e.seg[i];
                const int c = n - s.n0;
                const int u = c / s.unit, r = c - u * s.unit;
                const long long off = (long long)(u / s.maps) * s.group_stride + (long long)(u % s.maps) * s.unit_pitch + r;
                const int row0 = s.at_cache_row ? e.prefix[0] + e.write_off : 0;
                const int size = s.f32 ? 4 : (int)sizeof(T);
                op = s.op; f32 = s.f32;
                stride = s.row_stride * size;
                base = static_cast<char*>(s.dst) + off * size + row0 * stride;
                if (s.op == kOpForget) { p0 = s.p0[c]; p1 = s.p1[c]; }
                if (s.op == kOpSoftcap) {
                    p0 = e.cap;
                    if (e.half_copy != nullptr) half_base = e.half_copy + off;
                }
                if (s.op == kOpResidual) {
                    p0 = e.mult;
                    if (e.add != nullptr) add_base = reinterpret_cast<const char*>(e.add + off);
                }
            }
        }
    }
    __device__ __forceinline__ float finish(float acc, float residual) const {
        if (op == kOpSilu) return acc * sigmoid_f(acc);
        if (op == kOpSigmoid) return sigmoid_f(acc);
        if (op == kOpForget) return (1.0f - p1) * sigmoid_f(-(acc + p0));
        if (op == kOpResidual) return residual + p0 * acc;
        if (op == kOpSoftcap && p0 > 0.f) return p0 * tanhf(acc / p0);
        return acc;
    }
    __device__ __forceinline__ float residual(int m) const {
        float r = *reinterpret_cast<const float*>(base + (long long)m * stride);
        if (add_base != nullptr) r += *reinterpret_cast<const float*>(add_base + (long long)m * stride);
        return r;
    }
    __device__ __forceinline__ void put(int m, float v) const {
        char* p = base + (long long)m * stride;
        if (f32) *reinterpret_cast<float*>(p) = v;
        else *reinterpret_cast<T*>(p) = from_f32<T>(v);
        if (half_base != nullptr) half_base[(long long)m * (stride >> 2)] = __float2half_rn(v);
    }
    __device__ __forceinline__ void store(int m, float acc) const {
        if (base == nullptr) return;
        put(m, finish(acc, op == kOpResidual ? residual(m) : 0.f));
    }
    template <int OP, bool F32, int N>
    __device__ __forceinline__ void rows_of(int m0, int n, const uint32_t (&acc)[N]) const {
        char* p = base + (long long)m0 * stride;
        float r[N];
        if (OP == kOpResidual) {                     // all loads before the first store
#pragma unroll
            for (int i = 0; i < N; i++) r[i] = i < n ? *reinterpret_cast<const float*>(p + i * stride) : 0.f;
            if (add_base != nullptr) {
                const char* q = add_base + (long long)m0 * stride;
                float e[N];
#pragma unroll
                for (int i = 0; i < N; i++) e[i] = i < n ? *reinterpret_cast<const float*>(q + i * stride) : 0.f;
#pragma unroll
                for (int i = 0; i < N; i++) r[i] += e[i];
            }
        }
#pragma unroll
        for (int i = 0; i < N; i++) {
            float v = __uint_as_float(acc[i]);
            if (OP == kOpSilu) v = v * sigmoid_f(v);
            else if (OP == kOpSigmoid) v = sigmoid_f(v);
            else if (OP == kOpForget) v = (1.0f - p1) * sigmoid_f(-(v + p0));
            else if (OP == kOpResidual) v = r[i] + p0 * v;
            else if (OP == kOpSoftcap) v = p0 > 0.f ? p0 * tanhf(v / p0) : v;
            if (i < n) {
                if (F32) *reinterpret_cast<float*>(p + i * stride) = v;
                else *reinterpret_cast<T*>(p + i * stride) = from_f32<T>(v);
                if (OP == kOpSoftcap && half_base != nullptr) half_base[(long long)(m0 + i) * (stride >> 2)] = __float2half_rn(v);
            }
        }
    }
    // Rows m0 .. m0 + n - 1, n clipped to N: one branch on the operation, straight code for the rows.
    template <int N>
    __device__ __forceinline__ void store_rows(int m0, int n, const uint32_t (&acc)[N]) const {
        if (base == nullptr) return;
        switch (op) {
            case kOpNone: if (f32) rows_of<kOpNone, true>(m0, n, acc); else rows_of<kOpNone, false>(m0, n, acc); break;
            case kOpSilu: rows_of<kOpSilu, false>(m0, n, acc); break;
            case kOpSigmoid: rows_of<kOpSigmoid, false>(m0, n, acc); break;
            case kOpForget: rows_of<kOpForget, true>(m0, n, acc); break;
            case kOpResidual: rows_of<kOpResidual, true>(m0, n, acc); break;
            default: rows_of<kOpSoftcap, true>(m0, n, acc); break;
        }
    }
};

// ---------------------------------------------------------------- launches
// x: activations [x_rows][lin.pitch] of type act_type; x_rows bounds what may be read.
int launch_linear(int act_type, const b200_linear& lin, const void* x, int x_rows, const Epi& epi, int* error, cudaStream_t st);

int launch_embed(const b200_hybrid_model& m, const b200_hybrid_pass& p, cudaStream_t st);
int launch_norm_conv(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r,
                     const b200_hybrid_pass& p, cudaStream_t st);
// x / rms(x) * w into the product-input buffer; with `gather` the rows named by out_rows / row_index.
int launch_norm(const b200_hybrid_model& m, const float* w, const b200_hybrid_pass& p, bool gather, int rows, cudaStream_t st);
int launch_polynorm(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st);
int launch_add(float* x, const float* y, size_t n, cudaStream_t st);
int launch_attention(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r,
                     const b200_hybrid_pass& p, cudaStream_t st);
int launch_recurrence(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r,
                      const b200_hybrid_pass& p, cudaStream_t st);
// fixed_count > 0: rows 0 .. fixed_count-1 of the pending buffer; else count / rows as in b200_hybrid_commit.
int launch_commit(const b200_hybrid_model& m, void* cache, int cache_rows, int fixed_count, const int* count, const int* rows,
                  int tree_rows, const int* prefix, int states, int compact, cudaStream_t st);
size_t attention_part_bytes(const b200_hybrid_model& m, int rows);

inline int act_bytes(int act_type) { return act_type == B200_ACT_F32 ? 4 : 2; }
// The pending slot a committed chain row keeps its convolution input in (negative: none).
__host__ __device__ inline int chain_slot(int row, int M) {
    return M <= B200_HYBRID_PENDING ? row : row - (M - B200_HYBRID_PENDING);
}

}  // namespace hybrid
}  // namespace b200
