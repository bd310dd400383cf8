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

__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }

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
    kOpResidual = 4,    // dst += mult * (acc + b) (+ add), b optional
    kOpSoftcap = 5,     // cap * tanh(acc / cap), cap <= 0: acc
    kOpBias = 6,        // acc + b
    kOpDecay = 7        // exp(-rate softplus(acc + b)) - 1: what is lost keeps its precision where almost nothing is
};

// log(1 + e^z) = max(z, 0) + log(1 + x), x = e^-|z| in (0, 1]; log(1 + x) = 2 artanh(s), s = x / (2 + x) <= 1/3, by its odd
// series up to s^15.
__device__ __forceinline__ float softplus_f(float z) {
    const float x = expf(-fabsf(z)), s = __fdividef(x, 2.0f + x), q = s * s;
    float t = 1.0f / 15.0f;
    t = fmaf(t, q, 1.0f / 13.0f);
    t = fmaf(t, q, 1.0f / 11.0f);
    t = fmaf(t, q, 1.0f / 9.0f);
    t = fmaf(t, q, 1.0f / 7.0f);
    t = fmaf(t, q, 1.0f / 5.0f);
    t = fmaf(t, q, 1.0f / 3.0f);
    return fmaxf(z, 0.f) + fmaf(2.0f * s * q, t, 2.0f * s);
}

// Two-branch activations: a product whose columns alternate gate, up, or the same as a kernel of its own.
struct Gating {
    int kind;               // 0: none, B200_FF_GATED: gelu_tanh(g) u, B200_FF_EXPERTS: clipped, swish_alpha(g) (u + shift)
    float limit, alpha, shift;
};
__device__ __forceinline__ float gated_f(const Gating& p, float g, float u) {
    if (p.kind == B200_FF_GATED) {
        const float t = tanhf(0.79788456080286536f * (g + 0.044715f * g * g * g));
        return 0.5f * g * (1.0f + t) * u;
    }
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit);
    return g * sigmoid_f(p.alpha * g) * (u + p.shift);
}
inline Gating gating_of(const b200_hybrid_layer& l) { return Gating{l.ff_kind, l.act[0], l.act[1], l.act[2]}; }

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
    const float* p0;        // per column: bias (kOpForget, kOpDecay, kOpBias, kOpResidual: may be null there)
    const float* p1;        // lower bound (kOpForget), rate (kOpDecay)
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
    // gate.kind != 0: one segment of the activation type with half the product's columns; column 2c is the gate of channel c,
    // 2c + 1 its other branch
    Gating gate;
    const float* gate_bias; // per column of the product (or null)
    const float* row_scale; // per row, on the accumulator (or null)
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
    float bias;             // kOpResidual
    char* base;             // null: not a column of the product
    long long stride;       // bytes between rows
    float p0, p1;
    __half* half_base;
    const char* add_base;

    __device__ __forceinline__ void init(const Epi& e, int n) {
        op = kOpNone; f32 = 1; bias = 0.f; base = nullptr; stride = 0; p0 = p1 = 0.f; half_base = nullptr; add_base = nullptr;
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
                if (s.op == kOpForget || s.op == kOpDecay) { p0 = s.p0[c]; p1 = s.p1[c]; }
                if (s.op == kOpBias) p0 = s.p0[c];
                if (s.op == kOpSoftcap) {
                    p0 = e.cap;
                    if (e.half_copy != nullptr) half_base = e.half_copy + off;
                }
                if (s.op == kOpResidual) {
                    p0 = e.mult;
                    if (s.p0 != nullptr) bias = s.p0[c];
                    if (e.add != nullptr) add_base = reinterpret_cast<const char*>(e.add + off);
                }
            }
        }
    }
    __device__ __forceinline__ float finish(float acc, float residual) const {
        if (op == kOpSilu) return acc * sigmoid_f(acc);
        if (op == kOpSigmoid) return sigmoid_f(acc);
        if (op == kOpForget) return (1.0f - p1) * sigmoid_f(-(acc + p0));
        if (op == kOpResidual) return residual + p0 * (acc + bias);
        if (op == kOpBias) return acc + p0;
        if (op == kOpDecay) return expm1f(-p1 * softplus_f(acc + p0));
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
            if (i >= n) break;                       // (n is the same for the whole warp)
            float v = __uint_as_float(acc[i]);
            if (OP == kOpSilu) v = v * sigmoid_f(v);
            else if (OP == kOpSigmoid) v = sigmoid_f(v);
            else if (OP == kOpForget) v = (1.0f - p1) * sigmoid_f(-(v + p0));
            else if (OP == kOpResidual) v = r[i] + p0 * (v + bias);
            else if (OP == kOpBias) v = v + p0;
            else if (OP == kOpDecay) v = expm1f(-p1 * softplus_f(v + p0));
            else if (OP == kOpSoftcap) v = p0 > 0.f ? p0 * tanhf(v / p0) : v;
            if (F32) *reinterpret_cast<float*>(p + i * stride) = v;
            else *reinterpret_cast<T*>(p + i * stride) = from_f32<T>(v);
            if (OP == kOpSoftcap && half_base != nullptr) half_base[(long long)(m0 + i) * (stride >> 2)] = __float2half_rn(v);
        }
    }
    // Rows m0 .. m0 + n - 1, n clipped to N: one branch on the operation, straight code for the rows.
    template <int N>
    __device__ __forceinline__ void store_rows(int m0, int n, const uint32_t (&acc)[N]) const {
        if (base == nullptr) return;
        switch (op) {
            case kOpNone: if (f32) rows_of<kOpNone, true>(m0, n, acc); else rows_of<kOpNone, false>(m0, n, acc); break;
            case kOpSilu: rows_of<kOpSilu, false>(m0, n, acc); break;
            case kOpSigmoid: if (f32) rows_of<kOpSigmoid, true>(m0, n, acc); else rows_of<kOpSigmoid, false>(m0, n, acc); break;
            case kOpBias: rows_of<kOpBias, true>(m0, n, acc); break;
            case kOpDecay: rows_of<kOpDecay, true>(m0, n, acc); break;
            case kOpForget: rows_of<kOpForget, true>(m0, n, acc); break;
            case kOpResidual: rows_of<kOpResidual, true>(m0, n, acc); break;
            default: rows_of<kOpSoftcap, true>(m0, n, acc); break;
        }
    }
};

// Column n of a product whose columns alternate gate and up, rows m0 .. m0 + count - 1 (count clipped to N), called by whole
// warps with neighbouring lanes on neighbouring columns: each lane of a pair finishes every other row of their channel.
template <typename T, int N>
__device__ __forceinline__ void store_gated_rows(const Epi& e, int n, bool valid, int m0, int count, const uint32_t (&acc)[N]) {
    const bool odd = n & 1;
    const float b = valid && e.gate_bias != nullptr ? e.gate_bias[n] : 0.f;
    T* dst = static_cast<T*>(e.seg[0].dst) + (n >> 1);
#pragma unroll
    for (int i = 0; i < N; i += 2) {
        if (i >= count) break;                       // (the same for the whole warp)
        float a0 = __uint_as_float(acc[i]), a1 = __uint_as_float(acc[i + 1]);
        if (e.row_scale != nullptr) {
            a0 *= e.row_scale[m0 + i];
            a1 *= i + 1 < count ? e.row_scale[m0 + i + 1] : 0.f;
        }
        a0 += b;
        a1 += b;
        const float got = __shfl_xor_sync(0xffffffffu, odd ? a0 : a1, 1);
        const float y = gated_f(e.gate, odd ? got : a0, odd ? a1 : got);
        const int r = i + (odd ? 1 : 0);
        if (valid && r < count) dst[(long long)(m0 + r) * e.seg[0].row_stride] = from_f32<T>(y);
    }
}

// ---------------------------------------------------------------- launches
// x: activations [x_rows][x_pitch] of type act_type (x_pitch 0: pitch times groups); x_rows bounds what may be read.
int launch_linear(int act_type, const b200_linear& lin, const void* x, int x_pitch, int x_rows, const Epi& epi, int* error, cudaStream_t st);
// Products of an expert stack (bf16): rows offsets[e] .. offsets[e + 1] - 1 of x through group e of lin; `rows` in all.
int launch_linear_experts(const b200_linear& lin, const void* x, int x_rows, int rows, const int* offsets, const Epi& epi, int* error, cudaStream_t st);

int launch_embed(const b200_hybrid_model& m, const b200_hybrid_pass& p, cudaStream_t st);
int launch_norm_conv(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r,
                     const b200_hybrid_pass& p, cudaStream_t st);
// x / rms(x) * w into the product-input buffer; with `gather` the rows named by out_rows / row_index.
int launch_norm(const b200_hybrid_model& m, const float* w, const b200_hybrid_pass& p, bool gather, int rows, cudaStream_t st);
int launch_polynorm(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st);
int launch_gated(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st);
// x += norm(y) * w (w null: x += residual_mult * y) with y the sum of `slots` rows of m.y: row m, or with `place` the rows
// place[m * slots ..]; the new stream also goes to the product input.  x_add: added to the stream too (or null).
int launch_join(const b200_hybrid_model& m, const float* w, int rows, int slots, const int* place, const float* x_add, cudaStream_t st);
int launch_add(float* x, const float* y, size_t n, cudaStream_t st);
int launch_attention(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r,
                     const b200_hybrid_pass& p, cudaStream_t st);
int launch_recurrence(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r,
                      const b200_hybrid_pass& p, cudaStream_t st);
int launch_delta(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p, cudaStream_t st);
// Advances the state and convolution inputs of a delta run over pending rows, count / rows as in b200_hybrid_commit.
int launch_delta_commit(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, void* cache, const int* count,
                        const int* rows, int tree_rows, cudaStream_t st);
// Does the pass read the latent of every head's keys and values written out (prompts), or queries brought into its space?
bool latent_expands(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_pass& p);
constexpr int kLatentColumns = 512;      // latent sizes of the bf16 kernel over the latent itself
int launch_latent_attention(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p, cudaStream_t st);
size_t latent_attention_parts(int rows, int heads);      // partial vectors it may need
int launch_latent_prep(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p, cudaStream_t st);
bool router_in_rows(int rows);           // do that few rows get their logits from launch_router_rows?
int launch_router_rows(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st);
// Chooses the experts of every row (router logits in m.zr), runs them and leaves their outputs in rows of m.y; *place: where
// each (row, choice) is (null: in order).
int launch_experts(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, const int** place, cudaStream_t st);
// head_norm of m.o32 (vdim columns per head), times `gate` where there is one, to m.ab.
int launch_head_norm(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, const void* gate, cudaStream_t st);
// fixed_count > 0: rows 0 .. fixed_count-1 of the pending buffer; else count / rows as in b200_hybrid_commit.
int launch_commit(const b200_hybrid_model& m, void* cache, int cache_rows, int fixed_count, const int* count, const int* rows,
                  int tree_rows, const int* prefix, int states, int compact, cudaStream_t st);
size_t attention_part_bytes(const b200_hybrid_model& m, int rows);

inline int delta_channels(const b200_hybrid_layer& l) { return 2 * l.kv_heads * l.dim + l.heads * l.vdim; }
inline int delta_pitch(const b200_hybrid_layer& l) { return round_up(delta_channels(l), 8); }
__host__ __device__ inline int latent_pitch(const b200_hybrid_layer& l) { return round_up(l.kv_rank, 16) + round_up(l.rot_dim, 16); }
inline int act_bytes(int act_type) { return act_type == B200_ACT_F32 ? 4 : 2; }
// The pending slot a committed chain row keeps its convolution input in (negative: none).
__host__ __device__ inline int chain_slot(int row, int M) {
    return M <= B200_HYBRID_PENDING ? row : row - (M - B200_HYBRID_PENDING);
}

}  // namespace hybrid
}  // namespace b200
