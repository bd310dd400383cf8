// Mixture of experts of the hybrid decoders: each row goes through the `top` experts with the largest sigmoid scores of its
// router logits (fp32), the score multiplies the expert's input.
//
//   router_rows                         few rows: logits, a CTA per (expert, row).
//   expert_up_rows / expert_down_rows   few (row, choice) pairs, or fp32: a warp per channel of a pair; every CTA chooses the
//                                       row's experts itself from the logits (the choice is a few warp reductions).
//   route, sort, gather                 many pairs: choices of all rows, their places in expert order (counting sort, a warp
//                                       per expert), rows copied to their places; the products are the tcgen05 kernel's
//                                       with token tiles per expert.
#include "hybrid.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kThreads = 256;
constexpr int kPerLane = B200_HYBRID_MAX_EXPERTS / 32;

// The `top` largest scores of a row, in falling order (equal scores: the lower expert first); called by a whole warp.
// Lane s gets choice s (expert -1 where there is none).
struct Choice {
    int expert;
    float score;
};
__device__ __forceinline__ Choice choose(const float* z, int experts, int top, int lane) {
    float s[kPerLane];
#pragma unroll
    for (int i = 0; i < kPerLane; i++) s[i] = lane + 32 * i < experts ? sigmoid_f(z[lane + 32 * i]) : -1.f;
    Choice mine{-1, 0.f};
    for (int c = 0; c < top; c++) {
        float best = -1.f;
        int at = 1 << 30;
#pragma unroll
        for (int i = 0; i < kPerLane; i++)
            if (s[i] > best) { best = s[i]; at = lane + 32 * i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float b = __shfl_xor_sync(0xffffffffu, best, o);
            const int a = __shfl_xor_sync(0xffffffffu, at, o);
            if (b > best || (b == best && a < at)) { best = b; at = a; }
        }
        if (lane == c && at < experts) mine = Choice{at, best};
#pragma unroll
        for (int i = 0; i < kPerLane; i++)
            if (lane + 32 * i == at) s[i] = -1.f;
    }
    return mine;
}

// 16 bytes of bf16 weights times the activations beside them.
__device__ __forceinline__ float dot8(const uint4& w, const bf16* x, float acc) {
    const uint4 xr = *reinterpret_cast<const uint4*>(x);
    const uint32_t a[4] = {w.x, w.y, w.z, w.w}, b[4] = {xr.x, xr.y, xr.z, xr.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        acc = fmaf(__uint_as_float(a[i] << 16), __uint_as_float(b[i] << 16), acc);
        acc = fmaf(__uint_as_float(a[i] & 0xffff0000u), __uint_as_float(b[i] & 0xffff0000u), acc);
    }
    return acc;
}
__device__ __forceinline__ float dot8(const uint4& w, const float* x, float acc) {
    const float4 x0 = *reinterpret_cast<const float4*>(x), x1 = *reinterpret_cast<const float4*>(x + 4);
    const uint32_t a[4] = {w.x, w.y, w.z, w.w};
    const float b[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        acc = fmaf(__uint_as_float(a[i] << 16), b[2 * i], acc);
        acc = fmaf(__uint_as_float(a[i] & 0xffff0000u), b[2 * i + 1], acc);
    }
    return acc;
}

// Router logits of few rows (many: the matrix product kernels).
template <typename T>
__global__ void __launch_bounds__(128) router_rows_kernel(const bf16* w, const T* x, float* z, int experts, int pitch) {
    pdl_launch_dependents();
    const int e = blockIdx.x, m = blockIdx.y;
    __shared__ float red[33];
    const bf16* wr = w + (size_t)e * pitch;
    pdl_wait();
    float a = 0.f;
#pragma unroll 4
    for (int k = threadIdx.x * 8; k < pitch; k += 128 * 8) a = dot8(ldg_nc_v4(wr + k), x + (size_t)m * pitch + k, a);
    a = block_sum(a, red);
    if (threadIdx.x == 0) z[(size_t)m * experts + e] = a;
}

struct RowsParams {
    const float* z;               // router logits [M][experts]
    const bf16* w;                // stack [experts][stride rows][pitch]
    const void* x;                // up: [M][pitch], down: [M * top][pitch]
    void* out;                    // up: activations [M * top][out_pitch], down: fp32 [M * top][n]
    int experts, top, n, stride, pitch, out_pitch;
    Gating gate;
};

// CTA = (8 warps' channels, pair); a warp computes a channel's gate and up rows.
template <typename T>
__global__ void __launch_bounds__(kThreads) expert_up_rows_kernel(const RowsParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int pair = blockIdx.y, m = pair / p.top, slot = pair - m * p.top, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __shared__ int s_e;
    __shared__ float s_w;
    if (warp == 0) {
        const Choice c = choose(p.z + (size_t)m * p.experts, p.experts, p.top, lane);
        if (lane == slot) { s_e = c.expert; s_w = c.score; }
    }
    __syncthreads();
    const int c = blockIdx.x * (kThreads / 32) + warp;
    if (c >= p.n) return;
    const bf16* wg = p.w + ((size_t)max(s_e, 0) * p.stride + 2 * c) * p.pitch;
    const T* x = static_cast<const T*>(p.x) + (size_t)m * p.pitch;
    float g = 0.f, u = 0.f;
#pragma unroll 4
    for (int k = lane * 8; k < p.pitch; k += 256) {
        const uint4 a = ldg_nc_v4(wg + k), b = ldg_nc_v4(wg + p.pitch + k);
        g = dot8(a, x + k, g);
        u = dot8(b, x + k, u);
    }
    g = warp_sum(g) * s_w;
    u = warp_sum(u) * s_w;
    if (lane == 0) static_cast<T*>(p.out)[(size_t)pair * p.out_pitch + c] = from_f32<T>(gated_f(p.gate, g, u));
}

// CTA = (16 output channels, pair), two per warp.
template <typename T>
__global__ void __launch_bounds__(kThreads) expert_down_rows_kernel(const RowsParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int pair = blockIdx.y, m = pair / p.top, slot = pair - m * p.top, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __shared__ int s_e;
    if (warp == 0) {
        const Choice c = choose(p.z + (size_t)m * p.experts, p.experts, p.top, lane);
        if (lane == slot) s_e = c.expert;
    }
    __syncthreads();
    const int c = (blockIdx.x * (kThreads / 32) + warp) * 2;
    if (c >= p.n) return;
    const bf16* w = p.w + ((size_t)max(s_e, 0) * p.stride + c) * p.pitch;      // (the stack has rows past n)
    const T* x = static_cast<const T*>(p.x) + (size_t)pair * p.pitch;
    float a0 = 0.f, a1 = 0.f;
#pragma unroll 4
    for (int k = lane * 8; k < p.pitch; k += 256) {
        const uint4 a = ldg_nc_v4(w + k), b = ldg_nc_v4(w + p.pitch + k);
        a0 = dot8(a, x + k, a0);
        a1 = dot8(b, x + k, a1);
    }
    a0 = warp_sum(a0);
    a1 = warp_sum(a1);
    float* o = static_cast<float*>(p.out) + (size_t)pair * p.out_pitch + c;
    if (lane == 0) {
        o[0] = a0;
        if (c + 1 < p.n) o[1] = a1;
    }
}

// Parts of the route buffer.
struct Route {
    int* expert;                  // [rows * top]
    int* place;                   // [rows * top]
    float* score;                 // [rows * top], in expert order
    float* raw;                   // [rows * top], in row order
    int* offsets;                 // [experts + 1]
};
Route route_of(int* base, int max_rows, int top) {
    Route r;
    const size_t n = (size_t)max_rows * top;
    r.expert = base;
    r.place = base + n;
    r.score = reinterpret_cast<float*>(base + 2 * n);
    r.raw = reinterpret_cast<float*>(base + 3 * n);
    r.offsets = base + 4 * n;
    return r;
}

__global__ void __launch_bounds__(kThreads) route_kernel(const float* z, Route r, int M, int experts, int top) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (m >= M) return;
    const Choice c = choose(z + (size_t)m * experts, experts, top, lane);
    if (lane < top) {
        r.expert[m * top + lane] = max(c.expert, 0);
        r.raw[m * top + lane] = c.score;
    }
}

// One CTA: the pairs' places in expert order, in row order within an expert.  Each warp ranks a run of pairs by itself, then
// the warps' counts of an expert are added in order.
__global__ void __launch_bounds__(1024) sort_kernel(Route r, int pairs, int experts) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ int s_count[];                     // [32][experts], then (expert, rank) of every pair
    __shared__ int s_first[B200_HYBRID_MAX_EXPERTS + 1];
    unsigned short* s_e = reinterpret_cast<unsigned short*>(s_count + 32 * experts);
    unsigned short* s_rank = s_e + pairs;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int run = ((pairs + 31) / 32 + 31) / 32 * 32, i0 = warp * run, i1 = min(pairs, i0 + run);
    for (int i = tid; i < 32 * experts; i += 1024) s_count[i] = 0;
    for (int i = tid; i < pairs; i += 1024) s_e[i] = (unsigned short)r.expert[i];
    __syncthreads();
    int* mine = s_count + warp * experts;
    for (int i = i0 + lane; i - lane < i1; i += 32) {
        const int e = i < i1 ? s_e[i] : 0xffff;
        const unsigned peers = __match_any_sync(0xffffffffu, e);
        const int before = e != 0xffff ? mine[e] : 0;
        __syncwarp();
        if (e != 0xffff) {
            s_rank[i] = (unsigned short)(before + __popc(peers & ((1u << lane) - 1u)));
            if (lane == __ffs(peers) - 1) mine[e] = before + __popc(peers);
        }
        __syncwarp();
    }
    __syncthreads();
    for (int e = tid; e < experts; e += 1024) {
        int n = 0;
        for (int w = 0; w < 32; w++) {
            const int c = s_count[w * experts + e];
            s_count[w * experts + e] = n;
            n += c;
        }
        s_first[e + 1] = n;
    }
    if (tid == 0) s_first[0] = 0;
    __syncthreads();
    if (warp == 0) {
        int before = 0;
        for (int e0 = 1; e0 <= experts; e0 += 32) {
            const int e = e0 + lane;
            int n = e <= experts ? s_first[e] : 0;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int u = __shfl_up_sync(0xffffffffu, n, o);
                if (lane >= o) n += u;
            }
            if (e <= experts) s_first[e] = before + n;
            before += __shfl_sync(0xffffffffu, n, 31);
        }
    }
    __syncthreads();
    for (int e = tid; e <= experts; e += 1024) r.offsets[e] = s_first[e];
    for (int i = tid; i < pairs; i += 1024) {
        const int e = s_e[i], place = s_first[e] + s_count[i / run * experts + e] + s_rank[i];
        r.place[i] = place;
        r.score[place] = r.raw[i];
    }
}

__global__ void __launch_bounds__(kThreads) gather_kernel(const bf16* x, bf16* xg, const int* place, int top, int pitch) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x;
    for (int c = threadIdx.x * 8; c < pitch; c += kThreads * 8) {
        const uint4 v = *reinterpret_cast<const uint4*>(x + (size_t)m * pitch + c);
        for (int s = 0; s < top; s++) *reinterpret_cast<uint4*>(xg + (size_t)place[m * top + s] * pitch + c) = v;
    }
}

template <typename T>
int experts_rows(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st) {
    RowsParams p{};
    p.z = m.zr; p.experts = l.experts; p.top = l.top; p.gate = gating_of(l);
    p.w = static_cast<const bf16*>(l.up.w); p.x = m.hb; p.out = m.zab; p.n = l.ff; p.stride = round_up(l.up.n, 128); p.pitch = l.up.pitch;
    p.out_pitch = round_up(l.ff, 64);
    launch_kernel(expert_up_rows_kernel<T>, dim3((l.ff + 7) / 8, rows * l.top), dim3(kThreads), 0, st, p);
    p.w = static_cast<const bf16*>(l.down.w); p.x = m.zab; p.out = m.y; p.n = m.width; p.stride = round_up(m.width, 128); p.pitch = l.down.pitch;
    p.out_pitch = m.width;
    launch_kernel(expert_down_rows_kernel<T>, dim3((m.width + 15) / 16, rows * l.top), dim3(kThreads), 0, st, p);
    return check_launch();
}

constexpr int kFewPairs = 16, kFewRows = 16;

}  // namespace

bool router_in_rows(int rows) { return rows <= kFewRows; }

int launch_router_rows(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st) {
    const bf16* w = static_cast<const bf16*>(l.router.w);
    const dim3 grid(l.experts, rows);
    if (m.act_type == B200_ACT_F32) launch_kernel(router_rows_kernel<float>, grid, dim3(128), 0, st, w, static_cast<const float*>(m.hb), m.zr, l.experts, l.router.pitch);
    else launch_kernel(router_rows_kernel<bf16>, grid, dim3(128), 0, st, w, static_cast<const bf16*>(m.hb), m.zr, l.experts, l.router.pitch);
    return check_launch();
}

int launch_experts(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, const int** place, cudaStream_t st) {
    *place = nullptr;
    const int pairs = rows * l.top;
    if (m.act_type == B200_ACT_F32) return experts_rows<float>(m, l, rows, st);
    if (pairs <= kFewPairs) return experts_rows<bf16>(m, l, rows, st);
    const Route r = route_of(m.route, m.max_rows, l.top);
    launch_kernel(route_kernel, dim3((rows + 7) / 8), dim3(kThreads), 0, st, static_cast<const float*>(m.zr), r, rows, l.experts, l.top);
    const size_t smem = (size_t)pairs * 4 + (size_t)32 * l.experts * 4;
    if (smem > 200 * 1024) return B200_ELIMIT;
    if (smem > 40 * 1024 && cudaFuncSetAttribute(sort_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return check_launch();
    launch_kernel(sort_kernel, dim3(1), dim3(1024), smem, st, r, pairs, l.experts);
    launch_kernel(gather_kernel, dim3(rows), dim3(kThreads), 0, st, static_cast<const bf16*>(m.hb), static_cast<bf16*>(m.xg),
                  static_cast<const int*>(r.place), l.top, round_up(m.width, 64));
    if (check_launch() != B200_OK) return B200_ECUDA;
    const int x_rows = m.max_rows * l.top;
    Epi e{};
    e.nseg = 1;
    e.M = pairs;
    e.seg[0] = plain_seg(0, l.ff, kOpNone, 0, m.zab, round_up(l.ff, 64));
    e.gate = gating_of(l);
    e.row_scale = r.score;
    int rc = launch_linear_experts(l.up, m.xg, x_rows, pairs, r.offsets, e, m.error, st);
    if (rc != B200_OK) return rc;
    Epi d{};
    d.nseg = 1;
    d.M = pairs;
    d.seg[0] = plain_seg(0, m.width, kOpNone, 1, m.y, m.width);
    *place = r.place;
    return launch_linear_experts(l.down, m.zab, x_rows, pairs, r.offsets, d, m.error, st);
}

}  // namespace hybrid
}  // namespace b200

extern "C" size_t b200_hybrid_route_ints(int max_rows, int top, int experts) {
    return max_rows < 1 || top < 1 || experts < 1 ? 0 : (size_t)4 * max_rows * top + experts + 1;
}
