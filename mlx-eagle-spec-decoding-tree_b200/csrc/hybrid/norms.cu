// Element-wise and per-row steps of the hybrid decoders: embedding, RMS norm with the causal input convolution, RMS
// norm alone (feed-forward input, final norm with row gather), a sublayer's normed output joined to the stream, the
// polynomial and the gated activation, stream injection.  All
// statistics and the residual stream are fp32; outputs that feed a product have the activation type.
#include "hybrid.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kThreads = 256;
constexpr int kRowsPerCta = 8;       // chain rows of one CTA of the norm + convolution kernel
constexpr int kMaxTaps = B200_HYBRID_MAX_TAPS;

// V (1 or 4) neighbouring channels.
template <int V> struct Vec { float v[V]; };
template <int V> __device__ __forceinline__ Vec<V> ld(const float* p) {
    Vec<V> r;
    if (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        r.v[0] = t.x; r.v[V > 1 ? 1 : 0] = t.y; r.v[V > 1 ? 2 : 0] = t.z; r.v[V > 1 ? 3 : 0] = t.w;
        return r;
    }
    r.v[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ void st(float* p, const Vec<V>& r) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[V > 1 ? 1 : 0], r.v[V > 1 ? 2 : 0], r.v[V > 1 ? 3 : 0]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void st(bf16* p, const Vec<V>& r) {
    if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[V > 1 ? 1 : 0]), b = __floats2bfloat162_rn(r.v[V > 1 ? 2 : 0], r.v[V > 1 ? 3 : 0]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

struct EmbedParams {
    const int* tokens;
    const bf16* table;
    float* x;
    float* emb;                      // copy of the output, or null
    void* out;                       // product input [M][pitch], or null
    const int* pos;
    int* tail_pos;                   // tree: positions of the tail rows (null: chain)
    int width, vocab, pitch;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) embed_kernel(const EmbedParams p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int N = 4;                              // channels of a thread; all loads before the first store
    const int m = blockIdx.x, c0 = blockIdx.y * kThreads * N + threadIdx.x;
    const int tok = min(max(p.tokens[m], 0), p.vocab - 1);
    const bf16* src = p.table + (size_t)tok * p.width;
    bf16 v[N];
#pragma unroll
    for (int i = 0; i < N; i++) v[i] = c0 + i * kThreads < p.width ? src[c0 + i * kThreads] : __float2bfloat16_rn(0.f);
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int c = c0 + i * kThreads;
        if (c < p.width) {
            const float f = __bfloat162float(v[i]);
            p.x[(size_t)m * p.width + c] = f;
            if (p.emb != nullptr) p.emb[(size_t)m * p.width + c] = f;
            if (p.out != nullptr) static_cast<T*>(p.out)[(size_t)m * p.pitch + c] = from_f32<T>(f);
        }
    }
    if (p.tail_pos != nullptr && blockIdx.y == 0 && threadIdx.x == 0) p.tail_pos[m] = p.pos[m];
}

template <int V>
__device__ __forceinline__ float row_sumsq_warp(const float* row, int width, int lane) {
    float s[V] = {};
#pragma unroll 8
    for (int c = lane * V; c < width; c += 32 * V) {
        const Vec<V> t = ld<V>(row + c);
#pragma unroll
        for (int e = 0; e < V; e++) s[e] = fmaf(t.v[e], t.v[e], s[e]);
    }
    float r = 0.f;
#pragma unroll
    for (int e = 0; e < V; e++) r += s[e];
    return warp_sum(r);
}

struct NormConvParams {
    const float* x;
    const float* w;                  // norm weight
    const float* conv;               // [taps][width]
    const float* state;              // [taps - 1][width] committed inputs, oldest first
    float* pend;                     // [64][width] inputs of this pass's rows until they are committed
    void* out;                       // [M][pitch]
    const unsigned long long* mask;
    int M, width, pitch, write_off;
    float eps;
};

// h = x / rms(x) * w;  out = h + sum_j conv[j] * (input TAPS-1-j positions earlier on the row's path).
// Grid (rows, channel slices); every CTA computes the norms it needs from whole rows.
// Chain: kRowsPerCta consecutive rows per CTA, the inputs before them recomputed from x or taken from the state.
// Tree: one row per CTA; its predecessors are its ancestors (set bits of its mask), then the committed inputs.
template <typename T, int TAPS, int V, bool TREE>
__global__ void __launch_bounds__(kThreads) norm_conv_kernel(const NormConvParams p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int PREV = TAPS - 1;
    constexpr int ROWS = TREE ? 1 : kRowsPerCta;
    __shared__ float s_rstd[ROWS + PREV];
    __shared__ const float* s_src[kMaxTaps];      // tree: predecessor vectors, oldest first
    __shared__ int s_raw[kMaxTaps];               // ... row of this pass whose norm has to be applied (-1: vector as stored)
    const int W = p.width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r0 = blockIdx.x * ROWS, rows = min(ROWS, p.M - r0);
    const int self = p.write_off + r0;
    T* out = static_cast<T*>(p.out);
    if (TREE) {
        if (threadIdx.x == 0) {
            unsigned long long anc = p.mask[r0] & ((1ull << self) - 1ull);
            int have = 0;
            for (int j = PREV - 1; j >= 0; j--) {
                if (anc != 0ull) {
                    const int a = 63 - __clzll((long long)anc);
                    anc &= ~(1ull << a);
                    have++;
                    s_raw[j] = a >= p.write_off ? a - p.write_off : -1;
                    s_src[j] = a >= p.write_off ? p.x + (size_t)(a - p.write_off) * W : p.pend + (size_t)a * W;
                } else {
                    s_raw[j] = -1;
                    s_src[j] = p.state + (size_t)(j + have) * W;
                }
            }
        }
        __syncthreads();
    }
    for (int i = warp; i < rows + PREV; i += kThreads / 32) {
        const int row = TREE ? (i == PREV ? r0 : s_raw[i]) : r0 - PREV + i;
        if (row >= 0) {
            const float ss = row_sumsq_warp<V>(p.x + (size_t)row * W, W, lane);
            if (lane == 0) s_rstd[i] = rsqrtf(ss / (float)W + p.eps);
        }
    }
    __syncthreads();
    for (int c = (blockIdx.y * kThreads + threadIdx.x) * V; c < W; c += gridDim.y * kThreads * V) {
        const Vec<V> wc = ld<V>(p.w + c);
        Vec<V> hist[TAPS], cw[TAPS];                  // inputs, oldest first
#pragma unroll
        for (int k = 0; k < TAPS; k++) cw[k] = ld<V>(p.conv + (size_t)k * W + c);
#pragma unroll
        for (int k = 0; k < PREV; k++) {
            const int row = TREE ? s_raw[k] : r0 - PREV + k;
            const float* src = TREE ? s_src[k] : (row >= 0 ? p.x + (size_t)row * W : p.state + (size_t)(row + PREV) * W);
            hist[k] = ld<V>(src + c);
            if (row >= 0)
#pragma unroll
                for (int e = 0; e < V; e++) hist[k].v[e] *= s_rstd[k] * wc.v[e];
        }
#pragma unroll
        for (int r = 0; r < ROWS; r++) {
            if (r >= rows) break;
            const int m = r0 + r;
            Vec<V> h = ld<V>(p.x + (size_t)m * W + c), acc;
#pragma unroll
            for (int e = 0; e < V; e++) {
                h.v[e] *= s_rstd[PREV + r] * wc.v[e];
                acc.v[e] = fmaf(cw[PREV].v[e], h.v[e], h.v[e]);
            }
#pragma unroll
            for (int k = 0; k < PREV; k++)
#pragma unroll
                for (int e = 0; e < V; e++) acc.v[e] = fmaf(cw[k].v[e], hist[k].v[e], acc.v[e]);
            if (TREE) st<V>(p.pend + (size_t)self * W + c, h);
            else if (m >= p.M - PREV) st<V>(p.pend + (size_t)chain_slot(m, p.M) * W + c, h);
            st<V>(out + (size_t)m * p.pitch + c, acc);
#pragma unroll
            for (int k = 0; k + 1 < PREV; k++) hist[k] = hist[k + 1];
            if (PREV > 0) hist[PREV > 0 ? PREV - 1 : 0] = h;
        }
    }
}

template <typename T, int V>
__global__ void __launch_bounds__(1024) norm_kernel(const float* x, const float* w, T* out,
                                                    const int* rows, const int* row_index, int gather, int width,
                                                    int pitch, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[33];
    int src = blockIdx.x;
    if (gather) src = rows != nullptr ? rows[src] : (row_index != nullptr ? row_index[0] + src : src);
    const float* xr = x + (size_t)src * width;
    float ss = 0.f;
#pragma unroll 4
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        const Vec<V> t = ld<V>(xr + c);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(t.v[e], t.v[e], ss);
    }
    ss = block_sum(ss, red);
    const float rstd = rsqrtf(ss / (float)width + eps);
    T* o = out + (size_t)blockIdx.x * pitch;
#pragma unroll 4
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        Vec<V> t = ld<V>(xr + c);
        const Vec<V> g = ld<V>(w + c);
#pragma unroll
        for (int e = 0; e < V; e++) t.v[e] *= rstd * g.v[e];
        st<V>(o + c, t);
    }
}

// a N(z) + b N(z^2) + c N(z^3) + e, N: over the root mean square of the row.  16 bytes per thread and step; the padding of
// a row (zeros or finite leftovers that meet zero weights) is read but not counted.
template <typename T>
__global__ void __launch_bounds__(1024) polynorm_kernel(const T* z, T* out, int width, int pitch, float a, float b,
                                                        float c, float e, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int VE = 16 / (int)sizeof(T);
    __shared__ float red[99];
    const T* zr = z + (size_t)blockIdx.x * pitch;
    float3 s = make_float3(0.f, 0.f, 0.f);
#pragma unroll 2
    for (int i = threadIdx.x * VE; i < width; i += blockDim.x * VE) {
        const uint4 raw = *reinterpret_cast<const uint4*>(zr + i);
        const T* t = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int k = 0; k < VE; k++) {
            const float v = i + k < width ? to_f32<T>(t[k]) : 0.f, q = v * v, u = q * v;
            s.x += q;
            s.y = fmaf(q, q, s.y);
            s.z = fmaf(u, u, s.z);
        }
    }
    s = block_sum3(s, red);
    const float n = (float)width;
    const float ka = a * rsqrtf(s.x / n + eps), kb = b * rsqrtf(s.y / n + eps), kc = c * rsqrtf(s.z / n + eps);
    T* o = out + (size_t)blockIdx.x * pitch;
#pragma unroll 2
    for (int i = threadIdx.x * VE; i < width; i += blockDim.x * VE) {
        uint4 raw = *reinterpret_cast<const uint4*>(zr + i);
        T* t = reinterpret_cast<T*>(&raw);
#pragma unroll
        for (int k = 0; k < VE; k++) {
            const float v = to_f32<T>(t[k]);
            t[k] = from_f32<T>(i + k < width ? fmaf(v, fmaf(v, fmaf(v, kc, kb), ka), e) : 0.f);
        }
        *reinterpret_cast<uint4*>(o + i) = raw;
    }
}

// x += y / rms(y) * w (w null: x += mult * y), y the sum of `slots` rows; the new stream also goes to the product input.
struct JoinParams {
    const float* y;
    const float* w;
    const int* place;                // rows of y of every (row, slot), null: row * slots + slot
    const float* add;
    float* x;
    void* out;
    int slots, width, pitch;
    float eps, mult;
};

template <typename T, int V>
__global__ void __launch_bounds__(1024) join_kernel(const JoinParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float s_y[];      // the row's y
    __shared__ float red[33];
    __shared__ int s_row[B200_HYBRID_MAX_TOP];
    const int m = blockIdx.x;
    if (threadIdx.x < p.slots) s_row[threadIdx.x] = p.place != nullptr ? p.place[m * p.slots + threadIdx.x] : m * p.slots + threadIdx.x;
    __syncthreads();
    float ss = 0.f;
#pragma unroll 2
    for (int c = threadIdx.x * V; c < p.width; c += blockDim.x * V) {
        Vec<V> t = ld<V>(p.y + (size_t)s_row[0] * p.width + c);
        for (int s = 1; s < p.slots; s++) {
            const Vec<V> u = ld<V>(p.y + (size_t)s_row[s] * p.width + c);
#pragma unroll
            for (int e = 0; e < V; e++) t.v[e] += u.v[e];
        }
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(t.v[e], t.v[e], ss);
        st<V>(s_y + c, t);
    }
    float f = p.mult;
    if (p.w != nullptr) f = rsqrtf(block_sum(ss, red) / (float)p.width + p.eps);
    float* x = p.x + (size_t)m * p.width;
    T* o = static_cast<T*>(p.out) + (size_t)m * p.pitch;
#pragma unroll 2
    for (int c = threadIdx.x * V; c < p.width; c += blockDim.x * V) {      // (each thread its own channels)
        const Vec<V> t = ld<V>(s_y + c);
        Vec<V> g, r = ld<V>(x + c);
        if (p.w != nullptr) g = ld<V>(p.w + c);
#pragma unroll
        for (int e = 0; e < V; e++) r.v[e] += p.w != nullptr ? t.v[e] * f * g.v[e] : t.v[e] * f;
        if (p.add != nullptr) {
            const Vec<V> a = ld<V>(p.add + (size_t)m * p.width + c);
#pragma unroll
            for (int e = 0; e < V; e++) r.v[e] += a.v[e];
        }
        st<V>(x + c, r);
        st<V>(o + c, r);
    }
}

// Columns alternating gate and up -> the activation (fp32 products, whose epilogue does not pair columns).
__global__ void __launch_bounds__(kThreads) gated_kernel(const float* z, int z_pitch, float* out, int pitch, int ff, const float* bias, Gating gate) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.x * kThreads + threadIdx.x, m = blockIdx.y;
    if (c >= ff) return;
    float g = z[(size_t)m * z_pitch + 2 * c], u = z[(size_t)m * z_pitch + 2 * c + 1];
    if (bias != nullptr) { g += bias[2 * c]; u += bias[2 * c + 1]; }
    out[(size_t)m * pitch + c] = gated_f(gate, g, u);
}

__global__ void add_kernel(float* x, const float* y, size_t n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += y[i];
}

}  // namespace

int launch_embed(const b200_hybrid_model& m, const b200_hybrid_pass& p, cudaStream_t st) {
    EmbedParams q{};
    q.tokens = p.tokens; q.table = static_cast<const bf16*>(m.embed); q.x = m.x; q.emb = m.injects ? m.emb : nullptr;
    q.out = m.norm_out ? m.hb : nullptr; q.pos = p.pos; q.tail_pos = p.tree ? p.tail_pos + p.write_off : nullptr;
    q.width = m.width; q.vocab = m.vocab; q.pitch = round_up(m.width, 64);
    const dim3 grid(p.M, (m.width + 4 * kThreads - 1) / (4 * kThreads));
    if (m.act_type == B200_ACT_F32) launch_kernel(embed_kernel<float>, grid, dim3(kThreads), 0, st, q);
    else launch_kernel(embed_kernel<bf16>, grid, dim3(kThreads), 0, st, q);
    return check_launch();
}

namespace {

template <typename T, int TAPS, int V>
void launch_norm_conv_v(const NormConvParams& q, int tree, cudaStream_t st) {
    const int all = (q.width + kThreads * V - 1) / (kThreads * V);
    const int slices = q.M <= 32 ? all : 1;          // many rows: a CTA takes whole rows, or it would read them once per slice
    if (tree) launch_kernel(norm_conv_kernel<T, TAPS, V, true>, dim3(q.M, slices), dim3(kThreads), 0, st, q);
    else launch_kernel(norm_conv_kernel<T, TAPS, V, false>, dim3((q.M + kRowsPerCta - 1) / kRowsPerCta, slices), dim3(kThreads), 0, st, q);
}

template <typename T, int TAPS>
int launch_norm_conv_t(const NormConvParams& q, int taps, int tree, cudaStream_t st) {
    if constexpr (TAPS > kMaxTaps) {
        return B200_ELIMIT;
    } else {
        if (taps != TAPS) return launch_norm_conv_t<T, TAPS + 1>(q, taps, tree, st);
        if (q.width % 4 == 0) launch_norm_conv_v<T, TAPS, 4>(q, tree, st);
        else launch_norm_conv_v<T, TAPS, 1>(q, tree, st);
        return check_launch();
    }
}

// Threads of a CTA that works on one row: more when there are few rows.
int row_threads(int rows, int units) {
    const int most = rows < 148 ? 1024 : 256;
    const int t = round_up(units, 32);
    return t < 128 ? 128 : (t < most ? t : most);    // (block_sum3 needs three warps)
}

template <typename T>
int launch_norm_t(const b200_hybrid_model& m, const float* w, const b200_hybrid_pass& p, int gather, int rows, cudaStream_t st) {
    const int pitch = round_up(m.width, 64);
    const float* x = m.x;
    T* out = static_cast<T*>(m.hb);
    if (m.width % 4 == 0)
        launch_kernel(norm_kernel<T, 4>, dim3(rows), dim3(row_threads(rows, m.width / 4)), 0, st, x, w, out, p.out_rows, p.row_index, gather,
                      m.width, pitch, m.eps);
    else
        launch_kernel(norm_kernel<T, 1>, dim3(rows), dim3(row_threads(rows, m.width)), 0, st, x, w, out, p.out_rows, p.row_index, gather, m.width,
                      pitch, m.eps);
    return check_launch();
}

template <typename T>
int launch_polynorm_t(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st) {
    const int VE = 16 / (int)sizeof(T);
    launch_kernel(polynorm_kernel<T>, dim3(rows), dim3(row_threads(rows, (l.ff + VE - 1) / VE)), 0, st, static_cast<const T*>(m.zb),
                  static_cast<T*>(m.zab), l.ff, round_up(l.ff, 64), l.act[0], l.act[1], l.act[2], l.act[3], m.eps);
    return check_launch();
}

template <typename T>
int launch_join_t(const JoinParams& p, int rows, cudaStream_t st) {
    const size_t smem = (size_t)p.width * 4;
    if (smem > 160 * 1024) return B200_ELIMIT;
    auto k = p.width % 4 == 0 ? join_kernel<T, 4> : join_kernel<T, 1>;
    if (smem > 40 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return check_launch();
    launch_kernel(k, dim3(rows), dim3(row_threads(rows, p.width % 4 == 0 ? p.width / 4 : p.width)), smem, st, p);
    return check_launch();
}

}  // namespace

int launch_norm_conv(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p,
                     cudaStream_t st) {
    NormConvParams q{};
    q.x = m.x; q.w = l.norm1; q.conv = l.conv;
    q.state = reinterpret_cast<const float*>(static_cast<const char*>(p.cache) + r.conv_off);
    q.pend = reinterpret_cast<float*>(static_cast<char*>(m.pending) + r.pend_h);
    q.out = m.hb; q.mask = p.mask;
    q.M = p.M; q.width = m.width; q.pitch = round_up(m.width, 64); q.write_off = p.write_off;
    q.eps = m.eps;
    return m.act_type == B200_ACT_F32 ? launch_norm_conv_t<float, 1>(q, l.taps, p.tree, st) : launch_norm_conv_t<bf16, 1>(q, l.taps, p.tree, st);
}

int launch_norm(const b200_hybrid_model& m, const float* w, const b200_hybrid_pass& p, bool gather, int rows, cudaStream_t st) {
    return m.act_type == B200_ACT_F32 ? launch_norm_t<float>(m, w, p, gather ? 1 : 0, rows, st) : launch_norm_t<bf16>(m, w, p, gather ? 1 : 0, rows, st);
}

int launch_polynorm(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st) {
    return m.act_type == B200_ACT_F32 ? launch_polynorm_t<float>(m, l, rows, st) : launch_polynorm_t<bf16>(m, l, rows, st);
}

int launch_join(const b200_hybrid_model& m, const float* w, int rows, int slots, const int* place, const float* x_add, cudaStream_t st) {
    if (slots < 1 || slots > B200_HYBRID_MAX_TOP) return B200_ELIMIT;
    JoinParams p{};
    p.y = m.y; p.w = w; p.place = place; p.add = x_add; p.x = m.x; p.out = m.hb; p.slots = slots; p.width = m.width;
    p.pitch = round_up(m.width, 64); p.eps = m.eps; p.mult = m.residual_mult;
    return m.act_type == B200_ACT_F32 ? launch_join_t<float>(p, rows, st) : launch_join_t<bf16>(p, rows, st);
}

int launch_gated(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st) {
    if (m.act_type != B200_ACT_F32) return B200_EINVAL;
    launch_kernel(gated_kernel, dim3((l.ff + kThreads - 1) / kThreads, rows), dim3(kThreads), 0, st, static_cast<const float*>(m.zb),
                  round_up(2 * l.ff, 64), static_cast<float*>(m.zab), round_up(l.ff, 64), l.ff, l.up_bias, gating_of(l));
    return check_launch();
}

int launch_add(float* x, const float* y, size_t n, cudaStream_t st) {
    launch_kernel(add_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, x, y, n);
    return check_launch();
}

}  // namespace hybrid
}  // namespace b200
