// Element-wise and per-row steps of the hybrid decoders: embedding, RMS norm with the causal input convolution, RMS
// norm alone (feed-forward input, final norm with row gather), the polynomial activation, stream injection.  All
// statistics and the residual stream are fp32; outputs that feed a product have the activation type.
#include "hybrid.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kThreads = 256;
constexpr int kRowsPerCta = 4;       // chain rows of one CTA of the norm + convolution kernel
constexpr int kMaxTaps = B200_HYBRID_MAX_TAPS;

__global__ void __launch_bounds__(kThreads) embed_kernel(const int* __restrict__ tokens, const bf16* __restrict__ table, int width, int vocab,
                                                         float* __restrict__ x, float* __restrict__ emb) {
    pdl_wait();
    pdl_launch_dependents();
    const int m = blockIdx.x;
    const int tok = min(max(tokens[m], 0), vocab - 1);
    for (int c = threadIdx.x; c < width; c += kThreads) {
        const float v = __bfloat162float(table[(size_t)tok * width + c]);
        x[(size_t)m * width + c] = v;
        if (emb != nullptr) emb[(size_t)m * width + c] = v;
    }
}

__device__ __forceinline__ float row_sumsq_warp(const float* __restrict__ row, int width, int lane) {
    float s = 0.f;
    for (int c = lane; c < width; c += 32) { const float v = row[c]; s = fmaf(v, v, s); }
    return warp_sum(s);
}

struct NormConvParams {
    const float* x;
    const float* w;                  // norm weight
    const float* conv;               // [taps][width]
    const float* state;              // [taps - 1][width] committed inputs, oldest first
    float* pend;                     // [64][width] inputs of this pass's rows until they are committed
    void* out;                       // [M][pitch]
    const unsigned long long* mask;
    const int* pos;
    int* tail_pos;
    int M, width, pitch, taps, write_off, tree;
    float eps;
};

// h = x / rms(x) * w;  out = h + sum_j conv[j] * (input taps-1-j positions earlier on the row's path).
// Chain: kRowsPerCta consecutive rows per CTA, the inputs before them recomputed from x or taken from the state.
// Tree: one row per CTA; its predecessors are its ancestors (set bits of its mask), then the committed inputs.
template <typename T>
__global__ void __launch_bounds__(kThreads) norm_conv_kernel(const NormConvParams p) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float s_rstd[kRowsPerCta + kMaxTaps];
    __shared__ const float* s_src[kMaxTaps];      // tree: predecessor vectors, oldest first
    __shared__ int s_raw[kMaxTaps];               // ... row of this pass whose norm has to be applied (-1: vector as stored)
    const int W = p.width, prev = p.taps - 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    T* out = static_cast<T*>(p.out);
    if (p.tree) {
        const int m = blockIdx.x;
        const int self = p.write_off + m;
        if (threadIdx.x == 0) {
            unsigned long long anc = p.mask[m] & ((1ull << self) - 1ull);
            int have = 0;
            for (int j = prev - 1; j >= 0; j--) {
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
            p.tail_pos[self] = p.pos[m];
        }
        __syncthreads();
        if (warp <= prev) {
            const int row = warp == prev ? m : s_raw[warp];
            if (row >= 0) {
                const float ss = row_sumsq_warp(p.x + (size_t)row * W, W, lane);
                if (lane == 0) s_rstd[warp] = rsqrtf(ss / (float)W + p.eps);
            }
        }
        __syncthreads();
        for (int c = threadIdx.x; c < W; c += kThreads) {
            const float wc = p.w[c];
            const float h = p.x[(size_t)m * W + c] * s_rstd[prev] * wc;
            float acc = fmaf(p.conv[(size_t)prev * W + c], h, h);
            for (int j = 0; j < prev; j++) {
                float v = s_src[j][c];
                if (s_raw[j] >= 0) v = v * s_rstd[j] * wc;
                acc = fmaf(p.conv[(size_t)j * W + c], v, acc);
            }
            p.pend[(size_t)self * W + c] = h;
            out[(size_t)m * p.pitch + c] = from_f32<T>(acc);
        }
        return;
    }
    const int r0 = blockIdx.x * kRowsPerCta, rows = min(kRowsPerCta, p.M - r0);
    for (int i = warp; i < rows + prev; i += kThreads / 32) {
        const int row = r0 - prev + i;
        if (row >= 0) {
            const float ss = row_sumsq_warp(p.x + (size_t)row * W, W, lane);
            if (lane == 0) s_rstd[i] = rsqrtf(ss / (float)W + p.eps);
        }
    }
    __syncthreads();
    for (int c = threadIdx.x; c < W; c += kThreads) {
        const float wc = p.w[c];
        float hist[kMaxTaps], cw[kMaxTaps];           // the last entries are the ones in use: hist[kMaxTaps-1] is the newest
#pragma unroll
        for (int j = 0; j < kMaxTaps; j++) {
            const int k = j - (kMaxTaps - p.taps);    // tap index
            cw[j] = k >= 0 ? p.conv[(size_t)k * W + c] : 0.f;
            float v = 0.f;
            if (k >= 0 && k < prev) {                 // input k - prev positions before row r0 is tap k of row r0 - 0
                const int row = r0 - prev + k;
                v = row >= 0 ? p.x[(size_t)row * W + c] * s_rstd[k] * wc : p.state[(size_t)(row + prev) * W + c];
            }
            hist[j] = v;
        }
        // shift so that the loop below can push the newest input
#pragma unroll
        for (int r = 0; r < kRowsPerCta; r++) {
            if (r >= rows) break;
            const int m = r0 + r;
            const float h = p.x[(size_t)m * W + c] * s_rstd[prev + r] * wc;
            hist[kMaxTaps - 1] = h;
            float acc = h;
#pragma unroll
            for (int j = 0; j < kMaxTaps; j++) acc = fmaf(cw[j], hist[j], acc);
            const int slot = chain_slot(m, p.M);
            if (slot >= 0 && m >= p.M - prev) p.pend[(size_t)slot * W + c] = h;
            out[(size_t)m * p.pitch + c] = from_f32<T>(acc);
#pragma unroll
            for (int j = 0; j + 1 < kMaxTaps; j++) hist[j] = hist[j + 1];
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(kThreads) norm_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ out,
                                                        const int* __restrict__ rows, const int* __restrict__ row_index, int gather,
                                                        int width, int pitch, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[33];
    int src = blockIdx.x;
    if (gather) src = rows != nullptr ? rows[src] : (row_index != nullptr ? row_index[0] + src : src);
    const float* xr = x + (size_t)src * width;
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += kThreads) { const float v = xr[c]; ss = fmaf(v, v, ss); }
    ss = block_sum(ss, red);
    const float rstd = rsqrtf(ss / (float)width + eps);
    T* o = out + (size_t)blockIdx.x * pitch;
    for (int c = threadIdx.x; c < width; c += kThreads) o[c] = from_f32<T>(xr[c] * rstd * w[c]);
}

// a N(z) + b N(z^2) + c N(z^3) + e, N: over the root mean square of the row.
template <typename T>
__global__ void __launch_bounds__(kThreads) polynorm_kernel(const T* __restrict__ z, T* __restrict__ out, int width, int pitch, float a, float b,
                                                            float c, float e, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[33];
    const T* zr = z + (size_t)blockIdx.x * pitch;
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    for (int i = threadIdx.x; i < width; i += kThreads) {
        const float v = to_f32<T>(zr[i]), q = v * v, u = q * v;
        s1 += q;
        s2 = fmaf(q, q, s2);
        s3 = fmaf(u, u, s3);
    }
    s1 = block_sum(s1, red);
    s2 = block_sum(s2, red);
    s3 = block_sum(s3, red);
    const float n = (float)width;
    const float ka = a * rsqrtf(s1 / n + eps), kb = b * rsqrtf(s2 / n + eps), kc = c * rsqrtf(s3 / n + eps);
    T* o = out + (size_t)blockIdx.x * pitch;
    for (int i = threadIdx.x; i < width; i += kThreads) {
        const float v = to_f32<T>(zr[i]);
        o[i] = from_f32<T>(fmaf(v, fmaf(v, fmaf(v, kc, kb), ka), e));
    }
}

__global__ void add_kernel(float* __restrict__ x, const float* __restrict__ y, size_t n) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += y[i];
}

}  // namespace

int launch_embed(const b200_hybrid_model& m, const b200_hybrid_pass& p, cudaStream_t st) {
    launch_kernel(embed_kernel, dim3(p.M), dim3(kThreads), 0, st, p.tokens, static_cast<const bf16*>(m.embed), m.width, m.vocab, m.x,
                  m.injects ? m.emb : static_cast<float*>(nullptr));
    return check_launch();
}

int launch_norm_conv(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p,
                     cudaStream_t st) {
    NormConvParams q{};
    q.x = m.x; q.w = l.norm1; q.conv = l.conv;
    q.state = reinterpret_cast<const float*>(static_cast<const char*>(p.cache) + r.conv_off);
    q.pend = reinterpret_cast<float*>(static_cast<char*>(m.pending) + r.pend_h);
    q.out = m.hb; q.mask = p.mask; q.pos = p.pos; q.tail_pos = p.tail_pos;
    q.M = p.M; q.width = m.width; q.pitch = round_up(m.width, 64); q.taps = l.taps; q.write_off = p.write_off; q.tree = p.tree;
    q.eps = m.eps;
    const int grid = p.tree ? p.M : (p.M + kRowsPerCta - 1) / kRowsPerCta;
    if (m.act_type == B200_ACT_F32) launch_kernel(norm_conv_kernel<float>, dim3(grid), dim3(kThreads), 0, st, q);
    else launch_kernel(norm_conv_kernel<bf16>, dim3(grid), dim3(kThreads), 0, st, q);
    return check_launch();
}

int launch_norm(const b200_hybrid_model& m, const float* w, const b200_hybrid_pass& p, bool gather, int rows, cudaStream_t st) {
    const int pitch = round_up(m.width, 64), g = gather ? 1 : 0;
    if (m.act_type == B200_ACT_F32)
        launch_kernel(norm_kernel<float>, dim3(rows), dim3(kThreads), 0, st, static_cast<const float*>(m.x), w, static_cast<float*>(m.hb),
                      p.out_rows, p.row_index, g, m.width, pitch, m.eps);
    else
        launch_kernel(norm_kernel<bf16>, dim3(rows), dim3(kThreads), 0, st, static_cast<const float*>(m.x), w, static_cast<bf16*>(m.hb),
                      p.out_rows, p.row_index, g, m.width, pitch, m.eps);
    return check_launch();
}

int launch_polynorm(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, cudaStream_t st) {
    const int pitch = round_up(l.ff, 64);
    if (m.act_type == B200_ACT_F32)
        launch_kernel(polynorm_kernel<float>, dim3(rows), dim3(kThreads), 0, st, static_cast<const float*>(m.zb), static_cast<float*>(m.zab),
                      l.ff, pitch, l.act[0], l.act[1], l.act[2], l.act[3], m.eps);
    else
        launch_kernel(polynorm_kernel<bf16>, dim3(rows), dim3(kThreads), 0, st, static_cast<const bf16*>(m.zb), static_cast<bf16*>(m.zab),
                      l.ff, pitch, l.act[0], l.act[1], l.act[2], l.act[3], m.eps);
    return check_launch();
}

int launch_add(float* x, const float* y, size_t n, cudaStream_t st) {
    launch_kernel(add_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, x, y, n);
    return check_launch();
}

}  // namespace hybrid
}  // namespace b200
