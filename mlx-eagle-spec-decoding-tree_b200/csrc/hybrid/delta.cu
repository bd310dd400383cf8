// Gated delta rule of the hybrid decoders, one decay per head and key channel:
//     S <- g * S (rows);   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q,
// q and k unit vectors; q, k, v come out of short causal convolutions with silu.  Everything that enters the recurrence is
// fp32, the state [heads][vdim][dim] is carried in the request's cache, as are the convolutions' last inputs.  Decays are kept
// as g - 1 and applied as S <- S + (g - 1) S: a decay next to 1, rounded, would change a state by as much as it loses over
// thousands of tokens.
//
//   conv_kernel    convolution, silu and unit norm: a warp per head of q, k or v and block of rows.
//   scan_kernel    token by token.  CTA = (head, 32 state columns); 8 lanes share a column and hold its rows in registers (packed
//                  pairs), so the read-out of k before the write takes three shuffles; tokens come in blocks through shared
//                  memory and the lanes' parts of the outputs are added for 8 tokens at once.  Three forms:
//                    chain   the pass's rows in order; the new state and convolution inputs are written back;
//                    tree    a CTA per row replays the row's path from the state, nothing is written back;
//                    commit  pending rows are replayed and written back, no output.
//   step_kernel    one token: convolution, unit norms, the step of the state, head norm and output gate, a CTA per head.
//   conv_chunk_kernel, chunk_scan_kernel
//                  prompts: 8 tokens at a time.  With P_j the product of the chunk's decays up to token j and P_ij that of the
//                  tokens after i up to j (products of decays only, nothing is divided),
//                      u_j = beta_j (v_j - S^T (P_j k_j) - sum_{i<j} (k_j . P_ij k_i) u_i),
//                      o_j = S^T (P_j q_j) + sum_{i<=j} (q_j . P_ij k_i) u_i,      S <- P_7 S + sum_i (P_i7 k_i) u_i^T
//                  with S the state before the chunk: the read-outs of all 8 tokens are independent of each other.  The vectors
//                  and the 8 x 8 coefficients do not depend on the column and come out of the convolution kernel.
#include "scan.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kThreads = 256;
constexpr int kConvRows = 8;             // chain rows of a warp
constexpr int kLanes = 8;                // lanes of a state column
constexpr int kMaxDim = 256;
enum : int { kChain = 0, kTree = 1, kCommit = 2 };

struct ConvParams {
    const void* in;          // chain: [M][pitch]; tree: pending rows [64][pitch]
    const void* state;       // [taps - 1][pitch] committed inputs, oldest first
    const float* w;          // [taps][channels]
    const unsigned long long* mask;
    float* q;                // [M][G * d]
    float* k;                // [M][G * d], tree: pending rows from write_off on
    void* v;                 // [M][H * dv], likewise
    int M, G, H, d, dv, taps, pitch, channels, write_off;
};

// A lane holds NI vectors of V neighbouring channels.
template <typename T, int V> __device__ __forceinline__ void ld_vec(float (&r)[V], const T* p) {
    if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        r[0] = __uint_as_float(u.x << 16);
        r[1] = __uint_as_float(u.x & 0xffff0000u);
        r[2] = __uint_as_float(u.y << 16);
        r[3] = __uint_as_float(u.y & 0xffff0000u);
    } else {
#pragma unroll
        for (int e = 0; e < V; e++) r[e] = to_f32<T>(p[e]);
    }
}

template <typename T, int V, int NI, bool TREE>
__global__ void __launch_bounds__(kThreads) conv_kernel(const ConvParams p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int R = TREE ? 1 : kConvRows;
    __shared__ const T* s_src[B200_HYBRID_MAX_TAPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = blockIdx.y * R, rows = min(R, p.M - r0);
    const T* in = static_cast<const T*>(p.in);
    const T* state = static_cast<const T*>(p.state);
    if (TREE) {                              // the row's inputs along its path: ancestors (set bits of its mask), then committed ones
        if (threadIdx.x == 0) {
            const int self = p.write_off + r0;
            unsigned long long anc = p.mask[r0] & ((1ull << self) - 1ull);
            int have = 0;
            s_src[p.taps - 1] = in + (size_t)self * p.pitch;
            for (int j = p.taps - 2; j >= 0; j--) {
                if (anc != 0ull) {
                    const int a = 63 - __clzll((long long)anc);
                    anc &= ~(1ull << a);
                    have++;
                    s_src[j] = in + (size_t)a * p.pitch;
                } else {
                    s_src[j] = state + (size_t)(j + have) * p.pitch;
                }
            }
        }
        __syncthreads();
    }
    const int unit = blockIdx.x * (kThreads / 32) + warp;
    if (unit >= 2 * p.G + p.H) return;
    const bool value = unit >= 2 * p.G;
    const int n = value ? p.dv : p.d, c0 = value ? 2 * p.G * p.d + (unit - 2 * p.G) * p.dv : unit * p.d;
    float acc[R][NI][V];
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int e = 0; e < V; e++) acc[r][i][e] = 0.f;
    for (int j = 0; j < p.taps; j++) {
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const int c = (lane + 32 * i) * V;
            if (c >= n) continue;
            float w[V];
#pragma unroll
            for (int e = 0; e < V; e++) w[e] = p.w[(size_t)j * p.channels + c0 + c + e];
#pragma unroll
            for (int r = 0; r < R; r++) {
                if (r >= rows) continue;
                const int row = r0 + r - (p.taps - 1) + j;
                const T* src = TREE ? s_src[j] : (row >= 0 ? in + (size_t)row * p.pitch : state + (size_t)(row + p.taps - 1) * p.pitch);
                float x[V];
                ld_vec<T, V>(x, src + c0 + c);
#pragma unroll
                for (int e = 0; e < V; e++) acc[r][i][e] = fmaf(w[e], x[e], acc[r][i][e]);
            }
        }
    }
    const float scale = unit < p.G ? rsqrtf((float)p.d) : 1.f;
#pragma unroll
    for (int r = 0; r < R; r++) {
        if (r >= rows) continue;
        const int m = r0 + r;
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int e = 0; e < V; e++) {
                const float z = acc[r][i][e];        // (channels past the head are zero)
                acc[r][i][e] = z * sigmoid_f(z);
                ss = fmaf(acc[r][i][e], acc[r][i][e], ss);
            }
        float f = 1.f;
        if (!value) f = rsqrtf(warp_sum(ss) + 1e-6f) * scale;
#pragma unroll
        for (int i = 0; i < NI; i++) {
            const int c = (lane + 32 * i) * V;
            if (c >= n) continue;
            if (value) {
                T* dst = static_cast<T*>(p.v) + ((size_t)m * p.H + unit - 2 * p.G) * p.dv + c;
#pragma unroll
                for (int e = 0; e < V; e++) dst[e] = from_f32<T>(acc[r][i][e]);
            } else {
                float* dst = (unit < p.G ? p.q : p.k) + ((size_t)m * p.G + (unit < p.G ? unit : unit - p.G)) * p.d + c;
                if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(acc[r][i][0] * f, acc[r][i][1] * f, acc[r][i][2] * f, acc[r][i][3] * f);
                else dst[0] = acc[r][i][0] * f;
            }
        }
    }
}

// ---------------------------------------------------------------- 8 tokens at a time
constexpr int kChunk = 8;

// Sum of v[i] over the warp's lanes, for 32 values at once: lane i gets the total of v[i].
__device__ __forceinline__ float transpose_sum32(float (&v)[32], int lane) {
#pragma unroll
    for (int s = 16; s > 0; s >>= 1)
#pragma unroll
        for (int i = 0; i < s; i++) {
            const bool up = (lane & s) != 0;
            const float keep = up ? v[i + s] : v[i], send = up ? v[i] : v[i + s];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, s);
        }
    return v[0];
}

struct ChunkParams {
    ConvParams c;            // (q, k unused)
    const float* g;          // [M][H * d], decays - 1
    float* kt;               // [M][H * d]: P_j k_j
    float* qt;               // P_j q_j
    float* kh;               // P_j7 k_j
    float* decay;            // [chunks][H * d]: P_7 - 1
    float* coef;             // [chunks][H][2][8][8]: k_j . P_ij k_i (i < j), q_j . P_ij k_i (i <= j), zeros elsewhere
};

// silu(convolution) of 8 rows from r0 on, the lane's 4 channels from c on (n of them in the head).
template <typename T, int TAPS>
__device__ __forceinline__ void conv_rows(const ConvParams& p, int r0, int rows, int c, bool in_head, float (&y)[kChunk][4]) {
    constexpr int X = kChunk + TAPS - 1;
    const T* in = static_cast<const T*>(p.in);
    const T* state = static_cast<const T*>(p.state);
    float x[X][4], w[TAPS][4];
#pragma unroll
    for (int i = 0; i < X; i++) {
        const int row = r0 + i - (TAPS - 1);
#pragma unroll
        for (int e = 0; e < 4; e++) x[i][e] = 0.f;
        if (in_head && row < r0 + rows) ld_vec<T, 4>(x[i], (row >= 0 ? in + (size_t)row * p.pitch : state + (size_t)(row + TAPS - 1) * p.pitch) + c);
    }
#pragma unroll
    for (int j = 0; j < TAPS; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) w[j][e] = in_head ? p.w[(size_t)j * p.channels + c + e] : 0.f;
#pragma unroll
    for (int r = 0; r < kChunk; r++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            float z = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; j++) z = fmaf(w[j][e], x[r + j][e], z);
            y[r][e] = z * sigmoid_f(z);
        }
}

// Warp = (chunk, key head) or (chunk, value head); heads of at most 128 channels, multiples of 4.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_chunk_kernel(const ChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const ConvParams& cp = p.c;
    const int lane = threadIdx.x & 31, unit = blockIdx.x * 4 + (threadIdx.x >> 5), chunk = blockIdx.y, r0 = chunk * kChunk;
    const int rows = min(kChunk, cp.M - r0), c = lane * 4, d = cp.d, G = cp.G, H = cp.H;
    if (unit >= G + H) return;
    if (unit >= G) {
        const int h = unit - G;
        const bool in = c < cp.dv;
        float y[kChunk][4];
        conv_rows<T, TAPS>(cp, r0, rows, 2 * G * d + h * cp.dv + c, in, y);
#pragma unroll
        for (int r = 0; r < kChunk; r++) {
            if (!in || r >= rows) continue;
            T* dst = static_cast<T*>(cp.v) + ((size_t)(r0 + r) * H + h) * cp.dv + c;
            if constexpr (sizeof(T) == 4) {
                *reinterpret_cast<float4*>(dst) = make_float4(y[r][0], y[r][1], y[r][2], y[r][3]);
            } else {
                const __nv_bfloat162 a = __floats2bfloat162_rn(y[r][0], y[r][1]), b = __floats2bfloat162_rn(y[r][2], y[r][3]);
                *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
            }
        }
        return;
    }
    const bool in = c < d;
    float q[kChunk][4], k[kChunk][4];
    conv_rows<T, TAPS>(cp, r0, rows, unit * d + c, in, q);
    conv_rows<T, TAPS>(cp, r0, rows, (G + unit) * d + c, in, k);
    const float scale = rsqrtf((float)d);
#pragma unroll
    for (int r = 0; r < kChunk; r++) {
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int e = 0; e < 4; e++) { sq = fmaf(q[r][e], q[r][e], sq); sk = fmaf(k[r][e], k[r][e], sk); }
        const float fq = rsqrtf(warp_sum(sq) + 1e-6f) * scale, fk = rsqrtf(warp_sum(sk) + 1e-6f);
#pragma unroll
        for (int e = 0; e < 4; e++) { q[r][e] *= fq; k[r][e] *= fk; }
    }
    // (rows past the pass are zero: zero inputs, or a head's zero channels)
#pragma unroll
    for (int r = 0; r < kChunk; r++)
#pragma unroll
        for (int e = 0; e < 4; e++)
            if (r >= rows) q[r][e] = k[r][e] = 0.f;
    const int R = H / G;
    for (int h = unit * R; h < (unit + 1) * R; h++) {
        float g[kChunk][4];
#pragma unroll
        for (int r = 0; r < kChunk; r++) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (in && r < rows) x = *reinterpret_cast<const float4*>(p.g + ((size_t)(r0 + r) * H + h) * d + c);
            g[r][0] = x.x; g[r][1] = x.y; g[r][2] = x.z; g[r][3] = x.w;
        }
        float P[4] = {0.f, 0.f, 0.f, 0.f};                   // products - 1: (1 + a)(1 + b) - 1 = a + b + ab
#pragma unroll
        for (int r = 0; r < kChunk; r++) {
#pragma unroll
            for (int e = 0; e < 4; e++) P[e] = fmaf(P[e], g[r][e], P[e] + g[r][e]);
            if (in && r < rows) {
                const size_t at = ((size_t)(r0 + r) * H + h) * d + c;
                *reinterpret_cast<float4*>(p.kt + at) = make_float4(fmaf(P[0], k[r][0], k[r][0]), fmaf(P[1], k[r][1], k[r][1]), fmaf(P[2], k[r][2], k[r][2]), fmaf(P[3], k[r][3], k[r][3]));
                *reinterpret_cast<float4*>(p.qt + at) = make_float4(fmaf(P[0], q[r][0], q[r][0]), fmaf(P[1], q[r][1], q[r][1]), fmaf(P[2], q[r][2], q[r][2]), fmaf(P[3], q[r][3], q[r][3]));
            }
        }
        if (in) *reinterpret_cast<float4*>(p.decay + ((size_t)chunk * H + h) * d + c) = make_float4(P[0], P[1], P[2], P[3]);
        float* coef = p.coef + ((size_t)chunk * H + h) * 2 * kChunk * kChunk;
        *reinterpret_cast<float4*>(coef + lane * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
        __syncwarp();
        // for every i: k_j . P_ij k_i for j > i, then q_j . P_ij k_i for j >= i; 64 sums in all, 32 at a time
        float v[32];
#pragma unroll
        for (int i = 0, n = 0; i < kChunk; i++) {
            float qd[kChunk], w[4];
#pragma unroll
            for (int e = 0; e < 4; e++) w[e] = k[i][e];
            auto put = [&](float x) {
                v[n & 31] = x;
                n++;
                if ((n & 31) == 0) {
                    const float total = transpose_sum32(v, lane);
                    int at = n - 32 + lane, ii = 0;
                    while (at >= 15 - 2 * ii) { at -= 15 - 2 * ii; ii++; }
                    const bool first = at < 7 - ii;
                    const int jj = first ? ii + 1 + at : ii + at - (7 - ii);
                    coef[(first ? 0 : kChunk * kChunk) + jj * kChunk + ii] = total;
                }
            };
#pragma unroll
            for (int j = i; j < kChunk; j++) {
                if (j > i)
#pragma unroll
                    for (int e = 0; e < 4; e++) w[e] = fmaf(w[e], g[j][e], w[e]);
                qd[j] = w[0] * q[j][0] + w[1] * q[j][1] + w[2] * q[j][2] + w[3] * q[j][3];
                if (j > i) put(w[0] * k[j][0] + w[1] * k[j][1] + w[2] * k[j][2] + w[3] * k[j][3]);
            }
#pragma unroll
            for (int j = i; j < kChunk; j++) put(qd[j]);
            if (in && i < rows) *reinterpret_cast<float4*>(p.kh + ((size_t)(r0 + i) * H + h) * d + c) = make_float4(w[0], w[1], w[2], w[3]);
        }
    }
}

struct ScanParams {
    const float* q;          // [M][G * d]
    const float* k;          // chain: [M][G * d]; tree, commit: pending rows
    const float* g;          // [..][H * d], decays - 1
    const float* beta;       // [..][H]
    const void* v;           // [..][H * dv]
    float* state;            // [H][dv][d]
    float* o;                // [M][H * dv]
    const void* in;          // convolution inputs [..][pitch]
    void* conv_state;        // [taps - 1][pitch]
    const unsigned long long* mask;
    const int* count;        // commit: as b200_hybrid_commit
    const int* rows;
    int M, H, G, d, dv, taps, pitch, channels, tree_rows;
};

__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(dst), "l"(src) : "memory");
}

// Sum of v[i] over groups of 8 neighbouring lanes, for 8 values at once: lane i of a group gets the total of v[i].
__device__ __forceinline__ float transpose_sum8(float (&v)[8], int lane) {
#pragma unroll
    for (int s = 4; s > 0; s >>= 1)
#pragma unroll
        for (int i = 0; i < s; i++) {
            const bool up = (lane & s) != 0;
            const float keep = up ? v[i + s] : v[i], send = up ? v[i] : v[i + s];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, s);
        }
    return v[0];
}

// The convolutions' last inputs after n rows, channels over all CTAs of the grid.
template <typename T, typename RowOf>
__device__ __forceinline__ void roll_inputs(const ScanParams& p, int n, RowOf row_of) {
    const int prev = p.taps - 1, first = (blockIdx.y * gridDim.x + blockIdx.x) * blockDim.x + threadIdx.x;
    const T* in = static_cast<const T*>(p.in);
    T* cs = static_cast<T*>(p.conv_state);
    if (prev == 0) return;
    for (int c = first; c < p.channels; c += gridDim.x * gridDim.y * blockDim.x) {
        T nv[B200_HYBRID_MAX_TAPS];
#pragma unroll
        for (int e = 0; e < B200_HYBRID_MAX_TAPS; e++)
            if (e < prev) {
                const int i = n - prev + e;
                nv[e] = i >= 0 ? in[(size_t)row_of(i) * p.pitch + c] : cs[(size_t)(i + prev) * p.pitch + c];
            }
#pragma unroll
        for (int e = 0; e < B200_HYBRID_MAX_TAPS; e++)
            if (e < prev) cs[(size_t)e * p.pitch + c] = nv[e];
    }
}

struct ChunkScanParams {
    ScanParams s;
    const float* kt;
    const float* qt;
    const float* kh;
    const float* decay;
    const float* coef;
};

// CTA = (head, 32 state columns), warp = 4 columns: 16 lanes share 2 columns and hold their rows.
//
// The read-outs of 4 tokens, of k and of q, for 2 columns are 16 sums over 16 lanes.  Lane j keeps them in an order of its own, sum
// x in register x ^ j, so that adding them across lanes takes 15 shuffles and additions and no selection, and leaves sum j with
// lane j: in the step of bit s every lane keeps the registers without the bit and sends the others.
template <typename T, int RPL>           // state rows of a lane
__global__ void __launch_bounds__(kThreads, 1) chunk_scan_kernel(const ChunkScanParams cp) {
    pdl_launch_dependents();
    constexpr int D = 16 * RPL, C = kChunk;
    constexpr int STAGE = 3 * C * D + D + 2 * C * C + C + C * 32;       // floats (values: room for fp32)
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* stages = reinterpret_cast<float*>(smem_raw);
    __shared__ float s_read[8][2][C][4];                 // per warp
    __shared__ __align__(16) float2 s_u[8][C][4];        // (each value twice: a packed pair)
    const ScanParams& p = cp.s;
    const int h = blockIdx.y, c0 = blockIdx.x * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, j = lane & 15, grp = lane >> 4;
    const int d = p.d, dv = p.dv, n = p.M, ncol = min(32, dv - c0);
    const bool wide_v = dv * (int)sizeof(T) % 16 == 0;
    for (int i = tid; i < 2 * STAGE; i += kThreads) stages[i] = 0.f;      // rows past the head's width, columns past its values
    pdl_wait();
    __syncthreads();
    auto fetch = [&](int b) {
        float* st = stages + (b & 1) * STAGE;
        const int t0 = b * C, nt = min(C, n - t0), t = warp;
        const size_t row = (size_t)(t0 + t) * p.H + h, ch = (size_t)b * p.H + h;
        float* at = st + 3 * C * D;
        float* beta = at + D + 2 * C * C;
        T* v = reinterpret_cast<T*>(beta + C);
        if (t < nt) {
            fetch_row(st + t * D, cp.kt + row * d, d, true, lane);
            fetch_row(st + (C + t) * D, cp.qt + row * d, d, true, lane);
            fetch_row(st + (2 * C + t) * D, cp.kh + row * d, d, true, lane);
            fetch_row(v + t * 32, static_cast<const T*>(p.v) + row * dv + c0, ncol, wide_v, lane);
            if (lane == 0) cp_async4(smem_u32(beta + t), p.beta + row);
        } else {
            for (int c = lane; c < D; c += 32) st[t * D + c] = st[(C + t) * D + c] = st[(2 * C + t) * D + c] = 0.f;
            if (lane == 0) beta[t] = 0.f;
        }
        if (warp == 0) fetch_row(at, cp.decay + ch * d, d, true, lane);
        if (warp == 1) fetch_row(at + D, cp.coef + ch * 2 * C * C, 2 * C * C, true, lane);
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    fetch(0);
    // register column c of a lane: column c ^ (j & 1) of its group's two
    unsigned long long S[RPL / 2][2];                    // rows 64 i + 4 j + (0 .. 3), in pairs
    const int col = c0 + warp * 4 + grp * 2;
#pragma unroll
    for (int i = 0; i < RPL / 4; i++)
#pragma unroll
        for (int c = 0; c < 2; c++) {
            const int r = 64 * i + 4 * j, cc = col + (c ^ (j & 1));
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < d && cc < dv) x = *reinterpret_cast<const float4*>(p.state + ((size_t)h * dv + cc) * d + r);
            S[2 * i][c] = pack2(x.x, x.y);
            S[2 * i + 1][c] = pack2(x.z, x.w);
        }
    const int nb = (n + C - 1) / C, mycol = lane & 3, mytok = lane >> 2;
    // sum x = 8 (token bit 1) + 4 (token bit 0) + 2 (k or q) + column; where register x of this lane reads
    int src[4][2];
#pragma unroll
    for (int t = 0; t < 4; t++)
#pragma unroll
        for (int kind = 0; kind < 2; kind++) src[t][kind] = ((kind ^ ((j >> 1) & 1)) * C + (t ^ (j >> 2))) * D + 4 * j;
    for (int b = 0; b < nb; b++) {
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                                 // this chunk is here, the one before has been read
        if (b + 1 < nb) fetch(b + 1);
        const float* st = stages + (b & 1) * STAGE;
        const float* at = st + 3 * C * D;
        const float* beta = at + D + 2 * C * C;
        const T* v = reinterpret_cast<const T*>(beta + C);
        // read-outs of the state before the chunk, four tokens at a time
#pragma unroll
        for (int t0 = 0; t0 < C; t0 += 4) {
            float y[16];
#pragma unroll
            for (int t = 0; t < 4; t++)
#pragma unroll
                for (int kind = 0; kind < 2; kind++) {
                    unsigned long long a[2] = {0ull, 0ull};
#pragma unroll
                    for (int i = 0; i < RPL / 4; i++) {
                        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(st + src[t][kind] + t0 * D + 64 * i);
#pragma unroll
                        for (int c = 0; c < 2; c++) a[c] = fma2(w.y, S[2 * i + 1][c], fma2(w.x, S[2 * i][c], a[c]));
                    }
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        const float2 z = unpack2(a[c]);
                        y[t * 4 + kind * 2 + c] = z.x + z.y;
                    }
                }
#pragma unroll
            for (int s = 8; s > 0; s >>= 1)
#pragma unroll
                for (int x = 0; x < s; x++) y[x] += __shfl_xor_sync(0xffffffffu, y[x + s], s);
            s_read[warp][(j >> 1) & 1][t0 + (j >> 2)][grp * 2 + (j & 1)] = y[0];
        }
        __syncwarp();
        // what each token writes: every lane solves its column, and finishes one token's output
        float u[C];
#pragma unroll
        for (int t = 0; t < C; t++) {
            float r = s_read[warp][0][t][mycol];
            const float4 a0 = *reinterpret_cast<const float4*>(at + D + t * C), a1 = *reinterpret_cast<const float4*>(at + D + t * C + 4);
            const float a[C] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
#pragma unroll
            for (int i = 0; i < t; i++) r = fmaf(a[i], u[i], r);
            u[t] = beta[t] * (to_f32<T>(v[t * 32 + warp * 4 + mycol]) - r);
            if (t == mytok) s_u[warp][t][mycol] = make_float2(u[t], u[t]);
        }
        {
            float o = s_read[warp][1][mytok][mycol];
            const float4 b0 = *reinterpret_cast<const float4*>(at + D + C * C + mytok * C), b1 = *reinterpret_cast<const float4*>(at + D + C * C + mytok * C + 4);
            o = fmaf(b0.x, u[0], fmaf(b0.y, u[1], fmaf(b0.z, u[2], fmaf(b0.w, u[3], o))));
            o = fmaf(b1.x, u[4], fmaf(b1.y, u[5], fmaf(b1.z, u[6], fmaf(b1.w, u[7], o))));
            const int m = b * C + mytok, cc = c0 + warp * 4 + mycol;
            if (m < n && cc < dv) p.o[((size_t)m * p.H + h) * dv + cc] = o;
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < RPL / 4; i++) {
            const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(at + 64 * i + 4 * j);
#pragma unroll
            for (int c = 0; c < 2; c++) {
                S[2 * i][c] = fma2(w.x, S[2 * i][c], S[2 * i][c]);
                S[2 * i + 1][c] = fma2(w.y, S[2 * i + 1][c], S[2 * i + 1][c]);
            }
        }
#pragma unroll
        for (int t = 0; t < C; t++) {
            unsigned long long u2[2];
#pragma unroll
            for (int c = 0; c < 2; c++) u2[c] = *reinterpret_cast<const unsigned long long*>(&s_u[warp][t][grp * 2 + (c ^ (j & 1))]);
#pragma unroll
            for (int i = 0; i < RPL / 4; i++) {
                const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(st + (2 * C + t) * D + 64 * i + 4 * j);
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    S[2 * i][c] = fma2(w.x, u2[c], S[2 * i][c]);
                    S[2 * i + 1][c] = fma2(w.y, u2[c], S[2 * i + 1][c]);
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RPL / 4; i++)
#pragma unroll
        for (int c = 0; c < 2; c++) {
            const int r = 64 * i + 4 * j, cc = col + (c ^ (j & 1));
            const float2 x = unpack2(S[2 * i][c]), y = unpack2(S[2 * i + 1][c]);
            if (r < d && cc < dv) *reinterpret_cast<float4*>(p.state + ((size_t)h * dv + cc) * d + r) = make_float4(x.x, x.y, y.x, y.y);
        }
    roll_inputs<T>(p, n, [](int t) { return t; });
}

template <int RPL> __host__ __device__ constexpr int scan_block() { return RPL == 32 ? 8 : 16; }      // tokens of a shared-memory block

template <typename T, int RPL, int MODE>         // state rows of a lane
__global__ void __launch_bounds__(kThreads) scan_kernel(const ScanParams p) {
    pdl_launch_dependents();
    constexpr int D = kLanes * RPL, TB = scan_block<RPL>(), STAGES = 2;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* sg = reinterpret_cast<float*>(smem_raw);      // [STAGES][TB][D]
    float* sk = sg + STAGES * TB * D;
    float* sq = sk + STAGES * TB * D;
    float* sb = sq + STAGES * TB * D;                    // [STAGES][TB]
    T* sv = reinterpret_cast<T*>(sb + STAGES * TB);      // [STAGES][TB][32]
    __shared__ int s_row[B200_HYBRID_PENDING];
    const int h = blockIdx.y, c0 = blockIdx.x * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kh = h / (p.H / p.G), d = p.d, dv = p.dv, m = blockIdx.z;
    const int ncol = min(32, dv - c0), col = c0 + warp * 4 + (lane >> 3), j = lane & 7;
    const bool wide = d % 4 == 0, wide_v = dv * (int)sizeof(T) % 16 == 0;
    // what the copies never write stays zero: rows past the head's width, columns past its values, queries that are not asked for
    for (int i = tid; i < STAGES * TB * D; i += kThreads) { sg[i] = 0.f; sk[i] = 0.f; sq[i] = 0.f; }
    for (int i = tid; i < STAGES * TB * 32; i += kThreads) sv[i] = from_f32<T>(0.f);
    pdl_wait();
    int n = p.M;
    if (MODE == kTree) {
        const unsigned long long path = p.mask[m];
        n = __popcll(path);
        if (tid < B200_HYBRID_PENDING && ((path >> tid) & 1ull)) s_row[__popcll(path & ((1ull << tid) - 1ull))] = tid;
    } else if (MODE == kCommit) {
        n = min(max(p.count[0] + 1, 0), B200_HYBRID_PENDING);
        for (int i = tid; i < n; i += kThreads) {
            int s = i == 0 || p.rows == nullptr ? i : p.rows[i];
            if (s < 0) s += p.tree_rows;
            s_row[i] = min(max(s, 0), B200_HYBRID_PENDING - 1);
        }
    }
    __syncthreads();
    auto row_of = [&](int t) { return MODE == kChain ? t : s_row[t]; };
    auto fetch = [&](int b) {
        const int st = (b & 1) * TB, t0 = b * TB;
        for (int t = warp; t < TB && t0 + t < n; t += kThreads / 32) {
            const int row = row_of(t0 + t);
            fetch_row(sg + (st + t) * D, p.g + ((size_t)row * p.H + h) * d, d, wide, lane);
            fetch_row(sk + (st + t) * D, p.k + ((size_t)row * p.G + kh) * d, d, wide, lane);
            if (MODE == kChain) fetch_row(sq + (st + t) * D, p.q + ((size_t)row * p.G + kh) * d, d, wide, lane);
            if (MODE == kTree && t0 + t == n - 1) fetch_row(sq + (st + t) * D, p.q + ((size_t)m * p.G + kh) * d, d, wide, lane);
            fetch_row(sv + (st + t) * 32, static_cast<const T*>(p.v) + ((size_t)row * p.H + h) * dv + c0, ncol, wide_v, lane);
            if (lane == 0) cp_async4(smem_u32(sb + st + t), p.beta + (size_t)row * p.H + h);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    fetch(0);
    unsigned long long S[RPL / 2];                       // state rows 32 i + 4 j + (0 .. 3) of the column, in pairs
    float* sbase = p.state + ((size_t)h * dv + min(col, dv - 1)) * d;
#pragma unroll
    for (int i = 0; i < RPL / 4; i++) {
        const int r = 32 * i + 4 * j;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (wide) {
            if (r < d) x = *reinterpret_cast<const float4*>(sbase + r);
        } else {
            if (r < d) x.x = sbase[r];
            if (r + 1 < d) x.y = sbase[r + 1];
            if (r + 2 < d) x.z = sbase[r + 2];
            if (r + 3 < d) x.w = sbase[r + 3];
        }
        S[2 * i] = pack2(x.x, x.y);
        S[2 * i + 1] = pack2(x.z, x.w);
    }
    const int nb = (n + TB - 1) / TB;
    for (int b = 0; b < nb; b++) {
        const int st = (b & 1) * TB, t0 = b * TB;
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                                 // this block is here, the one before has been read
        if (b + 1 < nb) fetch(b + 1);
#pragma unroll 1
        for (int tg = 0; tg < TB && t0 + tg < n; tg += 8) {
            const int nt = min(8, n - t0 - tg);
            float y[8];                                  // this lane's rows
#pragma unroll
            for (int t = 0; t < 8; t++) {
                y[t] = 0.f;
                if (t >= nt) continue;
                const int at = st + tg + t;
                const ulonglong2* g4 = reinterpret_cast<const ulonglong2*>(sg + at * D + 4 * j);
                const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(sk + at * D + 4 * j);
                const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(sq + at * D + 4 * j);
                const float v = to_f32<T>(sv[at * 32 + warp * 4 + (lane >> 3)]), beta = sb[at];
                unsigned long long k2[RPL / 2], a0 = 0ull, a1 = 0ull;
#pragma unroll
                for (int i = 0; i < RPL / 4; i++) {
                    const ulonglong2 g = g4[8 * i], k = k4[8 * i];
                    k2[2 * i] = k.x;
                    k2[2 * i + 1] = k.y;
                    S[2 * i] = fma2(S[2 * i], g.x, S[2 * i]);
                    S[2 * i + 1] = fma2(S[2 * i + 1], g.y, S[2 * i + 1]);
                    a0 = fma2(k.x, S[2 * i], a0);
                    a1 = fma2(k.y, S[2 * i + 1], a1);
                }
                const float2 x0 = unpack2(a0), x1 = unpack2(a1);
                float r = (x0.x + x0.y) + (x1.x + x1.y);
#pragma unroll
                for (int o = 1; o < kLanes; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
                const float u = beta * (v - r);
                const unsigned long long u2 = pack2(u, u);
                a0 = 0ull;
                a1 = 0ull;
#pragma unroll
                for (int i = 0; i < RPL / 4; i++) {
                    S[2 * i] = fma2(k2[2 * i], u2, S[2 * i]);
                    S[2 * i + 1] = fma2(k2[2 * i + 1], u2, S[2 * i + 1]);
                    if (MODE != kCommit) {
                        const ulonglong2 q = q4[8 * i];
                        a0 = fma2(q.x, S[2 * i], a0);
                        a1 = fma2(q.y, S[2 * i + 1], a1);
                    }
                }
                if (MODE != kCommit) {
                    const float2 z0 = unpack2(a0), z1 = unpack2(a1);
                    y[t] = (z0.x + z0.y) + (z1.x + z1.y);
                }
            }
            if (MODE == kCommit) continue;
            const float out = transpose_sum8(y, lane);
            const int t = t0 + tg + j;
            if (MODE == kChain) {
                if (j < nt && col < dv) p.o[((size_t)t * p.H + h) * dv + col] = out;
            } else if (t == n - 1 && col < dv) {
                p.o[((size_t)m * p.H + h) * dv + col] = out;
            }
        }
    }
    if (MODE == kTree) return;
    if (col < dv) {
#pragma unroll
        for (int i = 0; i < RPL / 4; i++) {
            const int r = 32 * i + 4 * j;
            const float2 x = unpack2(S[2 * i]), y = unpack2(S[2 * i + 1]);
            if (wide) {
                if (r < d) *reinterpret_cast<float4*>(sbase + r) = make_float4(x.x, x.y, y.x, y.y);
            } else {
                if (r < d) sbase[r] = x.x;
                if (r + 1 < d) sbase[r + 1] = x.y;
                if (r + 2 < d) sbase[r + 2] = y.x;
                if (r + 3 < d) sbase[r + 3] = y.y;
            }
        }
    }
    roll_inputs<T>(p, n, row_of);
}

template <typename T, int RPL, int MODE>
int launch_scan_r(const ScanParams& p, int rows, cudaStream_t st) {
    constexpr int TB = scan_block<RPL>(), D = kLanes * RPL;
    const size_t smem = 2 * TB * ((size_t)3 * D * 4 + 4 + 32 * sizeof(T));
    auto k = scan_kernel<T, RPL, MODE>;
    if (smem > 40 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return check_launch();
    launch_kernel(k, dim3((p.dv + 31) / 32, p.H, rows), dim3(kThreads), smem, st, p);
    return check_launch();
}
template <typename T, int MODE>
int launch_scan(const ScanParams& p, int rows, cudaStream_t st) {
    if (p.d <= 64) return launch_scan_r<T, 8, MODE>(p, rows, st);
    if (p.d <= 128) return launch_scan_r<T, 16, MODE>(p, rows, st);
    return launch_scan_r<T, 32, MODE>(p, rows, st);
}

template <typename T, int V, int NI>
void launch_conv_v(const ConvParams& p, bool tree, cudaStream_t st) {
    const int units = (2 * p.G + p.H + kThreads / 32 - 1) / (kThreads / 32);
    if (tree) launch_kernel(conv_kernel<T, V, NI, true>, dim3(units, p.M), dim3(kThreads), 0, st, p);
    else launch_kernel(conv_kernel<T, V, NI, false>, dim3(units, (p.M + kConvRows - 1) / kConvRows), dim3(kThreads), 0, st, p);
}

// ---------------------------------------------------------------- one token
struct StepParams {
    const void* in;          // [pitch] convolution inputs of the token
    void* conv_state;        // [taps - 1][pitch]
    const float* w;          // [taps][channels]
    const float* g;          // [H * d], decays - 1
    const float* beta;       // [H]
    float* state;            // [H][dv][d]
    const float* norm;       // [dv]
    const void* gate;        // [H * dv]
    void* out;               // [H * dv]
    int H, G, d, dv, taps, pitch, channels;
    float eps;
};

// CTA = head; the heads of one key head form a cluster, so that the convolution inputs they share move on after all have read
// them.  8 lanes per state column hold its rows; heads of at most 128 x 128, multiples of 4.
template <typename T>
__global__ void __launch_bounds__(kThreads) step_kernel(const StepParams p) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr int IT = 4, MAX = 128;
    __shared__ __align__(16) float sq[MAX], sk[MAX], sg[MAX], sv[MAX], so[MAX];
    __shared__ float red[33];
    const int h = blockIdx.x, R = p.H / p.G, kh = h / R, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, j = lane & 7, d = p.d, dv = p.dv;
    float4 S[IT][4];                                     // rows 32 i + 4 j + (0 .. 3) of column 32 it + 4 warp + lane / 8
    float* sbase = p.state + (size_t)h * dv * d;
#pragma unroll
    for (int it = 0; it < IT; it++)
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int col = 32 * it + 4 * warp + (lane >> 3), r = 32 * i + 4 * j;
            S[it][i] = col < dv && r < d ? *reinterpret_cast<const float4*>(sbase + (size_t)col * d + r) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    const T* in = static_cast<const T*>(p.in);
    T* cs = static_cast<T*>(p.conv_state);
    if (tid < MAX) {
        sg[tid] = tid < d ? p.g[(size_t)h * d + tid] : 0.f;
        sq[tid] = sk[tid] = sv[tid] = 0.f;
    }
    __syncthreads();
    T moved[2][B200_HYBRID_MAX_TAPS];                    // the channel's inputs after the token
    int chan[2];
#pragma unroll
    for (int x = 0; x < 2; x++) {
        const int e = tid + x * kThreads, which = e / MAX, c = e % MAX;
        const bool mine = which < 3 && c < (which == 2 ? dv : d);
        chan[x] = !mine ? -1 : (which == 2 ? 2 * p.G * d + h * dv + c : (which * p.G + kh) * d + c);
        if (!mine) continue;
        float z = 0.f;
#pragma unroll
        for (int t = 0; t < B200_HYBRID_MAX_TAPS; t++) {
            if (t >= p.taps) break;
            moved[x][t] = t == p.taps - 1 ? in[chan[x]] : cs[(size_t)t * p.pitch + chan[x]];
            z = fmaf(p.w[(size_t)t * p.channels + chan[x]], to_f32<T>(moved[x][t]), z);
        }
        z *= sigmoid_f(z);
        (which == 0 ? sq : (which == 1 ? sk : sv))[c] = which == 2 ? to_f32<T>(from_f32<T>(z)) : z;
    }
    if (R > 1) asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;\n" ::: "memory");
#pragma unroll
    for (int x = 0; x < 2; x++) {
        const bool key = tid + x * kThreads < 2 * MAX;   // (the key head's inputs move once)
        if (chan[x] < 0 || (key && h % R != 0)) continue;
#pragma unroll
        for (int t = 1; t < B200_HYBRID_MAX_TAPS; t++)
            if (t < p.taps) cs[(size_t)(t - 1) * p.pitch + chan[x]] = moved[x][t];
    }
    __syncthreads();
    if (warp < 2) {
        float* v = warp == 0 ? sq : sk;
        float4 x = *reinterpret_cast<const float4*>(v + 4 * lane);
        const float f = rsqrtf(warp_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w) + 1e-6f) * (warp == 0 ? rsqrtf((float)d) : 1.f);
        *reinterpret_cast<float4*>(v + 4 * lane) = make_float4(x.x * f, x.y * f, x.z * f, x.w * f);
    }
    __syncthreads();
    const float beta = p.beta[h];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < IT; it++) {
        const int col = 32 * it + 4 * warp + (lane >> 3);
        if (32 * it >= dv) break;
        float r = 0.f, o = 0.f;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const float4 g = *reinterpret_cast<const float4*>(sg + 32 * i + 4 * j), k = *reinterpret_cast<const float4*>(sk + 32 * i + 4 * j);
            float4& s = S[it][i];
            s = make_float4(fmaf(s.x, g.x, s.x), fmaf(s.y, g.y, s.y), fmaf(s.z, g.z, s.z), fmaf(s.w, g.w, s.w));
            r = fmaf(k.x, s.x, fmaf(k.y, s.y, fmaf(k.z, s.z, fmaf(k.w, s.w, r))));
        }
#pragma unroll
        for (int x = 1; x < 8; x <<= 1) r += __shfl_xor_sync(0xffffffffu, r, x);
        const float u = beta * (sv[min(col, MAX - 1)] - r);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const float4 q = *reinterpret_cast<const float4*>(sq + 32 * i + 4 * j), k = *reinterpret_cast<const float4*>(sk + 32 * i + 4 * j);
            float4& s = S[it][i];
            s = make_float4(fmaf(k.x, u, s.x), fmaf(k.y, u, s.y), fmaf(k.z, u, s.z), fmaf(k.w, u, s.w));
            o = fmaf(q.x, s.x, fmaf(q.y, s.y, fmaf(q.z, s.z, fmaf(q.w, s.w, o))));
            const int row = 32 * i + 4 * j;
            if (col < dv && row < d) *reinterpret_cast<float4*>(sbase + (size_t)col * d + row) = s;
        }
#pragma unroll
        for (int x = 1; x < 8; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
        if (j == 0 && col < dv) {
            so[col] = o;
            ss = fmaf(o, o, ss);
        }
    }
    const float rstd = rsqrtf(block_sum(ss, red) / (float)dv + p.eps);
    for (int c = tid; c < dv; c += kThreads)
        static_cast<T*>(p.out)[(size_t)h * dv + c] = from_f32<T>(so[c] * rstd * p.norm[c] * to_f32<T>(static_cast<const T*>(p.gate)[(size_t)h * dv + c]));
}

// Single tokens that step_kernel takes.
bool single_step(const b200_hybrid_layer& l, const b200_hybrid_pass& p) {
    return !p.tree && p.M == 1 && l.dim % 4 == 0 && l.vdim % 4 == 0 && l.dim <= 128 && l.vdim <= 128 && l.heads / l.kv_heads <= 8;
}

template <typename T>
int delta_step(const b200_hybrid_model& m, const b200_hybrid_layer& l, const ScanParams& s, const float* w, cudaStream_t st) {
    StepParams p{};
    p.in = s.in; p.conv_state = s.conv_state; p.w = w; p.g = s.g; p.beta = s.beta; p.state = s.state; p.norm = l.head_norm; p.gate = m.gb;
    p.out = m.ab; p.H = s.H; p.G = s.G; p.d = s.d; p.dv = s.dv; p.taps = s.taps; p.pitch = s.pitch; p.channels = s.channels; p.eps = m.eps;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(p.H);
    cfg.blockDim = dim3(kThreads);
    cfg.stream = st;
    cudaLaunchAttribute attrs[2];
    int na = 0;
    if (p.H > p.G) {
        attrs[na].id = cudaLaunchAttributeClusterDimension;
        attrs[na].val.clusterDim.x = p.H / p.G;
        attrs[na].val.clusterDim.y = attrs[na].val.clusterDim.z = 1;
        na++;
    }
    if (g_use_pdl) {
        attrs[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attrs[na].val.programmaticStreamSerializationAllowed = 1;
        na++;
    }
    cfg.attrs = attrs;
    cfg.numAttrs = na;
    cudaLaunchKernelEx(&cfg, step_kernel<T>, p);
    return check_launch();
}

// Prompts of heads the chunk kernels take.
bool chunked(const b200_hybrid_layer& l, const b200_hybrid_pass& p) {
    return !p.tree && p.M > 2 * kChunk && l.dim % 4 == 0 && l.vdim % 4 == 0 && l.dim <= 128 && l.vdim <= 128 && l.conv_taps <= 4;
}

template <typename T, int RPL>
int launch_chunk_scan(const ChunkScanParams& p, cudaStream_t st) {
    constexpr int D = 16 * RPL;
    const size_t smem = 2 * (size_t)(3 * kChunk * D + D + 2 * kChunk * kChunk + kChunk + kChunk * 32) * 4;
    launch_kernel(chunk_scan_kernel<T, RPL>, dim3((p.s.dv + 31) / 32, p.s.H), dim3(kThreads), smem, st, p);
    return check_launch();
}

template <typename T>
int delta_chunks(const b200_hybrid_model& m, const b200_hybrid_layer& l, const ConvParams& c, const ScanParams& s, cudaStream_t st) {
    ChunkParams p{};
    const size_t nd = (size_t)m.max_rows * l.heads * l.dim, chunks = (m.max_rows + kChunk - 1) / kChunk;
    p.c = c; p.g = s.g; p.kt = m.chunk; p.qt = m.chunk + nd; p.kh = m.chunk + 2 * nd; p.decay = m.chunk + 3 * nd;
    p.coef = p.decay + chunks * l.heads * l.dim;
    const dim3 grid((l.kv_heads + l.heads + 3) / 4, (c.M + kChunk - 1) / kChunk);
    if (l.conv_taps == 1) launch_kernel(conv_chunk_kernel<T, 1>, grid, dim3(128), 0, st, p);
    else if (l.conv_taps == 2) launch_kernel(conv_chunk_kernel<T, 2>, grid, dim3(128), 0, st, p);
    else if (l.conv_taps == 3) launch_kernel(conv_chunk_kernel<T, 3>, grid, dim3(128), 0, st, p);
    else launch_kernel(conv_chunk_kernel<T, 4>, grid, dim3(128), 0, st, p);
    if (check_launch() != B200_OK) return B200_ECUDA;
    const ChunkScanParams q{s, p.kt, p.qt, p.kh, p.decay, p.coef};
    return l.dim <= 64 ? launch_chunk_scan<T, 4>(q, st) : launch_chunk_scan<T, 8>(q, st);
}

template <typename T>
int delta(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& ps, cudaStream_t st) {
    char* pend = static_cast<char*>(m.pending);
    char* cache = static_cast<char*>(ps.cache);
    const size_t off = ps.write_off;
    const int nk = l.kv_heads * l.dim, nv = l.heads * l.vdim;
    ConvParams c{};
    c.in = ps.tree ? pend + r.pend_c : static_cast<char*>(m.cb);
    c.state = cache + r.mix_off; c.w = l.mix_conv; c.mask = ps.mask; c.q = m.q32;
    c.k = ps.tree ? reinterpret_cast<float*>(pend + r.pend_k) + off * nk : m.k32;
    c.v = ps.tree ? static_cast<void*>(reinterpret_cast<T*>(pend + r.pend_v) + off * nv) : m.vb;
    c.M = ps.M; c.G = l.kv_heads; c.H = l.heads; c.d = l.dim; c.dv = l.vdim; c.taps = l.conv_taps; c.pitch = delta_pitch(l);
    c.channels = delta_channels(l); c.write_off = ps.write_off;
    ScanParams s{};
    s.q = m.q32; s.state = reinterpret_cast<float*>(cache + r.state_off); s.o = m.o32; s.in = c.in; s.conv_state = cache + r.mix_off;
    s.k = ps.tree ? reinterpret_cast<const float*>(pend + r.pend_k) : m.k32;
    s.g = ps.tree ? reinterpret_cast<const float*>(pend + r.pend_g) : m.gf;
    s.beta = ps.tree ? reinterpret_cast<const float*>(pend + r.pend_b) : m.beta;
    s.v = ps.tree ? static_cast<const void*>(pend + r.pend_v) : m.vb;
    s.mask = ps.mask; s.M = ps.M; s.H = l.heads; s.G = l.kv_heads; s.d = l.dim; s.dv = l.vdim; s.taps = l.conv_taps; s.pitch = c.pitch;
    s.channels = c.channels;
    if (single_step(l, ps)) return delta_step<T>(m, l, s, l.mix_conv, st);
    int rc;
    if (chunked(l, ps)) {
        rc = delta_chunks<T>(m, l, c, s, st);
    } else {
        const int most = l.dim > l.vdim ? l.dim : l.vdim;
        if (l.dim % 4 || l.vdim % 4) launch_conv_v<T, 1, 8>(c, ps.tree, st);
        else if (most <= 128) launch_conv_v<T, 4, 1>(c, ps.tree, st);
        else launch_conv_v<T, 4, 2>(c, ps.tree, st);
        if (check_launch() != B200_OK) return B200_ECUDA;
        rc = ps.tree ? launch_scan<T, kTree>(s, ps.M, st) : launch_scan<T, kChain>(s, 1, st);
    }
    return rc != B200_OK ? rc : launch_head_norm(m, l, ps.M, m.gb, st);
}

template <typename T>
int delta_commit(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, char* cache, const int* count, const int* rows,
                 int tree_rows, cudaStream_t st) {
    char* pend = static_cast<char*>(m.pending);
    ScanParams s{};
    s.state = reinterpret_cast<float*>(cache + r.state_off); s.in = pend + r.pend_c; s.conv_state = cache + r.mix_off;
    s.k = reinterpret_cast<const float*>(pend + r.pend_k);
    s.g = reinterpret_cast<const float*>(pend + r.pend_g);
    s.beta = reinterpret_cast<const float*>(pend + r.pend_b);
    s.v = pend + r.pend_v;
    s.count = count; s.rows = rows; s.tree_rows = tree_rows;
    s.H = l.heads; s.G = l.kv_heads; s.d = l.dim; s.dv = l.vdim; s.taps = l.conv_taps; s.pitch = delta_pitch(l); s.channels = delta_channels(l);
    return launch_scan<T, kCommit>(s, 1, st);
}

}  // namespace

int launch_delta(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p, cudaStream_t st) {
    if (l.dim > kMaxDim || l.vdim > kMaxDim) return B200_ELIMIT;
    return m.act_type == B200_ACT_F32 ? delta<float>(m, l, r, p, st) : delta<bf16>(m, l, r, p, st);
}

int launch_delta_commit(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, void* cache, const int* count,
                        const int* rows, int tree_rows, cudaStream_t st) {
    if (l.dim > kMaxDim || l.vdim > kMaxDim) return B200_ELIMIT;
    char* c = static_cast<char*>(cache);
    return m.act_type == B200_ACT_F32 ? delta_commit<float>(m, l, r, c, count, rows, tree_rows, st) : delta_commit<bf16>(m, l, r, c, count, rows, tree_rows, st);
}

}  // namespace hybrid
}  // namespace b200

extern "C" size_t b200_hybrid_chunk_floats(int max_rows, int heads, int dim) {
    if (max_rows < 1 || heads < 1 || dim < 1) return 0;
    const size_t nd = (size_t)heads * dim, chunks = ((size_t)max_rows + 7) / 8;
    return 3 * nd * max_rows + chunks * (nd + (size_t)heads * 128);
}
