// Gated linear recurrence of the hybrid decoders (the forget gate also decides what is written):
//     S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T   computed as   S += (1 - f) (v - S),      o_t = S_t^T q_t,
// all in fp32, the state [heads][dim][vdim] carried in the request's cache.
//
//   scan_kernel    chain passes, any number of rows: CTA = (head, 32 state columns), warp = 4 columns, lane = a slice of
//                  the state's rows; the slice lives in registers (packed pairs of rows), tokens come in blocks through
//                  shared memory, the lanes' parts of the outputs are added for 8 tokens at once.  The new state is
//                  written back.
//   tree_kernel    tree passes: nothing may change the state yet.  Row m's output is written out along its path:
//                  o = S_0^T (q prod f) + sum over the path's rows a of (q . (1 - f_a) prod of the later f) v_a.
//   commit_kernel  advances convolution inputs, states and K/V rows over accepted rows, for every layer run at once.
//   head_norm      per-head RMS norm of the outputs with the head weight (times a gate), to the activation type.
#include "scan.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kWarps = 8;
constexpr int kLaneCols = 4;         // state columns of a warp of the scan
constexpr int kMaxDim = 256;

constexpr unsigned long long kMinusOne2 = 0xbf800000bf800000ull;

// Sum of v[i] over the warp's lanes, for 32 values at once: lane i gets the total of v[i].
__device__ __forceinline__ float transpose_sum(float (&v)[32], int lane) {
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

// RPL neighbouring values of a shared-memory row as packed pairs.
template <int RPL> __device__ __forceinline__ void ld_pairs(unsigned long long (&r)[RPL / 2], const float* p) {
#pragma unroll
    for (int i = 0; i < RPL / 2; i++) r[i] = *reinterpret_cast<const unsigned long long*>(p + 2 * i);
}
template <int RPL> __device__ __forceinline__ void ld_pairs(unsigned long long (&r)[RPL / 2], const bf16* p) {
#pragma unroll
    for (int i = 0; i < RPL / 2; i++) {
        const uint32_t u = *reinterpret_cast<const uint32_t*>(p + 2 * i);
        r[i] = pack2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
    }
}

template <typename T, int RPL>           // state rows of a lane
__global__ void __launch_bounds__(kWarps * 32) scan_kernel(const T* q, const float* gf, const T* v, float* state, float* o, int M, int H,
                                                           int d, int dv) {
    pdl_launch_dependents();
    constexpr int D = 32 * RPL, TB = RPL == 8 ? 8 : 16, STAGES = 2;
    __shared__ __align__(16) float sg[STAGES][TB][D];
    __shared__ __align__(16) T sq[STAGES][TB][D];
    __shared__ __align__(16) T sv[STAGES][TB][32];
    const int h = blockIdx.y, c0 = blockIdx.x * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int col = c0 + warp * kLaneCols, ncol = min(32, dv - c0);
    const bool wide_g = d % 4 == 0, wide_q = d * (int)sizeof(T) % 16 == 0, wide_v = dv * (int)sizeof(T) % 16 == 0;
    // what the copies never write stays zero: rows past the head's width, columns past its values
    for (int i = tid; i < STAGES * TB; i += kWarps * 32) {
        for (int c = d; c < D; c++) { sg[i / TB][i % TB][c] = 0.f; sq[i / TB][i % TB][c] = from_f32<T>(0.f); }
        for (int c = ncol; c < 32; c++) sv[i / TB][i % TB][c] = from_f32<T>(0.f);
    }
    pdl_wait();
    auto fetch = [&](int b) {
        const int st = b % STAGES, t0 = b * TB;
        for (int t = warp; t < TB && t0 + t < M; t += kWarps) {
            const size_t row = (size_t)(t0 + t) * H + h;
            fetch_row(sg[st][t], gf + row * d, d, wide_g, lane);
            fetch_row(sq[st][t], q + row * d, d, wide_q, lane);
            fetch_row(sv[st][t], v + row * dv + c0, ncol, wide_v, lane);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    fetch(0);
    unsigned long long S[RPL / 2][kLaneCols];            // two neighbouring state rows each
    float* sbase = state + ((size_t)h * d + lane * RPL) * dv + col;
    const bool wide_s = dv % 4 == 0 && col < dv;
    float row[RPL][kLaneCols];
#pragma unroll
    for (int r = 0; r < RPL; r++) {
        const bool in = lane * RPL + r < d;
        if (wide_s) {
            const float4 x = in ? *reinterpret_cast<const float4*>(sbase + (size_t)r * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
            row[r][0] = x.x; row[r][1] = x.y; row[r][2] = x.z; row[r][3] = x.w;
        } else {
#pragma unroll
            for (int c = 0; c < kLaneCols; c++) row[r][c] = in && col + c < dv ? sbase[(size_t)r * dv + c] : 0.f;
        }
    }
#pragma unroll
    for (int r = 0; r < RPL; r += 2)
#pragma unroll
        for (int c = 0; c < kLaneCols; c++) S[r / 2][c] = pack2(row[r][c], row[r + 1][c]);
    const int nb = (M + TB - 1) / TB;
    for (int b = 0; b < nb; b++) {
        const int st = b % STAGES, t0 = b * TB;
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                                 // this block is here, the one before has been read
        if (b + 1 < nb) fetch(b + 1);
#pragma unroll 1
        for (int tg = 0; tg < TB && t0 + tg < M; tg += 8) {
            const int nt = min(8, M - t0 - tg);
            float y[32];                                 // [token][column], this lane's rows
#pragma unroll
            for (int t = 0; t < 8; t++) {
                if (t < nt) {
                    unsigned long long g2[RPL / 2], q2[RPL / 2], acc[kLaneCols], v2[kLaneCols];
                    ld_pairs<RPL>(g2, &sg[st][tg + t][lane * RPL]);
                    ld_pairs<RPL>(q2, &sq[st][tg + t][lane * RPL]);
#pragma unroll
                    for (int c = 0; c < kLaneCols; c++) {
                        const float x = to_f32<T>(sv[st][tg + t][warp * kLaneCols + c]);
                        v2[c] = pack2(x, x);
                        acc[c] = 0ull;
                    }
#pragma unroll
                    for (int r = 0; r < RPL / 2; r++) {
#pragma unroll
                        for (int c = 0; c < kLaneCols; c++) {
                            S[r][c] = fma2(g2[r], fma2(S[r][c], kMinusOne2, v2[c]), S[r][c]);
                            acc[c] = fma2(q2[r], S[r][c], acc[c]);
                        }
                    }
#pragma unroll
                    for (int c = 0; c < kLaneCols; c++) {
                        const float2 x = unpack2(acc[c]);
                        y[t * kLaneCols + c] = x.x + x.y;
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < kLaneCols; c++) y[t * kLaneCols + c] = 0.f;
                }
            }
            const float out = transpose_sum(y, lane);
            const int t = lane / kLaneCols, c = col + lane % kLaneCols;
            if (t < nt && c < dv) o[((size_t)(t0 + tg + t) * H + h) * dv + c] = out;
        }
    }
#pragma unroll
    for (int r = 0; r < RPL; r++) {
        if (lane * RPL + r >= d) break;
        float x[kLaneCols];
#pragma unroll
        for (int c = 0; c < kLaneCols; c++) {
            const float2 y = unpack2(S[r / 2][c]);
            x[c] = r & 1 ? y.y : y.x;
        }
        if (wide_s) {
            *reinterpret_cast<float4*>(sbase + (size_t)r * dv) = make_float4(x[0], x[1], x[2], x[3]);
        } else {
#pragma unroll
            for (int c = 0; c < kLaneCols; c++)
                if (col + c < dv) sbase[(size_t)r * dv + c] = x[c];
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(128) tree_kernel(const T* q, const float* pend_g, const T* pend_v,
                                                   const float* state, const unsigned long long* mask,
                                                   float* o, int H, int d, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float sw[B200_HYBRID_PENDING][4];
    __shared__ float sqs[kMaxDim];
    const int h = blockIdx.x, m = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const unsigned long long path = mask[m];             // the row itself and its ancestors among the tail rows
    float qi[2], suf[2];
#pragma unroll
    for (int k = 0; k < 2; k++) {
        const int i = tid + 128 * k;
        qi[k] = i < d ? to_f32<T>(q[((size_t)m * H + h) * d + i]) : 0.f;
        suf[k] = 1.f;
    }
    for (unsigned long long left = path; left != 0ull;) {   // newest row first
        const int a = 63 - __clzll((long long)left);
        left &= ~(1ull << a);
        float c = 0.f;
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int i = tid + 128 * k;
            if (i < d) {
                const float g = pend_g[((size_t)a * H + h) * d + i];
                c = fmaf(qi[k] * suf[k], g, c);
                suf[k] *= 1.f - g;
            }
        }
        c = warp_sum(c);
        if (lane == 0) sw[a][warp] = c;
    }
#pragma unroll
    for (int k = 0; k < 2; k++)
        if (tid + 128 * k < d) sqs[tid + 128 * k] = qi[k] * suf[k];
    __syncthreads();
    for (int c = tid; c < dv; c += 128) {
        float acc = 0.f;
        const float* s = state + (size_t)h * d * dv + c;
#pragma unroll 8
        for (int i = 0; i < d; i++) acc = fmaf(sqs[i], s[(size_t)i * dv], acc);
        for (unsigned long long left = path; left != 0ull; left &= left - 1ull) {
            const int a = __ffsll((long long)left) - 1;
            acc = fmaf(sw[a][0] + sw[a][1] + sw[a][2] + sw[a][3], to_f32<T>(pend_v[((size_t)a * H + h) * dv + c]), acc);
        }
        o[((size_t)m * H + h) * dv + c] = acc;
    }
}

template <typename T>
__global__ void __launch_bounds__(128) head_norm_kernel(const float* o, const float* w, const T* gate, T* out, int M, int H,
                                                        int dv, int pitch, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= M * H) return;
    const int m = unit / H, h = unit - m * H;
    const float* row = o + (size_t)unit * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) { const float x = row[c]; ss = fmaf(x, x, ss); }
    const float rstd = rsqrtf(warp_sum(ss) / (float)dv + eps);
    T* dst = out + (size_t)m * pitch + (size_t)h * dv;
    if (gate != nullptr) {
        const T* g = gate + (size_t)unit * dv;
        for (int c = lane; c < dv; c += 32) dst[c] = from_f32<T>(row[c] * rstd * w[c] * to_f32<T>(g[c]));
        return;
    }
    for (int c = lane; c < dv; c += 32) dst[c] = from_f32<T>(row[c] * rstd * w[c]);
}

struct CommitParams {
    const b200_hybrid_layer* layers;
    const b200_hybrid_run* runs;
    char* cache;
    char* pending;
    const int* count;
    const int* rows;
    const int* prefix;
    int width, cap, fixed_count, tree_rows, states, compact;
};

template <typename T>
__global__ void __launch_bounds__(256) commit_kernel(const CommitParams p) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ int srow[B200_HYBRID_PENDING];
    const b200_hybrid_run& r = p.runs[blockIdx.x];
    const b200_hybrid_layer& l = p.layers[r.layer];
    int n = p.fixed_count > 0 ? p.fixed_count : p.count[0] + 1;
    n = min(max(n, 0), B200_HYBRID_PENDING);
    for (int i = threadIdx.x; i < n; i += 256) {
        int s = (i == 0 || p.rows == nullptr || p.fixed_count > 0) ? i : p.rows[i];
        if (s < 0) s += p.tree_rows;
        srow[i] = min(max(s, 0), B200_HYBRID_PENDING - 1);
    }
    __syncthreads();
    const int first = blockIdx.y * 256 + threadIdx.x, step = gridDim.y * 256;
    const int prev = l.taps - 1;
    if (prev > 0) {
        float* state = reinterpret_cast<float*>(p.cache + r.conv_off);
        const float* pend = reinterpret_cast<const float*>(p.pending + r.pend_h);
        for (int c = first; c < p.width; c += step) {
            float nv[B200_HYBRID_MAX_TAPS];
#pragma unroll
            for (int j = 0; j < B200_HYBRID_MAX_TAPS; j++) {
                const int i = n - prev + j;
                nv[j] = 0.f;
                if (j < prev) nv[j] = i >= 0 ? pend[(size_t)srow[i] * p.width + c] : state[(size_t)(i + prev) * p.width + c];
            }
#pragma unroll
            for (int j = 0; j < B200_HYBRID_MAX_TAPS; j++)
                if (j < prev) state[(size_t)j * p.width + c] = nv[j];
        }
    }
    if (p.states && l.mixer == B200_MIXER_RECURRENCE) {
        float* state = reinterpret_cast<float*>(p.cache + r.state_off);
        const float* pg = reinterpret_cast<const float*>(p.pending + r.pend_g);
        const T* pv = reinterpret_cast<const T*>(p.pending + r.pend_v);
        const int per = l.dim * l.vdim, total = l.heads * per;
        for (int e = first; e < total; e += step) {
            const int h = e / per, x = e - h * per, i = x / l.vdim, c = x - i * l.vdim;
            float s = state[e];
            for (int t = 0; t < n; t++) {
                const float g = pg[((size_t)srow[t] * l.heads + h) * l.dim + i];
                const float v = to_f32<T>(pv[((size_t)srow[t] * l.heads + h) * l.vdim + c]);
                s = fmaf(g, v - s, s);
            }
            state[e] = s;
        }
    }
    if (p.compact && (l.mixer == B200_MIXER_ATTENTION || l.mixer == B200_MIXER_LATENT)) {
        const int P = p.prefix[0];
        const bool latent = l.mixer == B200_MIXER_LATENT;           // one row per token for all heads, no values of their own
        const int ke = latent ? latent_pitch(l) : l.maps * round_up(l.dim, 16), ve = latent ? 0 : round_up(l.vdim, 16), per = ke + ve;
        for (int e = first; e < (latent ? 1 : l.kv_heads) * per; e += step) {
            const int g = e / per, x = e - g * per;
            T* base = x < ke ? reinterpret_cast<T*>(p.cache + r.k_off) + (size_t)g * p.cap * ke + x
                             : reinterpret_cast<T*>(p.cache + r.v_off) + (size_t)g * p.cap * ve + (x - ke);
            const int pitch = x < ke ? ke : ve;
            // rows ascend along a path, so no source is overwritten before it is read
            for (int i = 1; i < n; i++)
                if (srow[i] != i && P + srow[i] < p.cap) base[(size_t)(P + i) * pitch] = base[(size_t)(P + srow[i]) * pitch];
        }
    }
}

template <typename T>
int launch_scan(const b200_hybrid_model& m, const b200_hybrid_layer& l, float* state, int M, cudaStream_t st) {
    const dim3 grid((l.vdim + 31) / 32, l.heads), block(kWarps * 32);
    const T* q = static_cast<const T*>(m.qb);
    const T* v = static_cast<const T*>(m.vb);
    const float* gf = m.gf;
    if (l.dim <= 64) launch_kernel(scan_kernel<T, 2>, grid, block, 0, st, q, gf, v, state, m.o32, M, l.heads, l.dim, l.vdim);
    else if (l.dim <= 128) launch_kernel(scan_kernel<T, 4>, grid, block, 0, st, q, gf, v, state, m.o32, M, l.heads, l.dim, l.vdim);
    else launch_kernel(scan_kernel<T, 8>, grid, block, 0, st, q, gf, v, state, m.o32, M, l.heads, l.dim, l.vdim);
    return check_launch();
}

template <typename T>
int recurrence(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p, cudaStream_t st) {
    float* state = reinterpret_cast<float*>(static_cast<char*>(p.cache) + r.state_off);
    int rc;
    if (p.tree) {
        launch_kernel(tree_kernel<T>, dim3(l.heads, p.M), dim3(128), 0, st, static_cast<const T*>(m.qb),
                      reinterpret_cast<const float*>(static_cast<const char*>(m.pending) + r.pend_g),
                      reinterpret_cast<const T*>(static_cast<const char*>(m.pending) + r.pend_v), static_cast<const float*>(state), p.mask,
                      m.o32, l.heads, l.dim, l.vdim);
        rc = check_launch();
    } else {
        rc = launch_scan<T>(m, l, state, p.M, st);
    }
    return rc != B200_OK ? rc : launch_head_norm(m, l, p.M, nullptr, st);
}

template <typename T>
void launch_head_norm_t(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, const void* gate, cudaStream_t st) {
    launch_kernel(head_norm_kernel<T>, dim3((rows * l.heads + 3) / 4), dim3(128), 0, st, static_cast<const float*>(m.o32), l.head_norm,
                  static_cast<const T*>(gate), static_cast<T*>(m.ab), rows, l.heads, l.vdim, round_up(l.heads * l.vdim, 64), m.eps);
}

}  // namespace

int launch_head_norm(const b200_hybrid_model& m, const b200_hybrid_layer& l, int rows, const void* gate, cudaStream_t st) {
    if (m.act_type == B200_ACT_F32) launch_head_norm_t<float>(m, l, rows, gate, st);
    else launch_head_norm_t<bf16>(m, l, rows, gate, st);
    return check_launch();
}

int launch_recurrence(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p,
                      cudaStream_t st) {
    if (l.dim > kMaxDim) return B200_ELIMIT;
    return m.act_type == B200_ACT_F32 ? recurrence<float>(m, l, r, p, st) : recurrence<bf16>(m, l, r, p, st);
}

int launch_commit(const b200_hybrid_model& m, void* cache, int cache_rows, int fixed_count, const int* count, const int* rows, int tree_rows,
                  const int* prefix, int states, int compact, cudaStream_t st) {
    CommitParams p{};
    p.layers = m.dev_layers; p.runs = m.dev_runs; p.cache = static_cast<char*>(cache); p.pending = static_cast<char*>(m.pending);
    p.count = count; p.rows = rows; p.prefix = prefix; p.width = m.width; p.cap = cache_rows; p.fixed_count = fixed_count;
    p.tree_rows = tree_rows; p.states = states; p.compact = compact;
    const dim3 grid(m.n_runs, states ? 32 : 4);
    if (m.act_type == B200_ACT_F32) launch_kernel(commit_kernel<float>, grid, dim3(256), 0, st, p);
    else launch_kernel(commit_kernel<bf16>, grid, dim3(256), 0, st, p);
    return check_launch();
}

}  // namespace hybrid
}  // namespace b200
