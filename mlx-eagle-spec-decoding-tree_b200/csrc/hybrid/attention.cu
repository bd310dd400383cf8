// Softmax attention of the hybrid decoders: one or two maps per head over the same values (two: differential
// attention, a1 - lambda a2, normed per head and scaled), a sliding window with kept first keys, an output gate,
// tree-masked tail rows.  Scores, weights and statistics are fp32.
//
// attention_rows: any activation type, few query rows (decoding, tree passes, fp32 prompts).  CTA = (key split, kv
// head and group of its query heads, query row).  Only visible keys are walked: the kept first keys, then the window's
// committed keys, then the tail rows.  Keys come in blocks of 64 through shared memory (read once for all query vectors
// of the group); partial (max, sum, output) per split go to a workspace, attention_merge adds them in split order and
// applies the head's ending (difference, norm, gate).
//
// attention_prompt: bf16, many query rows of one sequence.  CTA = (64 query rows, head), four warps of 16 rows,
// mma.sync with the key/value blocks double-buffered by cp.async; both maps share the value block.  The softmax weights
// enter the value product as a pair of bf16 terms (value + remainder), which keeps them at fp32-like precision.
//
// Latent attention (one low-rank latent and one rotated key part per token, shared by all heads) uses both: fp32 rows walk the
// latent itself, with queries brought into its space and the key row's first columns as values (SHARED; bf16: latent.cu);
// prompts walk keys and values written out per head, the rotated part taken from the cache (LATENT).
#include "mma.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kKeys = 64;                // keys of a block
constexpr int kMaxSplits = 32;
constexpr int kRowThreads = 128;

struct AttnParams {
    const void* q;            // [M][q_pitch]: (head, map) vectors of dp elements
    const void* kc;           // [G][cap][maps * dp]; LATENT: [H][cap][dp - rp]
    const void* vc;           // [G][cap][vp]
    const void* gate;         // [M][H * vdim], or null
    const void* krot;         // LATENT: [..][krot_pitch] rotated key parts of rp columns
    void* out;                // [M][out_pitch], heads out_head apart
    float* part;              // [M][H * maps][splits][vp + 2]
    const int* pos;
    const int* tail_pos;
    const unsigned long long* mask;
    const int* prefix;
    int M, H, G, maps, dim, dp, vdim, vp, cap, window, keep, tree, tail, q_pitch, out_pitch, out_head, rp, krot_pitch;
    int splits, qgroups, hpg; // key splits; query-head groups of a kv head and heads in each
    float scale_log2, lambda, out_scale, eps;
};

// The visible committed keys of a query row as one index range: kept first keys, then the window.
struct KeyWalk {
    int ns, wstart, nc, prefix, pos, total;
    __device__ __forceinline__ void init(const AttnParams& p, int m) {
        pos = p.pos[m];
        prefix = p.tree ? p.prefix[0] : pos + 1;
        const int w0 = max(0, pos - p.window + 1);
        wstart = min(w0, prefix);
        ns = min(p.keep, wstart);
        nc = ns + prefix - wstart;
        total = nc + (p.tree ? p.tail : 0);
    }
    __device__ __forceinline__ int blocks() const { return (total + kKeys - 1) / kKeys; }
    __device__ __forceinline__ int per_split(const AttnParams& p) const { return (blocks() + p.splits - 1) / p.splits; }
    __device__ __forceinline__ int row(int u) const { return u < ns ? u : (u < nc ? wstart + u - ns : prefix + u - nc); }
};

template <typename T, int QN, int CR, bool SHARED>    // query vectors (at most), columns per thread, values are the keys' first columns
__global__ void __launch_bounds__(kRowThreads) attention_rows_kernel(const AttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    constexpr int VE = 16 / (int)sizeof(T), SP = kKeys + 4;              // elements of 16 bytes, pitch of a score row
    const int KE = p.maps * p.dp, KP = KE + VE;                          // padded key row
    float* sq = reinterpret_cast<float*>(smem_raw);                      // [QN][dp]
    float* sc = sq + QN * p.dp;                                          // [QN][SP]
    float* sm = sc + QN * SP;                                            // [QN] running max
    float* sl = sm + QN;                                                 // [QN] running sum
    float* sr = sl + QN;                                                 // [2 QN] rescale factor of this block
    int* srow = reinterpret_cast<int*>(sr + 2 * QN);                     // [kKeys] cache row of the block's keys, -1: not visible
    T* sk = reinterpret_cast<T*>(srow + kKeys);                          // [kKeys][KP]
    T* sv = SHARED ? sk : sk + kKeys * KP;                               // [kKeys][VP]
    const int vload = SHARED ? 0 : p.vp, VP = SHARED ? KP : p.vp;
    const int split = blockIdx.x, g = blockIdx.y / p.qgroups, qg = blockIdx.y % p.qgroups, m = blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int R = p.H / p.G;
    const int h0 = g * R + qg * p.hpg;
    const int nh = min(p.hpg, R - qg * p.hpg), nq = nh * p.maps;
    KeyWalk kw;
    kw.init(p, m);
    const int nb = kw.blocks(), per = kw.per_split(p), b0 = split * per, b1 = min(nb, b0 + per);
    if (b0 >= b1) return;                                                // the merge knows which splits hold something

    const T* qrow = static_cast<const T*>(p.q) + (size_t)m * p.q_pitch + (size_t)h0 * p.maps * p.dp;
    for (int i = tid; i < QN * p.dp; i += kRowThreads) sq[i] = i < nq * p.dp ? to_f32<T>(qrow[i]) * p.scale_log2 : 0.f;
    for (int i = tid; i < QN; i += kRowThreads) { sm[i] = -INFINITY; sl[i] = 0.f; }
    float acc[QN][CR];
#pragma unroll
    for (int i = 0; i < QN; i++)
#pragma unroll
        for (int c = 0; c < CR; c++) acc[i][c] = 0.f;
    const T* kbase = static_cast<const T*>(p.kc) + (size_t)g * p.cap * KE;
    const T* vbase = static_cast<const T*>(p.vc) + (size_t)g * p.cap * p.vp;
    const unsigned long long mk = p.tree ? p.mask[m] : 0ull;

    for (int b = b0; b < b1; b++) {
        __syncthreads();
        if (tid < kKeys) {
            const int u = b * kKeys + tid;
            int r = -1;
            if (u < kw.total) {
                r = kw.row(u);
                if (u >= kw.nc) {
                    const int j = u - kw.nc, tp = p.tail_pos[j];
                    if (!((mk >> j) & 1ull) || !(kw.pos - tp < p.window || tp < p.keep)) r = -1;
                }
                if (r >= p.cap) r = -1;
            }
            srow[tid] = r;
        }
        __syncthreads();
        for (int k = warp; k < kKeys; k += kRowThreads / 32) {           // a warp per key row, 16 bytes per lane
            const int r = srow[k];
            for (int c = lane; c * VE < KE + vload; c += 32) {
                const bool key = c * VE < KE;
                T* dst = key ? sk + k * KP + c * VE : sv + k * VP + (c * VE - KE);
                const T* src = key ? kbase + (size_t)r * KE + c * VE : vbase + (size_t)r * p.vp + (c * VE - KE);
                if (r >= 0) cp_async16(smem_u32(dst), src);
                else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
            }
        }
        asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();
        {
            const int k = tid & (kKeys - 1);
            const bool vis = srow[k] >= 0;
            for (int qi = tid / kKeys; qi < nq; qi += kRowThreads / kKeys) {
                const T* kr = sk + k * KP + (p.maps == 2 ? (qi & 1) * p.dp : 0);
                const float* qv = sq + qi * p.dp;
                float s0 = 0.f, s1 = 0.f;
#pragma unroll 4
                for (int c = 0; c < p.dp; c += VE) {
                    const uint4 raw = *reinterpret_cast<const uint4*>(kr + c);
                    const T* kv = reinterpret_cast<const T*>(&raw);
#pragma unroll
                    for (int e = 0; e < VE; e += 4) {
                        const float4 q4 = *reinterpret_cast<const float4*>(qv + c + e);
                        s0 = fmaf(q4.x, to_f32<T>(kv[e]), s0);
                        s1 = fmaf(q4.y, to_f32<T>(kv[e + 1]), s1);
                        s0 = fmaf(q4.z, to_f32<T>(kv[e + 2]), s0);
                        s1 = fmaf(q4.w, to_f32<T>(kv[e + 3]), s1);
                    }
                }
                sc[qi * SP + k] = vis ? s0 + s1 : -INFINITY;
            }
        }
        __syncthreads();
        for (int qi = warp; qi < nq; qi += kRowThreads / 32) {
            const float a0 = sc[qi * SP + lane], a1 = sc[qi * SP + lane + 32];
            const float mo = sm[qi], mn = fmaxf(mo, warp_max(fmaxf(a0, a1)));
            const float base = mn == -INFINITY ? 0.f : mn;
            const float p0 = exp2f(a0 - base), p1 = exp2f(a1 - base);
            sc[qi * SP + lane] = p0;
            sc[qi * SP + lane + 32] = p1;
            const float ls = warp_sum(p0 + p1);
            __syncwarp();
            if (lane == 0) {
                const float f = mo == -INFINITY ? 0.f : exp2f(mo - base);
                sr[qi] = f;
                sl[qi] = sl[qi] * f + ls;
                sm[qi] = mn;
            }
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < CR; c++) {
            const int col = tid + c * kRowThreads;
            if (col < p.vdim) {
#pragma unroll
                for (int i = 0; i < QN; i++)
                    if (i < nq) acc[i][c] *= sr[i];
#pragma unroll 2
                for (int k = 0; k < kKeys; k += 4) {                     // rows that are not visible: weight 0, value 0
                    float v[4];
#pragma unroll
                    for (int e = 0; e < 4; e++) v[e] = to_f32<T>(sv[(k + e) * VP + col]);
#pragma unroll
                    for (int i = 0; i < QN; i++)
                        if (i < nq) {
                            const float4 w = *reinterpret_cast<const float4*>(sc + i * SP + k);
                            acc[i][c] = fmaf(w.x, v[0], fmaf(w.y, v[1], fmaf(w.z, v[2], fmaf(w.w, v[3], acc[i][c]))));
                        }
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < QN; i++) {
        if (i < nq) {
            float* dst = p.part + (((size_t)m * p.H * p.maps + (size_t)h0 * p.maps + i) * p.splits + split) * (p.vp + 2);
            if (tid == 0) { dst[0] = sm[i]; dst[1] = sl[i]; }
#pragma unroll
            for (int c = 0; c < CR; c++) {
                const int col = tid + c * kRowThreads;
                if (col < p.vdim) dst[2 + col] = acc[i][c];
            }
        }
    }
}

// Adds the key splits of one (row, head) and finishes the head.
template <typename T, int CR>
__global__ void __launch_bounds__(kRowThreads) attention_merge_kernel(const AttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[33];
    __shared__ float sw[2 * kMaxSplits];
    const int h = blockIdx.x, m = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    KeyWalk kw;
    kw.init(p, m);
    const int per = kw.per_split(p), ns = (kw.blocks() + per - 1) / per;          // splits that hold something
    const size_t stride = p.vp + 2;
    const float* base = p.part + ((size_t)m * p.H + h) * p.maps * p.splits * stride;
    if (warp < p.maps) {
        const float* b = base + (size_t)warp * p.splits * stride;
        const float mm = lane < ns ? b[lane * stride] : -INFINITY;
        const float ll = lane < ns ? b[lane * stride + 1] : 0.f;
        const float mx = warp_max(mm);
        const float f = mm == -INFINITY ? 0.f : exp2f(mm - mx);
        const float tot = warp_sum(f * ll);
        sw[warp * kMaxSplits + lane] = tot > 0.f ? f / tot : 0.f;
    }
    __syncthreads();
    float ss = 0.f;
    float o[CR];
#pragma unroll
    for (int c = 0; c < CR; c++) {
        const int col = tid + c * kRowThreads;
        o[c] = 0.f;
        if (col < p.vdim) {
            float a[2] = {0.f, 0.f};
            for (int mp = 0; mp < p.maps; mp++) {
                const float* src = base + (size_t)mp * p.splits * stride + 2 + col;
                float x = 0.f;
#pragma unroll 8
                for (int s = 0; s < ns; s++) x = fmaf(sw[mp * kMaxSplits + s], src[s * stride], x);
                a[mp] = x;
            }
            o[c] = p.maps == 2 ? a[0] - p.lambda * a[1] : a[0];
            ss = fmaf(o[c], o[c], ss);
        }
    }
    float f = 1.f;
    if (p.maps == 2) f = rsqrtf(block_sum(ss, red) / (float)p.vdim + p.eps) * p.out_scale;
#pragma unroll
    for (int c = 0; c < CR; c++) {
        const int col = tid + c * kRowThreads;
        if (col < p.vdim) {
            const float gt = p.gate != nullptr ? to_f32<T>(static_cast<const T*>(p.gate)[((size_t)m * p.H + h) * p.vdim + col]) : 1.f;
            static_cast<T*>(p.out)[(size_t)m * p.out_pitch + (size_t)h * p.out_head + col] = from_f32<T>(o[c] * f * gt);
        }
    }
}

// ---------------------------------------------------------------- prompts
constexpr int kQRows = 64;

template <int VT, int MAPS, bool LATENT> // 16-column value tiles, maps per head
__global__ void __launch_bounds__(128) attention_prompt_kernel(const AttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int KE = MAPS * p.dp, KP = KE + 8;
    constexpr int VP = VT * 16 + 8;
    bf16* sq = reinterpret_cast<bf16*>(smem_raw);                        // [64][KP]
    bf16* sk = sq + kQRows * KP;                                         // [2][64][KP]
    bf16* sv = sk + 2 * kKeys * KP;                                      // [2][64][VP]
    const int h = blockIdx.x, r0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * kQRows, g = h / (p.H / p.G);   // longest rows first
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t = lane & 3;
    const int base_pos = p.prefix[0], qpos0 = base_pos + r0, qlast = base_pos + min(p.M, r0 + kQRows) - 1;
    const int kown = LATENT ? KE - p.rp : KE;                            // key columns of the head's own
    const bf16* kbase = static_cast<const bf16*>(p.kc) + (size_t)g * p.cap * kown;
    const bf16* vbase = static_cast<const bf16*>(p.vc) + (size_t)g * p.cap * p.vp;

    const int kv = KE / 8, vv = p.vp / 8;
    for (int i = tid; i < kQRows * kv; i += 128) {
        const int r = i / kv, c = i - r * kv;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r0 + r < p.M) v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q) + (size_t)(r0 + r) * p.q_pitch + (size_t)h * KE + c * 8);
        *reinterpret_cast<uint4*>(sq + r * KP + c * 8) = v;
    }
    if (p.vp < VT * 16) {                // value columns past the head's width stay zero
        for (int i = tid; i < 2 * kKeys * (VT * 16 - p.vp); i += 128) {
            const int r = i / (VT * 16 - p.vp), c = i % (VT * 16 - p.vp);
            sv[r * VP + p.vp + c] = __float2bfloat16_rn(0.f);
        }
    }
    const int wb0 = max(0, qpos0 - p.window + 1) / kKeys;
    const int nsink = min((p.keep + kKeys - 1) / kKeys, wb0);
    const int nblk = nsink + qlast / kKeys - wb0 + 1;
    auto block_of = [&](int i) { return i < nsink ? i : wb0 + i - nsink; };
    auto load = [&](int i) {
        const int k0 = block_of(i) * kKeys, st = i & 1;
        for (int e = tid; e < kKeys * kv; e += 128) {
            const int r = e / kv, c = e - r * kv;
            bf16* dst = sk + (st * kKeys + r) * KP + c * 8;
            const bf16* src = kbase + (size_t)(k0 + r) * kown + c * 8;
            if (LATENT && c * 8 >= kown) src = static_cast<const bf16*>(p.krot) + (size_t)(k0 + r) * p.krot_pitch + (c * 8 - kown);
            if (k0 + r <= qlast) cp_async16(smem_u32(dst), src);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        for (int e = tid; e < kKeys * vv; e += 128) {
            const int r = e / vv, c = e - r * vv;
            bf16* dst = sv + (st * kKeys + r) * VP + c * 8;
            if (k0 + r <= qlast) cp_async16(smem_u32(dst), vbase + (size_t)(k0 + r) * p.vp + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };

    float o[MAPS][VT * 2][4];
    float mx[MAPS][2], ls[MAPS][2];
#pragma unroll
    for (int a = 0; a < MAPS; a++) {
        mx[a][0] = mx[a][1] = -INFINITY;
        ls[a][0] = ls[a][1] = 0.f;
#pragma unroll
        for (int n = 0; n < VT * 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[a][n][e] = 0.f;
    }
    const int qp0 = qpos0 + warp * 16 + gq, qp1 = qp0 + 8;
    load(0);
    for (int i = 0; i < nblk; i++) {
        if (i + 1 < nblk) {
            load(i + 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const int k0 = block_of(i) * kKeys;
        const bf16* kt = sk + (i & 1) * kKeys * KP;
        const bf16* vt = sv + (i & 1) * kKeys * VP;
#pragma unroll
        for (int a = 0; a < MAPS; a++) {
            float s[8][4];
#pragma unroll
            for (int n = 0; n < 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            const uint32_t qaddr = smem_u32(sq + (warp * 16 + (lane & 15)) * KP + a * p.dp + (lane >> 4) * 8);
            const uint32_t kaddr = smem_u32(kt + ((lane & 7) + ((lane >> 4) << 3)) * KP + a * p.dp + ((lane >> 3) & 1) * 8);
            for (int c = 0; c < p.dp; c += 16) {
                uint32_t qa[4];
                ldsm4(qa, qaddr + c * 2);
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    uint32_t kb[4];
                    ldsm4(kb, kaddr + (n * 8 * KP + c) * 2);
                    mma_bf16(s[n], qa, kb[0], kb[1]);
                    mma_bf16(s[n + 1], qa, kb[2], kb[3]);
                }
            }
            float m0 = mx[a][0], m1 = mx[a][1];
#pragma unroll
            for (int n = 0; n < 8; n++) {
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int j = k0 + n * 8 + 2 * t + e;
                    const bool v0 = j <= qp0 && (qp0 - j < p.window || j < p.keep);
                    const bool v1 = j <= qp1 && (qp1 - j < p.window || j < p.keep);
                    s[n][e] = v0 ? s[n][e] * p.scale_log2 : -INFINITY;
                    s[n][2 + e] = v1 ? s[n][2 + e] * p.scale_log2 : -INFINITY;
                    m0 = fmaxf(m0, s[n][e]);
                    m1 = fmaxf(m1, s[n][2 + e]);
                }
            }
            m0 = fmaxf(m0, __shfl_xor_sync(0xffffffffu, m0, 1));
            m0 = fmaxf(m0, __shfl_xor_sync(0xffffffffu, m0, 2));
            m1 = fmaxf(m1, __shfl_xor_sync(0xffffffffu, m1, 1));
            m1 = fmaxf(m1, __shfl_xor_sync(0xffffffffu, m1, 2));
            const float c0 = m0 == -INFINITY ? 0.f : m0, c1 = m1 == -INFINITY ? 0.f : m1;
            const float f0 = exp2f(mx[a][0] - c0), f1 = exp2f(mx[a][1] - c1);       // first block: exp2(-inf) = 0
            mx[a][0] = m0;
            mx[a][1] = m1;
            float l0 = 0.f, l1 = 0.f;
#pragma unroll
            for (int n = 0; n < 8; n++) {
                s[n][0] = exp2f(s[n][0] - c0); s[n][1] = exp2f(s[n][1] - c0);
                s[n][2] = exp2f(s[n][2] - c1); s[n][3] = exp2f(s[n][3] - c1);
                l0 += s[n][0] + s[n][1];
                l1 += s[n][2] + s[n][3];
            }
            ls[a][0] = ls[a][0] * f0 + l0;                                          // per lane; the quad is added at the end
            ls[a][1] = ls[a][1] * f1 + l1;
#pragma unroll
            for (int n = 0; n < VT * 2; n++) { o[a][n][0] *= f0; o[a][n][1] *= f0; o[a][n][2] *= f1; o[a][n][3] *= f1; }
#pragma unroll
            for (int kk = 0; kk < kKeys / 16; kk++) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float a0 = s[2 * kk + (e >> 1)][(e & 1) * 2], a1 = s[2 * kk + (e >> 1)][(e & 1) * 2 + 1];
                    hi[e] = pack_bf16(a0, a1);
                    const __nv_bfloat162 hv = *reinterpret_cast<const __nv_bfloat162*>(&hi[e]);
                    lo[e] = pack_bf16(a0 - __low2float(hv), a1 - __high2float(hv));
                }
                const uint32_t vaddr = smem_u32(vt + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VP + (lane >> 4) * 8);
#pragma unroll
                for (int n = 0; n < VT; n++) {
                    uint32_t vb[4];
                    ldsm4t(vb, vaddr + n * 32);
                    mma_bf16(o[a][2 * n], hi, vb[0], vb[1]);
                    mma_bf16(o[a][2 * n + 1], hi, vb[2], vb[3]);
                    mma_bf16(o[a][2 * n], lo, vb[0], vb[1]);
                    mma_bf16(o[a][2 * n + 1], lo, vb[2], vb[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int a = 0; a < MAPS; a++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float l = ls[a][e];
            l += __shfl_xor_sync(0xffffffffu, l, 1);
            l += __shfl_xor_sync(0xffffffffu, l, 2);
            ls[a][e] = l > 0.f ? 1.f / l : 0.f;
        }
    float ss0 = 0.f, ss1 = 0.f;
#pragma unroll
    for (int n = 0; n < VT * 2; n++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float x0 = o[0][n][e] * ls[0][0], x1 = o[0][n][2 + e] * ls[0][1];
            if (MAPS == 2) {
                x0 -= p.lambda * (o[MAPS - 1][n][e] * ls[MAPS - 1][0]);
                x1 -= p.lambda * (o[MAPS - 1][n][2 + e] * ls[MAPS - 1][1]);
            }
            o[0][n][e] = x0;
            o[0][n][2 + e] = x1;
            ss0 = fmaf(x0, x0, ss0);
            ss1 = fmaf(x1, x1, ss1);
        }
    float f0 = 1.f, f1 = 1.f;
    if (MAPS == 2) {
        ss0 += __shfl_xor_sync(0xffffffffu, ss0, 1);
        ss0 += __shfl_xor_sync(0xffffffffu, ss0, 2);
        ss1 += __shfl_xor_sync(0xffffffffu, ss1, 1);
        ss1 += __shfl_xor_sync(0xffffffffu, ss1, 2);
        f0 = rsqrtf(ss0 / (float)p.vdim + p.eps) * p.out_scale;
        f1 = rsqrtf(ss1 / (float)p.vdim + p.eps) * p.out_scale;
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int m = r0 + warp * 16 + gq + 8 * e;
        if (m >= p.M) continue;
        const bf16* gr = p.gate != nullptr ? static_cast<const bf16*>(p.gate) + ((size_t)m * p.H + h) * p.vdim : nullptr;
        bf16* orow = static_cast<bf16*>(p.out) + (size_t)m * p.out_pitch + (size_t)h * p.out_head;
        const float f = e ? f1 : f0;
#pragma unroll
        for (int n = 0; n < VT * 2; n++)
#pragma unroll
            for (int d = 0; d < 2; d++) {
                const int col = n * 8 + 2 * t + d;
                if (col < p.vdim) orow[col] = __float2bfloat16_rn(o[0][n][2 * e + d] * f * (gr != nullptr ? __bfloat162float(gr[col]) : 1.f));
            }
    }
}

int pick_splits(int M, int groups, int key_blocks) {
    int s = 592 / (M * groups);
    s = s < 1 ? 1 : (s > kMaxSplits ? kMaxSplits : s);
    return s < key_blocks ? s : (key_blocks < 1 ? 1 : key_blocks);
}
// Query heads of a CTA: at most 16 query vectors.
void pick_groups(int R, int maps, int* hpg, int* qgroups) {
    const int most = 16 / maps;
    *qgroups = (R + most - 1) / most;
    *hpg = (R + *qgroups - 1) / *qgroups;
}

constexpr size_t kMaxSmem = 227 * 1024;

size_t rows_smem(const AttnParams& p, int qn, int elem, bool shared) {
    const int KP = p.maps * p.dp + 16 / elem;
    return (size_t)(qn * p.dp + qn * (kKeys + 4) + 4 * qn + kKeys) * 4 + (size_t)kKeys * (KP + (shared ? 0 : p.vp)) * elem;
}

template <typename T, int QN, int CR, bool SHARED>
int launch_rows_c(AttnParams& p, cudaStream_t st) {
    const size_t smem = rows_smem(p, QN, sizeof(T), SHARED);
    if (smem > kMaxSmem) return B200_ELIMIT;
    auto k = attention_rows_kernel<T, QN, CR, SHARED>;
    if (smem > 48 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return check_launch();
    launch_kernel(k, dim3(p.splits, p.G * p.qgroups, p.M), dim3(kRowThreads), smem, st, p);
    if (check_launch() != B200_OK) return B200_ECUDA;
    launch_kernel(attention_merge_kernel<T, CR>, dim3(p.H, p.M), dim3(kRowThreads), 0, st, p);
    return check_launch();
}

template <typename T, int QN>
int launch_rows(AttnParams& p, cudaStream_t st) {
    return p.vdim <= kRowThreads ? launch_rows_c<T, QN, 1, false>(p, st) : launch_rows_c<T, QN, 2, false>(p, st);
}
template <typename T, int QN>
int launch_rows_shared(AttnParams& p, cudaStream_t st) {
    if (p.vdim <= 2 * kRowThreads) return launch_rows_c<T, QN, 2, true>(p, st);
    if (p.vdim <= 4 * kRowThreads) return launch_rows_c<T, QN, 4, true>(p, st);
    if constexpr (QN <= 8) {
        if (p.vdim <= 8 * kRowThreads) return launch_rows_c<T, QN, 8, true>(p, st);
    }
    return B200_ELIMIT;
}

template <typename T>
int launch_rows_any(AttnParams& p, cudaStream_t st) {
    const int nq = p.hpg * p.maps;
    if (nq <= 2) return launch_rows<T, 2>(p, st);
    if (nq <= 4) return launch_rows<T, 4>(p, st);
    if (nq <= 8) return launch_rows<T, 8>(p, st);
    return launch_rows<T, 16>(p, st);
}

template <typename T>
int launch_rows_latent(AttnParams& p, cudaStream_t st) {
    if (p.hpg <= 4) return launch_rows_shared<T, 4>(p, st);
    if (p.hpg <= 8) return launch_rows_shared<T, 8>(p, st);
    return launch_rows_shared<T, 16>(p, st);
}

template <int VT, int MAPS, bool LATENT>
int launch_prompt(const AttnParams& p, cudaStream_t st) {
    auto k = attention_prompt_kernel<VT, MAPS, LATENT>;
    const int KP = MAPS * p.dp + 8;
    const size_t smem = (size_t)(3 * kKeys * KP + 2 * kKeys * (VT * 16 + 8)) * 2;
    if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return check_launch();
    launch_kernel(k, dim3(p.H, (p.M + kQRows - 1) / kQRows), dim3(128), smem, st, p);
    return check_launch();
}

template <int MAPS, bool LATENT>
int launch_prompt_any(const AttnParams& p, cudaStream_t st) {
    if (p.vp <= 32) return launch_prompt<2, MAPS, LATENT>(p, st);
    if (p.vp <= 64) return launch_prompt<4, MAPS, LATENT>(p, st);
    if (p.vp <= 96) return launch_prompt<6, MAPS, LATENT>(p, st);
    return launch_prompt<8, MAPS, LATENT>(p, st);
}

// Passes of a latent layer that walk the latent itself, other than latent.cu's: all heads read the same rows.  Heads of a CTA:
// what the shared memory holds.
int launch_latent_rows(const b200_hybrid_model& m, const b200_hybrid_layer& l, AttnParams& p, int max_keys, cudaStream_t st) {
    const int elem = act_bytes(m.act_type);
    int most = p.vdim <= 4 * kRowThreads ? 16 : 8;
    while (most > 4 && rows_smem(p, most, elem, true) > kMaxSmem) most /= 2;
    p.qgroups = (p.H + most - 1) / most;
    p.hpg = (p.H + p.qgroups - 1) / p.qgroups;
    p.splits = pick_splits(p.M, p.qgroups, (max_keys + p.tail + kKeys - 1) / kKeys);
    if ((size_t)p.M * p.H * p.splits * (p.vp + 2) * 4 > m.attn_part_bytes) return B200_EWORKSPACE;
    return m.act_type == B200_ACT_F32 ? launch_rows_latent<float>(p, st) : launch_rows_latent<bf16>(p, st);
}

}  // namespace

size_t attention_part_bytes(const b200_hybrid_model& m, int rows) {
    size_t most = 0;
    for (int i = 0; i < m.n_layers; i++) {
        const b200_hybrid_layer& l = m.layers[i];
        if (l.mixer != B200_MIXER_ATTENTION && l.mixer != B200_MIXER_LATENT) continue;
        const size_t r = rows > 592 ? rows : 592;        // rows * splits never exceeds it (pick_splits)
        size_t b = r * l.heads * l.maps * (round_up(l.vdim, 16) + 2) * 4;
        if (l.mixer == B200_MIXER_LATENT) {
            const size_t vectors = r * l.heads, packed = latent_attention_parts(rows, l.heads);
            b = (vectors > packed ? vectors : packed) * (round_up(l.kv_rank, 16) + 2) * 4;
        }
        most = b > most ? b : most;
    }
    return most;
}

int launch_attention(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& ps,
                     cudaStream_t st) {
    AttnParams p{};
    char* cache = static_cast<char*>(ps.cache);
    if (l.mixer == B200_MIXER_LATENT) {
        const int cp = round_up(l.kv_rank, 16), rp = round_up(l.rot_dim, 16);
        p.q = m.qb; p.part = m.attn_part; p.pos = ps.pos; p.tail_pos = ps.tail_pos; p.mask = ps.mask; p.prefix = ps.prefix;
        p.M = ps.M; p.H = l.heads; p.maps = 1; p.window = l.window; p.keep = l.keep_first; p.tree = ps.tree;
        p.tail = ps.tree ? ps.tail : 0; p.scale_log2 = l.scale * kLog2e; p.out_scale = 1.f; p.eps = m.eps;
        if (latent_expands(m, l, ps)) {
            p.G = l.heads; p.rp = rp; p.dim = l.dim; p.dp = round_up(l.dim, 16) + rp; p.vdim = l.vdim; p.vp = round_up(l.vdim, 16);
            p.kc = m.kx; p.vc = m.vx; p.cap = m.x_rows; p.krot = cache + r.k_off + (size_t)cp * 2; p.krot_pitch = cp + rp;
            p.q_pitch = l.heads * p.dp; p.out = m.ab; p.out_pitch = round_up(l.heads * l.vdim, 64); p.out_head = l.vdim;
            return launch_prompt_any<1, true>(p, st);
        }
        if (m.act_type == B200_ACT_BF16 && cp <= kLatentColumns) return launch_latent_attention(m, l, r, ps, st);
        p.G = 1; p.dim = p.dp = cp + rp; p.vdim = l.kv_rank; p.vp = cp; p.kc = cache + r.k_off; p.cap = ps.cache_rows;
        p.q_pitch = l.heads * p.dp; p.out = m.ob; p.out_head = l.value.pitch; p.out_pitch = l.heads * l.value.pitch;
        return launch_latent_rows(m, l, p, ps.max_keys, st);
    }
    p.q = m.qb; p.kc = cache + r.k_off; p.vc = cache + r.v_off; p.gate = m.gb; p.out = m.ab; p.part = m.attn_part;
    p.pos = ps.pos; p.tail_pos = ps.tail_pos; p.mask = ps.mask; p.prefix = ps.prefix;
    p.M = ps.M; p.H = l.heads; p.G = l.kv_heads; p.maps = l.maps; p.dim = l.dim; p.dp = round_up(l.dim, 16); p.vdim = l.vdim;
    p.vp = round_up(l.vdim, 16); p.cap = ps.cache_rows; p.window = l.window; p.keep = l.keep_first; p.tree = ps.tree;
    p.tail = ps.tree ? ps.tail : 0; p.q_pitch = l.heads * l.maps * p.dp; p.out_pitch = round_up(l.heads * l.vdim, 64);
    p.out_head = l.vdim;
    p.scale_log2 = l.scale * kLog2e; p.lambda = l.lambda; p.out_scale = l.out_scale; p.eps = m.eps;
    if (m.act_type == B200_ACT_BF16 && !ps.tree && ps.M > 16 && p.dp <= 128 && p.vp <= 128)
        return l.maps == 2 ? launch_prompt_any<2, false>(p, st) : launch_prompt_any<1, false>(p, st);
    pick_groups(p.H / p.G, p.maps, &p.hpg, &p.qgroups);
    long long keys = (long long)l.window + l.keep_first;
    if (keys > ps.max_keys) keys = ps.max_keys;
    keys += p.tail;
    p.splits = pick_splits(p.M, p.G * p.qgroups, (int)((keys + kKeys - 1) / kKeys));
    if ((size_t)p.M * p.H * p.maps * p.splits * (p.vp + 2) * 4 > m.attn_part_bytes) return B200_EWORKSPACE;
    return m.act_type == B200_ACT_F32 ? launch_rows_any<float>(p, st) : launch_rows_any<bf16>(p, st);
}

}  // namespace hybrid
}  // namespace b200
