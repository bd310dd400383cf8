// Latent attention of the hybrid decoders.  A token's cache row is [latent | rotated key part], each padded to 16.
//
//   latent_prep      norm of the latent, interleaved rotation of the query parts and of the shared key part, cache row.
//   latent_rows      bf16, few query rows: queries are brought into the latent's space, so all heads read the same rows as keys
//                    and (their first columns) as values.  CTA = (key split, 16 (row, head) vectors): scores, softmax and
//                    weighted sum on mma.sync over blocks of 32 cache rows, double-buffered; the softmax weights enter as a
//                    pair of bf16 terms.  Partial (max, sum, output) per split, added in split order by latent_merge.
#include "mma.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kThreads = 256;
constexpr int kExpandRows = 32;          // more rows of a chain: keys and values of all heads are written out

struct PrepParams {
    const float* in;         // [M][heads * rot | rank | rot]
    const float* freq;       // [rot / 2]
    const float* w;          // [rank]
    const int* pos;
    const int* prefix;
    void* cache;             // [rows][cp + rp]
    void* q;                 // [M][heads][unit], rotated part at column q_off
    int write_off, heads, rank, rot, cp, rp, unit, q_len, q_off;
    float eps, mag;
};

// The pair at `x` turned by the angle whose cos, sin are at `cs`.
__device__ __forceinline__ void rotate(const float* x, const float* cs, float* u, float* v) {
    *u = x[0] * cs[0] - x[1] * cs[1];
    *v = x[1] * cs[0] + x[0] * cs[1];
}
__device__ __forceinline__ void put2(float* p, float u, float v) { *reinterpret_cast<float2*>(p) = make_float2(u, v); }
__device__ __forceinline__ void put2(bf16* p, float u, float v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(u, v); }

// Grid (rows, slices of the heads); the first slice also writes the cache row.
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_prep_kernel(const PrepParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float s_cs[];      // cos, sin of every pair
    __shared__ float red[33];
    const int m = blockIdx.x, tid = threadIdx.x, half = p.rot / 2;
    const float* row = p.in + (size_t)m * (p.heads * p.rot + p.rank + p.rot);
    const float* lat = row + p.heads * p.rot;
    const float* kr = lat + p.rank;
    const float at = (float)p.pos[m];
    for (int i = tid; i < half; i += kThreads) {
        float s, c;
        sincosf(at * p.freq[i], &s, &c);
        s_cs[2 * i] = c * p.mag;
        s_cs[2 * i + 1] = s * p.mag;
    }
    __syncthreads();
    const int per = (p.heads + gridDim.y - 1) / gridDim.y, h0 = blockIdx.y * per, nh = max(0, min(per, p.heads - h0)), pairs = p.rp / 2;
    T* q = static_cast<T*>(p.q) + ((size_t)m * p.heads + h0) * p.unit;
    for (int e = tid; e < nh * pairs; e += kThreads) {
        const int h = e / pairs, i = e - h * pairs;
        float u = 0.f, v = 0.f;
        if (i < half) rotate(row + (h0 + h) * p.rot + 2 * i, s_cs + 2 * i, &u, &v);
        put2(q + (size_t)h * p.unit + p.q_off + 2 * i, u, v);
    }
    const int pad = p.q_off - p.q_len;                                           // of the other query part
    for (int e = tid; e < nh * pad; e += kThreads) q[(size_t)(e / pad) * p.unit + p.q_len + e % pad] = from_f32<T>(0.f);
    if (blockIdx.y > 0) return;
    float ss = 0.f;
    for (int c = tid; c < p.rank; c += kThreads) ss = fmaf(lat[c], lat[c], ss);
    const float rstd = rsqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
    T* dst = static_cast<T*>(p.cache) + (size_t)(p.prefix[0] + p.write_off + m) * (p.cp + p.rp);
    for (int c = tid; c < p.cp; c += kThreads) dst[c] = from_f32<T>(c < p.rank ? lat[c] * rstd * p.w[c] : 0.f);
    for (int i = tid; i < pairs; i += kThreads) {
        float u = 0.f, v = 0.f;
        if (i < half) rotate(kr + 2 * i, s_cs + 2 * i, &u, &v);
        put2(dst + p.cp + 2 * i, u, v);
    }
}

constexpr int kBlock = 32;               // cache rows of a block
constexpr int kVecs = 16;                // (row, head) vectors of a CTA
constexpr int kRowThreads = 128;
constexpr int kSlots = 296;              // CTAs on the device
constexpr int kMostSplits = 64;

struct RowsParams {
    const bf16* q;           // [M * H][width]
    const bf16* cache;       // [rows][width], width = cp + rp
    float* part;             // [M * H][splits][cp + 2]
    bf16* out;               // [M * H][out_pitch]
    const int* pos;
    const unsigned long long* mask;
    const int* prefix;
    int M, H, cp, width, rows, tree, tail, splits, out_pitch;
    float scale_log2;

    // Cache rows of the pass: committed ones, then its own (chain) or the tail.
    __device__ __forceinline__ int total() const { return min(prefix[0] + (tree ? tail : M), rows); }
    __device__ __forceinline__ int per_split(int total) const { return ((total + kBlock - 1) / kBlock + splits - 1) / splits; }
};

template <int NV>                        // 8-column value tiles of a warp
__global__ void __launch_bounds__(kRowThreads) latent_rows_kernel(const RowsParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    constexpr int SP = kBlock + 1, PP = kBlock + 8;
    const int KP = round_up(max(p.width, 32 * NV), 64) + 8;
    bf16* sq = reinterpret_cast<bf16*>(smem_raw);                        // [16][KP]
    bf16* sk = sq + kVecs * KP;                                          // [2][32][KP]
    bf16* sp = sk + 2 * kBlock * KP;                                     // [2][16][PP] weights: value, remainder
    float* ss = reinterpret_cast<float*>(sp + 2 * kVecs * PP);           // [16][SP]
    __shared__ float sm[kVecs], sl[kVecs], sr[kVecs];
    __shared__ int spos[kVecs];
    __shared__ unsigned long long smask[kVecs];
    const int split = blockIdx.x, v0 = blockIdx.y * kVecs, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t = lane & 3;
    const int nvec = min(kVecs, p.M * p.H - v0);
    const int prefix = p.prefix[0], total = p.total(), per = p.per_split(total), blocks = (total + kBlock - 1) / kBlock;
    const int b0 = split * per, b1 = min(blocks, b0 + per);
    if (b0 >= b1) return;                                                // the merge knows which splits hold something
    const int chunks = p.width / 8;
    auto load = [&](int b) {
        bf16* dst = sk + (b & 1) * kBlock * KP;
        for (int e = tid; e < kBlock * chunks; e += kRowThreads) {
            const int r = e / chunks, c = e - r * chunks, j = b * kBlock + r;
            if (j < total) cp_async16(smem_u32(dst + r * KP + c * 8), p.cache + (size_t)j * p.width + c * 8);
            else *reinterpret_cast<uint4*>(dst + r * KP + c * 8) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    load(b0);
    for (int e = tid; e < kVecs * chunks; e += kRowThreads) {
        const int r = e / chunks, c = e - r * chunks;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < nvec) v = *reinterpret_cast<const uint4*>(p.q + (size_t)(v0 + r) * p.width + c * 8);
        *reinterpret_cast<uint4*>(sq + r * KP + c * 8) = v;
    }
    if (tid < kVecs) {
        const int row = (v0 + min(tid, nvec - 1)) / p.H;
        sm[tid] = -INFINITY;
        sl[tid] = 0.f;
        spos[tid] = p.pos[row];
        smask[tid] = p.tree ? p.mask[row] : 0ull;
    }
    float o[NV][4];
#pragma unroll
    for (int n = 0; n < NV; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    for (int b = b0; b < b1; b++) {
        if (b + 1 < b1) {
            load(b + 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const bf16* kt = sk + (b & 1) * kBlock * KP;
        {                                                                // scores: 8 cache rows per warp
            float s[2][4] = {};
            const uint32_t qaddr = smem_u32(sq + (lane & 15) * KP + (lane >> 4) * 8);
            const uint32_t kaddr = smem_u32(kt + (warp * 8 + (lane & 7)) * KP + (lane >> 3) * 8);
            int c = 0;
#pragma unroll 2
            for (; c + 32 <= p.width; c += 32) {
                uint32_t qa[4], qb[4], kb[4];
                ldsm4(qa, qaddr + c * 2);
                ldsm4(qb, qaddr + c * 2 + 32);
                ldsm4(kb, kaddr + c * 2);
                mma_bf16(s[0], qa, kb[0], kb[1]);
                mma_bf16(s[1], qb, kb[2], kb[3]);
            }
            if (c < p.width) {                                           // (16 columns; the row's padding is not used)
                uint32_t qa[4], kb[4];
                ldsm4(qa, qaddr + c * 2);
                ldsm4(kb, kaddr + c * 2);
                mma_bf16(s[0], qa, kb[0], kb[1]);
            }
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int v = gq + (e >> 1) * 8, key = warp * 8 + 2 * t + (e & 1), j = b * kBlock + key;
                bool vis;
                if (p.tree && j >= prefix) vis = j < total && ((smask[v] >> (j - prefix)) & 1ull);
                else vis = j < total && j <= spos[v];
                ss[v * SP + key] = vis ? (s[0][e] + s[1][e]) * p.scale_log2 : -INFINITY;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kVecs / 4; i++) {                            // softmax: 4 vectors per warp, a lane per cache row
            const int v = warp * (kVecs / 4) + i;
            const float a = ss[v * SP + lane], mo = sm[v], mn = fmaxf(mo, warp_max(a)), base = mn == -INFINITY ? 0.f : mn;
            const float w = exp2f(a - base), sum = warp_sum(w);
            const bf16 hi = __float2bfloat16_rn(w);
            sp[v * PP + lane] = hi;
            sp[(kVecs + v) * PP + lane] = __float2bfloat16_rn(w - __bfloat162float(hi));
            __syncwarp();
            if (lane == 0) {
                const float f = mo == -INFINITY ? 0.f : exp2f(mo - base);
                sr[v] = f;
                sl[v] = sl[v] * f + sum;
                sm[v] = mn;
            }
        }
        __syncthreads();
        const float f0 = sr[gq], f1 = sr[gq + 8];
#pragma unroll
        for (int n = 0; n < NV; n++) { o[n][0] *= f0; o[n][1] *= f0; o[n][2] *= f1; o[n][3] *= f1; }
#pragma unroll
        for (int kk = 0; kk < kBlock / 16; kk++) {
            uint32_t hi[4], lo[4];
            const uint32_t paddr = smem_u32(sp + (lane & 15) * PP + kk * 16 + (lane >> 4) * 8);
            ldsm4(hi, paddr);
            ldsm4(lo, paddr + kVecs * PP * 2);
            const uint32_t vaddr = smem_u32(kt + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * KP + warp * NV * 8 + (lane >> 4) * 8);
#pragma unroll
            for (int n = 0; n < NV; n += 2) {
                uint32_t vb[4];
                ldsm4t(vb, vaddr + n * 16);
                mma_bf16(o[n], hi, vb[0], vb[1]);
                mma_bf16(o[n + 1], hi, vb[2], vb[3]);
                mma_bf16(o[n], lo, vb[0], vb[1]);
                mma_bf16(o[n + 1], lo, vb[2], vb[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int v = gq + 8 * e;
        if (v >= nvec) continue;
        float* dst = p.part + ((size_t)(v0 + v) * p.splits + split) * (p.cp + 2);
        if (warp == 0 && t == 0) { dst[0] = sm[v]; dst[1] = sl[v]; }
#pragma unroll
        for (int n = 0; n < NV; n++) {
            const int col = (warp * NV + n) * 8 + 2 * t;
            if (col < p.cp) *reinterpret_cast<float2*>(dst + 2 + col) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
        }
    }
}

// Adds the splits of one (row, head).
__global__ void __launch_bounds__(kRowThreads) latent_merge_kernel(const RowsParams p) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float sw[kMostSplits];
    const int v = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
    const int total = p.total(), per = p.per_split(total), ns = ((total + kBlock - 1) / kBlock + per - 1) / per;      // splits that hold something
    const size_t stride = p.cp + 2;
    const float* base = p.part + (size_t)v * p.splits * stride;
    if (tid < 32) {
        float mm[2], ll[2];
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int s = lane + 32 * i;
            mm[i] = s < ns ? base[s * stride] : -INFINITY;
            ll[i] = s < ns ? base[s * stride + 1] : 0.f;
        }
        const float mx = warp_max(fmaxf(mm[0], mm[1]));
        const float f0 = mm[0] == -INFINITY ? 0.f : exp2f(mm[0] - mx), f1 = mm[1] == -INFINITY ? 0.f : exp2f(mm[1] - mx);
        const float sum = warp_sum(f0 * ll[0] + f1 * ll[1]), inv = sum > 0.f ? 1.f / sum : 0.f;
        sw[lane] = f0 * inv;
        sw[lane + 32] = f1 * inv;
    }
    __syncthreads();
    const int c = (blockIdx.y * kRowThreads + tid) * 2;
    if (c < p.cp) {
        float2 a = make_float2(0.f, 0.f);
#pragma unroll 16
        for (int s = 0; s < ns; s++) {
            const float2 x = *reinterpret_cast<const float2*>(base + s * stride + 2 + c);
            a.x = fmaf(sw[s], x.x, a.x);
            a.y = fmaf(sw[s], x.y, a.y);
        }
        *reinterpret_cast<uint32_t*>(p.out + (size_t)v * p.out_pitch + c) = pack_bf16(a.x, a.y);
    }
}

template <int NV>
int launch_rows(const RowsParams& p, cudaStream_t st) {
    const int most = p.width > 32 * NV ? p.width : 32 * NV, KP = round_up(most, 64) + 8;
    const size_t smem = (size_t)(kVecs + 2 * kBlock) * KP * 2 + (size_t)2 * kVecs * (kBlock + 8) * 2 + (size_t)kVecs * (kBlock + 1) * 4;
    if (smem > 227 * 1024) return B200_ELIMIT;
    auto k = latent_rows_kernel<NV>;
    if (smem > 40 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return check_launch();
    launch_kernel(k, dim3(p.splits, (p.M * p.H + kVecs - 1) / kVecs), dim3(kRowThreads), smem, st, p);
    launch_kernel(latent_merge_kernel, dim3(p.M * p.H, (p.cp + 2 * kRowThreads - 1) / (2 * kRowThreads)), dim3(kRowThreads), 0, st, p);
    return check_launch();
}

int splits_for(int groups, int blocks) {
    int s = kSlots / groups;
    s = s < 1 ? 1 : (s > kMostSplits ? kMostSplits : s);
    return s < blocks ? s : (blocks < 1 ? 1 : blocks);
}

}  // namespace

size_t latent_attention_parts(int rows, int heads) {
    const size_t groups = ((size_t)rows * heads + kVecs - 1) / kVecs;        // groups * splits is at most the larger of these
    return kVecs * (groups > (size_t)kSlots ? groups : (size_t)kSlots);
}

int launch_latent_attention(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& ps, cudaStream_t st) {
    RowsParams p{};
    p.cp = round_up(l.kv_rank, 16);
    p.width = latent_pitch(l);
    p.q = static_cast<const bf16*>(m.qb); p.cache = reinterpret_cast<const bf16*>(static_cast<const char*>(ps.cache) + r.k_off);
    p.part = m.attn_part; p.out = static_cast<bf16*>(m.ob); p.pos = ps.pos; p.mask = ps.mask; p.prefix = ps.prefix;
    p.M = ps.M; p.H = l.heads; p.rows = ps.cache_rows; p.tree = ps.tree; p.tail = ps.tree ? ps.tail : 0;
    p.out_pitch = l.value.pitch; p.scale_log2 = l.scale * kLog2e;
    const int keys = ps.max_keys + p.tail, groups = (p.M * p.H + kVecs - 1) / kVecs;
    p.splits = splits_for(groups, ((keys < ps.cache_rows ? keys : ps.cache_rows) + kBlock - 1) / kBlock);
    if ((size_t)p.M * p.H * p.splits * (p.cp + 2) * 4 > m.attn_part_bytes) return B200_EWORKSPACE;
    if (p.cp <= 128) return launch_rows<4>(p, st);
    if (p.cp <= 256) return launch_rows<8>(p, st);
    return launch_rows<16>(p, st);
}

bool latent_expands(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_pass& p) {
    return m.act_type == B200_ACT_BF16 && !p.tree && p.M > kExpandRows && m.kx && m.vx && p.max_keys <= m.x_rows && p.max_keys <= p.cache_rows &&
           round_up(l.dim, 16) + round_up(l.rot_dim, 16) <= 256 && l.vdim <= 128;
}

int launch_latent_prep(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& ps, cudaStream_t st) {
    PrepParams p{};
    const bool expands = latent_expands(m, l, ps);
    p.in = m.lat32; p.freq = l.rot_freq; p.w = l.latent_norm; p.pos = ps.pos; p.prefix = ps.prefix; p.cache = static_cast<char*>(ps.cache) + r.k_off;
    p.q = m.qb; p.write_off = ps.tree ? ps.write_off : 0; p.heads = l.heads; p.rank = l.kv_rank; p.rot = l.rot_dim;
    p.cp = round_up(l.kv_rank, 16); p.rp = round_up(l.rot_dim, 16); p.q_len = expands ? l.dim : l.kv_rank; p.q_off = round_up(p.q_len, 16);
    p.unit = p.q_off + p.rp; p.eps = m.eps; p.mag = l.rot_mag;
    const size_t smem = (size_t)l.rot_dim * 4;
    if (smem > 40 * 1024) return B200_ELIMIT;
    const dim3 grid(ps.M, ps.M <= 32 ? (l.heads + 7) / 8 : 1);
    if (m.act_type == B200_ACT_F32) launch_kernel(latent_prep_kernel<float>, grid, dim3(kThreads), smem, st, p);
    else launch_kernel(latent_prep_kernel<bf16>, grid, dim3(kThreads), smem, st, p);
    return check_launch();
}

}  // namespace hybrid
}  // namespace b200
