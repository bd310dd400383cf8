// Matrix products y = x W^T of the hybrid decoders, W bf16 [N][K padded to 64].
//
// bf16 activations: one tcgen05 kernel for every row count.  The tile is 128 weight rows (the M of the MMA) x NT token
// columns; a TMA producer warp streams 128 x 64 weight boxes and NT x 64 activation boxes (128-byte swizzle, K-major)
// through a shared-memory ring, one thread issues tcgen05.mma (kind::f16, bf16 operands, fp32 accumulator in tensor
// memory), four or eight warps read the accumulator back (thread = weight row, so stores of neighbouring threads are
// neighbouring columns of a token's row) and apply the epilogue.  With few tokens a product is a stream of weights:
// the K range of a tile is then cut over a cluster of up to 8 CTAs whose accumulators are added through distributed
// shared memory in rank order, so that every SM streams whatever the matrix height.  The weight copies of the first
// ring stages are issued before the grid dependency resolves (weights do not depend on earlier kernels).
// With many tokens the kernel is persistent and double-buffers the accumulator, so a tile's epilogue overlaps the next
// tile's products.
// Every wait is bounded: one that gives up raises the error word and the CTA runs to its end.  No copy is multicast.
//
// fp32 activations: plain fp32 multiply-adds (no reduced-precision tensor-core mode): a warp per output column for few
// rows, 64 x 64 shared-memory tiles for many.
#include <cuda.h>

#include "hybrid.cuh"
#include "../pipeline.cuh"

namespace b200 {
namespace hybrid {
namespace {

constexpr int kTileRows = 128;                    // weight rows of a tile
constexpr int kTileK = 64;                        // 128 bytes of bf16: one swizzle span
constexpr int kWBytes = kTileRows * kTileK * 2;
constexpr int kMaxSplit = 8;                      // CTAs of a cluster
constexpr uint32_t kPolls = 1u << 22;
constexpr uint32_t kPollNs = 64u;

template <int NT>
struct Geo {
    // epilogue warps (a quarter of the tile's rows each; eight: two per quarter, half of the columns each), so that every SM has eight
    static constexpr int EPI = NT >= 128 ? 8 : 4;
    static constexpr int THREADS = (EPI + 2) * 32;         // + TMA producer warp + MMA warp
    static constexpr int XBYTES = NT * kTileK * 2;
    static constexpr int STAGE = kWBytes + XBYTES;
    static constexpr int STAGES = NT == 16 || NT == 128 ? 6 : (NT == 32 || NT == 160 ? 5 : 4);
    static constexpr int PER_SM = NT <= 64 ? 2 : 1;        // resident CTAs the shared memory allows
    static constexpr int NACC = NT >= 128 ? 2 : 1;
    static constexpr int ACC_COLS = NT < 32 ? 32 : (NT == 160 ? 256 : NT);
    static constexpr int TMEM_COLS = ACC_COLS * NACC;
    static constexpr int SMEM = STAGES * STAGE + 1024 + 256;
};

struct GemmParams {
    CUtensorMap wmap, xmap;
    Epi epi;
    int kblocks, ntiles, ttiles;      // 128-row tiles of all groups, token tiles
    int gtiles, gn, xg;               // tiles, rows and x columns of a group
    int ksplit;                       // CTAs of a cluster that share a tile's K range (1: none)
    int groups;
    const int* offsets;               // expert stacks: first token row of every group
    int* error;
};

// What a tile multiplies: weight row, x column and token row of its corner, output column of its first row.
struct Tile {
    int wrow, xcol, tok0, tokend, col0, rows;
};
__device__ __forceinline__ Tile tile_at(const GemmParams& p, int t, int nt) {
    Tile r;
    const int w = t / p.ttiles, g = w / p.gtiles, lt = w - g * p.gtiles;
    r.wrow = w * kTileRows;
    r.xcol = g * p.xg;
    r.tok0 = (t - w * p.ttiles) * nt;
    r.tokend = p.epi.M;
    r.col0 = g * p.gn + lt * kTileRows;
    r.rows = p.gn - lt * kTileRows;
    return r;
}
// Expert stacks: tile0[g] token tiles before group g; a group's tiles are ordered token tile fastest.
__device__ __forceinline__ Tile expert_tile_at(const GemmParams& p, const int* off, const int* tile0, int t, int nt) {
    Tile r;
    int lo = 0, hi = p.groups - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (tile0[mid] * p.gtiles <= t) lo = mid;
        else hi = mid - 1;
    }
    const int rem = t - tile0[lo] * p.gtiles, tt = tile0[lo + 1] - tile0[lo], lt = rem / tt;
    r.wrow = (lo * p.gtiles + lt) * kTileRows;
    r.xcol = 0;
    r.tok0 = off[lo] + (rem - lt * tt) * nt;
    r.tokend = off[lo + 1];
    r.col0 = lt * kTileRows;
    r.rows = p.gn - lt * kTileRows;
    return r;
}

__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];\n" ::"r"(dst),
        "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(bar)
        : "memory");
}
// K-major operand tile, rows of 128 bytes, 128-byte swizzle: 8-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t sw128_desc(uint32_t saddr) {
    return (uint64_t)((saddr & 0x3ffffu) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) |
           ((uint64_t)2 << 61);
}
__device__ __forceinline__ bool gwait(uint32_t bar, uint32_t parity) { return mbar_wait_timed(bar, parity, kPolls, kPollNs); }
__device__ __forceinline__ uint32_t cluster_rank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;\n" : "=r"(r));
    return r;
}
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;\n" ::: "memory");
}
__device__ __forceinline__ float ld_cluster_f32(uint32_t saddr, uint32_t rank) {
    float v;
    asm volatile("{\n .reg .u32 a;\n mapa.shared::cluster.u32 a, %1, %2;\n ld.shared::cluster.f32 %0, [a];\n}\n"
                 : "=f"(v)
                 : "r"(saddr), "r"(rank)
                 : "memory");
    return v;
}

template <int NT, bool EXPERTS>
__global__ void __launch_bounds__(Geo<NT>::THREADS, Geo<NT>::PER_SM) gemm_kernel(const __grid_constant__ GemmParams p) {
    using G = Geo<NT>;
    constexpr int kEpiWarps = G::EPI, kThreads = G::THREADS;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + G::STAGES * G::STAGE);
    uint64_t* full = bars;
    uint64_t* empty = full + G::STAGES;
    uint64_t* accfull = empty + G::STAGES;
    uint64_t* accempty = accfull + G::NACC;
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort;
    __shared__ int s_off[EXPERTS ? B200_HYBRID_MAX_EXPERTS + 1 : 1], s_tile0[EXPERTS ? B200_HYBRID_MAX_EXPERTS + 1 : 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ks = p.ksplit;
    const uint32_t rank = ks > 1 ? cluster_rank() : 0u;
    // K blocks of this CTA, output tiles of this CTA
    const int kb0 = (int)((long long)p.kblocks * rank / ks), kb1 = (int)((long long)p.kblocks * (rank + 1) / ks);
    const int nk = kb1 - kb0;
    int tiles = EXPERTS ? 0 : p.ntiles * p.ttiles;
    const int tile0 = blockIdx.x / ks, tile_step = gridDim.x / ks;
    auto tile_of = [&](int t) { return EXPERTS ? expert_tile_at(p, s_off, s_tile0, t, NT) : tile_at(p, t, NT); };

    if (threadIdx.x == 0) {
        s_abort = 0;
        for (int s = 0; s < G::STAGES; s++) {
            mbar_init(smem_u32(full + s), 1);
            mbar_init(smem_u32(empty + s), 1);
        }
        for (int s = 0; s < G::NACC; s++) {
            mbar_init(smem_u32(accfull + s), 1);
            mbar_init(smem_u32(accempty + s), kEpiWarps);
        }
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == kEpiWarps + 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(&s_tmem)), "n"(G::TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    if (EXPERTS) {
        pdl_wait();
        for (int e = threadIdx.x; e <= p.groups; e += kThreads) s_off[e] = p.offsets[e];
        __syncthreads();
        if (warp == 0) {                                    // token tiles before each group
            int before = 0;
            for (int e0 = 0; e0 < p.groups; e0 += 32) {
                const int e = e0 + lane;
                int n = e < p.groups ? (s_off[e + 1] - s_off[e] + NT - 1) / NT : 0;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const int u = __shfl_up_sync(0xffffffffu, n, o);
                    if (lane >= o) n += u;
                }
                if (e < p.groups) s_tile0[e + 1] = before + n;
                before += __shfl_sync(0xffffffffu, n, 31);
            }
            if (lane == 0) s_tile0[0] = 0;
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    if (EXPERTS) tiles = s_tile0[p.groups] * p.gtiles;
    const uint32_t tmem = s_tmem;
    volatile int* abort_flag = &s_abort;
    uint32_t issued = 0;                                    // producer: stages whose copies were issued

    if (warp == kEpiWarps) {
        // ------------------------------------------------------------------ TMA producer
        if (lane == 0) {
            uint32_t n = 0;
            // weights of the first stages, before anything of an earlier kernel is read
            uint32_t pre = 0;
            if (tile0 < tiles) {
                const int row = tile_of(tile0).wrow;
                pre = nk < G::STAGES ? nk : G::STAGES;
                for (uint32_t s = 0; s < pre; s++) {
                    mbar_expect_tx(smem_u32(full + s), G::STAGE);
                    tma_load_2d(smem_u32(smem + s * G::STAGE), &p.wmap, (kb0 + (int)s) * kTileK, row, smem_u32(full + s));
                }
            }
            pdl_wait();
            pdl_launch_dependents();
            bool ok = true;
            for (int t = tile0; t < tiles && ok; t += tile_step) {
                const Tile at = tile_of(t);
                for (int kb = kb0; kb < kb1; kb++, n++) {
                    const uint32_t s = n % G::STAGES, use = n / G::STAGES;
                    if (use > 0) {
                        ok = !*abort_flag && gwait(smem_u32(empty + s), (use - 1) & 1u);
                        if (!ok) break;
                    }
                    const uint32_t bar = smem_u32(full + s), dst = smem_u32(smem + s * G::STAGE);
                    if (n >= pre) {
                        mbar_expect_tx(bar, G::STAGE);
                        tma_load_2d(dst, &p.wmap, kb * kTileK, at.wrow, bar);
                    }
                    tma_load_2d(dst + kWBytes, &p.xmap, at.xcol + kb * kTileK, at.tok0, bar);
                    issued = n + 1;
                }
            }
            if (!ok && !*abort_flag) { *abort_flag = 1; atomicCAS(p.error, 0, 21); }
            // leave no copy in flight behind: wait (bounded) for the newest use of every stage
            if (*abort_flag)
                for (uint32_t s = 0; s < (uint32_t)G::STAGES && s < issued; s++) {
                    const uint32_t last = (issued - 1 - s) / G::STAGES;
                    gwait(smem_u32(full + s), last & 1u);
                }
        }
        __syncwarp();
    } else if (warp == kEpiWarps + 1) {
        // ------------------------------------------------------------------ MMA issuer
        if (lane == 0) {
            // fp32 accumulator, bf16 A and B, both K-major
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NT >> 3) << 17) | ((uint32_t)(kTileRows >> 4) << 24);
            uint32_t n = 0, it = 0;
            bool ok = true;
            for (int t = tile0; t < tiles && ok; t += tile_step, it++) {
                const uint32_t ab = it % G::NACC, ause = it / G::NACC;
                if (ause > 0) ok = !*abort_flag && gwait(smem_u32(accempty + ab), (ause - 1) & 1u);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                const uint32_t d = tmem + ab * G::ACC_COLS;
                for (int kb = 0; kb < nk; kb++, n++) {
                    const uint32_t s = n % G::STAGES, use = n / G::STAGES;
                    ok = !*abort_flag && gwait(smem_u32(full + s), use & 1u);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                    const uint64_t da = sw128_desc(smem_u32(smem + s * G::STAGE));
                    const uint64_t db = sw128_desc(smem_u32(smem + s * G::STAGE + kWBytes));
#pragma unroll
                    for (int k = 0; k < kTileK / 16; k++) {            // 16 k values: 32 bytes further inside the swizzle span
                        const uint32_t accumulate = (kb > 0 || k > 0) ? 1u : 0u;
                        asm volatile(
                            "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                            "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}\n" ::"r"(d),
                            "l"(da + 2 * k), "l"(db + 2 * k), "r"(idesc), "r"(accumulate)
                            : "memory");
                    }
                    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n" ::"r"(smem_u32(empty + s)) : "memory");
                }
                if (ok)
                    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n" ::"r"(smem_u32(accfull + ab)) : "memory");
            }
            if (!ok && !*abort_flag) { *abort_flag = 1; atomicCAS(p.error, 0, 22); }
        }
        __syncwarp();
    } else {
        // ------------------------------------------------------------------ epilogue: thread = weight row of the tile
        pdl_wait();
        uint32_t it = 0;
        bool ok = true;
        for (int t = tile0; t < tiles && ok; t += tile_step, it++) {
            const uint32_t ab = it % G::NACC, ause = it / G::NACC;
            ok = __all_sync(0xffffffffu, !*abort_flag && gwait(smem_u32(accfull + ab), ause & 1u));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const Tile at = tile_of(t);
            const int tok0 = at.tok0;
            const int quarter = warp & 3, cpart = NT * 4 / kEpiWarps, cfirst = (warp >> 2) * cpart;
            const uint32_t taddr = tmem + ab * G::ACC_COLS + ((uint32_t)(quarter * 32) << 16);
            const int r = quarter * 32 + lane;
            ColumnOut<bf16> out;
            const bool gated = p.epi.gate.kind != 0;
            if (ks == 1 && !gated) out.init(p.epi, r < at.rows ? at.col0 + r : -1);
            float* part = reinterpret_cast<float*>(smem);          // split: [token][128], over the drained ring
#pragma unroll 1
            for (int c = cfirst; c < cfirst + cpart; c += 16) {
                if (tok0 + c >= at.tokend) break;
                uint32_t v[16];
                asm volatile(
                    "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n"
                    : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]),
                      "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
                    : "r"(taddr + c)
                    : "memory");
                asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
                if (ks > 1) {
#pragma unroll
                    for (int i = 0; i < 16; i++) part[(c + i) * kTileRows + r] = __uint_as_float(v[i]);
                } else if (gated) {
                    store_gated_rows<bf16, 16>(p.epi, at.col0 + r, r < at.rows, tok0 + c, at.tokend - tok0 - c, v);
                } else {
                    out.store_rows<16>(tok0 + c, at.tokend - tok0 - c, v);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(accempty + ab));
        }
        if (!ok && lane == 0 && !*abort_flag) { *abort_flag = 1; atomicCAS(p.error, 0, 23); }
    }

    if (ks > 1) {
        // Every CTA of the cluster adds its share of the tile's rows over all K slices, in rank order.
        pdl_wait();
        __syncthreads();
        cluster_sync_all();
        if (tile0 < tiles && !*abort_flag) {
            const Tile at = tile_of(tile0);
            const int r0 = kTileRows * (int)rank / ks, share = kTileRows * ((int)rank + 1) / ks - r0;
            const int tok0 = at.tok0, ntok = min(NT, at.tokend - tok0);
            const uint32_t part = smem_u32(smem);
            auto total = [&](int c, int r) {
                float v[kMaxSplit];
#pragma unroll
                for (int q = 0; q < kMaxSplit; q++)
                    v[q] = q < ks ? ld_cluster_f32(part + (uint32_t)((c * kTileRows + r) * 4), (uint32_t)q) : 0.f;
                float a = 0.f;
#pragma unroll
                for (int q = 0; q < kMaxSplit; q++) a += v[q];
                return a;
            };
            if (p.epi.gate.kind != 0) {
                for (int i = threadIdx.x; i < share / 2 * ntok; i += kThreads) {
                    const int c = i / (share / 2), r = r0 + 2 * (i - c * (share / 2)), n = at.col0 + r, m = tok0 + c;
                    if (r >= at.rows) continue;
                    const float sc = p.epi.row_scale != nullptr ? p.epi.row_scale[m] : 1.f;
                    float g = total(c, r) * sc, u = total(c, r + 1) * sc;
                    if (p.epi.gate_bias != nullptr) { g += p.epi.gate_bias[n]; u += p.epi.gate_bias[n + 1]; }
                    static_cast<bf16*>(p.epi.seg[0].dst)[(long long)m * p.epi.seg[0].row_stride + (n >> 1)] = __float2bfloat16_rn(gated_f(p.epi.gate, g, u));
                }
            } else {
                for (int i = threadIdx.x; i < share * ntok; i += kThreads) {
                    const int c = i / share, r = r0 + i - c * share;
                    ColumnOut<bf16> out;
                    out.init(p.epi, r < at.rows ? at.col0 + r : -1);
                    out.store(tok0 + c, total(c, r));
                }
            }
        }
        cluster_sync_all();                                        // no CTA leaves while its shared memory is read
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    if (warp == kEpiWarps + 1)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "n"(G::TMEM_COLS) : "memory");
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

int make_map(CUtensorMap* map, const void* base, int cols, int rows, int box_rows) {
    static EncodeTiledFn encode = nullptr;
    if (encode == nullptr) {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q) != cudaSuccess || fn == nullptr) {
            check_launch();
            return B200_ECUDA;
        }
        encode = reinterpret_cast<EncodeTiledFn>(fn);
    }
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kTileK, (cuuint32_t)box_rows};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        g_last_cuda_error = (int)r;
        return B200_ECUDA;
    }
    return B200_OK;
}

int sm_count() {
    static int sms = 0;
    if (sms == 0) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms < 1)
            sms = 148;
    }
    return sms;
}

template <int NT, bool EXPERTS>
int launch_gemm(const b200_linear& lin, const void* x, int x_pitch, int x_rows, const Epi& epi, int rows, const int* offsets, int* error, cudaStream_t st) {
    using G = Geo<NT>;
    auto kern = gemm_kernel<NT, EXPERTS>;
    static bool attr = false;
    if (!attr) {
        if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, G::SMEM) != cudaSuccess) return check_launch();
        attr = true;
    }
    GemmParams p;
    const int groups = lin.groups > 1 ? lin.groups : 1;
    int rc = make_map(&p.wmap, lin.w, lin.pitch, groups * round_up(lin.n, kTileRows), kTileRows);
    if (rc == B200_OK) rc = make_map(&p.xmap, x, x_pitch, x_rows, NT);
    if (rc != B200_OK) return rc;
    p.epi = epi;
    p.kblocks = lin.pitch / kTileK;
    p.gtiles = (lin.n + kTileRows - 1) / kTileRows;
    p.gn = lin.n;
    p.xg = lin.pitch;
    p.groups = groups;
    p.offsets = offsets;
    p.ntiles = groups * p.gtiles;
    p.ttiles = (rows + NT - 1) / NT;
    p.error = error;
    p.ksplit = 1;
    const int sms = sm_count(), tiles = p.ntiles * p.ttiles;
    if (NT <= 128 && !EXPERTS) {
        // Cut K while the slices of all tiles fit the device at once (two CTAs per SM keep enough copies in flight) and are
        // at least two blocks long.  Powers of two: clusters of other sizes do not fill the SM groups.
        while (p.ksplit < kMaxSplit && tiles * p.ksplit * 2 <= sms * G::PER_SM && p.kblocks >= 4 * p.ksplit) p.ksplit *= 2;
    }
    int grid = tiles * p.ksplit;
    if (EXPERTS) {
        // at most one partly filled token tile per expert
        const long long most = (long long)p.gtiles * (rows / NT + (rows < groups ? rows : groups));
        grid = most < sms * G::PER_SM ? (int)most : sms * G::PER_SM;
    } else if (p.ksplit == 1 && G::NACC > 1 && grid > sms) {
        grid = sms;                                                 // persistent
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(grid);
    cfg.blockDim = dim3(G::THREADS);
    cfg.dynamicSmemBytes = G::SMEM;
    cfg.stream = st;
    cudaLaunchAttribute attrs[2];
    int na = 0;
    if (p.ksplit > 1) {
        attrs[na].id = cudaLaunchAttributeClusterDimension;
        attrs[na].val.clusterDim.x = p.ksplit;
        attrs[na].val.clusterDim.y = 1;
        attrs[na].val.clusterDim.z = 1;
        na++;
    }
    if (g_use_pdl) {
        attrs[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attrs[na].val.programmaticStreamSerializationAllowed = 1;
        na++;
    }
    cfg.attrs = attrs;
    cfg.numAttrs = na;
    cudaLaunchKernelEx(&cfg, kern, p);
    return check_launch();
}

// ---------------------------------------------------------------- fp32 activations
struct F32Params {
    const bf16* w;
    const float* x;
    int n, npad, groups, pitch, x_pitch;      // rows of a group, as stored
};

// Few rows: one warp per output column, the rows in groups of 8.
__global__ void __launch_bounds__(256) linear_f32_rows_kernel(const F32Params p, const __grid_constant__ Epi epi) {
    pdl_wait();
    pdl_launch_dependents();
    const int nr = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, g = nr / p.npad, r = nr - g * p.npad;
    if (g >= p.groups || r >= p.n) return;
    ColumnOut<float> out;
    out.init(epi, g * p.n + r);
    const bf16* wr = p.w + (size_t)nr * p.pitch;
    const float* x = p.x + (size_t)g * p.pitch;
    for (int m0 = 0; m0 < epi.M; m0 += 8) {
        float acc[8] = {};
        for (int k = lane * 2; k < p.pitch; k += 64) {
            const float2 wv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(wr + k));
#pragma unroll
            for (int i = 0; i < 8; i++)
                if (m0 + i < epi.M) {
                    const float2 xv = *reinterpret_cast<const float2*>(x + (size_t)(m0 + i) * p.x_pitch + k);
                    acc[i] = fmaf(wv.x, xv.x, acc[i]);
                    acc[i] = fmaf(wv.y, xv.y, acc[i]);
                }
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float a = warp_sum(acc[i]);
            if (lane == 0 && m0 + i < epi.M) out.store(m0 + i, a);
        }
    }
}

// Many rows: 64 columns x 64 rows per CTA, 4 x 4 per thread.
__global__ void __launch_bounds__(256) linear_f32_tile_kernel(const F32Params p, const __grid_constant__ Epi epi) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float sw[16][68], sx[16][68];
    const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64, g = n0 / p.npad, c0 = n0 - g * p.npad;
    if (c0 >= p.n) return;
    const int tn = threadIdx.x & 15, tm = threadIdx.x >> 4;
    const float* x = p.x + (size_t)g * p.pitch;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.pitch; k0 += 16) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int e = threadIdx.x + 256 * i, r = e >> 4, k = e & 15;
            sw[k][r] = c0 + r < p.n ? __bfloat162float(p.w[(size_t)(n0 + r) * p.pitch + k0 + k]) : 0.f;
            sx[k][r] = m0 + r < epi.M ? x[(size_t)(m0 + r) * p.x_pitch + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; k++) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { a[i] = sw[k][tn + 16 * i]; b[i] = sx[k][tm + 16 * i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int c = c0 + tn + 16 * i;
        if (c >= p.n) continue;
        ColumnOut<float> out;
        out.init(epi, g * p.n + c);
#pragma unroll
        for (int j = 0; j < 4; j++)
            if (m0 + tm + 16 * j < epi.M) out.store(m0 + tm + 16 * j, acc[i][j]);
    }
}

}  // namespace

int launch_linear(int act_type, const b200_linear& lin, const void* x, int x_pitch, int x_rows, const Epi& epi, int* error, cudaStream_t st) {
    if (!lin.w || !x || lin.n < 1 || lin.pitch < 64 || lin.pitch % 64 != 0 || epi.M < 1 || x_rows < epi.M) return B200_EINVAL;
    const int groups = lin.groups > 1 ? lin.groups : 1;
    if (x_pitch == 0) x_pitch = groups * lin.pitch;
    if (!aligned16(lin.w) || !aligned16(x) || x_pitch % 8 != 0) return B200_EALIGN;
    if (act_type == B200_ACT_F32) {
        if (x_pitch < groups * lin.pitch || epi.gate.kind != 0) return B200_EINVAL;
        const int npad = round_up(lin.n, kTileRows);
        const F32Params p{static_cast<const bf16*>(lin.w), static_cast<const float*>(x), lin.n, npad, groups, lin.pitch, x_pitch};
        if (epi.M <= 16)
            launch_kernel(linear_f32_rows_kernel, dim3(groups * npad / 8), dim3(256), 0, st, p, epi);
        else
            launch_kernel(linear_f32_tile_kernel, dim3(groups * npad / 64, (epi.M + 63) / 64), dim3(256), 0, st, p, epi);
        return check_launch();
    }
    const int M = epi.M, tiles = groups * ((lin.n + kTileRows - 1) / kTileRows);
    if (M <= 16) return launch_gemm<16, false>(lin, x, x_pitch, x_rows, epi, M, nullptr, error, st);
    if (M <= 32) return launch_gemm<32, false>(lin, x, x_pitch, x_rows, epi, M, nullptr, error, st);
    // (few output columns: small token tiles, so that more SMs take part)
    if (M <= 64 || tiles * ((M + 255) / 256) * 2 <= sm_count()) return launch_gemm<64, false>(lin, x, x_pitch, x_rows, epi, M, nullptr, error, st);
    // (short K: a tile's epilogue is most of its time, and smaller tiles even out over the SMs)
    if (M <= 128 || lin.pitch <= 512) return launch_gemm<128, false>(lin, x, x_pitch, x_rows, epi, M, nullptr, error, st);
    return launch_gemm<256, false>(lin, x, x_pitch, x_rows, epi, M, nullptr, error, st);
}

int launch_linear_experts(const b200_linear& lin, const void* x, int x_rows, int rows, const int* offsets, const Epi& epi, int* error, cudaStream_t st) {
    if (!lin.w || !x || !offsets || lin.n < 1 || lin.pitch < 64 || lin.pitch % 64 != 0 || rows < 1 || x_rows < rows) return B200_EINVAL;
    if (lin.groups < 1 || lin.groups > B200_HYBRID_MAX_EXPERTS) return B200_ELIMIT;
    if (!aligned16(lin.w) || !aligned16(x)) return B200_EALIGN;
    // One token tile for most experts, with room for an uneven load: a second tile streams an expert's weights again.
    const int mean = rows / lin.groups;
    if (mean <= 20) return launch_gemm<32, true>(lin, x, lin.pitch, x_rows, epi, rows, offsets, error, st);
    if (mean <= 48) return launch_gemm<64, true>(lin, x, lin.pitch, x_rows, epi, rows, offsets, error, st);
    if (mean <= 100) return launch_gemm<128, true>(lin, x, lin.pitch, x_rows, epi, rows, offsets, error, st);
    if (mean <= 140) return launch_gemm<160, true>(lin, x, lin.pitch, x_rows, epi, rows, offsets, error, st);
    return launch_gemm<256, true>(lin, x, lin.pitch, x_rows, epi, rows, offsets, error, st);
}

}  // namespace hybrid
}  // namespace b200
