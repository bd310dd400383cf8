// Latent attention of the hybrid decoders, the steps around the attention itself: norm of the latent, interleaved rotation of
// the query parts and of the shared key part, cache row.  A token's cache row is [latent | rotated key part], each padded to 16.
#include "hybrid.cuh"

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
    float ss = 0.f;
    for (int c = tid; c < p.rank; c += kThreads) ss = fmaf(lat[c], lat[c], ss);
    const float rstd = rsqrtf(block_sum(ss, red) / (float)p.rank + p.eps);       // (its barriers publish the angles too)
    T* dst = static_cast<T*>(p.cache) + (size_t)(p.prefix[0] + p.write_off + m) * (p.cp + p.rp);
    for (int c = tid; c < p.cp; c += kThreads) dst[c] = from_f32<T>(c < p.rank ? lat[c] * rstd * p.w[c] : 0.f);
    for (int i = tid; i < p.rp / 2; i += kThreads) {
        float u = 0.f, v = 0.f;
        if (i < half) {
            const float a = kr[2 * i], b = kr[2 * i + 1], c = s_cs[2 * i], s = s_cs[2 * i + 1];
            u = a * c - b * s;
            v = b * c + a * s;
        }
        dst[p.cp + 2 * i] = from_f32<T>(u);
        dst[p.cp + 2 * i + 1] = from_f32<T>(v);
    }
    for (int e = tid; e < p.heads * (p.rp / 2); e += kThreads) {
        const int h = e / (p.rp / 2), i = e - h * (p.rp / 2);
        float u = 0.f, v = 0.f;
        if (i < half) {
            const float a = row[h * p.rot + 2 * i], b = row[h * p.rot + 2 * i + 1], c = s_cs[2 * i], s = s_cs[2 * i + 1];
            u = a * c - b * s;
            v = b * c + a * s;
        }
        T* q = static_cast<T*>(p.q) + ((size_t)m * p.heads + h) * p.unit + p.q_off + 2 * i;
        q[0] = from_f32<T>(u);
        q[1] = from_f32<T>(v);
    }
    for (int e = tid; e < p.heads * (p.q_off - p.q_len); e += kThreads) {        // padding of the other query part
        const int h = e / (p.q_off - p.q_len), i = e - h * (p.q_off - p.q_len);
        static_cast<T*>(p.q)[((size_t)m * p.heads + h) * p.unit + p.q_len + i] = from_f32<T>(0.f);
    }
}

}  // namespace

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
    if (m.act_type == B200_ACT_F32) launch_kernel(latent_prep_kernel<float>, dim3(ps.M), dim3(kThreads), smem, st, p);
    else launch_kernel(latent_prep_kernel<bf16>, dim3(ps.M), dim3(kThreads), smem, st, p);
    return check_launch();
}

}  // namespace hybrid
}  // namespace b200
