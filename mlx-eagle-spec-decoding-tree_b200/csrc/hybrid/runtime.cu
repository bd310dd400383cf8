// The pass driver: walks the layer runs and issues their launches; C entry points of libb200hybrid.so.
#include "hybrid.cuh"

#include <limits.h>

namespace b200 {
int g_last_cuda_error = 0;
int g_use_pdl = 1;
unsigned g_wait_limit = 0;

namespace hybrid {
namespace {

// q | k | v | gate of an attention layer: queries to the activation buffer (map vectors padded to 16), keys and values
// straight into the cache rows, the gate through its sigmoid.
Epi attention_in_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p) {
    Epi e{};
    const int dp = round_up(l.dim, 16), vp = round_up(l.vdim, 16), ke = l.maps * dp;
    char* cache = static_cast<char*>(p.cache);
    int n = 0;
    Seg s = plain_seg(n, n + l.heads * l.maps * l.dim, kOpNone, 0, m.qb, (long long)l.heads * ke);
    s.unit = l.dim; s.group_stride = dp;
    e.seg[0] = s;
    n = s.n1;
    s = plain_seg(n, n + l.kv_heads * l.maps * l.dim, kOpNone, 0, cache + r.k_off, ke);
    s.unit = l.dim; s.maps = l.maps; s.unit_pitch = dp; s.group_stride = (long long)p.cache_rows * ke; s.at_cache_row = 1;
    e.seg[1] = s;
    n = s.n1;
    s = plain_seg(n, n + l.kv_heads * l.vdim, kOpNone, 0, cache + r.v_off, vp);
    s.unit = l.vdim; s.group_stride = (long long)p.cache_rows * vp; s.at_cache_row = 1;
    e.seg[2] = s;
    n = s.n1;
    e.seg[3] = plain_seg(n, n + l.heads * l.vdim, kOpSigmoid, 0, m.gb, (long long)l.heads * l.vdim);
    e.nseg = 4;
    return e;
}

// q | f | v of a recurrence layer; tree passes leave f and v in the pending rows, from where a commit reads them.
Epi recurrence_in_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p) {
    Epi e{};
    const int nd = l.heads * l.dim, nv = l.heads * l.vdim;
    char* pend = static_cast<char*>(m.pending);
    float* g = p.tree ? reinterpret_cast<float*>(pend + r.pend_g) + (size_t)p.write_off * nd : m.gf;
    void* v = p.tree ? static_cast<void*>(pend + r.pend_v + (size_t)p.write_off * nv * act_bytes(m.act_type)) : m.vb;
    e.seg[0] = plain_seg(0, nd, kOpSilu, 0, m.qb, nd);
    e.seg[1] = plain_seg(nd, 2 * nd, kOpForget, 1, g, nd);
    e.seg[1].p0 = l.gate_bias;
    e.seg[1].p1 = l.gate_lower;
    e.seg[2] = plain_seg(2 * nd, 2 * nd + nv, kOpNone, 0, v, nv);
    e.nseg = 3;
    return e;
}

// q | k | v | beta | low-rank inputs of a delta layer; tree passes leave the convolution inputs and beta in the pending rows.
Epi delta_in_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p) {
    Epi e{};
    const int C = delta_channels(l), CP = delta_pitch(l);
    char* pend = static_cast<char*>(m.pending);
    void* c = p.tree ? static_cast<void*>(pend + r.pend_c + (size_t)p.write_off * CP * act_bytes(m.act_type)) : m.cb;
    float* b = p.tree ? reinterpret_cast<float*>(pend + r.pend_b) + (size_t)p.write_off * l.heads : m.beta;
    e.seg[0] = plain_seg(0, C, kOpNone, 0, c, CP);
    e.seg[1] = plain_seg(C, C + l.heads, kOpSigmoid, 1, b, l.heads);
    e.seg[2] = plain_seg(C + l.heads, C + l.heads + l.low_rank, kOpNone, 0, m.lowb, l.low.pitch);
    e.nseg = 3;
    return e;
}

// Low-rank inputs -> decay | output gate.
Epi delta_low_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p) {
    Epi e{};
    const int nd = l.heads * l.dim, nv = l.heads * l.vdim;
    float* g = p.tree ? reinterpret_cast<float*>(static_cast<char*>(m.pending) + r.pend_g) + (size_t)p.write_off * nd : m.gf;
    e.seg[0] = plain_seg(0, nd, kOpDecay, 1, g, nd);
    e.seg[0].p0 = l.decay_bias;
    e.seg[0].p1 = l.decay_rate;
    e.seg[1] = plain_seg(nd, nd + nv, kOpSigmoid, 0, m.gb, nv);
    e.nseg = 2;
    return e;
}

// Unrotated queries | rotated query parts, latent, rotated key part of a latent layer; what is normed or rotated stays fp32.
Epi latent_in_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l, bool expands) {
    Epi e{};
    const int nq = l.heads * l.dim, rest = l.heads * l.rot_dim + l.kv_rank + l.rot_dim;
    const int unit = expands ? round_up(l.dim, 16) + round_up(l.rot_dim, 16) : l.absorb.pitch;
    e.seg[0] = plain_seg(0, nq, kOpNone, 0, expands ? m.qb : m.qn, (long long)l.heads * unit);
    e.seg[0].unit = l.dim;
    e.seg[0].group_stride = unit;
    e.seg[1] = plain_seg(nq, nq + rest, kOpNone, 1, m.lat32, rest);
    e.nseg = 2;
    return e;
}

// Keys and values of all heads from the latent of the cache.
Epi latent_expand_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l) {
    Epi e{};
    const int dp = round_up(l.dim, 16), vp = round_up(l.vdim, 16), nk = l.heads * l.dim;
    e.seg[0] = plain_seg(0, nk, kOpNone, 0, m.kx, dp);
    e.seg[0].unit = l.dim;
    e.seg[0].group_stride = (long long)m.x_rows * dp;
    e.seg[1] = plain_seg(nk, nk + l.heads * l.vdim, kOpNone, 0, m.vx, vp);
    e.seg[1].unit = l.vdim;
    e.seg[1].group_stride = (long long)m.x_rows * vp;
    e.nseg = 2;
    return e;
}

Epi latent_absorb_epi(const b200_hybrid_model& m, const b200_hybrid_layer& l) {
    Epi e{};
    const int unit = latent_pitch(l);
    e.seg[0] = plain_seg(0, l.heads * l.kv_rank, kOpNone, 0, m.qb, (long long)l.heads * unit);
    e.seg[0].unit = l.kv_rank;
    e.seg[0].group_stride = unit;
    e.nseg = 1;
    return e;
}

Epi one_seg(const Seg& s) {
    Epi e{};
    e.nseg = 1;
    e.seg[0] = s;
    return e;
}

#define B200_TRY(x)                    \
    do {                               \
        const int rc_ = (x);           \
        if (rc_ != B200_OK) return rc_; \
    } while (0)

int product(const b200_hybrid_model& m, const b200_hybrid_pass& p, const b200_linear& lin, const void* x, Epi e, int rows, cudaStream_t st) {
    e.M = rows;
    e.prefix = p.prefix;
    e.write_off = p.tree ? p.write_off : 0;
    return launch_linear(m.act_type, lin, x, 0, m.max_rows, e, m.error, st);
}

int latent_mixer(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_run& r, const b200_hybrid_pass& p, cudaStream_t st) {
    const bool expands = latent_expands(m, l, p);
    B200_TRY(product(m, p, l.in, m.hb, latent_in_epi(m, l, expands), p.M, st));
    B200_TRY(launch_latent_prep(m, l, r, p, st));
    if (expands) {
        Epi e = latent_expand_epi(m, l);
        e.M = p.max_keys;
        B200_TRY(launch_linear(m.act_type, l.expand, static_cast<const char*>(p.cache) + r.k_off, latent_pitch(l), p.cache_rows, e, m.error, st));
        return launch_attention(m, l, r, p, st);
    }
    B200_TRY(product(m, p, l.absorb, m.qn, latent_absorb_epi(m, l), p.M, st));
    B200_TRY(launch_attention(m, l, r, p, st));
    return product(m, p, l.value, m.ob, one_seg(plain_seg(0, l.heads * l.vdim, kOpNone, 0, m.ab, round_up(l.heads * l.vdim, 64))), p.M, st);
}

// A sublayer's last product: into the stream, or into a buffer whose norm joins the stream.
int sublayer_out(const b200_hybrid_model& m, const b200_hybrid_pass& p, const b200_linear& lin, const void* x, const float* bias, const float* norm,
                 const float* inject, cudaStream_t st) {
    if (m.norm_out) {
        Seg s = plain_seg(0, m.width, bias ? kOpBias : kOpNone, 1, m.y, m.width);
        s.p0 = bias;
        B200_TRY(product(m, p, lin, x, one_seg(s), p.M, st));
        return launch_join(m, norm, p.M, 1, nullptr, inject, st);
    }
    Epi e = one_seg(plain_seg(0, m.width, kOpResidual, 1, m.x, m.width));
    e.seg[0].p0 = bias;
    e.mult = m.residual_mult;
    e.add = inject;
    return product(m, p, lin, x, e, p.M, st);
}

int feed_forward(const b200_hybrid_model& m, const b200_hybrid_layer& l, const b200_hybrid_pass& p, const float* inject, cudaStream_t st) {
    if (!m.norm_out) B200_TRY(launch_norm(m, l.norm2, p, false, p.M, st));
    const int pitch = round_up(l.ff, 64);
    if (l.ff_kind == B200_FF_EXPERTS) {
        const int* place = nullptr;
        if (router_in_rows(p.M)) B200_TRY(launch_router_rows(m, l, p.M, st));
        else B200_TRY(product(m, p, l.router, m.hb, one_seg(plain_seg(0, l.experts, kOpNone, 1, m.zr, l.experts)), p.M, st));
        B200_TRY(launch_experts(m, l, p.M, &place, st));
        return launch_join(m, m.norm_out ? l.norm2 : nullptr, p.M, l.top, place, inject, st);
    }
    if (l.ff_kind == B200_FF_GATED) {
        if (m.act_type == B200_ACT_F32) {
            B200_TRY(product(m, p, l.up, m.hb, one_seg(plain_seg(0, 2 * l.ff, kOpNone, 1, m.zb, round_up(2 * l.ff, 64))), p.M, st));
            B200_TRY(launch_gated(m, l, p.M, st));
        } else {
            Epi e = one_seg(plain_seg(0, l.ff, kOpNone, 0, m.zab, pitch));
            e.gate = gating_of(l);
            e.gate_bias = l.up_bias;
            B200_TRY(product(m, p, l.up, m.hb, e, p.M, st));
        }
    } else {
        B200_TRY(product(m, p, l.up, m.hb, one_seg(plain_seg(0, l.ff, kOpNone, 0, m.zb, pitch)), p.M, st));
        B200_TRY(launch_polynorm(m, l, p.M, st));
    }
    return sublayer_out(m, p, l.down, m.zab, l.down_bias, l.norm2, inject, st);
}

bool valid(const b200_hybrid_model& m, const b200_hybrid_pass& p) {
    if (m.act_type != B200_ACT_BF16 && m.act_type != B200_ACT_F32) return false;
    if (m.width < 1 || m.vocab < 1 || m.n_layers < 1 || m.n_runs < 1 || m.max_rows < 256 || !m.layers || !m.runs) return false;
    if (!m.dev_layers || !m.dev_runs || !m.embed || !m.final_norm || !m.x || !m.hb || !m.ab || !m.pending || !m.error) return false;
    if (m.injects && !m.emb) return false;
    if (p.M < 1 || p.M > m.max_rows || p.rows_out < 0 || p.rows_out > m.max_rows || p.cache_rows < 1) return false;
    if (!p.tokens || !p.pos || !p.prefix || !p.cache || (p.rows_out > 0 && !p.logits)) return false;
    if (p.tree && (!p.mask || !p.tail_pos || p.tail < 1 || p.tail > B200_HYBRID_PENDING || p.write_off < 0 || p.write_off + p.M > p.tail))
        return false;
    for (int i = 0; i < m.n_layers; i++) {
        const b200_hybrid_layer& l = m.layers[i];
        if (l.taps < 1 || l.taps > B200_HYBRID_MAX_TAPS || l.heads < 1 || l.dim < 1 || l.vdim < 1 || !l.norm1) return false;
        if (!m.norm_out && !l.conv) return false;
        if (l.ff > 0 && !l.norm2) return false;
        if (l.ff > 0 && l.ff_kind == B200_FF_EXPERTS) {
            if (l.experts < 1 || l.experts > B200_HYBRID_MAX_EXPERTS || l.top < 1 || l.top > l.experts || l.top > B200_HYBRID_MAX_TOP) return false;
            if (!m.zr || !m.route || (!m.xg && m.act_type == B200_ACT_BF16) || !m.y || m.route_top < l.top || m.route_experts < l.experts) return false;
        }
        if (m.norm_out && (!m.y || l.taps != 1)) return false;
        if (l.mixer == B200_MIXER_ATTENTION) {
            if (l.kv_heads < 1 || l.heads % l.kv_heads || l.maps < 1 || l.maps > 2 || l.window < 1 || l.keep_first < 0) return false;
            if (!m.attn_part) return false;
        } else if (l.mixer == B200_MIXER_RECURRENCE) {
            if (!l.gate_bias || !l.gate_lower || !l.head_norm) return false;
        } else if (l.mixer == B200_MIXER_DELTA) {
            if (l.kv_heads < 1 || l.heads % l.kv_heads || l.conv_taps < 1 || l.conv_taps > B200_HYBRID_MAX_TAPS || l.low_rank < 1) return false;
            if (!l.mix_conv || !l.decay_bias || !l.decay_rate || !l.head_norm || !m.cb || !m.lowb || !m.q32 || !m.k32 || !m.beta || !m.chunk) return false;
        } else if (l.mixer == B200_MIXER_LATENT) {
            if (l.kv_rank < 1 || l.rot_dim < 2 || l.rot_dim % 2 || l.maps != 1 || l.window != INT_MAX || l.keep_first != 0) return false;
            if (!l.rot_freq || !l.latent_norm || !m.lat32 || !m.qn || !m.ob || !m.attn_part) return false;
        } else {
            return false;
        }
    }
    return true;
}

}  // namespace
}  // namespace hybrid
}  // namespace b200

using namespace b200;
using namespace b200::hybrid;

extern "C" {

int b200_hybrid_version(void) { return 2; }
int b200_hybrid_last_cuda_error(void) { return g_last_cuda_error; }
void b200_hybrid_set_pdl(int enabled) { g_use_pdl = enabled ? 1 : 0; }

size_t b200_hybrid_attention_workspace_bytes(const b200_hybrid_model* model, int rows) {
    if (!model || !model->layers || rows < 1) return 0;
    return attention_part_bytes(*model, rows);
}

int b200_hybrid_forward(const b200_hybrid_model* model, const b200_hybrid_pass* pass, void* stream) {
    if (!model || !pass || !valid(*model, *pass)) return B200_EINVAL;
    const b200_hybrid_model& m = *model;
    const b200_hybrid_pass& p = *pass;
    for (int i = 0; i < m.n_layers; i++) {
        const b200_hybrid_layer& l = m.layers[i];
        if (l.mixer != B200_MIXER_LATENT && (l.dim > 256 || l.vdim > 256)) return B200_ELIMIT;
    }
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const size_t n = (size_t)p.M * m.width;
    B200_TRY(launch_embed(m, p, st));
    for (int i = 0; i < m.n_runs; i++) {
        const b200_hybrid_run& r = m.runs[i];
        const b200_hybrid_layer& l = m.layers[r.layer];
        const bool has_ff = l.ff > 0;
        const float* inject = r.inject && !p.dump ? m.emb : nullptr;       // rides on the run's last residual step
        const float* after_mixer = has_ff ? nullptr : inject;
        if (!m.norm_out) B200_TRY(launch_norm_conv(m, l, r, p, st));
        if (l.mixer == B200_MIXER_ATTENTION) {
            B200_TRY(product(m, p, l.in, m.hb, attention_in_epi(m, l, r, p), p.M, st));
            B200_TRY(launch_attention(m, l, r, p, st));
        } else if (l.mixer == B200_MIXER_RECURRENCE) {
            B200_TRY(product(m, p, l.in, m.hb, recurrence_in_epi(m, l, r, p), p.M, st));
            B200_TRY(launch_recurrence(m, l, r, p, st));
        } else if (l.mixer == B200_MIXER_DELTA) {
            B200_TRY(product(m, p, l.in, m.hb, delta_in_epi(m, l, r, p), p.M, st));
            B200_TRY(product(m, p, l.low, m.lowb, delta_low_epi(m, l, r, p), p.M, st));
            B200_TRY(launch_delta(m, l, r, p, st));
        } else {
            B200_TRY(latent_mixer(m, l, r, p, st));
        }
        B200_TRY(sublayer_out(m, p, l.out, m.ab, nullptr, l.norm1, after_mixer, st));
        if (has_ff) B200_TRY(feed_forward(m, l, p, inject, st));
        if (p.dump) {
            if (cudaMemcpyAsync(p.dump + i * n, m.x, n * sizeof(float), cudaMemcpyDeviceToDevice, st) != cudaSuccess) return check_launch();
            if (r.inject) B200_TRY(launch_add(m.x, m.emb, n, st));
        }
    }
    if (p.rows_out > 0) {
        B200_TRY(launch_norm(m, m.final_norm, p, true, p.rows_out, st));
        Epi e = one_seg(plain_seg(0, m.vocab, kOpSoftcap, 1, p.logits, m.vocab));
        e.cap = m.softcap;
        e.half_copy = static_cast<__half*>(p.logits16);
        B200_TRY(product(m, p, m.head, m.hb, e, p.rows_out, st));
    }
    if (!p.tree && m.conv_max_taps > 1)
        B200_TRY(launch_commit(m, p.cache, p.cache_rows, p.M < B200_HYBRID_PENDING ? p.M : B200_HYBRID_PENDING, nullptr, nullptr, 0, nullptr,
                               0, 0, st));
    return B200_OK;
}

int b200_hybrid_commit(const b200_hybrid_model* model, void* cache, int cache_rows, const int* count, const int* rows, int tree_rows,
                       const int* prefix, int compact, void* stream) {
    if (!model || !cache || !count || cache_rows < 1 || tree_rows < 1 || (compact && !prefix)) return B200_EINVAL;
    if (!model->layers || !model->runs || !model->dev_layers || !model->dev_runs || !model->pending || model->n_runs < 1) return B200_EINVAL;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    for (int i = 0; i < model->n_runs; i++) {
        const b200_hybrid_run& r = model->runs[i];
        const b200_hybrid_layer& l = model->layers[r.layer];
        if (l.mixer == B200_MIXER_DELTA) B200_TRY(launch_delta_commit(*model, l, r, cache, count, rows, tree_rows, st));
    }
    return launch_commit(*model, cache, cache_rows, 0, count, rows, tree_rows, prefix, 1, compact, st);
}

int b200_hybrid_linear(const b200_hybrid_model* model, const b200_linear* lin, const void* x, int x_pitch, int x_rows, float* y, int y_pitch,
                       int M, void* stream) {
    if (!model || !lin || !x || !y || M < 1 || x_pitch != lin->pitch || lin->groups > 1 || y_pitch < lin->n || !model->error) return B200_EINVAL;
    Epi e = one_seg(plain_seg(0, lin->n, kOpNone, 1, y, y_pitch));
    e.M = M;
    return launch_linear(model->act_type, *lin, x, 0, x_rows, e, model->error, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
