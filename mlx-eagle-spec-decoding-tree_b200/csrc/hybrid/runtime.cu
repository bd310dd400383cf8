// The pass driver: walks the layer runs and issues their launches; C entry points of libb200hybrid.so.
#include "hybrid.cuh"

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
    return launch_linear(m.act_type, lin, x, m.max_rows, e, m.error, st);
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
        if (l.taps < 1 || l.taps > B200_HYBRID_MAX_TAPS || l.heads < 1 || l.dim < 1 || l.vdim < 1 || !l.norm1 || !l.conv) return false;
        if (l.ff > 0 && !l.norm2) return false;
        if (l.mixer == B200_MIXER_ATTENTION) {
            if (l.kv_heads < 1 || l.heads % l.kv_heads || l.maps < 1 || l.maps > 2 || l.window < 1 || l.keep_first < 0) return false;
            if (!m.attn_part) return false;
        } else if (l.mixer != B200_MIXER_RECURRENCE || !l.gate_bias || !l.gate_lower || !l.head_norm) {
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

int b200_hybrid_version(void) { return 1; }
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
        if (l.dim > 256 || l.vdim > 256) return B200_ELIMIT;
    }
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const size_t n = (size_t)p.M * m.width;
    B200_TRY(launch_embed(m, p, st));
    for (int i = 0; i < m.n_runs; i++) {
        const b200_hybrid_run& r = m.runs[i];
        const b200_hybrid_layer& l = m.layers[r.layer];
        const bool has_ff = l.ff > 0;
        const float* inject = r.inject && !p.dump ? m.emb : nullptr;       // rides on the run's last residual product
        B200_TRY(launch_norm_conv(m, l, r, p, st));
        if (l.mixer == B200_MIXER_ATTENTION) {
            B200_TRY(product(m, p, l.in, m.hb, attention_in_epi(m, l, r, p), p.M, st));
            B200_TRY(launch_attention(m, l, r, p, st));
        } else {
            B200_TRY(product(m, p, l.in, m.hb, recurrence_in_epi(m, l, r, p), p.M, st));
            B200_TRY(launch_recurrence(m, l, r, p, st));
        }
        Epi e = one_seg(plain_seg(0, m.width, kOpResidual, 1, m.x, m.width));
        e.mult = m.residual_mult;
        e.add = has_ff ? nullptr : inject;
        B200_TRY(product(m, p, l.out, m.ab, e, p.M, st));
        if (has_ff) {
            B200_TRY(launch_norm(m, l.norm2, p, false, p.M, st));
            B200_TRY(product(m, p, l.up, m.hb, one_seg(plain_seg(0, l.ff, kOpNone, 0, m.zb, round_up(l.ff, 64))), p.M, st));
            B200_TRY(launch_polynorm(m, l, p.M, st));
            e.add = inject;
            B200_TRY(product(m, p, l.down, m.zab, e, p.M, st));
        }
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
    if (!model->dev_layers || !model->dev_runs || !model->pending || model->n_runs < 1) return B200_EINVAL;
    return launch_commit(*model, cache, cache_rows, 0, count, rows, tree_rows, prefix, 1, compact, static_cast<cudaStream_t>(stream));
}

int b200_hybrid_linear(const b200_hybrid_model* model, const b200_linear* lin, const void* x, int x_pitch, int x_rows, float* y, int y_pitch,
                       int M, void* stream) {
    if (!model || !lin || !x || !y || M < 1 || x_pitch != lin->pitch || y_pitch < lin->n || !model->error) return B200_EINVAL;
    Epi e = one_seg(plain_seg(0, lin->n, kOpNone, 1, y, y_pitch));
    e.M = M;
    return launch_linear(model->act_type, *lin, x, x_rows, e, model->error, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
