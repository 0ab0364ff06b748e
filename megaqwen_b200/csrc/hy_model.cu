// The layer-listed decoder: the kernel chains of one prefill portion and of one decode step,
// and the C ABI of include/megaqwen_hybrid.h.
//
// Prefill, per layer run:  input projection (segments) -> mixer -> output projection (fp32 planes)
//                          -> residual sum + what the next product reads.
// Decode, per layer run:   input projection (with the norms before it) -> mixer -> output projection.
// In the parallel form mixer and feed-forward read the same norm, so their input projections are one product, and so
// are their output projections (over the concatenation), which add to the residual stream.
// In the post-norm form they follow one another; each result is normed before it is added, which needs the whole
// result: prefill does it in the row kernel behind the product, decode in the head of the next product, where
// every CTA recomputes the sum it is about to read and CTA 0 stores it.
#include <vector>

#include "../../include/megaqwen_b200.h"
#include "hy_common.cuh"

namespace mq {
namespace hy {

static int seg_up(int n) { return (n + MQH_SEGMENT - 1) / MQH_SEGMENT * MQH_SEGMENT; }
static int up256(int n) { return (n + 255) / 256 * 256; }

struct Run { int layer; bool first; };      // first: the pass through the looped stretch begins here
static void list_runs(const MqhModel* m, std::vector<Run>* out) {
    const bool loop = m->loop_times > 0;
    const int a = loop ? m->loop_start : 0, b = loop ? m->loop_stop : 0;
    for (int i = 0; i < a; ++i) out->push_back({i, false});
    for (int t = 0; t < (loop ? m->loop_times : 0); ++t)
        for (int i = a; i < b; ++i) out->push_back({i, i == a});
    for (int i = b; i < m->num_layers; ++i) out->push_back({i, false});
}
static int hv_of(const MqhLayer& l) { return l.heads * l.vdim; }
// columns of w_out and of the buffer before it
static int cat_of(const MqhLayer& l, int form) { return hv_of(l) + (form == MQH_PARALLEL ? l.ff : 0); }
static int up16(int n) { return (n + 15) / 16 * 16; }
static int kv_dim(const MqhLayer& l) { return l.kv_heads * l.dim; }
static int conv_channels(const MqhLayer& l) { return hv_of(l) + 2 * kv_dim(l); }
static bool is_recurrent(const MqhLayer& l) { return l.kind == MQH_LIGHTNING || l.kind == MQH_GLA || l.kind == MQH_MAMBA2; }
static int decay_mode(const MqhLayer& l) { return l.kind == MQH_GLA ? DECAY_CHANNEL : l.kind == MQH_MAMBA2 ? DECAY_HEAD : DECAY_CONST; }

static bool mult16(int n) { return n > 0 && n % 16 == 0; }
static int check_layer(const MqhLayer& l, int form) {
    if (l.kind < MQH_LIGHTNING || l.kind > MQH_ATTENTION) return MQ_ERR_UNSUPPORTED;
    if (l.heads <= 0 || !mult16(l.dim) || !mult16(l.vdim) || l.ff < 0 || l.ff % 16 || l.mix_norm_n <= 0) return MQ_ERR_BAD_ARG;
    if (!l.norm || !l.w_in || !l.w_out) return MQ_ERR_BAD_ARG;
    if (form == MQH_POST_NORM && l.ff > 0 && (!l.norm2 || !l.w_gu || !l.w_down)) return MQ_ERR_BAD_ARG;
    if (is_recurrent(l) && (!l.mix_norm || l.norm_parts <= 0 || l.vdim_n <= 0 || l.vdim_n > l.vdim)) return MQ_ERR_BAD_ARG;
    if (is_recurrent(l) && (long long)l.norm_parts * l.mix_norm_n != (long long)l.heads * l.vdim_n) return MQ_ERR_BAD_ARG;
    switch (l.kind) {
    case MQH_LIGHTNING: return l.decay_pow ? (l.dim <= 512 ? MQ_OK : MQ_ERR_UNSUPPORTED) : MQ_ERR_BAD_ARG;
    case MQH_GLA: return mult16(l.rank) && l.gate_w && l.gate_b ? (l.dim <= 512 ? MQ_OK : MQ_ERR_UNSUPPORTED) : MQ_ERR_BAD_ARG;
    case MQH_MAMBA2:
        if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.conv <= 0 || !l.conv_w || !l.conv_b || !l.dt_bias || !l.a_neg || !l.skip) return MQ_ERR_BAD_ARG;
        return l.dim <= 512 && l.conv <= CONV_MAX_TAPS ? MQ_OK : MQ_ERR_UNSUPPORTED;
    case MQH_ATTENTION:
        if (l.kv_heads <= 0 || l.heads % l.kv_heads || l.vdim != l.dim || l.rot < 0 || l.rot % 2 || l.rot > l.dim || l.chunk < 0) return MQ_ERR_BAD_ARG;
        return l.q_norm && l.k_norm && (l.rope || !l.rot) ? (l.dim <= 512 ? MQ_OK : MQ_ERR_UNSUPPORTED) : MQ_ERR_BAD_ARG;
    default: break;
    }
    if (!l.mix_norm || !mult16(l.rank) || !mult16(l.rot) || !l.w_ukv || !l.w_uk_t || !l.rope) return MQ_ERR_BAD_ARG;
    return l.rank <= 2048 && l.vdim <= 512 ? MQ_OK : MQ_ERR_UNSUPPORTED;
}
static int check_model(const MqhModel* m) {
    if (!m || !m->layers || m->num_layers <= 0 || (m->dtype != MQH_BF16 && m->dtype != MQH_F32)) return MQ_ERR_BAD_ARG;
    if (!mult16(m->width) || m->norm_n <= 0 || m->vocab <= 0 || m->max_seq <= 0 || !m->embed || !m->head || !m->final_norm) return MQ_ERR_BAD_ARG;
    if ((m->form != MQH_PARALLEL && m->form != MQH_POST_NORM) || (m->form == MQH_POST_NORM && m->loop_times > 0)) return MQ_ERR_UNSUPPORTED;
    if (m->loop_times < 0 || (m->loop_times > 0 && (!m->w_loop || m->loop_start < 0 || m->loop_stop > m->num_layers || m->loop_start >= m->loop_stop)))
        return MQ_ERR_BAD_ARG;
    for (int i = 0; i < m->num_layers; ++i) {
        const int rc = check_layer(m->layers[i], m->form);
        if (rc) return rc;
    }
    return MQ_OK;
}

// ---------------------------------------------------------------- workspace
constexpr int MAX_PLANES = 4;
template <typename T>
struct Work {
    // residual stream [P, width]; parallel form: y the other one where a product may not overwrite its input, x0 the embedding;
    // post-norm form: y the result that is still to be normed, x0 the other residual stream
    float *x, *y, *x0;
    T *xin, *h;                     // [P, 2 width], [P, width]
    float* planes;                  // [MAX_PLANES][P][width rounded up to 256]
    T* cat;                         // [P, cat_of], or the feed-forward's activations [P, ff]
    T *a, *b, *c, *g;               // lightning, gla q, k, v, g / latent q unrotated, q rotated / attention q, k / mamba2 x|B|C before and after
                                    // the convolution, -, z
    float *down, *o;                // latent [P, rank + rot], gla low-rank decay input, mamba2 dt, attention gate; recurrences [P, heads*vdim]
    T *kx, *vx;                     // expanded keys, values [max_seq, ..]
    void* scratch;                  // chunk states
    T* qcat;
    float* parts;
    unsigned long long* slot;
    unsigned int* ticket;
    size_t bytes;
};
template <typename T>
static Work<T> carve(const MqhModel* m, void* base, int P) {
    Work<T> w;
    size_t off = 0;
    auto take = [&](size_t bytes) {
        uint8_t* p = reinterpret_cast<uint8_t*>(base) + off;
        off += (bytes + 255) / 256 * 256;
        return (void*)p;
    };
    size_t a = 0, b = 0, c = 0, g = 0, down = 0, o = 0, cat = 0, kx = 0, vx = 0, scr = 0, qcat = 0, parts = 0;
    auto grow = [](size_t& v, size_t n) { if (n > v) v = n; };
    for (int i = 0; i < m->num_layers; ++i) {
        const MqhLayer& l = m->layers[i];
        grow(cat, cat_of(l, m->form));
        grow(cat, l.ff);
        if (is_recurrent(l)) {
            grow(g, hv_of(l)); grow(o, hv_of(l));
            if (m->dtype == MQH_BF16) grow(scr, recurrence_scratch_bytes(P, l.heads, l.dim, l.vdim));
            if (l.kind == MQH_MAMBA2) {
                grow(a, conv_channels(l)); grow(b, conv_channels(l));
                grow(down, up16(l.heads));
            } else {
                grow(a, (size_t)l.heads * l.dim); grow(b, (size_t)l.heads * l.dim); grow(c, hv_of(l));
                if (l.kind == MQH_GLA) grow(down, l.rank);
            }
        } else if (l.kind == MQH_ATTENTION) {
            grow(a, (size_t)l.heads * l.dim); grow(b, kv_dim(l));
            grow(down, up16(l.heads));
        } else {
            grow(a, (size_t)l.heads * l.dim);
            grow(b, (size_t)l.heads * l.rot);
            grow(down, l.rank + l.rot);
            grow(kx, (size_t)l.heads * l.dim); grow(vx, hv_of(l));
            grow(qcat, (size_t)((l.heads + 15) / 16 * 16) * (l.rank + l.rot));
            grow(parts, latent_parts_floats(l.heads, l.rank, m->max_seq));
        }
    }
    const size_t p = P, W = m->width, t = sizeof(T);
    w.x = (float*)take(p * W * 4); w.y = (float*)take(p * W * 4); w.x0 = (float*)take(p * W * 4);
    w.xin = (T*)take(p * 2 * W * t); w.h = (T*)take(p * W * t);
    w.planes = (float*)take((size_t)MAX_PLANES * p * up256(m->width) * 4);
    w.cat = (T*)take(p * cat * t);
    w.a = (T*)take(p * a * t); w.b = (T*)take(p * b * t); w.c = (T*)take(p * c * t); w.g = (T*)take(p * g * t);
    w.down = (float*)take(p * down * 4); w.o = (float*)take(p * o * 4);
    w.kx = (T*)take((size_t)m->max_seq * kx * t); w.vx = (T*)take((size_t)m->max_seq * vx * t);
    w.scratch = take(scr);
    w.qcat = (T*)take(qcat * t);
    w.parts = (float*)take(parts * 4);
    w.slot = (unsigned long long*)take(8);
    w.ticket = (unsigned int*)take(4);
    w.bytes = off;
    return w;
}

// segments of a layer's input projection; one row of the outputs follows the other in each buffer
template <typename T>
static Segments in_segments(const MqhLayer& l, int form, const Work<T>& w) {
    Segments g = {};
    int row = 0;
    auto add = [&](void* out, int rows_, int ld, int act, int f32, const float* bias = nullptr) {
        g.s[g.n++] = {out, row, rows_, ld, (short)act, (short)f32, bias};
        row += seg_up(rows_);
    };
    const int hd = l.heads * l.dim, hv = hv_of(l), kd = kv_dim(l), h16 = up16(l.heads);
    switch (l.kind) {
    case MQH_LIGHTNING:
    case MQH_GLA: {
        const int act = l.kind == MQH_LIGHTNING ? ACT_SILU : ACT_NONE;
        add(w.a, hd, hd, act, 0);
        add(w.b, hd, hd, act, 0);
        add(w.c, hv, hv, act, 0);
        add(w.g, hv, hv, ACT_NONE, 0);
        if (l.kind == MQH_GLA) add(w.down, l.rank, l.rank, ACT_NONE, 1);
        break;
    }
    case MQH_MAMBA2:
        add(w.g, hv, hv, ACT_NONE, 0);
        add(w.a, hv, conv_channels(l), ACT_NONE, 0);
        add(w.a + hv, kd, conv_channels(l), ACT_NONE, 0);
        add(w.a + hv + kd, kd, conv_channels(l), ACT_NONE, 0);
        add(w.down, h16, h16, ACT_NONE, 1);
        break;
    case MQH_ATTENTION:
        add(w.a, hd, hd, ACT_NONE, 0, l.q_bias);
        add(w.b, kd, kd, ACT_NONE, 0, l.k_bias);
        add(w.down, h16, h16, ACT_NONE, 1);
        break;
    default:
        add(w.a, hd, hd, ACT_NONE, 0);
        add(w.b, l.heads * l.rot, l.heads * l.rot, ACT_NONE, 0);
        add(w.down, l.rank + l.rot, l.rank + l.rot, ACT_NONE, 1);
    }
    if (form == MQH_PARALLEL && l.ff > 0) add(w.cat + hv, 2 * l.ff, cat_of(l, form), ACT_SWIGLU, 0);
    return g;
}
static int in_rows(const MqhLayer& l, int form) {
    Work<float> none = {};
    const Segments g = in_segments<float>(l, form, none);
    return g.s[g.n - 1].row0 + seg_up(g.s[g.n - 1].rows);
}
template <typename T>
static Segments ff_segments(const MqhLayer& l, const Work<T>& w) {
    Segments g = {};
    g.n = 1;
    g.s[0] = {w.cat, 0, 2 * l.ff, l.ff, ACT_SWIGLU, 0, nullptr};
    return g;
}
static int ukv_rows(const MqhLayer& l) { return l.kind == MQH_LATENT ? seg_up(l.heads * l.dim) + seg_up(hv_of(l)) : 0; }

// parameters of a layer's recurrence; the caller adds the tensors
static RecurrenceArgs recurrence_of(const MqhLayer& l, float* state, int n) {
    RecurrenceArgs r = {};
    r.mode = decay_mode(l);
    r.n = n; r.heads = l.heads; r.dim = l.dim; r.vdim = l.vdim;
    r.kv_heads = l.kind == MQH_MAMBA2 ? l.kv_heads : l.heads;
    r.scale = l.kind == MQH_GLA ? l.scale : 1.0f;
    r.state = state;
    r.decay_pow = l.decay_pow;
    r.dt_bias = l.dt_bias; r.a_neg = l.a_neg; r.skip = l.skip;
    r.gate_w = l.gate_w; r.gate_b = l.gate_b; r.rank = l.rank; r.inv_tau = l.inv_tau;
    r.ldq = r.ldk = r.kv_heads * l.dim;
    r.ldv = hv_of(l);
    return r;
}
static size_t matrix_state_bytes(const MqhLayer& l) { return (size_t)l.heads * l.dim * l.vdim * sizeof(float); }
template <typename T>
static RecurrenceArgs recurrence_args(const MqhLayer& l, const Work<T>& w, void* state, int n) {
    RecurrenceArgs r = recurrence_of(l, (float*)state, n);
    r.o = w.o; r.scratch = w.scratch;
    r.decay_in = w.down;
    r.ld_decay = l.kind == MQH_MAMBA2 ? up16(l.heads) : l.rank;
    if (l.kind == MQH_MAMBA2) {
        r.v = w.b; r.k = w.b + hv_of(l); r.q = w.b + hv_of(l) + kv_dim(l);
        r.ldq = r.ldk = r.ldv = conv_channels(l);
    } else {
        r.q = w.a; r.k = w.b; r.v = w.c;
    }
    return r;
}
template <typename T>
static GatedNorm gated_args(const MqhLayer& l, const Work<T>& w, float eps) {
    return {w.o, l.mix_norm, w.g, hv_of(l), l.vdim, l.vdim_n, l.norm_parts, l.mix_norm_n,
            (short)(l.kind == MQH_LIGHTNING ? GATE_SIGMOID : GATE_SILU), (short)(l.kind == MQH_MAMBA2), eps};
}
static HeadNorm head_norm(const MqhLayer& l, const float* w, float eps) { return {w, l.mix_norm_n, l.dim, l.rot / 2, eps, l.rope}; }
// the caches of an attention run: keys, then values, a row per position
template <typename T>
static T* value_cache(const MqhModel* m, const MqhLayer& l, void* state) { return (T*)state + (size_t)m->max_seq * kv_dim(l); }

// From this many tokens on the chunked form of the recurrence is used.
constexpr int CHUNKED_FROM = 16;

// ---------------------------------------------------------------- prefill
#define MQH_TRY(expr) do { const int rc_ = (expr); if (rc_) return rc_; } while (0)

template <typename T>
static int mix_tokens(Stream& st, const MqhModel* m, const MqhLayer& l, const Work<T>& w, void* state, int n, int pos0, unsigned int* status) {
    const int hv = hv_of(l), ldc = cat_of(l, m->form);
    if (is_recurrent(l)) {
        const RecurrenceArgs a = recurrence_args(l, w, state, n);
        if (l.kind == MQH_MAMBA2)
            MQH_TRY(conv_rows<T>(st, w.a, l.conv_w, l.conv_b, (T*)((uint8_t*)state + matrix_state_bytes(l)), w.b, n, pos0, conv_channels(l), l.conv));
        if (m->dtype == MQH_BF16 && n >= CHUNKED_FROM && recurrence_chunked_fits(a.mode, l.dim)) MQH_TRY(recurrence_chunked(st, a));
        else MQH_TRY(recurrence_tokens<T>(st, a));
        return gated_norm<T>(st, n, gated_args(l, w, m->eps), w.cat, ldc);
    }
    if (l.kind == MQH_ATTENTION) {
        const int kd = kv_dim(l);
        T* vc = value_cache<T>(m, l, state);
        MQH_TRY(attn_rows<T>(st, {w.a, w.b, state, vc, head_norm(l, l.q_norm, m->eps), head_norm(l, l.k_norm, m->eps), n, pos0, l.heads, l.kv_heads}));
        const CausalArgs a = {w.a, nullptr, state, nullptr, vc, nullptr, w.cat, 0, ldc, n, pos0, l.heads, l.dim, 0, l.vdim, l.scale, status,
                              l.kv_heads, kd, kd, l.chunk, w.down, up16(l.heads)};
        if (m->dtype == MQH_BF16 && causal_tc_fits(l.dim, 0, l.vdim, l.scale)) return causal_tc(st, a);
        return causal_simt<T>(st, a);
    }
    const int D = l.rank + l.rot, keys = pos0 + n, hd = l.heads * l.dim;
    MQH_TRY(latent_rows<T>(st, {w.down, l.mix_norm, l.mix_norm_n, m->eps, l.rope, state, w.b, n, pos0, l.heads, l.rank, l.rot, m->max_seq}));
    Segments g = {};
    g.n = 2;
    g.s[0] = {w.kx, 0, hd, hd, ACT_NONE, 0, nullptr};
    g.s[1] = {w.vx, seg_up(hd), hv, hv, ACT_NONE, 0, nullptr};
    MQH_TRY(linear_segments<T>(st, (const T*)state, D, (const T*)l.w_ukv, keys, ukv_rows(l), l.rank, g, status));
    const CausalArgs a = {w.a, w.b, w.kx, (const T*)state + l.rank, w.vx, l.sink, w.cat, D, ldc, n, pos0, l.heads, l.dim, l.rot, l.vdim, l.scale, status,
                          l.heads, hd, hv, 0, nullptr, 0};
    if (m->dtype == MQH_BF16 && causal_tc_fits(l.dim, l.rot, l.vdim, l.scale)) return causal_tc(st, a);
    return causal_simt<T>(st, a);
}

template <typename T>
static int head_of(Stream& st, const MqhModel* m, const Work<T>& w, const float* x, const float* post_y, const float* post, float* logits, int* out_token,
                   unsigned int* status) {
    GemvArgs a = {};
    a.post_y = post_y; a.post = post;
    a.W = m->head; a.rows = m->vocab; a.K = m->width;
    a.x = x; a.gain = m->final_norm; a.eps = m->eps; a.norm_n = m->norm_n;
    a.logits = logits; a.slot = w.slot; a.ticket = w.ticket; a.out_token = out_token; a.status = status;
    return gemv<T>(st, post_y ? VEC_POST_NORM : VEC_NORM, OUT_HEAD, a);
}

template <typename T>
static int prefill(const MqhModel* m, const MqhBuffers* buf, const int* ids, int n, int pos0, const int* want_rows, int n_want, int* out_token,
                   float* logits, int* launches, cudaStream_t stream) {
    const Work<T> w = carve<T>(m, buf->workspace, buf->max_tokens);
    if (w.bytes > buf->workspace_bytes) return MQ_ERR_TOO_LONG;
    std::vector<Run> runs;
    list_runs(m, &runs);
    const int W = m->width, ldp = up256(W);
    Stream st = {stream, false, 0};         // the first kernel waits for everything before it on the stream
    RowsArgs r = {};
    r.eps = m->eps; r.norm_n = m->norm_n; r.width = W; r.status = buf->status;
    r.planes = w.planes; r.ldp = ldp; r.plane_stride = (size_t)n * ldp;
    // what run `i` reads first: the loop's input before a pass, its own norm otherwise
    auto next = [&](RowsArgs& q, size_t i) {
        q.gain = nullptr; q.xin = nullptr; q.x0_in = nullptr; q.h = nullptr;
        if (i >= runs.size()) return;
        if (m->form == MQH_POST_NORM) { q.h = w.h; return; }       // the product reads the residual stream itself
        if (runs[i].first) { q.xin = w.xin; q.x0_in = q.ids ? nullptr : w.x0; }
        else { q.gain = m->layers[runs[i].layer].norm; q.h = w.h; }
    };
    RowsArgs e = r;
    e.ids = ids; e.embed = m->embed; e.embed_scale = m->embed_scale; e.vocab = m->vocab; e.x = w.x; e.x0 = w.x0; e.nplanes = 0;
    next(e, 0);
    MQH_TRY(rows<T>(st, n, e));
    st.pdl = true;
    for (size_t i = 0; i < runs.size(); ++i) {
        const MqhLayer& l = m->layers[runs[i].layer];
        if (runs[i].first) {
            int np = MAX_PLANES;
            MQH_TRY(linear_planes<T>(st, w.xin, 2 * W, (const T*)m->w_loop, w.planes, n, W, 2 * W, ldp, &np, buf->status));
            RowsArgs q = r;
            q.nplanes = np; q.mult = 1.0f; q.x = w.x; q.gain = l.norm; q.h = w.h;
            MQH_TRY(rows<T>(st, n, q));
        }
        MQH_TRY(linear_segments<T>(st, w.h, W, (const T*)l.w_in, n, in_rows(l, m->form), W, in_segments(l, m->form, w), buf->status));
        MQH_TRY(mix_tokens<T>(st, m, l, w, buf->run_state[i], n, pos0, buf->status));
        const int cat = cat_of(l, m->form);
        int np = MAX_PLANES;
        MQH_TRY(linear_planes<T>(st, w.cat, cat, (const T*)l.w_out, w.planes, n, W, cat, ldp, &np, buf->status));
        RowsArgs q = r;
        q.base = w.x; q.nplanes = np; q.mult = m->residual_mult; q.x = w.x;
        if (m->form == MQH_POST_NORM) q.post = l.norm;
        if (m->form == MQH_POST_NORM && l.ff > 0) {
            q.h = w.h;
            MQH_TRY(rows<T>(st, n, q));
            MQH_TRY(linear_segments<T>(st, w.h, W, (const T*)l.w_gu, n, seg_up(2 * l.ff), W, ff_segments(l, w), buf->status));
            np = MAX_PLANES;
            MQH_TRY(linear_planes<T>(st, w.cat, l.ff, (const T*)l.w_down, w.planes, n, W, l.ff, ldp, &np, buf->status));
            q.nplanes = np; q.post = l.norm2;
        }
        next(q, i + 1);
        MQH_TRY(rows<T>(st, n, q));
    }
    if (n_want > 0) {
        RowsArgs q = r;
        q.base = w.x; q.nplanes = 0; q.gather = want_rows; q.gather_max = n - 1; q.gain = m->final_norm; q.h = w.h;
        MQH_TRY(rows<T>(st, n_want, q));
        int np = 1;
        MQH_TRY(linear_planes<T>(st, w.h, W, (const T*)m->head, logits, n_want, m->vocab, W, up256(m->vocab), &np, buf->status));
    }
    MQH_TRY(head_of<T>(st, m, w, w.x + (size_t)(n - 1) * W, nullptr, nullptr, nullptr, out_token, buf->status));
    if (launches) *launches = st.launches;
    return (int)cudaGetLastError();
}

// ---------------------------------------------------------------- decode
// the mixer of one token between its input and its output projection; what the latter's vector is made of goes to `b`, *vec
template <typename T>
static int mix_one(Stream& st, const MqhModel* m, const MqhLayer& l, const Work<T>& w, void* state, const int* position, unsigned int* status, GemvArgs& b,
                   int* vec) {
    b.cat = w.cat;
    *vec = VEC_PLAIN;
    if (is_recurrent(l)) {
        RecurrenceArgs r = recurrence_args(l, w, state, 1);
        if (l.kind == MQH_MAMBA2) {
            r.position = position; r.max_seq = m->max_seq; r.status = status;
            r.conv_in = w.a; r.conv_state = (uint8_t*)state + matrix_state_bytes(l);
            r.conv_w = l.conv_w; r.conv_b = l.conv_b; r.taps = l.conv; r.channels = conv_channels(l);
        }
        b.gn = gated_args(l, w, m->eps);
        *vec = l.norm_parts == 1 ? VEC_GATED : VEC_GATED_PARTS;
        return recurrence_tokens<T>(st, r);
    }
    if (l.kind == MQH_ATTENTION)
        return attn_decode<T>(st, {w.a, w.b, w.down, state, value_cache<T>(m, l, state), head_norm(l, l.q_norm, m->eps), head_norm(l, l.k_norm, m->eps),
                                   position, w.cat, l.heads, l.kv_heads, m->max_seq, l.chunk, l.scale, status});
    return latent_decode<T>(st, {w.a, w.b, w.down, l.mix_norm, l.mix_norm_n, m->eps, l.rope, position, state, l.w_uk_t,
                                 (const T*)l.w_ukv + (size_t)seg_up(l.heads * l.dim) * l.rank, l.sink, w.qcat, w.parts, w.cat, l.heads,
                                 l.dim, l.rot, l.vdim, l.rank, m->max_seq, l.scale, status});
}

template <typename T>
static int decode(const MqhModel* m, const MqhBuffers* buf, const int* in_token, int* out_token, const int* position, float* logits, int flags,
                  cudaStream_t stream) {
    const Work<T> w = carve<T>(m, buf->workspace, buf->max_tokens);
    if (w.bytes > buf->workspace_bytes) return MQ_ERR_TOO_LONG;
    std::vector<Run> runs;
    list_runs(m, &runs);
    const bool pdl = !(flags & MQ_FLAG_NO_PDL), post = m->form == MQH_POST_NORM;
    Stream st = {stream, pdl && (flags & MQ_FLAG_CHAINED), 0};
    const int W = m->width;
    float *x = w.x, *y = post ? w.x0 : w.y;     // y: the other residual stream
    GemvArgs base = {};
    base.eps = m->eps; base.norm_n = m->norm_n; base.status = buf->status; base.vocab = m->vocab; base.embed = m->embed; base.embed_scale = m->embed_scale;
    const float* pending = nullptr;             // post-norm: gain of the result in w.y that the residual stream still lacks
    // post-norm: a product that reads the residual stream completes it first
    auto complete = [&](GemvArgs& a) {
        a.x = x; a.x_store = y;
        if (pending) { a.post_y = w.y; a.post = pending; }
        float* t = x; x = y; y = t;
    };
    for (size_t i = 0; i < runs.size(); ++i) {
        const MqhLayer& l = m->layers[runs[i].layer];
        const bool embed = i == 0;          // the first product of the step looks the token up itself
        if (runs[i].first) {
            GemvArgs a = base;
            a.W = m->w_loop; a.rows = W; a.K = 2 * W; a.x = x; a.x0 = w.x0; a.y = y;
            if (embed) { a.token = in_token; a.x0_store = w.x0; }
            MQH_TRY(gemv<T>(st, VEC_CONCAT, OUT_STORE, a));
            st.pdl = pdl;
            float* t = x; x = y; y = t;
        }
        GemvArgs a = base;
        a.W = l.w_in; a.rows = in_rows(l, m->form); a.K = W; a.seg = in_segments(l, m->form, w);
        if (post) {
            complete(a);
            if (embed) a.token = in_token;
            MQH_TRY(gemv<T>(st, VEC_POST, OUT_SEGMENTS, a));
        } else {
            a.x = x; a.gain = l.norm;
            if (embed && !runs[i].first) { a.token = in_token; a.x_store = x; a.x0_store = w.x0; }
            MQH_TRY(gemv<T>(st, VEC_NORM, OUT_SEGMENTS, a));
        }
        st.pdl = pdl;
        GemvArgs b = base;
        int vec = VEC_PLAIN;
        MQH_TRY(mix_one<T>(st, m, l, w, buf->run_state[i], position, buf->status, b, &vec));
        b.W = l.w_out; b.rows = W; b.K = cat_of(l, m->form); b.y = post ? w.y : x; b.mult = m->residual_mult;
        MQH_TRY(gemv<T>(st, vec, post ? OUT_STORE : OUT_ADD, b));
        if (!post) continue;
        pending = l.norm;
        if (l.ff > 0) {
            GemvArgs f = base;
            f.W = l.w_gu; f.rows = seg_up(2 * l.ff); f.K = W; f.seg = ff_segments(l, w);
            complete(f);
            MQH_TRY(gemv<T>(st, VEC_POST, OUT_SEGMENTS, f));
            GemvArgs d = base;
            d.W = l.w_down; d.rows = W; d.K = l.ff; d.cat = w.cat; d.y = w.y;
            MQH_TRY(gemv<T>(st, VEC_PLAIN, OUT_STORE, d));
            pending = l.norm2;
        }
    }
    MQH_TRY(head_of<T>(st, m, w, x, post ? w.y : nullptr, pending, logits, out_token, buf->status));
    return (int)cudaGetLastError();
}

static bool misaligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 255u) != 0; }
static int check_call(const MqhModel* m, const MqhBuffers* buf) {
    const int rc = check_model(m);
    if (rc) return rc;
    if (!buf || !buf->workspace || !buf->run_state || !buf->status || buf->max_tokens <= 0) return MQ_ERR_BAD_ARG;
    if (misaligned(buf->workspace)) return MQ_ERR_ALIGNMENT;
    const int n = mqh_run_count(m);
    for (int i = 0; i < n; ++i) {
        if (!buf->run_state[i]) return MQ_ERR_BAD_ARG;
        if (misaligned(buf->run_state[i])) return MQ_ERR_ALIGNMENT;
    }
    return MQ_OK;
}

}  // namespace hy
}  // namespace mq

using namespace mq;
using namespace mq::hy;

extern "C" int mqh_run_count(const MqhModel* m) {
    if (!m) return 0;
    std::vector<Run> runs;
    list_runs(m, &runs);
    return (int)runs.size();
}
extern "C" int mqh_run_layer(const MqhModel* m, int run) {
    if (!m) return -1;
    std::vector<Run> runs;
    list_runs(m, &runs);
    return run >= 0 && run < (int)runs.size() ? runs[run].layer : -1;
}
extern "C" size_t mqh_state_bytes(const MqhModel* m, int run) {
    const int i = mqh_run_layer(m, run);
    if (i < 0) return 0;
    const MqhLayer& l = m->layers[i];
    const size_t elem = m->dtype == MQH_BF16 ? sizeof(bf16) : sizeof(float);
    if (l.kind == MQH_MAMBA2) return matrix_state_bytes(l) + (size_t)l.conv * conv_channels(l) * elem;
    if (is_recurrent(l)) return matrix_state_bytes(l);
    if (l.kind == MQH_ATTENTION) return (size_t)m->max_seq * 2 * kv_dim(l) * elem;
    return (size_t)m->max_seq * (l.rank + l.rot) * elem;
}
extern "C" int mqh_state_recurrent(const MqhModel* m, int run) {
    const int i = mqh_run_layer(m, run);
    return i >= 0 && is_recurrent(m->layers[i]);
}
extern "C" int mqh_in_rows(const MqhLayer* l, int form) { return l ? in_rows(*l, form) : 0; }
extern "C" int mqh_ukv_rows(const MqhLayer* l) { return l ? ukv_rows(*l) : 0; }
extern "C" size_t mqh_workspace_bytes(const MqhModel* m, int max_tokens) {
    if (check_model(m) || max_tokens <= 0) return 0;
    return m->dtype == MQH_BF16 ? carve<bf16>(m, nullptr, max_tokens).bytes : carve<float>(m, nullptr, max_tokens).bytes;
}
extern "C" int mqh_logits_ld(const MqhModel* m) { return m ? up256(m->vocab) : 0; }
extern "C" int mqh_decode_launch_count(const MqhModel* m) {
    if (!m) return 0;
    std::vector<Run> runs;
    list_runs(m, &runs);
    int n = 1;
    for (const Run& r : runs) {
        const MqhLayer& l = m->layers[r.layer];
        n += (r.first ? 1 : 0) + (l.kind == MQH_LATENT ? 5 : 3) + (m->form == MQH_POST_NORM && l.ff > 0 ? 2 : 0);
    }
    return n;
}
extern "C" int mqh_launch_decode(const MqhModel* m, const MqhBuffers* buf, const int* in_token, int* out_token, const int* position, float* logits,
                                 int flags, void* stream) {
    const int rc = check_call(m, buf);
    if (rc) return rc;
    if (!in_token || !out_token || !position) return MQ_ERR_BAD_ARG;
    return m->dtype == MQH_BF16 ? decode<bf16>(m, buf, in_token, out_token, position, logits, flags, (cudaStream_t)stream)
                                : decode<float>(m, buf, in_token, out_token, position, logits, flags, (cudaStream_t)stream);
}
extern "C" int mqh_launch_prefill(const MqhModel* m, const MqhBuffers* buf, const int* ids, int n, int pos0, const int* want_rows, int n_want,
                                  int* out_token, float* logits, int* launches, void* stream) {
    const int rc = check_call(m, buf);
    if (rc) return rc;
    if (!ids || !out_token || n <= 0 || pos0 < 0 || n_want < 0 || (n_want > 0 && (!want_rows || !logits))) return MQ_ERR_BAD_ARG;
    if (n > buf->max_tokens || n_want > n || pos0 + n > m->max_seq) return MQ_ERR_TOO_LONG;
    return m->dtype == MQH_BF16 ? prefill<bf16>(m, buf, ids, n, pos0, want_rows, n_want, out_token, logits, launches, (cudaStream_t)stream)
                                : prefill<float>(m, buf, ids, n, pos0, want_rows, n_want, out_token, logits, launches, (cudaStream_t)stream);
}

extern "C" size_t mqh_recurrence_scratch_bytes(int n, int heads, int dim, int vdim) { return recurrence_scratch_bytes(n, heads, dim, vdim); }
static int launch_recurrence(int dtype, const RecurrenceArgs& a, int chunked, void* stream) {
    if (!a.q || !a.k || !a.v || !a.state || !a.o || a.n <= 0) return MQ_ERR_BAD_ARG;
    if (chunked && (dtype != MQH_BF16 || !a.scratch)) return MQ_ERR_BAD_ARG;
    Stream st = {(cudaStream_t)stream, false, 0};
    if (chunked) return recurrence_chunked(st, a);
    return dtype == MQH_BF16 ? recurrence_tokens<bf16>(st, a) : recurrence_tokens<float>(st, a);
}
extern "C" int mqh_launch_lightning(int dtype, const void* q, const void* k, const void* v, const float* decay_pow, float* state, float* o, int n,
                                    int heads, int dim, int vdim, int chunked, void* scratch, void* stream) {
    if (!decay_pow || heads <= 0 || !mult16(dim) || !mult16(vdim)) return MQ_ERR_BAD_ARG;
    MqhLayer l = {};
    l.kind = MQH_LIGHTNING; l.heads = heads; l.dim = dim; l.vdim = vdim; l.decay_pow = decay_pow;
    RecurrenceArgs a = recurrence_of(l, state, n);
    a.q = q; a.k = k; a.v = v; a.o = o; a.scratch = scratch;
    return launch_recurrence(dtype, a, chunked, stream);
}
extern "C" int mqh_launch_recurrence(int dtype, const MqhLayer* l, const void* q, const void* k, const void* v, const float* decay_in, int ld_decay,
                                     float* state, float* o, int n, int chunked, void* scratch, void* stream) {
    if (!l || !decay_in || l->heads <= 0 || !mult16(l->dim) || !mult16(l->vdim)) return MQ_ERR_BAD_ARG;
    if (l->kind == MQH_GLA ? !l->gate_w || !l->gate_b || !mult16(l->rank) || ld_decay < l->rank || ld_decay % 4
                           : l->kind != MQH_MAMBA2 || !l->dt_bias || !l->a_neg || !l->skip || l->kv_heads <= 0 || l->heads % l->kv_heads || ld_decay < l->heads)
        return MQ_ERR_BAD_ARG;
    RecurrenceArgs a = recurrence_of(*l, state, n);
    a.q = q; a.k = k; a.v = v; a.o = o; a.scratch = scratch; a.decay_in = decay_in; a.ld_decay = ld_decay;
    return launch_recurrence(dtype, a, chunked, stream);
}
extern "C" int mqh_launch_conv(int dtype, const void* x, const float* w, const float* b, void* state, void* y, int n, int pos0, int channels, int taps,
                               void* stream) {
    if (!x || !w || !b || !state || !y || n <= 0 || pos0 < 0 || !mult16(channels) || taps <= 0) return MQ_ERR_BAD_ARG;
    Stream st = {(cudaStream_t)stream, false, 0};
    return dtype == MQH_BF16 ? conv_rows<bf16>(st, (const bf16*)x, w, b, (bf16*)state, (bf16*)y, n, pos0, channels, taps)
                             : conv_rows<float>(st, (const float*)x, w, b, (float*)state, (float*)y, n, pos0, channels, taps);
}
extern "C" int mqh_launch_causal_attention(int dtype, const void* q, const void* q_rot, const void* k, const void* k_rot, int ld_rot, const void* v,
                                           const float* sink, const float* gate, void* out, int n, int pos0, int heads, int kv_heads, int dim, int rot,
                                           int vdim, int chunk, float scale, int tensor_cores, unsigned int* status, void* stream) {
    if (!q || !k || !v || !out || !status || n <= 0 || pos0 < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || !mult16(dim) || !mult16(vdim) ||
        chunk < 0 || (rot != 0 && (!mult16(rot) || !q_rot || !k_rot)))
        return MQ_ERR_BAD_ARG;
    if (rot != 0 && (ld_rot < rot || ld_rot % 8)) return MQ_ERR_ALIGNMENT;
    Stream st = {(cudaStream_t)stream, false, 0};
    const CausalArgs a = {q, q_rot, k, k_rot, v, sink, out, ld_rot, heads * vdim, n, pos0, heads, dim, rot, vdim, scale, status,
                          kv_heads, kv_heads * dim, kv_heads * vdim, chunk, gate, heads};
    if (tensor_cores) return dtype == MQH_BF16 && causal_tc_fits(dim, rot, vdim, scale) ? causal_tc(st, a) : MQ_ERR_UNSUPPORTED;
    return dtype == MQH_BF16 ? causal_simt<bf16>(st, a) : causal_simt<float>(st, a);
}
