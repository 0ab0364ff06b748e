// The layer-listed decoder: the kernel chains of one prefill portion and of one decode step,
// and the C ABI of include/megaqwen_hybrid.h.
//
// Prefill, per layer run:  input projection (segments) -> mixer -> output projection (fp32 planes)
//                          -> residual sum + what the next product reads.
// Decode, per layer run:   norm + input projection -> mixer -> output projection + residual add.
// A layer is parallel: its mixer and its feed-forward read the same norm, so their input
// projections are one product, and so are their output projections (over the concatenation).
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
static int cat_of(const MqhLayer& l) { return hv_of(l) + l.ff; }

static bool mult16(int n) { return n > 0 && n % 16 == 0; }
static int check_layer(const MqhLayer& l) {
    if (l.kind != MQH_LIGHTNING && l.kind != MQH_LATENT) return MQ_ERR_UNSUPPORTED;
    if (l.heads <= 0 || !mult16(l.dim) || !mult16(l.vdim) || l.ff < 0 || l.ff % 16 || l.mix_norm_n <= 0) return MQ_ERR_BAD_ARG;
    if (!l.norm || !l.w_in || !l.w_out || !l.mix_norm) return MQ_ERR_BAD_ARG;
    if (l.kind == MQH_LIGHTNING) return l.decay_pow ? (l.dim <= 512 ? MQ_OK : MQ_ERR_UNSUPPORTED) : MQ_ERR_BAD_ARG;
    if (!mult16(l.rank) || !mult16(l.rot) || !l.w_ukv || !l.w_uk_t || !l.rope) return MQ_ERR_BAD_ARG;
    return l.rank <= 2048 && l.vdim <= 512 ? MQ_OK : MQ_ERR_UNSUPPORTED;
}
static int check_model(const MqhModel* m) {
    if (!m || !m->layers || m->num_layers <= 0 || (m->dtype != MQH_BF16 && m->dtype != MQH_F32)) return MQ_ERR_BAD_ARG;
    if (!mult16(m->width) || m->norm_n <= 0 || m->vocab <= 0 || m->max_seq <= 0 || !m->embed || !m->head || !m->final_norm) return MQ_ERR_BAD_ARG;
    if (m->loop_times < 0 || (m->loop_times > 0 && (!m->w_loop || m->loop_start < 0 || m->loop_stop > m->num_layers || m->loop_start >= m->loop_stop)))
        return MQ_ERR_BAD_ARG;
    for (int i = 0; i < m->num_layers; ++i) {
        const int rc = check_layer(m->layers[i]);
        if (rc) return rc;
    }
    return MQ_OK;
}

// ---------------------------------------------------------------- workspace
constexpr int MAX_PLANES = 4;
template <typename T>
struct Work {
    float *x, *y, *x0;              // residual stream [P, width]; y: the other one where a product may not overwrite its input
    T *xin, *h;                     // [P, 2 width], [P, width]
    float* planes;                  // [MAX_PLANES][P][width rounded up to 256]
    T* cat;                         // [P, heads*vdim + ff]
    T *a, *b, *c, *g;               // lightning q, k, v, g / latent q unrotated, q rotated
    float *down, *o;                // latent [P, rank + rot], lightning [P, heads*vdim]
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
        grow(cat, cat_of(l));
        grow(a, (size_t)l.heads * l.dim);
        if (l.kind == MQH_LIGHTNING) {
            grow(b, (size_t)l.heads * l.dim);
            grow(c, hv_of(l)); grow(g, hv_of(l)); grow(o, hv_of(l));
            if (m->dtype == MQH_BF16) grow(scr, lightning_scratch_bytes(P, l.heads, l.dim, l.vdim));
        } else {
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
static Segments in_segments(const MqhLayer& l, const Work<T>& w) {
    Segments g = {};
    int row = 0;
    auto add = [&](void* out, int rows_, int ld, int act, int f32) {
        g.s[g.n++] = {out, row, rows_, ld, act, f32};
        row += seg_up(rows_);
    };
    const int hd = l.heads * l.dim, hv = hv_of(l);
    if (l.kind == MQH_LIGHTNING) {
        add(w.a, hd, hd, ACT_SILU, 0);
        add(w.b, hd, hd, ACT_SILU, 0);
        add(w.c, hv, hv, ACT_SILU, 0);
        add(w.g, hv, hv, ACT_NONE, 0);
    } else {
        add(w.a, hd, hd, ACT_NONE, 0);
        add(w.b, l.heads * l.rot, l.heads * l.rot, ACT_NONE, 0);
        add(w.down, l.rank + l.rot, l.rank + l.rot, ACT_NONE, 1);
    }
    if (l.ff > 0) add(w.cat + hv, 2 * l.ff, cat_of(l), ACT_SWIGLU, 0);
    return g;
}
static int in_rows(const MqhLayer& l) {
    const int hd = l.heads * l.dim, hv = hv_of(l);
    const int mix = l.kind == MQH_LIGHTNING ? 2 * seg_up(hd) + 2 * seg_up(hv) : seg_up(hd) + seg_up(l.heads * l.rot) + seg_up(l.rank + l.rot);
    return mix + seg_up(2 * l.ff);
}
static int ukv_rows(const MqhLayer& l) { return l.kind == MQH_LATENT ? seg_up(l.heads * l.dim) + seg_up(hv_of(l)) : 0; }
template <typename T>
static LightningArgs lightning_args(const MqhLayer& l, const Work<T>& w, void* state, int n) {
    return {w.a, w.b, w.c, l.decay_pow, (float*)state, w.o, w.scratch, n, l.heads, l.dim, l.vdim};
}

// From this many tokens on the chunked form of the recurrence is used.
constexpr int CHUNKED_FROM = 16;

// ---------------------------------------------------------------- prefill
#define MQH_TRY(expr) do { const int rc_ = (expr); if (rc_) return rc_; } while (0)

template <typename T>
static int mix_tokens(Stream& st, const MqhModel* m, const MqhLayer& l, const Work<T>& w, void* state, int n, int pos0, unsigned int* status) {
    const int hv = hv_of(l), ldc = cat_of(l);
    if (l.kind == MQH_LIGHTNING) {
        const LightningArgs a = lightning_args(l, w, state, n);
        if (m->dtype == MQH_BF16 && n >= CHUNKED_FROM && lightning_chunked_fits(l.dim)) MQH_TRY(lightning_chunked(st, a));
        else MQH_TRY(lightning_tokens<T>(st, a));
        return gated_norm<T>(st, n, w.o, l.mix_norm, w.g, w.cat, ldc, hv, l.mix_norm_n, m->eps);
    }
    const int D = l.rank + l.rot, keys = pos0 + n, hd = l.heads * l.dim;
    MQH_TRY(latent_rows<T>(st, {w.down, l.mix_norm, l.mix_norm_n, m->eps, l.rope, state, w.b, n, pos0, l.heads, l.rank, l.rot, m->max_seq}));
    Segments g = {};
    g.n = 2;
    g.s[0] = {w.kx, 0, hd, hd, ACT_NONE, 0};
    g.s[1] = {w.vx, seg_up(hd), hv, hv, ACT_NONE, 0};
    MQH_TRY(linear_segments<T>(st, (const T*)state, D, (const T*)l.w_ukv, keys, ukv_rows(l), l.rank, g, status));
    const CausalArgs a = {w.a, w.b, w.kx, (const T*)state + l.rank, w.vx, l.sink, w.cat, D, ldc, n, pos0, l.heads, l.dim, l.rot, l.vdim, l.scale, status};
    if (m->dtype == MQH_BF16 && causal_tc_fits(l.dim, l.rot, l.vdim, l.scale)) return causal_tc(st, a);
    return causal_simt<T>(st, a);
}

template <typename T>
static int head_of(Stream& st, const MqhModel* m, const Work<T>& w, const float* x, float* logits, int* out_token, unsigned int* status) {
    GemvArgs a = {};
    a.W = m->head; a.rows = m->vocab; a.K = m->width;
    a.x = x; a.gain = m->final_norm; a.eps = m->eps; a.norm_n = m->norm_n;
    a.logits = logits; a.slot = w.slot; a.ticket = w.ticket; a.out_token = out_token; a.status = status;
    return gemv<T>(st, VEC_NORM, OUT_HEAD, a);
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
        q.gain = nullptr; q.xin = nullptr; q.x0_in = nullptr;
        if (i >= runs.size()) return;
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
        MQH_TRY(linear_segments<T>(st, w.h, W, (const T*)l.w_in, n, in_rows(l), W, in_segments(l, w), buf->status));
        MQH_TRY(mix_tokens<T>(st, m, l, w, buf->run_state[i], n, pos0, buf->status));
        int np = MAX_PLANES;
        MQH_TRY(linear_planes<T>(st, w.cat, cat_of(l), (const T*)l.w_out, w.planes, n, W, cat_of(l), ldp, &np, buf->status));
        RowsArgs q = r;
        q.base = w.x; q.nplanes = np; q.mult = m->residual_mult; q.x = w.x;
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
    MQH_TRY(head_of<T>(st, m, w, w.x + (size_t)(n - 1) * W, nullptr, out_token, buf->status));
    if (launches) *launches = st.launches;
    return (int)cudaGetLastError();
}

// ---------------------------------------------------------------- decode
template <typename T>
static int decode(const MqhModel* m, const MqhBuffers* buf, const int* in_token, int* out_token, const int* position, float* logits, int flags,
                  cudaStream_t stream) {
    const Work<T> w = carve<T>(m, buf->workspace, buf->max_tokens);
    if (w.bytes > buf->workspace_bytes) return MQ_ERR_TOO_LONG;
    std::vector<Run> runs;
    list_runs(m, &runs);
    const bool pdl = !(flags & MQ_FLAG_NO_PDL);
    Stream st = {stream, pdl && (flags & MQ_FLAG_CHAINED), 0};
    const int W = m->width;
    float *x = w.x, *y = w.y;
    GemvArgs base = {};
    base.eps = m->eps; base.norm_n = m->norm_n; base.status = buf->status; base.vocab = m->vocab; base.embed = m->embed; base.embed_scale = m->embed_scale;
    for (size_t i = 0; i < runs.size(); ++i) {
        const MqhLayer& l = m->layers[runs[i].layer];
        const int hv = hv_of(l), cat = cat_of(l);
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
        a.W = l.w_in; a.rows = in_rows(l); a.K = W; a.x = x; a.gain = l.norm; a.seg = in_segments(l, w);
        if (embed && !runs[i].first) { a.token = in_token; a.x_store = x; a.x0_store = w.x0; }
        MQH_TRY(gemv<T>(st, VEC_NORM, OUT_SEGMENTS, a));
        st.pdl = pdl;
        GemvArgs b = base;
        b.W = l.w_out; b.rows = W; b.K = cat; b.cat = w.cat; b.y = x; b.mult = m->residual_mult;
        if (l.kind == MQH_LIGHTNING) {
            MQH_TRY(lightning_tokens<T>(st, lightning_args(l, w, buf->run_state[i], 1)));
            b.o = w.o; b.gain = l.mix_norm; b.norm_n = l.mix_norm_n; b.g = w.g; b.hv = hv;
            MQH_TRY(gemv<T>(st, VEC_GATED, OUT_ADD, b));
        } else {
            MQH_TRY(latent_decode<T>(st, {w.a, w.b, w.down, l.mix_norm, l.mix_norm_n, m->eps, l.rope, position, buf->run_state[i], l.w_uk_t,
                                          (const T*)l.w_ukv + (size_t)seg_up(l.heads * l.dim) * l.rank, l.sink, w.qcat, w.parts, w.cat, l.heads,
                                          l.dim, l.rot, l.vdim, l.rank, m->max_seq, l.scale, buf->status}));
            MQH_TRY(gemv<T>(st, VEC_PLAIN, OUT_ADD, b));
        }
    }
    MQH_TRY(head_of<T>(st, m, w, x, logits, out_token, buf->status));
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
    if (l.kind == MQH_LIGHTNING) return (size_t)l.heads * l.dim * l.vdim * sizeof(float);
    return (size_t)m->max_seq * (l.rank + l.rot) * (m->dtype == MQH_BF16 ? sizeof(bf16) : sizeof(float));
}
extern "C" int mqh_state_recurrent(const MqhModel* m, int run) {
    const int i = mqh_run_layer(m, run);
    return i >= 0 && m->layers[i].kind == MQH_LIGHTNING;
}
extern "C" int mqh_in_rows(const MqhLayer* l) { return l ? in_rows(*l) : 0; }
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
    for (const Run& r : runs) n += (r.first ? 1 : 0) + (m->layers[r.layer].kind == MQH_LIGHTNING ? 3 : 5);
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

extern "C" size_t mqh_lightning_scratch_bytes(int n, int heads, int dim, int vdim) { return lightning_scratch_bytes(n, heads, dim, vdim); }
extern "C" int mqh_launch_lightning(int dtype, const void* q, const void* k, const void* v, const float* decay_pow, float* state, float* o, int n,
                                    int heads, int dim, int vdim, int chunked, void* scratch, void* stream) {
    if (!q || !k || !v || !decay_pow || !state || !o || n <= 0 || heads <= 0 || !mult16(dim) || !mult16(vdim)) return MQ_ERR_BAD_ARG;
    if (chunked && (dtype != MQH_BF16 || !scratch)) return MQ_ERR_BAD_ARG;
    Stream st = {(cudaStream_t)stream, false, 0};
    const LightningArgs a = {q, k, v, decay_pow, state, o, scratch, n, heads, dim, vdim};
    if (chunked) return lightning_chunked(st, a);
    return dtype == MQH_BF16 ? lightning_tokens<bf16>(st, a) : lightning_tokens<float>(st, a);
}
extern "C" int mqh_launch_causal_attention(int dtype, const void* q, const void* q_rot, const void* k, const void* k_rot, int ld_rot, const void* v,
                                           const float* sink, void* out, int n, int pos0, int heads, int dim, int rot, int vdim, float scale,
                                           int tensor_cores, unsigned int* status, void* stream) {
    if (!q || !q_rot || !k || !k_rot || !v || !out || !status || n <= 0 || pos0 < 0 || heads <= 0 || !mult16(dim) || !mult16(rot) || !mult16(vdim))
        return MQ_ERR_BAD_ARG;
    if (ld_rot < rot || ld_rot % 8) return MQ_ERR_ALIGNMENT;
    Stream st = {(cudaStream_t)stream, false, 0};
    const CausalArgs a = {q, q_rot, k, k_rot, v, sink, out, ld_rot, heads * vdim, n, pos0, heads, dim, rot, vdim, scale, status};
    if (tensor_cores) return dtype == MQH_BF16 && causal_tc_fits(dim, rot, vdim, scale) ? causal_tc(st, a) : MQ_ERR_UNSUPPORTED;
    return dtype == MQH_BF16 ? causal_simt<bf16>(st, a) : causal_simt<float>(st, a);
}
