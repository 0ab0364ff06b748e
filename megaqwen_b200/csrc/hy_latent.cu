// Latent attention: every head's keys and values are projections of one normed latent c per
// token, beside one rotated key part that all heads share; only c and that part are cached.
//
// More than one token: keys and values of all cached tokens are expanded once (a product) and
// the causal attention runs over them, on tcgen05 (tc_attention.cuh) or, for 32-bit models and
// head shapes that kernel does not hold, in k_causal_rows.
// One token: the query is carried into the latent space instead (W_uk^T q per head), so that
// scores and the weighted sum read the cache itself, once for all heads; the sum of latents is
// carried out again by W_uv.  Three kernels: k_latent_query (that product, rotations, the new
// cache row), k_latent_attention (splits of the cached tokens), k_latent_merge (sum of the splits
// with the sink, and W_uv).
// Scores, weights, rotations and norms are 32-bit; scores are kept in units of log2.
#include "hy_common.cuh"
#include "tc_attention.cuh"

namespace mq {
namespace hy {

// The interleaved rotation: elements 2i, 2i + 1 turn by the angle whose cos, sin are rope[i].
__device__ __forceinline__ float2 rotate_pair(float u, float v, float2 cs) { return make_float2(u * cs.x - v * cs.y, v * cs.x + u * cs.y); }
__device__ __forceinline__ float2 load2(const float* p) { return __ldcg(reinterpret_cast<const float2*>(p)); }
__device__ __forceinline__ float2 load2(const bf16* p) {
    const uint32_t u = ld_cg_u32(p);
    return make_float2(bf_lo(u), bf_hi(u));
}
__device__ __forceinline__ void store2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void store2(bf16* p, float2 v) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v.x, v.y); }

// acc + 16 bytes of a weight row times the vector elements at v
__device__ __forceinline__ float dot_row16(const uint4& u, const float* v, float acc, const bf16*) {
    const float4 a = load4(v), b = load4(v + 4);
    acc = fmaf(bf_lo(u.x), a.x, acc); acc = fmaf(bf_hi(u.x), a.y, acc); acc = fmaf(bf_lo(u.y), a.z, acc); acc = fmaf(bf_hi(u.y), a.w, acc);
    acc = fmaf(bf_lo(u.z), b.x, acc); acc = fmaf(bf_hi(u.z), b.y, acc); acc = fmaf(bf_lo(u.w), b.z, acc); acc = fmaf(bf_hi(u.w), b.w, acc);
    return acc;
}
__device__ __forceinline__ float dot_row16(const uint4& u, const float* v, float acc, const float*) {
    const float4 a = load4(v);
    acc = fmaf(__uint_as_float(u.x), a.x, acc); acc = fmaf(__uint_as_float(u.y), a.y, acc);
    acc = fmaf(__uint_as_float(u.z), a.z, acc); acc = fmaf(__uint_as_float(u.w), a.w, acc);
    return acc;
}

// The latent of a token from its down projection: c = rms(down[0, rank)) * norm.  NT threads of a CTA; nw: the norm weights
// of the thread's first two pairs, loaded ahead.
template <typename T, int NT>
__device__ __forceinline__ void write_latent(const float* down, const float* norm, const float2 (&nw)[2], int norm_n, float eps, T* row, int rank, float* red) {
    const int tid = threadIdx.x;
    float2 keep[2];
    float ss = 0.f;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = 2 * (tid + x * NT);
        keep[x] = i < rank ? load2(down + i) : make_float2(0.f, 0.f);
        ss += keep[x].x * keep[x].x + keep[x].y * keep[x].y;
    }
    for (int i = 2 * (tid + 2 * NT); i < rank; i += 2 * NT) {
        const float2 v = load2(down + i);
        ss += v.x * v.x + v.y * v.y;
    }
    const float inv = 1.0f / sqrtf(cta_sum<NT / 32>(ss, red) / (float)norm_n + eps);
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = 2 * (tid + x * NT);
        if (i < rank) store2(row + i, make_float2(keep[x].x * inv * nw[x].x, keep[x].y * inv * nw[x].y));
    }
    for (int i = 2 * (tid + 2 * NT); i < rank; i += 2 * NT) {
        const float2 v = load2(down + i);
        store2(row + i, make_float2(v.x * inv * norm[i], v.y * inv * norm[i + 1]));
    }
}

// ---------------------------------------------------------------- several tokens
template <typename T>
__global__ void __launch_bounds__(128) k_latent_rows(LatentRowsArgs a) {
    pdl_trigger();
    __shared__ float red[4];
    const int t = blockIdx.x, tid = threadIdx.x, pos = a.pos0 + t, D = a.rank + a.rot;
    const float2* rope = reinterpret_cast<const float2*>(a.rope + (size_t)pos * a.rot);
    float2 nw[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = 2 * (tid + x * 128);
        nw[x] = i < a.rank ? *reinterpret_cast<const float2*>(a.norm + i) : make_float2(0.f, 0.f);
    }
    pdl_wait();
    T* q = reinterpret_cast<T*>(a.q_rot) + (size_t)t * a.heads * a.rot;
    T* row = reinterpret_cast<T*>(a.cache) + (size_t)pos * D;
    const float* down = a.down + (size_t)t * D;
    const int half = a.rot / 2;
    for (int x = tid; x < a.heads * half; x += 128) {
        const float2 v = load2(q + 2 * x);
        store2(q + 2 * x, rotate_pair(v.x, v.y, rope[x % half]));
    }
    for (int i = tid; i < half; i += 128) {
        const float2 v = load2(down + a.rank + 2 * i);
        store2(row + a.rank + 2 * i, rotate_pair(v.x, v.y, rope[i]));
    }
    write_latent<T, 128>(down, a.norm, nw, a.norm_n, a.eps, row, a.rank, red);
}
template <typename T>
int latent_rows(Stream& st, const LatentRowsArgs& a) {
    return launch(st, k_latent_rows<T>, dim3(a.n), dim3(128), 0, a);
}
template int latent_rows<bf16>(Stream&, const LatentRowsArgs&);
template int latent_rows<float>(Stream&, const LatentRowsArgs&);

// Causal attention (all keys before a position, or those of its chunk) without tensor cores: one CTA per (row, head), tiles of 128 keys, online
// softmax.
constexpr int CR_KEYS = 128, CR_MAXV = 4;
template <typename T>
__global__ void __launch_bounds__(128) k_causal_rows(CausalArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float cr_q[];                      // [dim + rot]
    __shared__ float p[CR_KEYS];
    __shared__ float red[4];
    const int t = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nk = a.pos0 + t + 1, first = a.chunk > 0 ? (nk - 1) / a.chunk * a.chunk : 0, kvh = head / (a.heads / a.kv_heads);
    const T* q = reinterpret_cast<const T*>(a.q) + ((size_t)t * a.heads + head) * a.dim;
    const T* qr = reinterpret_cast<const T*>(a.q_rot) + ((size_t)t * a.heads + head) * a.rot;
    const T* kr = reinterpret_cast<const T*>(a.k_rot);
    const float c = a.scale * LOG2E;
    for (int i = tid; i < a.dim; i += 128) cr_q[i] = Elem<T>::get(q[i]);
    for (int i = tid; i < a.rot; i += 128) cr_q[a.dim + i] = Elem<T>::get(qr[i]);
    __syncthreads();
    float m = a.sink ? a.sink[head] * LOG2E : -INFINITY;
    float l = a.sink ? 1.0f : 0.0f;                      // the sink is a key without a value
    float acc[CR_MAXV] = {};
    for (int k0 = first; k0 < nk; k0 += CR_KEYS) {
        const int cnt = min(CR_KEYS, nk - k0);
        float best = -INFINITY;
        for (int j = warp; j < cnt; j += 4) {
            const T* k = reinterpret_cast<const T*>(a.k) + (size_t)(k0 + j) * a.ldk + (size_t)kvh * a.dim;
            float s = 0.f;
            for (int i = lane * 4; i < a.dim; i += 128) {
                const float4 kv = load4(k + i), qv = load4(cr_q + i);
                s = fmaf(kv.x, qv.x, fmaf(kv.y, qv.y, fmaf(kv.z, qv.z, fmaf(kv.w, qv.w, s))));
            }
            for (int i = lane; i < a.rot; i += 32) s = fmaf(Elem<T>::get(kr[(size_t)(k0 + j) * a.ld_rot + i]), cr_q[a.dim + i], s);
            s = warp_sum(s) * c;
            if (lane == 0) p[j] = s;
            best = fmaxf(best, s);
        }
        if (lane == 0) red[warp] = best;
        __syncthreads();
        const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
        const float alpha = exp2f(m - mn);
        if (tid < cnt) p[tid] = exp2f(p[tid] - mn);
        m = mn;
        __syncthreads();
        l = l * alpha + cta_sum<4>(tid < cnt ? p[tid] : 0.f, red);
#pragma unroll
        for (int x = 0; x < CR_MAXV; ++x) {
            const int j = tid + x * 128;
            if (j >= a.vdim) break;
            const T* v = reinterpret_cast<const T*>(a.v) + (size_t)k0 * a.ldv + (size_t)kvh * a.vdim + j;
            float s = 0.f;
            for (int y = 0; y < cnt; ++y) s = fmaf(p[y], Elem<T>::get(v[(size_t)y * a.ldv]), s);
            acc[x] = acc[x] * alpha + s;
        }
        __syncthreads();
    }
    const float gate = a.gate ? 1.0f / (1.0f + expf(-a.gate[(size_t)t * a.ld_gate + head])) : 1.0f;
    T* o = reinterpret_cast<T*>(a.out) + (size_t)t * a.ld_out + (size_t)head * a.vdim;
#pragma unroll
    for (int x = 0; x < CR_MAXV; ++x) {
        const int j = tid + x * 128;
        if (j < a.vdim) o[j] = Elem<T>::put(acc[x] / l * gate);
    }
}
template <typename T>
int causal_simt(Stream& st, const CausalArgs& a) {
    if (a.vdim > CR_MAXV * 128) return MQ_ERR_UNSUPPORTED;
    return launch(st, k_causal_rows<T>, dim3(a.n, a.heads), dim3(128), (size_t)(a.dim + a.rot) * 4, a);
}
template int causal_simt<bf16>(Stream&, const CausalArgs&);
template int causal_simt<float>(Stream&, const CausalArgs&);

// The tcgen05 kernel holds heads of up to 128 + 64 query / key and 128 value dimensions, and takes a positive scale.
bool causal_tc_fits(int dim, int rot, int vdim, float scale) { return dim <= 128 && rot <= 64 && vdim <= 128 && scale > 0.f; }
int causal_tc(Stream& st, const CausalArgs& a) {
    const uint64_t n = a.n, keys = a.pos0 + a.n, H = a.heads, G = a.kv_heads;
    CUtensorMap mq_, mk, mv, mqr, mkr;
    int rc = get_map(a.q, n, a.dim, H * a.dim, TA_BQ, &mq_, H, a.dim);
    if (!rc) rc = get_map(a.k, keys, a.dim, a.ldk, TA_BK, &mk, G, a.dim);
    if (!rc) rc = get_map(a.v, keys, a.vdim, a.ldv, TA_BK, &mv, G, a.vdim);
    if (!rc && a.rot) rc = get_map(a.q_rot, n, a.rot, H * a.rot, TA_BQ, &mqr, H, a.rot);
    if (!rc && a.rot) rc = get_map(a.k_rot, keys, a.rot, a.ld_rot, TA_BK, &mkr, 1, keys * a.ld_rot);
    if (rc) return rc;
    AttnTcArgs t = {(bf16*)a.out, a.ld_out, a.vdim, a.n, a.pos0, a.heads / a.kv_heads, 0, a.dim / 16, a.rot / 16, a.scale * LOG2E, a.sink, a.status};
    t.chunk = a.chunk; t.gate = a.gate; t.ld_gate = a.ld_gate;
    ++st.launches;
    const int qp = (a.dim + 63) / 64, vp = (a.vdim + 63) / 64;
    if (a.rot == 0) {                  // no shared key part
        if (qp == 1 && vp == 1) return launch_attention_tc<1, 0, 1>(a.heads, mq_, mk, mv, mq_, mk, t, st.s);
        if (qp == 1 && vp == 2) return launch_attention_tc<1, 0, 2>(a.heads, mq_, mk, mv, mq_, mk, t, st.s);
        if (qp == 2 && vp == 1) return launch_attention_tc<2, 0, 1>(a.heads, mq_, mk, mv, mq_, mk, t, st.s);
        if (qp == 2 && vp == 2) return launch_attention_tc<2, 0, 2>(a.heads, mq_, mk, mv, mq_, mk, t, st.s);
        return MQ_ERR_UNSUPPORTED;
    }
    if (qp == 1 && vp == 1) return launch_attention_tc<1, 1, 1>(a.heads, mq_, mk, mv, mqr, mkr, t, st.s);
    if (qp == 1 && vp == 2) return launch_attention_tc<1, 1, 2>(a.heads, mq_, mk, mv, mqr, mkr, t, st.s);
    if (qp == 2 && vp == 1) return launch_attention_tc<2, 1, 1>(a.heads, mq_, mk, mv, mqr, mkr, t, st.s);
    if (qp == 2 && vp == 2) return launch_attention_tc<2, 1, 2>(a.heads, mq_, mk, mv, mqr, mkr, t, st.s);
    return MQ_ERR_UNSUPPORTED;
}

// ---------------------------------------------------------------- one token: query
// CTA (x, h): q of head h times rows [64 x, 64 x + 64) of its W_uk^T -> qcat[h][..rank).  The extra CTA in x rotates
// all heads' rotated parts into qcat[h][rank..) and (h = 0) writes the new cache row.
constexpr int LQ_ROWS = 64, LQ_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(LQ_THREADS) k_latent_query(LatentDecodeArgs a) {
    extern __shared__ float lq_q[];                      // [dim]
    __shared__ float red[8];
    constexpr int EPL = Elem<T>::PER16;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, D = a.rank + a.rot;
    const bool extra = blockIdx.x == gridDim.x - 1;
    T* qc = reinterpret_cast<T*>(a.qcat) + (size_t)h * D;
    // a row of W_uk^T holds dim elements: `lanes` lanes of 16 bytes (a power of two, up to 32), 32 / lanes rows per load
    int lanes = 1;
    while (lanes < 32 && lanes * EPL < a.dim) lanes <<= 1;
    const int per = 32 / lanes, sub = lane / lanes, ln = lane % lanes;
    const int loads = (LQ_ROWS / 8 + per - 1) / per;     // of this warp's eight rows
    const T* W = reinterpret_cast<const T*>(a.w_uk_t) + (size_t)h * a.rank * a.dim;
    const int rbase = blockIdx.x * LQ_ROWS + warp * (LQ_ROWS / 8);
    uint4 w[8];
    if (!extra) {
#pragma unroll
        for (int x = 0; x < 8; ++x) {
            const int lr = x * per + sub, r = rbase + lr;
            const bool ok = x < loads && lr < LQ_ROWS / 8 && r < a.rank && ln * EPL < a.dim;
            w[x] = ok ? *reinterpret_cast<const uint4*>(W + (size_t)r * a.dim + ln * EPL) : make_uint4(0u, 0u, 0u, 0u);
        }
    }
    if (extra) {
        // what does not come from the kernel before is loaded before the wait (the position was set before this step began)
        int pos = *a.position;
        if (pos < 0 || pos >= a.max_seq) {
            if (tid == 0) atomicOr(a.status, MQ_STATUS_BAD_POSITION);
            pos = pos < 0 ? 0 : a.max_seq - 1;
        }
        const float2* rope = reinterpret_cast<const float2*>(a.rope + (size_t)pos * a.rot);
        const int pairs = a.rot / 2;
        float2 cs = tid < pairs ? rope[tid] : make_float2(1.f, 0.f);
        float2 nw[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int i = 2 * (tid + x * LQ_THREADS);
            nw[x] = h == 0 && i < a.rank ? *reinterpret_cast<const float2*>(a.norm + i) : make_float2(0.f, 0.f);
        }
        pdl_trigger();
        pdl_wait_cta();
        const T* qr = reinterpret_cast<const T*>(a.q_rot) + (size_t)h * a.rot;
        T* row = reinterpret_cast<T*>(a.cache) + (size_t)pos * D;
        for (int i = tid; i < pairs; i += LQ_THREADS) {
            if (i != tid) cs = rope[i];
            const float2 q = load2(qr + 2 * i);
            if (h == 0) {
                const float2 k = load2(a.down + a.rank + 2 * i);
                store2(row + a.rank + 2 * i, rotate_pair(k.x, k.y, cs));
            }
            store2(qc + a.rank + 2 * i, rotate_pair(q.x, q.y, cs));
        }
        if (h == 0) write_latent<T, LQ_THREADS>(a.down, a.norm, nw, a.norm_n, a.eps, row, a.rank, red);
        return;
    }
    pdl_trigger();
    pdl_wait_cta();
    const T* q = reinterpret_cast<const T*>(a.q) + (size_t)h * a.dim;
    for (int i = tid; i < a.dim; i += LQ_THREADS) lq_q[i] = Elem<T>::get(__ldcg(q + i));
    __syncthreads();
#pragma unroll
    for (int x = 0; x < 8; ++x) {
        if (x >= loads) break;
        const int lr = x * per + sub, r = rbase + lr;
        const bool ok = lr < LQ_ROWS / 8 && r < a.rank;
        float s = 0.f;
        for (int c0 = ln * EPL; c0 < a.dim && ok; c0 += 32 * EPL) {     // one pass unless dim > 32 * EPL
            const uint4 u = c0 == ln * EPL ? w[x] : *reinterpret_cast<const uint4*>(W + (size_t)r * a.dim + c0);
            s = dot_row16(u, lq_q + c0, s, (const T*)nullptr);
        }
        for (int o = lanes >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (ok && ln == 0) qc[r] = Elem<T>::put(s);
    }
}

// ---------------------------------------------------------------- one token: splits
// The cached tokens [0, ctx) are dealt to up to `splits` CTAs in equal pieces of whole 64-key tiles.
constexpr int LA_KEYS = 64;
int latent_splits(int max_seq) {
    const int n = (max_seq + LA_KEYS - 1) / LA_KEYS;
    return n < 148 ? n : 148;
}
__device__ __forceinline__ int keys_per_split(int ctx, int splits) {
    const int tiles = (ctx + LA_KEYS - 1) / LA_KEYS;
    return ((tiles + splits - 1) / splits) * LA_KEYS;
}
__device__ __forceinline__ int clamp_pos(int pos, int max_seq) { return pos < 0 ? 0 : pos >= max_seq ? max_seq - 1 : pos; }
// A split leaves behind, per head, the sum of its weighted latents (parts [split][head][rank]) and, after all of those, the
// maximum of its scores and the sum of its weights (pairs [split][head]).
size_t latent_parts_floats(int heads, int rank, int max_seq) { return (size_t)latent_splits(max_seq) * heads * (rank + 2); }

// bf16, up to 512 latent dimensions: sixteen heads are the M of mma.sync, so every cached row is read once for all of them.
constexpr int LA_THREADS = 256, LA_MAXT = 8, LA_PLD = LA_KEYS + 8;
static size_t la_smem(int D) { return (size_t)(LA_KEYS + 16) * (D + 8) * 2; }
__global__ void __launch_bounds__(LA_THREADS) k_latent_attention(LatentDecodeArgs a) {
    extern __shared__ __align__(16) uint8_t la_raw[];
    __shared__ __align__(16) bf16 sp[16 * LA_PLD];
    __shared__ float smax[8][16], ssum[8][16];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = a.rank + a.rot, ld = D + 8, d8 = D / 8;
    bf16* sk = reinterpret_cast<bf16*>(la_raw);
    bf16* sq = sk + LA_KEYS * ld;
    const bf16* cache = reinterpret_cast<const bf16*>(a.cache);
    const int h0 = blockIdx.y * 16, split = blockIdx.x;
    const int pos = clamp_pos(*a.position, a.max_seq), ctx = pos + 1;     // the position was set before this step began
    const int kps = keys_per_split(ctx, gridDim.x), kbeg = split * kps, kend = min(kbeg + kps, ctx);
    pdl_trigger();
    if (kbeg >= kend) return;
    auto fetch = [&](int k0, int lo, int hi) {            // rows lo .. hi - 1 of the tile at k0; those beyond kend as zeros
        for (int x = lo * d8 + tid; x < hi * d8; x += LA_THREADS) {
            const int j = x / d8, col = (x % d8) * 8;
            const bool ok = k0 + j < kend;
            cp_async16_zfill(sk + j * ld + col, ok ? cache + (size_t)(k0 + j) * D + col : cache, ok);
        }
        cp_async_commit();
    };
    // cached rows before the wait; the row of this token (written by the kernel before) after it
    const bool has_new = kend == ctx && kbeg + LA_KEYS >= ctx;
    const int jn = pos - kbeg;
    if (has_new) { fetch(kbeg, 0, jn); fetch(kbeg, jn + 1, LA_KEYS); }
    else fetch(kbeg, 0, LA_KEYS);
    pdl_wait_cta();
    if (has_new) fetch(kbeg, jn, jn + 1);
    for (int x = tid; x < 16 * d8; x += LA_THREADS) {
        const int r = x / d8, col = (x % d8) * 8;
        *reinterpret_cast<uint4*>(sq + r * ld + col) = ld_cg_u4(reinterpret_cast<const bf16*>(a.qcat) + (size_t)(h0 + r) * D + col);
    }
    const float c = a.scale * LOG2E;
    const int ntiles = a.rank / 8, tpw = 2 * ((ntiles + 15) / 16), tile0 = warp * tpw;
    float acc[LA_MAXT][4];
#pragma unroll
    for (int i = 0; i < LA_MAXT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};               // rows lane / 4, lane / 4 + 8
    const int row = lane >> 2;
    for (int k0 = kbeg; k0 < kend; k0 += LA_KEYS) {
        if (k0 > kbeg) fetch(k0, 0, LA_KEYS);
        cp_async_wait_all();
        __syncthreads();
        // scores of this warp's eight keys; two accumulators break the chain of dependent products
        float s0[4] = {}, s1[4] = {};
        const uint32_t qa = smem_u32(sq + (lane & 15) * ld + (lane >> 4) * 8);
        const uint32_t kb = smem_u32(sk + (warp * 8 + row) * ld + (lane & 3) * 2);
        int ks = 0;
#pragma unroll 3
        for (; ks + 1 < D / 16; ks += 2) {
            uint32_t q4[4], r4[4];
            ldsm4(q4, qa + ks * 32);
            ldsm4(r4, qa + ks * 32 + 32);
            mma16816(s0, q4, lds32(kb + ks * 32), lds32(kb + ks * 32 + 16));
            mma16816(s1, r4, lds32(kb + ks * 32 + 32), lds32(kb + ks * 32 + 48));
        }
        if (ks < D / 16) {
            uint32_t q4[4];
            ldsm4(q4, qa + ks * 32);
            mma16816(s0, q4, lds32(kb + ks * 32), lds32(kb + ks * 32 + 16));
        }
        float s[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int key = k0 + warp * 8 + 2 * (lane & 3) + (e & 1);
            s[e] = key < kend ? (s0[e] + s1[e]) * c : -INFINITY;
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float v = fmaxf(s[2 * h], s[2 * h + 1]);
            v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
            v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
            if ((lane & 3) == 0) smax[warp][row + 8 * h] = v;
        }
        __syncthreads();
        float alpha[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float mn = m[h];
#pragma unroll
            for (int w = 0; w < 8; ++w) mn = fmaxf(mn, smax[w][row + 8 * h]);
            alpha[h] = exp2f(m[h] - mn);
            m[h] = mn;
            const float p0 = exp2f(s[2 * h] - mn), p1 = exp2f(s[2 * h + 1] - mn);
            *reinterpret_cast<uint32_t*>(sp + (row + 8 * h) * LA_PLD + warp * 8 + 2 * (lane & 3)) = pack_bf16x2(p0, p1);
            float v = p0 + p1;
            v += __shfl_xor_sync(0xffffffffu, v, 1);
            v += __shfl_xor_sync(0xffffffffu, v, 2);
            if ((lane & 3) == 0) ssum[warp][row + 8 * h] = v;
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) v += ssum[w][row + 8 * h];
            l[h] = l[h] * alpha[h] + v;
        }
#pragma unroll
        for (int i = 0; i < LA_MAXT; ++i) { acc[i][0] *= alpha[0]; acc[i][1] *= alpha[0]; acc[i][2] *= alpha[1]; acc[i][3] *= alpha[1]; }
#pragma unroll
        for (int ks = 0; ks < LA_KEYS / 16; ++ks) {
            uint32_t p4[4];
            ldsm4(p4, smem_u32(sp + (lane & 15) * LA_PLD + ks * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int i = 0; i < LA_MAXT; i += 2) {
                if (i >= tpw || tile0 + i >= ntiles) break;
                uint32_t b[4];
                ldsm4_t(b, smem_u32(sk + (ks * 16 + (lane & 15)) * ld + (tile0 + i) * 8 + (lane >> 4) * 8));
                mma16816(acc[i], p4, b[0], b[1]);
                mma16816(acc[i + 1], p4, b[2], b[3]);
            }
        }
        __syncthreads();                                   // keys, weights and maxima are overwritten by the next tile
    }
    const int heads_here = min(16, a.heads - h0);
    const size_t part = (size_t)split * a.heads + h0;
    float2* ml = reinterpret_cast<float2*>(a.parts + (size_t)gridDim.x * a.heads * a.rank);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int r = row + 8 * h;
        if (r >= heads_here) continue;
        float* dst = a.parts + (part + r) * a.rank;
#pragma unroll
        for (int i = 0; i < LA_MAXT; ++i) {
            if (i >= tpw || tile0 + i >= ntiles) break;
            *reinterpret_cast<float2*>(dst + (tile0 + i) * 8 + 2 * (lane & 3)) = make_float2(acc[i][2 * h], acc[i][2 * h + 1]);
        }
        if (warp == 0 && (lane & 3) == 0) ml[part + r] = make_float2(m[h], l[h]);
    }
}

// The same split for 32-bit caches and larger latents: one CTA per (split, head).
constexpr int LP_THREADS = 128, LP_MAXC = 16;
template <typename T>
__global__ void __launch_bounds__(LP_THREADS) k_latent_attention_plain(LatentDecodeArgs a) {
    extern __shared__ float lp_q[];                        // [rank + rot]
    __shared__ float p[LA_KEYS];
    __shared__ float red[4];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = a.rank + a.rot, head = blockIdx.y, split = blockIdx.x;
    const T* cache = reinterpret_cast<const T*>(a.cache);
    pdl_trigger();
    pdl_wait_cta();
    const int pos = clamp_pos(*a.position, a.max_seq), ctx = pos + 1;
    const int kps = keys_per_split(ctx, gridDim.x), kbeg = split * kps, kend = min(kbeg + kps, ctx);
    if (kbeg >= kend) return;
    for (int i = tid; i < D; i += LP_THREADS) lp_q[i] = Elem<T>::get(__ldcg(reinterpret_cast<const T*>(a.qcat) + (size_t)head * D + i));
    __syncthreads();
    const float c = a.scale * LOG2E;
    float m = -INFINITY, l = 0.f, acc[LP_MAXC] = {};
    for (int k0 = kbeg; k0 < kend; k0 += LA_KEYS) {
        const int cnt = min(LA_KEYS, kend - k0);
        float best = -INFINITY;
        for (int j = warp; j < cnt; j += 4) {
            float s = 0.f;
            for (int i = lane * 4; i < D; i += 128) {
                const float4 kv = load4_cg(cache + (size_t)(k0 + j) * D + i), qv = load4(lp_q + i);
                s = fmaf(kv.x, qv.x, fmaf(kv.y, qv.y, fmaf(kv.z, qv.z, fmaf(kv.w, qv.w, s))));
            }
            s = warp_sum(s) * c;
            if (lane == 0) p[j] = s;
            best = fmaxf(best, s);
        }
        if (lane == 0) red[warp] = best;
        __syncthreads();
        const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
        const float alpha = exp2f(m - mn);
        m = mn;
        if (tid < cnt) p[tid] = exp2f(p[tid] - mn);
        __syncthreads();
        l = l * alpha + cta_sum<4>(tid < cnt ? p[tid] : 0.f, red);
#pragma unroll
        for (int x = 0; x < LP_MAXC; ++x) {
            const int i = tid + x * LP_THREADS;
            if (i >= a.rank) break;
            float s = 0.f;
            for (int j = 0; j < cnt; ++j) s = fmaf(p[j], Elem<T>::get(__ldcg(cache + (size_t)(k0 + j) * D + i)), s);
            acc[x] = acc[x] * alpha + s;
        }
        __syncthreads();
    }
    const size_t part = (size_t)split * a.heads + head;
    float* dst = a.parts + part * a.rank;
#pragma unroll
    for (int x = 0; x < LP_MAXC; ++x) {
        const int i = tid + x * LP_THREADS;
        if (i < a.rank) dst[i] = acc[x];
    }
    if (tid == 0) reinterpret_cast<float2*>(a.parts + (size_t)gridDim.x * a.heads * a.rank)[part] = make_float2(m, l);
}

// ---------------------------------------------------------------- one token: merge
// CTA (x, h): the latent sum of head h over all splits, the sink in the denominator, then rows [32 x, 32 x + 32) of its W_uv.
// Thread = (group of splits, four latent columns); the groups' sums meet in shared memory.
constexpr int LM_ROWS = 32, LM_THREADS = 512, LM_WARPS = LM_THREADS / 32, LM_PRE = 2, LM_FIRST = 8;
static __host__ __device__ __forceinline__ int lm_groups(int rank) { return rank >= 4 * LM_THREADS ? 1 : 4 * LM_THREADS / rank < 8 ? 4 * LM_THREADS / rank : 8; }
template <typename T>
__global__ void __launch_bounds__(LM_THREADS) k_latent_merge(LatentDecodeArgs a, int splits) {
    extern __shared__ float lm_c[];                        // [groups][rank], then the weight of every split
    __shared__ float red[LM_WARPS];
    constexpr int EPL = Elem<T>::PER16;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y;
    const int groups = lm_groups(a.rank), cols = a.rank / 4;
    float* ws = lm_c + groups * a.rank;
    const int r0 = blockIdx.x * LM_ROWS + warp * (LM_ROWS / LM_WARPS);
    const T* W = reinterpret_cast<const T*>(a.w_uv) + (size_t)h * a.vdim * a.rank;
    uint4 w[LM_ROWS / LM_WARPS][LM_PRE];
#pragma unroll
    for (int x = 0; x < LM_ROWS / LM_WARPS; ++x)
#pragma unroll
        for (int s = 0; s < LM_PRE; ++s) {
            const int c0 = (s * 32 + lane) * EPL;
            w[x][s] = r0 + x < a.vdim && c0 < a.rank ? *reinterpret_cast<const uint4*>(W + (size_t)(r0 + x) * a.rank + c0) : make_uint4(0u, 0u, 0u, 0u);
        }
    const int ctx = clamp_pos(*a.position, a.max_seq) + 1;                            // the position was set before this step began
    const int kps = keys_per_split(ctx, splits), active = (ctx + kps - 1) / kps;      // at most 148 < LM_THREADS
    const size_t hs = (size_t)h, stride = (size_t)a.heads;
    pdl_trigger();
    pdl_wait_cta();
    // the first latent sums are on their way while the weights are worked out
    float4 first[LM_FIRST];
#pragma unroll
    for (int y = 0; y < LM_FIRST; ++y) {
        const int k = tid / cols + y * groups;
        first[y] = tid < groups * cols && k < active ? load4_cg(a.parts + (k * stride + hs) * a.rank + (tid % cols) * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float2* ml = reinterpret_cast<const float2*>(a.parts + (size_t)splits * a.heads * a.rank);
    const float sink = a.sink ? a.sink[h] * LOG2E : -INFINITY;
    const float2 mine = tid < active ? __ldcg(ml + tid * stride + hs) : make_float2(-INFINITY, 0.f);
    float m = warp_max(mine.x);
    if (lane == 0) red[warp] = m;
    __syncthreads();
    m = sink;
#pragma unroll
    for (int i = 0; i < LM_WARPS; ++i) m = fmaxf(m, red[i]);
    __syncthreads();
    const float e = exp2f(mine.x - m);
    if (tid < active) ws[tid] = e;
    const float inv = 1.0f / (cta_sum<LM_WARPS>(e * mine.y, red) + exp2f(sink - m));
    for (int x = tid; x < groups * cols; x += LM_THREADS) {
        const int g = x / cols, c = (x % cols) * 4;
        const float* p = a.parts + hs * a.rank + c;
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
        auto add = [&](int k, const float4& v) {
            const float f = ws[k];
            s.x = fmaf(f, v.x, s.x); s.y = fmaf(f, v.y, s.y); s.z = fmaf(f, v.z, s.z); s.w = fmaf(f, v.w, s.w);
        };
        int k = g;
        if (x == tid) {
#pragma unroll
            for (int y = 0; y < LM_FIRST; ++y, k += groups)
                if (k < active) add(k, first[y]);
        }
#pragma unroll 8
        for (; k < active; k += groups) add(k, load4_cg(p + k * stride * a.rank));
        store4(lm_c + g * a.rank + c, make_float4(s.x * inv, s.y * inv, s.z * inv, s.w * inv));
    }
    __syncthreads();
    if (groups > 1) {
        for (int i = tid; i < a.rank; i += LM_THREADS) {
            float s = lm_c[i];
            for (int g = 1; g < groups; ++g) s += lm_c[g * a.rank + i];
            lm_c[i] = s;
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 0; x < LM_ROWS / LM_WARPS; ++x) {
        const int r = r0 + x;
        if (r >= a.vdim) break;
        float s = 0.f;
#pragma unroll
        for (int seg = 0; seg < LM_PRE; ++seg) {
            const int c0 = (seg * 32 + lane) * EPL;
            if (c0 < a.rank) s = dot_row16(w[x][seg], lm_c + c0, s, (const T*)nullptr);
        }
        for (int c0 = (LM_PRE * 32 + lane) * EPL; c0 < a.rank; c0 += 32 * EPL)
            s = dot_row16(*reinterpret_cast<const uint4*>(W + (size_t)r * a.rank + c0), lm_c + c0, s, (const T*)nullptr);
        s = warp_sum(s);
        if (lane == 0) reinterpret_cast<T*>(a.out)[(size_t)h * a.vdim + r] = Elem<T>::put(s);
    }
}

template <typename T> struct IsBf16 { static constexpr bool v = false; };
template <> struct IsBf16<bf16> { static constexpr bool v = true; };
template <typename T>
int latent_decode(Stream& st, const LatentDecodeArgs& a) {
    const int splits = latent_splits(a.max_seq), D = a.rank + a.rot;
    int rc = launch(st, k_latent_query<T>, dim3((a.rank + LQ_ROWS - 1) / LQ_ROWS + 1, a.heads), dim3(LQ_THREADS), (size_t)a.dim * 4, a);
    if (rc) return rc;
    if (IsBf16<T>::v && a.rank <= LA_MAXT * 64 && la_smem(D) <= 200 * 1024) {
        rc = allow_smem(k_latent_attention, la_smem(D));
        if (!rc) rc = launch(st, k_latent_attention, dim3(splits, (a.heads + 15) / 16), dim3(LA_THREADS), la_smem(D), a);
    } else {
        if (a.rank > LP_THREADS * LP_MAXC) return MQ_ERR_UNSUPPORTED;
        rc = launch(st, k_latent_attention_plain<T>, dim3(splits, a.heads), dim3(LP_THREADS), (size_t)D * 4, a);
    }
    if (rc) return rc;
    return launch(st, k_latent_merge<T>, dim3((a.vdim + LM_ROWS - 1) / LM_ROWS, a.heads), dim3(LM_THREADS), (size_t)(lm_groups(a.rank) * a.rank + splits) * 4, a, splits);
}
template int latent_decode<bf16>(Stream&, const LatentDecodeArgs&);
template int latent_decode<float>(Stream&, const LatentDecodeArgs&);

}  // namespace hy
}  // namespace mq
