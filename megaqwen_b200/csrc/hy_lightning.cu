// Lightning attention: per head the state S [dim, vdim] decays and takes up k v^T token by
// token, and the output is S^T q.  State, decays and scores are 32-bit.
//
// Two forms.  k_lightning_tokens walks token by token with the state in registers: decoding,
// short portions, 32-bit models, and head sizes that the other form does not hold.  The chunked
// form works on chunks of 128 tokens: k_lightning_kv computes what each chunk adds to the state,
// all chunks at once; k_lightning_scan walks over the chunks element by element and leaves behind
// the state BEFORE every chunk; k_lightning_out, again all chunks at once, adds q times that state
// and the causal product inside the chunk.  Its products run on mma.sync with q, k, v as they are (bf16) and every 32-bit
// factor (state, decayed keys, decayed scores) split into two bf16 terms, hi = bf16(x) and
// lo = bf16(x - hi), which keeps 16 to 17 bits of it; sums are 32-bit.  These products are a few per cent
// of a layer's work and bound by traffic, so they stay off tcgen05, whose operands would
// have to pass through shared memory twice for the split.
#include "hy_common.cuh"

namespace mq {
namespace hy {

constexpr int LC = MQH_CHUNK;

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(a, b);
    lo = pack_bf16x2(a - bf_lo(hi), b - bf_hi(hi));
}

// acc[2 np], acc[2 np + 1] += a * b[np]: NP independent pairs, so that the term that follows finds them finished
template <int NP>
__device__ __forceinline__ void mma_row(float (&acc)[2 * NP][4], const uint32_t (&a)[4], const uint32_t (&b)[NP][4]) {
#pragma unroll
    for (int np = 0; np < NP; ++np) {
        mma16816(acc[2 * np], a, b[np][0], b[np][1]);
        mma16816(acc[2 * np + 1], a, b[np][2], b[np][3]);
    }
}

// ---------------------------------------------------------------- token by token
// One CTA per (32 value columns, head).  Thread = (column quad, row group): rows ig, ig + 32, .. of S.
constexpr int LT_THREADS = 256;
template <typename T, int MAXI>
__global__ void __launch_bounds__(LT_THREADS) k_lightning_tokens(LightningArgs a) {
    __shared__ float part[8][32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y;
    const int j = blockIdx.x * 32 + (tid & 7) * 4, ig = tid >> 3;
    const int dim = a.dim, vdim = a.vdim;
    float* S = a.state + (size_t)head * dim * vdim;
    const bool live = j < vdim;                     // vdim is a multiple of 16
    float4 s[MAXI];
    // The state was last written by the same kernel of an earlier step (complete: see the LM head) or by an
    // unchained launch: it is read before the wait.
#pragma unroll
    for (int m = 0; m < MAXI; ++m) {
        const int i = ig + 32 * m;
        s[m] = live && i < dim ? load4_cg(S + (size_t)i * vdim + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float decay = a.decay_pow[head * (LC + 1) + 1];
    pdl_trigger();
    pdl_wait_cta();
    const T* q = reinterpret_cast<const T*>(a.q) + (size_t)head * dim;
    const T* k = reinterpret_cast<const T*>(a.k) + (size_t)head * dim;
    const T* v = reinterpret_cast<const T*>(a.v) + (size_t)head * vdim;
    const size_t ldk = (size_t)a.heads * dim, ldv = (size_t)a.heads * vdim;
    for (int t = 0; t < a.n; ++t) {
        const float4 vv = live ? load4_cg(v + t * ldv + j) : make_float4(0.f, 0.f, 0.f, 0.f);
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int m = 0; m < MAXI; ++m) {
            const int i = ig + 32 * m;
            if (i >= dim) break;
            const float ki = Elem<T>::get(__ldcg(k + t * ldk + i)), qi = Elem<T>::get(__ldcg(q + t * ldk + i));
            s[m].x = fmaf(decay, s[m].x, ki * vv.x); s[m].y = fmaf(decay, s[m].y, ki * vv.y);
            s[m].z = fmaf(decay, s[m].z, ki * vv.z); s[m].w = fmaf(decay, s[m].w, ki * vv.w);
            o.x = fmaf(qi, s[m].x, o.x); o.y = fmaf(qi, s[m].y, o.y); o.z = fmaf(qi, s[m].z, o.z); o.w = fmaf(qi, s[m].w, o.w);
        }
#pragma unroll
        for (int x = 8; x < 32; x <<= 1) {          // the four row groups of the warp
            o.x += __shfl_xor_sync(0xffffffffu, o.x, x); o.y += __shfl_xor_sync(0xffffffffu, o.y, x);
            o.z += __shfl_xor_sync(0xffffffffu, o.z, x); o.w += __shfl_xor_sync(0xffffffffu, o.w, x);
        }
        if (lane < 8) store4(&part[warp][lane * 4], o);
        __syncthreads();
        if (tid < 32 && blockIdx.x * 32 + tid < vdim) {
            float sum = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) sum += part[w][tid];
            a.o[t * ldv + (size_t)head * vdim + blockIdx.x * 32 + tid] = sum;
        }
        __syncthreads();
    }
#pragma unroll
    for (int m = 0; m < MAXI; ++m) {
        const int i = ig + 32 * m;
        if (live && i < dim) store4(S + (size_t)i * vdim + j, s[m]);
    }
}
template <typename T>
int lightning_tokens(Stream& st, const LightningArgs& a) {
    const dim3 grid((a.vdim + 31) / 32, a.heads), block(LT_THREADS);
    if (a.dim <= 128) return launch(st, k_lightning_tokens<T, 4>, grid, block, 0, a);
    if (a.dim <= 256) return launch(st, k_lightning_tokens<T, 8>, grid, block, 0, a);
    if (a.dim <= 512) return launch(st, k_lightning_tokens<T, 16>, grid, block, 0, a);
    return MQ_ERR_UNSUPPORTED;
}
template int lightning_tokens<bf16>(Stream&, const LightningArgs&);
template int lightning_tokens<float>(Stream&, const LightningArgs&);

// rows x cols bf16 (cols a multiple of 8) from a matrix of row length ld into shared memory of row length sld by
// asynchronous copies; rows from `live` on and columns from `cols_live` on become zeros.  PER threads share a row, so that
// no index is divided by a run-time value.
template <int THREADS, int PER>
__device__ __forceinline__ void copy_tile(bf16* dst, int sld, const bf16* src, size_t ld, int rows, int live, int cols, int cols_live) {
    const int r0 = threadIdx.x / PER, c0 = (threadIdx.x % PER) * 8;
    for (int col = c0; col < cols; col += PER * 8) {
        const bool cok = col < cols_live;
        const bf16* p = src + (size_t)r0 * ld + col;
        bf16* d = dst + r0 * sld + col;
        for (int r = r0; r < rows; r += THREADS / PER) {
            const bool ok = cok && r < live;
            cp_async16_zfill(d, ok ? p : src, ok);
            p += (size_t)(THREADS / PER) * ld;
            d += (THREADS / PER) * sld;
        }
    }
}

// ---------------------------------------------------------------- chunked: what every chunk adds to the state
// One CTA per (chunk, head, JT value columns): KV = sum over the chunk's n tokens of decay^(n - 1 - t) k_t v_t^T, fp32.
// Warp w takes rows 16 (w % 8) + 128 x of the head's dim and half of the columns.
constexpr int LK_THREADS = 512;
static size_t lk_smem(int dim, int jt) { return (size_t)LC * (dim + 8 + jt + 8) * 2; }
template <int JT>
__global__ void __launch_bounds__(LK_THREADS, 2) k_lightning_kv(LightningArgs a, float* __restrict__ kv) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t lk_raw[];
    __shared__ float pw[LC];                                   // by token: decay^(n - 1 - t)
    constexpr int VLD = JT + 8, NP = JT / 32;                   // 16-column pairs of tiles per warp
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, c = blockIdx.x, j0 = blockIdx.z * JT;
    const int dim = a.dim, vdim = a.vdim, kld = dim + 8, jw = (warp >> 3) * (JT / 2);
    bf16* sk = reinterpret_cast<bf16*>(lk_raw);
    bf16* sv = sk + LC * kld;
    const int cnt = min(LC, a.n - c * LC);
    const size_t ldk = (size_t)a.heads * dim, ldv = (size_t)a.heads * vdim, row0 = (size_t)c * LC;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * ldk + (size_t)head * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * ldv + (size_t)head * vdim + j0;
    copy_tile<LK_THREADS, 16>(sk, kld, kg, ldk, LC, cnt, dim, dim);
    copy_tile<LK_THREADS, JT / 8>(sv, VLD, vg, ldv, LC, cnt, JT, vdim - j0);
    cp_async_commit();
    if (tid < LC) pw[tid] = tid < cnt ? a.decay_pow[head * (LC + 1) + cnt - 1 - tid] : 0.f;
    cp_async_wait_all();
    __syncthreads();
    const int ksteps = (cnt + 15) / 16;
    if (j0 + jw >= vdim) return;
    for (int i0 = (warp & 7) * 16; i0 < dim; i0 += 128) {
        float acc[2 * NP][4];
#pragma unroll
        for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] = 0.f;
#pragma unroll 2
        for (int ks = 0; ks < ksteps; ++ks) {
            const int t0 = ks * 16, t = t0 + 2 * (lane & 3);
            uint32_t ka[4], ah[4], al[4];
            ldsm4_t(ka, smem_u32(sk + (t0 + (lane & 7) + ((lane >> 4) & 1) * 8) * kld + i0 + ((lane >> 3) & 1) * 8));
            const float w[4] = {pw[t], pw[t + 1], pw[t + 8], pw[t + 9]};
#pragma unroll
            for (int x = 0; x < 4; ++x) split_pair(bf_lo(ka[x]) * w[(x >> 1) * 2], bf_hi(ka[x]) * w[(x >> 1) * 2 + 1], ah[x], al[x]);
            uint32_t b[NP][4];
#pragma unroll
            for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sv + (t0 + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8));
            mma_row<NP>(acc, ah, b);
            mma_row<NP>(acc, al, b);
        }
        float* dst = kv + ((size_t)c * a.heads + head) * dim * vdim + (size_t)(i0 + (lane >> 2)) * vdim + j0 + jw + 2 * (lane & 3);
#pragma unroll
        for (int nt = 0; nt < 2 * NP; ++nt)
            if (j0 + jw + nt * 8 < vdim) {
                *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(acc[nt][0], acc[nt][1]);
                *reinterpret_cast<float2*>(dst + (size_t)8 * vdim + nt * 8) = make_float2(acc[nt][2], acc[nt][3]);
            }
    }
}

// ---------------------------------------------------------------- chunked: the state before every chunk
// Element by element over the chunks: hi[c], lo[c] = the two bf16 terms of the state, state <- decay^n state + KV[c].
constexpr int LN_THREADS = 128, LN_AHEAD = 8;
__global__ void __launch_bounds__(LN_THREADS) k_lightning_scan(LightningArgs a, const float* __restrict__ kv, bf16* __restrict__ hi, bf16* __restrict__ lo) {
    pdl_trigger();
    const size_t e = ((size_t)blockIdx.x * LN_THREADS + threadIdx.x) * 4, plane = (size_t)a.heads * a.dim * a.vdim;
    const bool live = e < plane;
    const int nchunks = (a.n + LC - 1) / LC, head = live ? (int)(e / ((size_t)a.dim * a.vdim)) : 0;
    const float* pw = a.decay_pow + head * (LC + 1);
    const float full = pw[LC], last = pw[a.n - (nchunks - 1) * LC];
    pdl_wait();
    if (!live) return;
    float4 s = load4_cg(a.state + e);
    for (int c0 = 0; c0 < nchunks; c0 += LN_AHEAD) {
        float4 v[LN_AHEAD];
#pragma unroll
        for (int x = 0; x < LN_AHEAD; ++x)
            if (c0 + x < nchunks) v[x] = load4_cg(kv + (c0 + x) * plane + e);
#pragma unroll
        for (int x = 0; x < LN_AHEAD; ++x)
            if (c0 + x < nchunks) {
                uint2 h, l;
                split_pair(s.x, s.y, h.x, l.x);
                split_pair(s.z, s.w, h.y, l.y);
                *reinterpret_cast<uint2*>(hi + (c0 + x) * plane + e) = h;
                *reinterpret_cast<uint2*>(lo + (c0 + x) * plane + e) = l;
                const float d = c0 + x == nchunks - 1 ? last : full;
                s.x = fmaf(d, s.x, v[x].x); s.y = fmaf(d, s.y, v[x].y); s.z = fmaf(d, s.z, v[x].z); s.w = fmaf(d, s.w, v[x].w);
            }
    }
    store4(a.state + e, s);
}

// ---------------------------------------------------------------- chunked: outputs
// One CTA per (chunk, head, JT value columns); each warp takes sixteen tokens t0 .. t0 + 15 of the chunk and half of the columns:
// o_t = decay^(t + 1) q_t S + sum over s <= t of (q_t k_s) decay^(t - s) v_s      (t, s within the chunk)
constexpr int LO_THREADS = 512;
static size_t lo_smem(int dim, int jt) { return ((size_t)2 * LC * (dim + 8) + (size_t)(LC + 2 * dim) * (jt + 8)) * 2; }
template <int JT>
__global__ void __launch_bounds__(LO_THREADS, 1) k_lightning_out(LightningArgs a, const bf16* __restrict__ hi, const bf16* __restrict__ lo) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t lo_raw[];
    __shared__ float pw[LC + 1];
    constexpr int VLD = JT + 8, NP = JT / 32;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, c = blockIdx.x, j0 = blockIdx.z * JT;
    const int dim = a.dim, vdim = a.vdim, qld = dim + 8;
    const int cnt = min(LC, a.n - c * LC);
    bf16* sq = reinterpret_cast<bf16*>(lo_raw);
    bf16* sk = sq + LC * qld;
    bf16* sv = sk + LC * qld;
    bf16* sh = sv + LC * VLD;
    bf16* sl = sh + dim * VLD;
    const size_t ldk = (size_t)a.heads * dim, ldv = (size_t)a.heads * vdim, row0 = (size_t)c * LC;
    const bf16* qg = reinterpret_cast<const bf16*>(a.q) + row0 * ldk + (size_t)head * dim;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * ldk + (size_t)head * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * ldv + (size_t)head * vdim + j0;
    const size_t plane = ((size_t)c * a.heads + head) * dim * vdim + j0;
    copy_tile<LO_THREADS, 16>(sq, qld, qg, ldk, LC, cnt, dim, dim);
    copy_tile<LO_THREADS, JT / 8>(sh, VLD, hi + plane, vdim, dim, dim, JT, vdim - j0);
    copy_tile<LO_THREADS, JT / 8>(sl, VLD, lo + plane, vdim, dim, dim, JT, vdim - j0);
    cp_async_commit();
    copy_tile<LO_THREADS, 16>(sk, qld, kg, ldk, LC, cnt, dim, dim);
    copy_tile<LO_THREADS, JT / 8>(sv, VLD, vg, ldv, LC, cnt, JT, vdim - j0);
    cp_async_commit();
    for (int i = tid; i <= LC; i += LO_THREADS) pw[i] = a.decay_pow[head * (LC + 1) + i];
    cp_async_wait<1>();
    __syncthreads();
    // the causal work grows with the tokens' place in the chunk: the four warps of a scheduler (warp % 4) take an early and a
    // late sixteen for each half of the columns
    const int wr = (warp >> 2) & 1 ? 7 - (warp & 3) : warp & 3, jw = (warp >> 3) * (JT / 2);
    const int t0 = wr * 16, tl = t0 + (lane >> 2), dk = dim / 16;      // this thread's rows: tl, tl + 8
    const uint32_t qaddr = smem_u32(sq + (wr * 16 + (lane & 15)) * qld + (lane >> 4) * 8);
    float acc[2 * NP][4], low[2 * NP][4];                        // the state's second terms have sums of their own
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] = low[nt][e] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < dk; ++kk) {
        uint32_t qa[4], b[NP][4], d[NP][4];
        ldsm4(qa, qaddr + kk * 32);
#pragma unroll
        for (int np = 0; np < NP; ++np) {
            const int off = (kk * 16 + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8;
            ldsm4_t(b[np], smem_u32(sh + off));
            ldsm4_t(d[np], smem_u32(sl + off));
        }
        mma_row<NP>(acc, qa, b);
        mma_row<NP>(low, qa, d);
    }
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] += low[nt][e];
    const float d0 = pw[tl + 1], d1 = pw[tl + 9];
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt) { acc[nt][0] *= d0; acc[nt][1] *= d0; acc[nt][2] *= d1; acc[nt][3] *= d1; }
    cp_async_wait<0>();
    __syncthreads();
    if (t0 >= cnt || j0 + jw >= vdim) return;
    for (int s0 = 0; s0 < t0 + 16; s0 += 32) {         // 32 keys each, up to the diagonal (a last half block is masked)
        float sc[4][4] = {};
        const uint32_t kaddr = smem_u32(sk + (s0 + (lane & 7) + ((lane >> 4) & 1) * 8) * qld + ((lane >> 3) & 1) * 8);
#pragma unroll 4
        for (int kk = 0; kk < dk; ++kk) {
            uint32_t qa[4], b[4], d[4];
            ldsm4(qa, qaddr + kk * 32);
            ldsm4(b, kaddr + kk * 32);
            ldsm4(d, kaddr + 32 * qld + kk * 32);      // 16 rows on
            mma16816(sc[0], qa, b[0], b[1]);
            mma16816(sc[1], qa, b[2], b[3]);
            mma16816(sc[2], qa, d[0], d[1]);
            mma16816(sc[3], qa, d[2], d[3]);
        }
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = tl + (e >> 1) * 8 - (s0 + nt * 8 + 2 * (lane & 3) + (e & 1));
                sc[nt][e] = d >= 0 ? sc[nt][e] * pw[d] : 0.f;
            }
#pragma unroll
        for (int hb = 0; hb < 2; ++hb) {
            uint32_t b[NP][4];
#pragma unroll
            for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sv + (s0 + hb * 16 + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8));
            uint32_t ph[4], pl[4];
            split_pair(sc[2 * hb][0], sc[2 * hb][1], ph[0], pl[0]);
            split_pair(sc[2 * hb][2], sc[2 * hb][3], ph[1], pl[1]);
            split_pair(sc[2 * hb + 1][0], sc[2 * hb + 1][1], ph[2], pl[2]);
            split_pair(sc[2 * hb + 1][2], sc[2 * hb + 1][3], ph[3], pl[3]);
            mma_row<NP>(acc, ph, b);
            mma_row<NP>(acc, pl, b);
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int t = tl + h * 8;
        if (t >= cnt) continue;
        float* orow = a.o + (row0 + t) * ldv + (size_t)head * vdim + j0;
#pragma unroll
        for (int nt = 0; nt < 2 * NP; ++nt) {
            const int j = jw + nt * 8 + 2 * (lane & 3);
            if (j0 + j < vdim) *reinterpret_cast<float2*>(orow + j) = make_float2(acc[nt][2 * h], acc[nt][2 * h + 1]);
        }
    }
}

size_t lightning_scratch_bytes(int n, int heads, int dim, int vdim) { return (size_t)((n + LC - 1) / LC) * heads * dim * vdim * (sizeof(float) + 2 * sizeof(bf16)); }
// value columns of one CTA: 128 unless the head has no more than 64, or its dim leaves no room for them
static int column_tile(int dim, int vdim) { return vdim > 64 && lo_smem(dim, 128) + 1024 <= 232448 ? 128 : 64; }
bool lightning_chunked_fits(int dim) { return lo_smem(dim, 64) + 1024 <= 232448; }
template <int JT>
static int chunked(Stream& st, const LightningArgs& a) {
    const int nchunks = (a.n + LC - 1) / LC, jt = (a.vdim + JT - 1) / JT;
    const size_t elems = (size_t)nchunks * a.heads * a.dim * a.vdim;
    float* kv = reinterpret_cast<float*>(a.scratch);
    bf16 *hi = reinterpret_cast<bf16*>(kv + elems), *lo = hi + elems;
    int rc = allow_smem(k_lightning_kv<JT>, lk_smem(a.dim, JT));
    if (!rc) rc = launch(st, k_lightning_kv<JT>, dim3(nchunks, a.heads, jt), dim3(LK_THREADS), lk_smem(a.dim, JT), a, kv);
    const size_t quads = (size_t)a.heads * a.dim * a.vdim / 4;
    if (!rc) rc = launch(st, k_lightning_scan, dim3((unsigned)((quads + LN_THREADS - 1) / LN_THREADS)), dim3(LN_THREADS), 0, a, (const float*)kv, hi, lo);
    if (!rc) rc = allow_smem(k_lightning_out<JT>, lo_smem(a.dim, JT));
    if (!rc) rc = launch(st, k_lightning_out<JT>, dim3(nchunks, a.heads, jt), dim3(LO_THREADS), lo_smem(a.dim, JT), a, (const bf16*)hi, (const bf16*)lo);
    return rc;
}
int lightning_chunked(Stream& st, const LightningArgs& a) {
    if (!lightning_chunked_fits(a.dim) || !a.scratch) return MQ_ERR_UNSUPPORTED;
    return column_tile(a.dim, a.vdim) == 128 ? chunked<128>(st, a) : chunked<64>(st, a);
}

}  // namespace hy
}  // namespace mq
