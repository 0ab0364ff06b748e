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

// ---------------------------------------------------------------- chunked: what every chunk adds to the state
// One CTA per (chunk, head, 64 value columns): KV = sum over the chunk's n tokens of decay^(n - 1 - t) k_t v_t^T, fp32.
// Warp w takes rows 16 w + 128 x of the head's dim.
constexpr int LK_THREADS = 256, LO_VLD = 64 + 8;
static size_t lk_smem(int dim) { return (size_t)LC * (dim + 8 + LO_VLD) * 2; }
__global__ void __launch_bounds__(LK_THREADS) k_lightning_kv(LightningArgs a, float* __restrict__ kv) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t lk_raw[];
    __shared__ float pw[LC];                                   // by token: decay^(n - 1 - t)
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, c = blockIdx.x, j0 = blockIdx.z * 64;
    const int dim = a.dim, vdim = a.vdim, kld = dim + 8, dv8 = dim / 8;
    bf16* sk = reinterpret_cast<bf16*>(lk_raw);
    bf16* sv = sk + LC * kld;
    const int cnt = min(LC, a.n - c * LC);
    const size_t ldk = (size_t)a.heads * dim, ldv = (size_t)a.heads * vdim, row0 = (size_t)c * LC;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * ldk + (size_t)head * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * ldv + (size_t)head * vdim + j0;
    for (int x = tid; x < LC * dv8; x += LK_THREADS) {
        const int t = x / dv8, col = (x % dv8) * 8;
        cp_async16_zfill(sk + t * kld + col, t < cnt ? kg + t * ldk + col : kg, t < cnt);
    }
    for (int x = tid; x < LC * 8; x += LK_THREADS) {
        const int t = x >> 3, col = (x & 7) * 8;
        const bool ok = t < cnt && j0 + col < vdim;
        cp_async16_zfill(sv + t * LO_VLD + col, ok ? vg + t * ldv + col : vg, ok);
    }
    cp_async_commit();
    if (tid < LC) pw[tid] = tid < cnt ? a.decay_pow[head * (LC + 1) + cnt - 1 - tid] : 0.f;
    cp_async_wait_all();
    __syncthreads();
    const int ksteps = (cnt + 15) / 16;
    for (int i0 = warp * 16; i0 < dim; i0 += 128) {
        float acc[8][4];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
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
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b[4];
                ldsm4_t(b, smem_u32(sv + (t0 + (lane & 15)) * LO_VLD + np * 16 + (lane >> 4) * 8));
                mma16816(acc[2 * np], ah, b[0], b[1]);
                mma16816(acc[2 * np + 1], ah, b[2], b[3]);
                mma16816(acc[2 * np], al, b[0], b[1]);
                mma16816(acc[2 * np + 1], al, b[2], b[3]);
            }
        }
        float* dst = kv + ((size_t)c * a.heads + head) * dim * vdim + (size_t)(i0 + (lane >> 2)) * vdim + j0 + 2 * (lane & 3);
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
            if (j0 + nt * 8 < vdim) {
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
// One CTA per (half chunk, head, 64 value columns); warp w takes the tokens t0 = 64 half + 16 w .. t0 + 15 of the chunk:
// o_t = decay^(t + 1) q_t S + sum over s <= t of (q_t k_s) decay^(t - s) v_s      (t, s within the chunk)
constexpr int LO_THREADS = 128;
static size_t lo_smem(int dim) { return ((size_t)(64 + LC) * (dim + 8) + (size_t)LC * LO_VLD + (size_t)2 * dim * LO_VLD) * 2; }
__global__ void __launch_bounds__(LO_THREADS) k_lightning_out(LightningArgs a, const bf16* __restrict__ hi, const bf16* __restrict__ lo) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t lo_raw[];
    __shared__ float pw[LC + 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, c = blockIdx.x >> 1, half = blockIdx.x & 1, j0 = blockIdx.z * 64;
    const int dim = a.dim, vdim = a.vdim, qld = dim + 8;
    const int cnt = min(LC, a.n - c * LC), q0 = half * 64;
    if (q0 >= cnt) return;
    bf16* sq = reinterpret_cast<bf16*>(lo_raw);                // 64 rows
    bf16* sk = sq + 64 * qld;
    bf16* sv = sk + LC * qld;
    bf16* sh = sv + LC * LO_VLD;
    bf16* sl = sh + dim * LO_VLD;
    const int nkeys = min(q0 + 64, LC);                        // rows of k, v this half may see
    const size_t ldk = (size_t)a.heads * dim, ldv = (size_t)a.heads * vdim, row0 = (size_t)c * LC;
    const bf16* qg = reinterpret_cast<const bf16*>(a.q) + row0 * ldk + (size_t)head * dim;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * ldk + (size_t)head * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * ldv + (size_t)head * vdim + j0;
    const size_t plane = ((size_t)c * a.heads + head) * dim * vdim + j0;
    const int dv8 = dim / 8;
    for (int x = tid; x < 64 * dv8; x += LO_THREADS) {
        const int t = x / dv8, col = (x % dv8) * 8;
        const bool ok = q0 + t < cnt;
        cp_async16_zfill(sq + t * qld + col, ok ? qg + (q0 + t) * ldk + col : qg, ok);
    }
    for (int x = tid; x < dim * 8; x += LO_THREADS) {
        const int i = x >> 3, col = (x & 7) * 8;
        const bool ok = j0 + col < vdim;
        cp_async16_zfill(sh + i * LO_VLD + col, ok ? hi + plane + (size_t)i * vdim + col : hi, ok);
        cp_async16_zfill(sl + i * LO_VLD + col, ok ? lo + plane + (size_t)i * vdim + col : lo, ok);
    }
    cp_async_commit();
    for (int x = tid; x < nkeys * dv8; x += LO_THREADS) {
        const int t = x / dv8, col = (x % dv8) * 8;
        const bool ok = t < cnt;
        cp_async16_zfill(sk + t * qld + col, ok ? kg + t * ldk + col : kg, ok);
    }
    for (int x = tid; x < nkeys * 8; x += LO_THREADS) {
        const int t = x >> 3, col = (x & 7) * 8;
        const bool ok = t < cnt && j0 + col < vdim;
        cp_async16_zfill(sv + t * LO_VLD + col, ok ? vg + t * ldv + col : vg, ok);
    }
    cp_async_commit();
    for (int i = tid; i <= LC; i += LO_THREADS) pw[i] = a.decay_pow[head * (LC + 1) + i];
    cp_async_wait<1>();
    __syncthreads();
    const int t0 = q0 + warp * 16, tl = t0 + (lane >> 2), dk = dim / 16;    // this thread's rows: tl, tl + 8
    const uint32_t qaddr = smem_u32(sq + (warp * 16 + (lane & 15)) * qld + (lane >> 4) * 8);
    float acc[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < dk; ++kk) {
        uint32_t qa[4];
        ldsm4(qa, qaddr + kk * 32);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
            uint32_t b[4], d[4];
            const int off = (kk * 16 + (lane & 15)) * LO_VLD + np * 16 + (lane >> 4) * 8;
            ldsm4_t(b, smem_u32(sh + off));
            ldsm4_t(d, smem_u32(sl + off));
            mma16816(acc[2 * np], qa, b[0], b[1]);
            mma16816(acc[2 * np + 1], qa, b[2], b[3]);
            mma16816(acc[2 * np], qa, d[0], d[1]);
            mma16816(acc[2 * np + 1], qa, d[2], d[3]);
        }
    }
    const float d0 = pw[tl + 1], d1 = pw[tl + 9];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) { acc[nt][0] *= d0; acc[nt][1] *= d0; acc[nt][2] *= d1; acc[nt][3] *= d1; }
    cp_async_wait<0>();
    __syncthreads();
    if (t0 >= cnt) return;
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
            uint32_t ph[4], pl[4];
            split_pair(sc[2 * hb][0], sc[2 * hb][1], ph[0], pl[0]);
            split_pair(sc[2 * hb][2], sc[2 * hb][3], ph[1], pl[1]);
            split_pair(sc[2 * hb + 1][0], sc[2 * hb + 1][1], ph[2], pl[2]);
            split_pair(sc[2 * hb + 1][2], sc[2 * hb + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b[4];
                ldsm4_t(b, smem_u32(sv + (s0 + hb * 16 + (lane & 15)) * LO_VLD + np * 16 + (lane >> 4) * 8));
                mma16816(acc[2 * np], ph, b[0], b[1]);
                mma16816(acc[2 * np + 1], ph, b[2], b[3]);
                mma16816(acc[2 * np], pl, b[0], b[1]);
                mma16816(acc[2 * np + 1], pl, b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int t = tl + h * 8;
        if (t >= cnt) continue;
        float* orow = a.o + (row0 + t) * ldv + (size_t)head * vdim + j0;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            const int j = nt * 8 + 2 * (lane & 3);
            if (j0 + j < vdim) *reinterpret_cast<float2*>(orow + j) = make_float2(acc[nt][2 * h], acc[nt][2 * h + 1]);
        }
    }
}

size_t lightning_scratch_bytes(int n, int heads, int dim, int vdim) { return (size_t)((n + LC - 1) / LC) * heads * dim * vdim * (sizeof(float) + 2 * sizeof(bf16)); }
bool lightning_chunked_fits(int dim) { return lo_smem(dim) + (LC + 1) * 4 + 64 <= 232448 && lk_smem(dim) + LC * 4 + 64 <= 232448; }
int lightning_chunked(Stream& st, const LightningArgs& a) {
    if (!lightning_chunked_fits(a.dim) || !a.scratch) return MQ_ERR_UNSUPPORTED;
    const int nchunks = (a.n + LC - 1) / LC, jt = (a.vdim + 63) / 64;
    const size_t elems = (size_t)nchunks * a.heads * a.dim * a.vdim;
    float* kv = reinterpret_cast<float*>(a.scratch);
    bf16 *hi = reinterpret_cast<bf16*>(kv + elems), *lo = hi + elems;
    int rc = allow_smem(k_lightning_kv, lk_smem(a.dim));
    if (!rc) rc = launch(st, k_lightning_kv, dim3(nchunks, a.heads, jt), dim3(LK_THREADS), lk_smem(a.dim), a, kv);
    const size_t quads = (size_t)a.heads * a.dim * a.vdim / 4;
    if (!rc) rc = launch(st, k_lightning_scan, dim3((unsigned)((quads + LN_THREADS - 1) / LN_THREADS)), dim3(LN_THREADS), 0, a, (const float*)kv, hi, lo);
    if (!rc) rc = allow_smem(k_lightning_out, lo_smem(a.dim));
    if (!rc) rc = launch(st, k_lightning_out, dim3(2 * nchunks, a.heads, jt), dim3(LO_THREADS), lo_smem(a.dim), a, (const bf16*)hi, (const bf16*)lo);
    return rc;
}

}  // namespace hy
}  // namespace mq
