// Grouped-query attention of the layer-listed decoder: heads share keys in groups, queries and keys are normed per
// head and rotated by halves, values are the keys as projected, positions may see only keys of their own
// chunk, and each head's output has a gate.
//
// More than one token: attn_rows norms and rotates the queries and writes the cache rows, then the causal attention
// of hy_latent.cu (tcgen05 or plain) runs over the caches.
// One token: ONE kernel.  A cluster of CTAs shares the visible keys of a key head; each CTA norms and rotates the
// group's queries for itself, takes its piece of the keys through mma.sync (the group's heads are the M of the
// product, so a cached row is read once for all of them), and the pieces meet through distributed shared memory.
// Cached rows are requested before the wait on the preceding kernel; the row of the token itself never
// passes through the cache: the CTA whose piece it ends computes it.
// Norms, rotations, scores and weights are 32-bit; scores are kept in units of log2.
#include "hy_common.cuh"

namespace mq {
namespace hy {

// ---------------------------------------------------------------- norm and rotation of one head, by one warp
// buf: dim floats of shared memory; on return it holds the head after norm and rotation.
template <typename T>
__device__ __forceinline__ void norm_rotate(const T* src, const HeadNorm& h, const float2* rope, float* buf) {
    const int lane = threadIdx.x & 31;
    float ss = 0.f;
    for (int i = lane * 4; i < h.dim; i += 128) {
        const float4 v = load4_cg(src + i);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        store4(buf + i, v);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)h.dim_n + h.eps);
    __syncwarp();
    for (int i = lane; i < h.dim; i += 32) buf[i] *= inv * h.w[i];
    __syncwarp();
    for (int i = lane; i < h.half; i += 32) {
        const float2 cs = rope[i];
        const float u = buf[i], v = buf[i + h.half];
        buf[i] = u * cs.x - v * cs.y;
        buf[i + h.half] = v * cs.x + u * cs.y;
    }
    __syncwarp();
}

// ---------------------------------------------------------------- several tokens
// One CTA per token, a warp per head: queries in place, keys and values into the caches.
constexpr int AR_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(AR_THREADS) k_attn_rows(AttnRowsArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float ar_buf[];                    // [warps][dim]
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, dim = a.qn.dim;
    const size_t pos = (size_t)a.pos0 + t;
    float* buf = ar_buf + warp * dim;
    const float2* rope = reinterpret_cast<const float2*>(a.qn.rope) + pos * a.qn.half;
    for (int x = warp; x < a.heads + a.kv_heads; x += AR_THREADS / 32) {
        const bool query = x < a.heads;
        const size_t kc = (pos * a.kv_heads + (x - a.heads)) * dim;
        T* dst = query ? reinterpret_cast<T*>(a.q) + ((size_t)t * a.heads + x) * dim : reinterpret_cast<T*>(a.k_cache) + kc;
        const T* src = query ? dst : reinterpret_cast<const T*>(a.k) + ((size_t)t * a.kv_heads + (x - a.heads)) * dim;
        norm_rotate(src, query ? a.qn : a.kn, rope, buf);
        for (int i = lane * 4; i < dim; i += 128) {
            store4(dst + i, load4(buf + i));
            if (!query) store4(reinterpret_cast<T*>(a.v_cache) + kc + i, load4_cg(src + i));
        }
        __syncwarp();
    }
}
template <typename T>
int attn_rows(Stream& st, const AttnRowsArgs& a) {
    const size_t smem = (size_t)(AR_THREADS / 32) * a.qn.dim * 4;
    const int rc = allow_smem(k_attn_rows<T>, smem);
    if (rc) return rc;
    return launch(st, k_attn_rows<T>, dim3(a.n), dim3(AR_THREADS), smem, a);
}
template int attn_rows<bf16>(Stream&, const AttnRowsArgs&);
template int attn_rows<float>(Stream&, const AttnRowsArgs&);

// ---------------------------------------------------------------- one token: what both kernels share
constexpr int AD_KEYS = 64;
struct Piece { int pos, first, kbeg, kend; };            // keys [kbeg, kend) of the visible [first, pos]
// the position was set before this step began
__device__ __forceinline__ Piece my_piece(const AttnDecodeArgs& a) {
    int pos = *a.position;
    if (pos < 0 || pos >= a.max_seq) {
        if (threadIdx.x == 0) atomicOr(a.status, MQ_STATUS_BAD_POSITION);
        pos = pos < 0 ? 0 : a.max_seq - 1;
    }
    const int first = a.chunk > 0 ? pos / a.chunk * a.chunk : 0, tiles = (pos - first) / AD_KEYS + 1;
    const int per = (tiles + (int)gridDim.x - 1) / (int)gridDim.x * AD_KEYS;
    const int kbeg = first + (int)blockIdx.x * per;
    return {pos, first, kbeg, min(kbeg + per, pos + 1)};
}
__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// a float in the shared memory of another CTA of the cluster
__device__ __forceinline__ float ld_cluster(const float* p, int rank) {
    uint32_t addr;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"(smem_u32(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
    return v;
}
// The pieces of all CTAs of the cluster -> out.  acc [rows][dim] and ml [rows][2] (maximum in log2 units, sum) of this CTA in
// shared memory; rows 0 .. rows - 1 are heads head0 ..  Every CTA writes its share of the elements.
template <typename T, int THREADS>
__device__ __forceinline__ void merge_pieces(const AttnDecodeArgs& a, const float* acc, const float* ml, int rows, int head0, int dim) {
    const int nc = gridDim.x, rank = blockIdx.x;
    __syncthreads();
    cluster_sync();
    for (int x = rank * THREADS + (int)threadIdx.x; x < rows * dim; x += nc * THREADS) {
        const int r = x / dim;
        float m = -INFINITY, l = 0.f, s = 0.f;
        for (int c = 0; c < nc; ++c) m = fmaxf(m, ld_cluster(ml + 2 * r, c));
        for (int c = 0; c < nc; ++c) {
            const float f = exp2f(ld_cluster(ml + 2 * r, c) - m);      // 0 for a CTA without keys
            l = fmaf(f, ld_cluster(ml + 2 * r + 1, c), l);
            s = fmaf(f, ld_cluster(acc + x, c), s);
        }
        const float gate = a.gate ? 1.0f / (1.0f + expf(-__ldcg(a.gate + head0 + r))) : 1.0f;
        reinterpret_cast<T*>(a.out)[(size_t)head0 * dim + x] = Elem<T>::put(s / l * gate);
    }
    cluster_sync();                                      // nobody leaves while its shared memory is read
}

// ---------------------------------------------------------------- one token: bf16
// Grid (pieces, key heads, groups of sixteen query heads), a cluster per (y, z).
constexpr int AD_THREADS = 256, AD_WARPS = 8, AD_MAXT = 4, AD_PLD = AD_KEYS + 8;
constexpr int AD_MAX_DIM = AD_MAXT * 64;
static size_t ad_smem(int dim, int stages) {
    return (size_t)(stages * 2 * AD_KEYS + 16 + 2) * (dim + 8) * 2 + (size_t)AD_WARPS * dim * 4 + (size_t)16 * dim * 4;
}
template <int STAGES>
__global__ void __launch_bounds__(AD_THREADS) k_attn_decode(AttnDecodeArgs a) {
    extern __shared__ __align__(16) uint8_t ad_raw[];
    __shared__ __align__(16) bf16 sp[16 * AD_PLD];
    __shared__ float smax[AD_WARPS][16], ssum[AD_WARPS][16], ml[32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, dim = a.qn.dim, ld = dim + 8, d8 = dim / 8;
    bf16* sk = reinterpret_cast<bf16*>(ad_raw);          // [STAGES][keys, then values][AD_KEYS][ld]
    bf16* sq = sk + STAGES * 2 * AD_KEYS * ld;           // [16][ld]
    bf16* snew = sq + 16 * ld;                           // key and value of the token itself
    float* buf = reinterpret_cast<float*>(snew + 2 * ld);    // [warps][dim]
    float* sacc = buf + AD_WARPS * dim;                  // [16][dim]
    const int g = blockIdx.y, group = a.heads / a.kv_heads, h0 = g * group + blockIdx.z * 16, nh = min(16, group - (int)blockIdx.z * 16);
    const Piece pc = my_piece(a);
    const int ntiles = pc.kend > pc.kbeg ? (pc.kend - pc.kbeg + AD_KEYS - 1) / AD_KEYS : 0;
    const bool has_new = ntiles > 0 && pc.kend == pc.pos + 1;
    const bf16 *kc = reinterpret_cast<const bf16*>(a.k_cache) + (size_t)g * dim, *vc = reinterpret_cast<const bf16*>(a.v_cache) + (size_t)g * dim;
    const size_t row = (size_t)a.kv_heads * dim;
    // A tile's cached rows; those beyond the piece become zeros, that of the token itself is left out
    auto fetch = [&](int t) {
        if (t < ntiles) {
            bf16* dst = sk + (t % STAGES) * 2 * AD_KEYS * ld;
            const int k0 = pc.kbeg + t * AD_KEYS;
            for (int x = tid; x < AD_KEYS * d8; x += AD_THREADS) {
                const int j = x / d8, col = (x - j * d8) * 8, key = k0 + j;
                if (key == pc.pos) continue;
                const bool ok = key < pc.kend;
                cp_async16_zfill(dst + j * ld + col, ok ? kc + key * row + col : kc, ok);
                cp_async16_zfill(dst + (AD_KEYS + j) * ld + col, ok ? vc + key * row + col : vc, ok);
            }
        }
        cp_async_commit();                               // an empty group beyond the last tile: the count stays in step
    };
    pdl_trigger();
#pragma unroll
    for (int t = 0; t < STAGES; ++t) fetch(t);
    pdl_wait_cta();
    const float2* rope = reinterpret_cast<const float2*>(a.qn.rope) + (size_t)pc.pos * a.qn.half;
    const bf16* knew = reinterpret_cast<const bf16*>(a.k) + (size_t)g * dim;
    for (int x = warp; x < 16 + (has_new ? 1 : 0); x += AD_WARPS) {
        float* b = buf + warp * dim;
        bf16* dst = x < 16 ? sq + x * ld : snew;
        if (x >= nh && x < 16) {
            for (int i = lane * 4; i < dim; i += 128) store4(dst + i, make_float4(0.f, 0.f, 0.f, 0.f));
            continue;
        }
        norm_rotate(x < 16 ? reinterpret_cast<const bf16*>(a.q) + (size_t)(h0 + x) * dim : knew, x < 16 ? a.qn : a.kn, rope, b);
        for (int i = lane * 4; i < dim; i += 128) store4(dst + i, load4(b + i));
        if (x == 16)
            for (int i = lane * 4; i < dim; i += 128) {
                const float4 v = load4_cg(knew + i);
                store4(snew + ld + i, v);
                if (blockIdx.z == 0) {
                    store4(reinterpret_cast<bf16*>(a.k_cache) + pc.pos * row + (size_t)g * dim + i, load4(b + i));
                    store4(reinterpret_cast<bf16*>(a.v_cache) + pc.pos * row + (size_t)g * dim + i, v);
                }
            }
        __syncwarp();
    }
    __syncthreads();
    const float c = a.scale * LOG2E;
    const int nt8 = dim / 8, tpw = 2 * ((nt8 + 15) / 16), tile0 = warp * tpw;      // this warp's 8-column tiles of the output
    float acc[AD_MAXT][4];
#pragma unroll
    for (int i = 0; i < AD_MAXT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};               // rows lane / 4, lane / 4 + 8
    const int r = lane >> 2;
    const uint32_t qa = smem_u32(sq + (lane & 15) * ld + (lane >> 4) * 8);
    for (int t = 0; t < ntiles; ++t) {
        bf16 *tk = sk + (t % STAGES) * 2 * AD_KEYS * ld, *tv = tk + AD_KEYS * ld;
        const int k0 = pc.kbeg + t * AD_KEYS;
        cp_async_wait<STAGES - 1>();
        if (has_new && t == ntiles - 1 && tid < 2 * d8) {
            const int j = pc.pos - k0, col = (tid % d8) * 8;
            *reinterpret_cast<uint4*>((tid < d8 ? tk : tv) + j * ld + col) = *reinterpret_cast<const uint4*>((tid < d8 ? snew : snew + ld) + col);
        }
        __syncthreads();
        // scores of this warp's eight keys
        float s0[4] = {}, s1[4] = {};
        const uint32_t kb = smem_u32(tk + (warp * 8 + r) * ld + (lane & 3) * 2);
        int ks = 0;
#pragma unroll 4
        for (; ks + 1 < dim / 16; ks += 2) {
            uint32_t q4[4], r4[4];
            ldsm4(q4, qa + ks * 32);
            ldsm4(r4, qa + ks * 32 + 32);
            mma16816(s0, q4, lds32(kb + ks * 32), lds32(kb + ks * 32 + 16));
            mma16816(s1, r4, lds32(kb + ks * 32 + 32), lds32(kb + ks * 32 + 48));
        }
        if (ks < dim / 16) {
            uint32_t q4[4];
            ldsm4(q4, qa + ks * 32);
            mma16816(s0, q4, lds32(kb + ks * 32), lds32(kb + ks * 32 + 16));
        }
        float s[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int key = k0 + warp * 8 + 2 * (lane & 3) + (e & 1);
            s[e] = key < pc.kend ? (s0[e] + s1[e]) * c : -INFINITY;
        }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float v = fmaxf(s[2 * h], s[2 * h + 1]);
            v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
            v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
            if ((lane & 3) == 0) smax[warp][r + 8 * h] = v;
        }
        __syncthreads();
        float alpha[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float mn = m[h];
#pragma unroll
            for (int w = 0; w < AD_WARPS; ++w) mn = fmaxf(mn, smax[w][r + 8 * h]);      // finite: every tile has a key
            alpha[h] = exp2f(m[h] - mn);
            m[h] = mn;
            const float p0 = exp2f(s[2 * h] - mn), p1 = exp2f(s[2 * h + 1] - mn);
            *reinterpret_cast<uint32_t*>(sp + (r + 8 * h) * AD_PLD + warp * 8 + 2 * (lane & 3)) = pack_bf16x2(p0, p1);
            float v = p0 + p1;
            v += __shfl_xor_sync(0xffffffffu, v, 1);
            v += __shfl_xor_sync(0xffffffffu, v, 2);
            if ((lane & 3) == 0) ssum[warp][r + 8 * h] = v;
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < AD_WARPS; ++w) v += ssum[w][r + 8 * h];
            l[h] = l[h] * alpha[h] + v;
        }
#pragma unroll
        for (int i = 0; i < AD_MAXT; ++i) { acc[i][0] *= alpha[0]; acc[i][1] *= alpha[0]; acc[i][2] *= alpha[1]; acc[i][3] *= alpha[1]; }
#pragma unroll
        for (int ks2 = 0; ks2 < AD_KEYS / 16; ++ks2) {
            uint32_t p4[4];
            ldsm4(p4, smem_u32(sp + (lane & 15) * AD_PLD + ks2 * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int i = 0; i < AD_MAXT; i += 2) {
                if (i >= tpw || tile0 + i >= nt8) break;
                uint32_t b[4];
                ldsm4_t(b, smem_u32(tv + (ks2 * 16 + (lane & 15)) * ld + (tile0 + i) * 8 + (lane >> 4) * 8));
                mma16816(acc[i], p4, b[0], b[1]);
                mma16816(acc[i + 1], p4, b[2], b[3]);
            }
        }
        __syncthreads();                                   // the stage, the weights and the maxima are overwritten next
        fetch(t + STAGES);
    }
    cp_async_wait_all();
#pragma unroll
    for (int h = 0; h < 2; ++h) {
#pragma unroll
        for (int i = 0; i < AD_MAXT; ++i) {
            if (i >= tpw || tile0 + i >= nt8) break;
            *reinterpret_cast<float2*>(sacc + (r + 8 * h) * dim + (tile0 + i) * 8 + 2 * (lane & 3)) = make_float2(acc[i][2 * h], acc[i][2 * h + 1]);
        }
        if (warp == 0 && (lane & 3) == 0) { ml[2 * (r + 8 * h)] = m[h]; ml[2 * (r + 8 * h) + 1] = l[h]; }
    }
    merge_pieces<bf16, AD_THREADS>(a, sacc, ml, nh, h0, dim);
}

// ---------------------------------------------------------------- one token: 32-bit caches, larger heads
// Grid (pieces, query heads), a cluster per head; a warp per key, then a thread per column.
constexpr int AP_THREADS = 128, AP_MAXC = 4;
template <typename T>
__global__ void __launch_bounds__(AP_THREADS) k_attn_decode_plain(AttnDecodeArgs a) {
    extern __shared__ float ap_buf[];                      // query, key of the token itself, output: [dim] each
    __shared__ float p[AD_KEYS], red[4], ml[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, dim = a.qn.dim, head = blockIdx.y, group = a.heads / a.kv_heads, g = head / group;
    float *sq = ap_buf, *snew = ap_buf + dim, *sacc = ap_buf + 2 * dim;
    pdl_trigger();
    pdl_wait_cta();
    const Piece pc = my_piece(a);
    const bool has_new = pc.kbeg < pc.kend && pc.kend == pc.pos + 1;
    const float2* rope = reinterpret_cast<const float2*>(a.qn.rope) + (size_t)pc.pos * a.qn.half;
    const T* knew = reinterpret_cast<const T*>(a.k) + (size_t)g * dim;
    const size_t row = (size_t)a.kv_heads * dim;
    T *kc = reinterpret_cast<T*>(a.k_cache) + (size_t)g * dim, *vc = reinterpret_cast<T*>(a.v_cache) + (size_t)g * dim;
    if (warp < 2) {
        float* b = warp ? snew : sq;
        norm_rotate(warp ? knew : reinterpret_cast<const T*>(a.q) + (size_t)head * dim, warp ? a.kn : a.qn, rope, b);
        for (int i = lane * 4; i < dim; i += 128) {
            float4 v = load4(b + i);
            if (warp && has_new && head % group == 0) {
                store4(kc + pc.pos * row + i, v);
                store4(vc + pc.pos * row + i, load4_cg(knew + i));
            }
            v = make_float4(Elem<T>::round(v.x), Elem<T>::round(v.y), Elem<T>::round(v.z), Elem<T>::round(v.w));      // as they are cached
            store4(b + i, v);
        }
    }
    __syncthreads();
    const float c = a.scale * LOG2E;
    float m = -INFINITY, l = 0.f, acc[AP_MAXC] = {};
    for (int k0 = pc.kbeg; k0 < pc.kend; k0 += AD_KEYS) {
        const int cnt = min(AD_KEYS, pc.kend - k0);
        float best = -INFINITY;
        for (int j = warp; j < cnt; j += 4) {
            const bool self = k0 + j == pc.pos;
            float s = 0.f;
            for (int i = lane * 4; i < dim; i += 128) {
                const float4 kv = self ? load4(snew + i) : load4_cg(kc + (k0 + j) * row + i), qv = load4(sq + i);
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
        for (int x = 0; x < AP_MAXC; ++x) {
            const int i = tid + x * AP_THREADS;
            if (i >= dim) break;
            float s = 0.f;
            for (int j = 0; j < cnt; ++j) {
                const T* v = k0 + j == pc.pos ? knew : vc + (k0 + j) * row;
                s = fmaf(p[j], Elem<T>::get(__ldcg(v + i)), s);
            }
            acc[x] = acc[x] * alpha + s;
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 0; x < AP_MAXC; ++x)
        if (tid + x * AP_THREADS < dim) sacc[tid + x * AP_THREADS] = acc[x];
    if (tid == 0) { ml[0] = m; ml[1] = l; }
    merge_pieces<T, AP_THREADS>(a, sacc, ml, 1, head, dim);
}

// ---------------------------------------------------------------- launches
template <typename T>
int attn_decode(Stream& st, const AttnDecodeArgs& a) {
    const int dim = a.qn.dim, most = a.chunk > 0 && a.chunk < a.max_seq ? a.chunk : a.max_seq;
    const int tiles = (most + AD_KEYS - 1) / AD_KEYS, pieces = tiles >= 8 ? 8 : tiles >= 4 ? 4 : tiles >= 2 ? 2 : 1;
    if (sizeof(T) == 2 && dim <= AD_MAX_DIM) {
        const dim3 grid(pieces, a.kv_heads, (a.heads / a.kv_heads + 15) / 16);
        const int per = (tiles + pieces - 1) / pieces;
        if (per >= 3 && ad_smem(dim, 4) <= 200 * 1024) {
            const int rc = allow_smem(k_attn_decode<4>, ad_smem(dim, 4));
            return rc ? rc : launch_cluster(st, k_attn_decode<4>, grid, dim3(AD_THREADS), ad_smem(dim, 4), pieces, a);
        }
        const int rc = allow_smem(k_attn_decode<2>, ad_smem(dim, 2));
        return rc ? rc : launch_cluster(st, k_attn_decode<2>, grid, dim3(AD_THREADS), ad_smem(dim, 2), pieces, a);
    }
    if (dim > AP_MAXC * AP_THREADS) return MQ_ERR_UNSUPPORTED;
    return launch_cluster(st, k_attn_decode_plain<T>, dim3(pieces, a.heads), dim3(AP_THREADS), (size_t)dim * 12, pieces, a);
}
template int attn_decode<bf16>(Stream&, const AttnDecodeArgs&);
template int attn_decode<float>(Stream&, const AttnDecodeArgs&);

}  // namespace hy
}  // namespace mq
