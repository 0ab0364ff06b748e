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

// The same in registers, a lane with four neighbouring elements, for heads of up to 128 whose rotated halves are whole quads.
__device__ __forceinline__ bool quad_head(const HeadNorm& h) { return h.dim <= 128 && h.half % 4 == 0; }
template <typename T>
__device__ __forceinline__ float4 norm_rotate_quad(const T* src, const HeadNorm& h, const float2* rope) {
    const int lane = threadIdx.x & 31, i = lane * 4, hq = h.half / 4;
    const bool in = i < h.dim, low = lane < hq, turns = lane < 2 * hq;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f), w = v, c0 = v, c1 = v;
    if (in) { v = load4_cg(src + i); w = load4(h.w + i); }
    if (turns) {
        const float4* p = reinterpret_cast<const float4*>(rope + (low ? i : i - h.half));
        c0 = p[0];                                       // cos, sin of two pairs
        c1 = p[1];
    }
    const float inv = 1.0f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / (float)h.dim_n + h.eps);
    v = make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w);
    const int other = !turns ? lane : low ? lane + hq : lane - hq;
    const float4 o = make_float4(__shfl_sync(0xffffffffu, v.x, other), __shfl_sync(0xffffffffu, v.y, other), __shfl_sync(0xffffffffu, v.z, other),
                                 __shfl_sync(0xffffffffu, v.w, other));
    if (!turns) return v;
    const float sg = low ? -1.0f : 1.0f;                 // u cos - v sin, v cos + u sin
    return make_float4(v.x * c0.x + sg * (o.x * c0.y), v.y * c0.z + sg * (o.y * c0.w), v.z * c1.x + sg * (o.z * c1.y), v.w * c1.z + sg * (o.w * c1.w));
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
    const bool quads = quad_head(a.qn);
    const float2* rope = reinterpret_cast<const float2*>(a.qn.rope) + pos * a.qn.half;
    for (int x = warp; x < a.heads + a.kv_heads; x += AR_THREADS / 32) {
        const bool query = x < a.heads;
        const size_t kc = (pos * a.kv_heads + (x - a.heads)) * dim;
        T* dst = query ? reinterpret_cast<T*>(a.q) + ((size_t)t * a.heads + x) * dim : reinterpret_cast<T*>(a.k_cache) + kc;
        const T* src = query ? dst : reinterpret_cast<const T*>(a.k) + ((size_t)t * a.kv_heads + (x - a.heads)) * dim;
        if (quads) {
            const float4 y = norm_rotate_quad(src, query ? a.qn : a.kn, rope);
            const int i = lane * 4;
            if (i < dim) {
                if (!query) store4(reinterpret_cast<T*>(a.v_cache) + kc + i, load4_cg(src + i));
                store4(dst + i, y);
            }
            continue;
        }
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
constexpr int AD_KEYS = 16;
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
// Grid (pieces, key heads, groups of sixteen query heads), a cluster per (y, z).  Every warp takes sixteen keys at a time
// through its own stages of shared memory and keeps its own maximum, sum and output, so that no tile needs a barrier; the
// weights of a tile stay in registers as the A operand of the second product.  The warps meet once, at the end.
// NT: 8-column tiles of the output, dim <= 8 NT.
constexpr int AD_THREADS = 256, AD_WARPS = 8;
constexpr int AD_MAX_DIM = 256;
static size_t ad_smem(int dim, int stages) {
    return (size_t)(AD_WARPS * stages * 2 * AD_KEYS + 16 + 2) * (dim + 8) * 2 + (size_t)AD_WARPS * dim * 4 + (size_t)16 * dim * 4;
}
template <int NT, int STAGES>
__global__ void __launch_bounds__(AD_THREADS) k_attn_decode(AttnDecodeArgs a) {
    extern __shared__ __align__(16) uint8_t ad_raw[];
    __shared__ float wm[AD_WARPS][16], wl[AD_WARPS][16], ml[32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, dim = a.qn.dim, ld = dim + 8, d8 = dim / 8;
    bf16* stages = reinterpret_cast<bf16*>(ad_raw);      // [warps][STAGES][keys, then values][AD_KEYS][ld]
    bf16* mine = stages + warp * STAGES * 2 * AD_KEYS * ld;
    bf16* sq = stages + AD_WARPS * STAGES * 2 * AD_KEYS * ld;    // [16][ld]
    bf16* snew = sq + 16 * ld;                           // key and value of the token itself
    float* buf = reinterpret_cast<float*>(snew + 2 * ld);    // [warps][dim]
    float* sacc = buf + AD_WARPS * dim;                  // [16][dim]
    const int g = blockIdx.y, group = a.heads / a.kv_heads, h0 = g * group + blockIdx.z * 16, nh = min(16, group - (int)blockIdx.z * 16);
    const Piece pc = my_piece(a);
    const int tiles = pc.kend > pc.kbeg ? (pc.kend - pc.kbeg + AD_KEYS - 1) / AD_KEYS : 0;
    const int count = tiles > warp ? (tiles - warp + AD_WARPS - 1) / AD_WARPS : 0;       // this warp's tiles: warp, warp + 8, ..
    const bool has_new = tiles > 0 && pc.kend == pc.pos + 1;
    const bf16 *kc = reinterpret_cast<const bf16*>(a.k_cache) + (size_t)g * dim, *vc = reinterpret_cast<const bf16*>(a.v_cache) + (size_t)g * dim;
    const size_t row = (size_t)a.kv_heads * dim;
    // A tile's cached rows; those beyond the piece become zeros, that of the token itself is left out
    auto fetch = [&](int i) {
        if (i < count) {
            bf16* dst = mine + (i % STAGES) * 2 * AD_KEYS * ld;
            const int k0 = pc.kbeg + (warp + i * AD_WARPS) * AD_KEYS;
            for (int x = lane; x < AD_KEYS * d8; x += 32) {
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
    for (int i = 0; i < STAGES; ++i) fetch(i);
    pdl_wait_cta();
    const float2* rope = reinterpret_cast<const float2*>(a.qn.rope) + (size_t)pc.pos * a.qn.half;
    const bf16* knew = reinterpret_cast<const bf16*>(a.k) + (size_t)g * dim;
    const bool quads = quad_head(a.qn);
    // query rows 0 .. nh - 1, the new key as row nh; the remaining rows of the product are zeros
    for (int x = warp; x < nh + (has_new ? 1 : 0); x += AD_WARPS) {
        float* b = buf + warp * dim;
        const bool key = x == nh;
        bf16* dst = key ? snew : sq + x * ld;
        const bf16* src = key ? knew : reinterpret_cast<const bf16*>(a.q) + (size_t)(h0 + x) * dim;
        if (quads) {
            const float4 y = norm_rotate_quad(src, key ? a.kn : a.qn, rope);
            if (lane * 4 < dim) store4(b + lane * 4, y);
        } else {
            norm_rotate(src, key ? a.kn : a.qn, rope, b);
        }
        for (int i = lane * 4; i < dim; i += 128) store4(dst + i, load4(b + i));
        if (key)
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
    for (int x = tid; x < (16 - nh) * d8; x += AD_THREADS)
        *reinterpret_cast<uint4*>(sq + (nh + x / d8) * ld + (x % d8) * 8) = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const float c = a.scale * LOG2E;
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};               // rows lane / 4, lane / 4 + 8; l: this lane's keys
    const int r = lane >> 2;
    const uint32_t qa = smem_u32(sq + (lane & 15) * ld + (lane >> 4) * 8);
    const int koff = ((lane & 7) + ((lane >> 4) & 1) * 8) * ld + ((lane >> 3) & 1) * 8, voff = (AD_KEYS + (lane & 15)) * ld + (lane >> 4) * 8;
    for (int i = 0; i < count; ++i) {
        bf16* tile = mine + (i % STAGES) * 2 * AD_KEYS * ld;
        const int k0 = pc.kbeg + (warp + i * AD_WARPS) * AD_KEYS;
        cp_async_wait<STAGES - 1>();
        if (pc.pos >= k0 && pc.pos < k0 + AD_KEYS)       // the token itself (in the last piece only)
            for (int x = lane; x < 2 * d8; x += 32) {
                const bool val = x >= d8;
                *reinterpret_cast<uint4*>(tile + ((val ? AD_KEYS : 0) + pc.pos - k0) * ld + (x % d8) * 8) =
                    *reinterpret_cast<const uint4*>(snew + (val ? ld : 0) + (x % d8) * 8);
            }
        __syncwarp();
        float s0[2][4] = {}, s1[2][4] = {};              // scores of keys 0-7, 8-15; two sums each break the chain of products
        const uint32_t ka = smem_u32(tile + koff);
        int ks = 0;
#pragma unroll 4
        for (; ks + 1 < dim / 16; ks += 2) {
            uint32_t q0[4], q1[4], b0[4], b1[4];
            ldsm4(q0, qa + ks * 32);
            ldsm4(b0, ka + ks * 32);
            ldsm4(q1, qa + ks * 32 + 32);
            ldsm4(b1, ka + ks * 32 + 32);
            mma16816(s0[0], q0, b0[0], b0[1]);
            mma16816(s0[1], q0, b0[2], b0[3]);
            mma16816(s1[0], q1, b1[0], b1[1]);
            mma16816(s1[1], q1, b1[2], b1[3]);
        }
        if (ks < dim / 16) {
            uint32_t q0[4], b0[4];
            ldsm4(q0, qa + ks * 32);
            ldsm4(b0, ka + ks * 32);
            mma16816(s0[0], q0, b0[0], b0[1]);
            mma16816(s0[1], q0, b0[2], b0[3]);
        }
        float s[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[n][e] = k0 + n * 8 + 2 * (lane & 3) + (e & 1) < pc.kend ? (s0[n][e] + s1[n][e]) * c : -INFINITY;
        uint32_t p4[4];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float v = fmaxf(fmaxf(s[0][2 * h], s[0][2 * h + 1]), fmaxf(s[1][2 * h], s[1][2 * h + 1]));
            v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
            v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
            const float mn = fmaxf(m[h], v), alpha = exp2f(m[h] - mn);   // finite: every tile has a key
            m[h] = mn;
            const float p0 = exp2f(s[0][2 * h] - mn), p1 = exp2f(s[0][2 * h + 1] - mn), p2 = exp2f(s[1][2 * h] - mn), p3 = exp2f(s[1][2 * h + 1] - mn);
            l[h] = l[h] * alpha + (p0 + p1) + (p2 + p3);
            p4[h] = pack_bf16x2(p0, p1);
            p4[2 + h] = pack_bf16x2(p2, p3);
#pragma unroll
            for (int n = 0; n < NT; ++n) { acc[n][2 * h] *= alpha; acc[n][2 * h + 1] *= alpha; }
        }
        const uint32_t va = smem_u32(tile + voff);
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
            if (n * 8 >= dim) break;
            uint32_t b[4];
            ldsm4_t(b, va + n * 16);
            mma16816(acc[n], p4, b[0], b[1]);
            mma16816(acc[n + 1], p4, b[2], b[3]);
        }
        __syncwarp();                                      // the stage is overwritten next
        fetch(i + STAGES);
    }
    cp_async_wait_all();
    __syncwarp();
    float* wacc = reinterpret_cast<float*>(mine);          // [16][dim] over this warp's stages
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        const int x = r + 8 * h;
        if ((lane & 3) == 0) { wm[warp][x] = m[h]; wl[warp][x] = l[h]; }
        if (x < nh) {
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                if (n * 8 >= dim) break;
                *reinterpret_cast<float2*>(wacc + x * dim + n * 8 + 2 * (lane & 3)) = make_float2(acc[n][2 * h], acc[n][2 * h + 1]);
            }
        }
    }
    __syncthreads();
    // the warps' shares -> this CTA's; one without keys has the maximum -inf and weighs nothing
    for (int x = tid; x < nh * dim; x += AD_THREADS) {
        const int y = x / dim;
        float mx = -INFINITY, lsum = 0.f, sum = 0.f;
#pragma unroll
        for (int w = 0; w < AD_WARPS; ++w) mx = fmaxf(mx, wm[w][y]);
        if (mx > -INFINITY)
#pragma unroll
            for (int w = 0; w < AD_WARPS; ++w) {
                const float f = exp2f(wm[w][y] - mx);
                lsum = fmaf(f, wl[w][y], lsum);
                sum = fmaf(f, reinterpret_cast<const float*>(stages + w * STAGES * 2 * AD_KEYS * ld)[x], sum);
            }
        sacc[x] = sum;
        if (x == y * dim) { ml[2 * y] = mx; ml[2 * y + 1] = lsum; }
    }
    merge_pieces<bf16, AD_THREADS>(a, sacc, ml, nh, h0, dim);
}

// ---------------------------------------------------------------- one token: 32-bit caches, larger heads
// Grid (pieces, query heads), a cluster per head; a warp per key, then a thread per column.
constexpr int AP_THREADS = 128, AP_MAXC = 4, AP_KEYS = 64;
template <typename T>
__global__ void __launch_bounds__(AP_THREADS) k_attn_decode_plain(AttnDecodeArgs a) {
    extern __shared__ float ap_buf[];                      // query, key of the token itself, output: [dim] each
    __shared__ float p[AP_KEYS], red[4], ml[2];
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
    for (int k0 = pc.kbeg; k0 < pc.kend; k0 += AP_KEYS) {
        const int cnt = min(AP_KEYS, pc.kend - k0);
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
    // one piece per 64 keys that a position may see, up to the portable cluster size
    const int tiles = (most + 63) / 64, pieces = tiles >= 8 ? 8 : tiles >= 4 ? 4 : tiles >= 2 ? 2 : 1;
    if (sizeof(T) == 2 && dim <= AD_MAX_DIM) {
        const dim3 grid(pieces, a.kv_heads, (a.heads / a.kv_heads + 15) / 16);
        auto go = [&](auto kernel, int stages) {
            const int rc = allow_smem(kernel, ad_smem(dim, stages));
            return rc ? rc : launch_cluster(st, kernel, grid, dim3(AD_THREADS), ad_smem(dim, stages), pieces, a);
        };
        if (dim <= 64) return go(k_attn_decode<8, 3>, 3);
        if (dim <= 128) return go(k_attn_decode<16, 2>, 2);
        return go(k_attn_decode<32, 1>, 1);
    }
    if (dim > AP_MAXC * AP_THREADS) return MQ_ERR_UNSUPPORTED;
    return launch_cluster(st, k_attn_decode_plain<T>, dim3(pieces, a.heads), dim3(AP_THREADS), (size_t)dim * 12, pieces, a);
}
template int attn_decode<bf16>(Stream&, const AttnDecodeArgs&);
template int attn_decode<float>(Stream&, const AttnDecodeArgs&);

}  // namespace hy
}  // namespace mq
