// Products of one token: y = W v.  A token reads every weight once, so the kernel is a
// stream of weight rows: each warp owns a contiguous range of row pairs, i.e. one
// contiguous piece of the matrix, and keeps a ring of 16-byte loads per lane in flight.
// The ring is filled BEFORE the wait on the preceding kernel (weights are written by nothing
// on the stream), so the first 64 KB per SM cross HBM while that kernel is still running.
// What the vector is made of (norm of the residual stream, the loop's input, the gated norm
// of lightning attention beside the feed-forward's activations) is computed by every CTA for
// itself; what becomes of the result (segments with activations, residual add, LM head with
// arg-max) follows from a shared-memory batch of finished rows, one lane per row pair.
#include "hy_common.cuh"

namespace mq {
namespace hy {

constexpr int GV_WARPS = 8, GV_THREADS = GV_WARPS * 32;
constexpr int GV_CS = 4;          // 16-byte loads per lane of one ring slot
constexpr int GV_D = 4;           // ring slots
constexpr int GV_BATCH = 64;      // finished rows per warp between two epilogues

// Position of element k of the vector in shared memory: a lane multiplies 16 bytes of a weight row (8 bf16 or 4 fp32
// elements) and reads its vector elements as float4 without bank conflicts.
template <typename T> __device__ __forceinline__ int vec_pos(int k);
template <> __device__ __forceinline__ int vec_pos<bf16>(int k) { return (k & ~255) + ((k >> 2) & 1) * 128 + ((k & 255) >> 3) * 4 + (k & 3); }
template <> __device__ __forceinline__ int vec_pos<float>(int k) { return k; }

__device__ __forceinline__ uint4 ld_weight(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ float dot16(const uint4& w, const float* v, int lane, const bf16*) {
    const float4 a = load4(v + lane * 4), b = load4(v + 128 + lane * 4);
    float s0 = bf_lo(w.x) * a.x, s1 = bf_hi(w.x) * a.y;
    s0 = fmaf(bf_lo(w.y), a.z, s0); s1 = fmaf(bf_hi(w.y), a.w, s1);
    s0 = fmaf(bf_lo(w.z), b.x, s0); s1 = fmaf(bf_hi(w.z), b.y, s1);
    s0 = fmaf(bf_lo(w.w), b.z, s0); s1 = fmaf(bf_hi(w.w), b.w, s1);
    return s0 + s1;
}
__device__ __forceinline__ float dot16(const uint4& w, const float* v, int lane, const float*) {
    const float4 a = load4(v + lane * 4);
    float s0 = __uint_as_float(w.x) * a.x, s1 = __uint_as_float(w.y) * a.y;
    s0 = fmaf(__uint_as_float(w.z), a.z, s0); s1 = fmaf(__uint_as_float(w.w), a.w, s1);
    return s0 + s1;
}
// larger value first, then the lower index
__device__ __forceinline__ unsigned long long best_key(float v, int i) {
    uint32_t u = __float_as_uint(v);
    u = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
    return ((unsigned long long)u << 32) | (unsigned long long)(0xffffffffu - (uint32_t)i);
}

template <typename T>
__device__ __forceinline__ void put_vec(float* vec, int i, float4 v) {   // i a multiple of 4
    store4(vec + vec_pos<T>(i), make_float4(Elem<T>::round(v.x), Elem<T>::round(v.y), Elem<T>::round(v.z), Elem<T>::round(v.w)));
}

template <typename T, int VEC, int OUT>
__global__ void __launch_bounds__(GV_THREADS, 2) k_gemv(GemvArgs a) {
    constexpr int EPL = Elem<T>::PER16;
    constexpr int SEG = 32 * EPL, CHUNK = GV_CS * SEG;       // elements of one warp-wide load, of one ring slot
    extern __shared__ float vec[];
    __shared__ float red[GV_WARPS];
    __shared__ float done[GV_WARPS][GV_BATCH];
    __shared__ unsigned long long wbest[GV_WARPS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int K = a.K, nch = (K + CHUNK - 1) / CHUNK;
    const T* W = reinterpret_cast<const T*>(a.W);
    const long long pairs = (a.rows + 1) / 2, gw = (long long)blockIdx.x * GV_WARPS + warp, tw = (long long)gridDim.x * GV_WARPS;
    const int r0 = 2 * (int)(pairs * gw / tw), r1 = min(2 * (int)(pairs * (gw + 1) / tw), a.rows);

    uint4 ring[GV_D][GV_CS];
    int lrow = r0, lch = 0;
    auto load = [&](uint4 (&b)[GV_CS]) {
        if (lrow < r1) {
            const int c0 = lch * CHUNK + lane * EPL;
            const T* p = W + (size_t)lrow * K + c0;
#pragma unroll
            for (int s = 0; s < GV_CS; ++s) b[s] = c0 + s * SEG < K ? ld_weight(p + s * SEG) : make_uint4(0u, 0u, 0u, 0u);
            if (++lch == nch) { lch = 0; ++lrow; }
        }
    };
#pragma unroll
    for (int d = 0; d < GV_D; ++d) load(ring[d]);
    // The rest of the warp's rows is asked into the L2 at the same time.
    if (lane == 0 && r1 > r0) {
        const size_t ahead = (size_t)GV_D * ((CHUNK < K ? CHUNK : K)), total = (size_t)(r1 - r0) * K;
        if (OUT != OUT_HEAD && total > ahead) l2_prefetch(W + (size_t)r0 * K + ahead, (uint32_t)((total - ahead) * sizeof(T)));
    }
    if (OUT != OUT_HEAD) pdl_trigger();
    pdl_wait_cta();
    // The LM head lets the next step begin only now: every kernel of this step has completed, so that the step after
    // may read cache rows and states ahead of its own waits.
    if (OUT == OUT_HEAD) pdl_trigger();

    // ---- the vector
    if (VEC == VEC_NORM || VEC == VEC_CONCAT) {
        const int width = VEC == VEC_CONCAT ? K / 2 : K;
        const T* erow = nullptr;
        if (a.token) {
            int tok = *a.token;
            if (tok < 0 || tok >= a.vocab) {
                if (tid == 0) atomicOr(a.status, MQ_STATUS_BAD_TOKEN);
                tok = tok < 0 ? 0 : a.vocab - 1;
            }
            erow = reinterpret_cast<const T*>(a.embed) + (size_t)tok * width;
        }
        float ss = 0.f;
        for (int i = tid * 4; i < width; i += GV_THREADS * 4) {
            float4 v;
            if (erow) {
                v = load4(erow + i);
                v.x *= a.embed_scale; v.y *= a.embed_scale; v.z *= a.embed_scale; v.w *= a.embed_scale;
                if (blockIdx.x == 0) {
                    if (a.x_store) store4(a.x_store + i, v);
                    if (a.x0_store) store4(a.x0_store + i, v);
                }
            } else {
                v = load4_cg(a.x + i);
            }
            if (VEC == VEC_CONCAT) {
                put_vec<T>(vec, i, v);
                put_vec<T>(vec, width + i, erow ? v : load4_cg(a.x0 + i));
            } else {
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                store4(vec + vec_pos<T>(i), v);
            }
        }
        if (VEC == VEC_NORM) {
            const float inv = 1.0f / sqrtf(cta_sum<GV_WARPS>(ss, red) / (float)a.norm_n + a.eps);
            for (int i = tid * 4; i < width; i += GV_THREADS * 4) {
                const float4 v = load4(vec + vec_pos<T>(i)), g = load4(a.gain + i);
                put_vec<T>(vec, i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
            }
        }
    } else {
        const int hv = VEC == VEC_GATED ? a.hv : 0;
        const T* cat = reinterpret_cast<const T*>(a.cat);
        float ss = 0.f;
        for (int i = tid * 4; i < K; i += GV_THREADS * 4) {
            if (i < hv) {
                const float4 v = load4_cg(a.o + i);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                store4(vec + vec_pos<T>(i), v);
            } else {
                store4(vec + vec_pos<T>(i), load4_cg(cat + i));
            }
        }
        if (VEC == VEC_GATED) {
            const float inv = 1.0f / sqrtf(cta_sum<GV_WARPS>(ss, red) / (float)a.norm_n + a.eps);
            for (int i = tid * 4; i < hv; i += GV_THREADS * 4) {
                const float4 v = load4(vec + vec_pos<T>(i)), w = load4(a.gain + i), g = load4_cg(reinterpret_cast<const T*>(a.g) + i);
                put_vec<T>(vec, i, make_float4(v.x * inv * w.x * Elem<T>::sigmoid(g.x), v.y * inv * w.y * Elem<T>::sigmoid(g.y),
                                               v.z * inv * w.z * Elem<T>::sigmoid(g.z), v.w * inv * w.w * Elem<T>::sigmoid(g.w)));
            }
        }
    }
    for (int i = K + tid * 4; i < nch * CHUNK; i += GV_THREADS * 4) store4(vec + vec_pos<T>(i), make_float4(0.f, 0.f, 0.f, 0.f));
    __syncthreads();

    // ---- the rows
    unsigned long long best = 0ull;
    auto flush = [&](int first, int cnt) {       // rows first .. first + cnt - 1 of this warp are in done[warp]
        __syncwarp();
        if (OUT == OUT_SEGMENTS) {
            for (int p = lane; 2 * p < cnt; p += 32) {
                const int r = first + 2 * p;     // rows of a pair are of one segment
                const Segment& s = a.seg.s[a.seg.find(r)];
                const int c = r - s.row0;
                if (c >= s.rows) continue;
                float y0 = done[warp][2 * p], y1 = done[warp][2 * p + 1];
                if (s.act == ACT_SWIGLU) {
                    reinterpret_cast<T*>(s.out)[c / 2] = Elem<T>::put(silu<T>(y0) * y1);
                } else {
                    if (s.act == ACT_SILU) { y0 = silu<T>(y0); y1 = silu<T>(y1); }
                    if (s.f32) {
                        reinterpret_cast<float*>(s.out)[c] = y0;
                        reinterpret_cast<float*>(s.out)[c + 1] = y1;
                    } else {
                        reinterpret_cast<T*>(s.out)[c] = Elem<T>::put(y0);
                        reinterpret_cast<T*>(s.out)[c + 1] = Elem<T>::put(y1);
                    }
                }
            }
        } else {
            for (int p = lane; p < cnt; p += 32) {
                const int r = first + p;
                const float v = done[warp][p];
                if (OUT == OUT_ADD) a.y[r] = fmaf(a.mult, v, __ldcg(a.y + r));
                else if (OUT == OUT_STORE) a.y[r] = v;
                else {
                    if (a.logits) a.logits[r] = v;
                    const unsigned long long k = best_key(v, r);
                    best = k > best ? k : best;
                }
            }
        }
        __syncwarp();
    };
    int crow = r0, cch = 0, first = r0;
    float acc = 0.f;
    while (crow < r1) {
#pragma unroll
        for (int d = 0; d < GV_D; ++d) {
            if (crow < r1) {
                const float* v = vec + cch * CHUNK;
#pragma unroll
                for (int s = 0; s < GV_CS; ++s) acc += dot16(ring[d][s], v + s * SEG, lane, (const T*)nullptr);
                load(ring[d]);
                if (++cch == nch) {
                    acc = warp_sum(acc);
                    if (lane == 0) done[warp][crow - first] = acc;
                    acc = 0.f;
                    cch = 0;
                    ++crow;
                    if (crow - first == GV_BATCH) { flush(first, GV_BATCH); first = crow; }
                }
            }
        }
    }
    if (crow > first) flush(first, crow - first);

    if (OUT == OUT_HEAD) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const unsigned long long other = __shfl_xor_sync(0xffffffffu, best, o);
            best = other > best ? other : best;
        }
        if (lane == 0) wbest[warp] = best;
        __syncthreads();
        if (tid == 0) {
            for (int i = 1; i < GV_WARPS; ++i) best = wbest[i] > best ? wbest[i] : best;
            atomicMax(a.slot, best);
            __threadfence();
            if (atomicAdd(a.ticket, 1u) == gridDim.x - 1) {
                __threadfence();
                const unsigned long long k = atomicExch(a.slot, 0ull);
                *a.out_token = (int)(0xffffffffu - (uint32_t)(k & 0xffffffffull));
                *a.ticket = 0u;
            }
        }
    }
}

template <typename T, int VEC, int OUT>
static int go(Stream& st, const GemvArgs& a) {
    constexpr int CHUNK = GV_CS * 32 * Elem<T>::PER16;
    const size_t smem = (size_t)((a.K + CHUNK - 1) / CHUNK) * CHUNK * sizeof(float);
    const int rc = allow_smem(k_gemv<T, VEC, OUT>, smem);
    if (rc) return rc;
    // The LM head is long enough to fill the device by itself: two CTAs per SM keep more loads in flight.  The products of
    // a layer take one, so that the next kernel's CTA fits beside it.
    return launch(st, k_gemv<T, VEC, OUT>, dim3(OUT == OUT_HEAD ? 2 * sm_count() : sm_count()), dim3(GV_THREADS), smem, a);
}
template <typename T>
int gemv(Stream& st, int vec, int out, const GemvArgs& a) {
    if (vec == VEC_NORM && out == OUT_SEGMENTS) return go<T, VEC_NORM, OUT_SEGMENTS>(st, a);
    if (vec == VEC_NORM && out == OUT_HEAD) return go<T, VEC_NORM, OUT_HEAD>(st, a);
    if (vec == VEC_CONCAT && out == OUT_STORE) return go<T, VEC_CONCAT, OUT_STORE>(st, a);
    if (vec == VEC_GATED && out == OUT_ADD) return go<T, VEC_GATED, OUT_ADD>(st, a);
    if (vec == VEC_PLAIN && out == OUT_ADD) return go<T, VEC_PLAIN, OUT_ADD>(st, a);
    return MQ_ERR_BAD_ARG;
}
template int gemv<bf16>(Stream&, int, int, const GemvArgs&);
template int gemv<float>(Stream&, int, int, const GemvArgs&);

}  // namespace hy
}  // namespace mq
