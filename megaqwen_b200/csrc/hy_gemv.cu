// Products of one token: y = W v.  A token reads every weight once, so these kernels stream
// weight rows: every CTA owns a contiguous range of rows, i.e. one contiguous piece of the
// matrix.  The first loads (a ring of registers) are issued and the rest of the piece is
// asked into the L2 BEFORE the wait on the preceding kernel (weights are written by nothing on
// the stream), so the weights cross HBM while that kernel is still running.
//
// bf16 (k_gemv_mma): sixteen rows are the M of mma.sync.m16n8k16, the vector fills all eight
// columns of N, the eight warps split K and meet in shared memory.  A lane's 16-byte load is
// eight consecutive elements of one row; a dot product does not care in which order the k's
// come, so its four words serve as the A words of two products and the same 16 bytes of the
// vector as their B words: five instructions for 16 rows x 32 columns.  On FMA pipes the
// unpacking alone would bound the kernel.
// 32-bit (k_gemv_f32): a warp per row, FMAs.
//
// What the vector is made of (norm of the residual stream, the loop's input, the gated norm of a
// recurrence's output beside the feed-forward's activations, the residual stream after the normed
// result of the sublayer before) is computed by every CTA for itself;
// what becomes of the result (segments with activations, residual add, LM head with arg-max) is
// decided row by row at the end.
#include "hy_common.cuh"

namespace mq {
namespace hy {

constexpr int GV_WARPS = 8, GV_THREADS = GV_WARPS * 32;
static __host__ __device__ constexpr bool is_gated(int vec) { return vec == VEC_GATED || vec == VEC_GATED_PARTS; }

__device__ __forceinline__ uint4 ld_weight(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
// larger value first, then the lower index
__device__ __forceinline__ unsigned long long best_key(float v, int i) {
    uint32_t u = __float_as_uint(v);
    u = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
    return ((unsigned long long)u << 32) | (unsigned long long)(0xffffffffu - (uint32_t)i);
}

// ---------------------------------------------------------------- the vector
// vec[0, K) in T; raw: K floats of shared memory (may be vec itself for T = float).  A decode step is a chain of
// latencies, so everything that can be asked for at once is: norm weights before the wait (`Ahead`), the activations
// that are taken as they are by asynchronous copies, the others in batches of registers.
constexpr int GV_AHEAD = 2;       // norm weights of the first 2 x 1024 elements
struct Ahead { float4 gain[GV_AHEAD], post[GV_AHEAD]; };
template <int VEC>
__device__ __forceinline__ void fetch_gain(const GemvArgs& a, Ahead& h) {
    const float* w = is_gated(VEC) ? a.gn.w : a.gain;
    const int n = VEC == VEC_NORM || VEC == VEC_POST_NORM ? a.K : is_gated(VEC) ? a.gn.hv : 0;
    const int np = (VEC == VEC_POST || VEC == VEC_POST_NORM) && a.post_y ? a.K : 0;
#pragma unroll
    for (int x = 0; x < GV_AHEAD; ++x) {
        const int i = (threadIdx.x + x * GV_THREADS) * 4;
        h.gain[x] = i < n ? load4(w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        h.post[x] = i < np ? load4(a.post + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
}
__device__ __forceinline__ float sum_sq(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
template <typename T, int VEC>
__device__ __forceinline__ void make_vector(const GemvArgs& a, const Ahead& ahead, T* vec, float* raw, float* scratch, float* red) {
    const int tid = threadIdx.x, K = a.K;
    constexpr int STRIDE = GV_THREADS * 4;
    if (VEC == VEC_POST || VEC == VEC_POST_NORM) {
        const T* erow = nullptr;
        if (a.token) {
            int tok = *a.token;
            if (tok < 0 || tok >= a.vocab) {
                if (tid == 0) atomicOr(a.status, MQ_STATUS_BAD_TOKEN);
                tok = tok < 0 ? 0 : a.vocab - 1;
            }
            erow = reinterpret_cast<const T*>(a.embed) + (size_t)tok * K;
        }
        auto stream = [&](int i) {
            if (!erow) return load4_cg(a.x + i);
            const float4 v = load4(erow + i);
            return make_float4(v.x * a.embed_scale, v.y * a.embed_scale, v.z * a.embed_scale, v.w * a.embed_scale);
        };
        // the first quads stay in registers, further ones of the result wait in shared memory
        float4 xk[GV_AHEAD], yk[GV_AHEAD];
        float ss = 0.f, inv = 0.f;
#pragma unroll
        for (int x = 0; x < GV_AHEAD; ++x) {
            const int i = tid * 4 + x * STRIDE;
            xk[x] = yk[x] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < K) {
                xk[x] = stream(i);
                if (a.post_y) yk[x] = load4_cg(a.post_y + i);
            }
        }
        if (a.post_y) {
#pragma unroll
            for (int x = 0; x < GV_AHEAD; ++x) ss += sum_sq(yk[x]);
            for (int i = tid * 4 + GV_AHEAD * STRIDE; i < K; i += STRIDE) {
                const float4 y = load4_cg(a.post_y + i);
                ss += sum_sq(y);
                store4(raw + i, y);
            }
            inv = 1.0f / sqrtf(cta_sum<GV_WARPS>(ss, red) / (float)a.norm_n + a.eps);
        }
        ss = 0.f;
        auto put = [&](int i, float4 v, const float4& y, const float4& g) {
            if (a.post_y) {
                v.x = fmaf(y.x * inv, g.x, v.x); v.y = fmaf(y.y * inv, g.y, v.y);
                v.z = fmaf(y.z * inv, g.z, v.z); v.w = fmaf(y.w * inv, g.w, v.w);
            }
            if (blockIdx.x == 0 && a.x_store) store4(a.x_store + i, v);
            if (VEC == VEC_POST_NORM) { ss += sum_sq(v); store4(raw + i, v); }
            else store4(vec + i, v);
        };
#pragma unroll
        for (int x = 0; x < GV_AHEAD; ++x) {
            const int i = tid * 4 + x * STRIDE;
            if (i < K) put(i, xk[x], yk[x], ahead.post[x]);
        }
        for (int i = tid * 4 + GV_AHEAD * STRIDE; i < K; i += STRIDE) {
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            put(i, stream(i), a.post_y ? load4(raw + i) : zero, a.post_y ? load4(a.post + i) : zero);
        }
        if (VEC == VEC_POST_NORM) {
            inv = 1.0f / sqrtf(cta_sum<GV_WARPS>(ss, red) / (float)a.norm_n + a.eps);
            int n = 0;
            for (int i = tid * 4; i < K; i += STRIDE, ++n) {
                const float4 v = load4(raw + i), g = n == 0 ? ahead.gain[0] : n == 1 ? ahead.gain[1] : load4(a.gain + i);
                store4(vec + i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
            }
        }
    } else if (VEC == VEC_NORM || VEC == VEC_CONCAT) {
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
        for (int i0 = tid * 4; i0 < width; i0 += 2 * STRIDE) {
            float4 v[2], y[2];
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int i = i0 + x * STRIDE;
                if (i >= width) break;
                v[x] = erow ? load4(erow + i) : load4_cg(a.x + i);
                if (VEC == VEC_CONCAT && !erow) y[x] = load4_cg(a.x0 + i);
            }
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int i = i0 + x * STRIDE;
                if (i >= width) break;
                if (erow) {
                    v[x].x *= a.embed_scale; v[x].y *= a.embed_scale; v[x].z *= a.embed_scale; v[x].w *= a.embed_scale;
                    if (blockIdx.x == 0) {
                        if (a.x_store) store4(a.x_store + i, v[x]);
                        if (a.x0_store) store4(a.x0_store + i, v[x]);
                    }
                }
                if (VEC == VEC_CONCAT) {
                    store4(vec + i, v[x]);
                    store4(vec + width + i, erow ? v[x] : y[x]);
                } else {
                    ss += v[x].x * v[x].x + v[x].y * v[x].y + v[x].z * v[x].z + v[x].w * v[x].w;
                    store4(raw + i, v[x]);
                }
            }
        }
        if (VEC == VEC_NORM) {
            const float inv = 1.0f / sqrtf(cta_sum<GV_WARPS>(ss, red) / (float)a.norm_n + a.eps);
            int n = 0;
            for (int i = tid * 4; i < width; i += STRIDE, ++n) {
                const float4 v = load4(raw + i), g = n == 0 ? ahead.gain[0] : n == 1 ? ahead.gain[1] : load4(a.gain + i);
                store4(vec + i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
            }
        }
    } else {
        const int hv = is_gated(VEC) ? a.gn.hv : 0;
        const T* cat = reinterpret_cast<const T*>(a.cat);
        constexpr int E = Elem<T>::PER16;
        for (int i = hv + tid * E; i < K; i += GV_THREADS * E) cp_async16(vec + i, cat + i);
        cp_async_commit();
        if (is_gated(VEC)) gated_norm_row<T, GV_WARPS, VEC == VEC_GATED>(a.gn, ahead.gain, raw, scratch, red, vec);
        cp_async_wait_all();
    }
}

// ---------------------------------------------------------------- the result
// Rows first .. first + cnt - 1, value(i) the i-th of them; threads me, me + of, .. of the caller share them.
template <typename T, int OUT, typename Value>
__device__ __forceinline__ void put_rows(const GemvArgs& a, int first, int cnt, int me, int of, Value value, float y_ahead, unsigned long long& best) {
    if (OUT == OUT_SEGMENTS) {
        for (int p = me; 2 * p < cnt; p += of) {       // rows of a pair are of one segment
            const int r = first + 2 * p;
            const Segment& s = a.seg.s[a.seg.find(r)];
            const int c = r - s.row0;
            if (c >= s.rows) continue;
            float y0 = value(2 * p), y1 = value(2 * p + 1);
            if (s.bias) { y0 += s.bias[c]; y1 += s.bias[c + 1]; }
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
        for (int p = me; p < cnt; p += of) {
            const int r = first + p;
            const float v = value(p);
            if (OUT == OUT_ADD) a.y[r] = fmaf(a.mult, v, p == me ? y_ahead : __ldcg(a.y + r));
            else if (OUT == OUT_STORE) a.y[r] = v;
            else {
                if (a.logits) a.logits[r] = v;
                const unsigned long long k = best_key(v, r);
                best = k > best ? k : best;
            }
        }
    }
}
// the arg-max over all CTAs; the last one writes the token and leaves slot and ticket as it found them
__device__ __forceinline__ void finish_head(const GemvArgs& a, unsigned long long best, unsigned long long* wbest) {
    const int tid = threadIdx.x;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const unsigned long long other = __shfl_xor_sync(0xffffffffu, best, o);
        best = other > best ? other : best;
    }
    if ((tid & 31) == 0) wbest[tid >> 5] = best;
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
// rows of this CTA (pairs where an epilogue needs them)
template <int OUT>
__device__ __forceinline__ void my_rows(int rows, int& r0, int& r1) {
    const int unit = OUT == OUT_SEGMENTS ? 2 : 1;
    const long long n = (rows + unit - 1) / unit;
    r0 = unit * (int)(n * blockIdx.x / gridDim.x);
    r1 = min(unit * (int)(n * (blockIdx.x + 1) / gridDim.x), rows);
}

// ---------------------------------------------------------------- bf16
// TALL: tiles of sixteen rows; otherwise eight (a CTA that owns no more), with half of the A words zero.
constexpr int GM_SLOT = 8;        // 16-byte loads per lane of one ring slot: k-steps (of 32 columns) x row halves
constexpr int GM_RING = 2;
constexpr int GM_BATCH = 128;     // rows that meet in shared memory at a time
template <int VEC, int OUT, bool TALL>
__global__ void __launch_bounds__(GV_THREADS, 2) k_gemv_mma(GemvArgs a) {
    constexpr int TR = TALL ? 16 : 8, STEPS = TALL ? GM_SLOT / 2 : GM_SLOT, BT = GM_BATCH / TR;
    extern __shared__ __align__(16) uint8_t gm_raw[];
    __shared__ float part[GV_WARPS][GM_BATCH];
    __shared__ float red[GV_WARPS];
    __shared__ unsigned long long wbest[GV_WARPS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c8 = (lane & 3) * 8;
    const int K = a.K, nsteps = (K + 31) / 32;
    bf16* xs = reinterpret_cast<bf16*>(gm_raw);                   // [nsteps * 32]
    float* raw = reinterpret_cast<float*>(xs + nsteps * 32);      // [K] (norms), then what the gated norm needs
    const bf16* W = reinterpret_cast<const bf16*>(a.W);
    int r0, r1;
    my_rows<OUT>(a.rows, r0, r1);
    const int s0 = nsteps * warp / GV_WARPS, s1 = nsteps * (warp + 1) / GV_WARPS;
    const int ntiles = (r1 - r0 + TR - 1) / TR, slots = (s1 - s0 + STEPS - 1) / STEPS;     // per tile

    uint4 ring[GM_RING][GM_SLOT];
    int lt = 0, ls = s0;                                          // tile and first step of the next slot to load
    auto load = [&](uint4 (&b)[GM_SLOT]) {
        if (lt >= ntiles || slots == 0) return;
        const int r = r0 + lt * TR + g;
        const bf16* p = W + (size_t)r * K + ls * 32 + c8;
#pragma unroll
        for (int u = 0; u < STEPS; ++u) {
            const bool in = ls + u < s1 && (ls + u) * 32 + c8 < K;
            b[u] = in && r < r1 ? ld_weight(p + u * 32) : make_uint4(0u, 0u, 0u, 0u);
            if (TALL) b[STEPS + u] = in && r + 8 < r1 ? ld_weight(p + (size_t)8 * K + u * 32) : make_uint4(0u, 0u, 0u, 0u);
        }
        ls += STEPS;
        if (ls >= s1) { ls = s0; ++lt; }
    };
#pragma unroll
    for (int d = 0; d < GM_RING; ++d) load(ring[d]);
    Ahead ahead;
    fetch_gain<VEC>(a, ahead);
    if (OUT != OUT_HEAD) {
        // one warp's share of the CTA's rows each, so that the requests leave side by side
        const size_t bytes = (size_t)(r1 - r0) * K * 2, each = (bytes / GV_WARPS) & ~(size_t)15;
        if (lane == 0 && each > 0) l2_prefetch(reinterpret_cast<const uint8_t*>(W + (size_t)r0 * K) + warp * each, (uint32_t)each);
        pdl_trigger();
    }
    pdl_wait_cta();
    // The LM head lets the next step begin only now: every kernel of this step has completed, so that the step after
    // may read cache rows and states ahead of its own waits.
    if (OUT == OUT_HEAD) pdl_trigger();
    const float y_ahead = OUT == OUT_ADD && tid < r1 - r0 ? __ldcg(a.y + r0 + tid) : 0.f;
    make_vector<bf16, VEC>(a, ahead, xs, raw, raw + K, red);
    if (tid < nsteps * 32 - K) xs[K + tid] = __float2bfloat16_rn(0.f);
    __syncthreads();

    unsigned long long best = 0ull;
    const bf16* xl = xs + c8;
    for (int tb = 0; tb < ntiles; tb += BT) {
        const int te = min(tb + BT, ntiles);
        if (slots == 0) {
            for (int i = lane; i < (te - tb) * TR; i += 32) part[warp][i] = 0.f;
        } else {
            int t = tb, s = s0;
            float acc[2][4] = {};
            const int items = (te - tb) * slots;
            // the ring position carries over from batch to batch: a batch takes an even number of slots or is the last
            for (int i = 0; i < items; i += GM_RING) {
#pragma unroll
                for (int d = 0; d < GM_RING; ++d) {
                    if (i + d < items) {
                        uint4 (&b)[GM_SLOT] = ring[d];
#pragma unroll
                        for (int u = 0; u < STEPS; ++u) {
                            if (s + u < s1) {
                                const uint4 x = *reinterpret_cast<const uint4*>(xl + (s + u) * 32);
                                const uint32_t a0[4] = {b[u].x, TALL ? b[STEPS + u].x : 0u, b[u].y, TALL ? b[STEPS + u].y : 0u};
                                const uint32_t a1[4] = {b[u].z, TALL ? b[STEPS + u].z : 0u, b[u].w, TALL ? b[STEPS + u].w : 0u};
                                mma16816(acc[0], a0, x.x, x.y);
                                mma16816(acc[1], a1, x.z, x.w);
                            }
                        }
                        load(ring[d]);
                        s += STEPS;
                        if (s >= s1) {
                            if ((lane & 3) == 0) {
                                part[warp][(t - tb) * TR + g] = acc[0][0] + acc[1][0];
                                if (TALL) part[warp][(t - tb) * TR + g + 8] = acc[0][2] + acc[1][2];
                            }
#pragma unroll
                            for (int e = 0; e < 4; ++e) acc[0][e] = acc[1][e] = 0.f;
                            s = s0;
                            ++t;
                        }
                    }
                }
            }
        }
        __syncthreads();
        const int first = r0 + tb * TR, cnt = min(r1, r0 + te * TR) - first;
        put_rows<bf16, OUT>(a, first, cnt, tid, GV_THREADS, [&](int i) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < GV_WARPS; ++w) v += part[w][i];
            return v;
        }, tb == 0 || OUT != OUT_ADD ? y_ahead : (tid < cnt ? __ldcg(a.y + first + tid) : 0.f), best);
        __syncthreads();
    }
    if (OUT == OUT_HEAD) finish_head(a, best, wbest);
}

// ---------------------------------------------------------------- 32-bit
template <int VEC, int OUT>
__global__ void __launch_bounds__(GV_THREADS, 2) k_gemv_f32(GemvArgs a) {
    extern __shared__ __align__(16) float gf_vec[];
    __shared__ float done[GV_WARPS][2];
    __shared__ float red[GV_WARPS];
    __shared__ unsigned long long wbest[GV_WARPS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, K = a.K;
    const float* W = reinterpret_cast<const float*>(a.W);
    int r0, r1;
    my_rows<OUT>(a.rows, r0, r1);
    Ahead ahead;
    fetch_gain<VEC>(a, ahead);
    if (OUT != OUT_HEAD) pdl_trigger();
    pdl_wait_cta();
    if (OUT == OUT_HEAD) pdl_trigger();
    make_vector<float, VEC>(a, ahead, gf_vec, gf_vec, gf_vec + K, red);
    __syncthreads();
    unsigned long long best = 0ull;
    for (int first = r0 + warp * 2; first < r1; first += GV_WARPS * 2) {      // two rows (a pair) at a time
        const int cnt = min(2, r1 - first);
        for (int p = 0; p < cnt; ++p) {
            const float* w = W + (size_t)(first + p) * K;
            float s = 0.f;
            for (int k = lane * 4; k < K; k += 128) {
                const float4 u = load4(w + k), v = load4(gf_vec + k);
                s = fmaf(u.x, v.x, fmaf(u.y, v.y, fmaf(u.z, v.z, fmaf(u.w, v.w, s))));
            }
            s = warp_sum(s);
            if (lane == 0) done[warp][p] = s;
        }
        __syncwarp();
        put_rows<float, OUT>(a, first, cnt, lane, 32, [&](int i) { return done[warp][i]; }, OUT == OUT_ADD && lane < cnt ? __ldcg(a.y + first + lane) : 0.f,
                             best);
        __syncwarp();
    }
    if (OUT == OUT_HEAD) finish_head(a, best, wbest);
}

// ---------------------------------------------------------------- launches
template <int VEC>
static size_t vec_scratch(const GemvArgs& a) { return is_gated(VEC) ? (size_t)gated_scratch(a.gn) * 4 : 0; }
template <int VEC, int OUT, bool TALL>
static int go_mma(Stream& st, const GemvArgs& a) {
    const size_t smem = (size_t)((a.K + 31) / 32) * 64 + (VEC == VEC_CONCAT || VEC == VEC_PLAIN ? 0 : (size_t)a.K * 4) + vec_scratch<VEC>(a);
    const int rc = allow_smem(k_gemv_mma<VEC, OUT, TALL>, smem);
    if (rc) return rc;
    // The LM head is long enough to fill the device by itself: two CTAs per SM keep more loads in flight.  The products of
    // a layer take one, so that the next kernel's CTA fits beside it.
    return launch(st, k_gemv_mma<VEC, OUT, TALL>, dim3(OUT == OUT_HEAD ? 2 * sm_count() : sm_count()), dim3(GV_THREADS), smem, a);
}
template <int VEC, int OUT>
static int go(Stream& st, const GemvArgs& a, const bf16*) {
    if (OUT != OUT_HEAD && a.rows <= 8 * sm_count()) return go_mma<VEC, OUT, false>(st, a);
    return go_mma<VEC, OUT, true>(st, a);
}
template <int VEC, int OUT>
static int go(Stream& st, const GemvArgs& a, const float*) {
    const size_t smem = (size_t)a.K * 4 + vec_scratch<VEC>(a);
    const int rc = allow_smem(k_gemv_f32<VEC, OUT>, smem);
    if (rc) return rc;
    return launch(st, k_gemv_f32<VEC, OUT>, dim3(sm_count()), dim3(GV_THREADS), smem, a);
}
template <typename T>
int gemv(Stream& st, int vec, int out, const GemvArgs& a) {
    const T* t = nullptr;
    if (vec == VEC_NORM && out == OUT_SEGMENTS) return go<VEC_NORM, OUT_SEGMENTS>(st, a, t);
    if (vec == VEC_NORM && out == OUT_HEAD) return go<VEC_NORM, OUT_HEAD>(st, a, t);
    if (vec == VEC_CONCAT && out == OUT_STORE) return go<VEC_CONCAT, OUT_STORE>(st, a, t);
    if (vec == VEC_GATED && out == OUT_ADD) return go<VEC_GATED, OUT_ADD>(st, a, t);
    if (vec == VEC_PLAIN && out == OUT_ADD) return go<VEC_PLAIN, OUT_ADD>(st, a, t);
    if (vec == VEC_GATED && out == OUT_STORE) return go<VEC_GATED, OUT_STORE>(st, a, t);
    if (vec == VEC_GATED_PARTS && out == OUT_ADD) return go<VEC_GATED_PARTS, OUT_ADD>(st, a, t);
    if (vec == VEC_GATED_PARTS && out == OUT_STORE) return go<VEC_GATED_PARTS, OUT_STORE>(st, a, t);
    if (vec == VEC_PLAIN && out == OUT_STORE) return go<VEC_PLAIN, OUT_STORE>(st, a, t);
    if (vec == VEC_POST && out == OUT_SEGMENTS) return go<VEC_POST, OUT_SEGMENTS>(st, a, t);
    if (vec == VEC_POST_NORM && out == OUT_HEAD) return go<VEC_POST_NORM, OUT_HEAD>(st, a, t);
    return MQ_ERR_BAD_ARG;
}
template int gemv<bf16>(Stream&, int, int, const GemvArgs&);
template int gemv<float>(Stream&, int, int, const GemvArgs&);

}  // namespace hy
}  // namespace mq
