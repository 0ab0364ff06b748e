// Shared by the kernels of the layer-listed decoder: element types, the segmented
// epilogue of its fused input projections, and the functions that launch each step.
// All sizes are run-time values, padded to multiples of 16 (include/megaqwen_hybrid.h).
#pragma once

#include "../../include/megaqwen_hybrid.h"
#include "mq_device.cuh"

namespace mq {
namespace hy {

// ---------------------------------------------------------------- element types
template <typename T> struct Elem;
template <> struct Elem<bf16> {
    static constexpr int PER16 = 8;      // elements in 16 bytes
    __device__ static __forceinline__ float get(bf16 v) { return __bfloat162float(v); }
    __device__ static __forceinline__ bf16 put(float v) { return __float2bfloat16_rn(v); }
    __device__ static __forceinline__ float round(float v) { return rbf(v); }
    __device__ static __forceinline__ float sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
};
template <> struct Elem<float> {
    static constexpr int PER16 = 4;
    __device__ static __forceinline__ float get(float v) { return v; }
    __device__ static __forceinline__ float put(float v) { return v; }
    __device__ static __forceinline__ float round(float v) { return v; }
    __device__ static __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
};
template <typename T> __device__ __forceinline__ float silu(float z) { return z * Elem<T>::sigmoid(z); }
// 32-bit in both modes: what enters a recurrence
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
constexpr float LOG2E = 1.4426950408889634f;
// four consecutive elements
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf_lo(u.x), bf_hi(u.x), bf_lo(u.y), bf_hi(u.y));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w)); }
// the same through the L2 (activations of the kernel before, see mq_device.cuh)
__device__ __forceinline__ float4 load4_cg(const float* p) { return __ldcg(reinterpret_cast<const float4*>(p)); }
__device__ __forceinline__ float4 load4_cg(const bf16* p) {
    const uint2 u = ld_cg_u2(p);
    return make_float4(bf_lo(u.x), bf_hi(u.x), bf_lo(u.y), bf_hi(u.y));
}

// Sum over a CTA of NW warps, the same value in every thread.  red: NW floats of shared memory.
template <int NW>
__device__ __forceinline__ float cta_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < NW; ++i) t += red[i];
    __syncthreads();
    return t;
}

// ---------------------------------------------------------------- segmented epilogue
// The rows of a fused projection belong to segments that go to different buffers through different activations.
enum { ACT_NONE = 0, ACT_SILU = 1, ACT_SWIGLU = 2 };   // SWIGLU: rows 2i, 2i + 1 are gate i, up i -> silu(gate) * up at column i
struct Segment {
    void* out;       // T, or fp32 if f32
    int row0, rows;  // rows without padding; the next segment starts at a multiple of MQH_SEGMENT
    int ld;
    short act, f32;
    const float* bias;   // per row, or null; not with SWIGLU
};
constexpr int MAX_SEGMENTS = 6;
struct Segments {
    Segment s[MAX_SEGMENTS];
    int n;
    __device__ __forceinline__ int find(int r) const {
        int i = 0;
        while (i + 1 < n && r >= s[i + 1].row0) ++i;
        return i;
    }
};
// Output columns n0 .. n0 + 31 (n0 a multiple of 32) of activation row `row`; v: fp32 bits.
template <typename T>
struct SegmentSink {
    Segments g;
    __device__ __forceinline__ void operator()(int row, int n0, const uint32_t (&v)[32]) const {
        const Segment& s = g.s[g.find(n0)];
        const int c = n0 - s.row0;
        if (c >= s.rows) return;
        const int nq = s.rows - c >= 32 ? 8 : (s.rows - c) / 4;   // rows is a multiple of 16
        if (s.act == ACT_SWIGLU) {
            T* o = reinterpret_cast<T*>(s.out) + (size_t)row * s.ld + c / 2;
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                if (2 * q >= nq) break;
                float4 r;
                r.x = silu<T>(__uint_as_float(v[8 * q])) * __uint_as_float(v[8 * q + 1]);
                r.y = silu<T>(__uint_as_float(v[8 * q + 2])) * __uint_as_float(v[8 * q + 3]);
                r.z = silu<T>(__uint_as_float(v[8 * q + 4])) * __uint_as_float(v[8 * q + 5]);
                r.w = silu<T>(__uint_as_float(v[8 * q + 6])) * __uint_as_float(v[8 * q + 7]);
                store4(o + 4 * q, r);
            }
            return;
        }
        float4 bias[8];                      // asked for side by side
#pragma unroll
        for (int q = 0; q < 8; ++q) bias[q] = s.bias && q < nq ? load4(s.bias + c + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int q = 0; q < 8; ++q) {
            if (q >= nq) break;
            float4 r = make_float4(__uint_as_float(v[4 * q]) + bias[q].x, __uint_as_float(v[4 * q + 1]) + bias[q].y,
                                   __uint_as_float(v[4 * q + 2]) + bias[q].z, __uint_as_float(v[4 * q + 3]) + bias[q].w);
            if (s.act == ACT_SILU) r = make_float4(silu<T>(r.x), silu<T>(r.y), silu<T>(r.z), silu<T>(r.w));
            if (s.f32) store4(reinterpret_cast<float*>(s.out) + (size_t)row * s.ld + c + 4 * q, r);
            else store4(reinterpret_cast<T*>(s.out) + (size_t)row * s.ld + c + 4 * q, r);
        }
    }
};

// ---------------------------------------------------------------- norm and gate of a mixer's output
// The concatenated heads are normed in `parts` equal parts (counted without the heads' padding) and gated by act(g):
// rms_part(o) * w * act(g), or, gate_first, rms_part(o * act(g)) * w.
enum { GATE_SIGMOID = 0, GATE_SILU = 1 };
struct GatedNorm {
    const float* o;          // [hv]
    const float* w;          // [hv]
    const void* g;           // T [hv]
    int hv, vp, vd;          // heads * vp; padded and true size of a head
    int parts, part_n;       // part_n elements each
    short act, gate_first;
    float eps;
};
// squares are kept per unit of four elements where no part ends inside one, else per element
__host__ __device__ __forceinline__ int gated_unit(const GatedNorm& a) { return (a.vd | a.part_n) % 4 == 0 ? 4 : 1; }
// quads of a part where parts are neighbouring lanes of a warp (no padding, a power of two up to 32 quads), else 0
__host__ __device__ __forceinline__ int gated_lanes(const GatedNorm& a) {
    const int n = a.part_n / 4;
    return a.vd == a.vp && a.part_n % 4 == 0 && n <= 32 && (n & (n - 1)) == 0 ? n : 0;
}
// floats of shared memory beside the hv of the values; none for one part, or parts inside a warp
__host__ __device__ __forceinline__ int gated_scratch(const GatedNorm& a) {
    return a.parts == 1 || gated_lanes(a) ? 0 : a.hv / gated_unit(a) + a.parts + 64;
}
template <typename T>
__device__ __forceinline__ float gate_act(int act, float z) { return act == GATE_SILU ? silu<T>(z) : Elem<T>::sigmoid(z); }
// One row by a CTA of NW warps.  raw: hv floats, scratch: gated_scratch floats, red: NW floats (all shared); out: T [hv] (may be
// raw itself for T = float).  w0: the weights of the thread's first two quads, loaded ahead (NW * 128 elements apart).
// ONE: a single part.
template <typename T, int NW, bool ONE>
__device__ __forceinline__ void gated_norm_row(const GatedNorm& a, const float4 (&w0)[2], float* raw, float* scratch, float* red, T* out) {
    constexpr int STRIDE = NW * 128;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const T* gate = reinterpret_cast<const T*>(a.g);
    const int unit = ONE ? 4 : gated_unit(a), lanes = ONE ? 0 : gated_lanes(a);
    float ss = 0.f;
    int n = 0;
    // whole warps go round: lanes beyond the end take part in the exchanges with zeros
    for (int i0 = tid * 4; (i0 & ~127) < a.hv; i0 += 2 * STRIDE, n += 2) {
        float4 v[2], g[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int i = i0 + x * STRIDE;
            v[x] = g[x] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i >= a.hv) continue;
            v[x] = load4_cg(a.o + i);
            g[x] = load4_cg(gate + i);
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int i = i0 + x * STRIDE;
            if ((i & ~127) >= a.hv) break;
            const bool in = i < a.hv;
            const float4 w = !in ? make_float4(0.f, 0.f, 0.f, 0.f) : n == 0 ? w0[x] : load4(a.w + i);
            const float4 s = make_float4(gate_act<T>(a.act, g[x].x), gate_act<T>(a.act, g[x].y), gate_act<T>(a.act, g[x].z), gate_act<T>(a.act, g[x].w));
            const float4 u = make_float4(v[x].x * s.x, v[x].y * s.y, v[x].z * s.z, v[x].w * s.w);
            const float4 m = a.gate_first ? u : v[x];
            const float4 q = make_float4(m.x * m.x, m.y * m.y, m.z * m.z, m.w * m.w);
            if (!ONE && lanes) {
                float t = q.x + q.y + q.z + q.w;
                for (int o = lanes >> 1; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
                const float inv = 1.0f / sqrtf(t / (float)a.part_n + a.eps);
                if (in) store4(out + i, make_float4(u.x * w.x * inv, u.y * w.y * inv, u.z * w.z * inv, u.w * w.w * inv));
                continue;
            }
            if (!in) continue;
            if (ONE) ss += q.x + q.y + q.z + q.w;
            else if (unit == 4) scratch[i >> 2] = q.x + q.y + q.z + q.w;
            else store4(scratch + i, q);
            store4(raw + i, make_float4(u.x * w.x, u.y * w.y, u.z * w.z, u.w * w.w));
        }
    }
    if (!ONE && lanes) return;
    if (ONE) {
        const float inv = 1.0f / sqrtf(cta_sum<NW>(ss, red) / (float)a.part_n + a.eps);
        for (int i = tid * 4; i < a.hv; i += STRIDE) {
            const float4 v = load4(raw + i);
            store4(out + i, make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv));
        }
        return;
    }
    // one warp per part, or `ways` warps per part where there are fewer parts than warps
    const int ways = a.parts >= NW ? 1 : NW / a.parts, units = a.part_n / unit, vu = a.vd / unit, pu = a.vp / unit;
    float* sums = scratch + a.hv / unit;                    // [parts * ways], then the factors in its place
    __syncthreads();
    for (int task = warp; task < a.parts * ways; task += NW) {
        const int part = task / ways, way = task % ways;
        float s = 0.f;
        for (int x = way * 32 + lane; x < units; x += ways * 32) {
            const int u = part * units + x;
            s += scratch[vu == pu ? u : (u / vu) * pu + u % vu];
        }
        s = warp_sum(s);
        if (lane == 0) sums[task] = s;
    }
    __syncthreads();
    for (int i = tid * 4; i < a.hv; i += STRIDE) {
        float4 v = load4(raw + i);
        float* e = &v.x;
        int last = -1;
        float inv = 0.f;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            if (x > 0 && unit == 4) { e[x] *= inv; continue; }
            const int y = i + x;
            int part = (a.vd == a.vp ? y : (y / a.vp) * a.vd + y % a.vp) / a.part_n;      // padding: any part, its weight is zero
            part = min(part, a.parts - 1);
            if (part != last) {
                float s = 0.f;
                for (int k = 0; k < ways; ++k) s += sums[part * ways + k];
                inv = 1.0f / sqrtf(s / (float)a.part_n + a.eps);
                last = part;
            }
            e[x] *= inv;
        }
        store4(out + i, v);
    }
}

// ---------------------------------------------------------------- steps (each launches its kernels on `stream`)
struct Stream {
    cudaStream_t s;
    bool pdl;                // programmatic stream serialisation
    int launches;
};
template <typename... KArgs, typename... Args>
static int launch_cluster(Stream& st, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, int cluster_x, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st.s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = st.pdl ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster_x;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = cluster_x > 1 ? 2 : 1;
    ++st.launches;
    return (int)cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}
template <typename... KArgs, typename... Args>
static int launch(Stream& st, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    return launch_cluster(st, kernel, grid, block, smem, 1, args...);
}
// Raises the dynamic shared memory limit of a kernel once per device.  Without it dynamic and static shared memory share
// 48 KB; no kernel here has more than 8 KB of the latter.
template <typename K>
static int allow_smem(K kernel, size_t bytes) {
    struct Seen { K kernel; size_t bytes; };
    static Seen seen[64][16] = {};       // kernels of one type share the table; one that finds no place is set every time
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) return MQ_ERR_UNSUPPORTED;
    if (bytes <= 40 * 1024) return MQ_OK;
    if (bytes > 232448) return MQ_ERR_UNSUPPORTED;
    Seen* e = nullptr;
    for (Seen& x : seen[dev]) {
        if (x.kernel != nullptr && x.kernel != kernel) continue;
        e = &x;
        break;
    }
    if (e && e->kernel == kernel && e->bytes >= bytes) return MQ_OK;
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (err != cudaSuccess) return (int)err;
    if (e) *e = {kernel, bytes};
    return MQ_OK;
}
int sm_count();

// hy_linear.cu: C[M, N] = A[M, K] W[N, K]^T
template <typename T>
int linear_segments(Stream& st, const T* A, int lda, const T* W, int M, int N, int K, const Segments& g, unsigned int* status);
// fp32 planes [n][M][ldp] whose sum is the product; *nplanes: at most that many on entry, the number used on return.  ldp: at least
// N rounded up to 256.
template <typename T>
int linear_planes(Stream& st, const T* A, int lda, const T* W, float* planes, int M, int N, int K, int ldp, int* nplanes, unsigned int* status);

// hy_rows.cu: row-wise kernels
struct RowsArgs {
    // value of the row: embed[ids[r]] * embed_scale (ids), or base[r] (base, may be null) + mult * sum of the planes
    const int* ids; const void* embed; float embed_scale; int vocab;
    // (with post: base[r] + rms(sum of the planes) * post)
    const float* base; const float* planes; int nplanes, ldp; size_t plane_stride; float mult; const float* post;
    const int* gather;              // row r reads base row gather[r]
    int gather_max;
    float* x; float* x0;            // where the value is stored (either may be null)
    // what the next product reads: h = rms(value) * gain (gain null: the value itself), or xin = [value; x0_in]
    const float* gain; float eps; int norm_n; void* h;
    const float* x0_in; void* xin;  // x0_in null: the value itself (the first pass)
    int width;
    unsigned int* status;
};
template <typename T> int rows(Stream& st, int n, const RowsArgs& a);
// cat[r, 0 .. hv) = the gated norm of row r of o, w, g (row length hv)
template <typename T>
int gated_norm(Stream& st, int n, const GatedNorm& a, T* cat, int ldc);

// hy_recurrence.cu: state S <- decay S + k v^T, output S^T q * scale (+ skip * v)
enum { DECAY_CONST = 0, DECAY_HEAD = 1, DECAY_CHANNEL = 2 };
struct RecurrenceArgs {
    int mode;
    const void *q, *k, *v;          // T rows of length ldq, ldk, ldv
    int ldq, ldk, ldv;
    int n, heads, dim, vdim, kv_heads;      // head h reads q, k of head h / (heads / kv_heads)
    float scale;
    float* state;                   // [heads, dim, vdim]
    float* o;                       // [n, heads*vdim]
    void* scratch;                  // recurrence_scratch_bytes (chunked only)
    const float* decay_in; int ld_decay;    // fp32 [n, ld_decay]
    // DECAY_CONST: [heads, MQH_CHUNK + 1]
    const float* decay_pow;
    // DECAY_HEAD: dt = softplus(decay_in[head] + dt_bias), log decay a_neg * dt, k weighted by dt
    const float *dt_bias, *a_neg, *skip;
    // DECAY_CHANNEL: decay = sigmoid(gate_w decay_in + gate_b)^inv_tau
    const void* gate_w; const float* gate_b; int rank; float inv_tau;
    // one token of a model whose q, k, v come from a convolution (DECAY_HEAD): position, its inputs and state instead of q, k, v
    const int* position; int max_seq;
    const void* conv_in; void* conv_state; const float *conv_w, *conv_b; int taps, channels;
    unsigned int* status;
};
size_t recurrence_scratch_bytes(int n, int heads, int dim, int vdim);
bool recurrence_chunked_fits(int mode, int dim);
template <typename T> int recurrence_tokens(Stream& st, const RecurrenceArgs& a);
int recurrence_chunked(Stream& st, const RecurrenceArgs& a);
template <typename T>
int conv_rows(Stream& st, const T* x, const float* w, const float* b, T* state, T* y, int n, int pos0, int channels, int taps);
constexpr int CONV_MAX_TAPS = 64;

// hy_latent.cu
struct LatentRowsArgs {             // after the input projection of n rows at positions pos0 ..
    const float* down;              // [n, rank + rot]
    const float* norm; int norm_n; float eps;
    const float* rope;
    void* cache;                    // T [max_seq, rank + rot]
    void* q_rot;                    // T [n, heads*rot], rotated in place
    int n, pos0, heads, rank, rot, max_seq;
};
template <typename T> int latent_rows(Stream& st, const LatentRowsArgs& a);
struct CausalArgs {
    const void *q, *q_rot, *k, *k_rot, *v;
    const float* sink;
    void* out;
    int ld_rot, ld_out;
    int n, pos0, heads, dim, rot, vdim;
    float scale;
    unsigned int* status;
    int kv_heads, ldk, ldv;         // query head h reads head h / (heads / kv_heads) of k, v (rows of length ldk, ldv)
    int chunk;                      // 0, or: position i sees keys from i / chunk * chunk on
    const float* gate; int ld_gate; // per row and head: the output is multiplied by sigmoid(gate); null for none
};
bool causal_tc_fits(int dim, int rot, int vdim, float scale);
int causal_tc(Stream& st, const CausalArgs& a);
template <typename T> int causal_simt(Stream& st, const CausalArgs& a);
struct LatentDecodeArgs {           // one token at *position
    const void *q, *q_rot;          // T [heads*dim], [heads*rot] (not rotated)
    const float* down;              // [rank + rot]
    const float* norm; int norm_n; float eps;
    const float* rope;
    const int* position;
    void* cache;
    const void *w_uk_t, *w_uv;      // T [heads*rank, dim], [heads*vdim, rank]
    const float* sink;
    void* qcat;                     // T [heads rounded up to 16, rank + rot], zeroed once
    float* parts;                   // latent_parts_floats
    void* out;                      // T [heads*vdim]
    int heads, dim, rot, vdim, rank, max_seq;
    float scale;
    unsigned int* status;
};
int latent_splits(int max_seq);
size_t latent_parts_floats(int heads, int rank, int max_seq);
template <typename T> int latent_decode(Stream& st, const LatentDecodeArgs& a);

// hy_attention.cu: grouped-query attention with normed, half-rotated keys
struct HeadNorm {                   // norm of a head, then the rotation of its first 2 * half elements
    const float* w; int dim_n, dim, half;   // weights [dim]; elements without and with padding
    float eps;
    const float* rope;              // [max_seq, half, 2]
};
struct AttnRowsArgs {               // after the input projection of n rows at positions pos0 ..: q in place, k and v into the caches
    void* q; const void* k;         // T [n, heads*dim], [n, kv_heads*dim]
    void *k_cache, *v_cache;        // T [max_seq, kv_heads*dim]
    HeadNorm qn, kn;
    int n, pos0, heads, kv_heads;
};
template <typename T> int attn_rows(Stream& st, const AttnRowsArgs& a);
struct AttnDecodeArgs {             // one token at *position
    const void *q, *k;              // T, neither normed nor rotated
    const float* gate;              // [heads] or null
    void *k_cache, *v_cache;
    HeadNorm qn, kn;
    const int* position;
    void* out;                      // T [heads*dim]
    int heads, kv_heads, max_seq, chunk;
    float scale;
    unsigned int* status;
};
template <typename T> int attn_decode(Stream& st, const AttnDecodeArgs& a);

// hy_gemv.cu: y = W v for one token, with what the vector is made of and where y goes
enum { VEC_NORM = 0, VEC_CONCAT = 1, VEC_GATED = 2, VEC_PLAIN = 3, VEC_POST = 4, VEC_POST_NORM = 5, VEC_GATED_PARTS = 6 };
enum { OUT_SEGMENTS = 0, OUT_ADD = 1, OUT_STORE = 2, OUT_HEAD = 3 };
struct GemvArgs {                   // what every product reads first: its other lines of the parameter bank are fetched behind the wait
    const void* W; int rows, K;
    float* y; float mult;           // OUT_ADD: y += mult * (W v); OUT_STORE: y = W v
    float eps; int norm_n;
    const void* cat;                // VEC_PLAIN: the vector; VEC_GATED: its elements from gn.hv on
    const float* x; const float* gain;      // VEC_NORM: rms(x) * gain
    Segments seg;                   // OUT_SEGMENTS (one row)
    const float* x0;                // VEC_CONCAT: [x; x0], K = 2 width
    // VEC_POST: x + rms(post_y) * post (post_y null: x); VEC_POST_NORM: the rms norm of that, times gain.  CTA 0 stores the sum
    // to x_store, which must not be x.
    const float* post_y; const float* post;
    // token != null: x (and x0) is row *token of embed times embed_scale; CTA 0 stores it to x_store / x0_store
    const int* token; const void* embed; float embed_scale; int vocab; float* x_store; float* x0_store;
    GatedNorm gn;                   // VEC_GATED (a norm of one part), VEC_GATED_PARTS: the first gn.hv elements
    float* logits; unsigned long long* slot; unsigned int* ticket; int* out_token;   // OUT_HEAD
    unsigned int* status;
};
template <typename T> int gemv(Stream& st, int vec, int out, const GemvArgs& a);

}  // namespace hy
}  // namespace mq
