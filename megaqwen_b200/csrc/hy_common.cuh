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
    int ld, act, f32;
};
constexpr int MAX_SEGMENTS = 5;
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
#pragma unroll
        for (int q = 0; q < 8; ++q) {
            if (q >= nq) break;
            float4 r = make_float4(__uint_as_float(v[4 * q]), __uint_as_float(v[4 * q + 1]), __uint_as_float(v[4 * q + 2]), __uint_as_float(v[4 * q + 3]));
            if (s.act == ACT_SILU) r = make_float4(silu<T>(r.x), silu<T>(r.y), silu<T>(r.z), silu<T>(r.w));
            if (s.f32) store4(reinterpret_cast<float*>(s.out) + (size_t)row * s.ld + c + 4 * q, r);
            else store4(reinterpret_cast<T*>(s.out) + (size_t)row * s.ld + c + 4 * q, r);
        }
    }
};

// ---------------------------------------------------------------- steps (each launches its kernels on `stream`)
struct Stream {
    cudaStream_t s;
    bool pdl;                // programmatic stream serialisation
    int launches;
};
template <typename... KArgs, typename... Args>
static int launch(Stream& st, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st.s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = st.pdl ? 1 : 0;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    ++st.launches;
    return (int)cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}
// Raises the dynamic shared memory limit of a kernel once per device.  Without it dynamic and static shared memory share
// 48 KB; no kernel here has more than 8 KB of the latter.
template <typename K>
static int allow_smem(K kernel, size_t bytes) {
    static size_t done[64] = {0};        // one array per kernel type; kernels of one type share the larger limit
    static K last[64] = {nullptr};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) return MQ_ERR_UNSUPPORTED;
    if (bytes <= 40 * 1024 || (last[dev] == kernel && done[dev] >= bytes)) return MQ_OK;
    if (bytes > 232448) return MQ_ERR_UNSUPPORTED;
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
    last[dev] = kernel;
    done[dev] = bytes;
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
    const float* base; const float* planes; int nplanes, ldp; size_t plane_stride; float mult;
    const int* gather;              // row r reads base row gather[r]
    int gather_max;
    float* x; float* x0;            // where the value is stored (either may be null)
    // what the next product reads: h = rms(value) * gain, or xin = [value; x0_in]
    const float* gain; float eps; int norm_n; void* h;
    const float* x0_in; void* xin;  // x0_in null: the value itself (the first pass)
    int width;
    unsigned int* status;
};
template <typename T> int rows(Stream& st, int n, const RowsArgs& a);
// cat[r, 0 .. hv) = rms(o[r]) * w * sigmoid(g[r])
template <typename T>
int gated_norm(Stream& st, int n, const float* o, const float* w, const T* g, T* cat, int ldc, int hv, int norm_n, float eps);

// hy_lightning.cu
struct LightningArgs {
    const void *q, *k, *v;          // T [n, heads*dim], [n, heads*dim], [n, heads*vdim]
    const float* decay_pow;         // [heads, MQH_CHUNK + 1]
    float* state;                   // [heads, dim, vdim]
    float* o;                       // [n, heads*vdim]
    void* scratch;                  // lightning_scratch_bytes (chunked only)
    int n, heads, dim, vdim;
};
size_t lightning_scratch_bytes(int n, int heads, int dim, int vdim);
bool lightning_chunked_fits(int dim);
template <typename T> int lightning_tokens(Stream& st, const LightningArgs& a);
int lightning_chunked(Stream& st, const LightningArgs& a);

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

// hy_gemv.cu: y = W v for one token, with what the vector is made of and where y goes
enum { VEC_NORM = 0, VEC_CONCAT = 1, VEC_GATED = 2, VEC_PLAIN = 3 };
enum { OUT_SEGMENTS = 0, OUT_ADD = 1, OUT_STORE = 2, OUT_HEAD = 3 };
struct GemvArgs {
    const void* W; int rows, K;
    // VEC_NORM: rms(x) * gain; VEC_CONCAT: [x; x0], K = 2 width
    const float* x; const float* x0; const float* gain; float eps; int norm_n;
    // token != null: x (and x0) is row *token of embed times embed_scale; CTA 0 stores it to x_store / x0_store
    const int* token; const void* embed; float embed_scale; int vocab; float* x_store; float* x0_store;
    // VEC_GATED: the first hv elements are rms(o) * gain * sigmoid(g) (norm_n elements), the others those of cat; VEC_PLAIN: cat
    const float* o; const void* g; int hv; const void* cat;
    Segments seg;                   // OUT_SEGMENTS (one row)
    float* y; float mult;           // OUT_ADD: y += mult * (W v); OUT_STORE: y = W v
    float* logits; unsigned long long* slot; unsigned int* ticket; int* out_token;   // OUT_HEAD
    unsigned int* status;
};
template <typename T> int gemv(Stream& st, int vec, int out, const GemvArgs& a);

}  // namespace hy
}  // namespace mq
