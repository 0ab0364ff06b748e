// Matrix products of the layer-listed decoder for more than one token: bf16 on the tcgen05
// tile GEMM (tc_gemm.cuh), 32-bit on plain FMA tiles (no reduced-precision tensor mode).
#include "hy_common.cuh"
#include "tc_gemm.cuh"

namespace mq {
namespace hy {

int sm_count() {
    static int n[64] = {0};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) return 148;
    if (!n[dev]) cudaDeviceGetAttribute(&n[dev], cudaDevAttrMultiProcessorCount, dev);
    return n[dev];
}

// ---------------------------------------------------------------- 32-bit
// 64 x 64 tiles, K in steps of 16, 256 threads with a 4 x 4 piece each.  The finished tile goes through shared memory
// so that the sink sees 32 columns of a row, as from the tensor-core kernel.
constexpr int FT = 64, FK = 16;
template <bool PLANES>
__global__ void __launch_bounds__(256) k_gemm_f32(const float* __restrict__ A, int lda, const float* __restrict__ W, int M, int N, int K,
                                                  SegmentSink<float> sink, float* __restrict__ plane, int ldp) {
    pdl_trigger();
    pdl_wait();
    __shared__ float sa[FK][FT + 4], sb[FK][FT + 4];
    __shared__ float sc[FT][FT + 4];
    const int tid = threadIdx.x, m0 = blockIdx.y * FT, n0 = blockIdx.x * FT;
    const int tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
    const int lr = tid >> 2, lk = (tid & 3) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += FK) {        // K is a multiple of 16
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
        if (m0 + lr < M) a = load4(A + (size_t)(m0 + lr) * lda + k0 + lk);
        if (n0 + lr < N) b = load4(W + (size_t)(n0 + lr) * K + k0 + lk);
        sa[lk][lr] = a.x; sa[lk + 1][lr] = a.y; sa[lk + 2][lr] = a.z; sa[lk + 3][lr] = a.w;
        sb[lk][lr] = b.x; sb[lk + 1][lr] = b.y; sb[lk + 2][lr] = b.z; sb[lk + 3][lr] = b.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < FK; ++k) {
            const float4 av = *reinterpret_cast<const float4*>(&sa[k][tr]), bv = *reinterpret_cast<const float4*>(&sb[k][tc]);
            const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], br[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(&sc[tr + i][tc]) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    __syncthreads();
    if (tid < 2 * FT) {
        const int r = tid >> 1, c = (tid & 1) * 32;
        if (m0 + r >= M || n0 + c >= N) return;
        uint32_t v[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(sc[r][c + j]);
        if (PLANES) {                            // the plane is at least as wide as the tiles
#pragma unroll
            for (int q = 0; q < 8; ++q)
                store4(plane + (size_t)(m0 + r) * ldp + n0 + c + 4 * q,
                       make_float4(__uint_as_float(v[4 * q]), __uint_as_float(v[4 * q + 1]), __uint_as_float(v[4 * q + 2]), __uint_as_float(v[4 * q + 3])));
        } else {
            sink(m0 + r, n0 + c, v);
        }
    }
}

// ---------------------------------------------------------------- tile shape
// Estimated cycles of one CTA round: a k-block costs the larger of its tensor time (256 cycles per 128 x 128) and its
// operand traffic (64 bytes per clock into an SM); a tile costs its start-up and epilogue on top.
struct TileShape { int bn, mt; };
static long long tile_cost(TileShape s, int M, int N, int kblocks, int split, int sms) {
    const long long tiles = (long long)((N + s.bn - 1) / s.bn) * ((M + 128 * s.mt - 1) / (128 * s.mt)) * split;
    const long long mma = 2LL * s.bn * s.mt, load = (16384LL * s.mt + 128LL * s.bn) / 64;
    const long long per_tile = ((kblocks + split - 1) / split) * (mma > load ? mma : load) + 3000 + 6LL * s.bn * s.mt;
    return ((tiles + sms - 1) / sms) * per_tile;
}
static TileShape pick_tile(int M, int N, int kblocks, int max_split, int* split) {
    static const TileShape shapes[] = {{256, 2}, {128, 2}, {256, 1}, {128, 1}, {64, 1}};
    TileShape best = shapes[3];
    long long cost = -1;
    for (const TileShape& s : shapes)
        for (int z = 1; z <= max_split && z * 4 <= kblocks + 3; z *= 2) {
            // every plane is written and read back once: 8 bytes per element over the memory of the whole device
            const long long c = tile_cost(s, M, N, kblocks, z, sm_count()) + (long long)(z - 1) * ((long long)M * N / 500 + 1500);
            if (cost < 0 || c < cost) { cost = c; best = s; *split = z; }
        }
    return best;
}

template <>
int linear_segments<float>(Stream& st, const float* A, int lda, const float* W, int M, int N, int K, const Segments& g, unsigned int*) {
    return launch(st, k_gemm_f32<false>, dim3((N + FT - 1) / FT, (M + FT - 1) / FT), dim3(256), 0, A, lda, W, M, N, K, SegmentSink<float>{g},
                  (float*)nullptr, 0);
}
template <>
int linear_planes<float>(Stream& st, const float* A, int lda, const float* W, float* planes, int M, int N, int K, int ldp, int* nplanes, unsigned int*) {
    *nplanes = 1;
    return launch(st, k_gemm_f32<true>, dim3((N + FT - 1) / FT, (M + FT - 1) / FT), dim3(256), 0, A, lda, W, M, N, K, SegmentSink<float>{}, planes, ldp);
}

template <>
int linear_segments<bf16>(Stream& st, const bf16* A, int lda, const bf16* W, int M, int N, int K, const Segments& g, unsigned int* status) {
    int z = 1;
    const TileShape s = pick_tile(M, N, (K + 63) / 64, 1, &z);
    const SegmentSink<bf16> sink{g};
    ++st.launches;
#define MQH_GO(BN, MT) \
    if (s.bn == BN && s.mt == MT) \
        return launch_gemm<BN, EPI_SINK, MT>(A, lda, W, nullptr, nullptr, nullptr, M, N, K, 0, status, st.s, nullptr, 0, 0, 1, -1, true, sink);
    MQH_GO(256, 2) MQH_GO(128, 2) MQH_GO(256, 1) MQH_GO(128, 1) MQH_GO(64, 1)
#undef MQH_GO
    return MQ_ERR_UNSUPPORTED;
}
template <>
int linear_planes<bf16>(Stream& st, const bf16* A, int lda, const bf16* W, float* planes, int M, int N, int K, int ldp, int* nplanes, unsigned int* status) {
    int z = 1;
    const TileShape s = pick_tile(M, N, (K + 63) / 64, *nplanes, &z);
    *nplanes = z;
    ++st.launches;
#define MQH_GO(BN, MT) \
    if (s.bn == BN && s.mt == MT) \
        return launch_gemm<BN, EPI_PARTIAL, MT>(A, lda, W, nullptr, (bf16*)planes, nullptr, M, N, K, ldp, status, st.s, nullptr, 0, 0, z);
    MQH_GO(256, 2) MQH_GO(128, 2) MQH_GO(256, 1) MQH_GO(128, 1) MQH_GO(64, 1)
#undef MQH_GO
    return MQ_ERR_UNSUPPORTED;
}

}  // namespace hy
}  // namespace mq
