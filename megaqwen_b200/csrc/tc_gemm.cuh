// Tile GEMM on tcgen05: C[M, N] = A[M, K] B[N, K]^T with the epilogues of the prefill chains.
#pragma once

#include "tc_core.cuh"

namespace mq {

// ---------------------------------------------------------------- GEMM  C[M,N] = A[M,K] * B[N,K]^T
constexpr int GM_BM = 128;
constexpr int GM_BK = 64;
constexpr int GM_THREADS = 192;    // skinny GEMM: warp 0 TMA, warp 1 MMA + TMEM owner, warps 2..5 epilogue
// Tile GEMM: eight epilogue warps.  Warps w and w + 4 read the same quarter of the TMEM lanes (a warp may
// only touch lanes 32 (w % 4) .. + 31) and split the accumulator columns; with four warps the SwiGLU
// epilogue of a 256 x 256 tile (65 536 silu + products on 128 threads) took as long as its main loop.
constexpr int GM_EPI_WARPS = 8;
constexpr int GM_TILE_THREADS = 64 + 32 * GM_EPI_WARPS;
enum { EPI_STORE = 0, EPI_RESID = 1, EPI_SWIGLU = 2, EPI_PARTIAL = 3, EPI_STORE_2CTA = 4, EPI_SINK = 5 };   // PARTIAL: fp32 plane blockIdx.z of a K split
// EPI_STORE_2CTA: EPI_STORE with a three-stage ring (97 KB), so that two CTAs share an SM.  For a GEMM of many short
// CTAs that stream weights (the batched LM head: 1187 column tiles of a 64-row matrix), where a lone CTA's start-up and
// epilogue leave the SM's memory pipeline idle.

#ifndef MQ_GEMM_BUDGET_KB
#define MQ_GEMM_BUDGET_KB 200   // shared memory for the operand ring of one CTA
#define MQ_GEMM_MIN_CTAS 1
#endif
// MT = 128-row A tiles per CTA.  With MT = 2 a CTA computes a 256-row output tile with two
// accumulators that share every B tile: the 128 x 128 tiles are bound by the operand traffic
// from the L2 into the SMs, and a 256-row tile moves a third less of it per FLOP.
template <int BN, int EPI, int MT = 1>
struct GemmCfg {
    static constexpr int NB = (EPI == EPI_SWIGLU) ? 2 : 1;                       // B operands per stage
    static constexpr int A_BYTES = MT * GM_BM * GM_BK * 2;
    static constexpr int STAGE_BYTES = A_BYTES + NB * BN * GM_BK * 2;
    static constexpr int STAGES = EPI == EPI_STORE_2CTA ? 3 : (MQ_GEMM_BUDGET_KB * 1024) / STAGE_BYTES > 6 ? 6 : (MQ_GEMM_BUDGET_KB * 1024) / STAGE_BYTES;
    static constexpr int ACC_COLS = MT * NB * BN;                                // accumulator columns in use
    static constexpr int TMEM_COLS = ACC_COLS <= 32 ? 32 : ACC_COLS <= 64 ? 64 : ACC_COLS <= 128 ? 128 : ACC_COLS <= 256 ? 256 : 512;   // allocations are powers of two
    static_assert(ACC_COLS <= 512 && BN % 32 == 0, "tensor memory holds 512 columns; the epilogue reads 32 at a time");
    static constexpr size_t SMEM = (size_t)STAGES * STAGE_BYTES + 1024 /*align*/ + 256 /*barriers*/;
};

// x / (1 + e^-x) with the hardware exponential and reciprocal (2 ulp of fp32; the result is rounded to bf16)
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.0f + __expf(-x)); }

// EPI_SINK hands every 32 accumulators of a row to sink(row, column, accumulators), a functor of the caller that is
// passed to the kernel by value.  The other epilogues take none.
struct NoSink {
    __device__ __forceinline__ void operator()(int, int, const uint32_t (&)[32]) const {}
};

template <int BN, int EPI, int MT, class Sink = NoSink>
__global__ void __launch_bounds__(GM_TILE_THREADS, MQ_GEMM_MIN_CTAS)
k_gemm(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const __grid_constant__ CUtensorMap tmB2,
       const __grid_constant__ CUtensorMap tmB3, int tiles0, int tiles1,
       bf16* __restrict__ C, const bf16* R, int M, int N, int K, int ldc, unsigned int* status, int drop_kb, int early_b, Sink sink) {
    // drop_kb >= 0 (test hook): the producer never requests k-block drop_kb, so the MMA thread's wait for it
    // runs out; -1 in every production launch.  early_b: B is constant over the stream's lifetime (a weight),
    // so its first tiles may be requested before the preceding grid has finished.
    pdl_trigger();   // the next grid may be scheduled already; it waits for this one below, after its own set-up
    // EPI_STORE / EPI_RESID may concatenate up to three B matrices along N (q|k|v): column tile
    // blockIdx.x < tiles0 reads tmB, < tiles0 + tiles1 tmB2, else tmB3.  EPI_SWIGLU uses tmB (gate)
    // and tmB2 (up) for the same tile.
    using Cfg = GemmCfg<BN, EPI, MT>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + (size_t)Cfg::STAGES * Cfg::STAGE_BYTES);
    uint64_t* empty = full + Cfg::STAGES;
    uint64_t* accum = empty + Cfg::STAGES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(accum + 1);
    // Set by the thread whose bounded wait expired (the sticky status bit is then set as well).  Everybody
    // stops issuing work; the epilogue stores nothing; the CTA drains what is in flight before it exits.
    volatile uint32_t* aborted = tmem_slot + 1;

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int m0 = blockIdx.y * GM_BM * MT, n0 = blockIdx.x * BN;
    const int kblocks = (K + GM_BK - 1) / GM_BK;   // the columns of a last, partial block beyond K arrive as zeros
    // EPI_PARTIAL: gridDim.z CTAs share an output tile, each takes a contiguous range of k-blocks
    const int kb_first = (int)(((long long)blockIdx.z * kblocks) / gridDim.z);
    const int nk = (int)(((long long)(blockIdx.z + 1) * kblocks) / gridDim.z) - kb_first;
    const int tile = blockIdx.x;
    const CUtensorMap* mapB = &tmB;
    int brow0 = n0;
    if (EPI != EPI_SWIGLU && tile >= tiles0) {
        mapB = tile < tiles0 + tiles1 ? &tmB2 : &tmB3;
        brow0 = (tile < tiles0 + tiles1 ? tile - tiles0 : tile - tiles0 - tiles1) * BN;
    }

    if (tid == 0) {
        for (int s = 0; s < Cfg::STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        mbar_init(accum, 1);
        mbar_fence_init();
    }
    if (tid == 64) *aborted = 0u;       // by a thread that is idle now (thread 0's set-up gates the first TMA request)
    if (warp == 1) tmem_alloc(tmem_slot, Cfg::TMEM_COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(tmem_slot);
    // Barriers and tensor memory are set up while the preceding grid may still be running.  Where the B operand is
    // a weight matrix that nothing on the stream writes, its tiles for the first ring of stages are requested now
    // and cross HBM while that grid finishes; the A tiles (its output) follow the wait, from which on its results
    // are complete and visible.
    const int npre = !early_b ? 0 : nk < Cfg::STAGES ? nk : Cfg::STAGES;
    if (tid == 0) {
        for (int kb = 0; kb < npre; ++kb) {
            if (kb == drop_kb) continue;
            uint8_t* st = smem + (size_t)kb * Cfg::STAGE_BYTES;
            mbar_expect_tx(&full[kb], (uint32_t)Cfg::STAGE_BYTES);
            tma_load_2d(st + Cfg::A_BYTES, mapB, (kb_first + kb) * GM_BK, brow0, &full[kb]);
            if (EPI == EPI_SWIGLU) tma_load_2d(st + Cfg::A_BYTES + BN * GM_BK * 2, &tmB2, (kb_first + kb) * GM_BK, n0, &full[kb]);
        }
    }
    pdl_wait();

    int issued = npre;                    // k-blocks the producer has requested, B tiles at least (thread 0 only)
    if (warp == 0) {
        if (lane == 0) {
            for (int kb = 0; kb < nk; ++kb) {
                const int s = kb % Cfg::STAGES;
                if (kb >= Cfg::STAGES && !mbar_wait(&empty[s], (uint32_t)((kb / Cfg::STAGES) - 1) & 1u, status)) { *aborted = 1u; break; }
                if (*aborted) break;
                issued = kb + 1;
                if (kb == drop_kb) continue;
                uint8_t* st = smem + (size_t)s * Cfg::STAGE_BYTES;
                if (kb >= npre) mbar_expect_tx(&full[s], (uint32_t)Cfg::STAGE_BYTES);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) tma_load_2d(st + mt * GM_BM * GM_BK * 2, &tmA, (kb_first + kb) * GM_BK, m0 + mt * GM_BM, &full[s]);
                if (kb >= npre) {
                    tma_load_2d(st + Cfg::A_BYTES, mapB, (kb_first + kb) * GM_BK, brow0, &full[s]);
                    if (EPI == EPI_SWIGLU) tma_load_2d(st + Cfg::A_BYTES + BN * GM_BK * 2, &tmB2, (kb_first + kb) * GM_BK, n0, &full[s]);
                }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            // instruction descriptor: D = f32, A = B = bf16, both K-major, N >> 3, M >> 4.  EPI_SWIGLU: the gate
            // and the up tile sit back to back in the stage (2 BN rows of one K-major operand), so ONE
            // instruction of N = 2 BN fills both accumulators (columns [0, BN) gate, [BN, 2 BN) up).  A
            // 128 x 128 x 16 instruction reads 8 KB of shared memory for 64 cycles of math, which is the
            // SM's whole shared-memory bandwidth; at N = 256 it is 12 KB for 128 cycles.
            constexpr int UMMA_N = Cfg::NB * BN;
            static_assert(UMMA_N <= 256, "one instruction spans at most 256 columns");
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(UMMA_N >> 3) << 17) | ((uint32_t)(GM_BM >> 4) << 24);
            for (int kb = 0; kb < nk; ++kb) {
                const int s = kb % Cfg::STAGES;
                if (!mbar_wait(&full[s], (uint32_t)(kb / Cfg::STAGES) & 1u, status)) { *aborted = 1u; break; }
                tc_fence_after();
                uint8_t* st = smem + (size_t)s * Cfg::STAGE_BYTES;
                const uint64_t db = smem_desc_sw128(st + Cfg::A_BYTES);
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {   // accumulator (mt, nb) lives at TMEM column (mt * NB + nb) * BN
                    const uint64_t da = smem_desc_sw128(st + mt * GM_BM * GM_BK * 2);
#pragma unroll
                    for (int k = 0; k < GM_BK / 16; ++k) {
                        const uint32_t acc = (kb > 0 || k > 0) ? 1u : 0u;
                        umma_bf16(tmem_base + mt * Cfg::NB * BN, da + 2 * k, db + 2 * k, idesc, acc);   // +32 bytes per K=16 step
                    }
                }
                umma_commit(&empty[s]);     // frees this stage once the MMAs above have read it
            }
            umma_commit(accum);             // accumulator complete (or, after an expired wait, the MMAs issued so far)
            if (*aborted) mbar_wait_drain(accum, 0);   // tensor memory is freed below: nothing may still be writing it
        }
        __syncwarp();
    } else {
        // epilogue: warp (2..9) owns TMEM lanes 32*(warp%4) .. +31 = tile rows and half of the columns
        const bool acc_ok = mbar_wait(accum, 0, status) && !*aborted;   // after an expired wait nothing is read or stored
        tc_fence_after();
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        // the two warps of a quarter take one 128-row accumulator each (MT = 2) or half of the columns (MT = 1)
        static_assert(GM_EPI_WARPS == 8 && (MT == 2 || (BN / 2) % 32 == 0), "epilogue split");
        const int cbeg = MT == 2 ? 0 : half * (BN / 2), cend = MT == 2 ? BN : cbeg + BN / 2;
#pragma unroll 1
        for (int mt = (MT == 2 ? half : 0); mt < (MT == 2 ? half + 1 : 1); ++mt) {
        if (!acc_ok) break;
        const int row = m0 + mt * GM_BM + quarter * 32 + lane;
        const uint32_t trow = tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(mt * Cfg::NB * BN);
#pragma unroll 1
        for (int c0 = cbeg; c0 < cend; c0 += 32) {
            uint32_t v[32];
            tmem_ld32(trow + c0, v);
            if (EPI == EPI_PARTIAL) {   // raw fp32 accumulators into plane blockIdx.z of C (a float [gridDim.z][M][ldc] array)
                if (row < M) {
                    float4* fp = reinterpret_cast<float4*>(reinterpret_cast<float*>(C) + ((size_t)blockIdx.z * M + row) * ldc + n0 + c0);
#pragma unroll
                    for (int q = 0; q < 8; ++q)
                        fp[q] = make_float4(__uint_as_float(v[4 * q]), __uint_as_float(v[4 * q + 1]), __uint_as_float(v[4 * q + 2]), __uint_as_float(v[4 * q + 3]));
                }
                continue;
            }
            if constexpr (EPI == EPI_SINK) {
                if (row < M) sink(row, n0 + c0, v);
                continue;
            }
            uint32_t out[16];
            if (EPI == EPI_SWIGLU) {
                uint32_t u[32];
                tmem_ld32(trow + BN + c0, u);
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    const float g0 = rbf(__uint_as_float(v[2 * j])), g1 = rbf(__uint_as_float(v[2 * j + 1]));
                    const float u0 = rbf(__uint_as_float(u[2 * j])), u1 = rbf(__uint_as_float(u[2 * j + 1]));
                    out[j] = pack_bf16x2(rbf(silu_fast(g0)) * u0, rbf(silu_fast(g1)) * u1);
                }
            } else if (EPI == EPI_RESID) {
                if (row < M) {
                    const uint4* rp = reinterpret_cast<const uint4*>(R + (size_t)row * ldc + n0 + c0);
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        const uint4 rr = rp[q];
                        const uint32_t rw[4] = {rr.x, rr.y, rr.z, rr.w};
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const int j = q * 4 + e;
                            out[j] = pack_bf16x2(bf_lo(rw[e]) + rbf(__uint_as_float(v[2 * j])), bf_hi(rw[e]) + rbf(__uint_as_float(v[2 * j + 1])));
                        }
                    }
                }
            } else {
#pragma unroll
                for (int j = 0; j < 16; ++j) out[j] = pack_bf16x2(__uint_as_float(v[2 * j]), __uint_as_float(v[2 * j + 1]));
            }
            if (row < M) {
                uint4* cp = reinterpret_cast<uint4*>(C + (size_t)row * ldc + n0 + c0);
#pragma unroll
                for (int q = 0; q < 4; ++q) cp[q] = make_uint4(out[4 * q], out[4 * q + 1], out[4 * q + 2], out[4 * q + 3]);
            }
        }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (*aborted) {
        // After an expired wait (anybody's: the flag is read behind the barrier): copies that were requested still
        // land in this CTA's shared memory, so the producer waits for the last one of every stage before the CTA exits.
        if (tid == 0)
            for (int s = 0; s < Cfg::STAGES && s < issued; ++s) {
                const int last = ((issued - 1 - s) / Cfg::STAGES) * Cfg::STAGES + s;      // last requested k-block of stage s
                if (last != drop_kb) mbar_wait_drain(&full[s], (uint32_t)(last / Cfg::STAGES) & 1u);
            }
        __syncthreads();
    }
    if (warp == 1) tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
}

template <int BN, int EPI, int MT = 1, class Sink = NoSink>
static int launch_gemm(const bf16* A, int lda, const bf16* B, const bf16* B2, bf16* C, const bf16* R, int M, int N, int K, int ldc,
                       unsigned int* status, cudaStream_t stream, const bf16* B3 = nullptr, int rows0 = 0, int rows1 = 0, int ksplit = 1,
                       int drop_kb = -1, bool early_b = true, Sink sink = Sink()) {
    // early_b: B (B2, B3) are weights, never written by work on this stream; false for caller-supplied operands
    // rows0 > 0: B, B2, B3 hold rows0, rows1 and N - rows0 - rows1 output columns (concatenated along N)
    using Cfg = GemmCfg<BN, EPI, MT>;
    static bool attr_set[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !attr_set[dev]) {
        cudaError_t e = cudaFuncSetAttribute(k_gemm<BN, EPI, MT, Sink>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM);
        if (e != cudaSuccess) return (int)e;
        attr_set[dev] = true;
    }
    // Whole tiles, except where the epilogue copes with a last, partial one: a sink looks at the column itself, and a
    // plane may be wider than N (the weight rows beyond N arrive as zeros, and so are its columns).
    const int tiles_n = (N + BN - 1) / BN, kblocks = (K + GM_BK - 1) / GM_BK;
    if (EPI != EPI_SINK && N % BN != 0 && !(EPI == EPI_PARTIAL && ldc >= tiles_n * BN)) return MQ_ERR_BAD_ARG;
    if (K % 8 != 0 || (EPI != EPI_SINK && EPI != EPI_PARTIAL && K % GM_BK != 0)) return MQ_ERR_BAD_ARG;
    CUtensorMap ma, mb, mb2;
    int rc = get_map(A, (uint64_t)M, (uint64_t)K, (uint64_t)lda, GM_BM, &ma);
    if (rc != MQ_OK) return rc;
    const bool concat = rows0 > 0;
    if (concat && (rows0 % BN || rows1 % BN || EPI == EPI_SWIGLU)) return MQ_ERR_BAD_ARG;
    rc = get_map(B, (uint64_t)(concat ? rows0 : N), (uint64_t)K, (uint64_t)K, BN, &mb);
    if (rc != MQ_OK) return rc;
    mb2 = mb;
    CUtensorMap mb3 = mb;
    if (EPI == EPI_SWIGLU) {
        rc = get_map(B2, (uint64_t)N, (uint64_t)K, (uint64_t)K, BN, &mb2);
        if (rc != MQ_OK) return rc;
    } else if (concat) {
        rc = get_map(B2, (uint64_t)rows1, (uint64_t)K, (uint64_t)K, BN, &mb2);
        if (rc != MQ_OK) return rc;
        rc = get_map(B3, (uint64_t)(N - rows0 - rows1), (uint64_t)K, (uint64_t)K, BN, &mb3);
        if (rc != MQ_OK) return rc;
    }
    if (ksplit < 1 || (ksplit > 1 && EPI != EPI_PARTIAL) || kblocks < ksplit) return MQ_ERR_BAD_ARG;
    dim3 grid(tiles_n, (M + GM_BM * MT - 1) / (GM_BM * MT), ksplit);
    launch_pdl(k_gemm<BN, EPI, MT, Sink>, dim3(grid), dim3(GM_TILE_THREADS), Cfg::SMEM, stream, ma, mb, mb2, mb3, concat ? rows0 / BN : (1 << 30), concat ? rows1 / BN : 0,
                                                             C, R, M, N, K, ldc, status, drop_kb, early_b ? 1 : 0, sink);
    return (int)cudaGetLastError();
}

}  // namespace mq
