// Causal attention on tcgen05 for a whole prompt or a portion of one.
#pragma once

#include "tc_gemm.cuh"

namespace mq {

// ---------------------------------------------------------------- causal attention on tcgen05 (one prompt)
// One CTA per (query head, 128-query tile); key tiles of 128 positions.  Both contractions run
// on the 5th-generation tensor cores with their accumulators in tensor memory:
//     S = Q K^T     A = Q tile [128 q x 128 d], B = K tile [128 keys x 128 d] straight from the KV cache
//     O_j = P V     A = P tile [128 q x 128 keys] (bf16) IN TENSOR MEMORY: the softmax warps write the probabilities
//                   over the scores they came from (tcgen05.st; 64 packed columns of S's 128), so the product
//                   reads only V from shared memory and nothing crosses the generic / async proxy boundary,
//                   B = V tile [128 keys x 128 d] straight from the KV cache, read as an MN-major operand
//                   (the cache rows are contiguous along d, the product contracts over the keys)
// (128-byte swizzle, fetched by TMA; the V map ends at the last key of the prompt, so the rows of the
// last tile beyond it arrive as zeros whatever the cache holds there).  Warp 0 feeds the K / V
// rings, warp 1 issues the MMAs, warps 2-9 hold HALF A QUERY ROW PER THREAD: they read the row's
// scores from tensor memory (tcgen05.ld), keep the running max / sum and write the probabilities
// rounded to bf16 as the next MMA's A operand; the output accumulates in tensor memory and is
// rescaled (tcgen05.ld / st) only when the maximum has grown by more than 2^8.  S is
// double-buffered: QK^T of tile j + 1 runs while tile j is in the softmax.  Replaces the reference's serial-per-warp kernel and its experimental tiles
// (csrc/megakernel/fused_prefill_kernels.inl:265-342, 347-445, 486-613).
constexpr int TA_BQ = 128, TA_BK = 128;
constexpr int TA_THREADS = 320;                             // warp 0 TMA, warp 1 MMA, warps 2-9 softmax
constexpr int TA_PANEL_BYTES = 128 * 128;                   // 128 rows of 64 columns
constexpr uint32_t TA_TMEM_COLS = 512;                      // S0 | S1 (128 columns each) | O (64 per value panel)

// Head shapes, in panels of 64 columns (narrower heads are filled up with zeros by TMA):
//   QP  query / key columns that each head has of its own
//   RP  query / key columns whose KEY is shared by all heads (the rotated part of latent attention), 0 for none
//   VP  value columns
template <int QP, int RP, int VP>
struct AttnTcCfg {
    static_assert(VP <= 4, "S0 | S1 | O fill the 512 columns of tensor memory");
    static constexpr int Q_BYTES = (QP + RP) * TA_PANEL_BYTES, V_BYTES = VP * TA_PANEL_BYTES;
    static constexpr size_t SMEM = (size_t)Q_BYTES + 2 * Q_BYTES + 2 * V_BYTES + 1024 /*align*/ + 256 /*barriers*/ + TA_BQ * 8 /*row exchange*/;
    static_assert(SMEM <= 232448, "shared memory of one CTA");
};
struct AttnTcArgs {
    bf16* out;               // [S, ld_out], head h at column h * head_cols
    int ld_out, head_cols;   // head_cols: value columns of a head, a multiple of 8
    int S, pos0;
    int kv_group, kv_plane0; // query head h reads plane kv_plane0 + h / kv_group of the K and V maps
    int ksteps, rsteps;      // 16-column steps of the two parts of the score (RP = 0: all of QP)
    float c;                 // score scale * log2(e), positive
    const float* sink;       // per head: the denominator also holds exp(sink); null for none
    unsigned int* status;
    int chunk = 0;           // > 0: position i sees keys from i / chunk * chunk on, else from 0
    const float* gate = nullptr;   // [S, ld_gate] per row and head: the output is multiplied by sigmoid(gate); null for none
    int ld_gate = 0;
};


// Maps: tmQ [head][token][d], tmK and tmV [plane][key][d] (the keys end at the last one of the prompt); with RP > 0
// tmQr [head][token][r] and tmKr [1][key][r].
template <int QP, int RP, int VP>
__global__ void __launch_bounds__(TA_THREADS, 1)
k_attention_tc(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
               const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmKr, AttnTcArgs a) {
    using Cfg = AttnTcCfg<QP, RP, VP>;
    constexpr int OC = VP * 32;                  // output columns of one softmax thread
    const int S = a.S, pos0 = a.pos0;
    unsigned int* status = a.status;
    pdl_trigger();
    pdl_wait();
    extern __shared__ uint8_t ta_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ta_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t* sQ = smem;
    uint8_t* sK = sQ + Cfg::Q_BYTES;             // [2]
    uint8_t* sV = sK + 2 * Cfg::Q_BYTES;         // [2]
    uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * Cfg::V_BYTES);
    uint64_t* q_full = bars;                     // 1
    uint64_t* k_full = bars + 1;                 // 2
    uint64_t* k_empty = bars + 3;                // 2
    uint64_t* v_full = bars + 5;                 // 2
    uint64_t* v_empty = bars + 7;                // 2
    uint64_t* s_full = bars + 9;                 // 2
    uint64_t* s_free = bars + 11;                // 2 (256 arrivals)
    uint64_t* p_full = bars + 13;                // 2 (256 arrivals)
    uint64_t* o_full = bars + 17;                // 1
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 18);
    float (*xm)[2] = reinterpret_cast<float(*)[2]>(bars + 20);   // [128][2]: the two half-row maxima (at the end: sums) of a query row

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head = blockIdx.x, plane = a.kv_plane0 + head / a.kv_group;
    const int q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * TA_BQ;        // longest query tiles first
    const int kv_end = min(pos0 + S, pos0 + q0 + TA_BQ);                  // keys any row of the tile may see
    const int kbase = a.chunk > 0 ? (pos0 + q0) / a.chunk * a.chunk : 0;  // first key of the tile's first row: key tiles start here
    const int nt = (kv_end - kbase + TA_BK - 1) / TA_BK;

    if (tid == 0) {
        mbar_init(q_full, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1);
            mbar_init(&s_full[i], 1); mbar_init(&s_free[i], 256); mbar_init(&p_full[i], 256);
        }
        mbar_init(o_full, 1);
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc(tmem_slot, TA_TMEM_COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(tmem_slot);
    const uint32_t tmem_o = tmem_base + 256;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(q_full, Cfg::Q_BYTES);
#pragma unroll
            for (int p = 0; p < QP; ++p) tma_load_3d(sQ + p * TA_PANEL_BYTES, &tmQ, p * 64, q0, head, q_full);
#pragma unroll
            for (int p = 0; p < RP; ++p) tma_load_3d(sQ + (QP + p) * TA_PANEL_BYTES, &tmQr, p * 64, q0, head, q_full);
            for (int j = 0; j < nt; ++j) {
                const int st = j & 1;
                if (j >= 2 && !mbar_wait(&k_empty[st], (uint32_t)((j >> 1) - 1) & 1u, status)) break;
                mbar_expect_tx(&k_full[st], Cfg::Q_BYTES);
#pragma unroll
                for (int p = 0; p < QP; ++p) tma_load_3d(sK + st * Cfg::Q_BYTES + p * TA_PANEL_BYTES, &tmK, p * 64, kbase + j * TA_BK, plane, &k_full[st]);
#pragma unroll
                for (int p = 0; p < RP; ++p) tma_load_3d(sK + st * Cfg::Q_BYTES + (QP + p) * TA_PANEL_BYTES, &tmKr, p * 64, kbase + j * TA_BK, 0, &k_full[st]);
                if (j >= 2 && !mbar_wait(&v_empty[st], (uint32_t)((j >> 1) - 1) & 1u, status)) break;
                mbar_expect_tx(&v_full[st], Cfg::V_BYTES);
#pragma unroll
                for (int p = 0; p < VP; ++p) tma_load_3d(sV + st * Cfg::V_BYTES + p * TA_PANEL_BYTES, &tmV, p * 64, kbase + j * TA_BK, plane, &v_full[st]);
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            // instruction descriptor: D = f32, A = B = bf16, both K-major, N = 128, M = 128
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
            // B (the V tile) is MN-major, N = the value panels
            const uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VP * 64 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
            bool ok = mbar_wait(q_full, 0, status);
            auto issue_s = [&](int j) {      // S[j & 1] = Q K_j^T
                const int st = j & 1;
                ok = ok && mbar_wait(&k_full[st], (uint32_t)(j >> 1) & 1u, status);
                if (j >= 2) ok = ok && mbar_wait(&s_free[st], (uint32_t)((j >> 1) - 1) & 1u, status);
                tc_fence_after();
                if (ok) {
                    auto step = [&](int panel, int kk, uint32_t acc) {
                        const uint64_t da = smem_desc_sw128(sQ + panel * TA_PANEL_BYTES) + 2 * kk;
                        const uint64_t db = smem_desc_sw128(sK + st * Cfg::Q_BYTES + panel * TA_PANEL_BYTES) + 2 * kk;
                        umma_bf16(tmem_base + st * 128, da, db, idesc, acc);
                    };
                    if constexpr (RP == 0) {
#pragma unroll
                        for (int kk = 0; kk < 4 * QP; ++kk) step(kk >> 2, kk & 3, kk > 0 ? 1u : 0u);
                    } else {
                        for (int kk = 0; kk < a.ksteps; ++kk) step(kk >> 2, kk & 3, kk > 0 ? 1u : 0u);
                        for (int kk = 0; kk < a.rsteps; ++kk) step(QP + (kk >> 2), kk & 3, 1u);
                    }
                }
                umma_commit(&k_empty[st]);
                umma_commit(&s_full[st]);
            };
            issue_s(0);
            for (int j = 0; j < nt; ++j) {
                const int st = j & 1;
                if (j + 1 < nt) issue_s(j + 1);
                ok = ok && mbar_wait(&p_full[st], (uint32_t)(j >> 1) & 1u, status);
                ok = ok && mbar_wait(&v_full[st], (uint32_t)(j >> 1) & 1u, status);
                tc_fence_after();
                if (ok) {
#pragma unroll
                    for (int kk = 0; kk < 8; ++kk) {
                        // A = the probabilities, written by the softmax threads over the scores they came from: 16 keys
                        // of a row are eight 32-bit columns.  B: 16 keys per step = two 1024-byte groups of the
                        // [keys][64 d] panels
                        const uint64_t db = smem_desc_mn_sw128(sV + st * Cfg::V_BYTES, TA_PANEL_BYTES) + (uint64_t)(kk * (2048 >> 4));
                        umma_bf16_ts(tmem_o, tmem_base + st * 128 + kk * 8, db, idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);   // O accumulates over all key tiles
                    }
                }
                umma_commit(&v_empty[st]);
                umma_commit(o_full);
            }
        }
        __syncwarp();
    } else {
        // softmax warps: TWO threads per query row r = TMEM lane r (warps w and w + 4 share a quarter of the
        // lanes); thread `half` owns keys [64 half, 64 half + 64) of every key tile and output columns
        // [OC half, +OC).  The two exchange their half-row maxima through shared memory (one 64-thread
        // named barrier per tile), so both scale by the same running maximum.  The output accumulates in
        // tensor memory over all key tiles; it is only rescaled when the running maximum has grown by
        // more than 2^8 since the value the accumulator is scaled to (then p <= 256 in between, exact in
        // fp32 and harmless in bf16), which after the first tiles practically never happens.  With one
        // thread per row the 128 exponentials per tile on four warps (one per scheduler) bounded the kernel.
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        const int r = quarter * 32 + lane;
        const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
        const uint32_t col_off = (uint32_t)(half * 64), out_off = (uint32_t)(half * OC);
        const int qpos = pos0 + q0 + r;                       // absolute position of this thread's query
        const int qfirst = a.chunk > 0 ? qpos / a.chunk * a.chunk : 0;
        const float c = a.c;
        float m = -INFINITY, l = 0.f;                         // m: the maximum the sums are scaled to (raw score units)
        bool ok = true;
        auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(1 + quarter) : "memory"); };
        for (int j = 0; j < nt; ++j) {
            const int st = j & 1;
            const uint32_t ts = tmem_base + st * 128 + lane_off + col_off;
            ok = ok && mbar_wait(&s_full[st], (uint32_t)(j >> 1) & 1u, status);
            tc_fence_after();
            const int k0 = kbase + j * TA_BK + half * 64;     // first key of this thread's half
            const bool diag = k0 + 63 > qpos || k0 < qfirst;  // some keys of this half lie beyond the query, or before its chunk
            uint32_t sv[64];
#pragma unroll
            for (int cb = 0; cb < 2; ++cb) tmem_ld32_nowait(ts + cb * 32, *reinterpret_cast<uint32_t(*)[32]>(&sv[cb * 32]));
            tmem_ld_wait();
            tc_fence_before();
            mbar_arrive(&s_free[st]);                         // the scores are in registers: S[st] may be overwritten
            float mh = -INFINITY;
            if (__any_sync(0xffffffffu, diag)) {              // without chunks only the last one or two key tiles of a query tile
#pragma unroll
                for (int i = 0; i < 64; ++i) {
                    if (k0 + i > qpos || k0 + i < qfirst) sv[i] = 0xff800000u;   // -inf
                    mh = fmaxf(mh, __uint_as_float(sv[i]));
                }
            } else {
                float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int i = 0; i < 64; ++i) m4[i & 3] = fmaxf(m4[i & 3], __uint_as_float(sv[i]));
                mh = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
            }
            xm[r][half] = mh;
            pair_sync();
            const float mx = fmaxf(xm[r][0], xm[r][1]);       // the same value in both threads of the row
            pair_sync();                                      // both have read it: the slot is free for the next tile
            // tcgen05.ld / st are warp-wide: the warp rescales together, rows that need none by 1
            const bool grow = (mx - m) * c > 8.0f;            // also true for the first tile (m = -inf)
            // o_full completes once per key tile and is waited on by parity, so every thread consumes EVERY
            // phase, in order (a parity wait that is two phases behind returns at once): phase j - 1 here if
            // the accumulator is rescaled, else just before this tile's probabilities are handed over.
            bool seen_prev = j == 0;
            if (__any_sync(0xffffffffu, grow)) {
                const float alpha = grow ? fast_exp2((m - mx) * c) : 1.0f;   // 0 for the first tile
                if (j > 0) {
                    // the previous P V product must have landed before the accumulator is touched
                    ok = ok && mbar_wait(o_full, (uint32_t)(j - 1) & 1u, status);
                    seen_prev = true;
                    tc_fence_after();
#pragma unroll
                    for (int cb = 0; cb < VP; ++cb) {
                        uint32_t v[32];
                        tmem_ld32(tmem_o + lane_off + out_off + cb * 32, v);
#pragma unroll
                        for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
                        tmem_st32(tmem_o + lane_off + out_off + cb * 32, v);
                    }
                    tc_fence_before();
                }
                l *= alpha;
                if (grow) m = mx;
            }
            // a row whose chunk begins in a later key tile has seen nothing yet: all its weights are 0
            const float mc = m == -INFINITY ? 0.f : m * c;
            // (S[st] last held the probabilities of tile j - 2; their product was issued before the Q K^T of this tile)
            // probabilities -> bf16 pairs -> A operand of the P V product in tensor memory; this thread's 64 keys
            // are 32 packed columns
            float rs = 0.f;
            uint32_t pk[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                const float p0 = fast_exp2(fmaf(__uint_as_float(sv[2 * i]), c, -mc));
                const float p1 = fast_exp2(fmaf(__uint_as_float(sv[2 * i + 1]), c, -mc));
                rs += p0 + p1;
                pk[i] = pack_bf16x2(p0, p1);
            }
            // into the columns the scores of keys 0-63 came from (both threads of the row have read theirs: the
            // exchange above lies in between); 64 keys of the row are 32 columns
            tmem_st32(tmem_base + st * 128 + lane_off + half * 32, pk);
            l += rs;
            if (!seen_prev) ok = ok && mbar_wait(o_full, (uint32_t)(j - 1) & 1u, status);   // P V of tile j - 1 (precedes this tile's anyway)
            tc_fence_before();
            mbar_arrive(&p_full[st]);
        }
        // the last P V product, then out = O / l (l = the sum of the two half-row sums)
        ok = ok && mbar_wait(o_full, (uint32_t)(nt - 1) & 1u, status);
        tc_fence_after();
        xm[r][half] = l;
        pair_sync();
        float den = xm[r][0] + xm[r][1];
        if (a.sink) den += fast_exp2(fmaf(a.sink[head], 1.4426950408889634f, -m * c));   // no value, and not scaled
        float inv = 1.0f / den;
        if (a.gate && q0 + r < S) inv *= 1.0f / (1.0f + __expf(-a.gate[(size_t)(q0 + r) * a.ld_gate + head]));
        bf16* orow = a.out + (size_t)(q0 + r) * a.ld_out + head * a.head_cols + half * OC;
        const int cols = a.head_cols - half * OC;             // value columns left for this thread
#pragma unroll
        for (int cb = 0; cb < VP; ++cb) {
            uint32_t v[32];
            tmem_ld32(tmem_o + lane_off + out_off + cb * 32, v);
            if (q0 + r < S) {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (cb * 32 + 8 * q < cols)
                    reinterpret_cast<uint4*>(orow + cb * 32)[q] =
                        make_uint4(pack_bf16x2(__uint_as_float(v[8 * q]) * inv, __uint_as_float(v[8 * q + 1]) * inv),
                                   pack_bf16x2(__uint_as_float(v[8 * q + 2]) * inv, __uint_as_float(v[8 * q + 3]) * inv),
                                   pack_bf16x2(__uint_as_float(v[8 * q + 4]) * inv, __uint_as_float(v[8 * q + 5]) * inv),
                                   pack_bf16x2(__uint_as_float(v[8 * q + 6]) * inv, __uint_as_float(v[8 * q + 7]) * inv));
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, TA_TMEM_COLS);
}

template <int QP, int RP, int VP>
static int launch_attention_tc(int heads, const CUtensorMap& mq_, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mqr,
                               const CUtensorMap& mkr, const AttnTcArgs& a, cudaStream_t stream) {
    using Cfg = AttnTcCfg<QP, RP, VP>;
    static bool attr_set[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !attr_set[dev]) {
        cudaError_t e = cudaFuncSetAttribute(k_attention_tc<QP, RP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM);
        if (e != cudaSuccess) return (int)e;
        attr_set[dev] = true;
    }
    launch_pdl(k_attention_tc<QP, RP, VP>, dim3(heads, (a.S + TA_BQ - 1) / TA_BQ), dim3(TA_THREADS), Cfg::SMEM, stream, mq_, mk, mv, mqr, mkr, a);
    return (int)cudaGetLastError();
}

}  // namespace mq
