// Recurrent mixers: per head the state S [dim, vdim] decays and takes up k v^T token by token, and
// the output is S^T q.  What decays it is a parameter: a constant per head (lightning attention),
// a factor per head and token with k weighted by the step size (Mamba-2), or a factor per key channel
// and token (gated linear attention).  State, decays and scores are 32-bit.
//
// Two forms.  k_recurrence_tokens walks token by token with the state in registers: decoding,
// short portions, 32-bit models, and head sizes that the other form does not hold.  The chunked
// form works on chunks of 128 tokens: k_chunk_kv computes what each chunk adds to the state,
// all chunks at once; k_chunk_scan walks over the chunks element by element and leaves behind
// the state BEFORE every chunk; k_chunk_out (k_channel_out), again all chunks at once, adds q times that state
// and the causal product inside the chunk.  Its products run on mma.sync with q, k, v as they are (bf16) and every 32-bit
// factor (state, decayed keys and queries, decayed scores) split into two bf16 terms, hi = bf16(x) and
// lo = bf16(x - hi), which keeps 16 to 17 bits of it; sums are 32-bit.  These products are a few per cent
// of a layer's work and bound by traffic, so they stay off tcgen05, whose operands would
// have to pass through shared memory twice for the split.
//
// Decays that the token sets are handled as running sums of logarithms (units of log2) inside a chunk, and only
// differences with a non-positive value are ever exponentiated, so that no factor overflows however fast a state decays.
#include "hy_common.cuh"

namespace mq {
namespace hy {

constexpr int LC = MQH_CHUNK;

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(a, b);
    lo = pack_bf16x2(a - bf_lo(hi), b - bf_hi(hi));
}

// acc[2 np], acc[2 np + 1] += a * b[np]: NP independent pairs, so that the term that follows finds them finished
template <int NP>
__device__ __forceinline__ void mma_row(float (&acc)[2 * NP][4], const uint32_t (&a)[4], const uint32_t (&b)[NP][4]) {
#pragma unroll
    for (int np = 0; np < NP; ++np) {
        mma16816(acc[2 * np], a, b[np][0], b[np][1]);
        mma16816(acc[2 * np + 1], a, b[np][2], b[np][3]);
    }
}

// log2 of the factor sigmoid(z)^inv_tau
__device__ __forceinline__ float channel_log_decay(float z, float inv_tau) { return -softplus(-z) * inv_tau * LOG2E; }
// the same by base-2 functions; 1 + e is rounded, an error of 2^-24 in the factor before it is raised to inv_tau
__device__ __forceinline__ float channel_log_decay_fast(float z, float inv_tau) {
    return -fmaf(fmaxf(-z, 0.f), LOG2E, log2f(1.0f + exp2f(-fabsf(z) * LOG2E))) * inv_tau;
}

// ---------------------------------------------------------------- short convolution
// y_t = silu(b + sum_j w[j] x_(t - taps + 1 + j)), channel by channel.  The state holds the input of position p in row p % taps:
// a token reads the taps - 1 rows before its own and overwrites the one row that nobody needs any more.  Positions before 0
// count as zeros, so a new sequence needs no clearing.
__device__ __forceinline__ int ring_row(int pos, int taps) { return pos % taps; }
constexpr int CV_THREADS = 512, CV_RUN = 8, CV_TOKENS = CONV_MAX_TAPS;     // tokens of one CTA: only the first CTA looks before the portion
static_assert(CV_THREADS / 64 * CV_RUN == CV_TOKENS, "runs of a CTA");
template <typename T>
__global__ void __launch_bounds__(CV_THREADS) k_conv_rows(const T* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, T* state,
                                                          T* __restrict__ y, int n, int pos0, int channels, int taps) {
    pdl_trigger();
    pdl_wait();
    const int c = (blockIdx.x * 64 + (threadIdx.x & 63)) * 4, t0 = blockIdx.y * CV_TOKENS, t1 = min(t0 + CV_TOKENS, n);
    const bool live = c < channels;
    if (live) {
        const float4 bias = load4(b + c);
        // a thread has a run of eight tokens; with four taps its inputs are read once, side by side, other filters read again
        const int ta = t0 + (threadIdx.x >> 6) * CV_RUN, te = min(ta + CV_RUN, t1);
        auto input = [&](int t) {
            if (t >= 0) return load4_cg(x + (size_t)t * channels + c);
            if (pos0 + t < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
            return load4_cg(state + (size_t)ring_row(pos0 + t, taps) * channels + c);
        };
        auto add = [](float4& s, const float4& u, const float4& v) {
            s.x = fmaf(u.x, v.x, s.x); s.y = fmaf(u.y, v.y, s.y); s.z = fmaf(u.z, v.z, s.z); s.w = fmaf(u.w, v.w, s.w);
        };
        auto put = [&](int t, const float4& s) {
            store4(y + (size_t)t * channels + c, make_float4(silu<T>(s.x), silu<T>(s.y), silu<T>(s.z), silu<T>(s.w)));
        };
        if (taps == 4 && ta < te) {
            const float4 w0 = load4(w + c), w1 = load4(w + channels + c), w2 = load4(w + 2 * channels + c), w3 = load4(w + 3 * channels + c);
            float4 in[CV_RUN + 3];
#pragma unroll
            for (int i = 0; i < CV_RUN + 3; ++i)
                if (ta + i - 3 < te) in[i] = input(ta + i - 3);
#pragma unroll
            for (int i = 0; i < CV_RUN; ++i)
                if (ta + i < te) {
                    float4 s = bias;
                    add(s, w0, in[i]); add(s, w1, in[i + 1]); add(s, w2, in[i + 2]); add(s, w3, in[i + 3]);
                    put(ta + i, s);
                }
        } else {
            for (int t = ta; t < te; ++t) {
                float4 s = bias;
                for (int j = 0; j < taps; ++j) add(s, load4(w + (size_t)j * channels + c), input(t - taps + 1 + j));
                put(t, s);
            }
        }
    }
    if (blockIdx.y != 0) return;
    __syncthreads();                                    // every read of the old rows lies before this
    if (live && threadIdx.x < 64)
        for (int t = max(0, n - (taps - 1)); t < n; ++t)
            store4(state + (size_t)ring_row(pos0 + t, taps) * channels + c, load4_cg(x + (size_t)t * channels + c));
}
template <typename T>
int conv_rows(Stream& st, const T* x, const float* w, const float* b, T* state, T* y, int n, int pos0, int channels, int taps) {
    if (taps > CONV_MAX_TAPS) return MQ_ERR_UNSUPPORTED;
    return launch(st, k_conv_rows<T>, dim3((channels / 4 + 63) / 64, (n + CV_TOKENS - 1) / CV_TOKENS), dim3(CV_THREADS), 0, x, w, b, state, y, n, pos0,
                  channels, taps);
}
template int conv_rows<bf16>(Stream&, const bf16*, const float*, const float*, bf16*, bf16*, int, int, int, int);
template int conv_rows<float>(Stream&, const float*, const float*, const float*, float*, float*, int, int, int, int);

// ---------------------------------------------------------------- token by token
// One CTA per (32 value columns, head).  Thread = (column quad, row group): rows ig, ig + 32, .. of S.
// CONV: one token whose q, k, v come out of the short convolution, which every CTA evaluates for what it needs.
constexpr int RT_THREADS = 256, RT_RANK = 16;
static size_t rt_smem(int mode, bool conv, int dim) { return (size_t)((mode == DECAY_CHANNEL ? dim : 0) + (conv ? 2 * dim + 32 : 0)) * 4; }
template <typename T, int MAXI, int MODE, bool CONV>
__global__ void __launch_bounds__(RT_THREADS) k_recurrence_tokens(RecurrenceArgs a) {
    extern __shared__ float rt_raw[];               // MODE channel: decays [dim]; CONV: q [dim], k [dim], v [32]
    __shared__ float part[8][32];
    constexpr int CPT = (MAXI * 32 + RT_THREADS - 1) / RT_THREADS;                  // key channels per thread
    constexpr int IPT = CONV ? (2 * MAXI * 32 + 32 + RT_THREADS - 1) / RT_THREADS : 1;  // convolution channels per thread
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y;
    const int j = blockIdx.x * 32 + (tid & 7) * 4, ig = tid >> 3;
    const int dim = a.dim, vdim = a.vdim, kvh = MODE == DECAY_HEAD ? head / (a.heads / a.kv_heads) : head;
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
    const T* q = reinterpret_cast<const T*>(a.q) + (size_t)kvh * dim;
    const T* k = reinterpret_cast<const T*>(a.k) + (size_t)kvh * dim;
    const T* v = reinterpret_cast<const T*>(a.v) + (size_t)head * vdim;
    const size_t ldq = a.ldq, ldk = a.ldk, ldv = a.ldv, ldo = (size_t)a.heads * vdim;
    float decay = 0.f, bias = 0.f, a_neg = 0.f, skip = 0.f;
    if (MODE == DECAY_CONST) decay = a.decay_pow[head * (LC + 1) + 1];
    if (MODE == DECAY_HEAD) { bias = a.dt_bias[head]; a_neg = a.a_neg[head]; skip = a.skip[head]; }
    // decay projection: the first weights of this thread's channels
    const T* gw = reinterpret_cast<const T*>(a.gate_w) + (size_t)head * a.rank * dim;
    float gk[MODE == DECAY_CHANNEL ? RT_RANK : 1][CPT], gb[CPT];
    float* al = rt_raw;
    if (MODE == DECAY_CHANNEL) {
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
            const int ch = tid + x * RT_THREADS;
            gb[x] = ch < dim ? a.gate_b[head * dim + ch] : 0.f;
#pragma unroll
            for (int r = 0; r < RT_RANK; ++r) gk[r][x] = ch < dim && r < a.rank ? Elem<T>::get(gw[(size_t)r * dim + ch]) : 0.f;
        }
    }
    // convolution: what the earlier tokens contribute.  Items: v columns, then k, then q channels
    float *cq = rt_raw, *ck = rt_raw + dim, *cv = rt_raw + 2 * dim;
    const int hv = a.heads * vdim, gn = a.kv_heads * dim, items = 32 + 2 * dim;
    int pos = 0;
    float past[IPT], wlast[IPT];
    auto channel = [&](int it) {
        if (it < 32) return blockIdx.x * 32 + it < vdim ? head * vdim + (int)blockIdx.x * 32 + it : -1;
        it -= 32;
        return it < dim ? hv + kvh * dim + it : it < 2 * dim ? hv + gn + kvh * dim + it - dim : -1;
    };
    if (CONV) {
        pos = *a.position;                          // set before this step began
        if (pos < 0 || pos >= a.max_seq) {
            if (tid == 0) atomicOr(a.status, MQ_STATUS_BAD_POSITION);
            pos = pos < 0 ? 0 : a.max_seq - 1;
        }
        const T* ring = reinterpret_cast<const T*>(a.conv_state);
#pragma unroll
        for (int x = 0; x < IPT; ++x) {
            const int it = tid + x * RT_THREADS, c = it < items ? channel(it) : -1;
            past[x] = wlast[x] = 0.f;
            if (c < 0) continue;
            past[x] = a.conv_b[c];
            for (int t = 0; t + 1 < a.taps; ++t) {
                const int p = pos - a.taps + 1 + t;
                if (p >= 0) past[x] = fmaf(a.conv_w[(size_t)t * a.channels + c], Elem<T>::get(__ldcg(ring + (size_t)ring_row(p, a.taps) * a.channels + c)), past[x]);
            }
            wlast[x] = a.conv_w[(size_t)(a.taps - 1) * a.channels + c];
        }
    }
    pdl_trigger();
    pdl_wait_cta();
    if (CONV) {
        const T* in = reinterpret_cast<const T*>(a.conv_in);
        T* ring = reinterpret_cast<T*>(a.conv_state) + (size_t)ring_row(pos, a.taps) * a.channels;
        const bool owner = blockIdx.x == 0 && head % (a.heads / a.kv_heads) == 0;     // of the channels that heads share
#pragma unroll
        for (int x = 0; x < IPT; ++x) {
            const int it = tid + x * RT_THREADS, c = it < items ? channel(it) : -1;
            if (c < 0) continue;
            const T now = __ldcg(in + c);
            const float y = Elem<T>::round(silu<T>(fmaf(wlast[x], Elem<T>::get(now), past[x])));
            if (it < 32) cv[it] = y;
            else if (it < 32 + dim) ck[it - 32] = y;
            else cq[it - 32 - dim] = y;
            if (it < 32 || owner) ring[c] = now;
        }
        __syncthreads();
    }
    for (int t = 0; t < a.n; ++t) {
        float4 vv = make_float4(0.f, 0.f, 0.f, 0.f);
        if (live) vv = CONV ? load4(cv + (tid & 7) * 4) : load4_cg(v + t * ldv + j);
        float vs = 0.f;                             // the value column whose output this thread stores
        if (MODE == DECAY_HEAD) {
            if (tid < 32 && blockIdx.x * 32 + tid < vdim) vs = CONV ? cv[tid] : Elem<T>::get(__ldcg(v + t * ldv + blockIdx.x * 32 + tid));
            const float dt = softplus(__ldcg(a.decay_in + (size_t)t * a.ld_decay + head) + bias);
            decay = expf(a_neg * dt);
            vv.x *= dt; vv.y *= dt; vv.z *= dt; vv.w *= dt;
        }
        if (MODE == DECAY_CHANNEL) {
            const float* in = a.decay_in + (size_t)t * a.ld_decay;
            float z[CPT];
#pragma unroll
            for (int x = 0; x < CPT; ++x) z[x] = gb[x];
#pragma unroll
            for (int r = 0; r < RT_RANK; ++r)
                if (r < a.rank) {
                    const float u = __ldcg(in + r);
#pragma unroll
                    for (int x = 0; x < CPT; ++x) z[x] = fmaf(u, gk[r][x], z[x]);
                }
            for (int r = RT_RANK; r < a.rank; ++r) {
                const float u = __ldcg(in + r);
#pragma unroll
                for (int x = 0; x < CPT; ++x)
                    if (tid + x * RT_THREADS < dim) z[x] = fmaf(u, Elem<T>::get(gw[(size_t)r * dim + tid + x * RT_THREADS]), z[x]);
            }
#pragma unroll
            for (int x = 0; x < CPT; ++x)
                if (tid + x * RT_THREADS < dim) al[tid + x * RT_THREADS] = exp2f(channel_log_decay(z[x], a.inv_tau));
            __syncthreads();
        }
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int m = 0; m < MAXI; ++m) {
            const int i = ig + 32 * m;
            if (i >= dim) break;
            const float ki = CONV ? ck[i] : Elem<T>::get(__ldcg(k + t * ldk + i)), qi = CONV ? cq[i] : Elem<T>::get(__ldcg(q + t * ldq + i));
            const float d = MODE == DECAY_CHANNEL ? al[i] : decay;
            s[m].x = fmaf(d, s[m].x, ki * vv.x); s[m].y = fmaf(d, s[m].y, ki * vv.y);
            s[m].z = fmaf(d, s[m].z, ki * vv.z); s[m].w = fmaf(d, s[m].w, ki * vv.w);
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
            a.o[t * ldo + (size_t)head * vdim + blockIdx.x * 32 + tid] = MODE == DECAY_HEAD ? fmaf(skip, vs, sum) : MODE == DECAY_CHANNEL ? sum * a.scale : sum;
        }
        __syncthreads();
    }
#pragma unroll
    for (int m = 0; m < MAXI; ++m) {
        const int i = ig + 32 * m;
        if (live && i < dim) store4(S + (size_t)i * vdim + j, s[m]);
    }
}
template <typename T, int MODE, bool CONV>
static int tokens(Stream& st, const RecurrenceArgs& a) {
    const dim3 grid((a.vdim + 31) / 32, a.heads), block(RT_THREADS);
    const size_t smem = rt_smem(MODE, CONV, a.dim);
    if (a.dim <= 128) return launch(st, k_recurrence_tokens<T, 4, MODE, CONV>, grid, block, smem, a);
    if (a.dim <= 256) return launch(st, k_recurrence_tokens<T, 8, MODE, CONV>, grid, block, smem, a);
    if (a.dim <= 512) return launch(st, k_recurrence_tokens<T, 16, MODE, CONV>, grid, block, smem, a);
    return MQ_ERR_UNSUPPORTED;
}
template <typename T>
int recurrence_tokens(Stream& st, const RecurrenceArgs& a) {
    if (a.mode == DECAY_CONST) return tokens<T, DECAY_CONST, false>(st, a);
    if (a.mode == DECAY_CHANNEL) return tokens<T, DECAY_CHANNEL, false>(st, a);
    return a.conv_in ? tokens<T, DECAY_HEAD, true>(st, a) : tokens<T, DECAY_HEAD, false>(st, a);
}
template int recurrence_tokens<bf16>(Stream&, const RecurrenceArgs&);
template int recurrence_tokens<float>(Stream&, const RecurrenceArgs&);

// rows x cols bf16 (cols a multiple of 8) from a matrix of row length ld into shared memory of row length sld by
// asynchronous copies; rows from `live` on and columns from `cols_live` on become zeros.  PER threads share a row, so that
// no index is divided by a run-time value.
template <int THREADS, int PER>
__device__ __forceinline__ void copy_tile(bf16* dst, int sld, const bf16* src, size_t ld, int rows, int live, int cols, int cols_live) {
    const int r0 = threadIdx.x / PER, c0 = (threadIdx.x % PER) * 8;
    for (int col = c0; col < cols; col += PER * 8) {
        const bool cok = col < cols_live;
        const bf16* p = src + (size_t)r0 * ld + col;
        bf16* d = dst + r0 * sld + col;
        for (int r = r0; r < rows; r += THREADS / PER) {
            const bool ok = cok && r < live;
            cp_async16_zfill(d, ok ? p : src, ok);
            p += (size_t)(THREADS / PER) * ld;
            d += (THREADS / PER) * sld;
        }
    }
}

// ---------------------------------------------------------------- chunked: decays
// Per head: step sizes dt and running sums (inclusive) of the log2 decays of a chunk's tokens, [HP][LC] for heads head ..;
// tokens beyond cnt add nothing.  Every thread of the CTA calls it; the results stand behind a barrier.
template <int HP>
__device__ __forceinline__ void head_decays(const RecurrenceArgs& a, int head, size_t row0, int cnt, float* dt, float* L, float* wsum) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, t = tid & (LC - 1), h = head + tid / LC;
    float x = 0.f, s = 0.f;
    if (tid < HP * LC) {
        if (t < cnt) x = softplus(__ldcg(a.decay_in + (row0 + t) * a.ld_decay + h) + a.dt_bias[h]);
        s = x * a.a_neg[h] * LOG2E;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += u;
        }
        if (lane == 31) wsum[warp] = s;
    }
    __syncthreads();
    if (tid < HP * LC) {
        for (int w = warp & ~(LC / 32 - 1); w < warp; ++w) s += wsum[w];
        dt[tid] = x;
        L[tid] = s;
    }
    __syncthreads();
}
// value columns (v or the state): JT columns of one head, or 64 each of two heads whose columns are `next` elements apart
template <int THREADS, int JT, bool PAIR>
__device__ __forceinline__ void copy_values(bf16* dst, const bf16* src, size_t ld, int rows, int live, int cols_live, size_t next) {
    if (PAIR) {
        copy_tile<THREADS, 8>(dst, JT + 8, src, ld, rows, live, 64, cols_live);
        copy_tile<THREADS, 8>(dst + 64, JT + 8, src + next, ld, rows, live, 64, cols_live);
    } else {
        copy_tile<THREADS, JT / 8>(dst, JT + 8, src, ld, rows, live, JT, cols_live);
    }
}
// Per key channel: cum [n, heads*dim] = running sums (inclusive, from the chunk's first token) of the log2 decays.
// One CTA per (32 channels, chunk): thread = (channel, run of CG_RUN tokens).
constexpr int CG_RUN = 16, CG_THREADS = 32 * (LC / CG_RUN), CG_RANK = 16;
__global__ void __launch_bounds__(CG_THREADS, 4) k_channel_decays(RecurrenceArgs a, float* __restrict__ cum) {
    pdl_trigger();
    __shared__ float in[LC][CG_RANK];
    __shared__ float total[LC / CG_RUN][32];
    const int tid = threadIdx.x, lane = tid & 31, run = tid >> 5, c = blockIdx.y;
    const int hd = a.heads * a.dim, ch = blockIdx.x * 32 + lane, cnt = min(LC, a.n - c * LC);
    const bool live = ch < hd;
    const int head = live ? ch / a.dim : 0;
    const bf16* gw = reinterpret_cast<const bf16*>(a.gate_w) + (size_t)head * a.rank * a.dim + (live ? ch - head * a.dim : 0);
    const float b = live ? a.gate_b[ch] : 0.f;
    float z[CG_RUN];
#pragma unroll
    for (int x = 0; x < CG_RUN; ++x) z[x] = b;
    float w[CG_RANK];
#pragma unroll
    for (int r = 0; r < CG_RANK; ++r) w[r] = live ? __bfloat162float(gw[(size_t)r * a.dim]) : 0.f;
    pdl_wait();
    for (int r0 = 0; r0 < a.rank; r0 += CG_RANK) {         // rank is a multiple of 16
        if (r0 > 0) {
#pragma unroll
            for (int r = 0; r < CG_RANK; ++r) w[r] = live ? __bfloat162float(gw[(size_t)(r0 + r) * a.dim]) : 0.f;
            __syncthreads();
        }
        for (int x = tid; x < LC * CG_RANK / 4; x += CG_THREADS) {
            const int t = x / (CG_RANK / 4), q = (x % (CG_RANK / 4)) * 4;
            store4(&in[t][q], t < cnt ? load4_cg(a.decay_in + (size_t)(c * LC + t) * a.ld_decay + r0 + q) : make_float4(0.f, 0.f, 0.f, 0.f));
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < CG_RUN; ++x) {
            const float* u = in[run * CG_RUN + x];
#pragma unroll
            for (int r = 0; r < CG_RANK; r += 4) {
                const float4 f = load4(u + r);
                z[x] = fmaf(f.x, w[r], z[x]); z[x] = fmaf(f.y, w[r + 1], z[x]); z[x] = fmaf(f.z, w[r + 2], z[x]); z[x] = fmaf(f.w, w[r + 3], z[x]);
            }
        }
    }
    float s = 0.f;
#pragma unroll
    for (int x = 0; x < CG_RUN; ++x) { s += channel_log_decay_fast(z[x], a.inv_tau); z[x] = s; }
    total[run][lane] = s;
    __syncthreads();
    float before = 0.f;
    for (int r = 0; r < run; ++r) before += total[r][lane];
#pragma unroll
    for (int x = 0; x < CG_RUN; ++x) {
        const int t = run * CG_RUN + x;
        if (live && t < cnt) cum[(size_t)(c * LC + t) * hd + ch] = before + z[x];
    }
}

// k of 8 channels times 2^e[..], as two bf16 terms
__device__ __forceinline__ void decay_split8(const uint4& k, const float4& e0, const float4& e1, uint4& hi, uint4& lo) {
    split_pair(bf_lo(k.x) * exp2f(e0.x), bf_hi(k.x) * exp2f(e0.y), hi.x, lo.x);
    split_pair(bf_lo(k.y) * exp2f(e0.z), bf_hi(k.y) * exp2f(e0.w), hi.y, lo.y);
    split_pair(bf_lo(k.z) * exp2f(e1.x), bf_hi(k.z) * exp2f(e1.y), hi.z, lo.z);
    split_pair(bf_lo(k.w) * exp2f(e1.z), bf_hi(k.w) * exp2f(e1.w), hi.w, lo.w);
}
__device__ __forceinline__ float4 sub4(const float4& a, const float4& b) { return make_float4(a.x - b.x, a.y - b.y, a.z - b.z, a.w - b.w); }

// ---------------------------------------------------------------- chunked: what every chunk adds to the state
// One CTA per (chunk, head, JT value columns): KV = sum over the chunk's n tokens of (decay from t to the chunk's end) k_t v_t^T, fp32.
// Warp w takes rows 16 (w % 8) + 128 x of the head's dim and half of the columns.  total [chunk, head] (per head): log2 of the
// whole chunk's decay.
constexpr int LK_THREADS = 512;
static size_t lk_smem(int mode, int dim, int jt) { return (size_t)LC * ((mode == DECAY_CHANNEL ? 2 : 1) * (dim + 8) + jt + 8) * 2; }
// PAIR: two heads that share q and k, one per half of the columns (JT = 128, vdim up to 64); blockIdx.y counts pairs.
template <int JT, int MODE, bool PAIR>
__global__ void __launch_bounds__(LK_THREADS, 2) k_chunk_kv(RecurrenceArgs a, float* __restrict__ kv, const float* __restrict__ cum, float* __restrict__ total) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t lk_raw[];
    constexpr int HP = PAIR ? 2 : 1;
    __shared__ float pws[HP * LC], sL[HP * LC], wsum[HP * LC / 32];             // pws by token: what k is scaled by
    constexpr int VLD = JT + 8, NP = JT / 32;                   // 16-column pairs of tiles per warp
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y * HP, c = blockIdx.x, j0 = blockIdx.z * JT;
    const int dim = a.dim, vdim = a.vdim, kld = dim + 8, jw = (warp >> 3) * (JT / 2), kvh = head / (a.heads / a.kv_heads);
    const float* pw = PAIR ? pws + (warp >> 3) * LC : pws;
    bf16* sk = reinterpret_cast<bf16*>(lk_raw);                 // MODE channel: the decayed keys' first terms, then the second
    bf16* sl = sk + LC * kld;
    bf16* sv = MODE == DECAY_CHANNEL ? sl + LC * kld : sl;
    const int cnt = min(LC, a.n - c * LC);
    const size_t row0 = (size_t)c * LC;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * a.ldk + (size_t)kvh * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * a.ldv + (size_t)head * vdim + j0;
    copy_values<LK_THREADS, JT, PAIR>(sv, vg, a.ldv, LC, cnt, vdim - j0, vdim);
    if (MODE != DECAY_CHANNEL) copy_tile<LK_THREADS, 16>(sk, kld, kg, a.ldk, LC, cnt, dim, dim);
    cp_async_commit();
    if (MODE == DECAY_CONST) {
        if (tid < LC) pws[tid] = tid < cnt ? a.decay_pow[head * (LC + 1) + cnt - 1 - tid] : 0.f;
    } else if (MODE == DECAY_HEAD) {
        head_decays<HP>(a, head, row0, cnt, pws, sL, wsum);
        if (tid < HP * LC) pws[tid] *= exp2f(sL[tid | (LC - 1)] - sL[tid]);
        if (tid < HP && blockIdx.z == 0) total[c * a.heads + head + tid] = sL[tid * LC + LC - 1];
    } else {
        const size_t hd = (size_t)a.heads * dim;
        const float* bg = cum + row0 * hd + (size_t)head * dim;
        const int r0 = tid / 16;
        for (int col = (tid % 16) * 8; col < dim; col += 128) {
            const float4 e0 = load4_cg(bg + (size_t)(cnt - 1) * hd + col), e1 = load4_cg(bg + (size_t)(cnt - 1) * hd + col + 4);
#pragma unroll 2
            for (int t = r0; t < LC; t += LK_THREADS / 16) {
                uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
                if (t < cnt)
                    decay_split8(ld_cg_u4(kg + (size_t)t * a.ldk + col), sub4(e0, load4_cg(bg + t * hd + col)), sub4(e1, load4_cg(bg + t * hd + col + 4)), hi, lo);
                *reinterpret_cast<uint4*>(sk + t * kld + col) = hi;
                *reinterpret_cast<uint4*>(sl + t * kld + col) = lo;
            }
        }
    }
    cp_async_wait_all();
    __syncthreads();
    const int ksteps = (cnt + 15) / 16;
    const int my = PAIR ? head + (warp >> 3) : head, col0 = PAIR ? 0 : j0 + jw;       // this warp's head and its first value column
    if (col0 >= vdim) return;
    for (int i0 = (warp & 7) * 16; i0 < dim; i0 += 128) {
        float acc[2 * NP][4];
#pragma unroll
        for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] = 0.f;
#pragma unroll 2
        for (int ks = 0; ks < ksteps; ++ks) {
            const int t0 = ks * 16, t = t0 + 2 * (lane & 3), koff = (t0 + (lane & 7) + ((lane >> 4) & 1) * 8) * kld + i0 + ((lane >> 3) & 1) * 8;
            uint32_t ah[4], al[4];
            if (MODE == DECAY_CHANNEL) {
                ldsm4_t(ah, smem_u32(sk + koff));
                ldsm4_t(al, smem_u32(sl + koff));
            } else {
                uint32_t ka[4];
                ldsm4_t(ka, smem_u32(sk + koff));
                const float w[4] = {pw[t], pw[t + 1], pw[t + 8], pw[t + 9]};
#pragma unroll
                for (int x = 0; x < 4; ++x) split_pair(bf_lo(ka[x]) * w[(x >> 1) * 2], bf_hi(ka[x]) * w[(x >> 1) * 2 + 1], ah[x], al[x]);
            }
            uint32_t b[NP][4];
#pragma unroll
            for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sv + (t0 + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8));
            mma_row<NP>(acc, ah, b);
            mma_row<NP>(acc, al, b);
        }
        float* dst = kv + ((size_t)c * a.heads + my) * dim * vdim + (size_t)(i0 + (lane >> 2)) * vdim + col0 + 2 * (lane & 3);
#pragma unroll
        for (int nt = 0; nt < 2 * NP; ++nt)
            if (col0 + nt * 8 < vdim) {
                *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(acc[nt][0], acc[nt][1]);
                *reinterpret_cast<float2*>(dst + (size_t)8 * vdim + nt * 8) = make_float2(acc[nt][2], acc[nt][3]);
            }
    }
}

// ---------------------------------------------------------------- chunked: the state before every chunk
// Element by element over the chunks: hi[c], lo[c] = the two bf16 terms of the state, state <- decay state + KV[c].
constexpr int LN_THREADS = 128, LN_AHEAD = 8;
template <int MODE>
__global__ void __launch_bounds__(LN_THREADS) k_chunk_scan(RecurrenceArgs a, const float* __restrict__ kv, const float* __restrict__ cum,
                                                           const float* __restrict__ total, bf16* __restrict__ hi, bf16* __restrict__ lo) {
    pdl_trigger();
    const size_t e = ((size_t)blockIdx.x * LN_THREADS + threadIdx.x) * 4, plane = (size_t)a.heads * a.dim * a.vdim;
    const bool live = e < plane;
    const int nchunks = (a.n + LC - 1) / LC, head = live ? (int)(e / ((size_t)a.dim * a.vdim)) : 0;
    const int hd = a.heads * a.dim, ch = live ? (int)(e / a.vdim) : 0;              // ch: head * dim + key channel
    float full = 0.f, last = 0.f;
    if (MODE == DECAY_CONST) {
        const float* pw = a.decay_pow + head * (LC + 1);
        full = pw[LC];
        last = pw[a.n - (nchunks - 1) * LC];
    }
    pdl_wait();
    if (!live) return;
    float4 s = load4_cg(a.state + e);
    for (int c0 = 0; c0 < nchunks; c0 += LN_AHEAD) {
        float4 v[LN_AHEAD];
        float d[LN_AHEAD];
#pragma unroll
        for (int x = 0; x < LN_AHEAD; ++x)
            if (c0 + x < nchunks) {
                v[x] = load4_cg(kv + (c0 + x) * plane + e);
                if (MODE == DECAY_CONST) d[x] = c0 + x == nchunks - 1 ? last : full;
                else if (MODE == DECAY_HEAD) d[x] = __ldcg(total + (size_t)(c0 + x) * a.heads + head);
                else d[x] = __ldcg(cum + (size_t)(min((c0 + x + 1) * LC, a.n) - 1) * hd + ch);
            }
#pragma unroll
        for (int x = 0; x < LN_AHEAD; ++x)
            if (c0 + x < nchunks) {
                uint2 h, l;
                split_pair(s.x, s.y, h.x, l.x);
                split_pair(s.z, s.w, h.y, l.y);
                *reinterpret_cast<uint2*>(hi + (c0 + x) * plane + e) = h;
                *reinterpret_cast<uint2*>(lo + (c0 + x) * plane + e) = l;
                const float f = MODE == DECAY_CONST ? d[x] : exp2f(d[x]);
                s.x = fmaf(f, s.x, v[x].x); s.y = fmaf(f, s.y, v[x].y); s.z = fmaf(f, s.z, v[x].z); s.w = fmaf(f, s.w, v[x].w);
            }
    }
    store4(a.state + e, s);
}

// ---------------------------------------------------------------- chunked: outputs
// Rows t0 + lane / 4 (+ 8) of a warp's accumulators -> columns col0 .. of the head's output.  vrow: the values of row t0 from
// column col0 on, for the skip.
template <int NT>
__device__ __forceinline__ void store_out(const RecurrenceArgs& a, const float (&acc)[NT][4], size_t row0, int cnt, int t0, int head, int col0, float skip,
                                          const bf16* vrow, int vld) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int r = (lane >> 2) + h * 8;
        if (t0 + r >= cnt) continue;
        float* orow = a.o + ((row0 + t0 + r) * a.heads + head) * a.vdim;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
            const int j = nt * 8 + 2 * (lane & 3);
            if (col0 + j >= a.vdim) continue;
            float2 y = make_float2(acc[nt][2 * h] * a.scale, acc[nt][2 * h + 1] * a.scale);
            if (skip != 0.f) {
                const uint32_t v = lds32(smem_u32(vrow + r * vld + j));
                y.x = fmaf(skip, bf_lo(v), y.x);
                y.y = fmaf(skip, bf_hi(v), y.y);
            }
            *reinterpret_cast<float2*>(orow + col0 + j) = y;
        }
    }
}
// One CTA per (chunk, head, JT value columns); each warp takes sixteen tokens t0 .. t0 + 15 of the chunk and half of the columns:
// o_t = D(start, t) q_t S + sum over s <= t of (q_t k_s) D(s, t) v_s      (t, s within the chunk; D: decay between two tokens)
constexpr int LO_THREADS = 512;
static size_t lo_smem(int dim, int jt) { return ((size_t)2 * LC * (dim + 8) + (size_t)(LC + 2 * dim) * (jt + 8)) * 2; }
template <int JT, int MODE, bool PAIR>
__global__ void __launch_bounds__(LO_THREADS, 1) k_chunk_out(RecurrenceArgs a, const bf16* __restrict__ hi, const bf16* __restrict__ lo) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t lo_raw[];
    constexpr int HP = PAIR ? 2 : 1;
    __shared__ float pws[HP * LC + 1], sdts[HP * LC], wsum[HP * LC / 32];       // pws: powers of the decay, or (per head and token) running log2 sums
    __shared__ float ends[MODE == DECAY_HEAD ? HP * LC : 1];                     // step size times the decay up to the end of the token's sixteen
    constexpr int VLD = JT + 8, NP = JT / 32;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y * HP, c = blockIdx.x, j0 = blockIdx.z * JT;
    const int dim = a.dim, vdim = a.vdim, qld = dim + 8, kvh = head / (a.heads / a.kv_heads);
    const float *pw = PAIR ? pws + (warp >> 3) * LC : pws, *sdt = PAIR ? sdts + (warp >> 3) * LC : sdts;
    const int cnt = min(LC, a.n - c * LC);
    bf16* sq = reinterpret_cast<bf16*>(lo_raw);
    bf16* sk = sq + LC * qld;
    bf16* sv = sk + LC * qld;
    bf16* sh = sv + LC * VLD;
    bf16* sl = sh + dim * VLD;
    const size_t row0 = (size_t)c * LC;
    const bf16* qg = reinterpret_cast<const bf16*>(a.q) + row0 * a.ldq + (size_t)kvh * dim;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * a.ldk + (size_t)kvh * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * a.ldv + (size_t)head * vdim + j0;
    const size_t plane = ((size_t)c * a.heads + head) * dim * vdim + j0;
    copy_tile<LO_THREADS, 16>(sq, qld, qg, a.ldq, LC, cnt, dim, dim);
    copy_values<LO_THREADS, JT, PAIR>(sh, hi + plane, vdim, dim, dim, vdim - j0, (size_t)dim * vdim);
    copy_values<LO_THREADS, JT, PAIR>(sl, lo + plane, vdim, dim, dim, vdim - j0, (size_t)dim * vdim);
    cp_async_commit();
    copy_tile<LO_THREADS, 16>(sk, qld, kg, a.ldk, LC, cnt, dim, dim);
    copy_values<LO_THREADS, JT, PAIR>(sv, vg, a.ldv, LC, cnt, vdim - j0, vdim);
    cp_async_commit();
    if (MODE == DECAY_CONST)
        for (int i = tid; i <= LC; i += LO_THREADS) pws[i] = a.decay_pow[head * (LC + 1) + i];
    else
        head_decays<HP>(a, head, row0, cnt, sdts, pws, wsum);
    if (MODE == DECAY_HEAD && tid < HP * LC) ends[tid] = sdts[tid] * exp2f(pws[tid | 15] - pws[tid]);
    cp_async_wait<1>();
    __syncthreads();
    // the causal work grows with the tokens' place in the chunk: the four warps of a scheduler (warp % 4) take an early and a
    // late sixteen for each half of the columns
    const int wr = (warp >> 2) & 1 ? 7 - (warp & 3) : warp & 3, jw = (warp >> 3) * (JT / 2);
    const int t0 = wr * 16, tl = t0 + (lane >> 2), dk = dim / 16;      // this thread's rows: tl, tl + 8
    const uint32_t qaddr = smem_u32(sq + (wr * 16 + (lane & 15)) * qld + (lane >> 4) * 8);
    float acc[2 * NP][4], low[2 * NP][4];                        // the state's second terms have sums of their own
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] = low[nt][e] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < dk; ++kk) {
        uint32_t qa[4], b[NP][4], d[NP][4];
        ldsm4(qa, qaddr + kk * 32);
#pragma unroll
        for (int np = 0; np < NP; ++np) {
            const int off = (kk * 16 + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8;
            ldsm4_t(b[np], smem_u32(sh + off));
            ldsm4_t(d[np], smem_u32(sl + off));
        }
        mma_row<NP>(acc, qa, b);
        mma_row<NP>(low, qa, d);
    }
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] += low[nt][e];
    const float l0 = MODE == DECAY_HEAD ? pw[tl] : 0.f, l1 = MODE == DECAY_HEAD ? pw[tl + 8] : 0.f;
    const float d0 = MODE == DECAY_HEAD ? exp2f(l0) : pw[tl + 1], d1 = MODE == DECAY_HEAD ? exp2f(l1) : pw[tl + 9];
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt) { acc[nt][0] *= d0; acc[nt][1] *= d0; acc[nt][2] *= d1; acc[nt][3] *= d1; }
    cp_async_wait<0>();
    __syncthreads();
    const int my = PAIR ? head + (warp >> 3) : head, col0 = PAIR ? 0 : j0 + jw;       // this warp's head and its first value column
    if (t0 >= cnt || col0 >= vdim) return;
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
        for (int hb = 0; hb < 2; ++hb) {                // sixteen keys each
            const int kb = s0 + hb * 16;
            if (MODE == DECAY_HEAD && kb < t0) {        // before this warp's tokens: by way of the sixteen's end
                const float* f = ends + (pw - pws) + kb;
                const float f0 = exp2f(l0 - pw[kb + 15]), f1 = exp2f(l1 - pw[kb + 15]);
#pragma unroll
                for (int x = 0; x < 8; ++x) {
                    const int nt = 2 * hb + (x >> 2), e = x & 3;
                    sc[nt][e] *= (e >> 1 ? f1 : f0) * f[(x >> 2) * 8 + 2 * (lane & 3) + (e & 1)];
                }
                continue;
            }
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                const int nt = 2 * hb + (x >> 2), e = x & 3, ts = s0 + nt * 8 + 2 * (lane & 3) + (e & 1), d = tl + (e >> 1) * 8 - ts;
                if (MODE == DECAY_CONST) sc[nt][e] = d >= 0 ? sc[nt][e] * pw[d] : 0.f;
                else sc[nt][e] = d >= 0 ? sc[nt][e] * exp2f((e >> 1 ? l1 : l0) - pw[ts]) * sdt[ts] : 0.f;
            }
        }
#pragma unroll
        for (int hb = 0; hb < 2; ++hb) {
            uint32_t b[NP][4];
#pragma unroll
            for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sv + (s0 + hb * 16 + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8));
            uint32_t ph[4], pl[4];
            split_pair(sc[2 * hb][0], sc[2 * hb][1], ph[0], pl[0]);
            split_pair(sc[2 * hb][2], sc[2 * hb][3], ph[1], pl[1]);
            split_pair(sc[2 * hb + 1][0], sc[2 * hb + 1][1], ph[2], pl[2]);
            split_pair(sc[2 * hb + 1][2], sc[2 * hb + 1][3], ph[3], pl[3]);
            mma_row<NP>(acc, ph, b);
            mma_row<NP>(acc, pl, b);
        }
    }
    store_out<2 * NP>(a, acc, row0, cnt, t0, my, col0, MODE == DECAY_HEAD ? a.skip[my] : 0.f, sv + t0 * VLD + jw, VLD);
}

// ---------------------------------------------------------------- chunked: outputs, a decay per key channel
// The same sums with b_t, the running log2 decays of the chunk (a vector over the key channels).  Sixteen tokens are a block; a
// warp has one block of queries and half of the columns:
//   its own block   score by score, sum over the channels of q k 2^(b_t - b_s), the two warps of a block taking half each
//   earlier blocks  the keys of block j are decayed to that block's end, k_s 2^(b_end(j) - b_s), once for everybody; the queries
//                   are decayed from the start of their own block and, while the warp walks back over the blocks, by each
//                   block it passes.  So every factor is a decay over a span of time, at most 1.
//   state           (q_t 2^b_t) S; the state takes the keys' place in shared memory while the values are multiplied
// STAGED: queries and decays stand in shared memory (dim up to 128), otherwise they are read where they are needed.
constexpr int BL = 16, NB = LC / BL;
static size_t co_smem(int dim, int jt, bool staged) {
    const size_t states = (size_t)2 * dim * (jt + 8), keys = (size_t)2 * LC * (dim + 8);
    return ((states > keys ? states : keys) + (size_t)LC * (jt + 8)) * 2 + (size_t)NB * dim * 4 + (size_t)NB * BL * (BL + 2) * 4 +
           (staged ? (size_t)LC * (dim + 8) * 6 : 0);
}
template <int JT, bool STAGED>
__global__ void __launch_bounds__(LO_THREADS, 1) k_channel_out(RecurrenceArgs a, const bf16* __restrict__ hi, const bf16* __restrict__ lo,
                                                               const float* __restrict__ cum) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t co_raw[];
    constexpr int VLD = JT + 8, NP = JT / 32, DLD = BL + 2;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, c = blockIdx.x, j0 = blockIdx.z * JT;
    const int dim = a.dim, vdim = a.vdim, kld = dim + 8;
    const int cnt = min(LC, a.n - c * LC);
    float* step = reinterpret_cast<float*>(co_raw);             // [NB][dim]: decay over a whole block
    float* diag = step + NB * dim;                              // [NB][BL][DLD]: scores inside the blocks
    bf16* sv = reinterpret_cast<bf16*>(diag + NB * BL * DLD);   // [LC][VLD]
    bf16* kh = sv + LC * VLD;                                   // keys: first terms (before: as they come) [LC][kld], second terms;
    bf16* kl = kh + LC * kld;
    bf16 *sh = kh, *sl = kh + dim * VLD;                        // later the state: first terms [dim][VLD], second terms
    const int region = max(2 * dim * VLD, 2 * LC * kld);
    bf16* sq = kh + region;                                     // STAGED: [LC][kld]
    float* sb = reinterpret_cast<float*>(sq + LC * kld);        // STAGED: [LC][kld]
    const size_t row0 = (size_t)c * LC, hd = (size_t)a.heads * dim;
    const bf16* qg = reinterpret_cast<const bf16*>(a.q) + row0 * a.ldq + (size_t)head * dim;
    const bf16* kg = reinterpret_cast<const bf16*>(a.k) + row0 * a.ldk + (size_t)head * dim;
    const bf16* vg = reinterpret_cast<const bf16*>(a.v) + row0 * a.ldv + (size_t)head * vdim + j0;
    const float* bg = cum + row0 * hd + (size_t)head * dim;
    const size_t plane = ((size_t)c * a.heads + head) * dim * vdim + j0;
    copy_tile<LO_THREADS, 16>(kh, kld, kg, a.ldk, LC, cnt, dim, dim);
    if (STAGED) {
        copy_tile<LO_THREADS, 16>(sq, kld, qg, a.ldq, LC, cnt, dim, dim);
        for (int t = tid / 32; t < LC; t += LO_THREADS / 32)
            for (int col = lane * 4; col < dim; col += 128)
                cp_async16_zfill(sb + t * kld + col, t < cnt ? bg + t * hd + col : bg, t < cnt);
    }
    cp_async_commit();
    copy_tile<LO_THREADS, JT / 8>(sv, VLD, vg, a.ldv, LC, cnt, JT, vdim - j0);
    cp_async_commit();
    // the decays and queries of a row (rows beyond cnt are not asked for)
    auto brow = [&](int t) { return STAGED ? sb + t * kld : bg + t * hd; };
    auto qrow = [&](int t) { return STAGED ? sq + t * kld : qg + (size_t)t * a.ldq; };
    const int wr = (warp >> 2) & 1 ? 7 - (warp & 3) : warp & 3, half = warp >> 3, jw = half * (JT / 2);
    const int t0 = wr * BL, tl = t0 + (lane >> 2), dk = dim / 16, c2 = 2 * (lane & 3);
    const bool on = t0 < cnt, cols = on && j0 + jw < vdim;
    cp_async_wait<1>();
    __syncthreads();
    // ---- scores inside the block: this warp's rows are t0 + 2 x + half, a lane has four channels of every 128
    if (on) {
        float mine[BL];                                         // [s]: this lane's share of rows x = 0 .. 7 after the exchange
#pragma unroll
        for (int s = 0; s < BL; ++s) mine[s] = 0.f;
        for (int base = 0; base < dim; base += 128) {           // lanes beyond the last channel add zeros
            const int d0 = base + lane * 4;
            const bool ok = d0 < dim;
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            float4 q[BL / 2], b[BL / 2];
#pragma unroll
            for (int x = 0; x < BL / 2; ++x) {
                const int t = t0 + 2 * x + half;
                q[x] = ok && t < cnt ? load4(qrow(t) + d0) : zero;
                b[x] = ok && t < cnt ? load4(brow(t) + d0) : zero;
            }
#pragma unroll
            for (int s = 0; s < BL; ++s) {
                if (t0 + s >= cnt) break;
                const float4 k = ok ? load4(kh + (t0 + s) * kld + d0) : zero, e = ok ? load4(brow(t0 + s) + d0) : zero;
                float p[BL / 2];
#pragma unroll
                for (int x = 0; x < BL / 2; ++x) {
                    p[x] = 0.f;
                    if (2 * x + half >= s && t0 + 2 * x + half < cnt)      // the same for the whole warp
                        p[x] = q[x].x * k.x * exp2f(b[x].x - e.x) + q[x].y * k.y * exp2f(b[x].y - e.y) + q[x].z * k.z * exp2f(b[x].z - e.z) +
                               q[x].w * k.w * exp2f(b[x].w - e.w);
                }
                // eight sums over the warp: after three exchanges lane l holds row (l & 7) over its group, then the groups meet
#pragma unroll
                for (int o = 4, w = 4; o > 0; o >>= 1, w >>= 1)
#pragma unroll
                    for (int x = 0; x < 4; ++x)
                        if (x < w) {
                            const bool up = lane & o;
                            const float send = up ? p[x] : p[x + w], keep = up ? p[x + w] : p[x];
                            p[x] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                        }
                p[0] += __shfl_xor_sync(0xffffffffu, p[0], 8);
                p[0] += __shfl_xor_sync(0xffffffffu, p[0], 16);
                mine[s] += p[0];
            }
        }
        if (lane < 8) {                                         // lane l ends with row x = l
            const int t = 2 * lane + half;
#pragma unroll
            for (int s = 0; s < BL; ++s) diag[(wr * BL + t) * DLD + s] = s <= t ? mine[s] : 0.f;
        }
    }
    __syncthreads();
    // ---- keys decayed to the end of their block (in place, with a second term), and the blocks' whole decays
    for (int col = (tid % 16) * 8; col < dim; col += 128)
#pragma unroll 2
        for (int t = tid / 16; t < LC; t += LO_THREADS / 16) {
            uint4 h = make_uint4(0u, 0u, 0u, 0u), l = h;
            if (t < cnt) {
                const float *e = brow(min(t | (BL - 1), cnt - 1)) + col, *f = brow(t) + col;
                decay_split8(*reinterpret_cast<const uint4*>(kh + t * kld + col), sub4(load4(e), load4(f)), sub4(load4(e + 4), load4(f + 4)), h, l);
            }
            *reinterpret_cast<uint4*>(kh + t * kld + col) = h;
            *reinterpret_cast<uint4*>(kl + t * kld + col) = l;
        }
    for (int j = tid / 64; j < NB; j += LO_THREADS / 64)
        for (int d = tid & 63; d < dim; d += 64)
            step[j * dim + d] = j * BL < cnt ? exp2f(brow(min(j * BL + BL - 1, cnt - 1))[d] - (j > 0 ? brow(j * BL - 1)[d] : 0.f)) : 0.f;
    cp_async_wait_all();
    __syncthreads();
    // rows beyond the end take the last token's place: their results are not stored
    const int ra = min(tl, cnt - 1), rb = min(tl + 8, cnt - 1);
    auto load_q = [&](int kk, int ref, float (&x)[8]) {         // the A fragment's eight elements, decayed since token ref (-1: the chunk's start)
        const int col = kk * 16 + c2;
        const bf16 *qa = qrow(ra) + col, *qb = qrow(rb) + col;
        const float *ba = brow(ra) + col, *bb = brow(rb) + col;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float2 r = make_float2(0.f, 0.f);
            if (ref >= 0) r = *reinterpret_cast<const float2*>(brow(ref) + col + 8 * h);
            const uint32_t u = *reinterpret_cast<const uint32_t*>(qa + 8 * h), v = *reinterpret_cast<const uint32_t*>(qb + 8 * h);
            const float2 f = *reinterpret_cast<const float2*>(ba + 8 * h), g = *reinterpret_cast<const float2*>(bb + 8 * h);
            x[4 * h] = bf_lo(u) * exp2f(f.x - r.x);
            x[4 * h + 1] = bf_hi(u) * exp2f(f.y - r.y);
            x[4 * h + 2] = bf_lo(v) * exp2f(g.x - r.x);
            x[4 * h + 3] = bf_hi(v) * exp2f(g.y - r.y);
        }
    };
    auto split_q = [](const float (&x)[8], uint32_t (&h)[4], uint32_t (&l)[4]) {
#pragma unroll
        for (int i = 0; i < 4; ++i) split_pair(x[2 * i], x[2 * i + 1], h[i], l[i]);
    };
    // ---- scores against the earlier blocks, block wr - 1 first
    float sc[NB - 1][2][4];
#pragma unroll
    for (int y = 0; y < NB - 1; ++y)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[y][0][e] = sc[y][1][e] = 0.f;
    if (cols && wr > 0) {
        const int koff = ((lane & 7) + ((lane >> 4) & 1) * 8) * kld + ((lane >> 3) & 1) * 8;
#pragma unroll 1
        for (int kk = 0; kk < dk; ++kk) {
            float x[8];
            load_q(kk, t0 - 1, x);
#pragma unroll
            for (int y = 0; y < NB - 1; ++y) {
                if (y >= wr) break;
                const int j = wr - 1 - y;
                uint32_t ah[4], al[4], bh[4], bl[4];
                split_q(x, ah, al);
                ldsm4(bh, smem_u32(kh + j * BL * kld + koff + kk * 16));
                ldsm4(bl, smem_u32(kl + j * BL * kld + koff + kk * 16));
                mma16816(sc[y][0], ah, bh[0], bh[1]);
                mma16816(sc[y][1], ah, bh[2], bh[3]);
                mma16816(sc[y][0], al, bh[0], bh[1]);
                mma16816(sc[y][1], al, bh[2], bh[3]);
                mma16816(sc[y][0], ah, bl[0], bl[1]);
                mma16816(sc[y][1], ah, bl[2], bl[3]);
                const float2 g0 = *reinterpret_cast<const float2*>(step + j * dim + kk * 16 + c2), g1 = *reinterpret_cast<const float2*>(step + j * dim + kk * 16 + c2 + 8);
                x[0] *= g0.x; x[1] *= g0.y; x[2] *= g0.x; x[3] *= g0.y;
                x[4] *= g1.x; x[5] *= g1.y; x[6] *= g1.x; x[7] *= g1.y;
            }
        }
    }
    __syncthreads();                                            // the keys have been read
    copy_tile<LO_THREADS, JT / 8>(sh, VLD, hi + plane, vdim, dim, dim, JT, vdim - j0);
    copy_tile<LO_THREADS, JT / 8>(sl, VLD, lo + plane, vdim, dim, dim, JT, vdim - j0);
    cp_async_commit();
    float acc[2 * NP][4];
#pragma unroll
    for (int nt = 0; nt < 2 * NP; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] = 0.f;
    auto add_values = [&](const float (&p0)[4], const float (&p1)[4], int j) {
        uint32_t b[NP][4], ph[4], pl[4];
#pragma unroll
        for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sv + (j * BL + (lane & 15)) * VLD + jw + np * 16 + (lane >> 4) * 8));
        split_pair(p0[0], p0[1], ph[0], pl[0]);
        split_pair(p0[2], p0[3], ph[1], pl[1]);
        split_pair(p1[0], p1[1], ph[2], pl[2]);
        split_pair(p1[2], p1[3], ph[3], pl[3]);
        mma_row<NP>(acc, ph, b);
        mma_row<NP>(acc, pl, b);
    };
    if (cols) {
#pragma unroll
        for (int y = 0; y < NB - 1; ++y) {
            if (y >= wr) break;
            add_values(sc[y][0], sc[y][1], wr - 1 - y);
        }
        const float* d = diag + (wr * BL + (lane >> 2)) * DLD + c2;
        const float2 u = *reinterpret_cast<const float2*>(d), v = *reinterpret_cast<const float2*>(d + 8 * DLD);
        const float2 w = *reinterpret_cast<const float2*>(d + 8), z = *reinterpret_cast<const float2*>(d + 8 * DLD + 8);
        const float p0[4] = {u.x, u.y, v.x, v.y}, p1[4] = {w.x, w.y, z.x, z.y};
        add_values(p0, p1, wr);
    }
    cp_async_wait_all();
    __syncthreads();
    if (!cols) return;
    // ---- state
#pragma unroll 2
    for (int kk = 0; kk < dk; ++kk) {
        float x[8];
        uint32_t ah[4], al[4], b[NP][4];
        load_q(kk, -1, x);
        split_q(x, ah, al);
        const int off = (kk * 16 + (lane & 15)) * VLD + jw + (lane >> 4) * 8;
#pragma unroll
        for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sh + off + np * 16));
        mma_row<NP>(acc, ah, b);
        mma_row<NP>(acc, al, b);
#pragma unroll
        for (int np = 0; np < NP; ++np) ldsm4_t(b[np], smem_u32(sl + off + np * 16));
        mma_row<NP>(acc, ah, b);
    }
    store_out<2 * NP>(a, acc, row0, cnt, t0, head, j0 + jw, 0.f, sv, VLD);
}

// ---------------------------------------------------------------- chunked: launches
// fp32 KV per chunk, two bf16 planes of the state before it, the running decays per channel and the chunks' decays per head
size_t recurrence_scratch_bytes(int n, int heads, int dim, int vdim) {
    const size_t chunks = (n + LC - 1) / LC;
    return chunks * heads * ((size_t)dim * vdim * (sizeof(float) + 2 * sizeof(bf16)) + (size_t)LC * dim * 4 + 4);
}
static bool staged(int dim, int jt) { return co_smem(dim, jt, true) + 2048 <= 232448; }
static size_t out_smem(int mode, int dim, int jt) { return mode == DECAY_CHANNEL ? co_smem(dim, jt, staged(dim, jt)) : lo_smem(dim, jt); }
static bool tile_fits(int mode, int dim, int jt) { return out_smem(mode, dim, jt) + 4096 <= 232448 && lk_smem(mode, dim, jt) + 4096 <= 232448; }
bool recurrence_chunked_fits(int mode, int dim) { return tile_fits(mode, dim, 64); }
template <int JT, int MODE, bool PAIR>
static int chunked(Stream& st, const RecurrenceArgs& a) {
    const int nchunks = (a.n + LC - 1) / LC;
    const dim3 grid = PAIR ? dim3(nchunks, a.heads / 2) : dim3(nchunks, a.heads, (a.vdim + JT - 1) / JT);
    const size_t elems = (size_t)nchunks * a.heads * a.dim * a.vdim;
    float* kv = reinterpret_cast<float*>(a.scratch);
    bf16 *hi = reinterpret_cast<bf16*>(kv + elems), *lo = hi + elems;
    float* cum = reinterpret_cast<float*>(lo + elems);                                 // [n, heads*dim]
    float* total = cum + (size_t)nchunks * LC * a.heads * a.dim;                        // [chunks, heads]
    int rc = 0;
    if (MODE == DECAY_CHANNEL) rc = launch(st, k_channel_decays, dim3((a.heads * a.dim + 31) / 32, nchunks), dim3(CG_THREADS), 0, a, cum);
    if (!rc) rc = allow_smem(k_chunk_kv<JT, MODE, PAIR>, lk_smem(MODE, a.dim, JT));
    if (!rc) rc = launch(st, k_chunk_kv<JT, MODE, PAIR>, grid, dim3(LK_THREADS), lk_smem(MODE, a.dim, JT), a, kv, (const float*)cum, total);
    const size_t quads = (size_t)a.heads * a.dim * a.vdim / 4;
    if (!rc) rc = launch(st, k_chunk_scan<MODE>, dim3((unsigned)((quads + LN_THREADS - 1) / LN_THREADS)), dim3(LN_THREADS), 0, a, (const float*)kv,
                         (const float*)cum, (const float*)total, hi, lo);
    const size_t smem = out_smem(MODE, a.dim, JT);
    if constexpr (MODE == DECAY_CHANNEL) {
        auto go = [&](auto kernel) {
            const int e = allow_smem(kernel, smem);
            return e ? e : launch(st, kernel, grid, dim3(LO_THREADS), smem, a, (const bf16*)hi, (const bf16*)lo, (const float*)cum);
        };
        if (!rc) rc = staged(a.dim, JT) ? go(k_channel_out<JT, true>) : go(k_channel_out<JT, false>);
    } else {
        if (!rc) rc = allow_smem(k_chunk_out<JT, MODE, PAIR>, smem);
        if (!rc) rc = launch(st, k_chunk_out<JT, MODE, PAIR>, grid, dim3(LO_THREADS), smem, a, (const bf16*)hi, (const bf16*)lo);
    }
    return rc;
}
int recurrence_chunked(Stream& st, const RecurrenceArgs& a) {
    if (!recurrence_chunked_fits(a.mode, a.dim) || !a.scratch) return MQ_ERR_UNSUPPORTED;
    // value columns of one CTA: 128 unless the head has no more than 64, or its dim leaves no room for them
    const bool roomy = tile_fits(a.mode, a.dim, 128), wide = a.vdim > 64 && roomy;
    if (a.mode == DECAY_CONST) return wide ? chunked<128, DECAY_CONST, false>(st, a) : chunked<64, DECAY_CONST, false>(st, a);
    if (a.mode == DECAY_HEAD) {
        if (wide) return chunked<128, DECAY_HEAD, false>(st, a);
        return a.vdim <= 64 && roomy && (a.heads / a.kv_heads) % 2 == 0 ? chunked<128, DECAY_HEAD, true>(st, a) : chunked<64, DECAY_HEAD, false>(st, a);
    }
    return wide ? chunked<128, DECAY_CHANNEL, false>(st, a) : chunked<64, DECAY_CHANNEL, false>(st, a);
}

}  // namespace hy
}  // namespace mq
