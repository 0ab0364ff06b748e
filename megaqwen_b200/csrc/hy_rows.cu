// Row-wise kernels of the layer-listed decoder's prefill: embedding, residual sum,
// norms, the loop's input, and the gated norm of a recurrence's output.  One CTA per row;
// the residual stream and every norm are 32-bit.
#include "hy_common.cuh"

namespace mq {
namespace hy {

// value of a row -> residual stream, then what the next product reads (see RowsArgs)
template <typename T>
__global__ void __launch_bounds__(256) k_rows(RowsArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float val[];               // [width]
    __shared__ float red[8];
    const int r = blockIdx.x, tid = threadIdx.x;
    size_t src = (size_t)r;
    if (a.gather) {
        int g = a.gather[r];
        src = (size_t)(g < 0 ? 0 : g > a.gather_max ? a.gather_max : g);
    }
    const T* erow = nullptr;
    if (a.ids) {
        int tok = a.ids[r];
        if (tok < 0 || tok >= a.vocab) {
            if (tid == 0) atomicOr(a.status, MQ_STATUS_BAD_TOKEN);
            tok = tok < 0 ? 0 : a.vocab - 1;
        }
        erow = reinterpret_cast<const T*>(a.embed) + (size_t)tok * a.width;
    }
    float ss = 0.f;
    auto plane_sum = [&](int i) {
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
        const float* p = a.planes + (size_t)r * a.ldp + i;
        for (int k = 0; k < a.nplanes; ++k) {
            const float4 q = load4(p + k * a.plane_stride);
            s.x += q.x; s.y += q.y; s.z += q.z; s.w += q.w;
        }
        return s;
    };
    float post_inv = 1.f;
    if (a.post) {                                // the sublayer's result is normed before it is added
        float ps = 0.f;
        for (int i = tid * 4; i < a.width; i += 1024) {
            const float4 s = plane_sum(i);
            ps += s.x * s.x + s.y * s.y + s.z * s.z + s.w * s.w;
            store4(val + i, s);
        }
        post_inv = 1.0f / sqrtf(cta_sum<8>(ps, red) / (float)a.norm_n + a.eps);
    }
    for (int i = tid * 4; i < a.width; i += 1024) {
        float4 v;
        if (erow) {
            v = load4(erow + i);
            v.x *= a.embed_scale; v.y *= a.embed_scale; v.z *= a.embed_scale; v.w *= a.embed_scale;
        } else {
            v = a.base ? load4(a.base + src * a.width + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (a.post) {
                const float4 s = load4(val + i), g = load4(a.post + i);
                v.x = fmaf(s.x * post_inv, g.x, v.x); v.y = fmaf(s.y * post_inv, g.y, v.y);
                v.z = fmaf(s.z * post_inv, g.z, v.z); v.w = fmaf(s.w * post_inv, g.w, v.w);
            } else if (a.nplanes > 0) {
                const float4 s = plane_sum(i);
                v.x = fmaf(a.mult, s.x, v.x); v.y = fmaf(a.mult, s.y, v.y); v.z = fmaf(a.mult, s.z, v.z); v.w = fmaf(a.mult, s.w, v.w);
            }
        }
        if (a.x) store4(a.x + (size_t)r * a.width + i, v);
        if (a.x0) store4(a.x0 + (size_t)r * a.width + i, v);
        if (a.h && !a.gain) store4(reinterpret_cast<T*>(a.h) + (size_t)r * a.width + i, v);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        store4(val + i, v);
    }
    if (a.gain) {
        const float inv = 1.0f / sqrtf(cta_sum<8>(ss, red) / (float)a.norm_n + a.eps);
        for (int i = tid * 4; i < a.width; i += 1024) {
            const float4 v = load4(val + i), g = load4(a.gain + i);
            store4(reinterpret_cast<T*>(a.h) + (size_t)r * a.width + i, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
        }
    }
    if (a.xin) {
        T* d = reinterpret_cast<T*>(a.xin) + (size_t)r * 2 * a.width;
        for (int i = tid * 4; i < a.width; i += 1024) {
            const float4 v = load4(val + i);
            store4(d + i, v);
            store4(d + a.width + i, a.x0_in ? load4(a.x0_in + (size_t)r * a.width + i) : v);
        }
    }
}
template <typename T>
int rows(Stream& st, int n, const RowsArgs& a) {
    const int rc = allow_smem(k_rows<T>, (size_t)a.width * 4);
    if (rc) return rc;
    return launch(st, k_rows<T>, dim3(n), dim3(256), (size_t)a.width * 4, a);
}
template int rows<bf16>(Stream&, int, const RowsArgs&);
template int rows<float>(Stream&, int, const RowsArgs&);

// the gated norm of a mixer's output, row by row
template <typename T, bool ONE>
__global__ void __launch_bounds__(256) k_gated_norm(GatedNorm a, T* __restrict__ cat, int ldc) {
    pdl_trigger();
    extern __shared__ float gn_raw[];            // [hv], gated_scratch
    __shared__ float red[8];
    float4 w0[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = threadIdx.x * 4 + x * 1024;
        w0[x] = i < a.hv ? load4(a.w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    const size_t r = blockIdx.x;
    a.o += r * a.hv;
    a.g = reinterpret_cast<const T*>(a.g) + r * a.hv;
    gated_norm_row<T, 8, ONE>(a, w0, gn_raw, gn_raw + a.hv, red, cat + r * ldc);
}
template <typename T>
int gated_norm(Stream& st, int n, const GatedNorm& a, T* cat, int ldc) {
    const size_t smem = (size_t)(a.hv + gated_scratch(a)) * 4;
    auto go = [&](auto kernel) {
        const int rc = allow_smem(kernel, smem);
        return rc ? rc : launch(st, kernel, dim3(n), dim3(256), smem, a, cat, ldc);
    };
    return a.parts == 1 ? go(k_gated_norm<T, true>) : go(k_gated_norm<T, false>);
}
template int gated_norm<bf16>(Stream&, int, const GatedNorm&, bf16*, int);
template int gated_norm<float>(Stream&, int, const GatedNorm&, float*, int);

}  // namespace hy
}  // namespace mq
