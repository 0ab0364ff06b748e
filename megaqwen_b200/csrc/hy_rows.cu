// Row-wise kernels of the layer-listed decoder's prefill: embedding, residual sum,
// norms, the loop's input, and the gated norm of lightning attention.  One CTA per row;
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
    for (int i = tid * 4; i < a.width; i += 1024) {
        float4 v;
        if (erow) {
            v = load4(erow + i);
            v.x *= a.embed_scale; v.y *= a.embed_scale; v.z *= a.embed_scale; v.w *= a.embed_scale;
        } else {
            v = a.base ? load4(a.base + src * a.width + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (a.nplanes > 0) {
                float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
                const float* p = a.planes + (size_t)r * a.ldp + i;
                for (int k = 0; k < a.nplanes; ++k) {
                    const float4 q = load4(p + k * a.plane_stride);
                    s.x += q.x; s.y += q.y; s.z += q.z; s.w += q.w;
                }
                v.x = fmaf(a.mult, s.x, v.x); v.y = fmaf(a.mult, s.y, v.y); v.z = fmaf(a.mult, s.z, v.z); v.w = fmaf(a.mult, s.w, v.w);
            }
        }
        if (a.x) store4(a.x + (size_t)r * a.width + i, v);
        if (a.x0) store4(a.x0 + (size_t)r * a.width + i, v);
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

// cat[r, i] = o[r, i] / rms(o[r]) * w[i] * sigmoid(g[r, i]): the concatenated heads are normed together
template <typename T>
__global__ void __launch_bounds__(256) k_gated_norm(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ g, T* __restrict__ cat,
                                                    int ldc, int hv, int norm_n, float eps) {
    pdl_trigger();
    pdl_wait();
    __shared__ float red[8];
    const int tid = threadIdx.x;
    const size_t r = blockIdx.x;
    float ss = 0.f;
    for (int i = tid * 4; i < hv; i += 1024) {
        const float4 v = load4(o + r * hv + i);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = 1.0f / sqrtf(cta_sum<8>(ss, red) / (float)norm_n + eps);
    for (int i = tid * 4; i < hv; i += 1024) {
        const float4 v = load4(o + r * hv + i), wv = load4(w + i), gv = load4(g + r * hv + i);
        store4(cat + r * ldc + i, make_float4(v.x * inv * wv.x * Elem<T>::sigmoid(gv.x), v.y * inv * wv.y * Elem<T>::sigmoid(gv.y),
                                              v.z * inv * wv.z * Elem<T>::sigmoid(gv.z), v.w * inv * wv.w * Elem<T>::sigmoid(gv.w)));
    }
}
template <typename T>
int gated_norm(Stream& st, int n, const float* o, const float* w, const T* g, T* cat, int ldc, int hv, int norm_n, float eps) {
    return launch(st, k_gated_norm<T>, dim3(n), dim3(256), 0, o, w, g, cat, ldc, hv, norm_n, eps);
}
template int gated_norm<bf16>(Stream&, int, const float*, const float*, const bf16*, bf16*, int, int, int, float);
template int gated_norm<float>(Stream&, int, const float*, const float*, const float*, float*, int, int, int, float);

}  // namespace hy
}  // namespace mq
