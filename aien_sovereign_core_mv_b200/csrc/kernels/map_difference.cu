// The difference of two attention maps over the same values, normed per head.
//
// a [T, lda] float32 holds, per key/value head g, the outputs of map 1 for its `per` query heads and then those of map 2:
// head r of map m of group g at columns ((g * 2 + m) * per + r) * V.  For query head h = g * per + r, element by element
//     o = a1 - lambda * a2;   out[t, h * V + i] = o_i / sqrt(mean(o^2) + eps) * mult
// in float32, rounded once to out's dtype.  A warp per (token, head); heads of up to 256 numbers stay in registers.
#include "common.cuh"

namespace aien {

template <typename TO, int VEC, int N>
__global__ void __launch_bounds__(256)
map_difference_norm_kernel(const float* __restrict__ a, long lda, TO* __restrict__ out, long ldo, int T, int H, int per, int V,
                           float lambda, float eps, float mult) {
    griddep_launch();
    const int lane = threadIdx.x & 31;
    const long unit = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (unit >= (long)T * H) return;
    const int t = (int)(unit / H), h = (int)(unit - (long)t * H), g = h / per, r = h - g * per;
    const float* p1 = a + (size_t)t * lda + (size_t)(2 * g * per + r) * V;
    const float* p2 = p1 + (size_t)per * V;
    griddep_wait();
    float o[N][VEC];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < N; ++j) {
        const int i = (j * 32 + lane) * VEC;
        if (i < V) {
            if constexpr (VEC == 4) {
                const float4 x = ld_act4(p1 + i), y = ld_act4(p2 + i);
                o[j][0] = fmaf(-lambda, y.x, x.x); o[j][1] = fmaf(-lambda, y.y, x.y);
                o[j][2] = fmaf(-lambda, y.z, x.z); o[j][3] = fmaf(-lambda, y.w, x.w);
            } else {
                o[j][0] = fmaf(-lambda, ld_act(p2 + i), ld_act(p1 + i));
            }
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) o[j][e] = 0.f;
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(o[j][e], o[j][e], ss);
    }
    const float f = mult / sqrtf(warp_sum(ss) / (float)V + eps);
    TO* dst = out + (size_t)t * ldo + (size_t)h * V;
#pragma unroll
    for (int j = 0; j < N; ++j) {
        const int i = (j * 32 + lane) * VEC;
        if (i >= V) continue;
        if constexpr (VEC == 4 && sizeof(TO) == 2) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(o[j][0] * f, o[j][1] * f), hi = __floats2bfloat162_rn(o[j][2] * f, o[j][3] * f);
            *reinterpret_cast<uint2*>(dst + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) dst[i + e] = from_f<TO>(o[j][e] * f);
        }
    }
}

}  // namespace aien

using namespace aien;

AIEN_API int aien_map_difference_norm(const float* a, long lda, void* out, int o_dt, long ldo, int T, int H, int per, int V, float lambda,
                                      float eps, float mult, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || per <= 0 || H % per != 0 || V <= 0 || V > 256) return AIEN_E_SHAPE;
    const long blocks = ((long)T * H + 7) / 8;
    if (blocks > 2147483647L) return AIEN_E_SHAPE;
    const bool vec = (V & 3) == 0 && (lda & 3) == 0 && (ldo & 3) == 0 && ((uintptr_t)a & 15) == 0 && ((uintptr_t)out & 15) == 0;
#define MD_LAUNCH(VEC, N)                                                                                                     \
    AIEN_DISPATCH_DTYPE(o_dt, TO, (launch_chain(map_difference_norm_kernel<TO, VEC, N>, dim3((unsigned)blocks), dim3(256), (size_t)0, stream, \
                                                a, lda, (TO*)out, ldo, T, H, per, V, lambda, eps, mult)))
    if (vec && V <= 128) MD_LAUNCH(4, 1);
    else if (vec) MD_LAUNCH(4, 2);
    else MD_LAUNCH(1, 8);
#undef MD_LAUNCH
    return launch_status();
}
