// Pending sums of several branches at once: what a layer whose sublayers read one norm leaves for the next norm.
//
// A term is a [T, H] tensor, or several of them to be added in order (float32 partial products, the parts of a routed
// feed-forward), optionally times sigmoid(gate[t]), one number per token.
//   sum_terms_rmsnorm   x = (x or, with `replace`, 0) + the terms + bias (one vector for every token), float32, in place;
//                       then, when asked, out = x / sqrt(mean(x^2) + eps) * w in the compute dtype
//   pass_rows           the rows of a product over [x; x0] with x = x + the terms: as float32 [x | x0], or in bfloat16 as
//                       [hi(x) | lo(x) | x0], hi the rounded value and lo the rounded rest, so that the product over the
//                       matching columns keeps 16 bits of the stream
#include "common.cuh"
#include <math.h>

namespace aien {

struct SumTerm { const void* p; int dt; int parts; size_t stride; const float* gate; long ldg; };
struct SumTerms { SumTerm t[3]; int n; };

__device__ __forceinline__ float term_gate(const SumTerm& a, size_t t) {
    return a.gate == nullptr ? 1.0f : 1.0f / (1.0f + expf(-a.gate[t * a.ldg]));
}

__device__ __forceinline__ float4 load4(const SumTerm& a, size_t at) {
    return a.dt == AIEN_DT_F32 ? ld_act4(reinterpret_cast<const float*>(a.p) + at) : ld_act4(reinterpret_cast<const __nv_bfloat16*>(a.p) + at);
}
// the loads of four parts in flight, then their sum in order
__device__ __forceinline__ float4 term_load4(const SumTerm& a, size_t at) {
    float4 s = load4(a, at);
    for (int p = 1; p < a.parts; p += 4) {
        float4 v[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = p + i < a.parts ? load4(a, (size_t)(p + i) * a.stride + at) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 4; ++i) { s.x += v[i].x; s.y += v[i].y; s.z += v[i].z; s.w += v[i].w; }
    }
    return s;
}
__device__ __forceinline__ float term_load(const SumTerm& a, size_t at) {
    float s = 0.f;
    for (int p = 0; p < a.parts; ++p) s += load_dyn(a.p, a.dt, (size_t)p * a.stride + at);
    return s;
}

template <typename TO> __device__ __forceinline__ void store4(TO* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}

// The row stays in registers between the sum and the norm: VPT groups of four numbers a thread.
template <typename TO, int VPT>
__global__ void __launch_bounds__(VPT == 8 ? 256 : 1024)
sum_terms_rmsnorm_vec_kernel(float* __restrict__ x, SumTerms a, const void* __restrict__ bias, int bdt, int replace,
                             const void* __restrict__ w, int wdt, float eps, TO* __restrict__ out, int H) {
    __shared__ float red[32];
    const size_t t = blockIdx.x, row = t * H;
    float g[3] = {1.f, 1.f, 1.f};
#pragma unroll
    for (int k = 0; k < 3; ++k) if (k < a.n) g[k] = term_gate(a.t[k], t);
    float4 v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = 4 * (threadIdx.x + i * blockDim.x);
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= H) continue;
        if (!replace) v[i] = ld_act4(x + row + c);
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            if (k < a.n) {
                const float4 d = term_load4(a.t[k], row + c);
                v[i].x = fmaf(g[k], d.x, v[i].x);
                v[i].y = fmaf(g[k], d.y, v[i].y);
                v[i].z = fmaf(g[k], d.z, v[i].z);
                v[i].w = fmaf(g[k], d.w, v[i].w);
            }
        }
        if (bias != nullptr) {
            v[i].x += load_dyn(bias, bdt, c);
            v[i].y += load_dyn(bias, bdt, c + 1);
            v[i].z += load_dyn(bias, bdt, c + 2);
            v[i].w += load_dyn(bias, bdt, c + 3);
        }
        if (a.n > 0 || bias != nullptr || replace) *reinterpret_cast<float4*>(x + row + c) = v[i];
        ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    if (out == nullptr) return;
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = 4 * (threadIdx.x + i * blockDim.x);
        if (c >= H) continue;
        store4<TO>(out + row + c, make_float4(v[i].x * r * load_dyn(w, wdt, c), v[i].y * r * load_dyn(w, wdt, c + 1),
                                              v[i].z * r * load_dyn(w, wdt, c + 2), v[i].w * r * load_dyn(w, wdt, c + 3)));
    }
}

template <typename TO>
__global__ void __launch_bounds__(256)
sum_terms_rmsnorm_kernel(float* __restrict__ x, SumTerms a, const void* __restrict__ bias, int bdt, int replace,
                         const void* __restrict__ w, int wdt, float eps, TO* __restrict__ out, int H) {
    __shared__ float red[32];
    const size_t t = blockIdx.x, row = t * H;
    float g[3] = {1.f, 1.f, 1.f};
#pragma unroll
    for (int k = 0; k < 3; ++k) if (k < a.n) g[k] = term_gate(a.t[k], t);
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += 256) {
        float v = replace ? 0.f : x[row + c];
#pragma unroll
        for (int k = 0; k < 3; ++k) if (k < a.n) v = fmaf(g[k], term_load(a.t[k], row + c), v);
        if (bias != nullptr) v += load_dyn(bias, bdt, c);
        x[row + c] = v;
        ss = fmaf(v, v, ss);
    }
    if (out == nullptr) return;
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += 256) out[row + c] = from_f<TO>(x[row + c] * r * load_dyn(w, wdt, c));
}

template <typename TO>
__global__ void __launch_bounds__(256)
pass_rows_kernel(const float* __restrict__ x, SumTerms a, const float* __restrict__ x0, TO* __restrict__ out, int H) {
    const size_t t = blockIdx.y, row = t * H;
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c >= H) return;
    float v = x[row + c];
#pragma unroll
    for (int k = 0; k < 3; ++k) if (k < a.n) v = fmaf(term_gate(a.t[k], t), term_load(a.t[k], row + c), v);
    if (sizeof(TO) == 4) {
        out[t * 2 * H + c] = from_f<TO>(v);
        out[t * 2 * H + H + c] = from_f<TO>(x0[row + c]);
    } else {
        const TO hi = from_f<TO>(v);
        out[t * 3 * H + c] = hi;
        out[t * 3 * H + H + c] = from_f<TO>(v - to_f(hi));
        out[t * 3 * H + 2 * H + c] = from_f<TO>(x0[row + c]);
    }
}

// The same, four numbers a thread.
template <typename TO>
__global__ void __launch_bounds__(256)
pass_rows_vec_kernel(const float* __restrict__ x, SumTerms a, const float* __restrict__ x0, TO* __restrict__ out, int H) {
    const size_t t = blockIdx.y, row = t * H;
    const int c = 4 * (blockIdx.x * 256 + threadIdx.x);
    if (c >= H) return;
    float4 v = ld_act4(x + row + c);
    const float4 e = ld_act4(x0 + row + c);
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        if (k < a.n) {
            const float g = term_gate(a.t[k], t);
            const float4 d = term_load4(a.t[k], row + c);
            v.x = fmaf(g, d.x, v.x);
            v.y = fmaf(g, d.y, v.y);
            v.z = fmaf(g, d.z, v.z);
            v.w = fmaf(g, d.w, v.w);
        }
    }
    if (sizeof(TO) == 4) {
        store4<TO>(out + t * 2 * H + c, v);
        store4<TO>(out + t * 2 * H + H + c, e);
    } else {
        store4<TO>(out + t * 3 * H + c, v);
        store4<TO>(out + t * 3 * H + H + c, make_float4(v.x - to_f(from_f<TO>(v.x)), v.y - to_f(from_f<TO>(v.y)), v.z - to_f(from_f<TO>(v.z)),
                                                        v.w - to_f(from_f<TO>(v.w))));
        store4<TO>(out + t * 3 * H + 2 * H + c, e);
    }
}

}  // namespace aien

using namespace aien;

#define TERM_ARGS(i) const void* p##i, int dt##i, int n##i, size_t st##i, const float* g##i, long lg##i
#define TERM_SET(i) SumTerm{p##i, dt##i, n##i, st##i, g##i, lg##i}

static bool terms_ok(const SumTerms& a, int H, bool* vec) {
    for (int k = 0; k < a.n; ++k) {
        const SumTerm& t = a.t[k];
        if (t.p == nullptr || t.parts <= 0 || (t.dt != AIEN_DT_F32 && t.dt != AIEN_DT_BF16)) return false;
        if ((uintptr_t)t.p & (t.dt == AIEN_DT_F32 ? 15 : 7)) *vec = false;
        if (t.stride & 3) *vec = false;
    }
    if (H & 3) *vec = false;
    return true;
}

// x float32 [T, H]; `terms` (0 to 3) of the term arguments are used, each dt / parts / distance between parts in elements / gate
// float32 (row distance ldg) or null; bias [H] in b_dt or null; replace != 0: x is overwritten; w [H] in w_dt; out [T, H] or null.
AIEN_API int aien_sum_terms_rmsnorm(float* x, int terms, TERM_ARGS(0), TERM_ARGS(1), TERM_ARGS(2), const void* bias, int b_dt, int replace,
                                    const void* w, int w_dt, float eps, void* out, int o_dt, int T, int H, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || terms < 0 || terms > 3) return AIEN_E_SHAPE;
    const SumTerms a{{TERM_SET(0), TERM_SET(1), TERM_SET(2)}, terms};
    bool vec = ((uintptr_t)x & 15) == 0 && ((uintptr_t)out & 15) == 0;
    if (!terms_ok(a, H, &vec)) return AIEN_E_SHAPE;
    // a step of few tokens has too few CTAs to hide a row's loads behind one another: wide CTAs then
    const int nv = H >> 2;
    int threads = (T <= 2 * 148) ? 1024 : 256;
    while (threads > 64 && threads / 2 >= nv) threads >>= 1;
    if (nv > 8 * 256) threads = 1024;
    if (nv > 4 * 1024) vec = false;
    const int per = vec ? (nv + threads - 1) / threads : 0;
#define ST_CASE(VP) AIEN_DISPATCH_DTYPE(o_dt, TO, (sum_terms_rmsnorm_vec_kernel<TO, VP><<<T, threads, 0, stream>>>(x, a, bias, b_dt, replace, w, w_dt, eps, (TO*)out, H)))
    if (!vec) AIEN_DISPATCH_DTYPE(o_dt, TO, (sum_terms_rmsnorm_kernel<TO><<<T, 256, 0, stream>>>(x, a, bias, b_dt, replace, w, w_dt, eps, (TO*)out, H)));
    else if (per <= 1) ST_CASE(1);
    else if (per <= 2) ST_CASE(2);
    else if (per <= 4) ST_CASE(4);
    else ST_CASE(8);
#undef ST_CASE
    return launch_status();
}

// out: bfloat16 [T, 3 * H] = [hi | lo | x0], or float32 [T, 2 * H] = [x | x0].
AIEN_API int aien_pass_rows(const float* x, int terms, TERM_ARGS(0), TERM_ARGS(1), TERM_ARGS(2), const float* x0, void* out, int o_dt, int T, int H,
                            cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || T > 65535 || terms < 0 || terms > 3 || x0 == nullptr) return AIEN_E_SHAPE;
    const SumTerms a{{TERM_SET(0), TERM_SET(1), TERM_SET(2)}, terms};
    bool vec = true;
    if (!terms_ok(a, H, &vec)) return AIEN_E_SHAPE;
    if (((uintptr_t)x | (uintptr_t)x0 | (uintptr_t)out) & 15) vec = false;
    if (vec) AIEN_DISPATCH_DTYPE(o_dt, TO, (pass_rows_vec_kernel<TO><<<dim3((H + 1023) / 1024, T), 256, 0, stream>>>(x, a, x0, (TO*)out, H)));
    else AIEN_DISPATCH_DTYPE(o_dt, TO, (pass_rows_kernel<TO><<<dim3((H + 255) / 256, T), 256, 0, stream>>>(x, a, x0, (TO*)out, H)));
    return launch_status();
}
