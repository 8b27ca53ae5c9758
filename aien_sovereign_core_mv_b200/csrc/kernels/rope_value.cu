// Bias, rotation of q and k and the cache write for attention whose values have a size of their own.
//
// q (nq heads of hd numbers), k (nkv heads of hd) and v (nv heads of hdv) are column blocks of one projection [T, ld], which
// may come as `nparts` float32 partial products [nparts][T][ld].  `bias` (float32, one number per column, or null) is added
// first.  The first `rot` dimensions of every q and k head turn by the token's angles, dimension i with dimension
// i + rot/2 (cos and sin float32 [T, rot/2]); the rest pass unchanged.  q leaves in the compute dtype, k and v go to the
// token's cache slot (slot < 0: nothing is written).  All of it float32.
//
// A thread takes VEC neighbouring columns, and with them their partners half a rotation further on, so every number is
// read once; the units of a step (rotated pairs, plain columns, values) are dealt out over the grid token by token.
#include "common.cuh"

namespace aien {

template <int VEC>
__device__ __forceinline__ void rv_load(const float* p, float* v) {
    if constexpr (VEC >= 4) {
#pragma unroll
        for (int i = 0; i < VEC; i += 4) {
            const float4 f = ld_act4(p + i);
            v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = ld_act(p + i);
    }
}
template <int VEC>
__device__ __forceinline__ void rv_load(const __nv_bfloat16* p, float* v) {
    if constexpr (VEC == 8) {
        const uint4 r = __ldcg(reinterpret_cast<const uint4*>(p));
        const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    } else if constexpr (VEC == 4) {
        const float4 f = ld_act4(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = ld_act(p + i);
    }
}
template <int VEC>
__device__ __forceinline__ void rv_store(float* p, const float* v) {
    if constexpr (VEC >= 4) {
#pragma unroll
        for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) p[i] = v[i];
    }
}
template <int VEC>
__device__ __forceinline__ void rv_store(__nv_bfloat16* p, const float* v) {
    if constexpr (VEC >= 4) {
        uint32_t w[VEC / 2];
#pragma unroll
        for (int i = 0; i < VEC / 2; ++i) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
            w[i] = *reinterpret_cast<const uint32_t*>(&b);
        }
        if constexpr (VEC == 8) *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
        else *reinterpret_cast<uint2*>(p) = make_uint2(w[0], w[1]);
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) p[i] = __float2bfloat16_rn(v[i]);
    }
}

// VEC columns at p, partial products added in order, bias added
template <int VEC, typename TI>
__device__ __forceinline__ void rv_fetch(const TI* p, int nparts, size_t part_stride, const float* bias, float* v) {
    rv_load<VEC>(p, v);
    for (int s = 1; s < nparts; ++s) {
        float w[VEC];
        rv_load<VEC>(p + (size_t)s * part_stride, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] += w[i];
    }
    if (bias != nullptr) {
        if constexpr (VEC >= 4) {
#pragma unroll
            for (int i = 0; i < VEC; i += 4) {
                const float4 b = __ldg(reinterpret_cast<const float4*>(bias + i));
                v[i] += b.x; v[i + 1] += b.y; v[i + 2] += b.z; v[i + 3] += b.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] += __ldg(bias + i);
        }
    }
}

template <int VEC, typename TI, typename TQ, typename TKV>
__global__ void __launch_bounds__(256)
rope_halves_value_write_kernel(const TI* __restrict__ proj, long ld, int nparts, size_t part_stride, const float* __restrict__ bias,
                               int q_off, int k_off, int v_off, int nq, int nkv, int hd, int nv, int hdv,
                               const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot,
                               const int* __restrict__ slot_map, TQ* __restrict__ q_out, long ldq,
                               TKV* __restrict__ k_cache, TKV* __restrict__ v_cache, int T) {
    griddep_launch();
    const int half = rot >> 1;
    const int pairs = half / VEC, per_head = (hd - half) / VEC, per_value = hdv / VEC;
    const int qk_units = (nq + nkv) * per_head, units = qk_units + nv * per_value;
    const int u = blockIdx.x * blockDim.x + threadIdx.x, t = blockIdx.y;
    if (u >= units) return;
    griddep_wait();
    const TI* row = proj + (size_t)t * ld;
    if (u >= qk_units) {                                       // a value: copied
        const int at = (u - qk_units) * VEC;
        const long slot = __ldcg(slot_map + t);
        if (slot < 0) return;
        float v[VEC];
        rv_fetch<VEC>(row + v_off + at, nparts, part_stride, bias != nullptr ? bias + v_off + at : nullptr, v);
        rv_store<VEC>(v_cache + (size_t)slot * nv * hdv + at, v);
        return;
    }
    const int head = u / per_head, w = u - head * per_head;
    const bool is_q = head < nq;
    const int hh = is_q ? head : head - nq;
    const long slot = is_q ? 0 : (long)__ldcg(slot_map + t);
    if (slot < 0) return;
    const int d = w < pairs ? w * VEC : rot + (w - pairs) * VEC;
    const int col = (is_q ? q_off : k_off) + hh * hd + d;
    float a[VEC];
    rv_fetch<VEC>(row + col, nparts, part_stride, bias != nullptr ? bias + col : nullptr, a);
    float b[VEC];
    if (w < pairs) {
        float c[VEC], s[VEC];
        rv_fetch<VEC>(row + col + half, nparts, part_stride, bias != nullptr ? bias + col + half : nullptr, b);
        rv_load<VEC>(cos_t + (size_t)t * half + d, c);
        rv_load<VEC>(sin_t + (size_t)t * half + d, s);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float x = a[i], y = b[i];
            a[i] = x * c[i] - y * s[i];
            b[i] = y * c[i] + x * s[i];
        }
    }
    if (is_q) {
        TQ* dst = q_out + (size_t)t * ldq + (size_t)hh * hd + d;
        rv_store<VEC>(dst, a);
        if (w < pairs) rv_store<VEC>(dst + half, b);
    } else {
        TKV* dst = k_cache + ((size_t)slot * nkv + hh) * hd + d;
        rv_store<VEC>(dst, a);
        if (w < pairs) rv_store<VEC>(dst + half, b);
    }
}

template <int VEC, typename TI, typename TQ, typename TKV>
static void launch_rope_value(const TI* proj, long ld, int nparts, size_t part_stride, const float* bias, int q_off, int k_off, int v_off,
                              int nq, int nkv, int hd, int nv, int hdv, const float* cos_t, const float* sin_t, int rot,
                              const int* slot_map, TQ* q_out, long ldq, TKV* k_cache, TKV* v_cache, int T, cudaStream_t stream) {
    const long units = ((long)(nq + nkv) * (hd - rot / 2) + (long)nv * hdv) / VEC;
    const long blocks = (units + 255) / 256, threads = ((units + blocks - 1) / blocks + 31) & ~31L;      // a token's units, evenly over its blocks
    launch_chain(rope_halves_value_write_kernel<VEC, TI, TQ, TKV>, dim3((unsigned)blocks, (unsigned)T), dim3((unsigned)threads), (size_t)0, stream,
                 proj, ld, nparts, part_stride, bias, q_off, k_off, v_off, nq, nkv, hd, nv, hdv, cos_t, sin_t, rot, slot_map, q_out, ldq,
                 k_cache, v_cache, T);
}

}  // namespace aien

using namespace aien;

// proj_dt: float32 or bfloat16 rows; nparts > 1: float32 partial products, part_stride numbers apart.  nv value heads.
AIEN_API int aien_rope_halves_value_write(const void* proj, int proj_dt, long ld, int nparts, size_t part_stride, const float* bias,
                                          int q_off, int k_off, int v_off, int nq, int nkv, int hd, int nv, int hdv,
                                          const float* cos_t, const float* sin_t, int rot, const int* slot_map, void* q_out, int q_dt,
                                          long ldq, void* k_cache, void* v_cache, int kv_dt, int T, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (nq <= 0 || nkv <= 0 || nv <= 0 || hd <= 0 || hdv <= 0 || rot < 0 || rot > hd || (rot & 1) ||
        (rot > 0 && (cos_t == nullptr || sin_t == nullptr)) || T > 65535 || nparts < 1 || (nparts > 1 && proj_dt != AIEN_DT_F32))
        return AIEN_E_SHAPE;
    // the widest vector that divides every size and whose accesses are aligned
    const long sizes = (long)hd | hdv | (rot / 2) | q_off | k_off | v_off | ld | ldq | (long)part_stride;
    const uintptr_t at = (uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)cos_t | (uintptr_t)sin_t | (uintptr_t)bias;
    const int vec = (at & 15) ? 1 : ((sizes & 7) == 0 ? 8 : ((sizes & 3) == 0 ? 4 : 1));
#define RV_LAUNCH(V)                                                                                                                   \
    AIEN_DISPATCH_DTYPE(proj_dt, TI, AIEN_DISPATCH_DTYPE(q_dt, TQ, AIEN_DISPATCH_DTYPE(kv_dt, TKV,                                       \
        (launch_rope_value<V, TI, TQ, TKV>((const TI*)proj, ld, nparts, part_stride, bias, q_off, k_off, v_off, nq, nkv, hd, nv, hdv,     \
                                           cos_t, sin_t, rot, slot_map, (TQ*)q_out, ldq, (TKV*)k_cache, (TKV*)v_cache, T, stream)))))
    if (vec == 8) RV_LAUNCH(8);
    else if (vec == 4) RV_LAUNCH(4);
    else RV_LAUNCH(1);
#undef RV_LAUNCH
    return launch_status();
}
