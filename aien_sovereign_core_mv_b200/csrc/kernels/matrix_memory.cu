// A matrix memory with exponential gates (the mLSTM recurrence).  Per head, with log gates i (input) and f (forget),
// a running maximum m that starts at 0, S [dim, vdim], n [dim]:
//     m_t = max(f + m_(t-1), i)      keep = exp(f - (m_t - m_(t-1)))      take = exp(i - m_t)
//     S_t = keep S_(t-1) + take k v^T      n_t = keep n_(t-1) + take k
//     o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + eps_den),      q already times dim^(-1/2)
// and then y = o / rms(o of the head) * w * sigmoid(g).  The log gates are i = cap tanh((z_i + b_i) / cap) and
// f = logsigmoid(cap tanh((z_f + b_f) / cap)).
//
// A slot holds S as [heads][dim][vdim], then n [heads][dim], then m [heads], float32.  The rules of a slot are those of
// every state group: the portion of request s is the tokens q_start[s] .. q_start[s+1], its slot slot_map[s]; a portion
// whose first token has position 0 starts from zeros.  Gates, m, keep, take, S, n, the products with them, the
// denominator and the norm are float32 in both engine precisions.
//
// Three forms:
//   token    every request brings one token: the state streams through once and the finished row y leaves;
//   walk     any sizes and dtypes: a state column's lanes walk the portion token by token (numerators and n . q leave,
//            a second kernel finishes the rows);
//   chunked  portions in bfloat16: chunks of 64 tokens side by side on the tensor cores (see below).
// m, and with it keep and take, is made once per step and head by the gate kernel ahead of the last two, so they are
// the same numbers whichever form follows.
#include "common.cuh"
#include <math.h>

namespace aien {

__device__ __forceinline__ float mm_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float mm_log_sigmoid(float v) { return fminf(v, 0.f) - log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float mm_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mm_forget_gate(float z, float cap) { return mm_log_sigmoid(cap * tanhf(z / cap)); }

struct MmSizes { int H, D, V; };
__device__ __forceinline__ size_t mm_n_off(MmSizes z) { return (size_t)z.H * z.D * z.V; }
__device__ __forceinline__ size_t mm_m_off(MmSizes z) { return mm_n_off(z) + (size_t)z.H * z.D; }

// ---------------------------------------------------------------- gates and the running maximum
// gates [T, 3 * H]: log keep = f - (m_t - m_(t-1)), then take = exp(i - m_t), then m_t.  One CTA per (request, head), 32 tokens a
// warp: the map of a run of tokens on m is m -> max(m + a, b), so the warps scan their own runs, the runs' maps follow one
// another from the state's m, and every token gets its m from its run's start.  The slot's m is rewritten at the end.
__global__ void __launch_bounds__(1024)
matrix_memory_gates_kernel(const float* __restrict__ z, long ldz, int i_off, int f_off, const float* __restrict__ bi,
                           const float* __restrict__ bf, float cap, float* __restrict__ state, size_t state_stride, size_t m_off,
                           const int* __restrict__ slot_map, const int* __restrict__ q_start, const int* __restrict__ positions,
                           float* __restrict__ gates, int H) {
    __shared__ float ra[32], rb[32];
    const int s = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int t0 = q_start[s], t1 = q_start[s + 1];
    if (t1 <= t0) return;
    float* ms = state + (size_t)slot_map[s] * state_stride + m_off + h;
    float m = positions[t0] == 0 ? 0.f : *ms;
    const float bih = bi[h], bfh = bf[h];
    for (int base = t0; base < t1; base += (int)blockDim.x) {
        const int t = base + (int)threadIdx.x;
        const bool in = t < t1;
        float li = -INFINITY, lf = 0.f;                     // beyond the portion's end: m stays
        if (in) {
            li = mm_input_gate(z[(size_t)t * ldz + i_off + h] + bih, cap);
            lf = mm_forget_gate(z[(size_t)t * ldz + f_off + h] + bfh, cap);
        }
        float a = lf, b = li;                               // this token's map, then the maps of the run up to this token
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, a, o), pb = __shfl_up_sync(0xffffffffu, b, o);
            if (lane >= o) { b = fmaxf(pb + a, b); a += pa; }
        }
        if (lane == 31) { ra[warp] = a; rb[warp] = b; }
        __syncthreads();
        float m_run = m;                                    // m before this warp's run, then after all runs
        float m_start = m;
        for (int w = 0; w < nwarps; ++w) {
            if (w == warp) m_start = m_run;
            m_run = fmaxf(m_run + ra[w], rb[w]);
        }
        const float mt = fmaxf(m_start + a, b);
        float mp = __shfl_up_sync(0xffffffffu, mt, 1);
        if (lane == 0) mp = m_start;
        if (in) {
            float* g = gates + (size_t)t * 3 * H + h;
            g[0] = lf - (mt - mp);          // exact to the last bit of lf while m only decays: m is far larger than lf
            g[H] = expf(li - mt);
            g[2 * H] = mt;
        }
        m = m_run;
        __syncthreads();
    }
    if (threadIdx.x == 0) *ms = m;
}

// ---------------------------------------------------------------- walk: token by token, any sizes
// 32 lanes share one column (head h, value column v; v = vdim is n, whose "value" is 1): lane ln keeps the rows
// d = ln * CH .. of the column in registers and the partial dot products with q meet by shuffles.
constexpr int MW_THREADS = 256;

template <typename TP, int CH, int U>
__global__ void __launch_bounds__(MW_THREADS)
matrix_memory_walk_kernel(const TP* __restrict__ proj, long ld, int q_off, int k_off, int v_off, float q_scale,
                          const float* __restrict__ gates, float* __restrict__ state, size_t state_stride,
                          const int* __restrict__ slot_map, const int* __restrict__ q_start, const int* __restrict__ positions,
                          float* __restrict__ num, float* __restrict__ nq, MmSizes z) {
    const int s = blockIdx.y, col = blockIdx.x * (MW_THREADS / 32) + (threadIdx.x >> 5), ln = threadIdx.x & 31;
    if (col >= z.H * (z.V + 1)) return;
    const int h = col / (z.V + 1), v = col % (z.V + 1), d0 = ln * CH;
    const bool norm_col = v == z.V;
    const int t0 = q_start[s], t1 = q_start[s + 1];
    if (t1 <= t0) return;
    const bool fresh = positions[t0] == 0;
    float* st = state + (size_t)slot_map[s] * state_stride +
                (norm_col ? mm_n_off(z) + (size_t)h * z.D : ((size_t)h * z.D) * z.V + v);
    const size_t rstride = norm_col ? 1 : z.V;
    float S[CH];
#pragma unroll
    for (int i = 0; i < CH; ++i) S[i] = (!fresh && d0 + i < z.D) ? st[(size_t)(d0 + i) * rstride] : 0.f;
    for (int t = t0; t < t1; t += U) {
        float keep[U], take[U], val[U], kk[U][CH], qq[U][CH];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int tt = t + u < t1 ? t + u : t1 - 1;
            const float* g = gates + (size_t)tt * 3 * z.H + h;
            const TP* row = proj + (size_t)tt * ld;
            keep[u] = g[0];
            take[u] = g[z.H];
            val[u] = norm_col ? 1.f : to_f(row[v_off + h * z.V + v]);
#pragma unroll
            for (int i = 0; i < CH; ++i) {
                const bool in = d0 + i < z.D;
                kk[u][i] = in ? to_f(row[k_off + h * z.D + d0 + i]) : 0.f;
                qq[u][i] = in ? to_f(row[q_off + h * z.D + d0 + i]) : 0.f;
            }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (t + u < t1) {
                const float e = expf(keep[u]), tv = take[u] * val[u];
                float y = 0.f;
#pragma unroll
                for (int i = 0; i < CH; ++i) {
                    S[i] = fmaf(e, S[i], kk[u][i] * tv);
                    y = fmaf(S[i], qq[u][i], y);
                }
                y = warp_sum(y) * q_scale;
                if (ln == 0) {
                    if (norm_col) nq[(size_t)(t + u) * z.H + h] = y;
                    else num[(size_t)(t + u) * z.H * z.V + h * z.V + v] = y;
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < CH; ++i) if (d0 + i < z.D) st[(size_t)(d0 + i) * rstride] = S[i];
}

// y = num / (max(|nq|, exp(-m)) + den_eps), divided by its own root mean square over the head, times w, times sigmoid(g).
// A warp per (token, head).
template <typename TG, typename TO>
__global__ void __launch_bounds__(256)
matrix_memory_finish_kernel(const float* __restrict__ num, const float* __restrict__ nq, const float* __restrict__ gates,
                            const TG* __restrict__ g, long ldg, const void* __restrict__ w, int wdt, float eps, float den_eps,
                            TO* __restrict__ out, long ldo, int T, int H, int V) {
    const long i = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (i >= (long)T * H) return;
    const int t = (int)(i / H), h = (int)(i % H);
    const float inv = 1.0f / (fmaxf(fabsf(nq[i]), expf(-gates[(size_t)t * 3 * H + 2 * H + h])) + den_eps);
    const float* o = num + (size_t)i * V;
    float ss = 0.f;
    for (int v = lane; v < V; v += 32) { const float x = o[v] * inv; ss = fmaf(x, x, ss); }
    const float r = inv / sqrtf(warp_sum(ss) / (float)V + eps);
    for (int v = lane; v < V; v += 32)
        out[(size_t)t * ldo + h * V + v] = from_f<TO>(o[v] * r * load_dyn(w, wdt, (size_t)h * V + v) * mm_sigmoid(to_f(g[(size_t)t * ldg + h * V + v])));
}

// ---------------------------------------------------------------- token: one token per request, everything in one pass
// A CTA per (head, request).  Thread (rg, c4) takes the rows d = rg, rg + RG, ... of four value columns: MT_ROWS rows in
// flight, updated, written back and added into the numerators; the row groups meet in shared memory.
constexpr int MT_THREADS = 512, MT_ROWS = 8;

template <typename TP, typename TO>
__global__ void __launch_bounds__(MT_THREADS)
matrix_memory_token_kernel(const TP* __restrict__ proj, long ld, int q_off, int k_off, int v_off, int g_off, float q_scale,
                           const float* __restrict__ z, long ldz, int i_off, int f_off, const float* __restrict__ bi,
                           const float* __restrict__ bf, float cap, float* __restrict__ state, size_t state_stride,
                           const int* __restrict__ slot_map, const int* __restrict__ q_start, const int* __restrict__ positions,
                           const void* __restrict__ w, int wdt, float eps, float den_eps, TO* __restrict__ out, long ldo, MmSizes sz) {
    extern __shared__ float sm[];
    __shared__ float red[32];
    const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, D = sz.D, V = sz.V;
    const int c4n = V >> 2, RG = MT_THREADS / c4n;
    float* part = sm;                        // [RG][V]
    float* qs = part + RG * V;               // [D]
    float* ks = qs + D;                      // [D]
    const int t = q_start[s];
    const bool fresh = positions[t] == 0;
    const TP* row = proj + (size_t)t * ld;
    float* slot = state + (size_t)slot_map[s] * state_stride;
    float* S = slot + (size_t)h * D * V;
    float* n = slot + mm_n_off(sz) + (size_t)h * D;
    float* ms = slot + mm_m_off(sz) + h;
    const int rg = tid / c4n, c4 = tid - rg * c4n;
    const bool works = rg < RG;
    float4 sv[MT_ROWS];
#pragma unroll
    for (int i = 0; i < MT_ROWS; ++i) {
        const int d = rg + i * RG;
        sv[i] = (works && !fresh && d < D) ? *reinterpret_cast<const float4*>(S + (size_t)d * V + 4 * c4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float m0 = fresh ? 0.f : *ms;
    const float li = mm_input_gate(z[(size_t)t * ldz + i_off + h] + bi[h], cap);
    const float lf = mm_forget_gate(z[(size_t)t * ldz + f_off + h] + bf[h], cap);
    const float m1 = fmaxf(lf + m0, li);
    const float keep = expf(lf - (m1 - m0)), take = expf(li - m1);
    float nqp = 0.f;
    for (int d = tid; d < D; d += MT_THREADS) {
        const float q = to_f(row[q_off + h * D + d]) * q_scale, k = to_f(row[k_off + h * D + d]) * take;
        qs[d] = q;
        ks[d] = k;
        const float nn = fmaf(keep, fresh ? 0.f : n[d], k);
        n[d] = nn;
        nqp = fmaf(nn, q, nqp);
    }
    const float nq = block_sum(nqp, red);    // its barriers also stand between the writes of qs, ks and their readers, and the reads of m and its write
    if (tid == 0) *ms = m1;
    if (works) {
        float vv[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) vv[j] = to_f(row[v_off + h * V + 4 * c4 + j]);
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int b = 0; b * MT_ROWS * RG < D; ++b) {
            const int db = rg + b * MT_ROWS * RG;
            if (b > 0) {
#pragma unroll
                for (int i = 0; i < MT_ROWS; ++i) {
                    const int d = db + i * RG;
                    sv[i] = (!fresh && d < D) ? *reinterpret_cast<const float4*>(S + (size_t)d * V + 4 * c4) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
            }
#pragma unroll
            for (int i = 0; i < MT_ROWS; ++i) {
                const int d = db + i * RG;
                if (d < D) {
                    const float k = ks[d], q = qs[d];
                    float4 x = sv[i];
                    x.x = fmaf(keep, x.x, k * vv[0]);
                    x.y = fmaf(keep, x.y, k * vv[1]);
                    x.z = fmaf(keep, x.z, k * vv[2]);
                    x.w = fmaf(keep, x.w, k * vv[3]);
                    *reinterpret_cast<float4*>(S + (size_t)d * V + 4 * c4) = x;
                    acc[0] = fmaf(x.x, q, acc[0]);
                    acc[1] = fmaf(x.y, q, acc[1]);
                    acc[2] = fmaf(x.z, q, acc[2]);
                    acc[3] = fmaf(x.w, q, acc[3]);
                }
            }
        }
        *reinterpret_cast<float4*>(part + (size_t)rg * V + 4 * c4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    }
    __syncthreads();
    const float inv = 1.0f / (fmaxf(fabsf(nq), expf(-m1)) + den_eps);
    float o = 0.f;
    if (tid < V) {                           // vdim <= MT_THREADS
        for (int r = 0; r < RG; ++r) o += part[(size_t)r * V + tid];
        o *= inv;
    }
    const float r = 1.0f / sqrtf(block_sum(o * o, red) / (float)V + eps);
    if (tid < V)
        out[(size_t)t * ldo + h * V + tid] =
            from_f<TO>(o * r * load_dyn(w, wdt, (size_t)h * V + tid) * mm_sigmoid(to_f(row[g_off + h * V + tid])));
}

}  // namespace aien

using namespace aien;

// gates float32 [T, 3 * H] for the T tokens of S requests; z float32 [T, ldz] with the gates' projections at i_off, f_off; bi, bf
// float32 [H]; the slot's m is at m_off.
AIEN_API int aien_matrix_memory_gates(const float* z, long ldz, int i_off, int f_off, const float* bi, const float* bf, float cap,
                                      float* state, size_t state_stride, size_t m_off, const int* slot_map, const int* q_start,
                                      const int* positions, float* gates, int T, int S, int H, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (H <= 0 || H > 65535 || !(cap > 0.f)) return AIEN_E_SHAPE;
    const int threads = T / S >= 512 ? 1024 : (T / S >= 128 ? 256 : 64);
    matrix_memory_gates_kernel<<<dim3(S, H), threads, 0, stream>>>(z, ldz, i_off, f_off, bi, bf, cap, state, state_stride, m_off, slot_map,
                                                                   q_start, positions, gates, H);
    return launch_status();
}

// proj [T, ld] in p_dt with q, k (H * D) and v (H * V) at their offsets; gates as above; num float32 [T, H * V], nq float32 [T, H].
AIEN_API int aien_matrix_memory_walk(const void* proj, int p_dt, long ld, int q_off, int k_off, int v_off, float q_scale,
                                     const float* gates, float* state, size_t state_stride, const int* slot_map, const int* q_start,
                                     const int* positions, float* num, float* nq, int S, int H, int D, int V, cudaStream_t stream) {
    if (S <= 0) return 0;
    if (H <= 0 || D <= 0 || V <= 0 || D > 512 || S > 65535) return AIEN_E_SHAPE;
    const MmSizes z{H, D, V};
    const dim3 grid((unsigned)(((long)H * (V + 1) + MW_THREADS / 32 - 1) / (MW_THREADS / 32)), S);
#define MW_CASE(CHV, UV)                                                                                                                  \
    AIEN_DISPATCH_DTYPE(p_dt, TP, (matrix_memory_walk_kernel<TP, CHV, UV><<<grid, MW_THREADS, 0, stream>>>(                                 \
        (const TP*)proj, ld, q_off, k_off, v_off, q_scale, gates, state, state_stride, slot_map, q_start, positions, num, nq, z)))
    if (D <= 32) MW_CASE(1, 4);
    else if (D <= 64) MW_CASE(2, 4);
    else if (D <= 128) MW_CASE(4, 4);
    else if (D <= 256) MW_CASE(8, 2);
    else MW_CASE(16, 1);
#undef MW_CASE
    return launch_status();
}

AIEN_API int aien_matrix_memory_finish(const float* num, const float* nq, const float* gates, const void* g, int g_dt, long ldg, const void* w,
                                       int w_dt, float eps, float den_eps, void* out, int o_dt, long ldo, int T, int H, int V, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || V <= 0) return AIEN_E_SHAPE;
    const unsigned blocks = (unsigned)(((long)T * H + 7) / 8);
    AIEN_DISPATCH_DTYPE(g_dt, TG, AIEN_DISPATCH_DTYPE(o_dt, TO,
        (matrix_memory_finish_kernel<TG, TO><<<blocks, 256, 0, stream>>>(num, nq, gates, (const TG*)g, ldg, w, w_dt, eps, den_eps, (TO*)out, ldo, T, H, V))));
    return launch_status();
}

AIEN_API int aien_matrix_memory_token_supports(int D, int V) { return D > 0 && D <= 1024 && V > 0 && (V & 3) == 0 && V <= MT_THREADS ? 1 : 0; }

// Every one of the S requests brings one token.  state 16-byte aligned, state_stride a multiple of 4.
AIEN_API int aien_matrix_memory_token(const void* proj, int p_dt, long ld, int q_off, int k_off, int v_off, int g_off, float q_scale,
                                      const float* z, long ldz, int i_off, int f_off, const float* bi, const float* bf, float cap,
                                      float* state, size_t state_stride, const int* slot_map, const int* q_start, const int* positions,
                                      const void* w, int w_dt, float eps, float den_eps, void* out, int o_dt, long ldo, int S, int H, int D, int V,
                                      cudaStream_t stream) {
    if (S <= 0) return 0;
    if (H <= 0 || S > 65535 || !(cap > 0.f) || !aien_matrix_memory_token_supports(D, V)) return AIEN_E_SHAPE;
    if (((uintptr_t)state & 15) || (state_stride & 3)) return AIEN_E_ALIGN;
    const MmSizes sz{H, D, V};
    const int RG = MT_THREADS / (V >> 2);
    const size_t smem = (size_t)(2 * D + RG * V) * sizeof(float);            // at most 8 KB + 8 KB
    const dim3 grid(H, S);
    AIEN_DISPATCH_DTYPE(p_dt, TP, AIEN_DISPATCH_DTYPE(o_dt, TO,
        (matrix_memory_token_kernel<TP, TO><<<grid, MT_THREADS, smem, stream>>>((const TP*)proj, ld, q_off, k_off, v_off, g_off, q_scale, z, ldz, i_off,
            f_off, bi, bf, cap, state, state_stride, slot_map, q_start, positions, w, w_dt, eps, den_eps, (TO*)out, ldo, sz))));
    return launch_status();
}
