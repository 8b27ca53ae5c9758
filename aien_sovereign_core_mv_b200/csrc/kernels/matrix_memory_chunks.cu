// The matrix memory (see matrix_memory.cu) for portions of prompts in bfloat16: chunks of 64 tokens side by side on the
// tensor cores.  With L_t the sum of log keep over the chunk's tokens up to t (from the gate kernel), the recurrence from
// the state (S, n) before a chunk is
//     S^T q_t = e^(L_t) (S^T q_t) + sum_{j <= t} A_tj v_j       n . q_t = e^(L_t) (n . q_t) + sum_{j <= t} A_tj
//     A_tj = (q_t . k_j) take_j e^(L_t - L_j)
// and the state after it e^(L_end) (S, n) + sum_j take_j e^(L_end - L_j) (k_j v_j^T, k_j).  Three launches:
//   1. every chunk's own contribution to the state, and its decay e^(L_end)           (chunks in parallel)
//   2. per request, over its chunks in order, the state before each chunk (in place)  (elements in parallel)
//   3. every chunk's outputs, with the denominator, the norm over the head, the weight and the gate
// q, k and v are bfloat16 (results of a product); everything else that enters the recurrence is float32, and a product of
// a float32 with a bfloat16 matrix runs as three bfloat16 products: the float32 value is cut into three bfloat16 numbers
// (8 bits each, so all 24), and the sums are float32.  L is summed in float64 and kept as two floats, so differences of
// neighbouring tokens stay exact to rounding however far the chunk has decayed.
//
// Between the launches a state lies in the order in which the third reads it: tiles of 16 rows (d) by 8 columns (v), in a
// tile four numbers per lane, lane = (v % 8) * 4 + (d % 8) / 2, number = d % 2 + 2 * (d % 16 / 8): the B fragment of
// mma.m16n8k16 as one float4.  Behind the D * V numbers of S come the D numbers of n.
#include "common.cuh"
#include <math.h>

namespace aien {

constexpr int MC = 64, MC_THREADS = 256;

__device__ __forceinline__ void mc_cp_async16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void mc_cp_async_wait() {
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
}
__device__ __forceinline__ void mc_ldmatrix_x4(uint32_t addr, uint32_t r[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mc_ldmatrix_x4_trans(uint32_t addr, uint32_t r[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mc_mma(float c[4], const uint32_t a[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t mc_pack(__nv_bfloat16 lo, __nv_bfloat16 hi) {
    __nv_bfloat162 p = __halves2bfloat162(lo, hi);
    return *reinterpret_cast<uint32_t*>(&p);
}
// x and y, each as the sum of three bfloat16 numbers, packed pairwise
__device__ __forceinline__ void mc_split2(float x, float y, uint32_t p[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        const __nv_bfloat16 a = __float2bfloat16_rn(x), b = __float2bfloat16_rn(y);
        p[i] = mc_pack(a, b);
        x -= __bfloat162float(a);
        y -= __bfloat162float(b);
    }
}

// Chunk number c of the step: its request, first token, tokens, and its number inside the portion.
__device__ __forceinline__ bool mc_locate(const int* __restrict__ q_start, int S, int c, int& s, int& t0, int& n, int& k) {
    int acc = 0;
    for (int i = 0; i < S; ++i) {
        const int len = q_start[i + 1] - q_start[i], nch = (len + MC - 1) / MC;
        if (c < acc + nch) {
            s = i;
            k = c - acc;
            t0 = q_start[i] + k * MC;
            n = min(MC, len - k * MC);
            return true;
        }
        acc += nch;
    }
    return false;
}

// One warp: L of the chunk's tokens as two floats each (tokens beyond n repeat the last one's).
__device__ __forceinline__ void mc_log_sums(const float* __restrict__ gates, int H, int h, int t0, int n, float* Lhi, float* Llo) {
    const int lane = threadIdx.x & 31, j = 2 * lane;
    const double a = j < n ? (double)gates[(size_t)(t0 + j) * 3 * H + h] : 0.0;
    const double b = j + 1 < n ? (double)gates[(size_t)(t0 + j + 1) * 3 * H + h] : 0.0;
    double run = a + b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
    }
    const double l0 = run - b, l1 = run;
    Lhi[j] = (float)l0;
    Llo[j] = (float)(l0 - (double)(float)l0);
    Lhi[j + 1] = (float)l1;
    Llo[j + 1] = (float)(l1 - (double)(float)l1);
}

// 64 rows of `cols` bfloat16 numbers into shared memory with row stride cols + 8; rows from n on are zeros.
__device__ __forceinline__ void mc_load_rows(uint32_t dst, const __nv_bfloat16* __restrict__ src, long ld, int cols, int n) {
    const int ch = cols >> 3;
    for (int idx = threadIdx.x; idx < MC * ch; idx += MC_THREADS) {
        const int r = idx / ch, c = idx - r * ch;
        mc_cp_async16(dst + (uint32_t)(r * (cols + 8) + c * 8) * 2, src + (size_t)(r < n ? r : 0) * ld + c * 8, r < n);
    }
}

// ---------------------------------------------------------------- 1: a chunk's own contribution to the state
// U^T = (w v)^T k with w_j = take_j e^(L_end - L_j): rows are value columns, so that an accumulator's two neighbouring
// tiles of eight k columns are one float4 of the state's order.
__global__ void __launch_bounds__(MC_THREADS)
mm_chunk_state_kernel(const __nv_bfloat16* __restrict__ proj, long ld, int k_off, int v_off, const float* __restrict__ gates,
                      const int* __restrict__ q_start, int S, float* __restrict__ U, float* __restrict__ decay, int H, int D, int V) {
    extern __shared__ __align__(16) uint8_t mc_smem[];
    __shared__ float Lhi[MC], Llo[MC], w[MC];
    int s, t0, n, kc;
    const int c = blockIdx.x, h = blockIdx.y;
    if (!mc_locate(q_start, S, c, s, t0, n, kc)) return;
    const int KSTR = D + 8, VSTR = V + 8;
    __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(mc_smem);              // [64][KSTR]
    __nv_bfloat16* Vs = Ks + MC * KSTR;                                         // three planes of [64][VSTR]
    const uint32_t Ks_u = (uint32_t)__cvta_generic_to_shared(Ks), Vs_u = (uint32_t)__cvta_generic_to_shared(Vs);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    mc_load_rows(Ks_u, proj + (size_t)t0 * ld + k_off + (size_t)h * D, ld, D, n);
    if (warp == 0) {
        mc_log_sums(gates, H, h, t0, n, Lhi, Llo);
        __syncwarp();
        const float eh = Lhi[MC - 1], el = Llo[MC - 1];
        for (int j = lane; j < MC; j += 32)
            w[j] = j < n ? gates[(size_t)(t0 + j) * 3 * H + H + h] * expf((eh - Lhi[j]) + (el - Llo[j])) : 0.f;
        if (lane == 0) decay[(size_t)c * H + h] = expf(eh + el);
    }
    __syncthreads();
    const int vch = V >> 3;
    for (int idx = tid; idx < MC * vch; idx += MC_THREADS) {
        const int j = idx / vch, v8 = (idx - j * vch) * 8;
        uint4 raw = make_uint4(0u, 0u, 0u, 0u);
        if (j < n) raw = *reinterpret_cast<const uint4*>(proj + (size_t)(t0 + j) * ld + v_off + (size_t)h * V + v8);
        const __nv_bfloat162* vp = reinterpret_cast<const __nv_bfloat162*>(&raw);
        uint32_t pl[3][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(vp[i]);
            uint32_t p[3];
            mc_split2(f.x * w[j], f.y * w[j], p);
            pl[0][i] = p[0]; pl[1][i] = p[1]; pl[2][i] = p[2];
        }
#pragma unroll
        for (int i = 0; i < 3; ++i)
            *reinterpret_cast<uint4*>(Vs + (size_t)i * MC * VSTR + j * VSTR + v8) = make_uint4(pl[i][0], pl[i][1], pl[i][2], pl[i][3]);
    }
    mc_cp_async_wait();
    __syncthreads();
    float* u = U + ((size_t)c * H + h) * ((size_t)D * V + D);
    const int dgroups = (D + 63) >> 6, items = (V >> 4) * dgroups, mi = lane >> 3, r8 = lane & 7;
    for (int it = warp; it < items; it += MC_THREADS / 32) {
        const int vt = it / dgroups, d0 = (it % dgroups) * 64, pairs = min(4, (D - d0) >> 4);
        float acc[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < MC / 16; ++ks) {
            if (ks * 16 >= n) break;                                            // uniform: the rest of the rows are zeros
            uint32_t a[3][4];
#pragma unroll
            for (int p = 0; p < 3; ++p)
                mc_ldmatrix_x4_trans(Vs_u + (uint32_t)(p * MC * VSTR + (ks * 16 + (mi >> 1) * 8 + r8) * VSTR + vt * 16 + (mi & 1) * 8) * 2, a[p]);
#pragma unroll
            for (int p = 0; p < 4; ++p) {
                if (p < pairs) {
                    uint32_t b[4];
                    mc_ldmatrix_x4_trans(Ks_u + (uint32_t)((ks * 16 + (lane & 15)) * KSTR + d0 + p * 16 + (lane >> 4) * 8) * 2, b);
#pragma unroll
                    for (int q = 2; q >= 0; --q) {
                        mc_mma(acc[2 * p], a[q], b[0], b[1]);
                        mc_mma(acc[2 * p + 1], a[q], b[2], b[3]);
                    }
                }
            }
        }
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            if (p < pairs) {
                const size_t tile = (size_t)((d0 >> 4) + p) * (V >> 3) + 2 * vt;
                *reinterpret_cast<float4*>(u + (tile * 32 + lane) * 4) = make_float4(acc[2 * p][0], acc[2 * p][1], acc[2 * p + 1][0], acc[2 * p + 1][1]);
                *reinterpret_cast<float4*>(u + ((tile + 1) * 32 + lane) * 4) = make_float4(acc[2 * p][2], acc[2 * p][3], acc[2 * p + 1][2], acc[2 * p + 1][3]);
            }
        }
    }
    for (int d = tid; d < D; d += MC_THREADS) {
        float sum = 0.f;
        for (int j = 0; j < n; ++j) sum = fmaf(w[j], __bfloat162float(Ks[j * KSTR + d]), sum);
        u[(size_t)D * V + d] = sum;
    }
}

// ---------------------------------------------------------------- 2: the states before the chunks
// A thread carries four numbers of the state over the request's chunks; the slot keeps S as [dim][vdim].
__global__ void __launch_bounds__(256)
mm_state_scan_kernel(float* __restrict__ U, const float* __restrict__ decay, float* __restrict__ state, size_t state_stride,
                     const int* __restrict__ slot_map, const int* __restrict__ q_start, const int* __restrict__ positions, int H, int D, int V) {
    const int s = blockIdx.z, h = blockIdx.y;
    const int DV = D * V, E = DV + D, e = 4 * (blockIdx.x * 256 + threadIdx.x);
    if (e >= E) return;
    int base = 0;
    for (int r = 0; r < s; ++r) base += (q_start[r + 1] - q_start[r] + MC - 1) / MC;
    const int t0 = q_start[s], len = q_start[s + 1] - t0;
    if (len <= 0) return;
    float* slot = state + (size_t)slot_map[s] * state_stride;
    float* at[4];
    if (e < DV) {
        const int tile = e >> 7, lane = (e & 127) >> 2, vb = V >> 3;
        const int d = (tile / vb) * 16 + 2 * (lane & 3), v = (tile % vb) * 8 + (lane >> 2);
        float* p = slot + ((size_t)h * D + d) * V + v;
        at[0] = p;
        at[1] = p + V;
        at[2] = p + 8 * (size_t)V;
        at[3] = p + 9 * (size_t)V;
    } else {
        float* p = slot + (size_t)H * DV + (size_t)h * D + (e - DV);
#pragma unroll
        for (int i = 0; i < 4; ++i) at[i] = p + i;
    }
    float4 sv = make_float4(0.f, 0.f, 0.f, 0.f);
    if (positions[t0] != 0) sv = make_float4(*at[0], *at[1], *at[2], *at[3]);
    const int nch = (len + MC - 1) / MC;
    const size_t cstride = (size_t)H * E;
    float* u0 = U + ((size_t)base * H + h) * E + e;
    constexpr int AHEAD = 8;                                                    // chunks whose loads are in flight
    for (int k0 = 0; k0 < nch; k0 += AHEAD) {
        float4 uv[AHEAD];
        float dk[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const bool in = k0 + i < nch;
            uv[i] = in ? __ldcg(reinterpret_cast<const float4*>(u0 + (size_t)(k0 + i) * cstride)) : make_float4(0.f, 0.f, 0.f, 0.f);
            dk[i] = in ? decay[(size_t)(base + k0 + i) * H + h] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (k0 + i < nch) {
                *reinterpret_cast<float4*>(u0 + (size_t)(k0 + i) * cstride) = sv;
                sv.x = fmaf(dk[i], sv.x, uv[i].x);
                sv.y = fmaf(dk[i], sv.y, uv[i].y);
                sv.z = fmaf(dk[i], sv.z, uv[i].z);
                sv.w = fmaf(dk[i], sv.w, uv[i].w);
            }
        }
    }
    *at[0] = sv.x;
    *at[1] = sv.y;
    *at[2] = sv.z;
    *at[3] = sv.w;
}

// ---------------------------------------------------------------- 3: the outputs
// Eight warps: warp & 3 is a slab of 16 tokens, warp >> 2 a half of the value columns (in pairs of 8-column tiles; both
// warps of a slab make the slab's scores).  PAIRS: pairs of tiles a warp holds at most.
template <int PAIRS>
__global__ void __launch_bounds__(MC_THREADS, PAIRS <= 4 ? 2 : 1)
mm_chunk_output_kernel(const __nv_bfloat16* __restrict__ proj, long ld, int q_off, int k_off, int v_off, int g_off, float q_scale,
                       const float* __restrict__ gates, const int* __restrict__ q_start, const int* __restrict__ positions, int S,
                       const float* __restrict__ P, const void* __restrict__ w, int wdt, float eps, float den_eps,
                       __nv_bfloat16* __restrict__ out, long ldo, int H, int D, int V) {
    extern __shared__ __align__(16) uint8_t mc_smem[];
    __shared__ float Lhi[MC], Llo[MC], take[MC], nq_before[MC], ssq[2][MC];
    int s, t0, n, kc;
    const int c = blockIdx.x, h = blockIdx.y;
    if (!mc_locate(q_start, S, c, s, t0, n, kc)) return;
    const int STR = D + 8, VSTR = V + 8;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(mc_smem);              // [64][STR]
    __nv_bfloat16* Ks = Qs + MC * STR;                                          // [64][STR]
    __nv_bfloat16* Vs = Ks + MC * STR;                                          // [64][VSTR]
    const uint32_t Qs_u = (uint32_t)__cvta_generic_to_shared(Qs), Ks_u = (uint32_t)__cvta_generic_to_shared(Ks);
    const uint32_t Vs_u = (uint32_t)__cvta_generic_to_shared(Vs);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const __nv_bfloat16* rows = proj + (size_t)t0 * ld;
    mc_load_rows(Qs_u, rows + q_off + (size_t)h * D, ld, D, n);
    mc_load_rows(Ks_u, rows + k_off + (size_t)h * D, ld, D, n);
    mc_load_rows(Vs_u, rows + v_off + (size_t)h * V, ld, V, n);
    if (warp == 0) mc_log_sums(gates, H, h, t0, n, Lhi, Llo);
    for (int j = tid; j < MC; j += MC_THREADS) take[j] = j < n ? gates[(size_t)(t0 + j) * 3 * H + H + h] : 0.f;
    const bool from_zero = kc == 0 && positions[t0] == 0;                       // the state before the chunk is zero
    const float* Pc = P + ((size_t)c * H + h) * ((size_t)D * V + D);
    mc_cp_async_wait();
    __syncthreads();
    {
        // n . q of the state before the chunk: four threads a token
        const int i = tid >> 2, q4 = tid & 3;
        float sum = 0.f;
        if (!from_zero) {
            const float* np = Pc + (size_t)D * V;
            for (int d = 2 * q4; d < D; d += 8) {
                const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Qs + i * STR + d));
                const float2 nn = *reinterpret_cast<const float2*>(np + d);
                sum = fmaf(q.x, nn.x, sum);
                sum = fmaf(q.y, nn.y, sum);
            }
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if (q4 == 0) nq_before[i] = sum;
    }
    __syncthreads();
    const int slab = warp & 3, half = warp >> 2, g = lane >> 2, cc = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const int i0 = slab * 16 + g, i1 = i0 + 8;
    const bool active = slab * 16 < n;
    const int all_pairs = V >> 4, first_pair = half == 0 ? 0 : (all_pairs + 1) >> 1;
    const int my_pairs = half == 0 ? (all_pairs + 1) >> 1 : all_pairs >> 1;
    float o[2 * PAIRS][4];
#pragma unroll
    for (int i = 0; i < 2 * PAIRS; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float nq0 = 0.f, nq1 = 0.f;
    if (active) {
        const uint32_t q_frag = Qs_u + (uint32_t)((slab * 16 + (mi & 1) * 8 + r8) * STR + (mi >> 1) * 8) * 2;
        // what the state before the chunk gives
        if (!from_zero) {
            const int vb = V >> 3;
            for (int kk = 0; kk < (D >> 4); ++kk) {
                uint32_t a[4];
                mc_ldmatrix_x4(q_frag + kk * 32, a);
                const float4* tiles = reinterpret_cast<const float4*>(Pc) + ((size_t)kk * vb + 2 * first_pair) * 32 + lane;
#pragma unroll
                for (int b = 0; b < 2 * PAIRS; b += 4) {                        // four tiles' loads in flight
                    float4 f[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        f[i] = b + i < 2 * my_pairs ? __ldg(tiles + (b + i) * 32) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (b + i < 2 * my_pairs) {
                            uint32_t p0[3], p1[3];
                            mc_split2(f[i].x, f[i].y, p0);
                            mc_split2(f[i].z, f[i].w, p1);
#pragma unroll
                            for (int q = 2; q >= 0; --q) mc_mma(o[b + i], a, p0[q], p1[q]);
                        }
                    }
                }
            }
        }
        const float e0 = expf(Lhi[i0] + Llo[i0]) * q_scale, e1 = expf(Lhi[i1] + Llo[i1]) * q_scale;
#pragma unroll
        for (int i = 0; i < 2 * PAIRS; ++i) { o[i][0] *= e0; o[i][1] *= e0; o[i][2] *= e1; o[i][3] *= e1; }
        nq0 = e0 * nq_before[i0];
        nq1 = e1 * nq_before[i1];
        // the slab's scores against the chunk's tokens up to its own last one
        float sc[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
        for (int kk = 0; kk < (D >> 4); ++kk) {
            uint32_t a[4];
            mc_ldmatrix_x4(q_frag + kk * 32, a);
#pragma unroll
            for (int jp = 0; jp < 4; ++jp) {
                if (jp <= slab) {
                    uint32_t b[4];
                    mc_ldmatrix_x4(Ks_u + (uint32_t)((jp * 16 + (mi >> 1) * 8 + r8) * STR + kk * 16 + (mi & 1) * 8) * 2, b);
                    mc_mma(sc[2 * jp], a, b[0], b[1]);
                    mc_mma(sc[2 * jp + 1], a, b[2], b[3]);
                }
            }
        }
        float rs0 = 0.f, rs1 = 0.f;
        const float h0 = Lhi[i0], l0 = Llo[i0], h1 = Lhi[i1], l1 = Llo[i1];
#pragma unroll
        for (int jt = 0; jt < 8; ++jt) {
            if ((jt >> 1) <= slab) {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = jt * 8 + 2 * cc + e;
                    const float tk = take[j] * q_scale, lh = Lhi[j], ll = Llo[j];
                    sc[jt][e] = j <= i0 ? sc[jt][e] * (tk * expf((h0 - lh) + (l0 - ll))) : 0.f;
                    sc[jt][2 + e] = j <= i1 ? sc[jt][2 + e] * (tk * expf((h1 - lh) + (l1 - ll))) : 0.f;
                    rs0 += sc[jt][e];
                    rs1 += sc[jt][2 + e];
                }
            }
        }
        rs0 += __shfl_xor_sync(0xffffffffu, rs0, 1); rs0 += __shfl_xor_sync(0xffffffffu, rs0, 2);
        rs1 += __shfl_xor_sync(0xffffffffu, rs1, 1); rs1 += __shfl_xor_sync(0xffffffffu, rs1, 2);
        nq0 += rs0;
        nq1 += rs1;
        // the scores times the chunk's values
#pragma unroll
        for (int jp = 0; jp < 4; ++jp) {
            if (jp <= slab) {
                uint32_t a[3][4], p[3];
                mc_split2(sc[2 * jp][0], sc[2 * jp][1], p);
                a[0][0] = p[0]; a[1][0] = p[1]; a[2][0] = p[2];
                mc_split2(sc[2 * jp][2], sc[2 * jp][3], p);
                a[0][1] = p[0]; a[1][1] = p[1]; a[2][1] = p[2];
                mc_split2(sc[2 * jp + 1][0], sc[2 * jp + 1][1], p);
                a[0][2] = p[0]; a[1][2] = p[1]; a[2][2] = p[2];
                mc_split2(sc[2 * jp + 1][2], sc[2 * jp + 1][3], p);
                a[0][3] = p[0]; a[1][3] = p[1]; a[2][3] = p[2];
#pragma unroll
                for (int vp = 0; vp < PAIRS; ++vp) {
                    if (vp < my_pairs) {
                        uint32_t b[4];
                        mc_ldmatrix_x4_trans(Vs_u + (uint32_t)((jp * 16 + (lane & 15)) * VSTR + (first_pair + vp) * 16 + (lane >> 4) * 8) * 2, b);
#pragma unroll
                        for (int q = 2; q >= 0; --q) {
                            mc_mma(o[2 * vp], a[q], b[0], b[1]);
                            mc_mma(o[2 * vp + 1], a[q], b[2], b[3]);
                        }
                    }
                }
            }
        }
        // denominators, and this half's sums of squares
        const float m0 = i0 < n ? gates[(size_t)(t0 + i0) * 3 * H + 2 * H + h] : 0.f, m1 = i1 < n ? gates[(size_t)(t0 + i1) * 3 * H + 2 * H + h] : 0.f;
        const float d0 = 1.0f / (fmaxf(fabsf(nq0), expf(-m0)) + den_eps), d1 = 1.0f / (fmaxf(fabsf(nq1), expf(-m1)) + den_eps);
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int i = 0; i < 2 * PAIRS; ++i) {
            o[i][0] *= d0; o[i][1] *= d0; o[i][2] *= d1; o[i][3] *= d1;
            s0 += o[i][0] * o[i][0] + o[i][1] * o[i][1];
            s1 += o[i][2] * o[i][2] + o[i][3] * o[i][3];
        }
        s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
        s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
        if (cc == 0) {
            ssq[half][i0] = s0;
            ssq[half][i1] = s1;
        }
    }
    __syncthreads();
    if (!active) return;
    const float r0 = 1.0f / sqrtf((ssq[0][i0] + ssq[1][i0]) / (float)V + eps), r1 = 1.0f / sqrtf((ssq[0][i1] + ssq[1][i1]) / (float)V + eps);
#pragma unroll
    for (int i = 0; i < 2 * PAIRS; ++i) {
        if (i < 2 * my_pairs) {
            const int v = first_pair * 16 + i * 8 + 2 * cc;
            const size_t at = (size_t)h * V + v;
            const float w0 = load_dyn(w, wdt, at), w1 = load_dyn(w, wdt, at + 1);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int row = e == 0 ? i0 : i1;
                if (row < n) {
                    const float2 gg = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rows + (size_t)row * ld + g_off + at));
                    const float r = e == 0 ? r0 : r1;
                    const float y0 = o[i][2 * e] * r * w0 / (1.0f + expf(-gg.x)), y1 = o[i][2 * e + 1] * r * w1 / (1.0f + expf(-gg.y));
                    *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(t0 + row) * ldo + at) = __floats2bfloat162_rn(y0, y1);
                }
            }
        }
    }
}

}  // namespace aien

using namespace aien;

AIEN_API int aien_matrix_memory_chunks_supports(int D, int V) {
    return D > 0 && D <= 256 && (D & 15) == 0 && V > 0 && V <= 256 && (V & 15) == 0 ? 1 : 0;
}

// proj bfloat16 [T, ld] with q, k (H * D), v, g (H * V) at their offsets, all 16-byte aligned; gates from aien_matrix_memory_gates;
// scratch float32, 16-byte aligned: (T / 64 + S) * H * (D * V + D + 1) numbers; out bfloat16 [T, ldo].
AIEN_API int aien_matrix_memory_chunked(const void* proj, long ld, int q_off, int k_off, int v_off, int g_off, float q_scale, const float* gates,
                                        float* state, size_t state_stride, const int* slot_map, const int* q_start, const int* positions,
                                        const void* w, int w_dt, float eps, float den_eps, void* out, long ldo, float* scratch, int T, int S,
                                        int H, int D, int V, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (H <= 0 || H > 65535 || S > 65535 || scratch == nullptr || !aien_matrix_memory_chunks_supports(D, V)) return AIEN_E_SHAPE;
    if (((uintptr_t)proj & 15) || (ld & 7) || ((q_off | k_off | v_off | g_off) & 7) || ((uintptr_t)scratch & 15) || ((uintptr_t)out & 3) || (ldo & 1)) return AIEN_E_ALIGN;
    const int NC = T / MC + S, E = D * V + D;
    float* U = scratch;
    float* decay = scratch + (size_t)NC * H * E;
    const __nv_bfloat16* p = (const __nv_bfloat16*)proj;
    const size_t smem1 = (size_t)MC * (D + 8) * 2 + (size_t)3 * MC * (V + 8) * 2, smem3 = (size_t)2 * MC * (D + 8) * 2 + (size_t)MC * (V + 8) * 2;
    if (cudaFuncSetAttribute(mm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1) != cudaSuccess) return AIEN_E_STATE;
    mm_chunk_state_kernel<<<dim3(NC, H), MC_THREADS, smem1, stream>>>(p, ld, k_off, v_off, gates, q_start, S, U, decay, H, D, V);
    mm_state_scan_kernel<<<dim3((E / 4 + 255) / 256, H, S), 256, 0, stream>>>(U, decay, state, state_stride, slot_map, q_start, positions, H, D, V);
#define MC_CASE(PV)                                                                                                                        \
    do {                                                                                                                                   \
        auto kern = mm_chunk_output_kernel<PV>;                                                                                            \
        if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3) != cudaSuccess) return AIEN_E_STATE;        \
        kern<<<dim3(NC, H), MC_THREADS, smem3, stream>>>(p, ld, q_off, k_off, v_off, g_off, q_scale, gates, q_start, positions, S, U, w, w_dt, \
                                                         eps, den_eps, (__nv_bfloat16*)out, ldo, H, D, V);                                 \
    } while (0)
    if (V <= 64) MC_CASE(2);
    else if (V <= 128) MC_CASE(4);
    else MC_CASE(8);
#undef MC_CASE
    return launch_status();
}
