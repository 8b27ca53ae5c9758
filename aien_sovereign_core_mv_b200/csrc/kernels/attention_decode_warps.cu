// Decode attention over the paged bfloat16 cache, a warp at a time: every warp walks tiles of 16 keys of its own with its own
// ring of shared memory and its own online softmax, so that nothing in the loop waits for another warp.
//
// For attention whose values have a size of their own, with an optional window or chunk mask, an optional cap on the score,
// and one or several attention maps over the same values: `maps` neighbouring key heads share a value head.  A value head
// with all its maps and query heads is one unit of work.  The maps' keys lie side by side in the cache, so a unit's key row is
// maps * hd numbers, and a query row holds its head's numbers in its own map's columns and zeros in the others: the maps are
// one score product S[16 heads x 16 keys] with keys and values fetched once for all of them.
//
// A CTA of four warps serves (range of tiles, value head, token); the ranges of a token are made so that the launch fills the
// GPU.  Per tile: cp.async brings the rows of K and V through the block table two or three tiles ahead (the table's entry one
// tile before that), m16n8k16 products with the query rows as A and the keys as B (ldmatrix), masks and softmax in float32 in
// log2 units, the probabilities go from accumulator to A fragment in registers, m16n8k16 products with V (transposing
// ldmatrix).  The running reference of the exponentials follows a row's maximum only when that has grown by more than 8
// (log2), so the sums are rescaled rarely.  At the end the warps' sums meet in shared memory; with several ranges the CTA that
// finishes last for a (token, value head) adds the ranges up in their order.
//
// With `diff` the two maps of a head (maps == 2) are combined before anything is written: o = a1 - lambda * a2, divided by
// sqrt(mean(o^2) + eps), times mult, per query head, in float32.
#include "common.cuh"
#include <math.h>

namespace aien {

constexpr int DW_WARPS = 4, DW_KEYS = 16, DW_MAX_SPLITS = 64;
constexpr int DW_RING_BYTES = 108 * 1024;

__device__ __forceinline__ void dw_cp16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void dw_ldsm4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dw_ldsm4t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dw_mma(float c[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t dw_pack(float lo, float hi) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&p);
}
__device__ __forceinline__ float dw_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// bytes between rows of KS 16-number (or DT 8-number) steps: an odd number of 16-byte pieces, so that eight rows of one piece
// column fall on different banks
__host__ __device__ constexpr int dw_row_bytes(int pieces) { return 16 * (pieces | 1); }

struct DwArgs {
    const __nv_bfloat16* q;
    long q_stride;
    const __nv_bfloat16 *k, *v;
    const int* block_table;
    int max_blocks;
    const int *seq_of_token, *positions, *token_list;
    void* out;
    long out_stride;
    int out_f32;
    float* part;                 // [T * nv * splits][heads * hdv + 2 * heads, rounded up to 4]: the sums, then per head the reference and the weight sum
    int* counters;               // [T * nv]: zero before and after
    int nv, maps, G, hd, hdv, page_size, window, chunk;
    float scale_log2e, cap_in, cap_l2;          // cap_in > 0: score = cap_l2 * tanh(dot * cap_in), in log2 units
    int splits;
    int diff;
    float lambda, eps, mult;
};

// KS: k16 steps of a key row (maps * hd, filled up with zeros); DT: n8 tiles of a value row (hdv, filled up)
template <int KS, int DT, int STAGES>
__global__ void __launch_bounds__(DW_WARPS * 32, 2)
paged_decode_warps_kernel(const DwArgs a) {
    constexpr int KROW = dw_row_bytes(2 * KS), VROW = dw_row_bytes(DT), TILE = DW_KEYS * (KROW + VROW);
    constexpr int V = DT * 8;
    extern __shared__ __align__(16) uint8_t dw_smem[];
    __shared__ float s_m[DW_WARPS][16], s_l[DW_WARPS][16];
    __shared__ int s_last;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
    const int split = blockIdx.x, vh = blockIdx.y, zt = blockIdx.z;
    const int t = a.token_list != nullptr ? a.token_list[zt] : zt;
    const int pos = a.positions[t];
    const int* bt = a.block_table + (size_t)(a.seq_of_token != nullptr ? a.seq_of_token[t] : t) * a.max_blocks;
    const int heads = a.maps * a.G, kd = a.maps * a.hd, hdv = a.hdv;
    int lo = (a.window > 0 && pos - a.window + 1 > 0) ? pos - a.window + 1 : 0;
    if (a.chunk > 0) lo = max(lo, (pos / a.chunk) * a.chunk);
    // this range's tiles of 16 positions, and this warp's among them
    const int t_lo = lo / DW_KEYS, t_hi = pos / DW_KEYS, per = (t_hi - t_lo + a.splits) / a.splits;
    const int t0 = t_lo + split * per, t1 = min(t_hi + 1, t0 + per);
    const uint32_t ring = (uint32_t)__cvta_generic_to_shared(dw_smem) + warp * (STAGES * TILE);
    // columns that no copy fills: zeros, once
    {
        uint8_t* base = dw_smem + warp * (STAGES * TILE);
        const int kp = kd / 8, vp = hdv / 8;
        for (int i = lane; i < STAGES * DW_KEYS; i += 32) {
            uint8_t* row = base + (i / DW_KEYS) * TILE + (i % DW_KEYS) * KROW;
            for (int pc = kp; pc < 2 * KS; ++pc) *reinterpret_cast<uint4*>(row + pc * 16) = make_uint4(0u, 0u, 0u, 0u);
            row = base + (i / DW_KEYS) * TILE + DW_KEYS * KROW + (i % DW_KEYS) * VROW;
            for (int pc = vp; pc < DT; ++pc) *reinterpret_cast<uint4*>(row + pc * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
    // lane's key of tile `tl`: its row of the cache, -1 when there is none or it is not seen
    auto slot_of = [&](int tl) {
        const int key = tl * DW_KEYS + (lane & 15);
        if (tl >= t1 || key < lo || key > pos) return -1;
        const int page = bt[key / a.page_size];
        return page < 0 ? -1 : page * a.page_size + key % a.page_size;
    };
    // a lane copies one 16-byte piece column of a row; 32 / pieces rows go out at a time (pieces: those of a padded row)
    constexpr int KP = 2 * KS, VP = DT, KR = 32 / KP, VR = 32 / VP;
    const int kpc = lane % KP, kr = lane / KP, vpc = lane % VP, vr = lane / VP;
    const bool k_in = kpc < kd / 8, v_in = vpc < hdv / 8;
    const size_t k_ld = (size_t)a.nv * kd, v_ld = (size_t)a.nv * hdv;
    const __nv_bfloat16* k_src = a.k + (size_t)vh * kd + kpc * 8;
    const __nv_bfloat16* v_src = a.v + (size_t)vh * hdv + vpc * 8;
    const uint32_t k_dst = ring + kr * KROW + kpc * 16, v_dst = ring + DW_KEYS * KROW + vr * VROW + vpc * 16;
    auto fetch = [&](int slot, int st) {
#pragma unroll
        for (int i = 0; i < DW_KEYS / KR; ++i) {
            const int sl = __shfl_sync(0xffffffffu, slot, i * KR + kr);
            if (k_in) dw_cp16(k_dst + st * TILE + i * KR * KROW, k_src + (sl >= 0 ? sl : 0) * k_ld, sl >= 0);
        }
#pragma unroll
        for (int i = 0; i < DW_KEYS / VR; ++i) {
            const int sl = __shfl_sync(0xffffffffu, slot, i * VR + vr);
            if (v_in) dw_cp16(v_dst + st * TILE + i * VR * VROW, v_src + (sl >= 0 ? sl : 0) * v_ld, sl >= 0);
        }
    };
    auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };

    // query rows as A fragments: rows g and g + 8 (heads), columns 16 ks + 2c (+ 1) and + 8
    uint32_t qa[KS][4];
    {
        const __nv_bfloat16* qrow = a.q + (size_t)t * a.q_stride + (size_t)vh * heads * a.hd;
        auto pair = [&](int head, int col) -> uint32_t {
            const int m = head / a.G, cc = col - m * a.hd;
            if (head >= heads || cc < 0 || cc >= a.hd) return 0u;
            return __ldcg(reinterpret_cast<const uint32_t*>(qrow + (size_t)head * a.hd + cc));
        };
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            qa[ks][0] = pair(g, ks * 16 + 2 * c);
            qa[ks][1] = pair(g + 8, ks * 16 + 2 * c);
            qa[ks][2] = pair(g, ks * 16 + 2 * c + 8);
            qa[ks][3] = pair(g + 8, ks * 16 + 2 * c + 8);
        }
    }

    float o[DT][4];
#pragma unroll
    for (int d = 0; d < DT; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
    float m_ref[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

    const int first_tile = t0 + warp;
#pragma unroll
    for (int st = 0; st < STAGES - 1; ++st) {
        const int tl = first_tile + st * DW_WARPS;
        if (tl < t1) fetch(slot_of(tl), st);
        commit();
    }
    int slot_next = slot_of(first_tile + (STAGES - 1) * DW_WARPS);
    int st = 0, st_fill = STAGES - 1;
    __syncwarp();
    for (int tl = first_tile; tl < t1; tl += DW_WARPS) {
        if (tl + (STAGES - 1) * DW_WARPS < t1) fetch(slot_next, st_fill);
        commit();
        slot_next = slot_of(tl + STAGES * DW_WARPS);
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 1) : "memory");
        __syncwarp();
        const uint32_t K_u = ring + st * TILE, V_u = K_u + DW_KEYS * KROW;
        float s[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
        const uint32_t k_at = K_u + (((lane >> 4) << 3) + (lane & 7)) * KROW + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            uint32_t b0, b1, b2, b3;
            dw_ldsm4(k_at + ks * 32, b0, b1, b2, b3);
            dw_mma(s[0], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], b0, b1);
            dw_mma(s[1], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], b2, b3);
        }
        // s[j][e], s[j][2 + e]: heads g and g + 8, key tl * 16 + j * 8 + 2c + e
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = tl * DW_KEYS + j * 8 + 2 * c + (e & 1);
                float x = a.cap_in > 0.f ? a.cap_l2 * tanh_ex2(s[j][e] * a.cap_in) : s[j][e] * a.scale_log2e;
                x = (key >= lo && key <= pos) ? x : -INFINITY;
                s[j][e] = x;
                mx[e >> 1] = fmaxf(mx[e >> 1], x);
            }
        bool grow = false;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            grow = grow || mx[r] > m_ref[r] + 8.0f;
        }
        if (__any_sync(0xffffffffu, grow)) {
            float f[2];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const float m_new = mx[r] > m_ref[r] + 8.0f ? mx[r] : m_ref[r];
                f[r] = m_ref[r] == -INFINITY ? 0.f : dw_ex2(m_ref[r] - m_new);
                m_ref[r] = m_new;
                l_run[r] *= f[r];
            }
#pragma unroll
            for (int d = 0; d < DT; ++d) { o[d][0] *= f[0]; o[d][1] *= f[0]; o[d][2] *= f[1]; o[d][3] *= f[1]; }
        }
        const float base0 = m_ref[0] == -INFINITY ? 0.f : m_ref[0], base1 = m_ref[1] == -INFINITY ? 0.f : m_ref[1];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            s[j][0] = dw_ex2(s[j][0] - base0);
            s[j][1] = dw_ex2(s[j][1] - base0);
            s[j][2] = dw_ex2(s[j][2] - base1);
            s[j][3] = dw_ex2(s[j][3] - base1);
            l_run[0] += s[j][0] + s[j][1];
            l_run[1] += s[j][2] + s[j][3];
        }
        const uint32_t p0 = dw_pack(s[0][0], s[0][1]), p1 = dw_pack(s[0][2], s[0][3]), p2 = dw_pack(s[1][0], s[1][1]), p3 = dw_pack(s[1][2], s[1][3]);
        const uint32_t v_at = V_u + (lane & 15) * VROW + (lane >> 4) * 16;
#pragma unroll
        for (int d = 0; d < DT; d += 2) {
            uint32_t b0, b1, b2, b3;
            dw_ldsm4t(v_at + d * 16, b0, b1, b2, b3);
            dw_mma(o[d], p0, p1, p2, p3, b0, b1);
            dw_mma(o[d + 1], p0, p1, p2, p3, b2, b3);
        }
        __syncwarp();                                        // every lane has read the tile: its stage may be filled again
        st = st + 1 == STAGES ? 0 : st + 1;
        st_fill = st_fill + 1 == STAGES ? 0 : st_fill + 1;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");

    // ---- the warps' sums, in shared memory
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
        if (c == 0) { s_m[warp][g + 8 * r] = m_ref[r]; s_l[warp][g + 8 * r] = l_run[r]; }
    }
    __syncthreads();                                         // the rings are used up: their place takes the sums
    float* acc = reinterpret_cast<float*>(dw_smem);          // [DW_WARPS][heads][V]
    {
        float* mine = acc + (size_t)warp * heads * V;
#pragma unroll
        for (int d = 0; d < DT; ++d) {
            if (g < heads) *reinterpret_cast<float2*>(mine + g * V + d * 8 + 2 * c) = make_float2(o[d][0], o[d][1]);
            if (g + 8 < heads) *reinterpret_cast<float2*>(mine + (g + 8) * V + d * 8 + 2 * c) = make_float2(o[d][2], o[d][3]);
        }
    }
    __syncthreads();
    const size_t unit = (size_t)zt * a.nv + vh;
    const int rec = heads * hdv + ((2 * heads + 3) & ~3);
    float* fin = acc + (size_t)DW_WARPS * heads * V;         // [heads][V]: the unit's normalised rows
    for (int i = tid; i < heads * hdv; i += DW_WARPS * 32) {
        const int h = i / hdv, d = i - h * hdv;
        float M = s_m[0][h];
#pragma unroll
        for (int w = 1; w < DW_WARPS; ++w) M = fmaxf(M, s_m[w][h]);
        float sum = 0.f, L = 0.f;
#pragma unroll
        for (int w = 0; w < DW_WARPS; ++w) {
            const float f = s_m[w][h] == -INFINITY ? 0.f : dw_ex2(s_m[w][h] - M);
            sum = fmaf(f, acc[((size_t)w * heads + h) * V + d], sum);
            L = fmaf(f, s_l[w][h], L);
        }
        if (a.splits > 1) {
            float* dst = a.part + (unit * a.splits + split) * rec;
            dst[h * hdv + d] = sum;
            if (d == 0) { dst[heads * hdv + 2 * h] = M; dst[heads * hdv + 2 * h + 1] = L; }
        } else {
            fin[h * V + d] = L > 0.f ? sum / L : 0.f;
        }
    }
    if (a.splits > 1) {
        __syncthreads();                                     // this range's record is written
        if (tid == 0) {
            __threadfence();
            const int ticket = atomicAdd(&a.counters[unit], 1);
            s_last = ticket == a.splits - 1;
            if (s_last) a.counters[unit] = 0;                // ready for the next launch
        }
        __syncthreads();
        if (!s_last) return;
        __threadfence();
        const float* src = a.part + unit * a.splits * rec;
        float* wt = acc;                                     // [splits][heads]: a range's weight over the sum of weights
        for (int h = warp; h < heads; h += DW_WARPS) {       // a lane per range (two of them from 33 on)
            float m[2], l[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int sp = u * 32 + lane;
                const bool in = sp < a.splits;
                const float2 ml = in ? __ldcg(reinterpret_cast<const float2*>(src + (size_t)sp * rec + heads * hdv + 2 * h)) : make_float2(-INFINITY, 0.f);
                m[u] = ml.x;
                l[u] = ml.y;
            }
            const float M = warp_max(fmaxf(m[0], m[1]));
            float f[2], L = 0.f;
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                f[u] = m[u] == -INFINITY ? 0.f : dw_ex2(m[u] - M);
                L = fmaf(f[u], l[u], L);
            }
            L = warp_sum(L);
            const float inv = L > 0.f ? 1.0f / L : 0.f;
#pragma unroll
            for (int u = 0; u < 2; ++u)
                if (u * 32 + lane < a.splits) wt[(u * 32 + lane) * heads + h] = f[u] * inv;
        }
        __syncthreads();
        for (int i = tid * 4; i < heads * hdv; i += DW_WARPS * 32 * 4) {
            const int h = i / hdv, d = i - h * hdv;
            float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int sp0 = 0; sp0 < a.splits; sp0 += 8) {
                float4 x[8];
#pragma unroll
                for (int u = 0; u < 8; ++u)
                    x[u] = sp0 + u < a.splits ? __ldcg(reinterpret_cast<const float4*>(src + (size_t)(sp0 + u) * rec + i)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const float f = sp0 + u < a.splits ? wt[(sp0 + u) * heads + h] : 0.f;
                    sum.x = fmaf(f, x[u].x, sum.x); sum.y = fmaf(f, x[u].y, sum.y);
                    sum.z = fmaf(f, x[u].z, sum.z); sum.w = fmaf(f, x[u].w, sum.w);
                }
            }
            *reinterpret_cast<float4*>(fin + h * V + d) = sum;
        }
    }
    __syncthreads();
    // ---- the result
    const size_t row = (size_t)t * a.out_stride;
    auto put = [&](size_t at, float x) {
        if (a.out_f32) reinterpret_cast<float*>(a.out)[row + at] = x;
        else reinterpret_cast<__nv_bfloat16*>(a.out)[row + at] = __float2bfloat16_rn(x);
    };
    if (!a.diff) {
        for (int i = tid; i < heads * hdv; i += DW_WARPS * 32) put((size_t)vh * heads * hdv + i, fin[(i / hdv) * V + i % hdv]);
        return;
    }
    for (int r = warp; r < a.G; r += DW_WARPS) {
        const float* a1 = fin + r * V;
        const float* a2 = fin + (a.G + r) * V;
        float x[DT / 4], ss = 0.f;
#pragma unroll
        for (int j = 0; j < DT / 4; ++j) {
            const int d = j * 32 + lane;
            x[j] = d < hdv ? fmaf(-a.lambda, a2[d], a1[d]) : 0.f;
            ss = fmaf(x[j], x[j], ss);
        }
        const float f = a.mult / sqrtf(warp_sum(ss) / (float)hdv + a.eps);
#pragma unroll
        for (int j = 0; j < DT / 4; ++j) {
            const int d = j * 32 + lane;
            if (d < hdv) put((size_t)(vh * a.G + r) * hdv + d, x[j] * f);
        }
    }
}

template <int KS, int DT>
static int launch_decode_warps(const DwArgs& a, int T, cudaStream_t stream) {
    constexpr int TILE = DW_KEYS * (dw_row_bytes(2 * KS) + dw_row_bytes(DT)), FIT = DW_RING_BYTES / (DW_WARPS * TILE);
    constexpr int STAGES = FIT > 4 ? 4 : (FIT < 2 ? 2 : FIT);
    const size_t ring = (size_t)DW_WARPS * STAGES * TILE;
    const int heads = a.maps * a.G;
    size_t sums = (size_t)(DW_WARPS + 1) * heads * DT * 8 * 4;
    if (a.splits > 1 && (size_t)a.splits > (size_t)DW_WARPS * DT * 8) return AIEN_E_SHAPE;       // the ranges' weights lie where the warps' sums were
    const size_t smem = ring > sums ? ring : sums;
    if (smem > 220 * 1024) return AIEN_E_SHAPE;
    auto kern = paged_decode_warps_kernel<KS, DT, STAGES>;
    static size_t configured = 0;
    if (smem > 48 * 1024 && smem > configured) {
        if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return AIEN_E_STATE;
        configured = smem;
    }
    kern<<<dim3(a.splits, a.nv, T), DW_WARPS * 32, smem, stream>>>(a);
    return launch_status();
}

}  // namespace aien

using namespace aien;

AIEN_API int aien_paged_attention_decode_warps_supports(int nq, int nkv, int hd, int hdv, int maps) {
    if (maps < 1 || nkv <= 0 || nkv % maps != 0 || nq % nkv != 0 || hd <= 0 || hdv <= 0) return 0;
    return ((hd & 7) == 0 && maps * hd <= 256 && (hdv & 7) == 0 && hdv <= 128 && maps * (nq / nkv) <= 16) ? 1 : 0;
}

// part: T * (nkv / maps) * splits records, see DwArgs; 16-byte aligned.
// T tokens (all of the step, or the entries of token_list); q [*, nq * hd], k_cache [slots, nkv, hd], v_cache [slots, nkv / maps,
// hdv]; out [*, nq * hdv], or with diff (maps == 2) [*, nq / 2 * hdv].  counters: T * (nkv / maps) ints, zero before and after.  At most one of window
// and chunk need be given; softcap 0: none.
AIEN_API int aien_paged_attention_decode_warps(
    const void* q, long q_stride, const void* k_cache, const void* v_cache, const int* block_table, int max_blocks,
    const int* seq_of_token, const int* positions, const int* token_list, void* out, long out_stride, int out_f32, float* part,
    int* counters, int nq, int nkv, int hd, int hdv, int maps, int page_size, int window, int chunk, float scale, float softcap,
    int splits, int T, int diff, float lambda, float eps, float mult, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (!aien_paged_attention_decode_warps_supports(nq, nkv, hd, hdv, maps) || page_size <= 0 || window < 0 || chunk < 0 || splits < 1 ||
        splits > DW_MAX_SPLITS || T > 65535 || nkv / maps > 65535 || (diff && maps != 2) || (splits > 1 && (part == nullptr || counters == nullptr)))
        return AIEN_E_SHAPE;
    if ((q_stride & 1) || ((uintptr_t)q & 3) || ((uintptr_t)k_cache & 15) || ((uintptr_t)v_cache & 15) || ((uintptr_t)part & 15)) return AIEN_E_ALIGN;
    const float L2E = 1.4426950408889634f;
    const bool cap = softcap > 0.f;
    const DwArgs a{(const __nv_bfloat16*)q, q_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, block_table, max_blocks,
                   seq_of_token, positions, token_list, out, out_stride, out_f32 ? 1 : 0, part, counters, nkv / maps, maps, nq / nkv, hd, hdv,
                   page_size, window, chunk, scale * L2E, cap ? scale / softcap : 0.f, cap ? softcap * L2E : 0.f, splits, diff ? 1 : 0,
                   lambda, eps, mult};
    const int kd = maps * hd;
    const int ks = kd <= 32 ? 2 : (kd <= 64 ? 4 : (kd <= 128 ? 8 : 16)), dt = hdv <= 32 ? 4 : (hdv <= 64 ? 8 : 16);
#define DW_CASE(K_, D_) if (ks == K_ && dt == D_) return launch_decode_warps<K_, D_>(a, T, stream);
    DW_CASE(2, 4) DW_CASE(2, 8) DW_CASE(2, 16) DW_CASE(4, 4) DW_CASE(4, 8) DW_CASE(4, 16)
    DW_CASE(8, 4) DW_CASE(8, 8) DW_CASE(8, 16) DW_CASE(16, 4) DW_CASE(16, 8) DW_CASE(16, 16)
#undef DW_CASE
    return AIEN_E_SHAPE;
}
