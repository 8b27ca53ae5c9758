// Attention over cached latent rows on the tensor cores (bfloat16 engine): the same result as the plain kernel in
// latent_attention.cu, for latents of up to 512 numbers and rotated parts that are multiples of 8.  A latent that is not
// 64, 128, 256 or 512 numbers long runs in the next of these sizes: its rows are filled up with zeros in shared memory.
//
// A cached row [c | k_rot] serves every head as key and (its first R numbers) as value, so the rows of the score
// product are (token, head) pairs: the queries of a request's portion, laid out [token][head][R + rot], are one
// matrix of len * heads rows.  One CTA owns 64 such rows (16 for steps of single tokens); a step has at most
// T * heads / 64 + S tiles, and a CTA finds its request and offset from q_start.  Keys are visited in blocks of 64 aligned
// to absolute positions, read through the block table into shared memory with cp.async (absent or unneeded rows
// zero-filled).  The warps of a 16-row slab deal out the block's keys for the scores and the latent's channels for the
// weighted sum, so they exchange their row maxima and their probabilities (bfloat16) through shared memory.  Products run
// on mma.sync.m16n8k16 (bfloat16 in, float32
// accumulate) with ldmatrix-fed fragments; masks, the online softmax and the sink are float32 per row.
#include "common.cuh"
#include <math.h>

namespace aien {

constexpr int LX_BM = 64, LX_BN = 64, LX_PSTR = LX_BN + 8;

// Numbers a row of D numbers takes in shared memory (without its padding): whole k-steps of 16, and all R columns of the sum.
__host__ __device__ __forceinline__ int lx_row_width(int R, int D) { return (D + 15) / 16 * 16 > R ? (D + 15) / 16 * 16 : R; }

__device__ __forceinline__ void lx_cp_async16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void lx_cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void lx_cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void lx_ldmatrix_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void lx_ldmatrix_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void lx_ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void lx_mma(float c[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t lx_pack(float lo, float hi) {
    __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&p);
}

// SLABS: 16-row slabs of a tile (4: tiles of 64 rows, for portions; 1: tiles of 16 rows, for steps of single tokens, where
// a request has only its heads as rows).  The WARPS / SLABS warps of a slab deal out the keys of a block for the scores and
// the channels for the weighted sum (tiles of 64 rows run 16 warps: four to a slab, so that a warp's share of the weighted
// sum, 16 rows x a quarter of the latent, leaves registers for loads in flight).
template <int R, int SLABS, int WARPS>
__global__ void __launch_bounds__(WARPS * 32, SLABS == 1 ? 2 : 1)
latent_attention_tc_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache,
                           const int* __restrict__ block_table, int max_blocks, const int* __restrict__ q_start,
                           const int* __restrict__ positions, int S, __nv_bfloat16* __restrict__ out,
                           int H, int r_lat, int rd, int page_size, int window, float scale_log2e, const float* __restrict__ sinks,
                           int ksplit, float* __restrict__ part_o, float* __restrict__ part_ml, int single_only) {
    constexpr int BM = SLABS * 16, PARTS = WARPS / SLABS, KP = LX_BN / PARTS, NJ = KP / 8, CHP = R / PARTS, THREADS = WARPS * 32;
    constexpr int DT = CHP / 8;                  // n8 tiles of this warp's share of the channels
    static_assert(DT >= 2 && DT % 2 == 0, "a warp's share of the latent must be whole pairs of n8 tiles");
    // r_lat <= R: the latent's own size; a row's D numbers are read, the rest of its width in shared memory is zeros
    const int D = r_lat + rd, CH = D / 8, KS = (D + 15) / 16, W = lx_row_width(R, D), CHW = W / 8, STR = W + 8;
    extern __shared__ __align__(16) uint8_t lx_smem[];
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(lx_smem);          // [BM][STR]
    __nv_bfloat16* Ks = Qs + BM * STR;                                      // [64][STR]
    __nv_bfloat16* Ps = Ks + LX_BN * STR;                                   // [BM][LX_PSTR]
    float* stat = reinterpret_cast<float*>(Ps + BM * LX_PSTR);              // [PARTS][BM]
    __shared__ int key_there[LX_BN];                                        // whether the block's key is in the cache and needed
    const uint32_t Qs_u = (uint32_t)__cvta_generic_to_shared(Qs), Ks_u = (uint32_t)__cvta_generic_to_shared(Ks);
    const uint32_t Ps_u = (uint32_t)__cvta_generic_to_shared(Ps);

    // which request, which rows
    int s = -1, row0 = 0, acc = 0, unit = 0;             // unit: how many served tokens come before a single one
    for (int i = 0; i < S; ++i) {
        const int n = q_start[i + 1] - q_start[i];
        const int tiles = single_only && n != 1 ? 0 : (n * H + BM - 1) / BM;         // single_only: portions are served elsewhere
        if ((int)blockIdx.x < acc + tiles) {
            s = i;
            row0 = ((int)blockIdx.x - acc) * BM;
            unit = acc / tiles;
            break;
        }
        acc += tiles;
    }
    if (s < 0) return;
    const int qs = q_start[s], len = q_start[s + 1] - qs;
    const int nrows = min(BM, len * H - row0);
    const int pos_first = positions[qs];
    const int pos_lo = pos_first + row0 / H, pos_hi = pos_first + (row0 + nrows - 1) / H;
    const int first = (window > 0 && pos_lo - window + 1 > 0) ? pos_lo - window + 1 : 0;
    const int* bt = block_table + (size_t)s * max_blocks;

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slab = warp % SLABS, half = warp / SLABS;                     // half: which share of the keys / channels
    const int g = lane >> 2, c = lane & 3;

    const __nv_bfloat16* qbase = q + ((size_t)qs * H + row0) * D;
    for (int idx = tid; idx < BM * CHW; idx += THREADS) {
        const int r = idx / CHW, ch = idx - r * CHW;
        const bool valid = r < nrows && ch < CH;
        lx_cp_async16(Qs_u + (uint32_t)(r * STR + ch * 8) * 2, qbase + (valid ? (size_t)r * D + ch * 8 : 0), valid);
    }
    lx_cp_async_commit();

    const uint32_t q_frag_u = Qs_u + (uint32_t)((slab * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * STR + (lane >> 4) * 8) * 2;
    const uint32_t p_frag_u = Ps_u + (uint32_t)((slab * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LX_PSTR + (lane >> 4) * 8) * 2;

    float o[DT][4];
#pragma unroll
    for (int d = 0; d < DT; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    const int ra = slab * 16 + g, rb = ra + 8;                              // this thread's two rows in the tile
    const int qpos0 = ra < nrows ? pos_first + (row0 + ra) / H : -1, qpos1 = rb < nrows ? pos_first + (row0 + rb) / H : -1;
    const int wlo0 = window > 0 ? qpos0 - window + 1 : 0, wlo1 = window > 0 ? qpos1 - window + 1 : 0;
    const bool active = slab * 16 < nrows;

    const int kb_begin = first / LX_BN, kb_end = pos_hi / LX_BN;
    if (ksplit > 1) {                                                      // Q must have landed even if this CTA gets no block
        lx_cp_async_wait_all();
        __syncthreads();
    }
    for (int kb = kb_begin + (int)blockIdx.y; kb <= kb_end; kb += ksplit) {
        for (int idx = tid; idx < LX_BN * CHW; idx += THREADS) {
            const int r = idx / CHW, ch = idx - r * CHW;
            const int key = kb * LX_BN + r;
            bool valid = key >= first && key <= pos_hi;
            long slot = 0;
            if (valid) {
                const int page = bt[key / page_size];
                valid = page >= 0;
                slot = (long)page * page_size + key % page_size;
            }
            const bool copy = valid && ch < CH;
            lx_cp_async16(Ks_u + (uint32_t)(r * STR + ch * 8) * 2, cache + (copy ? (size_t)slot * D + ch * 8 : 0), copy);
            if (ch == 0) key_there[r] = valid ? 1 : 0;
        }
        lx_cp_async_commit();
        lx_cp_async_wait_all();
        __syncthreads();                                                   // the block's rows (and, first time, Q) have landed

        float sc[NJ][4];
#pragma unroll
        for (int j = 0; j < NJ; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
        if (active) {
#pragma unroll 4
            for (int kk = 0; kk < KS; ++kk) {
                uint32_t q0r, q1r, q2r, q3r;
                lx_ldmatrix_x4(q_frag_u + kk * 32, q0r, q1r, q2r, q3r);
                if constexpr (NJ == 1) {
                    const int row = half * KP + (lane & 7), col = kk * 16 + ((lane >> 3) & 1) * 8;
                    uint32_t b0, b1;
                    lx_ldmatrix_x2(Ks_u + (uint32_t)(row * STR + col) * 2, b0, b1);
                    lx_mma(sc[0], q0r, q1r, q2r, q3r, b0, b1);
                } else {
#pragma unroll
                    for (int j = 0; j < NJ; j += 2) {
                        const int mi = lane >> 3;
                        const int row = half * KP + (j + (mi >> 1)) * 8 + (lane & 7), col = kk * 16 + (mi & 1) * 8;
                        uint32_t b0, b1, b2, b3;
                        lx_ldmatrix_x4(Ks_u + (uint32_t)(row * STR + col) * 2, b0, b1, b2, b3);
                        lx_mma(sc[j], q0r, q1r, q2r, q3r, b0, b1);
                        lx_mma(sc[j + (NJ > 1 ? 1 : 0)], q0r, q1r, q2r, q3r, b2, b3);
                    }
                }
            }
        }
        // masks and this half's row maxima (scores in log2 units)
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int kl = half * KP + j * 8 + 2 * c + e, key = kb * LX_BN + kl;
                const bool there = key_there[kl] != 0;
                const bool ok0 = there && key <= qpos0 && key >= wlo0, ok1 = there && key <= qpos1 && key >= wlo1;
                sc[j][e] = ok0 ? sc[j][e] * scale_log2e : -INFINITY;
                sc[j][2 + e] = ok1 ? sc[j][2 + e] * scale_log2e : -INFINITY;
                mx0 = fmaxf(mx0, sc[j][e]);
                mx1 = fmaxf(mx1, sc[j][2 + e]);
            }
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        if (c == 0) {
            stat[half * BM + ra] = mx0;
            stat[half * BM + rb] = mx1;
        }
        __syncthreads();                                                   // every share's maxima are there
#pragma unroll
        for (int pp = 0; pp < PARTS; ++pp) {
            mx0 = fmaxf(mx0, stat[pp * BM + ra]);
            mx1 = fmaxf(mx1, stat[pp * BM + rb]);
        }
        const float mn0 = fmaxf(m_run[0], mx0), mn1 = fmaxf(m_run[1], mx1);
        const float corr0 = (m_run[0] == -INFINITY) ? 0.f : exp2f(m_run[0] - mn0);
        const float corr1 = (m_run[1] == -INFINITY) ? 0.f : exp2f(m_run[1] - mn1);
        const float base0 = (mn0 == -INFINITY) ? 0.f : mn0, base1 = (mn1 == -INFINITY) ? 0.f : mn1;
        float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            float p00 = exp2f(sc[j][0] - base0), p01 = exp2f(sc[j][1] - base0);      // exp2(-inf) = 0 for masked keys
            float p10 = exp2f(sc[j][2] - base1), p11 = exp2f(sc[j][3] - base1);
            sum0 += p00 + p01;
            sum1 += p10 + p11;
            const int col = half * KP + j * 8 + 2 * c;
            *reinterpret_cast<uint32_t*>(Ps + ra * LX_PSTR + col) = lx_pack(p00, p01);
            *reinterpret_cast<uint32_t*>(Ps + rb * LX_PSTR + col) = lx_pack(p10, p11);
        }
        l_run[0] = l_run[0] * corr0 + sum0;
        l_run[1] = l_run[1] * corr1 + sum1;
        m_run[0] = mn0;
        m_run[1] = mn1;
#pragma unroll
        for (int d = 0; d < DT; ++d) { o[d][0] *= corr0; o[d][1] *= corr0; o[d][2] *= corr1; o[d][3] *= corr1; }
        __syncthreads();                                                   // the probabilities of every share are there
        if (active) {
#pragma unroll
            for (int ks = 0; ks < LX_BN / 16; ++ks) {
                uint32_t a0, a1, a2, a3;
                lx_ldmatrix_x4(p_frag_u + ks * 32, a0, a1, a2, a3);
#pragma unroll
                for (int d = 0; d < DT; d += 2) {
                    const int row = ks * 16 + (lane & 15), col = half * CHP + (d + (lane >> 4)) * 8;
                    uint32_t b0, b1, b2, b3;
                    lx_ldmatrix_x4_trans(Ks_u + (uint32_t)(row * STR + col) * 2, b0, b1, b2, b3);
                    lx_mma(o[d], a0, a1, a2, a3, b0, b1);
                    lx_mma(o[d + 1], a0, a1, a2, a3, b2, b3);
                }
            }
        }
        __syncthreads();                                                   // every warp is done with this block
    }

    if (ksplit > 1) {
        // this CTA saw only some of the key blocks: its running maximum, its sum and its unnormalised weighted sum go to
        // the scratch, and a second launch combines the CTAs of a row
        l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], 1); l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], 2);
        l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], 1); l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], 2);
        if (c == 0) {
            stat[half * BM + ra] = l_run[0];
            stat[half * BM + rb] = l_run[1];
        }
        __syncthreads();
        l_run[0] = l_run[1] = 0.f;
#pragma unroll
        for (int pp = 0; pp < PARTS; ++pp) {
            l_run[0] += stat[pp * BM + ra];
            l_run[1] += stat[pp * BM + rb];
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int row = r == 0 ? ra : rb;
            if (row >= nrows) continue;
            const size_t slot = ((size_t)(single_only ? unit : qs) * H + row0 + row) * ksplit + blockIdx.y;
            if (half == 0 && c == 0) {
                part_ml[slot * 2] = m_run[r];
                part_ml[slot * 2 + 1] = l_run[r];
            }
            float* dst = part_o + slot * r_lat + half * CHP;
#pragma unroll
            for (int d = 0; d < DT; ++d)
                if (half * CHP + d * 8 < r_lat) *reinterpret_cast<float2*>(dst + d * 8 + 2 * c) = make_float2(o[d][2 * r], o[d][2 * r + 1]);
        }
        return;
    }
    // the denominators: this thread's partial sums, its quad's, the other half's
    l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], 1); l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], 2);
    l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], 1); l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], 2);
    if (c == 0) {
        stat[half * BM + ra] = l_run[0];
        stat[half * BM + rb] = l_run[1];
    }
    __syncthreads();
    l_run[0] = l_run[1] = 0.f;
#pragma unroll
    for (int pp = 0; pp < PARTS; ++pp) {
        l_run[0] += stat[pp * BM + ra];
        l_run[1] += stat[pp * BM + rb];
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = r == 0 ? ra : rb;
        if (row >= nrows) continue;
        float corr = 1.f;
        if (sinks != nullptr) {                                            // the sink joins the denominator once (log2 units like the scores)
            const float sk = sinks[(row0 + row) % H] * 1.4426950408889634f;
            const float mn = fmaxf(m_run[r], sk);
            corr = (m_run[r] == -INFINITY) ? 0.f : exp2f(m_run[r] - mn);
            l_run[r] = l_run[r] * corr + exp2f(sk - mn);
        }
        const float inv = l_run[r] > 0.f ? corr / l_run[r] : 0.f;
        __nv_bfloat16* dst = out + ((size_t)qs * H + row0 + row) * r_lat + half * CHP;
#pragma unroll
        for (int d = 0; d < DT; ++d)
            if (half * CHP + d * 8 < r_lat) *reinterpret_cast<uint32_t*>(dst + d * 8 + 2 * c) = lx_pack(o[d][2 * r] * inv, o[d][2 * r + 1] * inv);
    }
}

// out[row] = sum_s 2^(m_s - M) o_s / (sum_s 2^(m_s - M) l_s + 2^(sink - M)), M = max over the row's parts and the sink.
// One CTA per (token, head) row; tokens (may be null): the tokens served.  The weights of the parts are made once, in shared
// memory; the sums run over the parts in order, eight requested at a time.
constexpr int LX_MAX_SPLIT = 512;
__global__ void __launch_bounds__(128)
latent_attention_merge_kernel(int R, const float* __restrict__ part_o, const float* __restrict__ part_ml, int ksplit,
                              const float* __restrict__ sinks, int H, __nv_bfloat16* __restrict__ out, const int* __restrict__ tokens) {
    __shared__ float wt[LX_MAX_SPLIT];
    __shared__ float red[32];
    const int unit = blockIdx.x / H, h = blockIdx.x - unit * H;
    const size_t row = blockIdx.x, to = (size_t)(tokens != nullptr ? tokens[unit] : unit) * H + h;
    const float sk = sinks != nullptr ? sinks[h] * 1.4426950408889634f : -INFINITY;
    float M = sk;
    for (int s = threadIdx.x; s < ksplit; s += 128) M = fmaxf(M, part_ml[(row * ksplit + s) * 2]);
    M = block_max(M, red);
    float den = 0.f;
    for (int s = threadIdx.x; s < ksplit; s += 128) {
        const float m = part_ml[(row * ksplit + s) * 2];
        const float w = m != -INFINITY ? exp2f(m - M) : 0.f;
        wt[s] = w;
        den += w * part_ml[(row * ksplit + s) * 2 + 1];
    }
    den = block_sum(den, red);                                             // its barriers also order the weights
    if (sinks != nullptr && M != -INFINITY) den += exp2f(sk - M);
    const float inv = den > 0.f ? 1.0f / den : 0.f;
    for (int ch = threadIdx.x * 2; ch < R; ch += 256) {                    // R is a multiple of 8
        const float* src = part_o + row * ksplit * R + ch;
        float2 acc = make_float2(0.f, 0.f);
        for (int s0 = 0; s0 < ksplit; s0 += 8) {
            float2 v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u)
                v[u] = s0 + u < ksplit && wt[s0 + u] != 0.f ? *reinterpret_cast<const float2*>(src + (size_t)(s0 + u) * R) : make_float2(0.f, 0.f);
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const float w = s0 + u < ksplit ? wt[s0 + u] : 0.f;
                acc.x = fmaf(w, v[u].x, acc.x);
                acc.y = fmaf(w, v[u].y, acc.y);
            }
        }
        *reinterpret_cast<uint32_t*>(out + to * R + ch) = lx_pack(acc.x * inv, acc.y * inv);
    }
}

template <int R, int SLABS, int WARPS>
static int launch_latent_tc(const void* q, const void* cache, const int* bt, int max_blocks, const int* q_start, const int* positions,
                            int T, int S, void* out, int H, int r_lat, int rd, int page_size, int window, float scale, const float* sinks,
                            int ksplit, float* part_o, float* part_ml, const int* tokens, int num_tokens, cudaStream_t stream) {
    const int D = r_lat + rd;
    constexpr int BM = SLABS * 16;
    const size_t smem = (size_t)(BM + LX_BN) * (lx_row_width(R, D) + 8) * 2 + (size_t)BM * LX_PSTR * 2 + (size_t)WARPS * 16 * sizeof(float);
    if (smem > 227 * 1024) return AIEN_E_SHAPE;
    auto kern = latent_attention_tc_kernel<R, SLABS, WARPS>;
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return AIEN_E_STATE;
    // tokens: only these, each a request's one token of the step
    const long tiles = tokens != nullptr ? (long)num_tokens * ((H + BM - 1) / BM) : ((long)T * H) / BM + S;
    kern<<<dim3((unsigned)tiles, ksplit), WARPS * 32, smem, stream>>>((const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, bt, max_blocks, q_start,
                                                                     positions, S, (__nv_bfloat16*)out, H, r_lat, rd, page_size, window,
                                                                     scale * 1.4426950408889634f, sinks, ksplit, part_o, part_ml, tokens != nullptr ? 1 : 0);
    if (ksplit > 1)
        latent_attention_merge_kernel<<<dim3((unsigned)((long)(tokens != nullptr ? num_tokens : T) * H)), 128, 0, stream>>>(
            r_lat, part_o, part_ml, ksplit, sinks, H, (__nv_bfloat16*)out, tokens);
    return launch_status();
}


// ---------------------------------------------------------------- one product per head, on the tensor cores
// C[m, h, n] = sum_k A[m, h, k] * W[h, n, k], times sigmoid(gate[m, h]) when given (see head_project_kernel), for bfloat16 A and W: tiles of 64 x 64 per CTA of
// four warps, k in steps of 64 through shared memory (cp.async), mma.sync.m16n8k16 with float32 accumulation.
constexpr int HT_BM = 64, HT_BN = 64, HT_BK = 64, HT_STR = HT_BK + 8;

// Two stages of k-steps: the next one's pieces are requested before the products of this one.  rows (or null): A's and C's rows
// are those that it lists, M of them.
template <typename TC>
__global__ void __launch_bounds__(128)
head_project_tc_kernel(const __nv_bfloat16* __restrict__ A, long lda, long a_head, const __nv_bfloat16* __restrict__ W, long w_head,
                       TC* __restrict__ C, long ldc, long c_head, int M, int N, int K, const void* __restrict__ gate, int gdt, long ldg, int gate_n,
                       const int* __restrict__ rows) {
    __shared__ __align__(16) __nv_bfloat16 As[2][HT_BM * HT_STR];
    __shared__ __align__(16) __nv_bfloat16 Ws[2][HT_BN * HT_STR];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int mh = warp & 1, nh = warp >> 1, g = lane >> 2, c = lane & 3;
    const int m0 = blockIdx.y * HT_BM, n0 = blockIdx.x * HT_BN, h = blockIdx.z;
    A += (size_t)h * a_head;
    W += (size_t)h * w_head;
    C += (size_t)h * c_head;
    float acc[2][4][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
    auto fetch = [&](int k0, int st) {
        const uint32_t As_u = (uint32_t)__cvta_generic_to_shared(As[st]), Ws_u = (uint32_t)__cvta_generic_to_shared(Ws[st]);
        for (int idx = tid; idx < HT_BM * (HT_BK / 8); idx += 128) {
            const int r = idx >> 3, ch = idx & 7;
            const bool kin = k0 + ch * 8 < K;
            const bool va = kin && m0 + r < M, vw = kin && n0 + r < N;
            const size_t ar = va ? (size_t)(rows != nullptr ? rows[m0 + r] : m0 + r) : 0;
            lx_cp_async16(As_u + (uint32_t)(r * HT_STR + ch * 8) * 2, A + ar * lda + (va ? k0 + ch * 8 : 0), va);
            lx_cp_async16(Ws_u + (uint32_t)(r * HT_STR + ch * 8) * 2, W + (size_t)(vw ? n0 + r : 0) * K + (vw ? k0 + ch * 8 : 0), vw);
        }
        lx_cp_async_commit();
    };
    fetch(0, 0);
    for (int k0 = 0, st = 0; k0 < K; k0 += HT_BK, st ^= 1) {
        if (k0 + HT_BK < K) {
            fetch(k0 + HT_BK, st ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            lx_cp_async_wait_all();
        }
        __syncthreads();
        const uint32_t As_u = (uint32_t)__cvta_generic_to_shared(As[st]), Ws_u = (uint32_t)__cvta_generic_to_shared(Ws[st]);
#pragma unroll
        for (int kk = 0; kk < HT_BK / 16; ++kk) {
            uint32_t a[2][4];
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
                lx_ldmatrix_x4(As_u + (uint32_t)((mh * 32 + mt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * HT_STR + kk * 16 + (lane >> 4) * 8) * 2,
                               a[mt][0], a[mt][1], a[mt][2], a[mt][3]);
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int mi = lane >> 3;
                uint32_t b0, b1, b2, b3;
                lx_ldmatrix_x4(Ws_u + (uint32_t)((nh * 32 + (j + (mi >> 1)) * 8 + (lane & 7)) * HT_STR + kk * 16 + (mi & 1) * 8) * 2, b0, b1, b2, b3);
#pragma unroll
                for (int mt = 0; mt < 2; ++mt) {
                    lx_mma(acc[mt][j], a[mt][0], a[mt][1], a[mt][2], a[mt][3], b0, b1);
                    lx_mma(acc[mt][j + 1], a[mt][0], a[mt][1], a[mt][2], a[mt][3], b2, b3);
                }
            }
        }
        __syncthreads();
    }
    const bool pairs = ((N | ldc | c_head) & 1) == 0 && ((uintptr_t)C & (2 * sizeof(TC) - 1)) == 0;     // two neighbouring columns at a time
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int ml = m0 + mh * 32 + mt * 16 + g + r * 8;
            if (ml >= M) continue;
            const size_t m = (size_t)(rows != nullptr ? rows[ml] : ml);
            const float gs = (gate != nullptr && gate_n == 0) ? 1.0f / (1.0f + expf(-load_dyn(gate, gdt, m * ldg + h))) : 1.0f;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int n = n0 + nh * 32 + j * 8 + 2 * c;
                float v[2] = {acc[mt][j][2 * r] * gs, acc[mt][j][2 * r + 1] * gs};
                if (gate_n > 0) {
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        if (n + e < N) v[e] *= __fdividef(1.0f, 1.0f + __expf(-load_dyn(gate, gdt, m * ldg + (size_t)h * gate_n + n + e)));
                }
                TC* dst = C + m * ldc + n;
                if (pairs && n + 1 < N) {
                    if constexpr (sizeof(TC) == 2) *reinterpret_cast<uint32_t*>(dst) = lx_pack(v[0], v[1]);
                    else *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
                } else {
                    if (n < N) dst[0] = from_f<TC>(v[0]);
                    if (n + 1 < N) dst[1] = from_f<TC>(v[1]);
                }
            }
        }
}

// ---------------------------------------------------------------- the latents of portions, for keys and values per head
// Portion p of the step (the p-th request that brings more than one token) gets rows p * len .. of `out`: its cached latents at
// positions 0 .. ctx_len - 1, then zeros.  table [S, len / 128]: the 128-row pages of those rows, in order, for requests
// with a portion.  One CTA per 8 rows; a warp finds the portion's request, then each of the eight copies a row.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, int r_lat, const int* __restrict__ block_table, int max_blocks, int page_size,
                     const int* __restrict__ q_start, const int* __restrict__ ctx_len, int S, int len, __nv_bfloat16* __restrict__ out,
                     int* __restrict__ table) {
    __shared__ int s_req;
    const int p = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (tid == 0) s_req = -1;
    __syncthreads();
    if (warp == 0) {
        int before = 0;
        for (int base = 0; base < S; base += 32) {
            const int i = base + lane;
            const bool has = i < S && q_start[i + 1] - q_start[i] > 1;
            const uint32_t mask = __ballot_sync(0xffffffffu, has);
            if (has && before + __popc(mask & ((1u << lane) - 1u)) == p) s_req = i;
            before += __popc(mask);
        }
    }
    __syncthreads();
    const int s = s_req, n = s >= 0 ? ctx_len[s] : 0;
    if (s >= 0 && blockIdx.x == 0)
        for (int b = tid; b < len / 128; b += 256) table[(size_t)s * (len / 128) + b] = p * (len / 128) + b;
    const int* bt = s >= 0 ? block_table + (size_t)s * max_blocks : nullptr;
    {
        const int key = blockIdx.x * 8 + warp;
        const int page = key < n ? bt[key / page_size] : -1;
        const uint4* src = reinterpret_cast<const uint4*>(cache + ((size_t)(page >= 0 ? page : 0) * page_size + key % page_size) * r_lat);
        uint4* dst = reinterpret_cast<uint4*>(out + ((size_t)p * len + key) * r_lat);
        for (int i = lane; i < r_lat / 8; i += 32) dst[i] = page >= 0 ? src[i] : make_uint4(0u, 0u, 0u, 0u);
    }
}

}  // namespace aien

using namespace aien;

static int lx_padded_rank(int kv_rank) { return kv_rank <= 64 ? 64 : (kv_rank <= 128 ? 128 : (kv_rank <= 256 ? 256 : 512)); }

AIEN_API int aien_latent_attention_tc_supports(int kv_rank, int rot_dim) {
    if (kv_rank <= 0 || kv_rank > 512 || (kv_rank & 7) || rot_dim < 0 || (rot_dim & 7)) return 0;
    const size_t smem = (size_t)(LX_BM + LX_BN) * (lx_row_width(lx_padded_rank(kv_rank), kv_rank + rot_dim) + 8) * 2 + (size_t)LX_BM * LX_PSTR * 2 + 16 * 16 * sizeof(float);
    return smem <= 227 * 1024 ? 1 : 0;
}

// q bfloat16 [T, H, kv_rank + rot_dim] (contiguous), cache bfloat16 [slots, kv_rank + rot_dim], out bfloat16 [T, H, kv_rank].
// The step's T tokens are the portions q_start[s] .. q_start[s + 1] of S requests; positions[t] is token t's position.
// ksplit > 1: the key blocks of every tile are dealt out to ksplit CTAs (for steps with few tiles); part_o (float32,
// T * H * ksplit * kv_rank) and part_ml (float32, T * H * ksplit * 2) hold their partial results for the merging launch.
// tokens (may be null), num_tokens: serve only these tokens, each the one token that its request brings (a mixed step's).
// small_tiles != 0: tiles of 16 rows instead of 64 (steps in which every request brings one token), for latents of more than 64.
AIEN_API int aien_latent_attention_tc(const void* q, const void* cache, const int* block_table, int max_blocks, const int* q_start,
                                      const int* positions, void* out, int T, int S, int H, int kv_rank, int rot_dim, int page_size,
                                      int window, float scale, const float* sinks, int ksplit, float* part_o, float* part_ml,
                                      int small_tiles, const int* tokens, int num_tokens, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (H <= 0 || page_size <= 0 || window < 0 || !aien_latent_attention_tc_supports(kv_rank, rot_dim)) return AIEN_E_SHAPE;
    if (((uintptr_t)q & 15) || ((uintptr_t)cache & 15) || ((uintptr_t)out & 3)) return AIEN_E_ALIGN;
    if (ksplit < 1 || ksplit > LX_MAX_SPLIT || num_tokens < 0 || (tokens != nullptr && num_tokens == 0) || (ksplit > 1 && (part_o == nullptr || part_ml == nullptr || ((uintptr_t)part_o & 7)))) return AIEN_E_SHAPE;
    const int padded = lx_padded_rank(kv_rank);
#define LX_CASE(RV, SL)                                                                                                          \
    if (padded == RV)                                                                                                            \
        return launch_latent_tc<RV, SL, (SL == 4 ? 16 : 8)>(q, cache, block_table, max_blocks, q_start, positions, T, S, out, H, kv_rank, rot_dim, page_size,  \
                                        window, scale, sinks, ksplit, part_o, part_ml, tokens, num_tokens, stream);
    if (small_tiles && padded >= 128) {                    // tiles of 16 rows: a latent of 64 would leave a warp half a pair of n8 tiles
        LX_CASE(128, 1) LX_CASE(256, 1) LX_CASE(512, 1)
    }
    LX_CASE(64, 4) LX_CASE(128, 4) LX_CASE(256, 4) LX_CASE(512, 4)
#undef LX_CASE
    return AIEN_E_SHAPE;
}

// A bfloat16 [M, lda] (head h at column h * a_head), W bfloat16 [heads, N, K], C [M, ldc] (head h at column h * c_head).
// K, lda and a_head multiples of 8, A and W 16-byte aligned.
AIEN_API int aien_head_project_tc(const void* A, long lda, long a_head, const void* W, void* C, int c_dt, long ldc, long c_head,
                                  int M, int N, int K, int heads, const void* gate, int gate_dt, long ldg, int gate_n, const int* rows,
                                  cudaStream_t stream) {
    if (M <= 0 || N <= 0 || heads <= 0) return 0;
    if (K <= 0 || heads > 65535 || gate_n < 0 || (gate_n > 0 && (gate == nullptr || gate_n != N))) return AIEN_E_SHAPE;
    if ((K & 7) || (lda & 7) || (a_head & 7) || ((uintptr_t)A & 15) || ((uintptr_t)W & 15)) return AIEN_E_ALIGN;
    dim3 grid((N + HT_BN - 1) / HT_BN, (M + HT_BM - 1) / HT_BM, heads);
    if (grid.y > 65535) return AIEN_E_SHAPE;
    AIEN_DISPATCH_DTYPE(c_dt, TC, (head_project_tc_kernel<TC><<<grid, 128, 0, stream>>>((const __nv_bfloat16*)A, lda, a_head, (const __nv_bfloat16*)W,
                                                                                     (long)N * K, (TC*)C, ldc, c_head, M, N, K, gate, gate_dt, ldg, gate_n, rows)));
    return launch_status();
}

// cache bfloat16 [slots, r_lat]; out bfloat16 [portions * len, r_lat]; table int32 [S, len / 128]; len a multiple of 128 that
// covers every portion's context; r_lat a multiple of 8.
AIEN_API int aien_latent_gather(const void* cache, int r_lat, const int* block_table, int max_blocks, int page_size, const int* q_start,
                                const int* ctx_len, int S, int portions, int len, void* out, int* table, cudaStream_t stream) {
    if (portions <= 0 || S <= 0) return 0;
    if (r_lat <= 0 || (r_lat & 7) || page_size <= 0 || len <= 0 || (len & 127) || portions > 65535) return AIEN_E_SHAPE;
    if (((uintptr_t)cache & 15) || ((uintptr_t)out & 15)) return AIEN_E_ALIGN;
    latent_gather_kernel<<<dim3(len / 8, portions), 256, 0, stream>>>((const __nv_bfloat16*)cache, r_lat, block_table, max_blocks, page_size, q_start,
                                                                      ctx_len, S, len, (__nv_bfloat16*)out, table);
    return launch_status();
}
