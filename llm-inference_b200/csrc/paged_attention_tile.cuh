// The bfloat16 prompt kernel of b200_paged_attention, instantiated by capped_attention.cu (the sizes and masks without a distance
// bias) and biased_attention.cu (with one).
#pragma once
#include "launch_count.h"
#include "paged_attention.cuh"

namespace b200 {

// ---------------------------------------------------------------------------------------------------------------
// bfloat16 prompt portions on tensor-core tiles (mma.sync m16n8k16, fp32 accumulation): a CTA of four warps owns 64
// consecutive rows of the packed batch for one query head; each warp keeps its 16 rows' Q fragments and output
// accumulators in registers and walks the keys in tiles of 64 that land in shared memory by cp.async (two buffers, the
// next tile in flight while this one is multiplied). Scores, cap, mask and the online softmax stay in fp32 registers;
// the probabilities are rounded to bfloat16 only as the operand of the second product. Rows of the tile that belong
// to different sequences are handled segment by segment (the other rows masked), so prompt portions, single tokens and
// mixed batches share the launch. The sink is the initial state of every row (m = 0, l = denom_bias; or a head's own score and 1).
// BIAS: a learned bias per distance joins the scaled scores. A tile of 64 rows x 64 keys sees 127 distances (the rows of a segment
// are consecutive positions), staged beside the tile; far tiles, where every distance has the table's last value, add a constant.
// These variants also take any dim <= D and vdim <= DV in multiples of 8 (the rest of the tile is zero and its products skipped).
// ---------------------------------------------------------------------------------------------------------------
constexpr int kTileM = 64, kTileN = 64;

// the special-function unit's power of two (relative error 2^-22)
__device__ __forceinline__ float pa_exp2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

enum { kNoBias = 0, kBias = 1, kBiasPadded = 2 };   // kBiasPadded: dim and vdim below the tile's

template <int D, int DV, bool BLOCKS, int KIND>   // dim == D (a multiple of 32), vdim == DV (a multiple of 16); BLOCKS: a block mask or a window
__global__ void __launch_bounds__(128, DV <= 128 ? 3 : 2) paged_attn_tile_kernel(const PA a) {
    using bf = __nv_bfloat16;
    constexpr bool BIAS = KIND != kNoBias, PADDED = KIND == kBiasPadded;
    constexpr int RS = D + 8;                 // row stride in elements: 16-byte aligned, conflict-free fragment loads
    constexpr int CH = D / 8;                 // 16-byte chunks per row
    constexpr int RSV = DV + 8;               // the same for value rows
    extern __shared__ __align__(16) unsigned char pa_smem[];
    bf* Ks = reinterpret_cast<bf*>(pa_smem);                  // [2][64][RS]
    bf* Vs = Ks + 2 * kTileN * RS;                            // [2][64][RSV]
    bf* Qs = Ks + kTileN * RS;                                // [64][RS]: the Q tile borrows the second K buffer until its
                                                              // fragments are in registers (three CTAs fit an SM this way)
    int* row_pos = reinterpret_cast<int*>(Vs + 2 * kTileN * RSV);   // [64], -1: no such row
    int* row_slot = row_pos + kTileM;
    float* bias_s = reinterpret_cast<float*>(row_slot + kTileM);       // BIAS: [2][128], entry 63 + (tile row - tile key)
    const int dim = PADDED ? a.dim : D, vdim = PADDED ? a.vdim : DV;
    // the last rows of a prompt see the most keys: those tiles are scheduled first, the short ones fill the tail
    const int t0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kTileM, h = blockIdx.y;   // h: query unit (head, map)
    const int g = (h / a.maps) / (a.heads / a.kv_heads), ku = g * a.maps + h % a.maps;
    const int k_units = a.kv_heads * a.maps, q_units = a.heads * a.maps;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    const int rows = min(kTileM, a.n_tokens - t0);
    for (int r = threadIdx.x; r < kTileM; r += blockDim.x) {
        row_pos[r] = r < rows ? a.pos[t0 + r] : -1;
        row_slot[r] = r < rows ? a.slot[t0 + r] : -1;
    }
    const bf* Q = reinterpret_cast<const bf*>(a.q);
    for (int i = threadIdx.x; i < kTileM * CH; i += blockDim.x) {
        const int r = i / CH, c = i % CH;
        Pack16 v{{0u, 0u, 0u, 0u}};
        if (r < rows && (!PADDED || c * 8 < dim)) v = ld16(Q + ((size_t)(t0 + r) * q_units + h) * dim + c * 8);
        st16(Qs + r * RS + c * 8, v);
    }
    __syncthreads();
    uint32_t qf[D / 16][4];
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
        pa_ldsm_x4(qf[ks], Qs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RS + ks * 16 + (lane >> 4) * 8);
    float o[DV / 8][4];
#pragma unroll
    for (int nt = 0; nt < DV / 8; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    const bool sig = !BIAS && a.sigmoid != 0;   // the host keeps sigmoid weights and caps away from the biased variants
    const float m0 = BIAS && a.sink ? a.sink[h / a.maps] : (a.denom_bias > 0.f || sig) ? 0.f : -1e30f, l0 = BIAS && a.sink ? 1.f : sig ? 1.f : a.denom_bias;
    const float* btab = BIAS && a.dist_bias ? a.dist_bias + (size_t)(h / a.maps) * a.dist_n : nullptr;
    const float far_bias = btab ? btab[a.dist_n - 1] : 0.f;
    float m_run[2] = {m0, m0}, l_run[2] = {l0, l0};
    const float hb = (sig && a.head_bias) ? a.head_bias[h / a.maps] : 0.f;
    const int r_lo = warp * 16 + gid, r_hi = r_lo + 8;
    const float sc_h = pa_scale(a, h / a.maps), scale_over_cap = a.softcap > 0.f ? sc_h / a.softcap : 0.f;
    const bf* Kp = reinterpret_cast<const bf*>(a.k_pool);
    const bf* Vp = reinterpret_cast<const bf*>(a.v_pool);

    for (int seg = 0; seg < rows;) {
        const int b = row_slot[seg];
        int seg_end = seg + 1;
        while (seg_end < rows && row_slot[seg_end] == b) ++seg_end;
        const int n_keys = row_pos[seg_end - 1] + 1;            // positions grow along an entry
        const int first_key = BLOCKS ? pa_first_key(a, row_pos[seg]) : 0;    // with a block mask the first row's block starts the walk
        const int* plist = a.pages + (size_t)b * a.max_pages;
        // this thread's two rows in this segment (last and first key each sees), and the keys any row of the warp sees
        const int p_lo = (r_lo >= seg && r_lo < seg_end) ? row_pos[r_lo] : -1;
        const int p_hi = (r_hi >= seg && r_hi < seg_end) ? row_pos[r_hi] : -1;
        const int f_lo = (BLOCKS && p_lo >= 0) ? pa_first_key(a, p_lo) : 0, f_hi = (BLOCKS && p_hi >= 0) ? pa_first_key(a, p_hi) : 0;
        const int w_first = max(seg, warp * 16), w_last = min(seg_end, warp * 16 + 16) - 1;
        const int warp_keys = w_last >= w_first ? row_pos[w_last] + 1 : 0;
        const int warp_first = (BLOCKS && w_last >= w_first) ? pa_first_key(a, row_pos[w_first]) : 0;
        const bool one_page = a.page_rows % kTileN == 0 && first_key % kTileN == 0;
        auto load_tile = [&](int k0, int buf) {
            bf* kd = Ks + buf * kTileN * RS;
            bf* vd = Vs + buf * kTileN * RSV;
            // a tile that lies inside one page (the usual page sizes, walks from a tile's edge) takes one lookup
            const size_t base = one_page ? (size_t)plist[k0 / a.page_rows] * a.page_rows + k0 % a.page_rows : 0;
            if constexpr (BIAS) {
                if (btab) {
                    const int dist = row_pos[seg] - seg - k0 + (int)threadIdx.x - 63;   // 128 threads, 127 distances
                    const uint32_t bdst = (uint32_t)__cvta_generic_to_shared(bias_s + buf * 128 + threadIdx.x);
                    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(bdst), "l"(btab + min(max(dist, 0), a.dist_n - 1)) : "memory");
                }
            }
            if constexpr (PADDED || (DV % D != 0)) {
                constexpr int CHV = DV / 8;
                for (int i = threadIdx.x; i < kTileN * CH; i += blockDim.x) {
                    const int kr = i / CH, c = i % CH, j = k0 + kr;
                    const bool ok = j < n_keys;
                    const size_t row = one_page ? base + kr : ok ? (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows : 0;
                    const uint32_t bytes = (ok && c * 8 < dim) ? 16u : 0u;
                    const int c0 = min(c * 8, dim - 8);
                    const uint32_t kdst = (uint32_t)__cvta_generic_to_shared(kd + kr * RS + c * 8);
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(kdst), "l"(Kp + (row * k_units + ku) * dim + c0), "r"(bytes) : "memory");
                }
                for (int i = threadIdx.x; i < kTileN * CHV; i += blockDim.x) {
                    const int kr = i / CHV, c = i % CHV, j = k0 + kr;
                    const bool ok = j < n_keys;
                    const size_t row = one_page ? base + kr : ok ? (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows : 0;
                    const uint32_t bytes = (ok && c * 8 < vdim) ? 16u : 0u;
                    const int c0 = min(c * 8, vdim - 8);
                    const uint32_t vdst = (uint32_t)__cvta_generic_to_shared(vd + kr * RSV + c * 8);
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(vdst), "l"(Vp + (row * a.kv_heads + g) * vdim + c0), "r"(bytes) : "memory");
                }
            } else   // a thread brings chunk c of key row kr, and the DV / D value chunks that go with it (one page lookup for all)
            for (int i = threadIdx.x; i < kTileN * CH; i += blockDim.x) {
                const int kr = i / CH, c = i % CH, j = k0 + kr;
                const bool ok = j < n_keys;
                const size_t row = one_page ? base + kr : ok ? (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows : 0;
                const uint32_t bytes = ok ? 16u : 0u;                 // beyond the sequence: zeros, nothing is read
                const uint32_t kdst = (uint32_t)__cvta_generic_to_shared(kd + kr * RS + c * 8);
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(kdst), "l"(Kp + (row * k_units + ku) * D + c * 8), "r"(bytes) : "memory");
#pragma unroll
                for (int e = 0; e < DV / D; ++e) {
                    const uint32_t vdst = (uint32_t)__cvta_generic_to_shared(vd + kr * RSV + (c + e * CH) * 8);
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(vdst), "l"(Vp + (row * a.kv_heads + g) * DV + (c + e * CH) * 8), "r"(bytes) : "memory");
                }
            }
            __syncwarp();   // lanes that left the loops one after another commit together: a group closed by
                            // part of a warp was seen not to cover the copies of the rest
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        __syncthreads();   // the buffers of the previous segment are no longer read
        load_tile(first_key, 0);
        int buf = 0;
        for (int k0 = first_key; k0 < n_keys; k0 += kTileN, buf ^= 1) {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();   // tile k0 has landed for everybody; the other buffer is no longer read
            if (k0 + kTileN < n_keys) load_tile(k0 + kTileN, buf ^ 1);
            if (k0 >= warp_keys || (BLOCKS && k0 + kTileN <= warp_first)) continue;   // nothing for this warp's rows in this tile (it keeps the barriers)
            const bf* Kb = Ks + buf * kTileN * RS;
            const bf* Vb = Vs + buf * kTileN * RSV;
            float s[kTileN / 8][4];
#pragma unroll
            for (int nt = 0; nt < kTileN / 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
            // k steps outside, key columns inside: consecutive MMAs feed different accumulators. One ldmatrix.x4 brings the
            // K fragments of two k steps: matrices (k 0-7 | 8-15 | 16-23 | 24-31) of 8 keys
#pragma unroll
            for (int ks = 0; ks < D / 16; ks += 2) {
                if (PADDED && ks * 16 >= dim) continue;
                uint32_t b4[kTileN / 8][4];
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt)
                    pa_ldsm_x4(b4[nt], Kb + (nt * 8 + (lane & 7)) * RS + (lane >> 3) * 8 + ks * 16);
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt) {
                    const uint32_t b0[2] = {b4[nt][0], b4[nt][1]};
                    pa_mma(s[nt], qf[ks], b0);
                }
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt) {
                    const uint32_t b1[2] = {b4[nt][2], b4[nt][3]};
                    pa_mma(s[nt], qf[ks + 1], b1);
                }
            }
            // cap * tanh(v / cap): when every score of this thread's tile is small against the cap (the usual case) the odd
            // series x - x^3/3 + 2x^5/15 - 17x^7/315 is exact to fp32 rounding below |x| = 0.25 and costs no special-function
            // unit; otherwise (t - 1) / (t + 1) with t = e^(2x) (absolute error ~1e-7 * cap)
            if (!BIAS && a.softcap > 0.f) {
                float big = 0.f;
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) { s[nt][e] *= scale_over_cap; big = fmaxf(big, fabsf(s[nt][e])); }
                if (__all_sync(0xffffffffu, big < 0.25f)) {
#pragma unroll
                    for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float x = s[nt][e], x2 = x * x;
                            s[nt][e] = a.softcap * x * fmaf(x2, fmaf(x2, fmaf(x2, -17.f / 315.f, 2.f / 15.f), -1.f / 3.f), 1.f);
                        }
                } else {
#pragma unroll
                    for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float t = __expf(fminf(fmaxf(2.f * s[nt][e], -30.f), 30.f));
                            s[nt][e] = a.softcap * __fdividef(t - 1.f, t + 1.f);
                        }
                }
            } else if (!BIAS || !btab) {
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[nt][e] *= sc_h;
            }
            if constexpr (BIAS) {
                if (btab) {
                    if (row_pos[seg] - (k0 + kTileN - 1) >= a.dist_n - 1) {   // every distance of the tile has the last value
#pragma unroll
                        for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                            for (int e = 0; e < 4; ++e) s[nt][e] = fmaf(s[nt][e], sc_h, far_bias);
                    } else {
                        const float* bl = bias_s + buf * 128 + 63 + r_lo - tig * 2;
#pragma unroll
                        for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                            for (int e = 0; e < 4; ++e) s[nt][e] = fmaf(s[nt][e], sc_h, bl[(e & 2) * 4 - nt * 8 - (e & 1)]);
                    }
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
            if (BIAS && !BLOCKS && __all_sync(0xffffffffu, k0 + kTileN - 1 <= min(p_lo, p_hi))) {   // every row sees the whole tile
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) mx[e >> 1] = fmaxf(mx[e >> 1], s[nt][e]);
            } else
#pragma unroll
            for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = k0 + nt * 8 + tig * 2 + (e & 1);
                    const float v = (j <= ((e & 2) ? p_hi : p_lo) && (!BLOCKS || j >= ((e & 2) ? f_hi : f_lo))) ? s[nt][e] : -INFINITY;
                    s[nt][e] = v;
                    mx[e >> 1] = fmaxf(mx[e >> 1], v);
                }
            if (sig) {   // weights that are not normalised over the keys: nothing runs along the row
#pragma unroll
                for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[nt][e] = s[nt][e] == -INFINITY ? 0.f : 1.f / (1.f + __expf(-(s[nt][e] + hb)));
            } else {
            float alpha[2];
#pragma unroll
            for (int hrow = 0; hrow < 2; ++hrow) {
                mx[hrow] = fmaxf(mx[hrow], __shfl_xor_sync(0xffffffffu, mx[hrow], 1));
                mx[hrow] = fmaxf(mx[hrow], __shfl_xor_sync(0xffffffffu, mx[hrow], 2));
                const float mn = fmaxf(m_run[hrow], mx[hrow]);   // finite: m starts at 0 (the sink) or at -1e30
                alpha[hrow] = __expf(m_run[hrow] - mn);
                m_run[hrow] = mn;
            }
            float sum[2] = {0.f, 0.f};
            constexpr float kLog2E = 1.4426950408889634f;
            const float ml[2] = {m_run[0] * kLog2E, m_run[1] * kLog2E};
#pragma unroll
            for (int nt = 0; nt < kTileN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    // masked: exp(-inf) = 0
                    const float pv = BIAS ? pa_exp2(fmaf(s[nt][e], kLog2E, -ml[e >> 1])) : __expf(s[nt][e] - m_run[e >> 1]);
                    s[nt][e] = pv;
                    sum[e >> 1] += pv;
                }
#pragma unroll
            for (int hrow = 0; hrow < 2; ++hrow) {
                sum[hrow] += __shfl_xor_sync(0xffffffffu, sum[hrow], 1);
                sum[hrow] += __shfl_xor_sync(0xffffffffu, sum[hrow], 2);
                l_run[hrow] = l_run[hrow] * alpha[hrow] + sum[hrow];
            }
#pragma unroll
            for (int nt = 0; nt < DV / 8; ++nt) { o[nt][0] *= alpha[0]; o[nt][1] *= alpha[0]; o[nt][2] *= alpha[1]; o[nt][3] *= alpha[1]; }
            }
#pragma unroll
            for (int kk = 0; kk < kTileN / 16; ++kk) {
                uint32_t pf[4];
                pf[0] = pa_pack(s[2 * kk][0], s[2 * kk][1]);
                pf[1] = pa_pack(s[2 * kk][2], s[2 * kk][3]);
                pf[2] = pa_pack(s[2 * kk + 1][0], s[2 * kk + 1][1]);
                pf[3] = pa_pack(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
                for (int nt = 0; nt < DV / 8; nt += 2) {
                    if (PADDED && nt * 8 >= vdim) continue;
                    // one transposed ldmatrix.x4: the V fragments of two column tiles
                    uint32_t b4[4];
                    pa_ldsm_x4_trans(b4, Vb + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RSV + (nt + (lane >> 4)) * 8);
                    const uint32_t b0[2] = {b4[0], b4[1]}, b1[2] = {b4[2], b4[3]};
                    pa_mma(o[nt], pf, b0);
                    pa_mma(o[nt + 1], pf, b1);
                }
            }
        }
        seg = seg_end;
    }
#pragma unroll
    for (int hrow = 0; hrow < 2; ++hrow) {
        const int r = hrow ? r_hi : r_lo;
        if (r >= rows) continue;
        const float inv = 1.0f / l_run[hrow];
        const size_t dst = ((size_t)(t0 + r) * q_units + h) * vdim + tig * 2;
        if (a.out_f32) {
#pragma unroll
            for (int nt = 0; nt < DV / 8; ++nt)
                if (!PADDED || nt * 8 < vdim) *reinterpret_cast<float2*>(reinterpret_cast<float*>(a.out) + dst + nt * 8) = make_float2(o[nt][hrow * 2] * inv, o[nt][hrow * 2 + 1] * inv);
        } else {
#pragma unroll
            for (int nt = 0; nt < DV / 8; ++nt)
                if (!PADDED || nt * 8 < vdim) *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf*>(a.out) + dst + nt * 8) = __floats2bfloat162_rn(o[nt][hrow * 2] * inv, o[nt][hrow * 2 + 1] * inv);
        }
    }
}

template <int D, int DV, int KIND, bool MASKED = true>   // MASKED: the block-mask / window variant is built too
static int launch_tile(const PA& a, cudaStream_t s) {
    static_assert(kTileM == kTileN, "the Q tile borrows a K buffer");
    constexpr int smem = 2 * kTileN * (D + 8) * 2 + 2 * kTileN * (DV + 8) * 2 + 2 * kTileM * 4 + (KIND != kNoBias ? 2 * 128 * 4 : 0);
    static unsigned long long done = 0;
    static_assert(KIND != kNoBias || DV % D == 0, "a thread brings DV / D value chunks with every key chunk");
    const dim3 grid((a.n_tokens + kTileM - 1) / kTileM, a.heads * a.maps);
    if constexpr (MASKED) if (a.chunk > 0 || a.window > 0) {
        static unsigned long long done_b = 0;
        const cudaError_t e = ensure_max_dynamic_smem((const void*)paged_attn_tile_kernel<D, DV, true, KIND>, smem, done_b);
        if (e != cudaSuccess) return (int)e;
        paged_attn_tile_kernel<D, DV, true, KIND><<<grid, 128, smem, s>>>(a);
        return (int)cudaGetLastError();
    }
    const cudaError_t e = ensure_max_dynamic_smem((const void*)paged_attn_tile_kernel<D, DV, false, KIND>, smem, done);
    if (e != cudaSuccess) return (int)e;
    paged_attn_tile_kernel<D, DV, false, KIND><<<grid, 128, smem, s>>>(a);
    return (int)cudaGetLastError();
}

}  // namespace b200
