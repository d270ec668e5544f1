// b200_paged_attention: causal attention over paged per-head keys and values with grouped query heads, a tanh cap on
// the scores and a constant added to the softmax denominator (a sink of score 0 that owns no value). Prompt portions,
// single decoded tokens and mixed batches run through the same launch: every token carries its sequence slot and
// position, and only sees its own sequence's pages. Two more masks and layouts are arguments: a block mask (a position
// only sees the keys of its own block of `chunk` positions) and several score maps per head over shared values (`maps`:
// query unit (h, m) scores against key unit (h / group, m) and weights the values of key head h / group). A sliding window
// (a position sees itself and the window - 1 positions before it) is a third mask, and the weights can be sigmoids of the
// score plus a number per head instead of a softmax: then nothing is normalised over the keys, which in the running
// (maximum, denominator, output) form is a maximum held at 0 and a denominator held at 1.
//
// A learned number per head and distance can be added to the scaled scores, and a head's sink can have a learned score.
// Scores can carry a factor per head; weights that are mixed across heads before they meet the values are the business of
// mixed_attention.cu.
//
//   paged_attn_row_kernel   one CTA per (token, query head), fp32 arithmetic on caches of either dtype: each warp
//                           takes blocks of 32 keys (a lane scores one key; the weighted value sum runs with a lane per
//                           output column), keeps its own running maximum / denominator / output and the warps merge at
//                           the end. The sink is the initial state of warp 0 (m = 0, l = denom_bias; or the head's own score, 1).
//   paged_attn_tile_kernel  bfloat16 prompt portions on mma.sync tiles (further down).
#include <cuda_bf16.h>
#include <math.h>
#include <stdlib.h>

#include <algorithm>

#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"
#include "paged_attention_tile.cuh"

namespace b200 {

__device__ __forceinline__ float pa_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
constexpr int kRowWarps = 4;
constexpr int kMaxSplits = 16;
constexpr int kMaxVPerLane = 8;   // vdim <= 256

template <typename T>
__device__ __forceinline__ float dot_row(const float* q, const T* k, int dim) {
    float acc = 0.f;
    if ((dim % DT<T>::kPer16B) == 0 && (reinterpret_cast<uintptr_t>(k) & 15u) == 0) {
        for (int i = 0; i < dim; i += DT<T>::kPer16B) {
            float f[DT<T>::kPer16B];
            const Pack16 pk = ld16(k + i);
            if constexpr (sizeof(T) == 4) {
#pragma unroll
                for (int e = 0; e < 4; ++e) f[e] = __uint_as_float(pk.w[e]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&pk.w[e]));
                    f[2 * e] = v.x;
                    f[2 * e + 1] = v.y;
                }
            }
#pragma unroll
            for (int e = 0; e < DT<T>::kPer16B; ++e) acc = fmaf(q[i + e], f[e], acc);
        }
    } else {
        for (int i = 0; i < dim; ++i) acc = fmaf(q[i], DT<T>::to_f(k[i]), acc);
    }
    return acc;
}

template <typename T>
__global__ void __launch_bounds__(kRowWarps * 32) paged_attn_row_kernel(const PA a) {
    extern __shared__ float sm[];
    float* qs = sm;                                   // [dim]
    float* om = sm + a.dim;                           // [kRowWarps][vdim]
    __shared__ float ms[kRowWarps], ls[kRowWarps];
    // h counts query units (head, map); ku is the key unit it scores against, g the key head whose values it weights
    const int t = blockIdx.x, h = blockIdx.y, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int g = (h / a.maps) / (a.heads / a.kv_heads), ku = g * a.maps + h % a.maps, p = a.pos[t];
    const int k_units = a.kv_heads * a.maps, q_units = a.heads * a.maps;
    const int* plist = a.pages + (size_t)a.slot[t] * a.max_pages;
    const T* q = reinterpret_cast<const T*>(a.q) + ((size_t)t * q_units + h) * a.dim;
    for (int i = threadIdx.x; i < a.dim; i += blockDim.x) qs[i] = DT<T>::to_f(q[i]);
    __syncthreads();
    const T* K = reinterpret_cast<const T*>(a.k_pool);
    const T* V = reinterpret_cast<const T*>(a.v_pool);
    float m = -INFINITY, l = 0.f, o[kMaxVPerLane];
#pragma unroll
    for (int c = 0; c < kMaxVPerLane; ++c) o[c] = 0.f;
    // this CTA's share of the keys: whole blocks of 32, the sink with the first share
    const int j_lo = pa_first_key(a, p);
    const int per = ((p - j_lo + a.splits) / a.splits + 31) & ~31;
    const int j_begin = j_lo + blockIdx.z * per, j_end = min(p + 1, j_begin + per);
    if (warp == 0 && blockIdx.z == 0) {
        if (a.sink) { m = a.sink[h / a.maps]; l = 1.f; }
        else if (a.denom_bias > 0.f) { m = 0.f; l = a.denom_bias; }
    }
    const float hb = (a.sigmoid && a.head_bias) ? a.head_bias[h / a.maps] : 0.f, sc_h = pa_scale(a, h / a.maps);
    if (a.sigmoid) { m = 0.f; l = (warp == 0 && blockIdx.z == 0) ? 1.f : 0.f; }
    for (int j0 = j_begin + warp * 32; j0 < j_end; j0 += kRowWarps * 32) {
        const int j = j0 + lane;
        const bool ok = j < j_end;
        size_t row = 0;   // the key's row in the page pool
        float s = -INFINITY;
        if (ok) {
            row = (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows;
            s = dot_row<T>(qs, K + (row * k_units + ku) * a.dim, a.dim) * sc_h;
            if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
            s += pa_dist_bias(a, h / a.maps, p - j);
        }
        float bm = s;
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, d));
        const float mn = a.sigmoid ? 0.f : fmaxf(m, bm);
        const float corr = expf(m - mn);   // m = -inf: 0
        const float pj = !ok ? 0.f : a.sigmoid ? pa_sigmoid(s + hb) : expf(s - mn);
        float ps = a.sigmoid ? 0.f : pj;
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, d);
        l = l * corr + ps;
        m = mn;
#pragma unroll
        for (int c = 0; c < kMaxVPerLane; ++c) o[c] *= corr;
        const int n = min(32, j_end - j0);
        for (int kk = 0; kk < n; ++kk) {
            const float pk = __shfl_sync(0xffffffffu, pj, kk);
            const size_t r = __shfl_sync(0xffffffffu, (unsigned long long)row, kk);
            const T* vr = V + (r * a.kv_heads + g) * a.vdim;
#pragma unroll
            for (int c = 0; c < kMaxVPerLane; ++c)
                if (lane + 32 * c < a.vdim) o[c] = fmaf(pk, DT<T>::to_f(vr[lane + 32 * c]), o[c]);
        }
    }
    if (lane == 0) { ms[warp] = m; ls[warp] = l; }
#pragma unroll
    for (int c = 0; c < kMaxVPerLane; ++c)
        if (lane + 32 * c < a.vdim) om[warp * a.vdim + lane + 32 * c] = o[c];
    __syncthreads();
    float M = ms[0];
    for (int w = 1; w < kRowWarps; ++w) M = fmaxf(M, ms[w]);
    float L = 0.f;
    for (int w = 0; w < kRowWarps; ++w) L += M == -INFINITY ? 0.f : ls[w] * expf(ms[w] - M);
    if (a.splits > 1) {   // an unnormalised share: (m, l, o); an empty share is (-inf, 0, 0)
        float* pr = a.part + (((size_t)t * q_units + h) * a.splits + blockIdx.z) * (a.vdim + 2);
        if (threadIdx.x == 0) { pr[0] = M; pr[1] = L; }
        for (int c = threadIdx.x; c < a.vdim; c += blockDim.x) {
            float v = 0.f;
            for (int w = 0; w < kRowWarps; ++w) v += M == -INFINITY ? 0.f : om[w * a.vdim + c] * expf(ms[w] - M);
            pr[2 + c] = v;
        }
        return;
    }
    const size_t dst = ((size_t)t * q_units + h) * a.vdim;
    for (int c = threadIdx.x; c < a.vdim; c += blockDim.x) {
        float v = 0.f;
        for (int w = 0; w < kRowWarps; ++w) v += om[w * a.vdim + c] * expf(ms[w] - M);
        pa_store<T>(a, dst + c, v / L);
    }
}

// Decode batches (few rows, long contexts): one CTA per (token, key head, share of the context) serves ALL query heads of
// the group from one pass over the keys and values. Eight lanes share a key row (16-byte loads, a row is read once,
// whole sectors), four keys per warp step; the scores of 32 keys go through shared memory to the softmax (a lane per
// key) and on to the weighted value sum (a lane per pair of output columns). fp32 arithmetic on caches of either dtype.
template <typename T, int R>   // R query heads per key head
__global__ void __launch_bounds__(kRowWarps * 32) paged_attn_group_kernel(const PA a) {
    extern __shared__ float sm[];
    float* qs = sm;                                        // [R][dim]
    float* sc = qs + R * a.dim;                            // [warps][R][32]
    float* om = sc + kRowWarps * R * 32;                   // [warps][R][vdim]
    __shared__ float ms[kRowWarps][R], ls[kRowWarps][R];
    __shared__ unsigned long long rows[kRowWarps][32];
    // blockIdx.y counts key units (key head g, map mp); query head g * R + r holds its map mp at unit (g * R + r) * maps + mp
    const int t = blockIdx.x, ku = blockIdx.y, g = ku / a.maps, mp = ku % a.maps, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int p = a.pos[t], dim = a.dim, vdim = a.vdim, k_units = a.kv_heads * a.maps, q_units = a.heads * a.maps;
    const int* plist = a.pages + (size_t)a.slot[t] * a.max_pages;
    const T* q = reinterpret_cast<const T*>(a.q) + (size_t)t * q_units * dim;
    for (int i = threadIdx.x; i < R * dim; i += blockDim.x) qs[i] = DT<T>::to_f(q[(size_t)((g * R + i / dim) * a.maps + mp) * dim + i % dim]);
    __syncthreads();
    const T* K = reinterpret_cast<const T*>(a.k_pool);
    const T* V = reinterpret_cast<const T*>(a.v_pool);
    float m[R], l[R], o[R][4][2];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const bool first = warp == 0 && blockIdx.z == 0, sink = first && a.denom_bias > 0.f;
        m[r] = (sink || a.sigmoid) ? 0.f : -INFINITY;
        l[r] = sink ? a.denom_bias : (a.sigmoid && first) ? 1.f : 0.f;
        if (a.sink && first) { m[r] = a.sink[g * R + r]; l[r] = 1.f; }
#pragma unroll
        for (int c = 0; c < 4; ++c) o[r][c][0] = o[r][c][1] = 0.f;
    }
    const int j_lo = pa_first_key(a, p);
    const int per = ((p - j_lo + a.splits) / a.splits + 31) & ~31;
    const int j_begin = j_lo + blockIdx.z * per, j_end = min(p + 1, j_begin + per);
    float* scw = sc + warp * R * 32;
    const int l8 = lane & 7;
    for (int j0 = j_begin + warp * 32; j0 < j_end; j0 += kRowWarps * 32) {
#pragma unroll
        for (int it = 0; it < 8; ++it) {   // scores of keys j0 + 4 it + (lane / 8); unrolled: the loads of all steps are in flight together
            const int kk = it * 4 + (lane >> 3), j = j0 + kk;
            float acc[R];
#pragma unroll
            for (int r = 0; r < R; ++r) acc[r] = 0.f;
            size_t row = 0;
            if (j < j_end) {
                row = (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows;
                const T* kr = K + (row * k_units + ku) * dim;
                for (int i = l8 * 8; i < dim; i += 64) {
                    float f[8];
                    if constexpr (sizeof(T) == 2) {   // eight bfloat16 in one 16-byte load
                        const Pack16 pk = ld16(kr + i);
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&pk.w[e]));
                            f[2 * e] = v.x;
                            f[2 * e + 1] = v.y;
                        }
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; e += 4) {
                            const Pack16 pk = ld16(kr + i + e);
#pragma unroll
                            for (int x = 0; x < 4; ++x) f[e + x] = __uint_as_float(pk.w[x]);
                        }
                    }
#pragma unroll
                    for (int r = 0; r < R; ++r)
#pragma unroll
                        for (int e = 0; e < 8; ++e) acc[r] = fmaf(qs[r * dim + i + e], f[e], acc[r]);
                }
            }
#pragma unroll
            for (int r = 0; r < R; ++r) {
                acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 1);
                acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 2);
                acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 4);
            }
            if (l8 == 0) {
                rows[warp][kk] = row;
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    float sv = acc[r] * pa_scale(a, g * R + r);
                    if (a.softcap > 0.f) sv = a.softcap * tanhf(sv / a.softcap);
                    if (a.dist_bias && j < j_end) sv += pa_dist_bias(a, g * R + r, p - j);
                    scw[r * 32 + kk] = j < j_end ? sv : -INFINITY;
                }
            }
        }
        __syncwarp();
#pragma unroll
        for (int r = 0; r < R; ++r) {   // softmax step, a lane per key
            const float sv = scw[r * 32 + lane];
            float bm = sv;
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, d));
            const float mn = a.sigmoid ? 0.f : fmaxf(m[r], bm);          // finite: the block holds at least one key
            const float corr = expf(m[r] - mn);
            // a masked key: exp(-inf) = 0
            const float pj = !a.sigmoid ? expf(sv - mn) : sv == -INFINITY ? 0.f : pa_sigmoid(sv + (a.head_bias ? a.head_bias[g * R + r] : 0.f));
            float ps = a.sigmoid ? 0.f : pj;
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, d);
            l[r] = l[r] * corr + ps;
            m[r] = mn;
#pragma unroll
            for (int c = 0; c < 4; ++c) { o[r][c][0] *= corr; o[r][c][1] *= corr; }
            scw[r * 32 + lane] = pj;
        }
        __syncwarp();
        const int n = min(32, j_end - j0);
#pragma unroll 4
        for (int kk = 0; kk < n; ++kk) {   // weighted values, a lane per pair of columns
            const T* vr = V + (rows[warp][kk] * a.kv_heads + g) * vdim;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int col = 2 * lane + 64 * c;
                if (col < vdim) {
                    const float2 v = Pair<T>::load(vr + col);
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        const float pk = scw[r * 32 + kk];
                        o[r][c][0] = fmaf(pk, v.x, o[r][c][0]);
                        o[r][c][1] = fmaf(pk, v.y, o[r][c][1]);
                    }
                }
            }
        }
        __syncwarp();
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (lane == 0) { ms[warp][r] = m[r]; ls[warp][r] = l[r]; }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int col = 2 * lane + 64 * c;
            if (col < vdim) { om[(warp * R + r) * vdim + col] = o[r][c][0]; om[(warp * R + r) * vdim + col + 1] = o[r][c][1]; }
        }
    }
    __syncthreads();
    for (int r = 0; r < R; ++r) {
        const int h = (g * R + r) * a.maps + mp;   // query unit
        float M = ms[0][r];
        for (int w = 1; w < kRowWarps; ++w) M = fmaxf(M, ms[w][r]);
        float L = 0.f;
        for (int w = 0; w < kRowWarps; ++w) L += M == -INFINITY ? 0.f : ls[w][r] * expf(ms[w][r] - M);
        float* pr = a.splits > 1 ? a.part + (((size_t)t * q_units + h) * a.splits + blockIdx.z) * (vdim + 2) : nullptr;
        if (pr && threadIdx.x == 0) { pr[0] = M; pr[1] = L; }
        const size_t dst = ((size_t)t * q_units + h) * vdim;
        for (int c = threadIdx.x; c < vdim; c += blockDim.x) {
            float v = 0.f;
            for (int w = 0; w < kRowWarps; ++w) v += M == -INFINITY ? 0.f : om[(w * R + r) * vdim + c] * expf(ms[w][r] - M);
            if (pr) pr[2 + c] = v;
            else pa_store<T>(a, dst + c, v / L);
        }
    }
}

template <typename T>
static bool launch_group(const PA& a, dim3 grid, cudaStream_t s) {
    const int R = a.heads / a.kv_heads;
    const size_t smem = ((size_t)R * a.dim + (size_t)kRowWarps * R * 32 + (size_t)kRowWarps * R * a.vdim) * sizeof(float);
    if (smem > 48 * 1024) return false;
    switch (R) {
        case 1: paged_attn_group_kernel<T, 1><<<grid, kRowWarps * 32, smem, s>>>(a); return true;
        case 2: paged_attn_group_kernel<T, 2><<<grid, kRowWarps * 32, smem, s>>>(a); return true;
        case 4: paged_attn_group_kernel<T, 4><<<grid, kRowWarps * 32, smem, s>>>(a); return true;
        case 8: paged_attn_group_kernel<T, 8><<<grid, kRowWarps * 32, smem, s>>>(a); return true;
    }
    return false;
}

// merges the shares of split contexts: one CTA per (token, head)
template <typename T>
__global__ void __launch_bounds__(128) paged_attn_combine_kernel(const float* __restrict__ part, T* __restrict__ out, int splits, int vdim) {
    const float* pr = part + (size_t)blockIdx.x * splits * (vdim + 2);
    float M = -INFINITY;
    for (int z = 0; z < splits; ++z) M = fmaxf(M, pr[(size_t)z * (vdim + 2)]);
    float L = 0.f, wz[kMaxSplits];
    for (int z = 0; z < splits; ++z) {
        const float mz = pr[(size_t)z * (vdim + 2)];
        wz[z] = mz == -INFINITY ? 0.f : expf(mz - M);
        L += pr[(size_t)z * (vdim + 2) + 1] * wz[z];
    }
    for (int c = threadIdx.x; c < vdim; c += blockDim.x) {
        float v = 0.f;
        for (int z = 0; z < splits; ++z) v += pr[(size_t)z * (vdim + 2) + 2 + c] * wz[z];
        out[(size_t)blockIdx.x * vdim + c] = DT<T>::from_f(v / L);
    }
}

// the (dim, vdim) pairs the tile kernel is built for: equal sizes, and values twice as wide as the keys
static int launch_tile_for(const PA& a, cudaStream_t s) {
    if (a.dim == a.vdim) return a.dim == 128 ? launch_tile<128, 128, kNoBias>(a, s) : a.dim == 64 ? launch_tile<64, 64, kNoBias>(a, s) : a.dim == 32 ? launch_tile<32, 32, kNoBias>(a, s) : -1;
    if (a.vdim == 2 * a.dim) return a.dim == 128 ? launch_tile<128, 256, kNoBias>(a, s) : a.dim == 64 ? launch_tile<64, 128, kNoBias>(a, s) : a.dim == 32 ? launch_tile<32, 64, kNoBias>(a, s) : -1;
    return -1;
}

}  // namespace b200

using namespace b200;

extern "C" size_t b200_paged_attention_workspace_bytes(int n_tokens, int heads, int vdim) {
    if (n_tokens < 1 || heads < 1 || vdim < 1 || (long long)n_tokens * heads >= 2 * sm_count()) return 0;
    return (size_t)n_tokens * heads * kMaxSplits * (vdim + 2) * sizeof(float);
}

extern "C" int b200_paged_attention(const b200_paged_attention_args* p, void* stream) {
    if (!p || !p->q || !p->out || !p->k_pool || !p->v_pool || !p->pages || !p->slot || !p->pos || p->n_tokens < 0 || p->heads < 1 ||
        p->kv_heads < 1 || p->heads % p->kv_heads || p->dim < 1 || p->vdim < 1 || p->page_rows < 1 || p->denom_bias < 0.f ||
        p->chunk < 0 || p->maps < 0 || p->window < 0)
        return B200_EINVAL;
    if (p->sigmoid_weights && (p->softcap > 0.f || p->denom_bias > 0.f || p->maps > 1)) return B200_EINVAL;
    if (p->head_mix && (p->softcap > 0.f || p->denom_bias > 0.f || p->sigmoid_weights || p->maps > 1)) return B200_EINVAL;
    if ((p->sink || p->dist_bias) && (p->sigmoid_weights || p->head_mix || (p->dist_bias && p->dist_n < 1) || (p->sink && p->denom_bias > 0.f))) return B200_EINVAL;
    const int maps = p->maps > 0 ? p->maps : 1, units = p->heads * maps;
    if (!p->head_mix && p->vdim > 32 * kMaxVPerLane) return B200_EUNSUPPORTED;
    if (p->n_tokens == 0) return B200_OK;
    PA a{p->q, p->out, p->k_pool, p->v_pool, p->pages, p->max_pages, p->page_rows, p->slot, p->pos, p->n_tokens, p->heads,
         p->kv_heads, p->dim, p->vdim, p->scale, p->softcap, p->denom_bias, 1, nullptr, p->chunk, maps, p->out_f32,
         p->window, p->sigmoid_weights != 0, p->head_bias, p->head_temp, p->head_mix, p->sink, p->dist_bias, p->dist_n};
    cudaStream_t s = (cudaStream_t)stream;
    if (p->head_mix) return mixed_attention(a, p->dtype, p->longest_entry, p->longest_context, p->workspace, p->workspace_bytes, s);
    const size_t smem = ((size_t)p->dim + (size_t)kRowWarps * p->vdim) * sizeof(float);
    if (smem > 48 * 1024) return B200_EUNSUPPORTED;
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    const char* env = getenv("B200_ATTN_ROWS");   // 1: every batch on the row kernel (debugging aid)
    if (p->dtype == B200_BF16 && p->longest_entry != 1 && (p->sink || p->dist_bias) && !(p->softcap > 0.f) && p->dim % 8 == 0 && p->vdim % 8 == 0 && al16(p->q) && al16(p->out) &&
        al16(p->k_pool) && al16(p->v_pool) && !(env && env[0] == '1')) {
        const int rc = biased_tile(a, s);
        if (rc == 0) count_launch();
        if (rc >= 0) return rc;
    }
    if (p->dtype == B200_BF16 && p->longest_entry != 1 && !p->sink && !p->dist_bias && (p->dim == p->vdim || p->vdim == 2 * p->dim) &&
        (p->dim == 64 || p->dim == 128 || p->dim == 32) && al16(p->q) && al16(p->out) && al16(p->k_pool) && al16(p->v_pool) &&
        !(env && env[0] == '1')) {
        const int rc = launch_tile_for(a, s);
        if (rc == 0) count_launch();
        if (rc >= 0) return rc;
    }
    // single tokens whose heads come in groups of 1, 2, 4 or 8 per key head: one pass over K / V serves the whole group
    const int R = p->heads / p->kv_heads;
    const bool group = p->longest_entry == 1 && (R == 1 || R == 2 || R == 4 || R == 8) && p->dim % 8 == 0 && p->vdim % 2 == 0 &&
                       al16(p->k_pool) && al16(p->v_pool) && !(env && env[0] == '1') &&
                       ((size_t)R * p->dim + (size_t)kRowWarps * R * (32 + p->vdim)) * sizeof(float) <= 48 * 1024;
    const long long ctas = (long long)p->n_tokens * (group ? p->kv_heads * maps : units);
    // few rows with long contexts (decode batches): split every context over several CTAs and merge the shares
    int longest_seen = p->chunk > 0 ? std::min(p->longest_context, p->chunk) : p->longest_context;
    if (p->window > 0) longest_seen = std::min(longest_seen, p->window);
    if (longest_seen > 256 && p->workspace && (long long)p->n_tokens * units < 2 * sm_count()) {
        int splits = (int)((4ll * sm_count() + ctas - 1) / ctas);
        splits = std::min(std::min(splits, kMaxSplits), (longest_seen + 127) / 128);
        if (splits > 1 && p->workspace_bytes >= (size_t)p->n_tokens * units * splits * (p->vdim + 2) * sizeof(float)) {
            a.splits = splits;
            a.part = reinterpret_cast<float*>(p->workspace);
        }
    }
    const dim3 grid3(p->n_tokens, units, a.splits);
    bool done = false;
    if (group) {
        const dim3 gridg(p->n_tokens, p->kv_heads * maps, a.splits);
        done = p->dtype == B200_BF16 ? launch_group<__nv_bfloat16>(a, gridg, s) : p->dtype == B200_F32 ? launch_group<float>(a, gridg, s) : false;
    }
    if (done) {
    } else if (p->dtype == B200_BF16) paged_attn_row_kernel<__nv_bfloat16><<<grid3, kRowWarps * 32, smem, s>>>(a);
    else if (p->dtype == B200_F32) paged_attn_row_kernel<float><<<grid3, kRowWarps * 32, smem, s>>>(a);
    else return B200_EINVAL;
    count_launch();
    if (a.splits > 1) {
        if (p->dtype == B200_BF16 && !p->out_f32) paged_attn_combine_kernel<__nv_bfloat16><<<p->n_tokens * units, 128, 0, s>>>(a.part, (__nv_bfloat16*)p->out, a.splits, p->vdim);
        else paged_attn_combine_kernel<float><<<p->n_tokens * units, 128, 0, s>>>(a.part, (float*)p->out, a.splits, p->vdim);
        count_launch();
    }
    return (int)cudaGetLastError();
}
