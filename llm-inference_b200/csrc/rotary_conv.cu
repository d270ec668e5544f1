// Between the q / k projection and the cache of an attention layer: rotary angles of a step (double-precision angle,
// one table per frequency set), the short causal convolution over time with its carried inputs, the per-head RMS norm,
// the rotation in either pairing, and the store of q, k (and of the convolved keys as values) — b200_qk_prepare — plus
// the update of the convolution's ring of carried inputs. All arithmetic fp32; only the stores take the serving dtype.
#include <cuda_bf16.h>

#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"
#include "rotary.cuh"

namespace b200 {

__global__ void rope_angles_kernel(const int* __restrict__ pos, const double* __restrict__ freq, int n_freq, int total,
                                   double amplitude, float* __restrict__ cos_out, float* __restrict__ sin_out) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const double a = (double)pos[i / n_freq] * freq[i % n_freq];
    double s, c;
    sincos(a, &s, &c);
    cos_out[i] = (float)(amplitude * c);
    sin_out[i] = (float)(amplitude * s);
}

struct QkPrep {
    const float* proj; long long ld_proj;
    const float* conv_w; int taps; const float* conv_state;
    const float* q_norm; const float* k_norm; float eps;
    const float* cos; const float* sin; int rot_dims, rot_layout;
    void* q_out; void* k_pool; void* v_pool; int v_from_conv;
    float* ring_out;   // non-NULL: every entry of the batch is one token, and the warp files its own inputs in the ring
    const int* pages; int max_pages, page_rows;
    const int* slot; const int* pos; const int* start;
    int heads, kv_heads, dim;
    int v_heads, vdim; long long v_off;
    const float* bias; const float* v_cos; const float* v_sin; int v_layout;
    int vals_per_warp;   // floats of shared memory per warp: max(dim, vdim)
    float temp_coef; int temp_every;
};

// what the queries of position p are multiplied by
__device__ __forceinline__ float query_temp(const QkPrep& a, int p) {
    return a.temp_every > 0 ? 1.f + a.temp_coef * logf((float)((p + 1) / a.temp_every + 1)) : 1.f;
}

// One warp per (token, head unit): units [0, heads) are query heads, [heads, heads + kv_heads) key heads; a lane owns the
// dimensions lane, lane + 32, ... (coalesced loads and stores); the head's sum of squares is a warp reduction and the
// rotation reads its partner through the warp's slice of shared memory, so no CTA-wide barrier is needed.
constexpr int kPrepWarps = 4, kMaxTapsUnrolled = 4;   // longer filters take the plain loop
template <typename T>
__global__ void __launch_bounds__(kPrepWarps * 32) qk_prepare_kernel(const QkPrep a, int n_units) {
    extern __shared__ float prep_sm[];
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, dim = a.dim;
    const int unit = blockIdx.x * kPrepWarps + warp, per_token = a.heads + a.kv_heads;
    if (unit >= n_units) return;
    float* vals = prep_sm + warp * a.vals_per_warp;   // the normed head before rotation
    const int t = unit / (per_token + a.v_heads), u = unit % (per_token + a.v_heads);
    if (u >= per_token) {   // a projected value head: to its cache row, with its bias and turned by its own position if asked
        const int g = u - per_token, pv = a.pos[t];
        const size_t vrow = ((size_t)a.pages[(size_t)a.slot[t] * a.max_pages + pv / a.page_rows] * a.page_rows + pv % a.page_rows) * a.v_heads + g;
        const size_t col0 = (size_t)a.v_off + (size_t)g * a.vdim;
        const float* src = a.proj + (size_t)t * a.ld_proj + col0;
        T* vd = reinterpret_cast<T*>(a.v_pool) + vrow * a.vdim;
        if (!a.v_cos) {
            for (int i = lane; i < a.vdim; i += 32) vd[i] = DT<T>::from_f(src[i] + (a.bias ? a.bias[col0 + i] : 0.f));
            return;
        }
        for (int i = lane; i < a.vdim; i += 32) vals[i] = src[i] + (a.bias ? a.bias[col0 + i] : 0.f);
        __syncwarp();
        const int vf = a.vdim / 2;
        for (int i = lane; i < a.vdim; i += 32)
            vd[i] = DT<T>::from_f(rotary_component(vals, i, 2 * vf, a.v_layout, a.v_cos + (size_t)t * vf, a.v_sin + (size_t)t * vf));
        return;
    }
    const bool is_k = u >= a.heads;
    const int ch0 = u * dim;          // first channel of this head in [q channels | k channels]
    const int channels = per_token * dim;
    const int p = a.pos[t], b = a.slot[t];
    size_t cache_row = 0;
    if (is_k) cache_row = ((size_t)a.pages[(size_t)b * a.max_pages + p / a.page_rows] * a.page_rows + p % a.page_rows) * a.kv_heads + (u - a.heads);
    const int first = a.conv_w ? a.start[t] : 0, taps = a.taps;
    float ss = 0.f;
    if (a.conv_w && taps <= kMaxTapsUnrolled) {
        // The rows that hold the taps' inputs (this step's batch, the slot's ring, or nothing before position 0) are found
        // once per warp; then four dimensions per lane and all their taps at once: every load of the group is in flight
        // before the first sum. A four-tap filter is one 16-byte load per channel.
        const float* rows[kMaxTapsUnrolled];
        bool ok[kMaxTapsUnrolled];
#pragma unroll
        for (int j = 0; j < kMaxTapsUnrolled; ++j) {
            const int back = taps - 1 - j, src = p - back;
            ok[j] = j < taps && src >= 0;
            rows[j] = !ok[j] ? a.proj
                      : src >= first ? a.proj + (size_t)(t - back) * a.ld_proj + ch0
                                     : a.conv_state + ((size_t)b * (taps - 1) + src % (taps - 1)) * channels + ch0;
        }
        const float* cw = a.conv_w + (size_t)ch0 * taps;
        const bool w4 = taps == 4 && (reinterpret_cast<uintptr_t>(a.conv_w) & 15u) == 0;
        float* ring = (a.ring_out && taps > 1) ? a.ring_out + ((size_t)b * (taps - 1) + p % (taps - 1)) * channels + ch0 : nullptr;
        T* vdst = (is_k && a.v_from_conv) ? reinterpret_cast<T*>(a.v_pool) + cache_row * dim : nullptr;
        for (int i0 = lane; i0 < dim; i0 += 128) {
            float xin[4][kMaxTapsUnrolled], w[4][kMaxTapsUnrolled];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int i = i0 + 32 * k;
                const bool in = i < dim;
#pragma unroll
                for (int j = 0; j < kMaxTapsUnrolled; ++j) xin[k][j] = in && ok[j] ? rows[j][i] : 0.f;
                if (w4) {
                    const float4 w4v = in ? *reinterpret_cast<const float4*>(cw + (size_t)i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
                    w[k][0] = w4v.x; w[k][1] = w4v.y; w[k][2] = w4v.z; w[k][3] = w4v.w;
                } else {
#pragma unroll
                    for (int j = 0; j < kMaxTapsUnrolled; ++j) w[k][j] = in && j < taps ? cw[(size_t)i * taps + j] : 0.f;
                }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int i = i0 + 32 * k;
                if (i >= dim) continue;
                float y = 0.f;
#pragma unroll
                for (int j = 0; j < kMaxTapsUnrolled; ++j) y = fmaf(w[k][j], xin[k][j], y);
                if (ring) ring[i] = a.proj[(size_t)t * a.ld_proj + ch0 + i];   // the token's own input (the last tap)
                if (vdst) vdst[i] = DT<T>::from_f(y);
                vals[i] = y;
                ss += y * y;
            }
        }
    } else
    for (int i = lane; i < dim; i += 32) {
        const int c = ch0 + i;
        float y;
        if (a.conv_w) {
            y = 0.f;
            for (int j = 0; j < taps; ++j) {
                const int back = taps - 1 - j, src = p - back;
                if (src < 0) continue;
                const float uin = src >= first ? a.proj[(size_t)(t - back) * a.ld_proj + c]
                                               : a.conv_state[((size_t)b * (taps - 1) + src % (taps - 1)) * channels + c];
                y = fmaf(a.conv_w[(size_t)c * taps + j], uin, y);
            }
            // a one-token entry: nobody else reads this sequence's ring in this launch, and this lane has read its own places
            if (a.ring_out && taps > 1) a.ring_out[((size_t)b * (taps - 1) + p % (taps - 1)) * channels + c] = a.proj[(size_t)t * a.ld_proj + c];
        } else
            y = a.proj[(size_t)t * a.ld_proj + c] + (a.bias ? a.bias[c] : 0.f);
        if (is_k && a.v_from_conv) reinterpret_cast<T*>(a.v_pool)[cache_row * dim + i] = DT<T>::from_f(y);
        vals[i] = y;
        ss += y * y;
    }
    const float* nw = is_k ? a.k_norm : a.q_norm;
    if (nw) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float rinv = 1.0f / sqrtf(ss / (float)dim + a.eps);
        for (int i = lane; i < dim; i += 32) vals[i] = vals[i] * rinv * nw[i];
    }
    __syncwarp();
    const int nf = a.rot_dims / 2;
    T* dst = is_k ? reinterpret_cast<T*>(a.k_pool) + cache_row * dim : reinterpret_cast<T*>(a.q_out) + ((size_t)t * a.heads + u) * dim;
    const float mul = is_k ? 1.f : query_temp(a, p);
    for (int i = lane; i < dim; i += 32)
        dst[i] = DT<T>::from_f(rotary_component(vals, i, a.rot_dims, a.rot_layout, a.cos + (size_t)t * nf, a.sin + (size_t)t * nf) * mul);
}

// Norms over the WHOLE query and the whole key projection (before they are split into heads): one CTA per token sums the squares of
// both parts, then norms, turns (through shared memory, where the design rotates), scales the queries and scatters q, k and the
// projected values. VEC consecutive dimensions per thread and step.
constexpr int kRowPrepThreads = 256;
template <typename T, int VEC>
__device__ __forceinline__ void prep_store(T* dst, const float (&v)[VEC]) {
    if constexpr (VEC == 1) dst[0] = DT<T>::from_f(v[0]);
    else if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
}
template <int VEC>
__device__ __forceinline__ void prep_load(float (&v)[VEC], const float* src) {
    if constexpr (VEC == 1) v[0] = src[0];
    else {
        const float4 f = *reinterpret_cast<const float4*>(src);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    }
}
template <typename T, int VEC>
__global__ void __launch_bounds__(kRowPrepThreads) qk_row_prepare_kernel(const QkPrep a) {
    extern __shared__ __align__(16) float prep_sm[];   // rotated designs: the normed q and k of the token
    __shared__ float red[2][kRowPrepThreads / 32];
    const int t = blockIdx.x, dim = a.dim, nq = a.heads * dim, nk = a.kv_heads * dim, nv = a.v_heads * a.vdim, p = a.pos[t];
    const float* row = a.proj + (size_t)t * a.ld_proj;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * VEC; i < nq + nk; i += kRowPrepThreads * VEC) {
        float v[VEC];
        prep_load<VEC>(v, row + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            if (a.bias) v[e] += a.bias[i + e];
            if (i < nq) sq += v[e] * v[e];
            else sk += v[e] * v[e];
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if (threadIdx.x % 32 == 0) { red[0][threadIdx.x / 32] = sq; red[1][threadIdx.x / 32] = sk; }
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < kRowPrepThreads / 32; ++w) { sq += red[0][w]; sk += red[1][w]; }
    const float rq = a.q_norm ? 1.0f / sqrtf(sq / (float)nq + a.eps) : 1.f, rk = a.k_norm && nk > 0 ? 1.0f / sqrtf(sk / (float)nk + a.eps) : 1.f;
    const float mul = query_temp(a, p);
    size_t cache_row = 0;
    if (nk + nv > 0) cache_row = (size_t)a.pages[(size_t)a.slot[t] * a.max_pages + p / a.page_rows] * a.page_rows + p % a.page_rows;
    T* qd = reinterpret_cast<T*>(a.q_out) + (size_t)t * nq;
    T* kd = reinterpret_cast<T*>(a.k_pool) + cache_row * nk;
    for (int i = threadIdx.x * VEC; i < nq + nk; i += kRowPrepThreads * VEC) {
        const bool is_k = i >= nq;
        const float* nw = is_k ? a.k_norm : a.q_norm;
        const int c = is_k ? i - nq : i;
        float v[VEC];
        prep_load<VEC>(v, row + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            if (a.bias) v[e] += a.bias[i + e];
            v[e] *= is_k ? rk : rq;
            if (nw) v[e] *= nw[c + e];
            if (a.rot_dims) prep_sm[i + e] = v[e];
            else if (!is_k) v[e] *= mul;
        }
        if (!a.rot_dims) prep_store<T, VEC>(is_k ? kd + c : qd + c, v);
    }
    for (int i = threadIdx.x * VEC; i < nv; i += kRowPrepThreads * VEC) {
        float v[VEC];
        prep_load<VEC>(v, row + a.v_off + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e)
            if (a.bias) v[e] += a.bias[a.v_off + i + e];
        prep_store<T, VEC>(reinterpret_cast<T*>(a.v_pool) + cache_row * nv + i, v);
    }
    if (!a.rot_dims) return;
    __syncthreads();
    const int nf = a.rot_dims / 2;
    for (int i = threadIdx.x; i < nq + nk; i += kRowPrepThreads) {
        const bool is_k = i >= nq;
        const float v = rotary_component(prep_sm + i / dim * dim, i % dim, a.rot_dims, a.rot_layout, a.cos + (size_t)t * nf, a.sin + (size_t)t * nf);
        if (is_k) kd[i - nq] = DT<T>::from_f(v);
        else qd[i] = DT<T>::from_f(v * mul);
    }
}

// The same without rotation and bias for rows of at most 4 * PER * THREADS query and key columns in whole groups of four: the row, the
// values and the weights are loaded up front and live in registers (one round trip to memory instead of two passes).
template <typename T, int THREADS, int PER>
__global__ void __launch_bounds__(THREADS) qk_row_prepare_reg_kernel(const QkPrep a) {
    __shared__ float red[2][THREADS / 32];
    const int t = blockIdx.x, nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.v_heads * a.vdim, p = a.pos[t];
    const float* row = a.proj + (size_t)t * a.ld_proj;
    float4 v[PER], w[PER];
    const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int i = 4 * (threadIdx.x + THREADS * k);
        v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        w[k] = one;
        if (i < nq + nk) {
            v[k] = *reinterpret_cast<const float4*>(row + i);
            const float* nw = i < nq ? a.q_norm : a.k_norm;
            if (nw) w[k] = *reinterpret_cast<const float4*>(nw + (i < nq ? i : i - nq));
        }
    }
    size_t cache_row = 0;
    if (nk + nv > 0) cache_row = (size_t)a.pages[(size_t)a.slot[t] * a.max_pages + p / a.page_rows] * a.page_rows + p % a.page_rows;
    for (int i = threadIdx.x * 4; i < nv; i += THREADS * 4) {
        const float4 f = *reinterpret_cast<const float4*>(row + a.v_off + i);
        const float vv[4] = {f.x, f.y, f.z, f.w};
        prep_store<T, 4>(reinterpret_cast<T*>(a.v_pool) + cache_row * nv + i, vv);
    }
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int i = 4 * (threadIdx.x + THREADS * k);
        const float ss = v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
        if (i < nq) sq += ss;
        else sk += ss;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if (threadIdx.x % 32 == 0) { red[0][threadIdx.x / 32] = sq; red[1][threadIdx.x / 32] = sk; }
    const float mul = query_temp(a, p);
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
    const float rq = a.q_norm ? 1.0f / sqrtf(sq / (float)nq + a.eps) : 1.f, rk = a.k_norm && nk > 0 ? 1.0f / sqrtf(sk / (float)nk + a.eps) : 1.f;
    T* qd = reinterpret_cast<T*>(a.q_out) + (size_t)t * nq;
    T* kd = reinterpret_cast<T*>(a.k_pool) + cache_row * nk;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int i = 4 * (threadIdx.x + THREADS * k);
        if (i >= nq + nk) continue;
        const bool is_k = i >= nq;
        const float r = is_k ? rk : rq, m = is_k ? 1.f : mul;
        const float f[4] = {v[k].x * r * w[k].x * m, v[k].y * r * w[k].y * m, v[k].z * r * w[k].z * m, v[k].w * r * w[k].w * m};
        prep_store<T, 4>(is_k ? kd + (i - nq) : qd + i, f);
    }
}
template <typename T>
static bool launch_row_prepare_reg(const QkPrep& a, int n_tokens, cudaStream_t s) {
    const int quads = (a.heads + a.kv_heads) * a.dim / 4;
    if (quads <= 256) qk_row_prepare_reg_kernel<T, 256, 1><<<n_tokens, 256, 0, s>>>(a);
    else if (quads <= 1024) qk_row_prepare_reg_kernel<T, 512, 2><<<n_tokens, 512, 0, s>>>(a);
    else if (quads <= 2048) qk_row_prepare_reg_kernel<T, 512, 4><<<n_tokens, 512, 0, s>>>(a);
    else return false;
    return true;
}

// Without convolution and head norm the preparation is a rotation and three scatters: a thread per four consecutive
// dimensions of one head (or value head) of one token. It loads its own four values and, inside the rotated part, the
// four of its rotate-half partner with 16-byte loads, and stores four values of the serving dtype at once.
template <typename T>
__global__ void __launch_bounds__(256) qk_rotate_store_kernel(const QkPrep a, long long total, int quads_per_token) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int t = (int)(idx / quads_per_token), qd = (int)(idx % quads_per_token);
    const int dim = a.dim, qk_quads = (a.heads + a.kv_heads) * (dim / 4);
    const float* row = a.proj + (size_t)t * a.ld_proj;
    float4 v;
    T* dst;
    if (qd < qk_quads) {
        const int u = qd / (dim / 4), i0 = (qd % (dim / 4)) * 4, half = a.rot_dims / 2;
        v = *reinterpret_cast<const float4*>(row + (size_t)u * dim + i0);
        if (i0 < a.rot_dims) {
            const bool low = i0 < half;
            const float4 w = *reinterpret_cast<const float4*>(row + (size_t)u * dim + (low ? i0 + half : i0 - half));
            const float* cs = a.cos + (size_t)t * half + (low ? i0 : i0 - half);
            const float* sn = a.sin + (size_t)t * half + (low ? i0 : i0 - half);
            // the pair (lo, hi) becomes (lo c - hi s, hi c + lo s)
            if (low) v = make_float4(v.x * cs[0] - w.x * sn[0], v.y * cs[1] - w.y * sn[1], v.z * cs[2] - w.z * sn[2], v.w * cs[3] - w.w * sn[3]);
            else v = make_float4(v.x * cs[0] + w.x * sn[0], v.y * cs[1] + w.y * sn[1], v.z * cs[2] + w.z * sn[2], v.w * cs[3] + w.w * sn[3]);
        }
        if (u < a.heads) dst = reinterpret_cast<T*>(a.q_out) + ((size_t)t * a.heads + u) * dim + i0;
        else {
            const int p = a.pos[t];
            const size_t prow = (size_t)a.pages[(size_t)a.slot[t] * a.max_pages + p / a.page_rows] * a.page_rows + p % a.page_rows;
            dst = reinterpret_cast<T*>(a.k_pool) + (prow * a.kv_heads + (u - a.heads)) * dim + i0;
        }
    } else {
        const int c0 = (qd - qk_quads) * 4, p = a.pos[t];   // value column (head g, dimension c0 % vdim)
        v = *reinterpret_cast<const float4*>(row + a.v_off + c0);
        const size_t prow = (size_t)a.pages[(size_t)a.slot[t] * a.max_pages + p / a.page_rows] * a.page_rows + p % a.page_rows;
        dst = reinterpret_cast<T*>(a.v_pool) + prow * a.v_heads * a.vdim + c0;
    }
    if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(dst) = v;
    else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
}

// the rotated part of every head's query, placed behind the head's absorbed part: a thread per (token, head, dimension)
__global__ void rotate_part_kernel(const float* __restrict__ src, long long ld_src, long long src_off, long long src_stride,
                                   float* __restrict__ dst, long long ld_dst, long long dst_off, long long dst_stride,
                                   const float* __restrict__ cs, const float* __restrict__ sn, int layout, int heads, int dims, size_t total) {
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int i = (int)(idx % dims), h = (int)((idx / dims) % heads);
    const size_t t = idx / ((size_t)dims * heads);
    const int nf = dims / 2;
    dst[t * ld_dst + dst_off + h * dst_stride + i] =
        rotary_component(src + t * ld_src + src_off + h * src_stride, i, 2 * nf, layout, cs + t * nf, sn + t * nf);
}

__global__ void conv_state_update_kernel(const float* __restrict__ proj, long long ld_proj, float* __restrict__ state,
                                         const int* __restrict__ slot, const int* __restrict__ pos, const int* __restrict__ end,
                                         int channels, int taps) {
    const int t = blockIdx.x, p = pos[t];
    if (p < end[t] - (taps - 1)) return;   // only the last taps-1 inputs of a sequence are carried
    float* dst = state + ((size_t)slot[t] * (taps - 1) + p % (taps - 1)) * channels;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) dst[c] = proj[(size_t)t * ld_proj + c];
}

}  // namespace b200

using namespace b200;

extern "C" int b200_rope_angles_amp(const int* pos, int n_tokens, const double* freq, int n_freq, double amplitude, float* cos_out,
                                    float* sin_out, void* stream) {
    if (!pos || !freq || !cos_out || !sin_out || n_tokens < 0 || n_freq < 0) return B200_EINVAL;
    const int total = n_tokens * n_freq;
    if (total == 0) return B200_OK;
    rope_angles_kernel<<<(total + 255) / 256, 256, 0, (cudaStream_t)stream>>>(pos, freq, n_freq, total, amplitude, cos_out, sin_out);
    count_launch();
    return (int)cudaGetLastError();
}
extern "C" int b200_rope_angles(const int* pos, int n_tokens, const double* freq, int n_freq, float* cos_out, float* sin_out,
                                void* stream) {
    return b200_rope_angles_amp(pos, n_tokens, freq, n_freq, 1.0, cos_out, sin_out, stream);
}

extern "C" int b200_qk_prepare(const b200_qk_prepare_args* p, void* stream) {
    if (!p || !p->proj || !p->q_out || (!p->k_pool && (!p->norm_rows || p->v_heads)) || !p->pages || !p->slot || !p->pos || p->n_tokens < 0 || p->heads < 1 ||
        p->kv_heads < 1 || p->dim < 1 || p->page_rows < 1)
        return B200_EINVAL;
    if (p->conv_w && (p->taps < 1 || !p->start || (p->taps > 1 && !p->conv_state))) return B200_EINVAL;
    if (p->v_from_conv && !p->v_pool) return B200_EINVAL;
    if (p->v_heads < 0 || (p->v_heads > 0 && (!p->v_pool || p->vdim < 1 || p->v_from_conv || p->v_off < 0))) return B200_EINVAL;
    if (p->rot_dims < 0 || (p->rot_dims & 1) || p->rot_dims > p->dim || (p->rot_dims && (!p->cos || !p->sin))) return B200_EINVAL;
    if (p->rot_layout != B200_ROPE_HALF && p->rot_layout != B200_ROPE_INTERLEAVED) return B200_EINVAL;
    if (p->norm_rows && (p->conv_w || p->v_from_conv || p->v_cos)) return B200_EINVAL;
    if (p->temp_every < 0) return B200_EINVAL;
    if (p->bias && p->conv_w) return B200_EINVAL;   // carried convolution inputs are raw projections
    if ((p->v_cos || p->v_sin) && (!p->v_cos || !p->v_sin || p->v_heads < 1 ||
                                   (p->v_rot_layout != B200_ROPE_HALF && p->v_rot_layout != B200_ROPE_INTERLEAVED)))
        return B200_EINVAL;
    if (p->n_tokens == 0) return B200_OK;
    QkPrep a{p->proj, p->ld_proj, p->conv_w, p->taps, p->conv_state, p->q_norm, p->k_norm, p->eps, p->cos, p->sin, p->rot_dims,
             p->rot_layout, p->q_out, p->k_pool, p->v_pool, p->v_from_conv, p->update_state_inline ? const_cast<float*>(p->conv_state) : nullptr, p->pages, p->max_pages, p->page_rows, p->slot, p->pos,
             p->start, p->heads, p->kv_heads, p->dim, p->v_heads, p->vdim, p->v_off, p->bias, p->v_cos, p->v_sin, p->v_rot_layout,
             p->v_heads > 0 && p->vdim > p->dim ? p->vdim : p->dim, p->temp_coef, p->temp_every};
    if (a.conv_w && a.taps == 1) a.conv_state = a.proj;   // never read: every input of a one-tap filter is the token's own
    cudaStream_t s = (cudaStream_t)stream;
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    if (p->norm_rows) {
        if (!p->k_pool) a.kv_heads = 0;
        const size_t smem = p->rot_dims ? (size_t)(a.heads + a.kv_heads) * p->dim * sizeof(float) : 0;
        if (smem > 48 * 1024 - 128) return B200_EUNSUPPORTED;
        const bool vec = p->dim % 4 == 0 && p->ld_proj % 4 == 0 && al16(p->proj) && al16(p->q_out) && al16(p->k_pool) &&
                         (p->v_heads == 0 || (p->vdim % 4 == 0 && p->v_off % 4 == 0 && al16(p->v_pool)));
        const bool reg = vec && !p->rot_dims && !p->bias && (!p->q_norm || al16(p->q_norm)) && (!p->k_norm || al16(p->k_norm));
        if (reg && (p->dtype == B200_BF16 ? launch_row_prepare_reg<__nv_bfloat16>(a, p->n_tokens, s) : p->dtype == B200_F32 && launch_row_prepare_reg<float>(a, p->n_tokens, s))) {
        } else if (p->dtype == B200_BF16) {
            if (vec) qk_row_prepare_kernel<__nv_bfloat16, 4><<<p->n_tokens, kRowPrepThreads, smem, s>>>(a);
            else qk_row_prepare_kernel<__nv_bfloat16, 1><<<p->n_tokens, kRowPrepThreads, smem, s>>>(a);
        } else if (p->dtype == B200_F32) {
            if (vec) qk_row_prepare_kernel<float, 4><<<p->n_tokens, kRowPrepThreads, smem, s>>>(a);
            else qk_row_prepare_kernel<float, 1><<<p->n_tokens, kRowPrepThreads, smem, s>>>(a);
        } else
            return B200_EINVAL;
        count_launch();
        return (int)cudaGetLastError();
    }
    {   // rotation and scatters only, everything in whole groups of four: the vector kernel
        const bool plain = !p->temp_every && !p->conv_w && !p->q_norm && !p->k_norm && !p->bias && !p->v_cos && p->rot_layout == B200_ROPE_HALF && p->dim % 4 == 0 && p->rot_dims % 8 == 0 &&
                           p->ld_proj % 4 == 0 && al16(p->proj) && al16(p->q_out) && al16(p->k_pool) &&
                           (p->v_heads == 0 || (p->vdim % 4 == 0 && p->v_off % 4 == 0 && al16(p->v_pool))) &&
                           (p->dtype == B200_BF16 || p->dtype == B200_F32);
        if (plain) {
            const int quads = (p->heads + p->kv_heads) * (p->dim / 4) + p->v_heads * (p->vdim / 4);
            const long long total = (long long)p->n_tokens * quads;
            const unsigned grid = (unsigned)((total + 255) / 256);
            if (p->dtype == B200_BF16) qk_rotate_store_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(a, total, quads);
            else qk_rotate_store_kernel<float><<<grid, 256, 0, s>>>(a, total, quads);
            count_launch();
            return (int)cudaGetLastError();
        }
    }
    const long long units = (long long)p->n_tokens * (p->heads + p->kv_heads + p->v_heads);
    if (units > 0x7fffffffll) return B200_EUNSUPPORTED;
    const unsigned grid = (unsigned)((units + kPrepWarps - 1) / kPrepWarps);
    const size_t smem = (size_t)kPrepWarps * a.vals_per_warp * sizeof(float);
    if (smem > 48 * 1024) return B200_EUNSUPPORTED;
    if (p->dtype == B200_BF16) qk_prepare_kernel<__nv_bfloat16><<<grid, kPrepWarps * 32, smem, s>>>(a, (int)units);
    else if (p->dtype == B200_F32) qk_prepare_kernel<float><<<grid, kPrepWarps * 32, smem, s>>>(a, (int)units);
    else return B200_EINVAL;
    count_launch();
    return (int)cudaGetLastError();
}

extern "C" int b200_rotate_part(const float* src, long long ld_src, long long src_off, long long src_stride, float* dst, long long ld_dst,
                                long long dst_off, long long dst_stride, const float* cos, const float* sin, int rot_layout, int n_tokens,
                                int heads, int dims, void* stream) {
    if (!src || !dst || !cos || !sin || n_tokens < 0 || heads < 1 || dims < 1) return B200_EINVAL;
    if (rot_layout != B200_ROPE_HALF && rot_layout != B200_ROPE_INTERLEAVED) return B200_EINVAL;
    if (n_tokens == 0) return B200_OK;
    const size_t total = (size_t)n_tokens * heads * dims;
    rotate_part_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(src, ld_src, src_off, src_stride, dst, ld_dst, dst_off,
                                                                                         dst_stride, cos, sin, rot_layout, heads, dims, total);
    count_launch();
    return (int)cudaGetLastError();
}

extern "C" int b200_conv_state_update(const float* proj, long long ld_proj, float* conv_state, const int* slot, const int* pos,
                                      const int* end, int n_tokens, int channels, int taps, void* stream) {
    if (!proj || !slot || !pos || !end || n_tokens < 0 || channels < 1 || taps < 1) return B200_EINVAL;
    if (n_tokens == 0 || taps == 1) return B200_OK;
    if (!conv_state) return B200_EINVAL;
    conv_state_update_kernel<<<n_tokens, 128, 0, (cudaStream_t)stream>>>(proj, ld_proj, conv_state, slot, pos, end, channels, taps);
    count_launch();
    return (int)cudaGetLastError();
}
