// State-space recurrence with one decay per head (the "dual" form of a selective state space): a matrix state S of
// n_state x vdim per head, S <- exp(A dt) S + dt B x^T, y = S^T C + D x, with step sizes dt = softplus(raw + bias) of the
// current token, B and C shared by the heads of a group, and S carried per sequence slot in fp32. And the gated norm behind
// it: y silu(z), RMS-normed in equal parts, times a weight.
//
//   ssd_walk_kernel    one CTA per (entry, head, block of value columns): a thread owns one column of a quarter of the state
//                      rows in registers and walks the entry's tokens; B, C, x and the decays of eight tokens are staged in
//                      shared memory at a time, the quarters' partial outputs are added there. All fp32. Decode batches,
//                      short portions and fp32 serving take this path.
//   chunk form (entries of 128 tokens and more, bfloat16 serving): 64-token chunks, four launches, products on tf32
//   tensor-core tiles (mma.sync m16n8k8) with fp32 accumulation:
//     ssd_cb_kernel        (C_i . B_j) of every chunk and group, once for all heads of the group;
//     ssd_state_kernel     U = sum_j exp(cum_end - cum_j) dt_j B_j x_j^T of every chunk and head, chunks in parallel;
//     ssd_carry_kernel     S at the start of every chunk, S' = exp(cum_end) S + U, and the state the entry leaves behind;
//     ssd_out_kernel       y_i = exp(cum_i) S^T C_i + sum_(j<=i) (C_i . B_j) exp(cum_i - cum_j) dt_j x_j + D x_i.
//   cum is the running sum of A dt inside the chunk, kept in double: the differences of two large sums are exact enough to
//   be exponentiated whatever the step sizes are.
#include <cuda_bf16.h>
#include <math.h>
#include <stdlib.h>

#include <algorithm>

#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"

namespace b200 {

struct SS {
    const float* u; long long ld_u; int x_off, b_off, c_off;
    const float* dt_raw; long long ld_dt; const float* dt_bias;
    const float* A; const float* D;
    float* state; float* out;
    const int* ent_row; const int* ent_len; const int* slot; const int* pos;
    int heads, groups, vdim, n_state;
    // chunk form: chunk c of entry e sits at place ent_row[e] / kSsdChunk + e + c
    float* chunk_state;   // [place, head, n_state, vdim]
    float* chunk_decay;   // [place, head]
    float* chunk_cb;      // [place, group, kSsdChunk, kSsdChunk]
    int col_blocks;
};

__device__ __forceinline__ float ssd_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }

constexpr int kSsdRowGroups = 4, kSsdTokens = 8;

template <int NPT, int PB>   // state rows per thread, value columns per CTA
__global__ void __launch_bounds__(kSsdRowGroups * PB) ssd_walk_kernel(const SS a) {
    constexpr int NP = NPT * kSsdRowGroups, NT = kSsdRowGroups * PB;
    __shared__ float Bs[kSsdTokens][NP], Cs[kSsdTokens][NP], xs[kSsdTokens][PB], part[kSsdTokens][kSsdRowGroups][PB];
    __shared__ float dts[kSsdTokens], decs[kSsdTokens];
    const int e = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PB;
    const int c = threadIdx.x % PB, rg = threadIdx.x / PB, n0 = rg * NPT, N = a.n_state, P = a.vdim;
    const int row0 = a.ent_row[e], len = a.ent_len[e], b = a.slot[row0], g = h / (a.heads / a.groups);
    const bool live = p0 + c < P, carried = a.pos[row0] > 0;
    float* st = a.state + (((size_t)b * a.heads + h) * N) * P + p0 + c;
    float S[NPT];
#pragma unroll
    for (int k = 0; k < NPT; ++k) S[k] = (carried && live && n0 + k < N) ? st[(size_t)(n0 + k) * P] : 0.f;
    const float A = a.A[h], Dh = a.D[h], bias = a.dt_bias[h];
    for (int t0 = 0; t0 < len; t0 += kSsdTokens) {
        const int nt = min(kSsdTokens, len - t0);
        __syncthreads();   // the previous group's readers are done
        for (int i = threadIdx.x; i < nt * NP; i += NT) {
            const int k = i / NP, n = i % NP;
            const float* row = a.u + (size_t)(row0 + t0 + k) * a.ld_u;
            Bs[k][n] = n < N ? row[a.b_off + g * N + n] : 0.f;
            Cs[k][n] = n < N ? row[a.c_off + g * N + n] : 0.f;
        }
        for (int i = threadIdx.x; i < nt * PB; i += NT) {
            const int k = i / PB, p = i % PB;
            xs[k][p] = p0 + p < P ? a.u[(size_t)(row0 + t0 + k) * a.ld_u + a.x_off + h * P + p0 + p] : 0.f;
        }
        if (threadIdx.x < nt) {
            const float dt = ssd_softplus(a.dt_raw[(size_t)(row0 + t0 + threadIdx.x) * a.ld_dt + h] + bias);
            dts[threadIdx.x] = dt;
            decs[threadIdx.x] = expf(A * dt);
        }
        __syncthreads();
        for (int k = 0; k < nt; ++k) {
            const float dec = decs[k], dx = dts[k] * xs[k][c];
            float y = 0.f;
#pragma unroll
            for (int j = 0; j < NPT; ++j) {
                S[j] = fmaf(dec, S[j], dx * Bs[k][n0 + j]);
                y = fmaf(S[j], Cs[k][n0 + j], y);
            }
            part[k][rg][c] = y;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * PB; i += NT) {
            const int k = i / PB, p = i % PB;
            if (p0 + p >= P) continue;
            float y = Dh * xs[k][p];
#pragma unroll
            for (int q = 0; q < kSsdRowGroups; ++q) y += part[k][q][p];
            a.out[(size_t)(row0 + t0 + k) * ((size_t)a.heads * P) + h * P + p0 + p] = y;
        }
    }
    if (live) {
#pragma unroll
        for (int k = 0; k < NPT; ++k)
            if (n0 + k < N) st[(size_t)(n0 + k) * P] = S[k];
    }
}

// ---------------------------------------------------------------------------------------------------------------
// chunk form
// ---------------------------------------------------------------------------------------------------------------
constexpr int kSsdChunk = 64, kSsdCols = 64, kSsdXs = kSsdCols + 8, kSsdMs = kSsdChunk + 4;
// row strides in floats: stride % 32 == 4 for operands whose rows run along the fragment's 8-wide index, 8 for those whose
// rows run along its 4-wide index (every fragment load then touches 32 different banks)
__host__ __device__ __forceinline__ int ssd_stride4(int n) { return ((n + 31) & ~31) + 4; }
__host__ __device__ __forceinline__ int ssd_stride8(int n) { return ((n + 31) & ~31) + 8; }

__device__ __forceinline__ float ssd_tf32(float v) {
    uint32_t r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(v));
    return __uint_as_float(r);
}
__device__ __forceinline__ void ssd_mma(float (&d)[4], const float (&a)[4], float b0, float b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])),
          "r"(__float_as_uint(b0)), "r"(__float_as_uint(b1)));
}

// the chunk's step sizes and running sums of A dt (double) by warp 0: two tokens per lane; places beyond the chunk hold
// dt = 0 and the last sum
__device__ __forceinline__ void ssd_chunk_sums(const SS& a, int h, int row0, int len, float* dts, double* cum) {
    if (threadIdx.x < 32) {
        const int l = threadIdx.x;
        const float bias = a.dt_bias[h], A = a.A[h];
        float d[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int i = 2 * l + k;
            d[k] = i < len ? ssd_softplus(a.dt_raw[(size_t)(row0 + i) * a.ld_dt + h] + bias) : 0.f;
            dts[i] = d[k];
        }
        const double v0 = (double)A * d[0], v1 = v0 + (double)A * d[1];
        double run = v1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, run, o);
            if (l >= o) run += up;
        }
        cum[2 * l] = run - v1 + v0;
        cum[2 * l + 1] = run;
    }
}

// `rows` rows of `cols` columns from global (leading dimension ld) into shared memory, rows beyond `live` and columns beyond
// cols (up to cpad) zero. Rows that allow it travel by cp.async (nothing waits for a load here: ssd_landed() before the first
// read); the values are rounded to tf32 when a fragment picks them up.
__device__ __forceinline__ void ssd_stage(float* dst, int stride, const float* src, long long ld, int rows, int live, int cols, int cpad) {
    if ((cols & 3) == 0 && (ld & 3) == 0 && (reinterpret_cast<uintptr_t>(src) & 15u) == 0 && cpad == cols) {
        const int q = cols / 4;
        for (int i = threadIdx.x; i < rows * q; i += blockDim.x) {
            const int r = i / q, c = (i - r * q) * 4;
            const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst + r * stride + c);
            const float* g = src + (r < live ? (size_t)r * ld + c : 0);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(g), "r"(r < live ? 16 : 0) : "memory");
        }
        return;
    }
    for (int i = threadIdx.x; i < rows * cpad; i += blockDim.x) {
        const int r = i / cpad, c = i - r * cpad;
        dst[r * stride + c] = (r < live && c < cols) ? src[(size_t)r * ld + c] : 0.f;
    }
}
__device__ __forceinline__ void ssd_landed() {
    __syncwarp();   // the lanes close their group of copies together
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();
}

struct SsdChunk {
    int row0, len, place;
    bool on;
};
__device__ __forceinline__ SsdChunk ssd_chunk_of(const SS& a, int e, int c) {
    const int row_e = a.ent_row[e], n = a.ent_len[e];
    return {row_e + c * kSsdChunk, min(kSsdChunk, n - c * kSsdChunk), row_e / kSsdChunk + e + c, c * kSsdChunk < n};
}

__global__ void __launch_bounds__(128) ssd_cb_kernel(const SS a) {
    extern __shared__ __align__(16) float sm[];
    const SsdChunk ck = ssd_chunk_of(a, blockIdx.x, blockIdx.y);
    if (!ck.on) return;
    const int g = blockIdx.z, N = a.n_state, npad = (N + 7) & ~7, st = ssd_stride4(npad);
    float* Cs = sm;                      // [64][st]
    float* Bs = sm + kSsdChunk * st;     // [64][st]
    const float* row = a.u + (size_t)ck.row0 * a.ld_u + g * N;
    ssd_stage(Cs, st, row + a.c_off, a.ld_u, kSsdChunk, ck.len, N, npad);
    ssd_stage(Bs, st, row + a.b_off, a.ld_u, kSsdChunk, ck.len, N, npad);
    ssd_landed();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3, m0 = warp * 16;
    float acc[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    for (int k0 = 0; k0 < npad; k0 += 8) {
        const float* ar = Cs + (m0 + gid) * st + k0 + tig;
        const float av[4] = {ssd_tf32(ar[0]), ssd_tf32(ar[8 * st]), ssd_tf32(ar[4]), ssd_tf32(ar[8 * st + 4])};
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            const float* br = Bs + (nt * 8 + gid) * st + k0 + tig;
            ssd_mma(acc[nt], av, ssd_tf32(br[0]), ssd_tf32(br[4]));
        }
    }
    float* dst = a.chunk_cb + ((size_t)ck.place * a.groups + g) * kSsdChunk * kSsdChunk;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
        const int j = nt * 8 + tig * 2;
        *reinterpret_cast<float2*>(dst + (m0 + gid) * kSsdChunk + j) = make_float2(acc[nt][0], acc[nt][1]);
        *reinterpret_cast<float2*>(dst + (m0 + gid + 8) * kSsdChunk + j) = make_float2(acc[nt][2], acc[nt][3]);
    }
}

__global__ void __launch_bounds__(128) ssd_state_kernel(const SS a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ double cum[kSsdChunk];
    __shared__ float dts[kSsdChunk], wts[kSsdChunk];
    const int e = blockIdx.x / a.col_blocks, p0 = (blockIdx.x % a.col_blocks) * kSsdCols;
    const SsdChunk ck = ssd_chunk_of(a, e, blockIdx.y);
    if (!ck.on) return;
    const int h = blockIdx.z, g = h / (a.heads / a.groups), N = a.n_state, P = a.vdim, npad = (N + 15) & ~15, st = ssd_stride8(npad);
    float* Xs = sm;                        // [64][kSsdXs]
    float* Bs = sm + kSsdChunk * kSsdXs;   // [64][st]
    const int cols = min(kSsdCols, P - p0);
    const float* row = a.u + (size_t)ck.row0 * a.ld_u;
    ssd_stage(Bs, st, row + a.b_off + g * N, a.ld_u, kSsdChunk, ck.len, N, npad);
    ssd_stage(Xs, kSsdXs, row + a.x_off + h * P + p0, a.ld_u, kSsdChunk, ck.len, cols, kSsdCols);
    ssd_chunk_sums(a, h, ck.row0, ck.len, dts, cum);
    ssd_landed();
    if (threadIdx.x < kSsdChunk) wts[threadIdx.x] = dts[threadIdx.x] * expf((float)(cum[kSsdChunk - 1] - cum[threadIdx.x]));
    if (threadIdx.x == 0 && p0 == 0) a.chunk_decay[(size_t)ck.place * a.heads + h] = expf((float)cum[kSsdChunk - 1]);
    __syncthreads();
    // the weights dt_j exp(cum_end - cum_j) go into the value rows, in place
    for (int i = threadIdx.x; i < kSsdChunk * (kSsdCols / 4); i += 128) {
        float4* x4 = reinterpret_cast<float4*>(Xs + (i / (kSsdCols / 4)) * kSsdXs) + i % (kSsdCols / 4);
        const float w = wts[i / (kSsdCols / 4)];
        const float4 v = *x4;
        *x4 = make_float4(ssd_tf32(v.x * w), ssd_tf32(v.y * w), ssd_tf32(v.z * w), ssd_tf32(v.w * w));
    }
    __syncthreads();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    float* U = a.chunk_state + (((size_t)ck.place * a.heads + h) * N) * P + p0;
    const bool pair = (P & 1) == 0;
    for (int m0 = warp * 16; m0 < npad; m0 += 64) {
        float acc[8][4];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
#pragma unroll 2
        for (int k0 = 0; k0 < kSsdChunk; k0 += 8) {
            const float* ar = Bs + (k0 + tig) * st + m0 + gid;
            const float av[4] = {ssd_tf32(ar[0]), ssd_tf32(ar[8]), ssd_tf32(ar[4 * st]), ssd_tf32(ar[4 * st + 8])};
            const float* br = Xs + (k0 + tig) * kSsdXs + gid;
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) ssd_mma(acc[nt], av, br[nt * 8], br[4 * kSsdXs + nt * 8]);
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int n = m0 + gid + half * 8, p = nt * 8 + tig * 2;
                if (n >= N || p0 + p >= P) continue;
                float* d = U + (size_t)n * P + p;
                if (pair) *reinterpret_cast<float2*>(d) = make_float2(acc[nt][half * 2], acc[nt][half * 2 + 1]);
                else {
                    d[0] = acc[nt][half * 2];
                    if (p0 + p + 1 < P) d[1] = acc[nt][half * 2 + 1];
                }
            }
    }
}

// element-wise over the state (VEC consecutive elements per thread): walks the entry's chunks, leaves S at each chunk's start in
// place of its U
template <int VEC> struct SsdVec;
template <> struct SsdVec<1> { using T = float; };
template <> struct SsdVec<4> { using T = float4; };
__device__ __forceinline__ float ssd_next(float S, float d, float u) { return fmaf(d, S, u); }
__device__ __forceinline__ float4 ssd_next(float4 S, float d, float4 u) {
    return make_float4(fmaf(d, S.x, u.x), fmaf(d, S.y, u.y), fmaf(d, S.z, u.z), fmaf(d, S.w, u.w));
}

template <int VEC>
__global__ void __launch_bounds__(128) ssd_carry_kernel(const SS a) {
    using V = typename SsdVec<VEC>::T;
    const int e = blockIdx.x, h = blockIdx.y, i = blockIdx.z * blockDim.x + threadIdx.x, per = a.n_state * a.vdim / VEC;
    if (i >= per) return;
    const int row_e = a.ent_row[e], n = a.ent_len[e], b = a.slot[row_e], chunks = (n + kSsdChunk - 1) / kSsdChunk;
    V* sp = reinterpret_cast<V*>(a.state) + ((size_t)b * a.heads + h) * per + i;
    V S{};
    if (a.pos[row_e] > 0) S = *sp;
    const size_t first = (size_t)(row_e / kSsdChunk + e), step = (size_t)a.heads * per;
    V* U = reinterpret_cast<V*>(a.chunk_state) + (first * a.heads + h) * per + i;
    const float* dec = a.chunk_decay + first * a.heads + h;
    constexpr int F = 8;
    for (int c0 = 0; c0 < chunks; c0 += F) {   // F loads in flight, then the dependent chain
        V u[F];
        float d[F];
#pragma unroll
        for (int k = 0; k < F; ++k)
            if (c0 + k < chunks) {
                u[k] = U[(size_t)(c0 + k) * step];
                d[k] = dec[(size_t)(c0 + k) * a.heads];
            }
#pragma unroll
        for (int k = 0; k < F; ++k)
            if (c0 + k < chunks) {
                U[(size_t)(c0 + k) * step] = S;
                S = ssd_next(S, d[k], u[k]);
            }
    }
    *sp = S;
}

__global__ void __launch_bounds__(256) ssd_out_kernel(const SS a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ double cum[kSsdChunk];
    __shared__ float dts[kSsdChunk];
    const int e = blockIdx.x / a.col_blocks, p0 = (blockIdx.x % a.col_blocks) * kSsdCols;
    const SsdChunk ck = ssd_chunk_of(a, e, blockIdx.y);
    if (!ck.on) return;
    const int h = blockIdx.z, g = h / (a.heads / a.groups), N = a.n_state, P = a.vdim, npad = (N + 7) & ~7, st = ssd_stride4(npad);
    float* Xs = sm;                               // [64][kSsdXs]
    float* Ms = Xs + kSsdChunk * kSsdXs;          // [64][kSsdMs]
    float* Cs = Ms + kSsdChunk * kSsdMs;          // [64][st]
    float* Ss = Cs + kSsdChunk * st;              // [npad][kSsdXs]
    const int cols = min(kSsdCols, P - p0);
    const float* row = a.u + (size_t)ck.row0 * a.ld_u;
    ssd_stage(Cs, st, row + a.c_off + g * N, a.ld_u, kSsdChunk, ck.len, N, npad);
    ssd_stage(Xs, kSsdXs, row + a.x_off + h * P + p0, a.ld_u, kSsdChunk, ck.len, cols, kSsdCols);
    ssd_stage(Ss, kSsdXs, a.chunk_state + (((size_t)ck.place * a.heads + h) * N) * P + p0, P, npad, N, cols, kSsdCols);
    ssd_stage(Ms, kSsdMs, a.chunk_cb + ((size_t)ck.place * a.groups + g) * kSsdChunk * kSsdChunk, kSsdChunk, kSsdChunk, kSsdChunk, kSsdChunk, kSsdChunk);
    ssd_chunk_sums(a, h, ck.row0, ck.len, dts, cum);
    ssd_landed();
#pragma unroll 4
    for (int i = threadIdx.x; i < kSsdChunk * kSsdChunk; i += 256) {
        const int r = i / kSsdChunk, j = i % kSsdChunk;
        float* v = Ms + r * kSsdMs + j;
        *v = j <= r ? ssd_tf32(*v * expf((float)(cum[r] - cum[j])) * dts[j]) : 0.f;
    }
    __syncthreads();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    const int m0 = (warp & 3) * 16, q0 = (warp >> 2) * 32;   // eight warps: 16 rows x 32 value columns each
    float acc[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    for (int k0 = 0; k0 < npad; k0 += 8) {   // what older chunks left
        const float* ar = Cs + (m0 + gid) * st + k0 + tig;
        const float av[4] = {ssd_tf32(ar[0]), ssd_tf32(ar[8 * st]), ssd_tf32(ar[4]), ssd_tf32(ar[8 * st + 4])};
        const float* br = Ss + (k0 + tig) * kSsdXs + q0 + gid;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) ssd_mma(acc[nt], av, ssd_tf32(br[nt * 8]), ssd_tf32(br[4 * kSsdXs + nt * 8]));
    }
    const float e_lo = expf((float)cum[m0 + gid]), e_hi = expf((float)cum[m0 + gid + 8]);
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) { acc[nt][0] *= e_lo; acc[nt][1] *= e_lo; acc[nt][2] *= e_hi; acc[nt][3] *= e_hi; }
    for (int k0 = 0; k0 < m0 + 16; k0 += 8) {   // this chunk's own tokens, up to the warp's last row
        const float* ar = Ms + (m0 + gid) * kSsdMs + k0 + tig;
        const float av[4] = {ar[0], ar[8 * kSsdMs], ar[4], ar[8 * kSsdMs + 4]};   // rounded above
        const float* br = Xs + (k0 + tig) * kSsdXs + q0 + gid;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) ssd_mma(acc[nt], av, ssd_tf32(br[nt * 8]), ssd_tf32(br[4 * kSsdXs + nt * 8]));
    }
    const float Dh = a.D[h];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int i = m0 + gid + (k >> 1) * 8, p = q0 + nt * 8 + tig * 2 + (k & 1);
            if (i < ck.len && p < cols)
                a.out[(size_t)(ck.row0 + i) * ((size_t)a.heads * P) + h * P + p0 + p] =
                    fmaf(Dh, Xs[i * kSsdXs + p], acc[nt][k]);
        }
}

// one CTA per (token, part): v = y silu(z) kept in shared memory between the sum of squares and the output
template <typename T>
__global__ void __launch_bounds__(128) gated_group_rms_kernel(const float* __restrict__ y, const float* __restrict__ z, long long ld_z,
                                                              const float* __restrict__ w, T* __restrict__ out, int n, int per, float eps) {
    extern __shared__ __align__(16) float vs[];
    __shared__ float red[4];
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * per;
    const float* yr = y + t * n + c0;
    const float* zr = z + t * ld_z + c0;
    float ss = 0.f;
    for (int i = threadIdx.x; i < per; i += 128) {
        const float g = zr[i], v = yr[i] * (g / (1.f + expf(-g)));
        vs[i] = v;
        ss += v * v;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = ss;
    __syncthreads();
    const float rinv = 1.0f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)per + eps);
    T* dst = out + t * n + c0;
    for (int i = threadIdx.x; i < per; i += 128) dst[i] = DT<T>::from_f(vs[i] * rinv * w[c0 + i]);
}

// the same for parts of at most 16 * THREADS columns in whole groups of four: everything is loaded up front and lives in registers
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS) gated_group_rms_reg_kernel(const float* __restrict__ y, const float* __restrict__ z, long long ld_z,
                                                                      const float* __restrict__ w, T* __restrict__ out, int n, int per, float eps) {
    __shared__ float red[THREADS / 32];
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * per;
    const float* yr = y + t * n + c0;
    const float* zr = z + t * ld_z + c0;
    float4 v[4], g[4], w4[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int i = 4 * (threadIdx.x + THREADS * k);
        v[k] = g[k] = w4[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < per) {
            v[k] = *reinterpret_cast<const float4*>(yr + i);
            g[k] = *reinterpret_cast<const float4*>(zr + i);
            w4[k] = *reinterpret_cast<const float4*>(w + c0 + i);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        v[k].x *= g[k].x / (1.f + expf(-g[k].x)); v[k].y *= g[k].y / (1.f + expf(-g[k].y));
        v[k].z *= g[k].z / (1.f + expf(-g[k].z)); v[k].w *= g[k].w / (1.f + expf(-g[k].w));
        ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int k = 0; k < THREADS / 32; ++k) tot += red[k];
    const float r = 1.0f / sqrtf(tot / (float)per + eps);
    T* dst = out + t * n + c0;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int i = 4 * (threadIdx.x + THREADS * k);
        if (i >= per) continue;
        const float f[4] = {v[k].x * r * w4[k].x, v[k].y * r * w4[k].y, v[k].z * r * w4[k].z, v[k].w * r * w4[k].w};
        if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(dst + i) = make_float4(f[0], f[1], f[2], f[3]);
        else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(f[0], f[1]), hi = __floats2bfloat162_rn(f[2], f[3]);
            *reinterpret_cast<uint2*>(dst + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

static size_t ssd_places(int n_tokens, int n_entries) { return (size_t)n_tokens / kSsdChunk + (size_t)n_entries + 1; }

template <int PB>
static int launch_walk(const SS& a, int n_entries, cudaStream_t s) {
    const dim3 grid(n_entries, a.heads, (a.vdim + PB - 1) / PB);
    constexpr int nt = kSsdRowGroups * PB;
    if (a.n_state <= 16) ssd_walk_kernel<4, PB><<<grid, nt, 0, s>>>(a);
    else if (a.n_state <= 32) ssd_walk_kernel<8, PB><<<grid, nt, 0, s>>>(a);
    else if (a.n_state <= 64) ssd_walk_kernel<16, PB><<<grid, nt, 0, s>>>(a);
    else if (a.n_state <= 128) ssd_walk_kernel<32, PB><<<grid, nt, 0, s>>>(a);
    else ssd_walk_kernel<64, PB><<<grid, nt, 0, s>>>(a);
    count_launch();
    return (int)cudaGetLastError();
}

}  // namespace b200

using namespace b200;

extern "C" size_t b200_ssd_scan_workspace_bytes(int n_tokens, int n_entries, int heads, int groups, int vdim, int n_state) {
    if (n_tokens < 2 * kSsdChunk || n_entries < 1 || heads < 1 || groups < 1 || vdim < 1 || n_state < 1) return 0;
    const size_t places = ssd_places(n_tokens, n_entries);
    return places * ((size_t)heads * n_state * vdim + ((heads + 3) & ~3) + (size_t)groups * kSsdChunk * kSsdChunk) * sizeof(float) + 256;
}

extern "C" int b200_ssd_scan(const b200_ssd_scan_args* p, void* stream) {
    if (!p || !p->u || !p->dt_raw || !p->dt_bias || !p->A || !p->D || !p->state || !p->out || !p->ent_row || !p->ent_len || !p->slot || !p->pos ||
        p->n_entries < 0 || p->n_tokens < 0 || p->heads < 1 || p->groups < 1 || p->heads % p->groups || p->vdim < 1 || p->n_state < 1 ||
        p->x_off < 0 || p->b_off < 0 || p->c_off < 0)
        return B200_EINVAL;
    if (p->n_state > 256 || p->heads > 65535 || p->vdim > 65535) return B200_EUNSUPPORTED;
    if (p->n_entries == 0 || p->n_tokens == 0) return B200_OK;
    SS a{p->u, p->ld_u, p->x_off, p->b_off, p->c_off, p->dt_raw, p->ld_dt, p->dt_bias, p->A, p->D, p->state, p->out,
         p->ent_row, p->ent_len, p->slot, p->pos, p->heads, p->groups, p->vdim, p->n_state, nullptr, nullptr, nullptr, 1};
    cudaStream_t s = (cudaStream_t)stream;
    const size_t need = b200_ssd_scan_workspace_bytes(p->n_tokens, p->n_entries, p->heads, p->groups, p->vdim, p->n_state);
    const int chunks = (p->longest_entry + kSsdChunk - 1) / kSsdChunk;
    if (p->chunked && p->longest_entry >= 2 * kSsdChunk && need > 0 && p->workspace && p->workspace_bytes >= need && chunks <= 65535) {
        const size_t places = ssd_places(p->n_tokens, p->n_entries);
        a.chunk_state = reinterpret_cast<float*>(p->workspace);
        a.chunk_cb = a.chunk_state + ((places * p->heads * p->n_state * p->vdim + 3) & ~(size_t)3);
        a.chunk_decay = a.chunk_cb + places * p->groups * kSsdChunk * kSsdChunk;
        a.col_blocks = (p->vdim + kSsdCols - 1) / kSsdCols;
        const int n8 = (p->n_state + 7) & ~7, n16 = (p->n_state + 15) & ~15;
        const size_t sm_cb = (size_t)2 * kSsdChunk * ssd_stride4(n8) * 4, sm_st = (size_t)kSsdChunk * (kSsdXs + ssd_stride8(n16)) * 4,
                     sm_out = ((size_t)kSsdChunk * (kSsdXs + kSsdMs + ssd_stride4(n8)) + (size_t)n8 * kSsdXs) * 4;
        // the attribute is set once per kernel: to the most any supported state size (256) needs
        static unsigned long long d0 = 0, d1 = 0, d2 = 0;
        cudaError_t e = ensure_max_dynamic_smem((const void*)ssd_cb_kernel, 2 * kSsdChunk * 260 * 4, d0);
        if (e == cudaSuccess) e = ensure_max_dynamic_smem((const void*)ssd_state_kernel, kSsdChunk * (kSsdXs + 264) * 4, d1);
        if (e == cudaSuccess) e = ensure_max_dynamic_smem((const void*)ssd_out_kernel, (kSsdChunk * (kSsdXs + kSsdMs + 260) + 256 * kSsdXs) * 4, d2);
        if (e != cudaSuccess) return (int)e;
        ssd_cb_kernel<<<dim3(p->n_entries, chunks, p->groups), 128, sm_cb, s>>>(a);
        const dim3 grid(p->n_entries * a.col_blocks, chunks, p->heads);
        ssd_state_kernel<<<grid, 128, sm_st, s>>>(a);
        const int per = p->n_state * p->vdim;   // a head's state starts on a multiple of `per` floats
        if (per % 4 == 0 && (reinterpret_cast<uintptr_t>(p->state) & 15u) == 0)
            ssd_carry_kernel<4><<<dim3(p->n_entries, p->heads, (per / 4 + 127) / 128), 128, 0, s>>>(a);
        else
            ssd_carry_kernel<1><<<dim3(p->n_entries, p->heads, (per + 127) / 128), 128, 0, s>>>(a);
        ssd_out_kernel<<<grid, 256, sm_out, s>>>(a);
        count_launch(4);
        return (int)cudaGetLastError();
    }
    return p->vdim <= 32 ? launch_walk<32>(a, p->n_entries, s) : launch_walk<64>(a, p->n_entries, s);
}

extern "C" int b200_gated_group_rms(const float* y, const float* z, long long ld_z, const float* w, void* out, int n_tokens, int n, int parts,
                                    float eps, int out_dtype, void* stream) {
    if (!y || !z || !w || !out || n_tokens < 0 || n < 1 || parts < 1 || n % parts || ld_z < n) return B200_EINVAL;
    if (n_tokens == 0) return B200_OK;
    const size_t smem = (size_t)(n / parts) * sizeof(float);
    if (smem > 200 * 1024 || parts > 65535) return B200_EUNSUPPORTED;
    const dim3 grid(n_tokens, parts);
    cudaStream_t s = (cudaStream_t)stream;
    const int per = n / parts;
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    if (per % 4 == 0 && per <= 16 * 512 && ld_z % 4 == 0 && al16(y) && al16(z) && al16(w) && al16(out) && (out_dtype == B200_BF16 || out_dtype == B200_F32)) {
        const bool bf = out_dtype == B200_BF16;
        if (per <= 16 * 128) {
            if (bf) gated_group_rms_reg_kernel<__nv_bfloat16, 128><<<grid, 128, 0, s>>>(y, z, ld_z, w, (__nv_bfloat16*)out, n, per, eps);
            else gated_group_rms_reg_kernel<float, 128><<<grid, 128, 0, s>>>(y, z, ld_z, w, (float*)out, n, per, eps);
        } else {
            if (bf) gated_group_rms_reg_kernel<__nv_bfloat16, 512><<<grid, 512, 0, s>>>(y, z, ld_z, w, (__nv_bfloat16*)out, n, per, eps);
            else gated_group_rms_reg_kernel<float, 512><<<grid, 512, 0, s>>>(y, z, ld_z, w, (float*)out, n, per, eps);
        }
        count_launch();
        return (int)cudaGetLastError();
    }
    if (out_dtype == B200_BF16) {
        static unsigned long long done = 0;
        if (smem > 48 * 1024) ensure_max_dynamic_smem((const void*)gated_group_rms_kernel<__nv_bfloat16>, 200 * 1024, done);
        gated_group_rms_kernel<__nv_bfloat16><<<grid, 128, smem, s>>>(y, z, ld_z, w, (__nv_bfloat16*)out, n, n / parts, eps);
    } else if (out_dtype == B200_F32) {
        static unsigned long long done = 0;
        if (smem > 48 * 1024) ensure_max_dynamic_smem((const void*)gated_group_rms_kernel<float>, 200 * 1024, done);
        gated_group_rms_kernel<float><<<grid, 128, smem, s>>>(y, z, ld_z, w, (float*)out, n, n / parts, eps);
    } else
        return B200_EINVAL;
    count_launch();
    return (int)cudaGetLastError();
}
