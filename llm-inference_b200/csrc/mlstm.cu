// Matrix memory with exponential input gates and sigmoid forget gates (the mLSTM cell), stabilised by a running maximum. Per head
// a state S (dim x vdim) with a normaliser n (dim) and a maximum m, all fp32 and carried per sequence slot:
//   i = cap tanh(raw_i / cap), f = log sigmoid(cap tanh(raw_f / cap)),  m' = max(f + m, i),
//   S' = exp(f + m - m') S + exp(i - m') k v^T, n' = exp(f + m - m') n + exp(i - m') k,
//   o = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6),   S, n, m start at zero.
//
//   mlstm_walk_kernel   one CTA per (entry, head, block of value columns): a thread owns one column of a share of the state rows
//                       in registers and walks the entry's tokens; one more warp carries n and forms the denominators. Every block
//                       of columns carries its own copy of (n, m), so no CTA reads what another one writes. All fp32. Decode
//                       batches, short portions and fp32 serving take this path.
//   chunk form (entries of 128 tokens and more, bfloat16 serving): 64-token chunks. With F the running sum of f inside the chunk,
//   a_j = i_j - F_j, A_i = max_(j<=i) a_j and m the maximum at the chunk's start, the recurrence gives m_i = F_i + g_i with
//   g_i = max(m, A_i), and a token j counts exp(a_j - g_i) at token i, the older state exp(m - g_i): every exponent is <= 0.
//     mlstm_qk_kernel     M_ij = exp(a_j - A_i) (q_i . k_j), j <= i, and its row sums, chunks in parallel;
//     mlstm_state_kernel  U = sum_j exp(a_j - A_end) k_j v_j^T and the same sum of the k_j, chunks in parallel;
//     mlstm_chain_kernel  the maximum at every chunk's start and the two factors of its carry;
//     mlstm_carry_kernel  S and n at the start of every chunk, and what the entry leaves behind;
//     mlstm_out_kernel    o_i = (exp(m - g_i) S^T q_i + exp(A_i - g_i) sum_j M_ij v_j) / denominator.
//   Products run on tf32 tensor-core tiles (mma.sync m16n8k8) with fp32 accumulation. q, k and v, which are projections, enter as one
//   tf32 number; what the recurrence itself made (the state, the weighted values, the weights M) enters as a sum of two, so it keeps
//   21 bits. Gates, maxima, factors, states, normalisers and everything between chunks are fp32, F and a are kept in double
//   (differences of two large sums are exponentiated).
#include <cuda_bf16.h>
#include <math.h>
#include <stdlib.h>

#include <algorithm>

#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"

namespace b200 {

struct ML {
    const float* proj; long long ld; int q_off, k_off, v_off, i_off, f_off;
    const float* i_bias; const float* f_bias; float cap, q_scale;
    float* state; float* norm; float* out;
    const int* ent_row; const int* ent_len; const int* slot; const int* pos;
    int heads, dim, vdim, norm_stride, copies;   // norm: [slot, head, copy, norm_stride] = n, padding, m last
    // chunk form: chunk c of entry e sits at place ent_row[e] / kMlChunk + e + c
    float* c_state;    // [place, head, dim, vdim]
    float* c_norm;     // [place, head, dim rounded up to 4]
    float* c_qk;       // [place, head, kMlChunk, kMlChunk]
    float* c_sum;      // [place, head, kMlChunk]: row sums of M
    float2* c_end;     // [place, head]: F_end, A_end
    float4* c_fac;     // [place, head]: m at the start, exp(m - g_end), exp(A_end - g_end)
    int col_blocks;
};

__device__ __forceinline__ float ml_gate_i(const ML& a, size_t row, int h) {
    return a.cap * tanhf((a.proj[row * a.ld + a.i_off + h] + a.i_bias[h]) / a.cap);
}
__device__ __forceinline__ float ml_gate_f(const ML& a, size_t row, int h) {
    const float z = a.cap * tanhf((a.proj[row * a.ld + a.f_off + h] + a.f_bias[h]) / a.cap);
    return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));   // log sigmoid
}

template <int NPT, int RG, int PB, int TOK>   // state rows per thread, row groups, value columns per CTA, tokens staged together
__global__ void __launch_bounds__(RG* PB + 32) mlstm_walk_kernel(const ML a) {
    constexpr int NP = NPT * RG, NT = RG * PB, ALL = NT + 32, NN = (NP + 31) / 32;
    __shared__ float ks[TOK][NP], qs[TOK][NP], vs[TOK][PB], part[TOK][RG][PB];
    __shared__ float keep[TOK], wr[TOK], floor_[TOK], inv_den[TOK];
    const int e = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PB, tid = threadIdx.x, lane = tid & 31;
    const bool walker = tid < NT;
    const int c = tid % PB, rg = walker ? tid / PB : 0, n0 = rg * NPT, N = a.dim, P = a.vdim;
    const int row0 = a.ent_row[e], len = a.ent_len[e], b = a.slot[row0];
    const bool live = walker && p0 + c < P, carried = a.pos[row0] > 0;
    float* st = a.state + (((size_t)b * a.heads + h) * N) * P + p0 + c;
    float* nm = a.norm + (((size_t)b * a.heads + h) * a.copies + blockIdx.z) * a.norm_stride;
    float S[NPT], nv[NN], m = 0.f;
#pragma unroll
    for (int k = 0; k < NPT; ++k) S[k] = (carried && live && n0 + k < N) ? st[(size_t)(n0 + k) * P] : 0.f;
#pragma unroll
    for (int k = 0; k < NN; ++k) nv[k] = (!walker && carried && lane + 32 * k < N) ? nm[lane + 32 * k] : 0.f;
    if (tid < 32 && carried) m = nm[a.norm_stride - 1];
    for (int t0 = 0; t0 < len; t0 += TOK) {
        const int nt = min(TOK, len - t0);
        __syncthreads();   // the previous group's readers are done
        for (int i = tid; i < nt * NP; i += ALL) {
            const int k = i / NP, n = i % NP;
            const float* row = a.proj + (size_t)(row0 + t0 + k) * a.ld + h * N + n;
            ks[k][n] = n < N ? row[a.k_off] : 0.f;
            qs[k][n] = n < N ? row[a.q_off] * a.q_scale : 0.f;
        }
        for (int i = tid; i < nt * PB; i += ALL) {
            const int k = i / PB, p = i % PB;
            vs[k][p] = p0 + p < P ? a.proj[(size_t)(row0 + t0 + k) * a.ld + a.v_off + h * P + p0 + p] : 0.f;
        }
        if (tid < 32) {   // gates of the group, a lane per token; the maximum runs along it in every lane
            const bool in = lane < nt;
            const float gi = in ? ml_gate_i(a, (size_t)(row0 + t0 + lane), h) : 0.f, gf = in ? ml_gate_f(a, (size_t)(row0 + t0 + lane), h) : 0.f;
            float my_fm = 0.f, my_m = 0.f;
            for (int k = 0; k < nt; ++k) {
                const float fm = __shfl_sync(0xffffffffu, gf, k) + m;
                m = fmaxf(fm, __shfl_sync(0xffffffffu, gi, k));
                if (lane == k) { my_fm = fm; my_m = m; }
            }
            if (in) {
                keep[lane] = expf(my_fm - my_m);
                wr[lane] = expf(gi - my_m);
                floor_[lane] = expf(-my_m);
            }
        }
        __syncthreads();
        if (walker) {
            for (int k = 0; k < nt; ++k) {
                const float dec = keep[k], vx = wr[k] * vs[k][c];
                float y = 0.f;
#pragma unroll
                for (int j = 0; j < NPT; ++j) {
                    S[j] = fmaf(dec, S[j], vx * ks[k][n0 + j]);
                    y = fmaf(S[j], qs[k][n0 + j], y);
                }
                part[k][rg][c] = y;
            }
        } else {
            for (int k = 0; k < nt; ++k) {
                const float dec = keep[k], w = wr[k];
                float y = 0.f;
#pragma unroll
                for (int j = 0; j < NN; ++j)
                    if (lane + 32 * j < NP) {
                        nv[j] = fmaf(dec, nv[j], w * ks[k][lane + 32 * j]);
                        y = fmaf(nv[j], qs[k][lane + 32 * j], y);
                    }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
                if (lane == 0) inv_den[k] = 1.f / (fmaxf(fabsf(y), floor_[k]) + 1e-6f);
            }
        }
        __syncthreads();
        for (int i = tid; i < nt * PB; i += ALL) {
            const int k = i / PB, p = i % PB;
            if (p0 + p >= P) continue;
            float y = 0.f;
#pragma unroll
            for (int q = 0; q < RG; ++q) y += part[k][q][p];
            a.out[(size_t)(row0 + t0 + k) * ((size_t)a.heads * P) + h * P + p0 + p] = y * inv_den[k];
        }
    }
    if (live) {
#pragma unroll
        for (int k = 0; k < NPT; ++k)
            if (n0 + k < N) st[(size_t)(n0 + k) * P] = S[k];
    }
    if (!walker) {
#pragma unroll
        for (int k = 0; k < NN; ++k)
            if (lane + 32 * k < N) nm[lane + 32 * k] = nv[k];
    }
    if (tid == 0) nm[a.norm_stride - 1] = m;
}

// ---------------------------------------------------------------------------------------------------------------
// chunk form
// ---------------------------------------------------------------------------------------------------------------
constexpr int kMlChunk = 64, kMlCols = 64, kMlVs = kMlCols + 8, kMlMs = kMlChunk + 4, kMlMaxDim = 256;
// row strides in floats: stride % 32 == 4 for operands whose rows run along the fragment's 8-wide index, 8 for those whose
// rows run along its 4-wide index (every fragment load then touches 32 different banks)
__host__ __device__ __forceinline__ int ml_stride4(int n) { return ((n + 31) & ~31) + 4; }
__host__ __device__ __forceinline__ int ml_stride8(int n) { return ((n + 31) & ~31) + 8; }

__device__ __forceinline__ float ml_tf32(float v) {
    uint32_t r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(v));
    return __uint_as_float(r);
}
__device__ __forceinline__ void ml_mma(float (&d)[4], const float (&a)[4], float b0, float b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])),
          "r"(__float_as_uint(b0)), "r"(__float_as_uint(b1)));
}

// v as the sum of two tf32 numbers
__device__ __forceinline__ void ml_split(float v, float& hi, float& lo) {
    hi = ml_tf32(v);
    lo = ml_tf32(v - hi);
}

// F, a and A of a chunk (double) by warp 0, two tokens per lane; places beyond the chunk hold the last F and A and a = -inf
struct MlGates {
    double F[kMlChunk], a[kMlChunk], A[kMlChunk];
};
__device__ __forceinline__ void ml_chunk_gates(const ML& a, int h, int row0, int len, MlGates& g) {
    if (threadIdx.x < 32) {
        const int l = threadIdx.x;
        double f[2], iv[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int i = 2 * l + k;
            f[k] = i < len ? (double)ml_gate_f(a, (size_t)(row0 + i), h) : 0.0;
            iv[k] = i < len ? (double)ml_gate_i(a, (size_t)(row0 + i), h) : -INFINITY;
        }
        double run = f[0] + f[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, run, o);
            if (l >= o) run += up;
        }
        const double F1 = run, F0 = run - f[1];
        const double a0 = iv[0] - F0, a1 = iv[1] - F1;
        double mx = fmax(a0, a1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, mx, o);
            if (l >= o) mx = fmax(mx, up);
        }
        const double before = __shfl_up_sync(0xffffffffu, mx, 1);
        g.F[2 * l] = F0;
        g.F[2 * l + 1] = F1;
        g.a[2 * l] = a0;
        g.a[2 * l + 1] = a1;
        g.A[2 * l] = l > 0 ? fmax(before, a0) : a0;
        g.A[2 * l + 1] = mx;
    }
}

// `rows` rows of `cols` columns from global (leading dimension ld) into shared memory, rows beyond `live` and columns beyond cols
// (up to cpad) zero; rows that allow it travel by cp.async (ml_landed() before the first read)
__device__ __forceinline__ void ml_stage(float* dst, int stride, const float* src, long long ld, int rows, int live, int cols, int cpad) {
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
__device__ __forceinline__ void ml_landed() {
    __syncwarp();   // the lanes close their group of copies together
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();
}

struct MlChunkAt {
    int row0, len, place;
    bool on;
};
__device__ __forceinline__ MlChunkAt ml_chunk_of(const ML& a, int e, int c) {
    const int row_e = a.ent_row[e], n = a.ent_len[e];
    return {row_e + c * kMlChunk, min(kMlChunk, n - c * kMlChunk), row_e / kMlChunk + e + c, c * kMlChunk < n};
}

__global__ void __launch_bounds__(128) mlstm_qk_kernel(const ML a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ MlGates gt;
    const MlChunkAt ck = ml_chunk_of(a, blockIdx.x, blockIdx.y);
    if (!ck.on) return;
    const int h = blockIdx.z, N = a.dim, npad = (N + 7) & ~7, st = ml_stride4(npad);
    float* Qs = sm;                      // [64][st]
    float* Ks = sm + kMlChunk * st;      // [64][st]
    const float* row = a.proj + (size_t)ck.row0 * a.ld + h * N;
    ml_stage(Qs, st, row + a.q_off, a.ld, kMlChunk, ck.len, N, npad);
    ml_stage(Ks, st, row + a.k_off, a.ld, kMlChunk, ck.len, N, npad);
    ml_chunk_gates(a, h, ck.row0, ck.len, gt);
    ml_landed();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3, m0 = warp * 16;
    float acc[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    for (int k0 = 0; k0 < npad; k0 += 8) {
        const float* ar = Qs + (m0 + gid) * st + k0 + tig;
        const float av[4] = {ml_tf32(ar[0]), ml_tf32(ar[8 * st]), ml_tf32(ar[4]), ml_tf32(ar[8 * st + 4])};
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            if (nt * 8 > m0 + 15) continue;   // keys behind all of the warp's rows
            const float* br = Ks + (nt * 8 + gid) * st + k0 + tig;
            ml_mma(acc[nt], av, ml_tf32(br[0]), ml_tf32(br[4]));
        }
    }
    const size_t at = (size_t)ck.place * a.heads + h;
    float* dst = a.c_qk + at * kMlChunk * kMlChunk;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int i = m0 + gid + half * 8;
        const double A = gt.A[i];
        float sum = 0.f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            float v[2];
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int j = nt * 8 + tig * 2 + x;
                v[x] = j <= i ? acc[nt][half * 2 + x] * a.q_scale * expf((float)(gt.a[j] - A)) : 0.f;
                sum += v[x];
            }
            *reinterpret_cast<float2*>(dst + i * kMlChunk + nt * 8 + tig * 2) = make_float2(v[0], v[1]);
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if (tig == 0) a.c_sum[at * kMlChunk + i] = sum;
    }
    if (threadIdx.x == 0) a.c_end[at] = make_float2((float)gt.F[kMlChunk - 1], (float)gt.A[kMlChunk - 1]);
}

__global__ void __launch_bounds__(128) mlstm_state_kernel(const ML a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ MlGates gt;
    __shared__ float wts[kMlChunk];
    const int e = blockIdx.x / a.col_blocks, p0 = (blockIdx.x % a.col_blocks) * kMlCols;
    const MlChunkAt ck = ml_chunk_of(a, e, blockIdx.y);
    if (!ck.on) return;
    const int h = blockIdx.z, N = a.dim, P = a.vdim, npad = (N + 15) & ~15, st = ml_stride8(npad);
    float* Vs = sm;                      // [64][kMlVs]
    float* Ks = sm + kMlChunk * kMlVs;   // [64][st]
    const int cols = min(kMlCols, P - p0);
    const float* row = a.proj + (size_t)ck.row0 * a.ld;
    ml_stage(Ks, st, row + a.k_off + h * N, a.ld, kMlChunk, ck.len, N, npad);
    ml_stage(Vs, kMlVs, row + a.v_off + h * P + p0, a.ld, kMlChunk, ck.len, cols, kMlCols);
    ml_chunk_gates(a, h, ck.row0, ck.len, gt);
    ml_landed();
    if (threadIdx.x < kMlChunk) wts[threadIdx.x] = expf((float)(gt.a[threadIdx.x] - gt.A[kMlChunk - 1]));   // beyond the chunk: exp(-inf) = 0
    __syncthreads();
    // the weights go into the value rows, in place
    for (int i = threadIdx.x; i < kMlChunk * (kMlCols / 4); i += 128) {
        float4* v4 = reinterpret_cast<float4*>(Vs + (i / (kMlCols / 4)) * kMlVs) + i % (kMlCols / 4);
        const float w = wts[i / (kMlCols / 4)];
        const float4 v = *v4;
        *v4 = make_float4(v.x * w, v.y * w, v.z * w, v.w * w);
    }
    const size_t at = (size_t)ck.place * a.heads + h;
    if (p0 == 0)   // the normaliser's share of the chunk, fp32
        for (int d = threadIdx.x; d < N; d += 128) {
            float s = 0.f;
            for (int j = 0; j < kMlChunk; ++j) s = fmaf(wts[j], Ks[j * st + d], s);
            a.c_norm[at * ((N + 3) & ~3) + d] = s;
        }
    __syncthreads();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    float* U = a.c_state + at * N * P + p0;
    const bool pair = (P & 1) == 0;
    for (int m0 = warp * 16; m0 < npad; m0 += 64) {
        float acc[8][4];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
#pragma unroll 2
        for (int k0 = 0; k0 < kMlChunk; k0 += 8) {
            const float* ar = Ks + (k0 + tig) * st + m0 + gid;
            const float av[4] = {ml_tf32(ar[0]), ml_tf32(ar[8]), ml_tf32(ar[4 * st]), ml_tf32(ar[4 * st + 8])};
            const float* br = Vs + (k0 + tig) * kMlVs + gid;
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) {
                float h0, l0, h1, l1;
                ml_split(br[nt * 8], h0, l0);
                ml_split(br[4 * kMlVs + nt * 8], h1, l1);
                ml_mma(acc[nt], av, h0, h1);
                ml_mma(acc[nt], av, l0, l1);
            }
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

// the maximum along the chunks of every (entry, head), a thread each; it leaves the entry's last maximum in every copy
__global__ void __launch_bounds__(128) mlstm_chain_kernel(const ML a) {
    const int e = blockIdx.x, h = blockIdx.y * blockDim.x + threadIdx.x;
    if (h >= a.heads) return;
    const int row_e = a.ent_row[e], n = a.ent_len[e], b = a.slot[row_e], chunks = (n + kMlChunk - 1) / kMlChunk;
    float* nm = a.norm + ((size_t)b * a.heads + h) * a.copies * a.norm_stride + a.norm_stride - 1;
    float m = a.pos[row_e] > 0 ? *nm : 0.f;
    const size_t first = (size_t)(row_e / kMlChunk + e) * a.heads + h;
    constexpr int F = 8;
    for (int c0 = 0; c0 < chunks; c0 += F) {   // F loads in flight, then the dependent chain
        float2 end[F];
#pragma unroll
        for (int k = 0; k < F; ++k)
            if (c0 + k < chunks) end[k] = a.c_end[first + (size_t)(c0 + k) * a.heads];
#pragma unroll
        for (int k = 0; k < F; ++k)
            if (c0 + k < chunks) {
                const float g = fmaxf(m, end[k].y);
                a.c_fac[first + (size_t)(c0 + k) * a.heads] = make_float4(m, expf(m - g), expf(end[k].y - g), 0.f);
                m = end[k].x + g;
            }
    }
    for (int z = 0; z < a.copies; ++z) nm[(size_t)z * a.norm_stride] = m;
}

// element-wise over the state and the normaliser (VEC consecutive elements per thread): leaves both at each chunk's start in place
// of the chunk's own share
template <int VEC> struct MlVec;
template <> struct MlVec<1> { using T = float; };
template <> struct MlVec<4> { using T = float4; };
__device__ __forceinline__ float ml_next(float S, float d, float u, float w) { return fmaf(d, S, w * u); }
__device__ __forceinline__ float4 ml_next(float4 S, float d, float4 u, float w) {
    return make_float4(fmaf(d, S.x, w * u.x), fmaf(d, S.y, w * u.y), fmaf(d, S.z, w * u.z), fmaf(d, S.w, w * u.w));
}

template <int VEC>
__global__ void __launch_bounds__(128) mlstm_carry_kernel(const ML a) {
    using V = typename MlVec<VEC>::T;
    const int e = blockIdx.x, h = blockIdx.y, per = a.dim * a.vdim / VEC, nper = (a.dim + VEC - 1) / VEC, npad4 = ((a.dim + 3) & ~3) / VEC;
    int i = blockIdx.z * blockDim.x + threadIdx.x;
    if (i >= per + nper) return;
    const bool is_n = i >= per;
    const int row_e = a.ent_row[e], n = a.ent_len[e], b = a.slot[row_e], chunks = (n + kMlChunk - 1) / kMlChunk;
    const size_t unit = (size_t)b * a.heads + h, first = (size_t)(row_e / kMlChunk + e);
    V *sp, *U;
    size_t step;
    if (!is_n) {
        sp = reinterpret_cast<V*>(a.state) + unit * per + i;
        U = reinterpret_cast<V*>(a.c_state) + (first * a.heads + h) * per + i;
        step = (size_t)a.heads * per;
    } else {
        i -= per;
        sp = reinterpret_cast<V*>(a.norm + unit * a.copies * a.norm_stride) + i;
        U = reinterpret_cast<V*>(a.c_norm) + (first * a.heads + h) * npad4 + i;
        step = (size_t)a.heads * npad4;
    }
    V S{};
    if (a.pos[row_e] > 0) S = *sp;
    const float4* fac = a.c_fac + first * a.heads + h;
    constexpr int F = 8;
    for (int c0 = 0; c0 < chunks; c0 += F) {   // F loads in flight, then the dependent chain
        V u[F];
        float2 d[F];
#pragma unroll
        for (int k = 0; k < F; ++k)
            if (c0 + k < chunks) {
                u[k] = U[(size_t)(c0 + k) * step];
                const float4 f4 = fac[(size_t)(c0 + k) * a.heads];
                d[k] = make_float2(f4.y, f4.z);
            }
#pragma unroll
        for (int k = 0; k < F; ++k)
            if (c0 + k < chunks) {
                U[(size_t)(c0 + k) * step] = S;
                S = ml_next(S, d[k].x, u[k], d[k].y);
            }
    }
    if (!is_n) *sp = S;
    else
        for (int z = 0; z < a.copies; ++z) *(reinterpret_cast<V*>(a.norm + (unit * a.copies + z) * a.norm_stride) + i) = S;
}

__global__ void __launch_bounds__(256) mlstm_out_kernel(const ML a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ MlGates gt;
    __shared__ float r_old[kMlChunk], r_new[kMlChunk], inv_den[kMlChunk];
    const int e = blockIdx.x / a.col_blocks, p0 = (blockIdx.x % a.col_blocks) * kMlCols;
    const MlChunkAt ck = ml_chunk_of(a, e, blockIdx.y);
    if (!ck.on) return;
    const int h = blockIdx.z, N = a.dim, P = a.vdim, npad = (N + 7) & ~7, st = ml_stride4(npad);
    float* Vs = sm;                               // [64][kMlVs]
    float* Ms = Vs + kMlChunk * kMlVs;            // [64][kMlMs]
    float* Qs = Ms + kMlChunk * kMlMs;            // [64][st]
    float* Ss = Qs + kMlChunk * st;               // [npad][kMlVs]
    const int cols = min(kMlCols, P - p0);
    const float* row = a.proj + (size_t)ck.row0 * a.ld;
    const size_t at = (size_t)ck.place * a.heads + h;
    ml_stage(Qs, st, row + a.q_off + h * N, a.ld, kMlChunk, ck.len, N, npad);
    ml_stage(Vs, kMlVs, row + a.v_off + h * P + p0, a.ld, kMlChunk, ck.len, cols, kMlCols);
    ml_stage(Ss, kMlVs, a.c_state + at * N * P + p0, P, npad, N, cols, kMlCols);
    ml_stage(Ms, kMlMs, a.c_qk + at * kMlChunk * kMlChunk, kMlChunk, kMlChunk, kMlChunk, kMlChunk, kMlChunk);
    ml_chunk_gates(a, h, ck.row0, ck.len, gt);
    ml_landed();
    {   // factors and denominators: four threads per row share the product of q with the older normaliser
        const int i = threadIdx.x >> 2, l4 = threadIdx.x & 3;
        const float* nrm = a.c_norm + at * ((N + 3) & ~3);
        float nq = 0.f;
        for (int d = l4; d < N; d += 4) nq = fmaf(Qs[i * st + d], nrm[d], nq);
        nq += __shfl_xor_sync(0xffffffffu, nq, 1);
        nq += __shfl_xor_sync(0xffffffffu, nq, 2);
        if (l4 == 0) {
            const double m = (double)a.c_fac[at].x, A = gt.A[i], g = fmax(m, A);
            const float ro = expf((float)(m - g)), rn = expf((float)(A - g));
            r_old[i] = ro * a.q_scale;
            r_new[i] = rn;
            inv_den[i] = 1.f / (fmaxf(fabsf(fmaf(ro * a.q_scale, nq, rn * a.c_sum[at * kMlChunk + i])), expf((float)(-(gt.F[i] + g)))) + 1e-6f);
        }
    }
    __syncthreads();
#pragma unroll 4
    for (int i = threadIdx.x; i < kMlChunk * kMlChunk; i += 256) {
        float* v = Ms + (i / kMlChunk) * kMlMs + i % kMlChunk;
        *v *= r_new[i / kMlChunk];
    }
    __syncthreads();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    const int m0 = (warp & 3) * 16, q0 = (warp >> 2) * 32;   // eight warps: 16 rows x 32 value columns each
    float acc[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    for (int k0 = 0; k0 < npad; k0 += 8) {   // what older chunks left
        const float* ar = Qs + (m0 + gid) * st + k0 + tig;
        const float av[4] = {ml_tf32(ar[0]), ml_tf32(ar[8 * st]), ml_tf32(ar[4]), ml_tf32(ar[8 * st + 4])};
        const float* br = Ss + (k0 + tig) * kMlVs + q0 + gid;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            float h0, l0, h1, l1;
            ml_split(br[nt * 8], h0, l0);
            ml_split(br[4 * kMlVs + nt * 8], h1, l1);
            ml_mma(acc[nt], av, h0, h1);
            ml_mma(acc[nt], av, l0, l1);
        }
    }
    const float e_lo = r_old[m0 + gid], e_hi = r_old[m0 + gid + 8];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) { acc[nt][0] *= e_lo; acc[nt][1] *= e_lo; acc[nt][2] *= e_hi; acc[nt][3] *= e_hi; }
    for (int k0 = 0; k0 < m0 + 16; k0 += 8) {   // this chunk's own tokens, up to the warp's last row
        const float* ar = Ms + (m0 + gid) * kMlMs + k0 + tig;
        float ah[4], al[4];
        ml_split(ar[0], ah[0], al[0]);
        ml_split(ar[8 * kMlMs], ah[1], al[1]);
        ml_split(ar[4], ah[2], al[2]);
        ml_split(ar[8 * kMlMs + 4], ah[3], al[3]);
        const float* br = Vs + (k0 + tig) * kMlVs + q0 + gid;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            const float b0 = ml_tf32(br[nt * 8]), b1 = ml_tf32(br[4 * kMlVs + nt * 8]);
            ml_mma(acc[nt], ah, b0, b1);
            ml_mma(acc[nt], al, b0, b1);
        }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int i = m0 + gid + (k >> 1) * 8, p = q0 + nt * 8 + tig * 2 + (k & 1);
            if (i < ck.len && p < cols)
                a.out[(size_t)(ck.row0 + i) * ((size_t)a.heads * P) + h * P + p0 + p] = acc[nt][k] * inv_den[i];
        }
}

static size_t ml_places(int n_tokens, int n_entries) { return (size_t)n_tokens / kMlChunk + (size_t)n_entries + 1; }
static int ml_copies(int vdim) { return vdim <= 32 ? 1 : (vdim + 63) / 64; }
static int ml_norm_stride(int dim) { return ((dim + 3) & ~3) + 4; }

template <int PB>
static int launch_ml_walk(const ML& a, int n_entries, cudaStream_t s) {
    const dim3 grid(n_entries, a.heads, (a.vdim + PB - 1) / PB);
    if (a.dim <= 16) mlstm_walk_kernel<4, 4, PB, 8><<<grid, 4 * PB + 32, 0, s>>>(a);
    else if (a.dim <= 32) mlstm_walk_kernel<8, 4, PB, 8><<<grid, 4 * PB + 32, 0, s>>>(a);
    else if (a.dim <= 64) mlstm_walk_kernel<16, 4, PB, 8><<<grid, 4 * PB + 32, 0, s>>>(a);
    else if (a.dim <= 128) mlstm_walk_kernel<32, 4, PB, 8><<<grid, 4 * PB + 32, 0, s>>>(a);
    else if (a.dim <= 256) mlstm_walk_kernel<64, 4, PB, 8><<<grid, 4 * PB + 32, 0, s>>>(a);
    else mlstm_walk_kernel<64, 8, PB, 4><<<grid, 8 * PB + 32, 0, s>>>(a);
    count_launch();
    return (int)cudaGetLastError();
}

}  // namespace b200

using namespace b200;

extern "C" size_t b200_mlstm_norm_floats(int dim, int vdim) {
    return dim > 0 && vdim > 0 ? (size_t)ml_copies(vdim) * ml_norm_stride(dim) : 0;
}

extern "C" size_t b200_mlstm_workspace_bytes(int n_tokens, int n_entries, int heads, int dim, int vdim) {
    if (n_tokens < 2 * kMlChunk || n_entries < 1 || heads < 1 || dim < 1 || vdim < 1 || dim > kMlMaxDim) return 0;
    const size_t per = (((size_t)dim * vdim + 3) & ~(size_t)3) + ((dim + 3) & ~3) + kMlChunk * kMlChunk + kMlChunk + 2 + 4;
    return ml_places(n_tokens, n_entries) * heads * per * sizeof(float) + 6 * 256;
}

extern "C" int b200_mlstm(const b200_mlstm_args* p, void* stream) {
    if (!p || !p->proj || !p->i_bias || !p->f_bias || !p->state || !p->norm || !p->out || !p->ent_row || !p->ent_len || !p->slot || !p->pos ||
        p->n_entries < 0 || p->n_tokens < 0 || p->heads < 1 || p->dim < 1 || p->vdim < 1 || p->q_off < 0 || p->k_off < 0 || p->v_off < 0 ||
        p->i_off < 0 || p->f_off < 0 || !(p->gate_cap > 0.f) || (reinterpret_cast<uintptr_t>(p->norm) & 15u))
        return B200_EINVAL;
    if (p->dim > 512 || p->heads > 65535 || p->vdim > 65535) return B200_EUNSUPPORTED;
    if (p->n_entries == 0 || p->n_tokens == 0) return B200_OK;
    ML a{p->proj, p->ld_proj, p->q_off, p->k_off, p->v_off, p->i_off, p->f_off, p->i_bias, p->f_bias, p->gate_cap, p->q_scale,
         p->state, p->norm, p->out, p->ent_row, p->ent_len, p->slot, p->pos, p->heads, p->dim, p->vdim, ml_norm_stride(p->dim), ml_copies(p->vdim),
         nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, 1};
    cudaStream_t s = (cudaStream_t)stream;
    const size_t need = b200_mlstm_workspace_bytes(p->n_tokens, p->n_entries, p->heads, p->dim, p->vdim);
    const int chunks = (p->longest_entry + kMlChunk - 1) / kMlChunk;
    if (p->chunked && p->longest_entry >= 2 * kMlChunk && need > 0 && p->workspace && p->workspace_bytes >= need && chunks <= 65535 &&
        (reinterpret_cast<uintptr_t>(p->workspace) & 15u) == 0) {
        const size_t units = ml_places(p->n_tokens, p->n_entries) * p->heads;
        char* w = reinterpret_cast<char*>(p->workspace);
        auto take = [&](auto*& dst, size_t bytes) { dst = reinterpret_cast<std::remove_reference_t<decltype(dst)>>(w); w += (bytes + 255) & ~(size_t)255; };
        take(a.c_state, units * p->dim * p->vdim * 4);
        take(a.c_norm, units * ((p->dim + 3) & ~3) * 4);
        take(a.c_qk, units * kMlChunk * kMlChunk * 4);
        take(a.c_sum, units * kMlChunk * 4);
        take(a.c_end, units * sizeof(float2));
        take(a.c_fac, units * sizeof(float4));
        a.col_blocks = (p->vdim + kMlCols - 1) / kMlCols;
        const int n8 = (p->dim + 7) & ~7, n16 = (p->dim + 15) & ~15;
        const size_t sm_qk = (size_t)2 * kMlChunk * ml_stride4(n8) * 4, sm_st = (size_t)kMlChunk * (kMlVs + ml_stride8(n16)) * 4,
                     sm_out = ((size_t)kMlChunk * (kMlVs + kMlMs + ml_stride4(n8)) + (size_t)n8 * kMlVs) * 4;
        // the attribute is set once per kernel: to the most any supported state size needs
        static unsigned long long d0 = 0, d1 = 0, d2 = 0;
        cudaError_t e = ensure_max_dynamic_smem((const void*)mlstm_qk_kernel, 2 * kMlChunk * (kMlMaxDim + 4) * 4, d0);
        if (e == cudaSuccess) e = ensure_max_dynamic_smem((const void*)mlstm_state_kernel, kMlChunk * (kMlVs + kMlMaxDim + 8) * 4, d1);
        if (e == cudaSuccess) e = ensure_max_dynamic_smem((const void*)mlstm_out_kernel, (kMlChunk * (kMlVs + kMlMs + kMlMaxDim + 4) + kMlMaxDim * kMlVs) * 4, d2);
        if (e != cudaSuccess) return (int)e;
        mlstm_qk_kernel<<<dim3(p->n_entries, chunks, p->heads), 128, sm_qk, s>>>(a);
        const dim3 grid(p->n_entries * a.col_blocks, chunks, p->heads);
        mlstm_state_kernel<<<grid, 128, sm_st, s>>>(a);
        mlstm_chain_kernel<<<dim3(p->n_entries, (p->heads + 127) / 128), 128, 0, s>>>(a);
        const int per = p->dim * p->vdim;   // a head's state starts on a multiple of `per` floats
        if (per % 4 == 0 && (reinterpret_cast<uintptr_t>(p->state) & 15u) == 0)
            mlstm_carry_kernel<4><<<dim3(p->n_entries, p->heads, (per / 4 + (p->dim + 3) / 4 + 127) / 128), 128, 0, s>>>(a);
        else
            mlstm_carry_kernel<1><<<dim3(p->n_entries, p->heads, (per + p->dim + 127) / 128), 128, 0, s>>>(a);
        mlstm_out_kernel<<<grid, 256, sm_out, s>>>(a);
        count_launch(5);
        return (int)cudaGetLastError();
    }
    return p->vdim <= 32 ? launch_ml_walk<32>(a, p->n_entries, s) : launch_ml_walk<64>(a, p->n_entries, s);
}
