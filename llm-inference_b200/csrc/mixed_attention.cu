// b200_paged_attention for designs that mix the softmax weights across the heads before they meet the values:
//   w_h(i, j) = softmax_j(scale temp[h] <q_i,h, k_j>),   o_h(i) = sum_j (sum_g mix[h, g] w_g(i, j)) v_j(key head of h),
// over the keys that position i sees (causal, block mask, sliding window). Every head needs every other head's NORMALISED
// weight of the same key, so nothing can run along the keys in one pass: the row's maxima and denominators come first.
//
//   mixed_attn_row_kernel   one CTA, or a cluster of up to sixteen CTAs that share the context, per token: ALL heads' scores of a
//                           tile of keys in shared memory, the row statistics (exchanged through distributed shared memory
//                           when several CTAs share the context), then weights, mix and weighted values, and the CTAs' partial
//                           outputs added in rank order. A share of keys that fits one tile keeps its scores, a longer one
//                           forms them again. fp32 arithmetic on caches of either dtype: single tokens, fp32 serving, odd
//                           sizes.
//   bfloat16 prompt portions, three launches per block of rows (scores and weights of a block live in the workspace, sized
//   to stay mostly in L2):
//     mixed_scores_kernel   64 rows x one head per CTA: scores on mma.sync tiles -> fp32 workspace, row maxima and
//                           denominators (online over the key tiles), and per row the range of columns it owns there;
//     mixed_mix_kernel      a thread per (row, two or four keys): the heads' weights in registers, the mix in fp32, rounded to
//                           bfloat16 only as the operand of the last product;
//     mixed_values_kernel   64 rows x one head per CTA: weights times values on mma.sync tiles.
#include <cooperative_groups.h>
#include <math.h>

#include <algorithm>

#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"
#include "paged_attention.cuh"

namespace b200 {

namespace cg = cooperative_groups;

constexpr int kMxThreads = 256, kMxWarps = kMxThreads / 32, kMxMaxCluster = 16;   // more than 8 CTAs per cluster: opt-in

struct MxRow {
    PA a;
    int kt;        // keys per tile (a multiple of 4)
    int vec;       // rows of K can be read in 16-byte pieces
    int vec4;      // rows of V can be read four values at a time
};

// scores of the tile's n keys (page rows in `rows`) for all heads; R heads of one key head share a pass over the key rows
template <typename T, int R>
__device__ __forceinline__ void mx_scores(const PA& a, const float* qs, const int* rows, float* sc, int kt, int n, int vec) {
    const T* K = reinterpret_cast<const T*>(a.k_pool);
    const int dim = a.dim, G = a.kv_heads, per = a.heads / G, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    if (vec) {
        constexpr int B = 4;   // four groups of four keys: their loads are in flight together
        const int blocks = (n + 4 * B - 1) / (4 * B), l8 = lane & 7;
        for (int w = warp; w < (a.heads / R) * blocks; w += kMxWarps) {
            const int u = w / blocks, k0 = (w - u * blocks) * 4 * B, g = u * R / per;
            float acc[B][R];
#pragma unroll
            for (int b = 0; b < B; ++b)
#pragma unroll
                for (int r = 0; r < R; ++r) acc[b][r] = 0.f;
            for (int i = l8 * 8; i < dim; i += 64) {
                float f[B][8];
#pragma unroll
                for (int b = 0; b < B; ++b) {
                    const int kk = min(k0 + 4 * b + (lane >> 3), n - 1);
                    const T* kr = K + ((size_t)rows[kk] * G + g) * dim + i;
                    if constexpr (sizeof(T) == 2) {
                        const Pack16 pk = ld16(kr);
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&pk.w[e]));
                            f[b][2 * e] = v.x;
                            f[b][2 * e + 1] = v.y;
                        }
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; e += 4) {
                            const Pack16 pk = ld16(kr + e);
#pragma unroll
                            for (int x = 0; x < 4; ++x) f[b][e + x] = __uint_as_float(pk.w[x]);
                        }
                    }
                }
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float* qr = qs + (u * R + r) * dim + i;
                    const float4 qa = *reinterpret_cast<const float4*>(qr), qb = *reinterpret_cast<const float4*>(qr + 4);
                    const float q8[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
                    for (int e = 0; e < 8; ++e)
#pragma unroll
                        for (int b = 0; b < B; ++b) acc[b][r] = fmaf(q8[e], f[b][e], acc[b][r]);
                }
            }
#pragma unroll
            for (int b = 0; b < B; ++b)
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    float v = acc[b][r];
                    v += __shfl_xor_sync(0xffffffffu, v, 1);
                    v += __shfl_xor_sync(0xffffffffu, v, 2);
                    v += __shfl_xor_sync(0xffffffffu, v, 4);
                    const int kk = k0 + 4 * b + (lane >> 3);
                    if (l8 == 0 && kk < n) sc[(u * R + r) * kt + kk] = v * pa_scale(a, u * R + r);
                }
        }
    } else {
        for (int i = threadIdx.x; i < a.heads * n; i += kMxThreads) {
            const int h = i / n, kk = i - h * n;
            const T* kr = K + ((size_t)rows[kk] * G + h / per) * dim;
            const float* q = qs + h * dim;
            float v = 0.f;
            for (int d = 0; d < dim; ++d) v = fmaf(q[d], DT<T>::to_f(kr[d]), v);
            sc[h * kt + kk] = v * pa_scale(a, h);
        }
    }
}

template <typename T, int VC> struct MxVal;   // VC consecutive values of one key
template <typename T> struct MxVal<T, 2> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[2]) {
        const float2 t = Pair<T>::load(p);
        v[0] = t.x; v[1] = t.y;
    }
};
template <> struct MxVal<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
};
template <> struct MxVal<__nv_bfloat16, 4> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
};
// om += mixed weights times values over the tile's n keys: a thread per VC value columns and R heads of one key head
template <typename T, int R, int VC>
__device__ __forceinline__ void mx_values(const T* V, const int* rows, const float* mx, float* om, int H, int G, int dv, int kt, int n) {
    const int hv = dv / VC, per = H / G;
    for (int i = threadIdx.x; i < (H / R) * hv; i += kMxThreads) {
        const int u = i / hv, c = VC * (i - u * hv), g = u * R / per;
        const float* w = mx + u * R * kt;
        float acc[R][VC];
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int x = 0; x < VC; ++x) acc[r][x] = 0.f;
        constexpr int F = R <= 4 ? 8 : 4;   // keys whose values are in flight together
        for (int k = 0; k < n; k += F) {
            float v[F][VC];
#pragma unroll
            for (int y = 0; y < F; ++y) MxVal<T, VC>::load(V + ((size_t)rows[min(k + y, n - 1)] * G + g) * dv + c, v[y]);
#pragma unroll
            for (int y0 = 0; y0 < F; y0 += 4) {
                if (k + y0 >= n) break;
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float4 w4 = *reinterpret_cast<const float4*>(w + r * kt + k + y0);
#pragma unroll
                    for (int x = 0; x < VC; ++x)
                        acc[r][x] = fmaf(w4.w, v[y0 + 3][x], fmaf(w4.z, v[y0 + 2][x], fmaf(w4.y, v[y0 + 1][x], fmaf(w4.x, v[y0][x], acc[r][x]))));
                }
            }
        }
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int x = 0; x < VC; ++x) om[(u * R + r) * dv + c + x] += acc[r][x];
    }
}

template <typename T, int R>
__global__ void __launch_bounds__(kMxThreads) mixed_attn_row_kernel(const MxRow m) {
    extern __shared__ __align__(16) float sm[];
    const PA& a = m.a;
    cg::cluster_group cluster = cg::this_cluster();
    const int C = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
    const int H = a.heads, G = a.kv_heads, dim = a.dim, dv = a.vdim, kt = m.kt, per = H / G;
    float* sc = sm;                       // [H][kt] scores, then weights
    float* mx = sc + H * kt;              // [H][kt] mixed weights
    float* qs = mx + H * kt;              // [H][dim]
    float* om = qs + H * dim;             // [H][dv]
    float* tk = om + H * dv;              // [H][H]
    float* st = tk + H * H;               // [2][H]: this CTA's maximum and denominator per head
    float* gl = st + 2 * H;               // [2][H]: the row's maximum and 1 / denominator
    int* rows = reinterpret_cast<int*>(gl + 2 * H);   // [kt]
    const int t = blockIdx.x / C, warp = threadIdx.x / 32, lane = threadIdx.x % 32, p = a.pos[t];
    const int* plist = a.pages + (size_t)a.slot[t] * a.max_pages;
    const T* q = reinterpret_cast<const T*>(a.q) + (size_t)t * H * dim;
    for (int i = threadIdx.x; i < H * dim; i += kMxThreads) qs[i] = DT<T>::to_f(q[i]);
    for (int i = threadIdx.x; i < H * H; i += kMxThreads) tk[i] = a.head_mix[i];
    for (int i = threadIdx.x; i < H * dv; i += kMxThreads) om[i] = 0.f;
    for (int i = threadIdx.x; i < H; i += kMxThreads) { st[i] = -INFINITY; st[H + i] = 0.f; }
    // this CTA's share of the visible keys
    const int lo = pa_first_key(a, p), share = ((p - lo + C) / C + 3) & ~3;
    const int j_begin = min(p + 1, lo + rank * share), j_end = min(p + 1, j_begin + share);
    const bool keep = j_end - j_begin <= kt;
    for (int j0 = j_begin; j0 < j_end; j0 += kt) {
        const int n = min(kt, j_end - j0);
        __syncthreads();
        for (int i = threadIdx.x; i < n; i += kMxThreads) rows[i] = plist[(j0 + i) / a.page_rows] * a.page_rows + (j0 + i) % a.page_rows;
        __syncthreads();
        mx_scores<T, R>(a, qs, rows, sc, kt, n, m.vec);
        __syncthreads();
        for (int h = warp; h < H; h += kMxWarps) {
            float bm = -INFINITY;
            for (int k = lane; k < n; k += 32) bm = fmaxf(bm, sc[h * kt + k]);
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, d));
            const float mo = st[h], mn = fmaxf(mo, bm);
            float s = 0.f;
            for (int k = lane; k < n; k += 32) s += expf(sc[h * kt + k] - mn);
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
            __syncwarp();
            if (lane == 0) {
                st[H + h] = st[H + h] * expf(mo - mn) + s;
                st[h] = mn;
            }
        }
    }
    // the row's statistics over all shares, in rank order (an empty share holds -inf, 0)
    if (C > 1) cluster.sync();
    else __syncthreads();
    for (int h = threadIdx.x; h < H; h += kMxThreads) {
        float M = -INFINITY, L = 0.f;
        for (int r = 0; r < C; ++r) M = fmaxf(M, C > 1 ? cluster.map_shared_rank(st, r)[h] : st[h]);
        for (int r = 0; r < C; ++r) {
            const float* s = C > 1 ? cluster.map_shared_rank(st, r) : st;
            if (s[H + h] > 0.f) L += s[H + h] * expf(s[h] - M);
        }
        gl[h] = M;
        gl[H + h] = 1.0f / L;
    }
    const T* V = reinterpret_cast<const T*>(a.v_pool);
    for (int j0 = j_begin; j0 < j_end; j0 += kt) {
        const int n = min(kt, j_end - j0), n4 = (n + 3) & ~3;
        __syncthreads();
        if (!keep) {
            for (int i = threadIdx.x; i < n; i += kMxThreads) rows[i] = plist[(j0 + i) / a.page_rows] * a.page_rows + (j0 + i) % a.page_rows;
            __syncthreads();
            mx_scores<T, R>(a, qs, rows, sc, kt, n, m.vec);
            __syncthreads();
        }
        for (int i = threadIdx.x; i < H * n; i += kMxThreads) {
            const int h = i / n, k = i - h * n;
            sc[h * kt + k] = expf(sc[h * kt + k] - gl[h]) * gl[H + h];
        }
        __syncthreads();
        for (int i = threadIdx.x; i < H * n4; i += kMxThreads) {   // consecutive threads: consecutive keys of one head
            const int h = i / n4, k = i - h * n4;
            float v = 0.f;
            if (k < n)
                for (int g = 0; g < H; ++g) v = fmaf(tk[h * H + g], sc[g * kt + k], v);
            mx[h * kt + k] = v;   // places behind the last key are 0
        }
        __syncthreads();
        if (dv % 4 == 0 && m.vec4)
            mx_values<T, R, 4>(V, rows, mx, om, H, G, dv, kt, n);
        else if (dv % 2 == 0) {
            mx_values<T, R, 2>(V, rows, mx, om, H, G, dv, kt, n);
        } else {
            for (int i = threadIdx.x; i < H * dv; i += kMxThreads) {
                const int h = i / dv, c = i - h * dv, g = h / per;
                float acc = 0.f;
                for (int k = 0; k < n; ++k) acc = fmaf(mx[h * kt + k], DT<T>::to_f(V[((size_t)rows[k] * G + g) * dv + c]), acc);
                om[i] += acc;
            }
        }
    }
    const size_t dst = (size_t)t * H * dv;
    if (C == 1) {
        __syncthreads();
        for (int i = threadIdx.x; i < H * dv; i += kMxThreads) pa_store<T>(a, dst + i, om[i]);
        return;
    }
    cluster.sync();
    for (int i = rank * kMxThreads + threadIdx.x; i < H * dv; i += C * kMxThreads) {
        float v = 0.f;
        for (int r = 0; r < C; ++r) v += cluster.map_shared_rank(om, r)[i];
        pa_store<T>(a, dst + i, v);
    }
    cluster.sync();   // nobody leaves while its shared memory is read
}

static size_t mx_row_floats(int H, int dim, int dv) { return (size_t)H * dim + (size_t)H * dv + (size_t)H * H + 4 * (size_t)H; }
constexpr size_t kMxSmem = 200 * 1024;

template <typename T, int R>
static int launch_mx_row(MxRow m, int cluster, size_t smem, cudaStream_t s) {
    static unsigned long long done = 0;
    cudaError_t e = ensure_max_dynamic_smem((const void*)mixed_attn_row_kernel<T, R>, (int)kMxSmem, done);
    if (e == cudaSuccess && cluster > 8) {
        static unsigned long long wide = 0;
        const int dev = current_device();
        if (!(wide & (1ull << dev))) {
            e = cudaFuncSetAttribute((const void*)mixed_attn_row_kernel<T, R>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
            if (e == cudaSuccess) wide |= 1ull << dev;
        }
    }
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3((unsigned)m.a.n_tokens * cluster);
    cfg.blockDim = dim3(kMxThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = (unsigned)cluster;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    cfg.attrs = at;
    cfg.numAttrs = 1;
    e = cudaLaunchKernelEx(&cfg, mixed_attn_row_kernel<T, R>, m);
    if (e != cudaSuccess) return (int)e;
    count_launch();
    return (int)cudaGetLastError();
}
template <typename T>
static int launch_mx_row_for(const MxRow& m, int cluster, size_t smem, cudaStream_t s) {
    const int per = m.a.heads / m.a.kv_heads;
    if (per % 8 == 0) return launch_mx_row<T, 8>(m, cluster, smem, s);
    if (per % 4 == 0) return launch_mx_row<T, 4>(m, cluster, smem, s);
    if (per % 2 == 0) return launch_mx_row<T, 2>(m, cluster, smem, s);
    return launch_mx_row<T, 1>(m, cluster, smem, s);
}

// ---------------------------------------------------------------------------------------------------------------
// prompt portions: tiles of 64 rows x 64 keys
// ---------------------------------------------------------------------------------------------------------------
constexpr int kMxTile = 64;

struct MxTile {
    PA a;
    int row0, n_rows;      // rows [row0, row0 + n_rows) of the batch; row0 a multiple of 64
    int width;             // columns per (row, head) of the workspace, a multiple of 64
    float* s;              // [n_rows, heads, width] scores
    __nv_bfloat16* w;      // [n_rows, heads, width] mixed weights
    float2* stat;          // [n_rows, heads] (maximum, 1 / denominator)
    int2* range;           // [n_rows] (key of column 0, columns in use: whole tiles)
};

// one segment of a row tile: consecutive rows of one sequence
struct MxSeg {
    int end, slot, base, n_keys;
};
__device__ __forceinline__ MxSeg mx_segment(const PA& a, const int* row_pos, const int* row_slot, int rows, int seg) {
    MxSeg g;
    g.slot = row_slot[seg];
    g.end = seg + 1;
    while (g.end < rows && row_slot[g.end] == g.slot) ++g.end;
    g.n_keys = row_pos[g.end - 1] + 1;                                     // positions grow along an entry
    g.base = pa_first_key(a, row_pos[seg]) / kMxTile * kMxTile;            // whole tiles from the first row's first key
    return g;
}
__device__ __forceinline__ void mx_cp16(void* dst, const void* src, bool on) {   // 16 bytes, zeros when off (nothing is read)
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(on ? 16 : 0) : "memory");
}

__global__ void __launch_bounds__(128) mixed_scores_kernel(const MxTile m) {
    using bf = __nv_bfloat16;
    extern __shared__ __align__(16) unsigned char mx_smem[];
    const PA& a = m.a;
    const int dim = a.dim, dpad = (dim + 15) & ~15, RS = dpad + 8, CH = dpad / 8;
    bf* Qs = reinterpret_cast<bf*>(mx_smem);          // [64][RS]
    bf* Ks = Qs + kMxTile * RS;                       // [2][64][RS]
    int* row_pos = reinterpret_cast<int*>(Ks + 2 * kMxTile * RS);
    int* row_slot = row_pos + kMxTile;
    const int l0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kMxTile, t0 = m.row0 + l0, h = blockIdx.y;
    const int G = a.kv_heads, g = h / (a.heads / G), warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    const int rows = min(kMxTile, m.n_rows - l0);
    for (int r = threadIdx.x; r < kMxTile; r += blockDim.x) {
        row_pos[r] = r < rows ? a.pos[t0 + r] : -1;
        row_slot[r] = r < rows ? a.slot[t0 + r] : -1;
    }
    const bf* Q = reinterpret_cast<const bf*>(a.q);
    for (int i = threadIdx.x; i < kMxTile * CH; i += blockDim.x) {
        const int r = i / CH, c = (i - r * CH) * 8;
        mx_cp16(Qs + r * RS + c, Q + ((size_t)(t0 + (r < rows ? r : 0)) * a.heads + h) * dim + (c < dim ? c : 0), r < rows && c < dim);
    }
    __syncwarp();   // the lanes close their group of copies together
    asm volatile("cp.async.commit_group;" ::: "memory");
    __syncthreads();
    const bf* Kp = reinterpret_cast<const bf*>(a.k_pool);
    const int r_lo = warp * 16 + gid, r_hi = r_lo + 8;
    const float sc_h = pa_scale(a, h);
    // a thread keeps its 16-byte column of a key tile when the columns divide the threads and a page holds whole tiles
    const bool one_page = a.page_rows % kMxTile == 0 && 128 % CH == 0;
    const int c_own = (threadIdx.x % CH) * 8, r_own = threadIdx.x / CH, r_step = 128 / CH;
    float m_run[2] = {-1e30f, -1e30f}, l_run[2] = {0.f, 0.f};
    for (int seg = 0; seg < rows;) {
        const MxSeg sg = mx_segment(a, row_pos, row_slot, rows, seg);
        const int* plist = a.pages + (size_t)sg.slot * a.max_pages;
        const int p_lo = (r_lo >= seg && r_lo < sg.end) ? row_pos[r_lo] : -1, p_hi = (r_hi >= seg && r_hi < sg.end) ? row_pos[r_hi] : -1;
        const int f_lo = p_lo >= 0 ? pa_first_key(a, p_lo) : 0, f_hi = p_hi >= 0 ? pa_first_key(a, p_hi) : 0;
        const int w_first = max(seg, warp * 16), w_last = min(sg.end, warp * 16 + 16) - 1;
        const int warp_keys = w_last >= w_first ? row_pos[w_last] + 1 : 0, warp_first = w_last >= w_first ? pa_first_key(a, row_pos[w_first]) : 0;
        if (h == 0)
            for (int r = seg + threadIdx.x; r < sg.end; r += blockDim.x)
                m.range[l0 + r] = make_int2(sg.base, (sg.n_keys - sg.base + kMxTile - 1) / kMxTile * kMxTile);
        auto load_tile = [&](int k0, int buf) {
            bf* kd = Ks + buf * kMxTile * RS;
            if (one_page) {   // whole rows per step of the threads: one lookup, no divisions
                const size_t row = (size_t)plist[k0 / a.page_rows] * a.page_rows + k0 % a.page_rows;
                const bf* src = Kp + (row * G + g) * dim + c_own;
                for (int kr = r_own; kr < kMxTile; kr += r_step) {
                    const bool ok = k0 + kr < sg.n_keys && c_own < dim;
                    mx_cp16(kd + kr * RS + c_own, ok ? src + (size_t)kr * G * dim : Kp, ok);
                }
            } else
                for (int i = threadIdx.x; i < kMxTile * CH; i += blockDim.x) {
                    const int kr = i / CH, c = (i - kr * CH) * 8, j = k0 + kr;
                    const bool ok = j < sg.n_keys && c < dim;
                    const size_t row = ok ? (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows : 0;
                    mx_cp16(kd + kr * RS + c, Kp + (row * G + g) * dim + (ok ? c : 0), ok);
                }
            __syncwarp();   // the lanes close their group of copies together
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        __syncthreads();   // the buffers of the previous segment are no longer read
        load_tile(sg.base, 0);
        int buf = 0;
        for (int k0 = sg.base; k0 < sg.n_keys; k0 += kMxTile, buf ^= 1) {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();   // tile k0 (and Q) has landed for everybody; the other buffer is no longer read
            if (k0 + kMxTile < sg.n_keys) load_tile(k0 + kMxTile, buf ^ 1);
            if (k0 >= warp_keys || k0 + kMxTile <= warp_first) continue;   // nothing for this warp's rows in this tile
            const bf* Kb = Ks + buf * kMxTile * RS;
            float s[8][4];
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
            for (int ks = 0; ks < dpad; ks += 16) {
                uint32_t qf[4];
                pa_ldsm_x4(qf, Qs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RS + ks + (lane >> 4) * 8);
#pragma unroll
                for (int nt = 0; nt < 8; nt += 2) {   // fragments of two key columns: (keys 0-7 | 8-15) x (k 0-7 | 8-15)
                    uint32_t b4[4];
                    pa_ldsm_x4(b4, Kb + (nt * 8 + (lane & 7) + ((lane >> 4) & 1) * 8) * RS + ks + ((lane >> 3) & 1) * 8);
                    const uint32_t b0[2] = {b4[0], b4[1]}, b1[2] = {b4[2], b4[3]};
                    pa_mma(s[nt], qf, b0);
                    pa_mma(s[nt + 1], qf, b1);
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = k0 + nt * 8 + tig * 2 + (e & 1);
                    const bool seen = j <= ((e & 2) ? p_hi : p_lo) && j >= ((e & 2) ? f_hi : f_lo);
                    s[nt][e] = seen ? s[nt][e] * sc_h : -INFINITY;
                    mx[e >> 1] = fmaxf(mx[e >> 1], s[nt][e]);
                }
#pragma unroll
            for (int hr = 0; hr < 2; ++hr) {
                const int r = hr ? r_hi : r_lo;
                if ((hr ? p_hi : p_lo) < 0) continue;   // (uniform over the four lanes of the row)
                float* dst = m.s + ((size_t)(l0 + r) * a.heads + h) * m.width + (k0 - sg.base) + tig * 2;
#pragma unroll
                for (int nt = 0; nt < 8; ++nt) *reinterpret_cast<float2*>(dst + nt * 8) = make_float2(s[nt][hr * 2], s[nt][hr * 2 + 1]);
            }
#pragma unroll
            for (int hr = 0; hr < 2; ++hr) {
                mx[hr] = fmaxf(mx[hr], __shfl_xor_sync(0xffffffffu, mx[hr], 1));
                mx[hr] = fmaxf(mx[hr], __shfl_xor_sync(0xffffffffu, mx[hr], 2));
                const float mn = fmaxf(m_run[hr], mx[hr]);   // finite: m starts at -1e30
                float sum = 0.f;
#pragma unroll
                for (int nt = 0; nt < 8; ++nt) sum += __expf(s[nt][hr * 2] - mn) + __expf(s[nt][hr * 2 + 1] - mn);
                sum += __shfl_xor_sync(0xffffffffu, sum, 1);
                sum += __shfl_xor_sync(0xffffffffu, sum, 2);
                l_run[hr] = l_run[hr] * __expf(m_run[hr] - mn) + sum;
                m_run[hr] = mn;
            }
        }
        seg = sg.end;
    }
    if (tig == 0) {
        if (r_lo < rows) m.stat[(size_t)(l0 + r_lo) * a.heads + h] = make_float2(m_run[0], 1.0f / l_run[0]);
        if (r_hi < rows) m.stat[(size_t)(l0 + r_hi) * a.heads + h] = make_float2(m_run[1], 1.0f / l_run[1]);
    }
}

template <int CW> struct MxCols;   // CW consecutive columns of one head
template <> struct MxCols<2> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[2]) {
        const float2 t = *reinterpret_cast<const float2*>(p);
        v[0] = t.x; v[1] = t.y;
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[2]) {
        *reinterpret_cast<uint32_t*>(p) = pa_pack(v[0], v[1]);
    }
};
template <> struct MxCols<4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
        *reinterpret_cast<uint2*>(p) = make_uint2(pa_pack(v[0], v[1]), pa_pack(v[2], v[3]));
    }
};

template <int HP, int CW>   // heads rounded up (8, 16, 32 or 64), columns per thread
__global__ void __launch_bounds__(128) mixed_mix_kernel(const MxTile m) {
    extern __shared__ __align__(16) float tk[];   // [heads][HP] mix, columns behind the last head zero; then [heads] (max, 1 / den)
    const PA& a = m.a;
    const int H = a.heads, l = blockIdx.x;
    const int2 rg = m.range[l];
    if (blockIdx.y * 128 * CW >= rg.y) return;
    float2* st = reinterpret_cast<float2*>(tk + H * HP);
    for (int i = threadIdx.x; i < H * HP; i += 128) {
        const int h = i / HP, g = i % HP;
        tk[i] = g < H ? a.head_mix[h * H + g] : 0.f;
    }
    for (int i = threadIdx.x; i < H; i += 128) st[i] = m.stat[(size_t)l * H + i];
    const int col = (blockIdx.y * 128 + threadIdx.x) * CW;
    const bool mine = col < rg.y;                 // whole tiles of 64 columns: a thread's columns are all inside or all outside
    const int p = a.pos[m.row0 + l], f = pa_first_key(a, p), j = rg.x + col;
    const bool any = mine && j + CW > f && j <= p;
    const size_t row = (size_t)l * H * m.width + col;
    float w[HP][CW];
#pragma unroll
    for (int g = 0; g < HP; ++g) {
#pragma unroll
        for (int c = 0; c < CW; ++c) w[g][c] = 0.f;
        if (any && g < H) MxCols<CW>::load(m.s + row + (size_t)g * m.width, w[g]);
    }
    __syncthreads();
    if (!mine) return;
    __nv_bfloat16* dst = m.w + row;
    if (any) {
#pragma unroll
        for (int g = 0; g < HP; ++g)
            if (g < H) {
                const float2 sg = st[g];
#pragma unroll
                for (int c = 0; c < CW; ++c) w[g][c] = (j + c >= f && j + c <= p) ? __expf(w[g][c] - sg.x) * sg.y : 0.f;
            }
    }
    for (int h = 0; h < H; ++h) {
        float v[CW];
#pragma unroll
        for (int c = 0; c < CW; ++c) v[c] = 0.f;
        if (any) {
#pragma unroll
            for (int g = 0; g < HP; g += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(tk + h * HP + g);
#pragma unroll
                for (int c = 0; c < CW; ++c)
                    v[c] = fmaf(k4.w, w[g + 3][c], fmaf(k4.z, w[g + 2][c], fmaf(k4.y, w[g + 1][c], fmaf(k4.x, w[g][c], v[c]))));
            }
        }
        MxCols<CW>::store(dst + (size_t)h * m.width, v);   // columns that the row does not see: weights of zero
    }
}

template <int NT>   // n8 tiles of the values: vdim <= 8 * NT
__global__ void __launch_bounds__(128) mixed_values_kernel(const MxTile m) {
    using bf = __nv_bfloat16;
    extern __shared__ __align__(16) unsigned char mx_smem[];
    const PA& a = m.a;
    constexpr int PS = kMxTile + 8, RSV = NT * 8 + 8;
    bf* Ws = reinterpret_cast<bf*>(mx_smem);          // [2][64][PS]
    bf* Vs = Ws + 2 * kMxTile * PS;                   // [2][64][RSV]
    int* row_pos = reinterpret_cast<int*>(Vs + 2 * kMxTile * RSV);
    int* row_slot = row_pos + kMxTile;
    const int l0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kMxTile, t0 = m.row0 + l0, h = blockIdx.y;
    const int G = a.kv_heads, g = h / (a.heads / G), dv = a.vdim, warp = threadIdx.x / 32, lane = threadIdx.x % 32, gid = lane >> 2, tig = lane & 3;
    const int rows = min(kMxTile, m.n_rows - l0);
    for (int r = threadIdx.x; r < kMxTile; r += blockDim.x) {
        row_pos[r] = r < rows ? a.pos[t0 + r] : -1;
        row_slot[r] = r < rows ? a.slot[t0 + r] : -1;
    }
    __syncthreads();
    const bf* Vp = reinterpret_cast<const bf*>(a.v_pool);
    float o[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    for (int seg = 0; seg < rows;) {
        const MxSeg sg = mx_segment(a, row_pos, row_slot, rows, seg);
        const int* plist = a.pages + (size_t)sg.slot * a.max_pages;
        const int w_first = max(seg, warp * 16), w_last = min(sg.end, warp * 16 + 16) - 1;
        const int warp_keys = w_last >= w_first ? row_pos[w_last] + 1 : 0, warp_first = w_last >= w_first ? pa_first_key(a, row_pos[w_first]) : 0;
        auto load_tile = [&](int k0, int buf) {
            bf* wd = Ws + buf * kMxTile * PS;
            bf* vd = Vs + buf * kMxTile * RSV;
            for (int i = threadIdx.x; i < kMxTile * 8; i += blockDim.x) {
                const int r = i / 8, c = (i & 7) * 8;
                const bool ok = r >= seg && r < sg.end;   // rows of other sequences: zero weights
                mx_cp16(wd + r * PS + c, m.w + ((size_t)(l0 + (ok ? r : 0)) * a.heads + h) * m.width + (ok ? k0 - sg.base + c : 0), ok);
            }
            const bool one_page = a.page_rows % kMxTile == 0;
            const size_t base = one_page ? (size_t)plist[k0 / a.page_rows] * a.page_rows + k0 % a.page_rows : 0;
#pragma unroll
            for (int i = threadIdx.x; i < kMxTile * NT; i += 128) {
                const int kr = i / NT, c = (i - kr * NT) * 8, j = k0 + kr;
                const bool ok = j < sg.n_keys && c < dv;
                const size_t row = !ok ? 0 : one_page ? base + kr : (size_t)plist[j / a.page_rows] * a.page_rows + j % a.page_rows;
                mx_cp16(vd + kr * RSV + c, Vp + (row * G + g) * dv + (ok ? c : 0), ok);
            }
            __syncwarp();   // the lanes close their group of copies together
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        __syncthreads();
        load_tile(sg.base, 0);
        int buf = 0;
        for (int k0 = sg.base; k0 < sg.n_keys; k0 += kMxTile, buf ^= 1) {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
            if (k0 + kMxTile < sg.n_keys) load_tile(k0 + kMxTile, buf ^ 1);
            if (k0 >= warp_keys || k0 + kMxTile <= warp_first) continue;
            const bf* Wb = Ws + buf * kMxTile * PS;
            const bf* Vb = Vs + buf * kMxTile * RSV;
#pragma unroll
            for (int kk = 0; kk < kMxTile / 16; ++kk) {
                uint32_t pf[4];
                pa_ldsm_x4(pf, Wb + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int nt = 0; nt < NT; nt += 2) {
                    uint32_t b4[4];
                    pa_ldsm_x4_trans(b4, Vb + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RSV + (nt + (lane >> 4)) * 8);
                    const uint32_t b0[2] = {b4[0], b4[1]}, b1[2] = {b4[2], b4[3]};
                    pa_mma(o[nt], pf, b0);
                    pa_mma(o[nt + 1], pf, b1);
                }
            }
        }
        seg = sg.end;
    }
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
        const int r = warp * 16 + gid + hr * 8;
        if (r >= rows) continue;
        const size_t dst = ((size_t)(t0 + r) * a.heads + h) * dv + tig * 2;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
            if (nt * 8 >= dv) continue;   // vdim is a multiple of 8
            if (a.out_f32) *reinterpret_cast<float2*>(reinterpret_cast<float*>(a.out) + dst + nt * 8) = make_float2(o[nt][hr * 2], o[nt][hr * 2 + 1]);
            else *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf*>(a.out) + dst + nt * 8) = __floats2bfloat162_rn(o[nt][hr * 2], o[nt][hr * 2 + 1]);
        }
    }
}

// columns of the workspace per (row, head): what the rows of one tile can see together, whole key tiles
static long long mx_width(int span, int longest) {
    const long long all = ((long long)longest + kMxTile - 1) / kMxTile * kMxTile;
    return span > 0 ? std::min(all, ((long long)span + 2 * kMxTile - 2 + kMxTile - 1) / kMxTile * kMxTile) : all;
}
static size_t mx_row_bytes(int heads, long long width) { return (size_t)heads * width * 6 + (size_t)heads * 8 + 8; }
constexpr size_t kMxBlockBytes = 256ull << 20, kMxMostBytes = 1024ull << 20;   // a block of rows: mostly L2; never more than 1 GB

// rows per block: whole tiles
static int mx_block_rows(int n_tokens, size_t row_bytes) {
    const long long tiles = std::max<long long>(1, (long long)(kMxBlockBytes / row_bytes) / kMxTile);
    return (int)std::min<long long>(tiles * kMxTile, ((long long)n_tokens + kMxTile - 1) / kMxTile * kMxTile);
}

template <int NT>
static int launch_values(const MxTile& m, dim3 grid, cudaStream_t s) {
    constexpr int smem = 2 * kMxTile * (kMxTile + 8) * 2 + 2 * kMxTile * (NT * 8 + 8) * 2 + 2 * kMxTile * 4;
    static unsigned long long done = 0;
    const cudaError_t e = ensure_max_dynamic_smem((const void*)mixed_values_kernel<NT>, smem, done);
    if (e != cudaSuccess) return (int)e;
    mixed_values_kernel<NT><<<grid, 128, smem, s>>>(m);
    return (int)cudaGetLastError();
}

static int mixed_tiles(const PA& a, int span, int longest_context, void* workspace, size_t workspace_bytes, cudaStream_t s) {
    const long long width = mx_width(span, longest_context);
    const size_t rb = mx_row_bytes(a.heads, width);
    const int block = mx_block_rows(a.n_tokens, rb);
    if (width > 0x7fffffff || (size_t)block * rb > workspace_bytes) return B200_EUNSUPPORTED;
    MxTile m{a, 0, 0, (int)width, nullptr, nullptr, nullptr, nullptr};
    m.s = reinterpret_cast<float*>(workspace);
    m.w = reinterpret_cast<__nv_bfloat16*>(m.s + (size_t)block * a.heads * width);
    m.stat = reinterpret_cast<float2*>(m.w + (size_t)block * a.heads * width);
    m.range = reinterpret_cast<int2*>(m.stat + (size_t)block * a.heads);
    const int dpad = (a.dim + 15) & ~15;
    const int sm1 = 3 * kMxTile * (dpad + 8) * 2 + 2 * kMxTile * 4;
    static unsigned long long done1 = 0;
    const cudaError_t e = ensure_max_dynamic_smem((const void*)mixed_scores_kernel, 3 * kMxTile * (256 + 8) * 2 + 2 * kMxTile * 4, done1);
    if (e != cudaSuccess) return (int)e;
    for (m.row0 = 0; m.row0 < a.n_tokens; m.row0 += block) {
        m.n_rows = std::min(block, a.n_tokens - m.row0);
        const dim3 grid((m.n_rows + kMxTile - 1) / kMxTile, a.heads);
        mixed_scores_kernel<<<grid, 128, sm1, s>>>(m);
        const dim3 gm4(m.n_rows, (unsigned)((width + 511) / 512)), gm2(m.n_rows, (unsigned)((width + 255) / 256));
        auto mix_smem = [&](int hp) { return (size_t)a.heads * hp * 4 + (size_t)a.heads * 8; };
        if (a.heads <= 8) mixed_mix_kernel<8, 4><<<gm4, 128, mix_smem(8), s>>>(m);
        else if (a.heads <= 16) mixed_mix_kernel<16, 4><<<gm4, 128, mix_smem(16), s>>>(m);
        else if (a.heads <= 32) mixed_mix_kernel<32, 4><<<gm4, 128, mix_smem(32), s>>>(m);
        else mixed_mix_kernel<64, 2><<<gm2, 128, mix_smem(64), s>>>(m);
        const int rc = a.vdim <= 32 ? launch_values<4>(m, grid, s) : a.vdim <= 64 ? launch_values<8>(m, grid, s)
                       : a.vdim <= 128 ? launch_values<16>(m, grid, s) : launch_values<32>(m, grid, s);
        if (rc != 0) return rc;
        count_launch(3);
    }
    return (int)cudaGetLastError();
}

int mixed_attention(const PA& a, int dtype, int longest_entry, int longest_context, void* workspace, size_t workspace_bytes, cudaStream_t s) {
    if (dtype != B200_BF16 && dtype != B200_F32) return B200_EINVAL;
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    int span = a.chunk;   // most keys a position sees, 0: no bound
    if (a.window > 0) span = span > 0 ? std::min(span, a.window) : a.window;
    if (dtype == B200_BF16 && longest_entry != 1 && longest_context > 0 && workspace && a.heads <= 64 && a.dim % 8 == 0 && a.vdim % 8 == 0 &&
        a.dim <= 256 && a.vdim <= 256 && al16(a.q) && al16(a.out) && al16(a.k_pool) && al16(a.v_pool) && al16(workspace)) {
        const int rc = mixed_tiles(a, span, longest_context, workspace, workspace_bytes, s);
        if (rc != B200_EUNSUPPORTED) return rc;
    }
    // The context is shared by a cluster when the tokens alone do not fill the GPU. Sizes follow the context rounded up, so that a
    // launch captured into a graph fits the contexts of its replays (a longer share is walked in several tiles).
    int seen = longest_context <= 256 ? 256 : (longest_context + 127) / 128 * 128;
    if (span > 0) seen = std::min(seen, span);
    int cluster = 1;
    while (cluster < kMxMaxCluster && (long long)a.n_tokens * cluster * 2 <= 2 * sm_count() && seen / (2 * cluster) >= 32) cluster *= 2;
    const size_t fixed = mx_row_floats(a.heads, a.dim, a.vdim) * sizeof(float);
    const size_t per_key = (size_t)2 * a.heads * sizeof(float) + sizeof(int);
    if (fixed + 8 * per_key > kMxSmem) return B200_EUNSUPPORTED;
    const int share = ((seen + cluster - 1) / cluster + 3) & ~3;
    const int kt = (int)std::min<size_t>(std::min(share, 512), (kMxSmem - fixed) / per_key) & ~3;
    MxRow m{a, kt, a.dim % 8 == 0 && al16(a.k_pool), al16(a.v_pool)};
    const size_t smem = fixed + (size_t)kt * per_key;
    return dtype == B200_BF16 ? launch_mx_row_for<__nv_bfloat16>(m, cluster, smem, s) : launch_mx_row_for<float>(m, cluster, smem, s);
}

}  // namespace b200

using namespace b200;

extern "C" size_t b200_mixed_attention_workspace_bytes(int n_tokens, int heads, int window, int longest_seen) {
    if (n_tokens < 2 || heads < 1 || window < 0 || longest_seen < 1) return 0;
    const size_t rb = mx_row_bytes(heads, mx_width(window, longest_seen));
    const size_t need = (size_t)mx_block_rows(n_tokens, rb) * rb;
    return need <= kMxMostBytes ? need : 0;
}
