// What the paged attention kernels share: their argument block, the masks, and the tensor-core fragment helpers of the
// bfloat16 tile kernels (mma.sync m16n8k16, ldmatrix).
#pragma once
#include <cuda_bf16.h>

#include "b200_serve.h"
#include "common.cuh"

namespace b200 {

struct PA {
    const void* q; void* out; const void* k_pool; const void* v_pool;
    const int* pages; int max_pages, page_rows;
    const int* slot; const int* pos;
    int n_tokens, heads, kv_heads, dim, vdim;
    float scale, softcap, denom_bias;
    int splits; float* part;   // row kernel: shares of a context split over gridDim.z CTAs, [token, head, split, 2 + vdim]
    int chunk, maps, out_f32;
    int window, sigmoid; const float* head_bias;
    const float* head_temp; const float* head_mix;
    const float* sink; const float* dist_bias; int dist_n;
};
// first key that position p sees
__device__ __forceinline__ int pa_first_key(const PA& a, int p) {
    const int f = a.chunk > 0 ? (p / a.chunk) * a.chunk : 0;
    return a.window > 0 ? max(f, p - a.window + 1) : f;
}
// what the scores of head h are multiplied by
__device__ __forceinline__ float pa_scale(const PA& a, int h) { return a.head_temp ? a.scale * a.head_temp[h] : a.scale; }
// what the scaled score of a key `dist` positions back gains in head h
__device__ __forceinline__ float pa_dist_bias(const PA& a, int h, int dist) {
    return a.dist_bias ? a.dist_bias[(size_t)h * a.dist_n + min(dist, a.dist_n - 1)] : 0.f;
}
template <typename T>
__device__ __forceinline__ void pa_store(const PA& a, size_t idx, float v) {
    if (a.out_f32) reinterpret_cast<float*>(a.out)[idx] = v;
    else reinterpret_cast<T*>(a.out)[idx] = DT<T>::from_f(v);
}

template <typename T> struct Pair;
template <> struct Pair<float> {
    static __device__ __forceinline__ float2 load(const float* p) { return *reinterpret_cast<const float2*>(p); }
};
template <> struct Pair<__nv_bfloat16> {
    static __device__ __forceinline__ float2 load(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
};

__device__ __forceinline__ void pa_ldsm_x4(uint32_t (&r)[4], const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void pa_ldsm_x4_trans(uint32_t (&r)[4], const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
// (not volatile: a pure function of its registers, so the compiler may interleave independent accumulators)
__device__ __forceinline__ void pa_mma(float (&d)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ uint32_t pa_pack(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}

// tensor-core tiles with a distance bias and / or a learned sink (biased_attention.cu); -1: no tile for these sizes
int biased_tile(const PA& a, cudaStream_t s);
// b200_paged_attention with weights mixed across heads (mixed_attention.cu); a.head_mix is set
int mixed_attention(const PA& a, int dtype, int longest_entry, int longest_context, void* workspace, size_t workspace_bytes, cudaStream_t s);

}  // namespace b200
