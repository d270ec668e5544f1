// What surrounds the sublayers of a parallel layer: the residual update that joins both sublayers (each mixer output
// optionally RMS-normed with its own weight first, the feed-forward's row or the weighted rows of its routed experts) with
// one multiplier, fused with the layer norm that reads the residual next; and the activation of a dense feed-forward that
// is a polynomial of RMS-normed powers. One CTA per row, everything fp32 up to the store of the next operand.
#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"

namespace b200 {

constexpr int kPrMaxTop = 16;

// sums of two values over a CTA, the same order in every thread
template <int THREADS>
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        a += __shfl_xor_sync(0xffffffffu, a, o);
        b += __shfl_xor_sync(0xffffffffu, b, o);
    }
    __syncthreads();   // red may still be read from the previous call
    if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = make_float2(a, b);
    __syncthreads();
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int k = 0; k < THREADS / 32; ++k) { s.x += red[k].x; s.y += red[k].y; }
    return s;
}

// rows of at most THREADS * PER values: every operand of the row is loaded up front and lives in registers
template <typename T, int THREADS, int PER>
__global__ void __launch_bounds__(THREADS) parallel_residual_reg_kernel(const b200_parallel_residual_args a) {
    __shared__ float2 red[THREADS / 32];
    __shared__ int e_dest[kPrMaxTop];
    __shared__ float e_w[kPrMaxTop];
    const int i = blockIdx.x, width = a.width;
    const size_t base = (size_t)i * width;
    if (a.expert_out) {
        if (threadIdx.x < a.top) {
            e_dest[threadIdx.x] = a.dest[(size_t)i * a.top + threadIdx.x];
            e_w[threadIdx.x] = a.weight[(size_t)i * a.top + threadIdx.x];
        }
        __syncthreads();
    }
    float v[PER], p1[PER], p2[PER], p3[PER], w1[PER], w2[PER], lw[PER], lb[PER];
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x + THREADS * k;
        const bool in = c < width;
        v[k] = in ? a.x[base + c] : 0.f;
        p1[k] = (in && a.y1) ? a.y1[base + c] : 0.f;
        p2[k] = (in && a.y2) ? a.y2[base + c] : 0.f;
        p3[k] = (in && a.y3) ? a.y3[base + c] : 0.f;
        w1[k] = (in && a.w1) ? a.w1[c] : 1.f;
        w2[k] = (in && a.w2) ? a.w2[c] : 1.f;
        lw[k] = (in && a.ln_w) ? a.ln_w[c] : 0.f;
        lb[k] = (in && a.ln_b) ? a.ln_b[c] : 0.f;
    }
    if (a.expert_out) {
#pragma unroll 2
        for (int j = 0; j < a.top; ++j) {   // an expert's row at a time: its loads are in flight together
            const int d = e_dest[j];
            if (d < 0) continue;
            const float* er = a.expert_out + (size_t)d * width;
            float e[PER];
#pragma unroll
            for (int k = 0; k < PER; ++k) e[k] = threadIdx.x + THREADS * k < width ? er[threadIdx.x + THREADS * k] : 0.f;
#pragma unroll
            for (int k = 0; k < PER; ++k) p3[k] = fmaf(e_w[j], e[k], p3[k]);
        }
    }
    float r1 = 1.f, r2 = 1.f;
    if (a.w1 || a.w2) {
        float s1 = 0.f, s2 = 0.f;
#pragma unroll
        for (int k = 0; k < PER; ++k) { s1 += p1[k] * p1[k]; s2 += p2[k] * p2[k]; }
        const float2 s = block_sum2<THREADS>(s1, s2, red);
        r1 = a.w1 ? 1.0f / sqrtf(s.x / (float)width + a.eps) : 1.f;
        r2 = a.w2 ? 1.0f / sqrtf(s.y / (float)width + a.eps) : 1.f;
    }
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x + THREADS * k;
        if (c < width) {
            float y = 0.f;
            if (a.y1) y += a.s1 * (p1[k] * r1 * w1[k]);   // no norm: both factors are 1
            if (a.y2) y += a.s2 * (p2[k] * r2 * w2[k]);
            y += p3[k];
            v[k] += a.mult * y;
            a.x[base + c] = v[k];
            sum += v[k];
        }
    }
    if (!a.ln_w) return;
    const float mean = block_sum2<THREADS>(sum, 0.f, red).x / (float)width;
    float q = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const float d = threadIdx.x + THREADS * k < width ? v[k] - mean : 0.f;
        q += d * d;
    }
    const float rstd = 1.0f / sqrtf(block_sum2<THREADS>(q, 0.f, red).x / (float)width + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + base;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x + THREADS * k;
        if (c < width) out[c] = DT<T>::from_f((v[k] - mean) * rstd * lw[k] + lb[k]);
    }
}

// longer rows: the new residual row stays in shared memory, the addends are read again
template <typename T>
__global__ void __launch_bounds__(256) parallel_residual_kernel(const b200_parallel_residual_args a) {
    extern __shared__ float pr_row[];
    __shared__ float2 red[8];
    const int i = blockIdx.x, width = a.width;
    const size_t base = (size_t)i * width;
    float r1 = 1.f, r2 = 1.f;
    if (a.w1 || a.w2) {
        float s1 = 0.f, s2 = 0.f;
        for (int c = threadIdx.x; c < width; c += 256) {
            const float u = a.y1 ? a.y1[base + c] : 0.f, w = a.y2 ? a.y2[base + c] : 0.f;
            s1 += u * u;
            s2 += w * w;
        }
        const float2 s = block_sum2<256>(s1, s2, red);
        r1 = a.w1 ? 1.0f / sqrtf(s.x / (float)width + a.eps) : 1.f;
        r2 = a.w2 ? 1.0f / sqrtf(s.y / (float)width + a.eps) : 1.f;
    }
    float sum = 0.f;
    for (int c = threadIdx.x; c < width; c += 256) {
        float y = 0.f, r = a.y3 ? a.y3[base + c] : 0.f;
        if (a.expert_out)
            for (int j = 0; j < a.top; ++j) {
                const int d = a.dest[(size_t)i * a.top + j];
                if (d >= 0) r = fmaf(a.weight[(size_t)i * a.top + j], a.expert_out[(size_t)d * width + c], r);
            }
        if (a.y1) y += a.s1 * (a.w1 ? a.y1[base + c] * r1 * a.w1[c] : a.y1[base + c]);
        if (a.y2) y += a.s2 * (a.w2 ? a.y2[base + c] * r2 * a.w2[c] : a.y2[base + c]);
        y += r;
        const float v = a.x[base + c] + a.mult * y;
        a.x[base + c] = v;
        pr_row[c] = v;
        sum += v;
    }
    if (!a.ln_w) return;
    const float mean = block_sum2<256>(sum, 0.f, red).x / (float)width;
    float q = 0.f;
    for (int c = threadIdx.x; c < width; c += 256) {
        const float d = pr_row[c] - mean;
        q += d * d;
    }
    const float rstd = 1.0f / sqrtf(block_sum2<256>(q, 0.f, red).x / (float)width + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + base;
    for (int c = threadIdx.x; c < width; c += 256) out[c] = DT<T>::from_f((pr_row[c] - mean) * rstd * a.ln_w[c] + (a.ln_b ? a.ln_b[c] : 0.f));
}

template <typename T>
static void launch_pr(const b200_parallel_residual_args& a, size_t smem, cudaStream_t s) {
    if (a.width <= 512) parallel_residual_reg_kernel<T, 128, 4><<<a.n_rows, 128, 0, s>>>(a);
    else if (a.width <= 2048) parallel_residual_reg_kernel<T, 512, 4><<<a.n_rows, 512, 0, s>>>(a);
    else if (a.width <= 4096) parallel_residual_reg_kernel<T, 1024, 4><<<a.n_rows, 1024, 0, s>>>(a);
    else {
        static unsigned long long done = 0;
        if (smem > 48 * 1024) ensure_max_dynamic_smem((const void*)parallel_residual_kernel<T>, 200 * 1024, done);
        parallel_residual_kernel<T><<<a.n_rows, 256, smem, s>>>(a);
    }
}

// c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3; the row is read twice (the second time from cache)
template <typename T>
__global__ void __launch_bounds__(256) poly_norm_kernel(const float* __restrict__ z, const float* __restrict__ c4, float eps, T* __restrict__ out,
                                                        int width) {
    __shared__ float2 red[8];
    const size_t base = (size_t)blockIdx.x * width;
    const float* row = z + base;
    const bool vec = width % 4 == 0 && (reinterpret_cast<uintptr_t>(z) & 15u) == 0;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    auto add = [&](float v) {
        const float q = v * v, q2 = q * q;
        s2 += q;
        s4 += q2;
        s6 += q2 * q;
    };
    if (vec) {
        for (int c = 4 * threadIdx.x; c < width; c += 1024) {
            const float4 v = *reinterpret_cast<const float4*>(row + c);
            add(v.x); add(v.y); add(v.z); add(v.w);
        }
    } else
        for (int c = threadIdx.x; c < width; c += 256) add(row[c]);
    const float2 s = block_sum2<256>(s2, s4, red);
    const float n = (float)width;
    const float f1 = c4[0] / sqrtf(s.x / n + eps), f2 = c4[1] / sqrtf(s.y / n + eps), f0 = c4[3];
    const float f3 = c4[2] / sqrtf(block_sum2<256>(s6, 0.f, red).x / n + eps);
    auto act = [&](float v) { return f1 * v + f2 * (v * v) + f3 * (v * v * v) + f0; };
    T* dst = out + base;
    if (vec) {
        for (int c = 4 * threadIdx.x; c < width; c += 1024) {
            const float4 v = *reinterpret_cast<const float4*>(row + c);
            dst[c] = DT<T>::from_f(act(v.x)); dst[c + 1] = DT<T>::from_f(act(v.y));
            dst[c + 2] = DT<T>::from_f(act(v.z)); dst[c + 3] = DT<T>::from_f(act(v.w));
        }
    } else
        for (int c = threadIdx.x; c < width; c += 256) dst[c] = DT<T>::from_f(act(row[c]));
}

}  // namespace b200

using namespace b200;

extern "C" int b200_parallel_residual(const b200_parallel_residual_args* a, void* stream) {
    if (!a || !a->x || a->n_rows < 0 || a->width < 1 || (a->ln_w && !a->out) || (a->w1 && !a->y1) || (a->w2 && !a->y2)) return B200_EINVAL;
    if (a->expert_out && (!a->dest || !a->weight || a->top < 1)) return B200_EINVAL;
    if (a->expert_out && a->top > kPrMaxTop) return B200_EUNSUPPORTED;
    if (a->n_rows == 0) return B200_OK;
    const size_t smem = (size_t)a->width * sizeof(float);
    if (smem > 200 * 1024) return B200_EUNSUPPORTED;
    if (a->out_dtype == B200_BF16 || !a->ln_w) launch_pr<__nv_bfloat16>(*a, smem, (cudaStream_t)stream);
    else if (a->out_dtype == B200_F32) launch_pr<float>(*a, smem, (cudaStream_t)stream);
    else return B200_EINVAL;
    count_launch();
    return (int)cudaGetLastError();
}

extern "C" int b200_poly_norm(const float* z, const float* c4, float eps, void* out, int n_rows, int width, int out_dtype, void* stream) {
    if (!z || !c4 || !out || n_rows < 0 || width < 1) return B200_EINVAL;
    if (n_rows == 0) return B200_OK;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == B200_BF16) poly_norm_kernel<__nv_bfloat16><<<n_rows, 256, 0, s>>>(z, c4, eps, (__nv_bfloat16*)out, width);
    else if (out_dtype == B200_F32) poly_norm_kernel<float><<<n_rows, 256, 0, s>>>(z, c4, eps, (float*)out, width);
    else return B200_EINVAL;
    count_launch();
    return (int)cudaGetLastError();
}
