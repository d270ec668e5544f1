// Residual streams with learned connections: instead of one residual row per token there are S rows, every sublayer reads one
// weighted sum of them and writes back into all of them through an S x S mixing matrix.
//
//   b200_embed_streams    token row * scale + fixed sinusoids of the position, copied into every stream
//   b200_hyper_residual   the boundary between two sublayers in one launch: the finished sublayer's output (a plain row, a row
//                         with a sigmoid gate per token, the rows of routed experts) goes into all streams at once, the next
//                         sublayer's weighted sum is formed from the new streams while they are in registers, RMS-normed and
//                         stored as the operand of its projections. With a row list it only reads and norms (the final norm);
//                         without weights it sums the streams.
// Everything fp32 up to the store of the normed row. One CTA per token: S rows are read once and written once.
#include "b200_serve.h"
#include "common.cuh"
#include "launch_count.h"

namespace b200 {

// Angles: turns[i] = 10000^(-2i/width) / pi (double). position * turns[i] is brought into [-1, 1] in double, then sincospif:
// a position of 10^6 is as exact as position 1.
template <typename T>
__global__ void __launch_bounds__(128) embed_streams_kernel(const int* __restrict__ ids, const int* __restrict__ pos, const T* __restrict__ table,
                                                            float scale, const double* __restrict__ turns, float* __restrict__ out,
                                                            int streams, int width) {
    const int t = blockIdx.x;
    const T* row = table + (size_t)ids[t] * width;
    const double p = turns ? (double)pos[t] : 0.0;
    float* dst = out + (size_t)t * streams * width;
    for (int i = threadIdx.x; 2 * i < width; i += blockDim.x) {
        float s = 0.f, c = 0.f;
        if (turns) {
            const double a = p * turns[i];
            sincospif((float)(a - 2.0 * rint(0.5 * a)), &s, &c);
        }
        const float v0 = fmaf(DT<T>::to_f(row[2 * i]), scale, s);
        const bool two = 2 * i + 1 < width;
        const float v1 = two ? fmaf(DT<T>::to_f(row[2 * i + 1]), scale, c) : 0.f;
        for (int k = 0; k < streams; ++k) {
            dst[(size_t)k * width + 2 * i] = v0;
            if (two) dst[(size_t)k * width + 2 * i + 1] = v1;
        }
    }
}

struct HyArgs {
    float* x; int streams;
    const float* mix; const float* w_out;
    const float* y1; const float* y2; const float* gate2;
    const float* eo; const int* dest; const float* weight; int top;
    const float* w_in; const int* rows;
    const float* w; float eps;
    void* out; float* sum_out;
    int width;
};

constexpr int kHyMaxTop = 16, kHyMaxStreams = 16;

__device__ __forceinline__ float4 hy_fma(float s, float4 a, float4 b) {
    return make_float4(fmaf(s, a.x, b.x), fmaf(s, a.y, b.y), fmaf(s, a.z, b.z), fmaf(s, a.w, b.w));
}

// the token's S x S matrix, output and input vectors, expert rows and the gate, once per CTA
template <int MAXS>
struct HyShared {
    float mix[MAXS * MAXS], w_out[MAXS], w_in[MAXS], gate;
    int e_dest[kHyMaxTop];
    float e_w[kHyMaxTop];
};
template <int MAXS>
__device__ __forceinline__ void hy_load_shared(HyShared<MAXS>& sh, const HyArgs& a, int i) {
    const int S = a.streams, tid = threadIdx.x;
    if (a.mix) {
        for (int k = tid; k < S * S; k += blockDim.x) sh.mix[k] = a.mix[k];
        if (tid < S) sh.w_out[tid] = a.w_out[tid];
        if (a.eo && tid < a.top) {
            sh.e_dest[tid] = a.dest[(size_t)i * a.top + tid];
            sh.e_w[tid] = a.weight ? a.weight[(size_t)i * a.top + tid] : 1.f;
        }
        if (tid == 0) sh.gate = (a.y2 && a.gate2) ? a.gate2[i] : 1.f;
    }
    if (tid < S) sh.w_in[tid] = a.w_in ? a.w_in[tid] : 1.f;
    __syncthreads();
}

// Rows in whole groups of four columns, at most PER groups per thread: the S streams, the sublayer's output and the norm weight
// are loaded up front (all loads in flight together) and live in registers.
template <typename T, int S, int THREADS, int PER>
__global__ void __launch_bounds__(THREADS) hyper_residual_reg_kernel(const HyArgs a) {
    __shared__ HyShared<S> sh;
    __shared__ float red[THREADS / 32];
    const int i = blockIdx.x, width = a.width, quads = width / 4;
    const size_t row = a.rows ? a.rows[i] : i;
    float4* x = reinterpret_cast<float4*>(a.x) + row * S * quads;
    float4 v[S][PER], y[PER], w4[PER];
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x + THREADS * k;
        const bool in = c < quads;
#pragma unroll
        for (int s = 0; s < S; ++s) v[s][k] = in ? x[s * quads + c] : zero;
        y[k] = (in && a.mix && a.y1) ? reinterpret_cast<const float4*>(a.y1)[row * quads + c] : zero;
        w4[k] = (in && a.w) ? reinterpret_cast<const float4*>(a.w)[c] : zero;
    }
    hy_load_shared<S>(sh, a, i);
    if (a.mix) {
        if (a.y2) {
#pragma unroll
            for (int k = 0; k < PER; ++k) {
                const int c = threadIdx.x + THREADS * k;
                if (c < quads) y[k] = hy_fma(sh.gate, reinterpret_cast<const float4*>(a.y2)[row * quads + c], y[k]);
            }
        }
        if (a.eo) {
            float4 r[PER];
#pragma unroll
            for (int k = 0; k < PER; ++k) r[k] = zero;
            for (int j = 0; j < a.top; ++j) {
                if (sh.e_dest[j] < 0) continue;
                const float4* er = reinterpret_cast<const float4*>(a.eo) + (size_t)sh.e_dest[j] * quads;
                const float ew = sh.e_w[j];
#pragma unroll
                for (int k = 0; k < PER; ++k) {
                    const int c = threadIdx.x + THREADS * k;
                    if (c < quads) r[k] = hy_fma(ew, er[c], r[k]);
                }
            }
#pragma unroll
            for (int k = 0; k < PER; ++k) y[k] = hy_fma(1.f, r[k], y[k]);
        }
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int c = threadIdx.x + THREADS * k;
            float4 n[S];
#pragma unroll
            for (int t = 0; t < S; ++t) {
                n[t] = zero;
#pragma unroll
                for (int s = 0; s < S; ++s) n[t] = hy_fma(sh.mix[s * S + t], v[s][k], n[t]);
                n[t] = hy_fma(sh.w_out[t], y[k], n[t]);
            }
#pragma unroll
            for (int t = 0; t < S; ++t) {
                v[t][k] = n[t];
                if (c < quads) x[t * quads + c] = n[t];
            }
        }
    }
    if (!a.w && !a.sum_out) return;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        float4 u = zero;
#pragma unroll
        for (int s = 0; s < S; ++s) u = hy_fma(sh.w_in[s], v[s][k], u);
        y[k] = u;
        ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
        const int c = threadIdx.x + THREADS * k;
        if (a.sum_out && c < quads) reinterpret_cast<float4*>(a.sum_out)[(size_t)i * quads + c] = u;
    }
    if (!a.w) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int k = 0; k < THREADS / 32; ++k) tot += red[k];
    const float rinv = 1.0f / sqrtf(tot / (float)width + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)i * width;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x + THREADS * k;
        if (c >= quads) continue;
        const float4 f = make_float4(y[k].x * rinv * w4[k].x, y[k].y * rinv * w4[k].y, y[k].z * rinv * w4[k].z, y[k].w * rinv * w4[k].w);
        if constexpr (sizeof(T) == 4) reinterpret_cast<float4*>(out)[c] = f;
        else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(f.x, f.y), hi = __floats2bfloat162_rn(f.z, f.w);
            reinterpret_cast<uint2*>(out)[c] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

// any width and up to kHyMaxStreams streams: a column at a time, the weighted sum kept in shared memory between the sum of squares
// and the output
template <typename T>
__global__ void __launch_bounds__(256) hyper_residual_kernel(const HyArgs a) {
    extern __shared__ float hy_row[];
    __shared__ HyShared<kHyMaxStreams> sh;
    __shared__ float red[8];
    const int i = blockIdx.x, width = a.width, S = a.streams;
    const size_t row = a.rows ? a.rows[i] : i;
    float* x = a.x + row * S * width;
    hy_load_shared<kHyMaxStreams>(sh, a, i);
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += 256) {
        float v[kHyMaxStreams];
        for (int s = 0; s < S; ++s) v[s] = x[(size_t)s * width + c];
        if (a.mix) {
            float y = a.y1 ? a.y1[row * width + c] : 0.f;
            if (a.y2) y = fmaf(sh.gate, a.y2[row * width + c], y);
            if (a.eo) {
                float r = 0.f;
                for (int j = 0; j < a.top; ++j)
                    if (sh.e_dest[j] >= 0) r = fmaf(sh.e_w[j], a.eo[(size_t)sh.e_dest[j] * width + c], r);
                y += r;
            }
            float n[kHyMaxStreams];
            for (int t = 0; t < S; ++t) {
                n[t] = 0.f;
                for (int s = 0; s < S; ++s) n[t] = fmaf(sh.mix[s * S + t], v[s], n[t]);
                n[t] = fmaf(sh.w_out[t], y, n[t]);
            }
            for (int t = 0; t < S; ++t) {
                v[t] = n[t];
                x[(size_t)t * width + c] = n[t];
            }
        }
        if (!a.w && !a.sum_out) continue;
        float u = 0.f;
        for (int s = 0; s < S; ++s) u = fmaf(sh.w_in[s], v[s], u);
        if (a.sum_out) a.sum_out[(size_t)i * width + c] = u;
        if (a.w) hy_row[c] = u;
        ss += u * u;
    }
    if (!a.w) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int k = 0; k < 8; ++k) tot += red[k];
    const float rinv = 1.0f / sqrtf(tot / (float)width + a.eps);
    T* out = reinterpret_cast<T*>(a.out) + (size_t)i * width;
    for (int c = threadIdx.x; c < width; c += 256) out[c] = DT<T>::from_f(hy_row[c] * rinv * a.w[c]);
}

template <typename T, int S>
static bool launch_hyper_reg(const HyArgs& a, int n_rows, cudaStream_t s) {
    const int quads = a.width / 4;
    if (quads <= 128) hyper_residual_reg_kernel<T, S, 128, 1><<<n_rows, 128, 0, s>>>(a);
    else if (quads <= 256) hyper_residual_reg_kernel<T, S, 256, 1><<<n_rows, 256, 0, s>>>(a);
    else if (quads <= 512) hyper_residual_reg_kernel<T, S, 256, 2><<<n_rows, 256, 0, s>>>(a);
    else if (quads <= 1024) hyper_residual_reg_kernel<T, S, 512, 2><<<n_rows, 512, 0, s>>>(a);
    else if (quads <= 2048 && S <= 2) hyper_residual_reg_kernel<T, S, 1024, 2><<<n_rows, 1024, 0, s>>>(a);
    else return false;
    return true;
}

template <typename T>
static int launch_hyper(const HyArgs& a, int n_rows, bool vec, cudaStream_t s) {
    bool done = false;
    if (vec) {
        switch (a.streams) {
            case 1: done = launch_hyper_reg<T, 1>(a, n_rows, s); break;
            case 2: done = launch_hyper_reg<T, 2>(a, n_rows, s); break;
            case 3: done = launch_hyper_reg<T, 3>(a, n_rows, s); break;
            case 4: done = launch_hyper_reg<T, 4>(a, n_rows, s); break;
        }
    }
    if (!done) {
        const size_t smem = a.w ? (size_t)a.width * sizeof(float) : 0;
        if (smem > 200 * 1024) return B200_EUNSUPPORTED;
        static unsigned long long set = 0;
        if (smem > 40 * 1024) {
            const cudaError_t e = ensure_max_dynamic_smem((const void*)hyper_residual_kernel<T>, 200 * 1024, set);
            if (e != cudaSuccess) return (int)e;
        }
        hyper_residual_kernel<T><<<n_rows, 256, smem, s>>>(a);
    }
    count_launch();
    return (int)cudaGetLastError();
}

}  // namespace b200

using namespace b200;

extern "C" int b200_embed_streams(const int* ids, const int* pos, const void* table, float scale, const double* turns, float* out, int streams,
                                  int n_tokens, int width, int dtype, void* stream) {
    if (!ids || !table || !out || (turns && !pos) || streams < 1 || n_tokens < 0 || width < 1) return B200_EINVAL;
    if (n_tokens == 0) return B200_OK;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == B200_BF16)
        embed_streams_kernel<__nv_bfloat16><<<n_tokens, 128, 0, s>>>(ids, pos, (const __nv_bfloat16*)table, scale, turns, out, streams, width);
    else if (dtype == B200_F32)
        embed_streams_kernel<float><<<n_tokens, 128, 0, s>>>(ids, pos, (const float*)table, scale, turns, out, streams, width);
    else
        return B200_EINVAL;
    count_launch();
    return (int)cudaGetLastError();
}

extern "C" int b200_hyper_residual(const b200_hyper_residual_args* p, void* stream) {
    if (!p || !p->x || p->streams < 1 || p->n_rows < 0 || p->width < 1) return B200_EINVAL;
    if (p->mix && !p->w_out) return B200_EINVAL;
    if (!p->mix && (p->y1 || p->y2 || p->expert_out)) return B200_EINVAL;
    if (p->rows && p->mix) return B200_EINVAL;
    if (p->w && !p->out) return B200_EINVAL;
    if (p->expert_out && (!p->dest || p->top < 1)) return B200_EINVAL;
    if (p->streams > kHyMaxStreams || (p->expert_out && p->top > kHyMaxTop)) return B200_EUNSUPPORTED;
    if (p->n_rows == 0) return B200_OK;
    HyArgs a{p->x, p->streams, p->mix, p->w_out, p->y1, p->y2, p->gate2, p->expert_out, p->dest, p->weight, p->top, p->w_in, p->rows,
             p->w, p->eps, p->out, p->sum_out, p->width};
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    const bool vec = p->width % 4 == 0 && al16(p->x) && al16(p->y1) && al16(p->y2) && al16(p->expert_out) && al16(p->w) && al16(p->out) && al16(p->sum_out);
    cudaStream_t s = (cudaStream_t)stream;
    if (p->out_dtype == B200_BF16 || !p->w) return launch_hyper<__nv_bfloat16>(a, p->n_rows, vec, s);
    if (p->out_dtype == B200_F32) return launch_hyper<float>(a, p->n_rows, vec, s);
    return B200_EINVAL;
}
