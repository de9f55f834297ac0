// The residual stream between two sublayers in one pass over each row: the previous sublayer's output (summed over
// its parts) is normalised and added, the new stream normalised for the next sublayer.  The stream and everything
// computed here is fp32; one CTA per row, the row in registers, 8 elements per access.
#include "../ktk_vec.cuh"
#include "ktk_layers.h"

namespace ktk {

constexpr int kRnThreads = 256;
constexpr int kRnMaxVec = 8;      // 8 x 8 elements per thread: rows of up to 16384 columns

struct ResidualNormParams {
    const int64_t* tokens;
    const void* embed;
    int64_t vocab;
    float embed_scale;
    float* x;
    const void* y;
    int parts;
    const float *post_w, *post_b;
    float mult;
    const float *pre_w, *pre_b;
    void* h;
    float eps;
    int center, cols, stride;
    int32_t* zero;
    int zero_n;
    int32_t* status;
};

__device__ __forceinline__ float row_sum(float v, float* part) {
    v = warp_sum_f(v);
    const int warps = blockDim.x >> 5;
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
    for (int i = 0; i < warps; ++i) t += part[i];
    __syncthreads();
    return t;
}

// v <- norm(v; w, b), in registers; elements past `cols` are zero before and after (their w and b are)
template <int NV>
__device__ __forceinline__ void norm_regs(float (&v)[NV][8], const float* w, const float* b, float eps, bool center,
                                          int cols, int nvec, float* part) {
    float c = 0.0f;
    if (center) {
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) s += v[i][e];
        c = row_sum(s, part) / (float)cols;
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int k = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
        for (int e = 0; e < 8; ++e)
            if (k + e < cols) { const float d = v[i][e] - c; ss += d * d; }
    }
    const float inv = 1.0f / sqrtf(row_sum(ss, part) / (float)cols + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int k = threadIdx.x + i * blockDim.x;
        if (k < nvec) {
            float wv[8], bv[8] = {0, 0, 0, 0, 0, 0, 0, 0};
            Vec8<float>::load(w + k * 8, wv);
            if (b != nullptr) Vec8<float>::load(b + k * 8, bv);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[i][e] = k * 8 + e < cols ? (v[i][e] - c) * inv * wv[e] + bv[e] : 0.0f;
        }
    }
}

template <typename T, int NV>
__global__ void __launch_bounds__(kRnThreads) residual_norm_kernel(const ResidualNormParams p) {
    __shared__ float part[kRnThreads / 32];
    const int64_t r = blockIdx.x;
    const int nvec = p.stride / 8;
    if (p.zero != nullptr && blockIdx.x == 0)
        for (int i = threadIdx.x; i < p.zero_n; i += blockDim.x) p.zero[i] = 0;
    float x[NV][8];
    float* xrow = p.x + r * p.stride;
    int64_t tok = 0;
    if (p.tokens != nullptr) {
        tok = p.tokens[r];
        if (tok < 0 || tok >= p.vocab) {
            if (threadIdx.x == 0) report(p.status, KTK_STATUS_BAD_TABLE);
            tok = 0;
        }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int k = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int e = 0; e < 8; ++e) x[i][e] = 0.0f;
        if (k < nvec) {
            if (p.tokens != nullptr) {
                Vec8<T>::load((const T*)p.embed + tok * p.stride + k * 8, x[i]);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[i][e] *= p.embed_scale;
            } else Vec8<float>::load(xrow + k * 8, x[i]);
        }
    }
    if (p.y != nullptr) {
        float y[NV][8];
        const T* yrow = (const T*)p.y + r * p.parts * p.stride;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int k = threadIdx.x + i * blockDim.x;
#pragma unroll
            for (int e = 0; e < 8; ++e) y[i][e] = 0.0f;
            if (k < nvec)
                for (int j = 0; j < p.parts; ++j) {
                    float t[8];
                    Vec8<T>::load(yrow + (int64_t)j * p.stride + k * 8, t);
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[i][e] += t[e];
                }
        }
        if (p.post_w != nullptr) norm_regs<NV>(y, p.post_w, p.post_b, p.eps, p.center != 0, p.cols, nvec, part);
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) x[i][e] += p.mult * y[i][e];
    }
    if (p.y != nullptr || p.tokens != nullptr) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int k = threadIdx.x + i * blockDim.x;
            if (k < nvec) Vec8<float>::store(xrow + k * 8, x[i]);
        }
    }
    if (p.h != nullptr) {
        if (p.pre_w != nullptr) norm_regs<NV>(x, p.pre_w, p.pre_b, p.eps, p.center != 0, p.cols, nvec, part);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int k = threadIdx.x + i * blockDim.x;
            if (k < nvec) Vec8<T>::store((T*)p.h + r * p.stride + k * 8, x[i]);
        }
    }
}

template <typename T>
static int residual_norm_launch(const ResidualNormParams& p, int64_t rows, cudaStream_t st) {
    const int nvec = p.stride / 8;
    const int threads = nvec >= kRnThreads ? kRnThreads : (nvec + 31) / 32 * 32;
    const int nv = (nvec + threads - 1) / threads;
    const unsigned grid = (unsigned)rows;
    if (nv <= 1) residual_norm_kernel<T, 1><<<grid, threads, 0, st>>>(p);
    else if (nv <= 2) residual_norm_kernel<T, 2><<<grid, threads, 0, st>>>(p);
    else if (nv <= 4) residual_norm_kernel<T, 4><<<grid, threads, 0, st>>>(p);
    else residual_norm_kernel<T, kRnMaxVec><<<grid, threads, 0, st>>>(p);
    KTK_CUDA_TRY(cudaGetLastError(), "ktk_residual_norm");
    return KTK_OK;
}

}  // namespace ktk

using namespace ktk;

extern "C" int ktk_residual_norm(const int64_t* tokens, const void* embed, int64_t vocab, float embed_scale, float* x,
                                 const void* y, int32_t parts, const float* post_w, const float* post_b, float mult,
                                 const float* pre_w, const float* pre_b, void* h, float eps, int32_t center,
                                 int64_t rows, int32_t cols, int32_t stride, int32_t* zero, int32_t zero_n,
                                 int32_t dtype, int32_t* status, void* stream) {
    const char* who = "ktk_residual_norm";
    if (rows < 0 || rows > 2147483647LL || cols <= 0 || stride < cols || stride % 8 != 0 || parts < 1 || zero_n < 0 ||
        (dtype != KTK_F32 && dtype != KTK_BF16)) {
        set_error("%s: rows=%lld cols=%d stride=%d parts=%d zero_n=%d dtype=%d", who, (long long)rows, cols, stride,
                  parts, zero_n, dtype);
        return KTK_ERR_ARG;
    }
    if (stride > 8 * kRnThreads * kRnMaxVec) {
        set_error("%s: rows of at most %d columns are built (got %d)", who, 8 * kRnThreads * kRnMaxVec, stride);
        return KTK_ERR_UNSUPPORTED;
    }
    if (rows == 0) return KTK_OK;
    if (!x || (tokens && (!embed || vocab <= 0)) || (!h && !y && !tokens)) {
        set_error("%s: null pointer argument", who);
        return KTK_ERR_ARG;
    }
    const uintptr_t al = (uintptr_t)embed | (uintptr_t)x | (uintptr_t)y | (uintptr_t)post_w | (uintptr_t)post_b |
                         (uintptr_t)pre_w | (uintptr_t)pre_b | (uintptr_t)h;
    if ((al & 15u) != 0) { set_error("%s: pointers must be 16-byte aligned", who); return KTK_ERR_ARG; }
    const ResidualNormParams p{tokens, embed, vocab, embed_scale, x, y, parts, post_w, post_b, mult, pre_w, pre_b, h, eps,
                               center, cols, stride, zero, zero ? zero_n : 0, status};
    return dtype == KTK_F32 ? residual_norm_launch<float>(p, rows, (cudaStream_t)stream)
                            : residual_norm_launch<__nv_bfloat16>(p, rows, (cudaStream_t)stream);
}
