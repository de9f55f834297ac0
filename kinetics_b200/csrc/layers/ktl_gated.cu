// Element-wise steps of free size: the gated activation of a dense feed-forward, and the scaled, soft-capped logits.
#include "ktl_common.cuh"

namespace ktk {

constexpr int kGtThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kGtThreads)
gated_rows_kernel(const T* __restrict__ in, T* __restrict__ out, int64_t rows, int nvec, float limit, float slope, float shift) {
    const int64_t n = rows * nvec;
    for (int64_t i = (int64_t)blockIdx.x * kGtThreads + threadIdx.x; i < n; i += (int64_t)gridDim.x * kGtThreads) {
        const int64_t r = i / nvec;
        const int c = (int)(i - r * nvec);
        float g[8], u[8];
        load8(in + (2 * r * nvec + c) * 8, g);
        load8(in + ((2 * r + 1) * nvec + c) * 8, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) g[e] = gated<sizeof(T) == 2>(g[e], u[e], limit, slope, shift);
        Vec8<T>::store(out + i * 8, g);
    }
}

__global__ void __launch_bounds__(kGtThreads) scale_cap_kernel(float* z, int64_t n, float scale, float cap) {
    for (int64_t i = (int64_t)blockIdx.x * kGtThreads + threadIdx.x; i < n; i += (int64_t)gridDim.x * kGtThreads) {
        const float v = z[i] * scale;
        z[i] = cap > 0.0f ? cap * tanhf(v / cap) : v;
    }
}

static unsigned rows_grid(int64_t work) {
    const int64_t blocks = (work + kGtThreads - 1) / kGtThreads, cap = (int64_t)sm_count() * 16;
    return (unsigned)(blocks < cap ? blocks : cap);
}

}  // namespace ktk

using namespace ktk;

extern "C" int ktk_gated_rows(const void* in, void* out, int64_t rows, int32_t cols_stride, float limit, float slope,
                              float shift, int32_t dtype, void* stream) {
    const char* who = "ktk_gated_rows";
    if (rows < 0 || cols_stride <= 0 || cols_stride % 8 != 0 || !(limit > 0.0f) || (dtype != KTK_F32 && dtype != KTK_BF16)) {
        set_error("%s: rows=%lld cols_stride=%d limit=%g dtype=%d", who, (long long)rows, cols_stride, (double)limit, dtype);
        return KTK_ERR_ARG;
    }
    if (rows == 0) return KTK_OK;
    if (!in || !out || (((uintptr_t)in | (uintptr_t)out) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    const int nvec = cols_stride / 8;
    const unsigned grid = rows_grid(rows * nvec);
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == KTK_F32)
        gated_rows_kernel<float><<<grid, kGtThreads, 0, st>>>((const float*)in, (float*)out, rows, nvec, limit, slope, shift);
    else
        gated_rows_kernel<__nv_bfloat16><<<grid, kGtThreads, 0, st>>>((const __nv_bfloat16*)in, (__nv_bfloat16*)out, rows, nvec,
                                                                     limit, slope, shift);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}

extern "C" int ktk_scale_cap(float* z, int64_t n, float scale, float cap, void* stream) {
    const char* who = "ktk_scale_cap";
    if (n < 0 || (n > 0 && !z)) { set_error("%s: n=%lld", who, (long long)n); return KTK_ERR_ARG; }
    if (n == 0) return KTK_OK;
    scale_cap_kernel<<<rows_grid(n), kGtThreads, 0, (cudaStream_t)stream>>>(z, n, scale, cap);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}
