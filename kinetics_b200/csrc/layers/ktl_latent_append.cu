// Latent attention, the step in front of the attention itself: the queries' rotated parts are turned, the latent is
// normalised, the shared rotated key is turned, and both go to the token's page row.  One CTA per row; norm, angles and
// rotation in fp32.
#include "ktl_common.cuh"

namespace ktk {

constexpr int kLaThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kLaThreads)
latent_append_kernel(T* proj, int64_t row_stride, int64_t q_col, int64_t kv_col, const int32_t* __restrict__ new_indptr,
                     const float* __restrict__ norm_w, const double* __restrict__ turns, T* q_out, T* pages,
                     const ktk_paged t, const ktk_latent a, int32_t* status) {
    extern __shared__ float2 la_turn[];                   // cos, sin of every pair
    __shared__ float part[kLaThreads / 32];
    const int64_t r = blockIdx.x;
    const int tid = threadIdx.x;
    const int b = new_indptr ? sequence_of_row(new_indptr, t.batch, r) : (int)r;
    const Span s = span_of(t, b);
    const int pos = new_indptr ? s.total - (new_indptr[b + 1] - (int)r) : s.total - 1;
    if (s.bad || pos < 0 || pos >= s.total) {             // uniform for the CTA
        if (tid == 0) report(status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const int half = a.rot_dim / 2, vecs = a.rot_stride / 8;           // vecs: 8 columns, 4 pairs each
    for (int i = tid; i < 4 * vecs; i += kLaThreads) {
        float sn = 0.0f, cs = 0.0f;                       // behind the rotated columns: zeros
        if (i < half) {
            // the whole turns are taken off before rounding: far positions keep their angle
            const double whole = (double)pos * turns[i];
            sincospif((float)(2.0 * (whole - rint(whole))), &sn, &cs);
        }
        la_turn[i] = make_float2(cs * a.rot_factor, sn * a.rot_factor);
    }
    __syncthreads();
    const int head_cols = a.dim_stride + a.rot_stride, row_cols = a.rank_stride + a.rot_stride;
    T* row = proj + r * row_stride;
    auto turn = [&](const T* src, T* dst, int i) {
        float v[8];
        Vec8<T>::load(src + 8 * i, v);
#pragma unroll
        for (int e = 0; e < 8; e += 2) {
            const float2 cs = la_turn[4 * i + e / 2];
            const float x = v[e], y = v[e + 1];
            v[e] = x * cs.x - y * cs.y;
            v[e + 1] = y * cs.x + x * cs.y;
        }
        Vec8<T>::store(dst + 8 * i, v);
    };
    for (int j = tid; j < a.heads * vecs; j += kLaThreads) {
        const int h = j / vecs, i = j - h * vecs;
        T* src = row + q_col + (int64_t)h * head_cols + a.dim_stride;
        turn(src, q_out ? q_out + (r * a.heads + h) * row_cols + a.rank_stride : src, i);
    }
    if (kv_col < 0) return;
    const int64_t page = t.kv_indices[s.start + pos / t.page_size];
    if (page < 0 || page >= t.num_pages) {
        if (tid == 0) report(status, KTK_STATUS_BAD_PAGE);
        return;
    }
    const T* kv = row + kv_col;
    T* dst = pages + (page * t.page_size + pos % t.page_size) * row_cols;
    for (int i = tid; i < vecs; i += kLaThreads) turn(kv + a.rank_stride, dst + a.rank_stride, i);
    float ss = 0.0f;
    for (int c = tid * 8; c < a.rank_stride; c += kLaThreads * 8) {
        float v[8];
        Vec8<T>::load(kv + c, v);                         // columns behind the rank are zero
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
    }
    ss = warp_sum_f(ss);
    if ((tid & 31) == 0) part[tid >> 5] = ss;
    __syncthreads();
    const float inv = 1.0f / sqrtf((part[0] + part[1] + part[2] + part[3]) / (float)a.rank + a.eps);
    for (int c = tid * 8; c < a.rank_stride; c += kLaThreads * 8) {
        float v[8], w[8];
        Vec8<T>::load(kv + c, v);
        load8(norm_w + c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= inv * w[e];
        Vec8<T>::store(dst + c, v);
    }
}

}  // namespace ktk

using namespace ktk;

extern "C" int ktk_latent_append(void* proj, int64_t row_stride, int64_t q_col, int64_t kv_col, const int32_t* new_indptr,
                                 int64_t rows, const float* norm_w, const double* turns, void* q_out, void* pages,
                                 const ktk_paged* table, const ktk_latent* shape, int32_t* status, void* stream) {
    const char* who = "ktk_latent_append";
    int rc = check_latent(shape, who);
    if (rc != KTK_OK) return rc;
    const ktk_attn rows_of = latent_rows(*shape);
    rc = check_attn(&rows_of, table, who);
    if (rc != KTK_OK) return rc;
    if (rows < 0 || rows > 2147483647LL || (!new_indptr && rows != table->batch)) {
        set_error("%s: %lld rows for %d sequences", who, (long long)rows, table->batch);
        return KTK_ERR_ARG;
    }
    if (rows == 0) return KTK_OK;
    const int64_t q_cols = (int64_t)shape->heads * (shape->dim_stride + shape->rot_stride);
    const int kv_cols = shape->rank_stride + shape->rot_stride;
    if (!proj || !turns || !table->kv_indices || !table->kv_indptr || !table->kv_last_page_len || row_stride % 8 != 0 ||
        q_col % 8 != 0 || q_col < 0 || q_col + q_cols > row_stride ||
        (kv_col >= 0 && (kv_col % 8 != 0 || kv_col + kv_cols > row_stride || !norm_w || !pages)) ||
        (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)pages | (uintptr_t)norm_w) & 15u) != 0) {
        set_error("%s: null or misaligned pointer, or columns outside the row", who);
        return KTK_ERR_ARG;
    }
    const size_t smem = (size_t)shape->rot_stride / 2 * sizeof(float2);
    cudaStream_t st = (cudaStream_t)stream;
    if (shape->dtype == KTK_F32)
        latent_append_kernel<float><<<(unsigned)rows, kLaThreads, smem, st>>>(
            (float*)proj, row_stride, q_col, kv_col, new_indptr, norm_w, turns, (float*)q_out, (float*)pages, *table, *shape,
            status);
    else
        latent_append_kernel<__nv_bfloat16><<<(unsigned)rows, kLaThreads, smem, st>>>(
            (__nv_bfloat16*)proj, row_stride, q_col, kv_col, new_indptr, norm_w, turns, (__nv_bfloat16*)q_out,
            (__nv_bfloat16*)pages, *table, *shape, status);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}
