// Keys and values of new tokens -> pages with free head sizes, and the entry point of the attention kernels.
#include "ktl_common.cuh"

namespace ktk {

// one CTA per row: 16-byte copies of its K and its V row
template <typename T>
__global__ void __launch_bounds__(128)
kv_append_kernel(const T* __restrict__ proj, int64_t row_stride, int64_t k_col, int64_t v_col,
                 const int32_t* __restrict__ new_indptr, T* __restrict__ k_pages, T* __restrict__ v_pages,
                 const ktk_paged t, int k_heads, int v_heads, int dim, int vdim, int32_t* status) {
    const int64_t r = blockIdx.x;
    const int b = new_indptr ? sequence_of_row(new_indptr, t.batch, r) : (int)r;
    const Span s = span_of(t, b);
    const int pos = new_indptr ? s.total - (new_indptr[b + 1] - (int)r) : s.total - 1;
    if (s.bad || pos < 0 || pos >= s.total) {
        if (threadIdx.x == 0) report(status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const int64_t page = t.kv_indices[s.start + pos / t.page_size];
    if (page < 0 || page >= t.num_pages) {
        if (threadIdx.x == 0) report(status, KTK_STATUS_BAD_PAGE);
        return;
    }
    const int slot = pos % t.page_size;
    constexpr int kPer = 16 / sizeof(T);
    // 16-byte pieces of the row, head by head: head g of the page starts at (page * heads + g) * page_size tokens
    auto copy = [&](const T* src, T* dst, int heads, int size) {
        const int per = size / kPer;
        for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
            const int g = i / per, c = i - g * per;
            reinterpret_cast<uint4*>(dst + (((int64_t)page * heads + g) * t.page_size + slot) * size)[c] =
                reinterpret_cast<const uint4*>(src)[i];
        }
    };
    copy(proj + r * row_stride + k_col, k_pages, k_heads, dim);
    copy(proj + r * row_stride + v_col, v_pages, v_heads, vdim);
}

template <typename T>
static int append_launch(const void* proj, int64_t row_stride, int64_t k_col, int64_t v_col, const int32_t* ni,
                         int64_t rows, void* k, void* v, const ktk_paged& t, const ktk_attn& a, int32_t* status,
                         cudaStream_t st) {
    kv_append_kernel<T><<<(unsigned)rows, 128, 0, st>>>((const T*)proj, row_stride, k_col, v_col, ni, (T*)k, (T*)v, t,
                                                         a.kv_heads * a.maps, a.kv_heads, a.dim_stride, a.vdim_stride,
                                                         status);
    KTK_CUDA_TRY(cudaGetLastError(), "ktk_kv_append");
    return KTK_OK;
}

}  // namespace ktk

using namespace ktk;

extern "C" int ktk_kv_append(const void* proj, int64_t row_stride, int64_t k_col, int64_t v_col,
                             const int32_t* new_indptr, int64_t rows, void* k_pages, void* v_pages,
                             const ktk_paged* table, const ktk_attn* shape, int32_t* status, void* stream) {
    const char* who = "ktk_kv_append";
    const int rc = check_attn(shape, table, who);
    if (rc != KTK_OK) return rc;
    if (rows < 0 || rows > 2147483647LL || (!new_indptr && rows != table->batch)) {
        set_error("%s: %lld rows for %d sequences", who, (long long)rows, table->batch);
        return KTK_ERR_ARG;
    }
    if (rows == 0) return KTK_OK;
    const int k_row = shape->kv_heads * shape->maps * shape->dim_stride, v_row = shape->kv_heads * shape->vdim_stride;
    if (!proj || !k_pages || !v_pages || !table->kv_indices || !table->kv_indptr || !table->kv_last_page_len ||
        row_stride % 8 != 0 || k_col % 8 != 0 || v_col % 8 != 0 || k_col < 0 || v_col < 0 ||
        k_col + k_row > row_stride || v_col + v_row > row_stride ||
        (((uintptr_t)proj | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15u) != 0) {
        set_error("%s: null or misaligned pointer, or columns outside the row", who);
        return KTK_ERR_ARG;
    }
    if (shape->v_row_stride != 0) { set_error("%s: values inside the keys are written by ktk_latent_append", who); return KTK_ERR_UNSUPPORTED; }
    cudaStream_t st = (cudaStream_t)stream;
    return shape->dtype == KTK_F32
               ? append_launch<float>(proj, row_stride, k_col, v_col, new_indptr, rows, k_pages, v_pages, *table, *shape,
                                      status, st)
               : append_launch<__nv_bfloat16>(proj, row_stride, k_col, v_col, new_indptr, rows, k_pages, v_pages,
                                              *table, *shape, status, st);
}

extern "C" int32_t ktk_paged_attention_splits(const ktk_attn* shape, int32_t batch, int32_t new_rows, int64_t max_keys) {
    if (attn_shared_supported(*shape)) return attn_shared_splits(*shape, batch, new_rows, max_keys);
    if (new_rows > 0) return 1;
    return attn_decode_supported(*shape) ? attn_decode_splits(*shape, batch, max_keys) : 1;
}

extern "C" size_t ktk_paged_attention_workspace(const ktk_attn* shape, int64_t rows, int32_t splits) {
    if (attn_shared_supported(*shape)) return attn_shared_workspace(*shape, rows, splits);
    return attn_decode_supported(*shape) ? attn_decode_workspace(*shape, rows, splits) : 0;
}

extern "C" int ktk_paged_attention(const void* q, int64_t q_stride, const int32_t* new_indptr, int64_t rows,
                                   int32_t max_new, const void* k_pages, const void* v_pages, const ktk_paged* table,
                                   const float* sink, const void* gate, int64_t gate_stride, void* o, void* workspace,
                                   size_t workspace_bytes, int32_t splits, int32_t variant, const ktk_attn* shape,
                                   int32_t* status, void* stream) {
    const char* who = "ktk_paged_attention";
    const int rc = check_attn(shape, table, who);
    if (rc != KTK_OK) return rc;
    if (rows < 0 || rows > 2147483647LL || (!new_indptr && rows != table->batch) || (new_indptr && max_new < 0)) {
        set_error("%s: %lld rows for %d sequences, at most %d each", who, (long long)rows, table->batch, max_new);
        return KTK_ERR_ARG;
    }
    if (rows == 0) return KTK_OK;
    const int q_row = shape->heads * shape->maps * shape->dim_stride;
    if (!q || !k_pages || !v_pages || !o || !table->kv_indices || !table->kv_indptr || !table->kv_last_page_len ||
        q_stride < q_row || q_stride % 8 != 0 ||
        (((uintptr_t)q | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)o | (uintptr_t)workspace) & 15u) != 0) {
        set_error("%s: null or misaligned pointer, or a row stride of %lld", who, (long long)q_stride);
        return KTK_ERR_ARG;
    }
    if (variant < KTK_VARIANT_AUTO || variant > KTK_VARIANT_UMMA) {
        set_error("%s: unknown variant %d", who, variant);
        return KTK_ERR_ARG;
    }
    if ((sink || gate) && shape->maps != 1) { set_error("%s: sinks and gates go with one map", who); return KTK_ERR_UNSUPPORTED; }
    if (gate && gate_stride < shape->heads) { set_error("%s: gate_stride %lld", who, (long long)gate_stride); return KTK_ERR_ARG; }
    AttnParams p{*shape, *table, q, q_stride, new_indptr, rows, max_new, k_pages, v_pages, sink, gate, gate_stride, o,
                 (float*)workspace, splits, status};
    const bool can_decode = !new_indptr && attn_decode_supported(*shape);
    const bool can_umma = new_indptr && attn_umma_supported(*shape), can_shared = attn_shared_supported(*shape);
    if ((variant == KTK_VARIANT_MMA && !can_decode) || (variant == KTK_VARIANT_UMMA && !can_umma && !can_shared)) {
        set_error("%s: variant %d is not built for this case", who, variant);
        return KTK_ERR_UNSUPPORTED;
    }
    if (variant != KTK_VARIANT_SIMT && can_shared) {
        if (p.splits <= 0) p.splits = attn_shared_splits(*shape, table->batch, new_indptr ? max_new : 0, 1 << 20);
        const size_t need = attn_shared_workspace(*shape, rows, p.splits);
        if (need && (!workspace || workspace_bytes < need)) {
            set_error("%s: workspace of %zu bytes needed, got %zu", who, need, workspace ? workspace_bytes : (size_t)0);
            return KTK_ERR_WORKSPACE;
        }
        return launch_attn_shared(p, (cudaStream_t)stream);
    }
    if (variant != KTK_VARIANT_SIMT && can_umma) return launch_attn_umma(p, (cudaStream_t)stream);
    if (variant != KTK_VARIANT_SIMT && can_decode) {
        if (p.splits <= 0) p.splits = attn_decode_splits(*shape, table->batch, 1 << 20);
        const size_t need = attn_decode_workspace(*shape, rows, p.splits);
        if (need && (!workspace || workspace_bytes < need)) {
            set_error("%s: workspace of %zu bytes needed, got %zu", who, need, workspace ? workspace_bytes : (size_t)0);
            return KTK_ERR_WORKSPACE;
        }
        return launch_attn_decode(p, (cudaStream_t)stream);
    }
    return launch_attn_simt(p, (cudaStream_t)stream);
}
