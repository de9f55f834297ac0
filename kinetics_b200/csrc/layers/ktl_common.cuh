// Shared by the kernels of libktk_layers.so: the page table of a layer with free head sizes, its argument checks,
// and how the rows routed to experts are cut into tiles.
#pragma once

#include "../ktk_vec.cuh"
#include "ktk_layers.h"

namespace ktk {

// sequence b of the table: first entry of its page list, pages, tokens
struct Span {
    int start, pages, total;
    bool bad;
};
__device__ __forceinline__ Span span_of(const ktk_paged& t, int b) {
    Span s;
    s.start = t.kv_indptr[b];
    s.pages = t.kv_indptr[b + 1] - s.start;
    const int last = s.pages > 0 ? t.kv_last_page_len[b] : 0;
    s.bad = s.pages < 0 || (s.pages > 0 && (last < 1 || last > t.page_size));
    s.total = s.pages > 0 && !s.bad ? (s.pages - 1) * t.page_size + last : 0;
    return s;
}

// sequence whose rows [indptr[b], indptr[b + 1]) hold row r
__device__ __forceinline__ int sequence_of_row(const int32_t* indptr, int batch, int64_t r) {
    int lo = 0, hi = batch;
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if ((int64_t)indptr[mid] <= r) lo = mid; else hi = mid;
    }
    return lo;
}

// row of head `head` (of `heads`) at token slot `slot` = page * page_size + place, in pages stored head by head
__device__ __forceinline__ int64_t row_in_pages(int64_t slot, int page_size, int heads, int head) {
    const int64_t page = slot / page_size;
    return (page * heads + head) * page_size + (slot - page * page_size);
}

// factor of the query at position pos (coef 0: none)
__device__ __forceinline__ float query_temperature(float coef, float every, int pos) {
    if (coef == 0.0f) return 1.0f;
    return 1.0f + coef * logf(floorf(__fdiv_rn((float)(pos + 1), every)) + 1.0f);
}

inline int check_attn(const ktk_attn* a, const ktk_paged* t, const char* who) {
    if (a == nullptr || t == nullptr) { set_error("%s: null shape or table", who); return KTK_ERR_ARG; }
    if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->dim <= 0 || a->vdim <= 0 ||
        a->dim_stride < a->dim || a->vdim_stride < a->vdim || a->dim_stride % 8 != 0 || a->vdim_stride % 8 != 0 ||
        (a->maps != 1 && a->maps != 2) || (a->dtype != KTK_F32 && a->dtype != KTK_BF16) ||
        (a->temp_coef != 0.0f && !(a->temp_every > 0.0f)) ||
        (a->v_row_stride != 0 && (a->v_row_stride != a->dim_stride || a->vdim_stride > a->dim_stride || a->maps != 1))) {
        set_error("%s: heads=%d kv_heads=%d maps=%d dim=%d (stride %d) vdim=%d (stride %d) dtype=%d temp_every=%g", who,
                  a->heads, a->kv_heads, a->maps, a->dim, a->dim_stride, a->vdim, a->vdim_stride, a->dtype,
                  (double)a->temp_every);
        return KTK_ERR_ARG;
    }
    if (t->page_size != 16 && t->page_size != 32 && t->page_size != 64) {
        set_error("%s: page_size %d (16, 32 and 64 are built)", who, t->page_size);
        return KTK_ERR_UNSUPPORTED;
    }
    if (t->batch < 0 || t->num_pages < 0 || t->num_pages > 2147483647LL / t->page_size ||
        t->num_pages > 2147483647LL / ((int64_t)a->kv_heads * a->maps)) {
        set_error("%s: batch=%d num_pages=%lld", who, t->batch, (long long)t->num_pages);
        return KTK_ERR_ARG;
    }
    return KTK_OK;
}

// elements between two value rows of a head
__host__ __device__ __forceinline__ int value_row(const ktk_attn& a) { return a.v_row_stride ? a.v_row_stride : a.vdim_stride; }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

struct AttnParams {
    ktk_attn a;
    ktk_paged t;
    const void* q;
    int64_t q_stride;
    const int32_t* new_indptr;
    int64_t rows;
    int max_new;
    const void *k, *v;
    const float* sink;
    const void* gate;
    int64_t gate_stride;
    void* o;
    float* ws;
    int splits;
    int32_t* status;
};

// latent attention: its sizes, and the attention over its cached rows
inline int check_latent(const ktk_latent* a, const char* who) {
    if (a == nullptr || a->heads <= 0 || a->dim <= 0 || a->rot_dim < 0 || a->rot_dim % 2 != 0 || a->vdim <= 0 || a->rank <= 0 ||
        a->dim_stride < a->dim || a->rot_stride < a->rot_dim || a->vdim_stride < a->vdim || a->rank_stride < a->rank ||
        (a->dim_stride | a->rot_stride | a->vdim_stride | a->rank_stride) % 8 != 0 || a->rot_stride > 4096 ||
        (a->dtype != KTK_F32 && a->dtype != KTK_BF16)) {
        set_error("%s: bad sizes", who);
        return KTK_ERR_ARG;
    }
    return KTK_OK;
}
inline ktk_attn latent_rows(const ktk_latent& a) {
    ktk_attn r{};
    r.heads = a.heads;
    r.kv_heads = r.maps = 1;
    r.dim = r.dim_stride = r.v_row_stride = a.rank_stride + a.rot_stride;
    r.vdim = a.rank;
    r.vdim_stride = a.rank_stride;
    r.dtype = a.dtype;
    r.scale = a.scale;
    r.temp_every = 1.0f;
    return r;
}

// splits of each of `units` pieces of work: between `lo_rounds` and `hi_rounds` rounds of `resident` CTAs, and among those
// the count that leaves the last round fullest
inline int32_t fill_rounds(int64_t units, int64_t resident, int lo_rounds, int hi_rounds, int64_t most, int64_t cap) {
    if (units <= 0) return 1;
    if (most > cap) most = cap;
    int64_t lo = (lo_rounds * resident + units - 1) / units, hi = (hi_rounds * resident + units - 1) / units, best = 1;
    if (lo > most) lo = most;
    if (hi > most) hi = most;
    double best_fill = 0.0;
    for (int64_t s = lo < 1 ? 1 : lo; s <= hi; ++s) {
        const int64_t ctas = units * s, rounds = (ctas + resident - 1) / resident;
        const double fill = (double)ctas / (double)(rounds * resident);
        if (fill > best_fill + 0.01) { best_fill = fill; best = s; }
    }
    return (int32_t)best;
}

int launch_attn_simt(const AttnParams& p, cudaStream_t st);
bool attn_decode_supported(const ktk_attn& a);
int32_t attn_decode_splits(const ktk_attn& a, int batch, int64_t max_keys);
size_t attn_decode_workspace(const ktk_attn& a, int64_t rows, int splits);
int make_cache_maps(const AttnParams& p, struct CUtensorMap_st* k_map, struct CUtensorMap_st* v_map, unsigned box_rows, const char* who);
int launch_attn_decode(const AttnParams& p, cudaStream_t st);
bool attn_umma_supported(const ktk_attn& a);
bool attn_shared_supported(const ktk_attn& a);
int32_t attn_shared_splits(const ktk_attn& a, int batch, int new_rows, int64_t max_keys);
size_t attn_shared_workspace(const ktk_attn& a, int64_t rows, int splits);
int launch_attn_shared(const AttnParams& p, cudaStream_t st);
int launch_attn_umma(const AttnParams& p, cudaStream_t st);

// ---- experts ------------------------------------------------------------------------------------------------
constexpr int kMaxExperts = 1024;

struct MoeParams {
    ktk_moe m;
    const void* in;
    const void* w;
    void* out;
    const float* weights;
    const int32_t* counts;
    const int32_t* bucket;
    int64_t rows;
    int32_t* status;
};
int launch_moe_simt(int stage, const MoeParams& p, cudaStream_t st);
bool moe_umma_supported(const ktk_moe& m);
int launch_moe_umma(int stage, const MoeParams& p, cudaStream_t st);

// g' sigmoid(slope g') (u' + shift), g' = min(g, limit), u' = clamp(u, -limit, limit).  FAST: with the special-function
// unit's exponential.
template <bool FAST> __device__ __forceinline__ float gated(float g, float u, float limit, float slope, float shift) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit) + shift;
    if (FAST) return __fdividef(g, 1.0f + __expf(-slope * g)) * u;
    return g / (1.0f + expf(-slope * g)) * u;
}

// How the rows of all experts are cut into tiles of at most `tile` rows; one warp fills this from `counts`.
struct ExpertPlan {
    int first_tile[kMaxExperts + 1];   // tiles of the experts before e
    int first_row[kMaxExperts + 1];    // rows of the experts before e
};
__device__ __forceinline__ void plan_experts(ExpertPlan& pl, const int32_t* counts, int experts, int64_t rows,
                                             int tile) {
    const int lane = threadIdx.x & 31;
    int tiles = 0, done = 0;
    for (int base = 0; base < experts; base += 32) {
        const int e = base + lane;
        int n = e < experts ? counts[e] : 0;
        n = n < 0 ? 0 : (n > rows ? (int)rows : n);
        int tn = (n + tile - 1) / tile, t0 = tn, n0 = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int a = __shfl_up_sync(0xffffffffu, t0, o), b = __shfl_up_sync(0xffffffffu, n0, o);
            if (lane >= o) { t0 += a; n0 += b; }
        }
        if (e < experts) { pl.first_tile[e] = tiles + t0 - tn; pl.first_row[e] = done + n0 - n; }
        tiles += __shfl_sync(0xffffffffu, t0, 31);
        done += __shfl_sync(0xffffffffu, n0, 31);
    }
    if (lane == 0) { pl.first_tile[experts] = tiles; pl.first_row[experts] = done; }
}
// expert of tile t
__device__ __forceinline__ int expert_of_tile(const ExpertPlan& pl, int experts, int t) {
    int lo = 0, hi = experts;
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (pl.first_tile[mid] <= t) lo = mid; else hi = mid;
    }
    return lo;
}

}  // namespace ktk
