/*
 * ktk_layers.h -- C ABI of libktk_layers.so: layer mechanisms whose sizes and constants are parameters.
 *
 *   residual_norm    residual stream in fp32: add a (normalised) sublayer output, normalise for the next one
 *   kv_append        keys and values of new tokens into a paged cache with free head sizes
 *   paged_attention  causal attention over that cache: one or two softmax maps per head over shared values
 *                    (with two: their weighted difference, unit norm), score softcap, query temperature
 *   moe_route        router logits, the top experts of each row and their softmax weights, rows per expert
 *   moe_gemm         the experts' matrix products over the rows routed to them
 *
 * Conventions of ktk.h: raw device pointers, cudaStream_t as void*, nothing synchronises or allocates, host-side
 * argument errors come back as KTK_ERR_*, device-side faults go to a status word and the access is skipped.
 * The library also carries the page pool and ktk_last_error of ktk.h, so that it can be used alone.
 *
 * Row strides are counted in elements and are multiples of 8; columns between the true width and the stride hold
 * zeros, and every kernel keeps them that way.  `dtype` is that of activations, weights and cache.
 */
#ifndef KTK_LAYERS_H_
#define KTK_LAYERS_H_

#include "ktk.h"

#ifdef __cplusplus
extern "C" {
#endif

/* Paged cache of one layer, head by head so that a head's tokens of a page lie together:
 *   k_pages [num_pages, kv_heads * maps, page_size, dim_stride], v_pages [num_pages, kv_heads, page_size, vdim_stride]
 * page_size is 16, 32 or 64.  CSR page table as in ktk.h, describing the state AFTER the step's append. */
typedef struct ktk_paged {
    const int32_t* kv_indices;
    const int32_t* kv_indptr;        /* [batch + 1] */
    const int32_t* kv_last_page_len; /* [batch], in [1, page_size] where a sequence holds pages */
    int32_t batch;
    int32_t page_size;
    int64_t num_pages;
} ktk_paged;

typedef struct ktk_attn {
    int32_t heads, kv_heads;         /* query head h reads kv head h / (heads / kv_heads)        */
    int32_t maps;                    /* 1: softmax(q k) v.  2: a1 - lambda a2 over the same v,
                                        then / sqrt(mean square + eps), times out_scale          */
    int32_t dim, vdim;               /* sizes per map and of a value head                        */
    int32_t dim_stride, vdim_stride; /* the same in memory: multiples of 8, zeros in between     */
    int32_t dtype;
    float scale;                     /* score = (q . k) * scale * temperature                    */
    float softcap;                   /* > 0: score <- softcap * tanh(score / softcap)            */
    float temp_coef, temp_every;     /* temperature at position p: 1 + temp_coef ln(floor((p + 1) / temp_every) + 1) */
    float lambda, eps, out_scale;    /* maps = 2 */
    int32_t v_row_stride;            /* 0: v_pages as above.  dim_stride: a key row's first vdim columns are the value
                                        (v_pages = k_pages), as in attention over latents                */
} ktk_attn;

/*
 * One pass over rows of the fp32 residual stream x [rows, stride]:
 *   start:   x = embed[token] * embed_scale (tokens and embed given; x is then only written), or x as it lies
 *   add:     y given: s = sum over `parts` of y[row, part, :];  x += mult * norm(s; post_w, post_b), or
 *            x += mult * s where post_w is null
 *   output:  h given: h = norm(x; pre_w, pre_b), or x itself where pre_w is null, in `dtype`
 * norm(v; w, b) = (v - c) / sqrt(mean((v - c)^2) + eps) * w + b over the first `cols` columns, with c the mean of v
 * (center != 0) or 0, and b null for none.  Norm weights are fp32 [stride].
 * zero (nullable): zero_n ints that the launch clears (the expert counters of the router behind it).
 */
KTK_API int ktk_residual_norm(const int64_t* tokens, const void* embed, int64_t vocab, float embed_scale, float* x,
                              const void* y, int32_t parts, const float* post_w, const float* post_b, float mult, const float* pre_w,
                              const float* pre_b, void* h, float eps, int32_t center, int64_t rows, int32_t cols,
                              int32_t stride, int32_t* zero, int32_t zero_n, int32_t dtype, int32_t* status,
                              void* stream);

/*
 * Write K and V of new tokens into their pages.  proj [rows, row_stride] holds each token's keys
 * (kv_heads * maps * dim_stride) from column k_col and its values (kv_heads * vdim_stride) from column v_col.
 * new_indptr int32 [batch + 1]: rows of each sequence, its newest tokens; null: one row per sequence.
 */
KTK_API int ktk_kv_append(const void* proj, int64_t row_stride, int64_t k_col, int64_t v_col,
                          const int32_t* new_indptr, int64_t rows, void* k_pages, void* v_pages,
                          const ktk_paged* table, const ktk_attn* shape, int32_t* status, void* stream);

/*
 * Causal attention of new tokens (already in their pages) over their sequence.
 * q [rows, q_stride]: heads * maps * dim_stride columns, head by head and map by map; o [rows, heads * vdim_stride].
 * variant: KTK_VARIANT_AUTO, _SIMT (any size, fp32 math), _MMA (bf16, one row per sequence), _UMMA (bf16 on tcgen05).
 * splits: parts that a sequence's keys are cut into (0: policy); with new_indptr only where values lie in the keys.
 * The policy's new_rows: 0 for one row per sequence, else the rows of each.
 * sink fp32 [heads] (nullable, maps = 1): exp(sink) joins each row's denominator, without key, value or scale.
 * gate (nullable, maps = 1), in `dtype`: head h of row r is multiplied by sigmoid(gate[r * gate_stride + h]).
 */
KTK_API int32_t ktk_paged_attention_splits(const ktk_attn* shape, int32_t batch, int32_t new_rows, int64_t max_keys);
KTK_API size_t ktk_paged_attention_workspace(const ktk_attn* shape, int64_t rows, int32_t splits);
KTK_API int ktk_paged_attention(const void* q, int64_t q_stride, const int32_t* new_indptr, int64_t rows,
                                int32_t max_new, const void* k_pages, const void* v_pages, const ktk_paged* table,
                                const float* sink, const void* gate, int64_t gate_stride, void* o, void* workspace,
                                size_t workspace_bytes, int32_t splits, int32_t variant, const ktk_attn* shape,
                                int32_t* status, void* stream);

/*
 * Latent attention: heads share one cached row per token, [latent (rank_stride) | rotated key (rot_stride)]; the page
 * tensor is [num_pages, page_size, rank_stride + rot_stride].  The attention itself is ktk_paged_attention over those
 * rows (kv_heads = 1, dim = rank_stride + rot_stride, vdim = rank, v_row_stride = dim_stride) with queries that carry
 * the key expansion, or ktk_expanded_attention.
 */
typedef struct ktk_latent {
    int32_t heads, dim, rot_dim, vdim, rank;              /* true sizes; dim: the unrotated part of a query head */
    int32_t dim_stride, rot_stride, vdim_stride, rank_stride;
    int32_t dtype;
    float scale;
    float eps;                                            /* of the latent's norm */
    float rot_factor;                                     /* of cos and sin */
} ktk_latent;

/*
 * One launch per layer over rows of proj [rows, row_stride]:
 *   queries at q_col: heads of [dim_stride | rot_stride]; the rotated part (pairs 2 i, 2 i + 1 turned by position *
 *   turns[i] whole turns, fp64 [rot_dim / 2]) goes to q_out [rows, heads, rank_stride + rot_stride], columns rank_stride.., or back
 *   in place where q_out is null;
 *   latents at kv_col (< 0: none): [rank_stride | rot_stride]; norm(latent) * norm_w (fp32 [rank_stride]) and the
 *   rotated key go to the token's page row.
 */
KTK_API int ktk_latent_append(void* proj, int64_t row_stride, int64_t q_col, int64_t kv_col, const int32_t* new_indptr,
                              int64_t rows, const float* norm_w, const double* turns, void* q_out, void* pages,
                              const ktk_paged* table, const ktk_latent* shape, int32_t* status, void* stream);

/*
 * The newest `rows` of a sequence of `total` tokens over keys and values expanded from its latents:
 *   q: rows of [dim_stride | rot_stride] per head, rotated;  kv [total, heads * dim_stride | heads * vdim_stride], the
 *   unrotated keys and the values of every head;  latents [total, rank_stride + rot_stride] (ktk_gather_rows), whose
 *   rotated keys all heads share;  sink, gate as in ktk_paged_attention;  o [rows, heads * vdim_stride].
 * bf16; ktk_expanded_attention_supported tells whether it is built for the sizes.
 */
KTK_API int ktk_expanded_attention_supported(const ktk_latent* shape);
KTK_API int ktk_expanded_attention(const void* q, int64_t q_stride, int64_t rows, int64_t total, const void* kv,
                                   const void* latents, const float* sink, const void* gate, int64_t gate_stride, void* o,
                                   const ktk_latent* shape, int32_t* status, void* stream);
/* The first `total` token rows of a table's only sequence out of pages [num_pages, page_size, row_bytes], in order. */
KTK_API int ktk_gather_rows(const void* pages, void* out, int64_t total, int32_t row_bytes, const ktk_paged* table,
                            int32_t* status, void* stream);

/* Linear recurrence with real gates, per channel (blocks of block_stride channels, the first `block` of them real):
 *   u = conv_b + sum_k conv_w[k] x_(t - taps + 1 + k)                     causal, zeros before the sequence
 *   r = sigmoid(zr + rb), i = sigmoid(zi + ib)                            zr, zi: block-diagonal products of u
 *   a = exp(-r decay);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu_tanh(y)
 * `state` fp32 [slots, width] and `ring` [slots, taps, width] (the newest inputs, that of position p at p % taps) belong
 * to slots; a sequence that starts at position 0 reads neither.  width = blocks * block_stride.
 */
typedef struct ktk_lru {
    int32_t blocks, block, block_stride, taps;
    int32_t dtype;
} ktk_lru;

/* x: rows of proj at column x_col; u [rows, width]; conv_w fp32 [taps, width], conv_b fp32 [width].  slots int32 [batch];
 * new_indptr as in ktk_kv_append.  Updates the ring. */
KTK_API int ktk_lru_conv(const void* proj, int64_t row_stride, int64_t x_col, const int32_t* new_indptr, int64_t rows,
                         int32_t max_new, const int32_t* slots, int64_t num_slots, const float* conv_w,
                         const float* conv_b, void* ring, void* u, const ktk_paged* table, const ktk_lru* shape,
                         int32_t* status, void* stream);

/* z fp32 [blocks, rows, 2 * block_stride]: zr, then zi of a block; y: rows of proj at y_col; out [rows, width] in dtype. */
KTK_API int ktk_lru_scan(const float* z, const void* u, const void* proj, int64_t row_stride, int64_t y_col,
                         const int32_t* new_indptr, int64_t rows, int32_t max_new, const int32_t* slots,
                         int64_t num_slots, const float* rb, const float* ib, const float* decay, float* state,
                         void* out, const ktk_paged* table, const ktk_lru* shape, int32_t* status, void* stream);

/* ktk_lru_conv, the gate products and ktk_lru_scan of one token of every sequence in one launch (bf16; blocks of channels
 * up to what ktk_lru_decode_supported accepts).  gates [blocks, 2, block_stride, block_stride]: r's rows, then i's. */
KTK_API int ktk_lru_decode_supported(const ktk_lru* shape);
KTK_API int ktk_lru_decode(const void* proj, int64_t row_stride, int64_t y_col, int64_t x_col, int64_t rows,
                           const int32_t* slots, int64_t num_slots, const float* conv_w, const float* conv_b,
                           const void* gates, const float* rb, const float* ib, const float* decay, void* ring, float* state,
                           void* out, const ktk_paged* table, const ktk_lru* shape, int32_t* status, void* stream);

/* Mixture of experts over rows h [rows, width_stride]. */
typedef struct ktk_moe {
    int32_t experts, top;
    int32_t width, ff;               /* true sizes */
    int32_t width_stride, ff_stride;
    int32_t dtype;
    int32_t scoring;                 /* weights: 0 softmax over the chosen logits, 1 softmax over all of them */
    float limit, slope, shift;       /* gated activation, see ktk_gated_rows */
} ktk_moe;

/*
 * logits = W h + b in fp32 (W [experts, width_stride], b fp32 or null); the `top` largest of each row (ties to the
 * lower expert) and their weights (`scoring`).  ids / weights [rows, top].  counts [experts] (cleared by the caller):
 * rows of each expert; bucket [experts, rows]: their row * top + place, in no particular order.
 */
KTK_API int ktk_moe_route(const void* h, const void* w, const float* b, int32_t* ids, float* weights, int32_t* counts,
                          int32_t* bucket, int64_t rows, const ktk_moe* shape, int32_t variant, void* stream);

/*
 * Expert products.  Rows of expert e take the places [sum of counts before e, + counts[e]) of `act`.
 *   stage 0: act [rows * top, ff_stride] = gated(G h, U h);  w = [experts, ff_stride, 2, width_stride] (a row of G, then
 *            the row of U of the same inner column)
 *   stage 1: y [rows, top, width_stride] = weight * (D act);   w = [experts, width_stride, ff_stride]
 * variant: KTK_VARIANT_AUTO, _SIMT (fp32 math), _UMMA (bf16 on tcgen05).
 */
KTK_API int ktk_moe_gemm(int32_t stage, const void* in, const void* w, void* out, const float* weights,
                         const int32_t* counts, const int32_t* bucket, int64_t rows, const ktk_moe* shape,
                         int32_t variant, int32_t* status, void* stream);

/*
 * out [rows, cols_stride] = gated(in[:, 0 .. cols_stride), in[:, cols_stride .. 2 cols_stride)):
 *   gated(g, u) = g' sigmoid(slope g') (u' + shift),  g' = min(g, limit),  u' = clamp(u, -limit, limit)
 * (limit = infinity, slope = 1, shift = 0: silu(g) u).
 */
KTK_API int ktk_gated_rows(const void* in, void* out, int64_t rows, int32_t cols_stride, float limit, float slope,
                           float shift, int32_t dtype, void* stream);

/* z [n] <- cap tanh(z scale / cap), fp32, in place (cap <= 0: z scale). */
KTK_API int ktk_scale_cap(float* z, int64_t n, float scale, float cap, void* stream);

#ifdef __cplusplus
}
#endif
#endif
