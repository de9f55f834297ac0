// Causal attention of a prompt's tokens over keys and values expanded from latents: per head an unrotated key and a value
// of its own, one rotated key part for all heads; a sink in the denominator, a gate on the output.  bf16 on the
// fifth-generation tensor cores, fp32 scores and sums.
//
// One CTA per (head, two tiles of 128 tokens): both tiles share every block of 64 keys that comes into shared memory.
// Softmax warps 0..3 hold the first tile, 4..7 the second, thread r of each the tile's row r = lane r of tensor memory.
// Roles:
//     loading warp (one lane)   TMA: K (unrotated columns of the head, then the shared rotated ones) and V of a block,
//                               two blocks in flight
//     issuing warp              S_m[128 x 64] = Q_m . K^T, then O_m[128 x vdim] += P_m . V with P_m from tensor memory;
//                               S of block j + 1 is issued before O += P . V of block j
//     softmax thread            S row -> registers; scale, mask, 2^x against a reference, at first the largest of the sink
//                               and the first block's scores, that moves in jumps of at least 2^8; P as bf16 pairs over that S
// Tensor memory: S of two blocks and two tiles in columns [0, 256), O_1 and O_2 behind.  Every wait is bounded.
#include "ktl_score.cuh"

namespace ktk {

constexpr int kAeKeys = 64;
constexpr int kAeThreads = 320;
constexpr int kAeTmemCols = 512;
constexpr int kAeColO = 256;
constexpr int kAeQTile = kUmRows * 128;       // [128 rows][64 columns]
constexpr int kAeKTile = kAeKeys * 128;       // [64 keys][64 columns]
constexpr int kAeMaxChunks = 4;               // of the key: 64 columns each
constexpr float kAeSlack = 8.0f;

struct ExpandedParams {
    ktk_latent a;
    const __nv_bfloat16* q;
    int64_t q_stride;
    int n, total;
    const float* sink;
    const __nv_bfloat16* gate;
    int64_t gate_stride;
    __nv_bfloat16* o;
    int32_t* status;
};

template <int VC>
__global__ void __launch_bounds__(kAeThreads, 1)
attn_expanded_kernel(const ExpandedParams p, const __grid_constant__ CUtensorMap k_map,
                     const __grid_constant__ CUtensorMap r_map, const __grid_constant__ CUtensorMap v_map) {
    extern __shared__ uint8_t ae_raw[];
    // S complete (tile, buffer) | P in place (tile, buffer) | K, V landed (buffer) | K, V read out (buffer) | O complete (tile)
    __shared__ __align__(8) uint64_t bar_s[2][2], bar_p[2][2], bar_k[2], bar_v[2], bar_kfree[2], bar_vfree[2], bar_o[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int abort_flag;
    const ktk_latent& a = p.a;
    const int nc = (a.dim_stride + 63) / 64, dc = nc + (a.rot_stride + 63) / 64;     // chunks of a key
    uint8_t* sQ = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ae_raw) + 1023) & ~uintptr_t(1023));   // [tile][chunk]
    uint8_t* sK = sQ + 2 * dc * kAeQTile;              // [buffer][chunk]
    uint8_t* sV = sK + 2 * dc * kAeKTile;              // [buffer][chunk]
    const int k_buf = dc * kAeKTile;
    constexpr int kVBuf = VC * kAeKTile;

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool issuer = warp == 8, loader = warp == 9;
    const int head = blockIdx.y;
    const int tok0 = (int)(gridDim.x - 1 - blockIdx.x) * 2 * kUmRows;      // the tiles with the longest history first
    const int base = p.total - p.n;
    int blocks[2];                                      // key blocks of each tile
#pragma unroll
    for (int m = 0; m < 2; ++m) {
        const int t0 = tok0 + m * kUmRows, t1 = t0 + kUmRows < p.n ? t0 + kUmRows : p.n;
        blocks[m] = t0 < p.n ? (base + t1 + kAeKeys - 1) / kAeKeys : 0;
    }
    const int n_blocks = blocks[1] > blocks[0] ? blocks[1] : blocks[0];

    const int tile = warp >> 2, row = tid & (kUmRows - 1);
    const int tok = tok0 + tile * kUmRows + row;
    const bool row_on = warp < 8 && tok < p.n;
    const int vis = row_on ? base + tok + 1 : 0;        // keys at positions < vis are seen

    if (tid == 0) {
        for (int i = 0; i < 2; ++i) {
            for (int m = 0; m < 2; ++m) { mbar_init(&bar_s[m][i], 1); mbar_init(&bar_p[m][i], 4); }
            mbar_init(&bar_k[i], 1); mbar_init(&bar_v[i], 1);
            mbar_init(&bar_kfree[i], 1); mbar_init(&bar_vfree[i], 1);
            mbar_init(&bar_o[i], 1);
        }
        abort_flag = 0;
        mbar_init_fence();
    }
    if (warp < 8) {
        const __nv_bfloat16* src = p.q + (int64_t)(row_on ? tok : 0) * p.q_stride + (int64_t)head * (a.dim_stride + a.rot_stride);
        uint8_t* dst = sQ + tile * dc * kAeQTile;
        for (int c = 0; c < dc * 8; ++c) {
            const bool rot = c >= nc * 8;
            const int col = (rot ? c - nc * 8 : c) * 8, size = rot ? a.rot_stride : a.dim_stride;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (row_on && col < size) v = *reinterpret_cast<const uint4*>(src + (rot ? a.dim_stride : 0) + col);
            *reinterpret_cast<uint4*>(dst + (c >> 3) * kAeQTile + swz(row, c & 7)) = v;
        }
        fence_proxy_async();
    } else if (issuer) {
        tmem_alloc(&tmem_base_s, kAeTmemCols);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_base_s;

    if (issuer) {
        const int ksteps = (a.dim_stride + 15) / 16, rsteps = (a.rot_stride + 15) / 16;
        const uint32_t idesc_s = umma_idesc(kAeKeys, false), idesc_o = umma_idesc((a.vdim_stride + 15) / 16 * 16, true);
        const uint64_t q_desc = umma_desc(smem_u32(sQ), 0, 1024), k_desc = umma_desc(smem_u32(sK), 0, 1024);
        const uint64_t v_desc = umma_desc(smem_u32(sV), kAeKTile, 1024);
        auto wait = [&](uint64_t* bar, int round) {
            return mbar_wait_all(bar, round & 1, &abort_flag);
        };
        auto issue_s = [&](int blk) {
            const int buf = blk & 1;
            if (!wait(&bar_k[buf], blk >> 1)) return false;
            tc_fence_after();
            if (elect_one()) {
                const uint64_t ka = umma_desc_at(k_desc, buf * k_buf);
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    if (blk >= blocks[m]) continue;
                    const uint64_t qa = umma_desc_at(q_desc, m * dc * kAeQTile);
                    const uint32_t d = tmem + m * 128 + buf * kAeKeys;
                    for (int k = 0; k < ksteps; ++k)
                        umma_f16(d, umma_desc_at(qa, (k >> 2) * kAeQTile + (k & 3) * 32),
                                 umma_desc_at(ka, (k >> 2) * kAeKTile + (k & 3) * 32), idesc_s, k > 0 ? 1u : 0u);
                    for (int k = 0; k < rsteps; ++k)
                        umma_f16(d, umma_desc_at(qa, (nc + (k >> 2)) * kAeQTile + (k & 3) * 32),
                                 umma_desc_at(ka, (nc + (k >> 2)) * kAeKTile + (k & 3) * 32), idesc_s, 1u);
                    umma_commit(&bar_s[m][buf]);
                }
                umma_commit(&bar_kfree[buf]);
            }
            __syncwarp();
            return true;
        };
        bool ok = issue_s(0);
        for (int j = 0; j < n_blocks && ok; ++j) {
            const int buf = j & 1;
            if (j + 1 < n_blocks) ok = issue_s(j + 1);
            ok = ok && wait(&bar_v[buf], j >> 1);
            const uint64_t va = umma_desc_at(v_desc, buf * kVBuf);
#pragma unroll
            for (int m = 0; m < 2; ++m) {
                if (j >= blocks[m]) continue;
                ok = ok && wait(&bar_p[m][buf], j >> 1);
                if (!ok) break;
                tc_fence_after();
                if (elect_one()) {
#pragma unroll
                    for (int k = 0; k < kAeKeys / 16; ++k)
                        umma_f16_ts(tmem + kAeColO + m * 128, tmem + m * 128 + buf * kAeKeys + k * 8,
                                    umma_desc_at(va, k * (16 * 128)), idesc_o, (j > 0 || k > 0) ? 1u : 0u);
                    if (j + 1 == blocks[m]) umma_commit(&bar_o[m]);
                }
                __syncwarp();
            }
            if (ok && elect_one()) umma_commit(&bar_vfree[buf]);
            __syncwarp();
        }
    } else if (loader) {
        if (lane == 0) {
            // K (which = 0) or V (which = 1) of block `blk`; columns and tokens outside come as zeros
            auto load = [&](int blk, int which) {
                const int buf = blk & 1;
                uint64_t* bar = which ? &bar_v[buf] : &bar_k[buf];
                mbar_arrive_expect_tx(bar, (uint32_t)((which ? VC : dc) * kAeKTile));
                if (which) {
#pragma unroll
                    for (int c = 0; c < VC; ++c)
                        tma_load_3d(sV + buf * kVBuf + c * kAeKTile, &v_map, bar, c * 64, head, blk * kAeKeys);
                } else {
                    for (int c = 0; c < dc; ++c) {
                        uint8_t* dst = sK + buf * k_buf + c * kAeKTile;
                        if (c < nc) tma_load_3d(dst, &k_map, bar, c * 64, head, blk * kAeKeys);
                        else tma_load_3d(dst, &r_map, bar, (c - nc) * 64, 0, blk * kAeKeys);
                    }
                }
            };
            prefetch_tensormap(&k_map);
            prefetch_tensormap(&r_map);
            prefetch_tensormap(&v_map);
            int k_issued = 1, v_issued = 1;
            load(0, 0);
            load(0, 1);
            if (n_blocks > 1) { load(1, 0); ++k_issued; }
            bool alive = true;
            for (int j = 0; j < n_blocks && alive; ++j) {
                if (j + 1 < n_blocks) {                          // V of block j + 1 over that of block j - 1
                    alive = j == 0 || mbar_wait_fast(&bar_vfree[(j + 1) & 1], ((j - 1) >> 1) & 1, &abort_flag);
                    if (alive) { load(j + 1, 1); ++v_issued; }
                }
                if (alive && j + 2 < n_blocks) {                 // K of block j + 2 over that of block j
                    alive = mbar_wait_fast(&bar_kfree[j & 1], (j >> 1) & 1, &abort_flag);
                    if (alive) { load(j + 2, 0); ++k_issued; }
                }
            }
            if (!alive) {                                        // the copies in flight still write shared memory
                volatile int never = 0;
                for (int i = k_issued > 2 ? k_issued - 2 : 0; i < k_issued; ++i) mbar_wait(&bar_k[i & 1], (i >> 1) & 1, &never);
                for (int i = v_issued > 2 ? v_issued - 2 : 0; i < v_issued; ++i) mbar_wait(&bar_v[i & 1], (i >> 1) & 1, &never);
            }
        }
    }
    else {
        const uint32_t my = tmem + ((uint32_t)((warp & 3) * 32) << 16);
        const float f = a.scale * kLog2eF;
        const int mine = blocks[tile], tile_min_vis = base + tok0 + tile * kUmRows + 1;
        float m_ref = p.sink ? p.sink[head] * kLog2eF : -1e30f, l_run = p.sink ? 1.0f : 0.0f;
        bool alive = true;
        for (int j = 0; j < mine; ++j) {
            const int buf = j & 1;
            const uint32_t s_col = tile * 128 + buf * kAeKeys;
            if (!mbar_wait_all(&bar_s[tile][buf], (j >> 1) & 1, &abort_flag)) { alive = false; break; }
            tc_fence_after();
            float lo[32], hi[32];
            tmem_ld64(my + s_col, lo, hi);
            if ((j + 1) * kAeKeys > tile_min_vis || !row_on) {         // some row of the tile does not see the whole block
                const int first = j * kAeKeys;
#pragma unroll
                for (int c = 0; c < 32; ++c) {
                    lo[c] = first + c < vis ? lo[c] : -INFINITY;
                    hi[c] = first + 32 + c < vis ? hi[c] : -INFINITY;
                }
            }
            float mx = fmaxf(lo[0], hi[0]);
#pragma unroll
            for (int c = 1; c < 32; ++c) mx = fmaxf(mx, fmaxf(lo[c], hi[c]));
            mx *= f;                                                   // f > 0
            float alpha = 1.0f;
            if (mx > m_ref + (j == 0 ? 0.0f : kAeSlack)) {
                alpha = ex2(m_ref - mx);
                m_ref = mx;
                l_run *= alpha;
            }
            uint32_t packed[32];
            float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
            for (int c = 0; c < 16; ++c) {
                const float p0 = ex2(fmaf(lo[2 * c], f, -m_ref)), p1 = ex2(fmaf(lo[2 * c + 1], f, -m_ref));
                const float p2 = ex2(fmaf(hi[2 * c], f, -m_ref)), p3 = ex2(fmaf(hi[2 * c + 1], f, -m_ref));
                sum0 += p0 + p1;
                sum1 += p2 + p3;
                packed[c] = pack_bf16(p0, p1);
                packed[16 + c] = pack_bf16(p2, p3);
            }
            l_run += sum0 + sum1;
            if (j > 0 && __any_sync(0xffffffffu, alpha != 1.0f)) {
                if (!mbar_wait_all(&bar_vfree[(j - 1) & 1], ((j - 1) >> 1) & 1, &abort_flag)) alive = false;
                tc_fence_after();
#pragma unroll
                for (int c = 0; c < VC * 64; c += 32) {
                    float o[32];
                    tmem_ld32(my + kAeColO + tile * 128 + c, o);
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] *= alpha;
                    tmem_st32(my + kAeColO + tile * 128 + c, o);
                }
            }
            tmem_st32_u32(my + s_col, packed);
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&bar_p[tile][buf]);
        }
        if (mine > 0 && alive && !mbar_wait_all(&bar_o[tile], 0, &abort_flag)) alive = false;
        tc_fence_after();
        if (mine > 0 && __all_sync(0xffffffffu, alive)) {
            float g = l_run > 0.0f ? 1.0f / l_run : 0.0f;
            if (row_on && p.gate) g *= sigmoid_f(__bfloat162float(p.gate[(int64_t)tok * p.gate_stride + head]));
            __nv_bfloat16* dst = p.o + ((int64_t)tok * a.heads + head) * a.vdim_stride;
#pragma unroll
            for (int c = 0; c < VC * 64; c += 32) {
                float o[32];
                tmem_ld32(my + kAeColO + tile * 128 + c, o);
#pragma unroll
                for (int i = 0; i < 32; i += 8)
                    if (row_on && c + i < a.vdim_stride) {
                        float e[8];
#pragma unroll
                        for (int x = 0; x < 8; ++x) e[x] = o[i + x] * g;
                        Vec8<__nv_bfloat16>::store(dst + c + i, e);
                    }
                __syncwarp();
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (abort_flag && tid == 0) report(p.status, KTK_STATUS_TIMEOUT);
    if (issuer) {
        __syncwarp();
        tmem_free(tmem, kAeTmemCols);
    }
}

// The rows of one sequence out of their pages, in order: 16 bytes per thread.
__global__ void __launch_bounds__(256)
gather_rows_kernel(const uint4* __restrict__ pages, uint4* __restrict__ out, const ktk_paged t, int pieces, int total, int32_t* status) {
    const Span s = span_of(t, 0);
    if (s.bad || s.total < total) {
        if (threadIdx.x == 0) report(status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const int64_t n = (int64_t)total * pieces;
    for (int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (int64_t)gridDim.x * 256) {
        const int tok = (int)(i / pieces), c = (int)(i - (int64_t)tok * pieces);
        const int64_t page = t.kv_indices[s.start + tok / t.page_size];
        if (page < 0 || page >= t.num_pages) { report(status, KTK_STATUS_BAD_PAGE); continue; }
        out[i] = pages[(page * t.page_size + tok % t.page_size) * pieces + c];
    }
}

static int chunks_of(const ktk_latent& a) { return (a.dim_stride + 63) / 64 + (a.rot_stride + 63) / 64; }

template <int VC>
static int expanded_launch(const ExpandedParams& p, const __nv_bfloat16* kv, const __nv_bfloat16* rows, cudaStream_t st) {
    const char* who = "ktk_expanded_attention";
    const ktk_latent& a = p.a;
    const uint64_t H = a.heads, line = H * (a.dim_stride + a.vdim_stride) * 2, row = (uint64_t)(a.rank_stride + a.rot_stride) * 2;
    CUtensorMap km, rm, vm;
    const uint32_t box[3] = {64, 1, kAeKeys};
    // innermost first: columns of a head, heads, tokens
    const uint64_t kd[3] = {(uint64_t)a.dim_stride, H, (uint64_t)p.total}, ks[2] = {(uint64_t)a.dim_stride * 2, line};
    const uint64_t vd[3] = {(uint64_t)a.vdim_stride, H, (uint64_t)p.total}, vs[2] = {(uint64_t)a.vdim_stride * 2, line};
    const uint64_t rd[3] = {(uint64_t)a.rot_stride, 1, (uint64_t)p.total}, rs[2] = {row, row};
    int rc = make_tensor_map_3d(&km, kv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, kd, ks, box, CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc == KTK_OK)
        rc = make_tensor_map_3d(&vm, kv + H * a.dim_stride, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, vd, vs, box,
                                CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc == KTK_OK)
        rc = make_tensor_map_3d(&rm, rows + a.rank_stride, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rd, rs, box,
                                CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc != KTK_OK) return rc;
    const int dc = chunks_of(a), smem = 2 * dc * kAeQTile + 2 * dc * kAeKTile + 2 * VC * kAeKTile + 1024;
    auto kernel = attn_expanded_kernel<VC>;
    KTK_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), who);
    kernel<<<dim3((unsigned)((p.n + 2 * kUmRows - 1) / (2 * kUmRows)), (unsigned)H), kAeThreads, smem, st>>>(p, km, rm, vm);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}

static bool expanded_supported(const ktk_latent& a) {
    return a.dtype == KTK_BF16 && a.rot_stride > 0 && a.scale > 0.0f && chunks_of(a) <= kAeMaxChunks && a.vdim_stride <= 128 && a.heads <= 65535;
}

}  // namespace ktk

using namespace ktk;

extern "C" int ktk_expanded_attention_supported(const ktk_latent* shape) {
    return check_latent(shape, "ktk_expanded_attention_supported") == KTK_OK && expanded_supported(*shape) ? 1 : 0;
}

extern "C" int ktk_gather_rows(const void* pages, void* out, int64_t total, int32_t row_bytes, const ktk_paged* table,
                               int32_t* status, void* stream) {
    const char* who = "ktk_gather_rows";
    if (total < 0 || total > 2147483647LL || row_bytes <= 0 || row_bytes % 16 != 0 || table == nullptr || table->batch != 1 ||
        table->page_size <= 0 || (total > 0 && (!pages || !out || (((uintptr_t)pages | (uintptr_t)out) & 15u) != 0))) {
        set_error("%s: total=%lld row_bytes=%d", who, (long long)total, row_bytes);
        return KTK_ERR_ARG;
    }
    if (total == 0) return KTK_OK;
    const int pieces = row_bytes / 16;
    const int64_t blocks = (total * pieces + 255) / 256, cap = (int64_t)sm_count() * 16;
    gather_rows_kernel<<<(unsigned)(blocks < cap ? blocks : cap), 256, 0, (cudaStream_t)stream>>>(
        (const uint4*)pages, (uint4*)out, *table, pieces, (int)total, status);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}

extern "C" int ktk_expanded_attention(const void* q, int64_t q_stride, int64_t rows, int64_t total, const void* kv,
                                      const void* latents, const float* sink, const void* gate, int64_t gate_stride, void* o,
                                      const ktk_latent* shape, int32_t* status, void* stream) {
    const char* who = "ktk_expanded_attention";
    const int rc = check_latent(shape, who);
    if (rc != KTK_OK) return rc;
    if (!expanded_supported(*shape)) { set_error("%s: not built for these sizes", who); return KTK_ERR_UNSUPPORTED; }
    if (rows < 0 || total < rows || total > (1 << 30) || q_stride % 8 != 0 ||
        q_stride < (int64_t)shape->heads * (shape->dim_stride + shape->rot_stride) || (gate && gate_stride < shape->heads)) {
        set_error("%s: %lld rows of %lld, stride %lld", who, (long long)rows, (long long)total, (long long)q_stride);
        return KTK_ERR_ARG;
    }
    if (rows == 0) return KTK_OK;
    if (!q || !kv || !latents || !o || (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)latents | (uintptr_t)o) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    const ExpandedParams p{*shape, (const __nv_bfloat16*)q, q_stride, (int)rows, (int)total, sink, (const __nv_bfloat16*)gate,
                           gate_stride, (__nv_bfloat16*)o, status};
    return shape->vdim_stride <= 64 ? expanded_launch<1>(p, (const __nv_bfloat16*)kv, (const __nv_bfloat16*)latents, (cudaStream_t)stream)
                                    : expanded_launch<2>(p, (const __nv_bfloat16*)kv, (const __nv_bfloat16*)latents, (cudaStream_t)stream);
}
