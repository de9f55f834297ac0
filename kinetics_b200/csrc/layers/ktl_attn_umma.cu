// Causal attention of a prompt's tokens on the fifth-generation tensor cores: two softmax maps per head over shared
// values, head sizes up to 128, softcap, query temperature; the difference of the maps and its unit norm in the
// epilogue.  bf16 operands, fp32 scores and sums.
//
// One CTA per (sequence, kv head, tile of 128 (token, head of the group) rows).  A row exists once per map: softmax
// warps 0..3 hold map 1, warps 4..7 map 2, thread r of each the tile's row r = lane r of tensor memory.  The history
// is walked in blocks of 64 keys.  Roles:
//     loading warp (one lane)   TMA: both maps' K and the shared V of a block -> shared memory, two blocks in flight
//     issuing warp (one lane)   S_m[128 x 64] = Q_m . K_m^T, then O_m[128 x vdim] += P_m . V with P_m from tensor
//                               memory; S of block j + 1 is issued before O += P.V of block j
//     softmax thread            S row -> registers; scale, softcap, mask, 2^x; P as bf16 pairs over that S
// With a softcap the exponentials have a fixed reference (ktl_score.cuh): nothing is ever rescaled.  Without one (or
// with a large one) the reference follows the running maximum in jumps, and O rows are rescaled when it moves.
// Tensor memory: S of two blocks and two maps in columns [0, 256), O_1 and O_2 behind.  Every wait is bounded.
#include "ktl_score.cuh"

namespace ktk {

constexpr int kAuKeys = 64;
constexpr int kAuThreads = 320;          // 8 softmax warps, the issuing warp, the loading warp
constexpr int kAuTmemCols = 512;
constexpr int kAuColO = 256;
constexpr int kAuQTile = kUmRows * 128;  // [128 rows][64 dims]
constexpr int kAuKTile = kAuKeys * 128;  // [64 keys][64 columns]
constexpr uint32_t kAuVLbo = kAuKTile, kAuVSbo = 1024;    // V read MN-major: distance of two 64-column tiles, of 8 rows

template <int DC, int VC> constexpr int au_smem() { return 2 * DC * kAuQTile + 2 * (2 * DC + VC) * kAuKTile + 1024; }

__device__ __forceinline__ void st_row16(__nv_bfloat16* d, const float* o, float f) {
    uint4 v;
    v.x = pack_bf16(o[0] * f, o[1] * f);
    v.y = pack_bf16(o[2] * f, o[3] * f);
    v.z = pack_bf16(o[4] * f, o[5] * f);
    v.w = pack_bf16(o[6] * f, o[7] * f);
    *reinterpret_cast<uint4*>(d) = v;
}

template <int DC, int VC, bool FIXED>
__global__ void __launch_bounds__(kAuThreads, 1)
attn_umma_kernel(const AttnParams p, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map) {
    extern __shared__ uint8_t au_raw[];
    // S complete (map, buffer) | P in place (map, buffer) | K, V landed (buffer) | K, V read out (buffer)
    __shared__ __align__(8) uint64_t bar_s[2][2], bar_p[2][2], bar_k[2], bar_v[2], bar_kfree[2], bar_vfree[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int abort_flag;
    __shared__ float row_l[2][kUmRows], row_ss[2][kUmRows];
    uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(au_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sQ = sm;                                  // [map][chunk]
    uint8_t* sK = sQ + 2 * DC * kAuQTile;              // [buffer][map][chunk]
    uint8_t* sV = sK + 2 * 2 * DC * kAuKTile;          // [buffer][chunk]
    constexpr int kKBuf = 2 * DC * kAuKTile, kVBuf = VC * kAuKTile;

    const ktk_attn& a = p.a;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool issuer = warp == 8, loader = warp == 9;
    const int b = blockIdx.z, kvh = blockIdx.y;
    const int group = a.heads / a.kv_heads, tpc = kUmRows / group;
    const int q0 = p.new_indptr[b], n_new = p.new_indptr[b + 1] - q0;
    const int tok0 = (int)(gridDim.x - 1 - blockIdx.x) * tpc;      // the tiles with the longest history first
    if (tok0 >= n_new) return;                          // uniform for the CTA: nothing allocated yet
    const Span s = span_of(p.t, b);
    const int base_pos = s.total - n_new;
    if (s.bad || base_pos < 0) {
        if (tid == 0) report(p.status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const int tok_hi = (tok0 + tpc < n_new ? tok0 + tpc : n_new) - 1;
    const int seen = base_pos + tok_hi + 1;             // keys the tile's last row sees
    const int n_blocks = (seen + kAuKeys - 1) / kAuKeys;
    const int ps = p.t.page_size;

    const int map = warp >> 2, row = tid & (kUmRows - 1);
    const int my_tok = tok0 + row / group, my_head = kvh * group + row % group;
    const bool row_on = warp < 8 && row / group < tpc && my_tok < n_new;
    const int vis = row_on ? base_pos + my_tok + 1 : 0; // keys at positions < vis are seen

    if (tid == 0) {
        for (int i = 0; i < 2; ++i) {
            for (int m = 0; m < 2; ++m) { mbar_init(&bar_s[m][i], 1); mbar_init(&bar_p[m][i], kUmRows); }
            mbar_init(&bar_k[i], 1); mbar_init(&bar_v[i], 1);
            mbar_init(&bar_kfree[i], 1); mbar_init(&bar_vfree[i], 1);
        }
        abort_flag = 0;
        mbar_init_fence();
    }
    if (warp < 8) {
        const uint4* src = reinterpret_cast<const uint4*>(
            (const __nv_bfloat16*)p.q + (int64_t)(q0 + (row_on ? my_tok : 0)) * p.q_stride +
            ((int64_t)(row_on ? my_head : 0) * 2 + map) * a.dim_stride);
        uint8_t* dst = sQ + map * DC * kAuQTile;
#pragma unroll
        for (int c = 0; c < DC * 8; ++c) {
            const uint4 v = row_on && c * 8 < a.dim_stride ? __ldg(src + c) : make_uint4(0u, 0u, 0u, 0u);
            *reinterpret_cast<uint4*>(dst + (c >> 3) * kAuQTile + swz(row, c & 7)) = v;
        }
        fence_proxy_async();
    } else if (issuer) {
        tmem_alloc(&tmem_base_s, kAuTmemCols);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_base_s;

    if (issuer) {
        const int ksteps = (a.dim_stride + 15) / 16;
        const uint32_t idesc_s = umma_idesc(kAuKeys, false);
        const uint32_t idesc_o = umma_idesc((a.vdim_stride + 15) / 16 * 16, true);
        const uint64_t q_desc = umma_desc(smem_u32(sQ), 0, 1024), k_desc = umma_desc(smem_u32(sK), 0, 1024);
        const uint64_t v_desc = umma_desc(smem_u32(sV), kAuVLbo, kAuVSbo);
        auto wait = [&](uint64_t* bar, int round) {
            return __all_sync(0xffffffffu, mbar_wait_fast(bar, round & 1, &abort_flag)) != 0;
        };
        auto issue_s = [&](int blk) {
            const int buf = blk & 1;
            if (!wait(&bar_k[buf], blk >> 1)) return false;
            tc_fence_after();
            if (elect_one()) {
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    const uint64_t qa = umma_desc_at(q_desc, m * DC * kAuQTile);
                    const uint64_t ka = umma_desc_at(k_desc, buf * kKBuf + m * DC * kAuKTile);
#pragma unroll
                    for (int k = 0; k < DC * 4; ++k)
                        if (k < ksteps)
                            umma_f16(tmem + m * 128 + buf * kAuKeys, umma_desc_at(qa, (k >> 2) * kAuQTile + (k & 3) * 32),
                                     umma_desc_at(ka, (k >> 2) * kAuKTile + (k & 3) * 32), idesc_s, k > 0 ? 1u : 0u);
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
                ok = ok && wait(&bar_p[m][buf], j >> 1);
                if (!ok) break;
                tc_fence_after();
                if (elect_one()) {
#pragma unroll
                    for (int k = 0; k < kAuKeys / 16; ++k)
                        umma_f16_ts(tmem + kAuColO + m * 128, tmem + m * 128 + buf * kAuKeys + k * 8,
                                    umma_desc_at(va, k * (16 * 128)), idesc_o, (j > 0 || k > 0) ? 1u : 0u);
                    if (m == 1) umma_commit(&bar_vfree[buf]);
                }
                __syncwarp();
            }
        }
    } else if (loader) {
        if (lane == 0) {
            const int rows = ps < kAuKeys ? ps : kAuKeys;        // rows of a box: a page, or a block of it
            const int pages = kAuKeys / rows;
            // K (which = 0) or V (which = 1) of block `blk`; returns false if the wait for its buffer ran out
            auto load = [&](int blk, int which) {
                const int buf = blk & 1;
                uint64_t* bar = which ? &bar_v[buf] : &bar_k[buf];
                int64_t z[kAuKeys / 16];                              // pages
                uint32_t bytes = 0;
#pragma unroll
                for (int i = 0; i < kAuKeys / 16; ++i) {
                    z[i] = -1;
                    const int tok = blk * kAuKeys + i * rows;
                    if (i < pages && tok < seen) {
                        const int64_t pg = p.t.kv_indices[s.start + tok / ps];
                        if (pg < 0 || pg >= p.t.num_pages) report(p.status, KTK_STATUS_BAD_PAGE);
                        else { z[i] = pg; bytes += (uint32_t)((which ? VC : 2 * DC) * rows * 128); }
                    }
                }
                if (bytes) mbar_arrive_expect_tx(bar, bytes);
                else mbar_arrive(bar);
#pragma unroll
                for (int i = 0; i < kAuKeys / 16; ++i) {
                    if (z[i] < 0) continue;
                    if (which) {
#pragma unroll
                        for (int c = 0; c < VC; ++c)
                            tma_load_3d(sV + buf * kVBuf + c * kAuKTile + i * rows * 128, &v_map, bar, c * 64, 0,
                                        (int)(z[i] * a.kv_heads) + kvh);
                    } else {
#pragma unroll
                        for (int mc = 0; mc < 2 * DC; ++mc)
                            tma_load_3d(sK + buf * kKBuf + mc * kAuKTile + i * rows * 128, &k_map, bar, (mc % DC) * 64, 0,
                                        (int)(z[i] * (2 * a.kv_heads)) + kvh * 2 + mc / DC);
                    }
                }
            };
            prefetch_tensormap(&k_map);
            prefetch_tensormap(&v_map);
            load(0, 0);
            load(0, 1);
            if (n_blocks > 1) load(1, 0);
            for (int j = 0; j < n_blocks; ++j) {
                if (j + 1 < n_blocks) {                          // V of block j + 1 over that of block j - 1
                    if (j > 0 && !mbar_wait_fast(&bar_vfree[(j + 1) & 1], ((j - 1) >> 1) & 1, &abort_flag)) break;
                    load(j + 1, 1);
                }
                if (j + 2 < n_blocks) {                          // K of block j + 2 over that of block j
                    if (!mbar_wait_fast(&bar_kfree[j & 1], (j >> 1) & 1, &abort_flag)) break;
                    load(j + 2, 0);
                }
            }
        }
    } else {
        const uint32_t my = tmem + ((uint32_t)((warp & 3) * 32) << 16);
        const float factor = a.scale * query_temperature(a.temp_coef, a.temp_every, vis > 0 ? vis - 1 : 0);
        const bool capped = FIXED || a.softcap > 0.0f;
        const float plain = factor * kLog2eF;
        CapPoly poly;
        CapCoef exact;
        poly.set(factor, capped ? a.softcap : 1.0f);
        exact.set(factor, capped ? a.softcap : 1.0f);
        float m_run = -INFINITY, m_ref = 0.0f, l_run = 0.0f;
        const int tile_min_vis = base_pos + tok0 + 1;
        bool alive = true;
        for (int j = 0; j < n_blocks; ++j) {
            const int buf = j & 1;
            const uint32_t s_col = map * 128 + buf * kAuKeys;
            const bool clean = (j + 1) * kAuKeys <= tile_min_vis && row_on;   // every row of the tile sees the block
            const bool ok = mbar_wait_fast(&bar_s[map][buf], (j >> 1) & 1, &abort_flag);
            if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
            tc_fence_after();
            float lo[32], hi[32];
            tmem_ld64(my + s_col, lo, hi);
            if (capped) {
                float mx = 0.0f;
#pragma unroll
                for (int c = 0; c < 32; ++c) mx = fmaxf(mx, fmaxf(fabsf(lo[c]), fabsf(hi[c])));
                // rows without a token and keys behind a row's own hold stale numbers: they decide the branch at most
                if (__any_sync(0xffffffffu, !(mx <= poly.limit))) {
#pragma unroll
                    for (int c = 0; c < 32; ++c) { lo[c] = exact(lo[c]); hi[c] = exact(hi[c]); }
                } else {
#pragma unroll
                    for (int c = 0; c < 32; c += 2) { poly.two(lo[c], lo[c + 1]); poly.two(hi[c], hi[c + 1]); }
                }
            } else {
#pragma unroll
                for (int c = 0; c < 32; ++c) { lo[c] *= plain; hi[c] *= plain; }
            }
            if (!clean) {
                const int first = j * kAuKeys;
#pragma unroll
                for (int c = 0; c < 32; ++c) {
                    lo[c] = first + c < vis ? lo[c] : -INFINITY;
                    hi[c] = first + 32 + c < vis ? hi[c] : -INFINITY;
                }
            }
            float alpha = 1.0f;
            if (!FIXED) {
                float mx = m_run;
#pragma unroll
                for (int c = 0; c < 32; ++c) mx = fmaxf(mx, fmaxf(lo[c], hi[c]));
                float use = m_ref;
                if (mx == -INFINITY) use = 0.0f;                       // a row that has seen nothing yet
                else if (m_run == -INFINITY || mx - m_ref > 8.0f) use = mx;
                alpha = m_run == -INFINITY ? 0.0f : ex2(m_ref - use);
                m_ref = use;
                m_run = mx;
            }
            uint32_t packed[32];
            float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
            for (int c = 0; c < 16; ++c) {
                const float p0 = ex2(lo[2 * c] - m_ref), p1 = ex2(lo[2 * c + 1] - m_ref);
                const float p2 = ex2(hi[2 * c] - m_ref), p3 = ex2(hi[2 * c + 1] - m_ref);
                sum0 += p0 + p1;
                sum1 += p2 + p3;
                packed[c] = pack_bf16(p0, p1);
                packed[16 + c] = pack_bf16(p2, p3);
            }
            l_run = FIXED ? l_run + (sum0 + sum1) : l_run * alpha + (sum0 + sum1);
            if (!FIXED && j > 0 && __any_sync(0xffffffffu, alpha != 1.0f)) {
                if (!mbar_wait_fast(&bar_vfree[(j - 1) & 1], ((j - 1) >> 1) & 1, &abort_flag)) alive = false;
                tc_fence_after();
#pragma unroll
                for (int c = 0; c < VC * 64; c += 32) {
                    float o[32];
                    tmem_ld32(my + kAuColO + map * 128 + c, o);
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] *= alpha;
                    tmem_st32(my + kAuColO + map * 128 + c, o);
                }
            }
            tmem_st32_u32(my + s_col, packed);
            tmem_st_wait();
            if (map == 0 && (j + 1) * kAuKeys > seen) {        // the last block: rows of V without a key are cleared
                if (tid < kAuKeys && j * kAuKeys + tid >= seen) {
                    if (!mbar_wait_fast(&bar_v[buf], (j >> 1) & 1, &abort_flag)) alive = false;
#pragma unroll
                    for (int c = 0; c < VC * 8; ++c)
                        *reinterpret_cast<uint4*>(sV + buf * kVBuf + (c >> 3) * kAuKTile + swz(tid, c & 7)) =
                            make_uint4(0u, 0u, 0u, 0u);
                }
                fence_proxy_async();
            }
            tc_fence_before();
            mbar_arrive(&bar_p[map][buf]);
        }
        if (alive && !mbar_wait_fast(&bar_vfree[(n_blocks - 1) & 1], ((n_blocks - 1) >> 1) & 1, &abort_flag)) alive = false;
        tc_fence_after();
        // ---- o = O_1 / l_1 - lambda O_2 / l_2, unit norm: warps 0..3 the first half of the columns, 4..7 the second
        row_l[map][row] = l_run;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        constexpr int kHalf = VC * 32;
        const float i1 = row_l[0][row] > 0.0f ? 1.0f / row_l[0][row] : 0.0f;
        const float i2 = row_l[1][row] > 0.0f ? a.lambda / row_l[1][row] : 0.0f;
        float o[kHalf], ss = 0.0f;
        if (!abort_flag) {
#pragma unroll
            for (int c = 0; c < kHalf; c += 32) {
                float t1[32], t2[32];
                tmem_ld32(my + kAuColO + map * kHalf + c, t1);
                tmem_ld32(my + kAuColO + 128 + map * kHalf + c, t2);
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    o[c + i] = map * kHalf + c + i < a.vdim ? t1[i] * i1 - t2[i] * i2 : 0.0f;
                    ss += o[c + i] * o[c + i];
                }
            }
        }
        row_ss[map][row] = ss;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (row_on && !abort_flag) {
            const float f = a.out_scale / sqrtf((row_ss[0][row] + row_ss[1][row]) / (float)a.vdim + a.eps);
            __nv_bfloat16* dst = (__nv_bfloat16*)p.o + ((int64_t)(q0 + my_tok) * a.heads + my_head) * a.vdim_stride;
#pragma unroll
            for (int c = 0; c < kHalf; c += 8)
                if (map * kHalf + c < a.vdim_stride) st_row16(dst + map * kHalf + c, o + c, f);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (abort_flag && tid == 0) report(p.status, KTK_STATUS_TIMEOUT);
    if (issuer) {
        __syncwarp();
        tmem_free(tmem, kAuTmemCols);
    }
}

bool attn_umma_supported(const ktk_attn& a) {
    return a.dtype == KTK_BF16 && a.maps == 2 && a.dim_stride <= 128 && a.vdim_stride <= 128 &&
           a.heads / a.kv_heads <= kUmRows;
}

template <int DC, int VC, bool FIXED> static int umma_launch(const AttnParams& p, cudaStream_t st) {
    const char* who = "ktk_paged_attention";
    CUtensorMap km, vm;
    const int rc = make_cache_maps(p, &km, &vm, (uint32_t)(p.t.page_size < kAuKeys ? p.t.page_size : kAuKeys), who);
    if (rc != KTK_OK) return rc;
    constexpr int smem = au_smem<DC, VC>();
    auto kernel = attn_umma_kernel<DC, VC, FIXED>;
    KTK_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), who);
    const int tpc = kUmRows / (p.a.heads / p.a.kv_heads);
    const dim3 grid((unsigned)((p.max_new + tpc - 1) / tpc), (unsigned)p.a.kv_heads, (unsigned)p.t.batch);
    kernel<<<grid, kAuThreads, smem, st>>>(p, km, vm);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}

int launch_attn_umma(const AttnParams& p, cudaStream_t st) {
    if (p.max_new <= 0) return KTK_OK;
    if (p.t.batch > 65535 || p.a.kv_heads > 65535) {
        set_error("ktk_paged_attention: more than 65535 sequences or kv heads in one launch");
        return KTK_ERR_TOO_LARGE;
    }
    const bool d1 = p.a.dim_stride <= 64, v1 = p.a.vdim_stride <= 64, fx = fixed_reference(p.a);
    if (d1 && v1) return fx ? umma_launch<1, 1, true>(p, st) : umma_launch<1, 1, false>(p, st);
    if (d1) return fx ? umma_launch<1, 2, true>(p, st) : umma_launch<1, 2, false>(p, st);
    return fx ? umma_launch<2, 2, true>(p, st) : umma_launch<2, 2, false>(p, st);
}

}  // namespace ktk
