// The experts' matrix products on the fifth-generation tensor cores, for prompts and for decode steps alike.
//
// The weights are the M operand and the routed rows the N operand: D[128 weight rows x N rows] += A[128 x 64] . B^T[64
// x N].  A work item is one tile of up to 128 rows of an expert and two blocks of 128 weight rows (stage 0: the gate
// and the up rows of the same inner columns, so that silu(g) * u happens inside one thread; stage 1: two neighbouring
// blocks of output columns), i.e. two accumulators over a shared B.  N follows the tile's row count, so a decode step
// with a few rows per expert streams the weights and little else.  Persistent CTAs; the item list follows from the
// experts' row counts, which each CTA reads and scans itself.  Roles:
//     loading warp    lane 0: A tiles by TMA; every lane: four routed rows of B by TMA gather (box of one row), from
//                     the row numbers in the expert's bucket (stage 0) or in place (stage 1); ring of 4 x 48 KiB
//     issuing warp    8 x tcgen05.mma per ring stage, accumulators double-buffered in tensor memory (2 x 256 columns)
//     warps 0..3      epilogue of the previous item: tcgen05.ld, activation or routing weight, bf16 stores to the
//                     rows' places
// Every wait is bounded; a wait that runs out ends the CTA's roles, drains the copies in flight and frees tensor
// memory.
#include "../ktk_umma.cuh"
#include "ktl_common.cuh"

namespace ktk {

constexpr int kMuThreads = 192;
constexpr int kMuRows = 128;                       // routed rows of a tile
constexpr int kMuK = 64;                           // columns per ring stage
constexpr int kMuStages = 4;
constexpr int kMuABytes = kUmRows * kMuK * 2;      // 16 KiB
constexpr int kMuBBytes = kMuRows * kMuK * 2;      // 16 KiB
constexpr int kMuStageBytes = 2 * kMuABytes + kMuBBytes;
constexpr int kMuSmem = kMuStages * kMuStageBytes + 1024;
constexpr int kMuTmemCols = 512;

template <int STAGE>
__global__ void __launch_bounds__(kMuThreads, 1)
moe_umma_kernel(const MoeParams p, const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap in_map) {
    extern __shared__ uint8_t mu_raw[];
    __shared__ ExpertPlan plan;
    __shared__ __align__(8) uint64_t full[kMuStages], empty[kMuStages], acc_full[2], acc_free[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int abort_flag;
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(mu_raw) + 1023) & ~uintptr_t(1023));
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int N = STAGE == 0 ? p.m.ff_stride : p.m.width_stride, K = STAGE == 0 ? p.m.width_stride : p.m.ff_stride;
    const int steps = (K + kMuK - 1) / kMuK;
    const int blocks = STAGE == 0 ? (N + kUmRows - 1) / kUmRows : (N + 2 * kUmRows - 1) / (2 * kUmRows);

    if (tid == 0) {
        for (int s = 0; s < kMuStages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_free[i], 4); }
        abort_flag = 0;
        mbar_init_fence();
    }
    if (warp == 0) plan_experts(plan, p.counts, p.m.experts, p.rows, kMuRows);
    if (warp == 4) tmem_alloc(&tmem_base_s, kMuTmemCols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_base_s;
    const int work = plan.first_tile[p.m.experts] * blocks;

    // item w: expert, first row of the tile within the expert, rows, block of weight rows
    struct Item { int e, r0, n, mb; };
    auto item = [&](int w) {
        Item it;
        const int t = w / blocks;
        it.mb = w - t * blocks;
        it.e = expert_of_tile(plan, p.m.experts, t);
        it.r0 = (t - plan.first_tile[it.e]) * kMuRows;
        const int left = plan.first_row[it.e + 1] - plan.first_row[it.e] - it.r0;
        it.n = left < kMuRows ? left : kMuRows;
        return it;
    };

    if (warp == 5) {
        // ---------------- loads ----------------
        if (lane == 0) { prefetch_tensormap(&w_map); prefetch_tensormap(&in_map); }
        int issued = 0;
        bool alive = true;
        for (int w = blockIdx.x; w < work && alive; w += gridDim.x) {
            const Item it = item(w);
            const int groups = (it.n + 3) / 4;
            int rows[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                int r = lane * 4 + i;
                r = it.r0 + (r < it.n ? r : it.n - 1);       // past the tile: its last row once more
                rows[i] = STAGE == 0 ? p.bucket[(int64_t)it.e * p.rows + r] / p.m.top : plan.first_row[it.e] + r;
            }
            const uint32_t bytes = 2u * kMuABytes + (uint32_t)groups * 512u;
            for (int k = 0; k < steps; ++k, ++issued) {
                const int s = issued % kMuStages;
                bool ok = true;
                if (issued >= kMuStages) ok = mbar_wait_fast(&empty[s], ((issued / kMuStages) - 1) & 1, &abort_flag);
                if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
                uint8_t* st = ring + s * kMuStageBytes;
                if (lane == 0) {
                    mbar_arrive_expect_tx(&full[s], bytes);
                    if (STAGE == 0) {
                        tma_load_3d(st, &w_map, &full[s], k * kMuK, it.mb * kUmRows, 2 * it.e);
                        tma_load_3d(st + kMuABytes, &w_map, &full[s], k * kMuK, it.mb * kUmRows, 2 * it.e + 1);
                    } else {
                        tma_load_3d(st, &w_map, &full[s], k * kMuK, it.mb * 2 * kUmRows, it.e);
                        tma_load_3d(st + kMuABytes, &w_map, &full[s], k * kMuK, (it.mb * 2 + 1) * kUmRows, it.e);
                    }
                }
                __syncwarp();
                if (lane < groups) tma_gather4(st + 2 * kMuABytes + lane * 512, &in_map, &full[s], k * kMuK, rows);
            }
        }
        if (!alive && lane == 0) {                           // gave up: the copies in flight still write shared memory
            volatile int never = 0;
            for (int i = issued > kMuStages ? issued - kMuStages : 0; i < issued; ++i)
                mbar_wait(&full[i % kMuStages], (i / kMuStages) & 1, &never);
        }
    } else if (warp == 4) {
        // ---------------- tensor cores ----------------
        if (lane == 0) {
            int used = 0, j = 0;
            bool alive = true;
            for (int w = blockIdx.x; w < work && alive; w += gridDim.x, ++j) {
                const Item it = item(w);
                const uint32_t idesc = umma_idesc((it.n + 15) / 16 * 16, false);
                const int buf = j & 1;
                const uint32_t d = tmem + buf * 256;
                if (j >= 2 && !mbar_wait_fast(&acc_free[buf], ((j >> 1) - 1) & 1, &abort_flag)) break;
                tc_fence_after();
                for (int k = 0; k < steps; ++k, ++used) {
                    const int s = used % kMuStages;
                    if (!mbar_wait_fast(&full[s], (used / kMuStages) & 1, &abort_flag)) { alive = false; break; }
                    tc_fence_after();
                    const uint32_t a = smem_u32(ring + s * kMuStageBytes), b = a + 2 * kMuABytes;
#pragma unroll
                    for (int q = 0; q < kMuK / 16; ++q) {
                        const uint64_t bd = umma_desc(b + q * 32, 0, 1024);
                        umma_f16(d, umma_desc(a + q * 32, 0, 1024), bd, idesc, (k > 0 || q > 0) ? 1u : 0u);
                        umma_f16(d + 128, umma_desc(a + kMuABytes + q * 32, 0, 1024), bd, idesc,
                                 (k > 0 || q > 0) ? 1u : 0u);
                    }
                    umma_commit(&empty[s]);
                }
                if (alive) umma_commit(&acc_full[buf]);
            }
        }
    } else {
        // ---------------- epilogue ----------------
        const uint32_t lanes = tmem + ((uint32_t)(warp * 32) << 16);
        __nv_bfloat16* out = (__nv_bfloat16*)p.out;
        int j = 0;
        for (int w = blockIdx.x; w < work; w += gridDim.x, ++j) {
            const Item it = item(w);
            const int buf = j & 1;
            int entry[4];
            float weight[4];
            if (STAGE == 1) {
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const int r = c * 32 + lane;
                    entry[c] = r < it.n ? p.bucket[(int64_t)it.e * p.rows + it.r0 + r] : 0;
                    weight[c] = r < it.n ? p.weights[entry[c]] : 0.0f;
                }
            }
            const bool ok = mbar_wait_fast(&acc_full[buf], (j >> 1) & 1, &abort_flag);
            if (!__all_sync(0xffffffffu, ok)) break;
            tc_fence_after();
#pragma unroll
            for (int c0 = 0; c0 < kMuRows; c0 += 32) {
                if (c0 >= it.n) break;                       // uniform for the CTA
                float v[2][32];
                tmem_ld32(lanes + buf * 256 + c0, v[0]);
                tmem_ld32(lanes + buf * 256 + 128 + c0, v[1]);
                if (STAGE == 0) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[0][i] = __fdividef(v[0][i], 1.0f + __expf(-v[0][i])) * v[1][i];
                }
                // neighbouring lanes hold neighbouring output columns: even lanes store row i, odd lanes row i + 1
#pragma unroll
                for (int half = 0; half < (STAGE == 0 ? 1 : 2); ++half) {
                    const int col = STAGE == 0 ? it.mb * kUmRows + warp * 32 + (lane & ~1)
                                               : (it.mb * 2 + half) * kUmRows + warp * 32 + (lane & ~1);
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        const float give = (lane & 1) ? v[half][i] : v[half][i + 1];
                        const float got = __shfl_xor_sync(0xffffffffu, give, 1);
                        const int row = c0 + i + (lane & 1);
                        float lo = (lane & 1) ? got : v[half][i], hi = (lane & 1) ? v[half][i + 1] : got;
                        int64_t dst;
                        if (STAGE == 0) {
                            dst = plan.first_row[it.e] + it.r0 + row;
                        } else {
                            const int src = i + (lane & 1);
                            dst = __shfl_sync(0xffffffffu, entry[c0 / 32], src);
                            const float f = __shfl_sync(0xffffffffu, weight[c0 / 32], src);
                            lo *= f;
                            hi *= f;
                        }
                        if (row < it.n && col < N)
                            *reinterpret_cast<uint32_t*>(out + dst * N + col) = pack_bf16(lo, hi);
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_free[buf]);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (abort_flag && tid == 0) report(p.status, KTK_STATUS_TIMEOUT);
    if (warp == 4) {
        __syncwarp();
        tmem_free(tmem, kMuTmemCols);
    }
}

bool moe_umma_supported(const ktk_moe& m) { return m.dtype == KTK_BF16; }

template <int STAGE> static int moe_umma(const MoeParams& p, cudaStream_t st) {
    const char* who = "ktk_moe_gemm";
    const uint64_t N = STAGE == 0 ? p.m.ff_stride : p.m.width_stride, K = STAGE == 0 ? p.m.width_stride : p.m.ff_stride;
    CUtensorMap w_map, in_map;
    const uint64_t wd[3] = {K, N, (uint64_t)p.m.experts * (STAGE == 0 ? 2 : 1)}, ws[2] = {K * 2, K * N * 2};
    const uint32_t wb[3] = {kMuK, kUmRows, 1};
    int rc = make_tensor_map(&w_map, p.w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, wd, ws, wb, CU_TENSOR_MAP_SWIZZLE_128B,
                             who);
    if (rc != KTK_OK) return rc;
    const uint64_t id[2] = {K, (uint64_t)p.rows * (STAGE == 0 ? 1 : p.m.top)}, is[1] = {K * 2};
    const uint32_t ib[2] = {kMuK, 1};
    rc = make_tensor_map(&in_map, p.in, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, id, is, ib, CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc != KTK_OK) return rc;
    KTK_CUDA_TRY(cudaFuncSetAttribute(moe_umma_kernel<STAGE>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMuSmem), who);
    const int64_t per = STAGE == 0 ? (N + kUmRows - 1) / kUmRows : (N + 2 * kUmRows - 1) / (2 * kUmRows);
    const int64_t routed = p.rows * p.m.top;
    const int64_t tiles = routed / kMuRows + (routed < p.m.experts ? routed : p.m.experts);
    if (tiles * per > 2147483647LL) { set_error("%s: too many rows", who); return KTK_ERR_TOO_LARGE; }
    const int64_t grid = tiles * per < sm_count() ? tiles * per : sm_count();
    moe_umma_kernel<STAGE><<<(unsigned)grid, kMuThreads, kMuSmem, st>>>(p, w_map, in_map);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}

int launch_moe_umma(int stage, const MoeParams& p, cudaStream_t st) {
    return stage == 0 ? moe_umma<0>(p, st) : moe_umma<1>(p, st);
}

}  // namespace ktk
