// The experts' matrix products on the fifth-generation tensor cores, for prompts and for decode steps alike.
//
// The weights are the M operand and the routed rows the N operand: D[128 weight rows x N rows] += A[128 x 64] . B^T[64
// x N].  A work item is one tile of up to 256 rows of an expert and a block of 128 weight rows: stage 0 has the gate
// and the up row of an inner column side by side, so gating needs one exchange between neighbouring lanes.  N
// follows the tile's row count, and the ring's stages shrink with the rows a tile can have: a decode step with a few
// rows per expert keeps many weight tiles in flight and moves little else.  Persistent CTAs; the item list follows
// from the experts' row counts, which each CTA reads and scans itself.  Roles:
//     loading warp      weight tiles by TMA; stage 1 also the rows, which lie in place
//     gathering warps   stage 0: the bucket's rows of h, 16 bytes per cp.async, into the layout of the operand
//     issuing warp      4 x tcgen05.mma per ring stage, accumulators double-buffered in tensor memory (2 x 256 columns)
//     warps 0..3        epilogue of the previous item: tcgen05.ld, activation or routing weight, bf16 stores to the
//                       rows' places
// Full tiles (prompts) run on pairs of CTAs (cta_group::2): 256 weight rows x 256 routed rows per item, each CTA with its
// half of both in shared memory, which takes a third off the traffic from L2.  The second CTA's issuing warp tells the
// first one's when its part of a stage has landed.
// Every wait is bounded; a wait that runs out ends the CTA's roles, drains the copies in flight and frees tensor
// memory.
#include "../ktk_umma.cuh"
#include "ktl_common.cuh"

namespace ktk {

constexpr int kMuRows = 256;                       // most routed rows of a tile; of a CTA: half of that in a pair
constexpr int kMuK = 64;                           // columns per ring stage
constexpr int kMuMaxStages = 12;
constexpr int kMuABytes = kUmRows * kMuK * 2;      // 16 KiB
constexpr int kMuRing = 200 * 1024;                // bytes for the ring
constexpr int kMuTmemCols = 512;
constexpr int kMuGatherers = 128;                  // threads
constexpr int kMuBox = 32;                         // rows per TMA box of the rows in place

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, uint32_t bytes) {      // bytes 16, or 0: zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
// arrives on the barrier when all cp.async of this thread so far have landed (one of the barrier's expected arrivals)
__device__ __forceinline__ void cp_async_arrive(uint64_t* bar) {
    asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}

// Position in a ring of `stages` stages: advanced by one, without a division.
struct RingPos {
    int stage = 0;
    uint32_t round = 0;                                      // parity of a full barrier's next phase = round & 1
    __device__ __forceinline__ void next(int stages) {
        if (++stage == stages) { stage = 0; ++round; }
    }
};

// tile_rows: most rows of a tile; cta_rows: of them in a CTA's ring stage (half in a pair)
template <int STAGE, bool PAIR>
__global__ void __launch_bounds__(STAGE == 0 ? 320 : 192, 1)
moe_umma_kernel(const MoeParams p, const int tile_rows, const int cta_rows, const int stages,
                const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap in_map) {
    extern __shared__ uint8_t mu_raw[];
    __shared__ ExpertPlan plan;
    __shared__ __align__(8) uint64_t full[kMuMaxStages], empty[kMuMaxStages], peer_full[kMuMaxStages],
        acc_full[2], acc_free[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int abort_flag;
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(mu_raw) + 1023) & ~uintptr_t(1023));
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int N = STAGE == 0 ? 2 * p.m.ff_stride : p.m.width_stride;       // weight rows
    const int K = STAGE == 0 ? p.m.width_stride : p.m.ff_stride;
    const int steps = (K + kMuK - 1) / kMuK;
    constexpr int kCtas = PAIR ? 2 : 1;
    constexpr int kPer = kMuRows / kCtas / 16;               // gathered rows per thread
    const int rank = PAIR ? (int)cluster_rank() : 0;
    const int unit = blockIdx.x / kCtas, num_units = gridDim.x / kCtas;
    const int blocks = (N + kCtas * kUmRows - 1) / (kCtas * kUmRows);
    const int stage_bytes = kMuABytes + cta_rows * 128;

    if (tid == 0) {
        for (int s = 0; s < stages; ++s) {
            mbar_init(&full[s], STAGE == 0 ? 1 + kMuGatherers : 1);
            mbar_init(&empty[s], 1);
            mbar_init(&peer_full[s], 1);
        }
        for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_free[i], 4 * kCtas); }
        abort_flag = 0;
        mbar_init_fence();
    }
    if (warp == 0) plan_experts(plan, p.counts, p.m.experts, p.rows, tile_rows);
    if (warp == 4) {
        if (PAIR) tmem_alloc_pair(&tmem_base_s, kMuTmemCols);
        else tmem_alloc(&tmem_base_s, kMuTmemCols);
    }
    tc_fence_before();
    __syncthreads();
    if (PAIR) cluster_sync();                                // both CTAs' barriers are initialised
    tc_fence_after();
    const uint32_t tmem = tmem_base_s;
    const int work = plan.first_tile[p.m.experts] * blocks;

    // item w: expert, first row of the tile within the expert, rows; this CTA's part of the rows (m0, m); its first weight
    // row.  An expert's rows are shared out evenly over its tiles, in multiples of what a matrix instruction takes.
    constexpr int kStep = 16 * kCtas;
    struct Item { int e, r0, n, m0, m, wrow; };
    auto item = [&](int w) {
        Item it;
        const int t = w / blocks;
        it.wrow = ((w - t * blocks) * kCtas + rank) * kUmRows;
        it.e = expert_of_tile(plan, p.m.experts, t);
        const int rows = plan.first_row[it.e + 1] - plan.first_row[it.e];
        const int tiles = plan.first_tile[it.e + 1] - plan.first_tile[it.e];
        const int each = ((rows + tiles - 1) / tiles + kStep - 1) / kStep * kStep;
        it.r0 = (t - plan.first_tile[it.e]) * each;
        it.n = rows - it.r0 < each ? rows - it.r0 : each;
        const int half = (it.n + kStep - 1) / kStep * 16;    // a CTA's share
        it.m0 = rank * half;
        it.m = it.n - it.m0 < half ? (it.n > it.m0 ? it.n - it.m0 : 0) : half;
        return it;                                           // n <= 0 for a tile that the rounding left empty
    };

    if (warp == 5) {
        // ---------------- loads ----------------
        if (lane == 0) { prefetch_tensormap(&w_map); prefetch_tensormap(&in_map); }
        RingPos pos;
        int issued = 0;
        bool alive = true;
        for (int w = unit; w < work && alive; w += num_units) {
            const Item it = item(w);
            if (it.n <= 0) continue;
            const int boxes = STAGE == 0 ? 0 : (it.m + kMuBox - 1) / kMuBox;
            const uint32_t bytes = (uint32_t)(kMuABytes + boxes * kMuBox * 128);
            const int row = plan.first_row[it.e] + it.r0 + it.m0;
            for (int k = 0; k < steps; ++k, ++issued, pos.next(stages)) {
                const int s = pos.stage;
                bool ok = true;
                if (pos.round > 0) ok = mbar_wait_fast(&empty[s], (pos.round - 1) & 1, &abort_flag);
                if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
                uint8_t* st = ring + s * stage_bytes;
                if (elect_one()) {
                    mbar_arrive_expect_tx(&full[s], bytes);
                    tma_load_3d(st, &w_map, &full[s], k * kMuK, it.wrow, it.e);
                    for (int i = 0; i < boxes; ++i)
                        tma_load_3d(st + kMuABytes + i * kMuBox * 128, &in_map, &full[s], k * kMuK, row + i * kMuBox, 0);
                }
                __syncwarp();
            }
        }
        if (!alive && lane == 0) {                           // gave up: the copies in flight still write shared memory
            volatile int never = 0;
            for (int i = issued > stages ? issued - stages : 0; i < issued; ++i)
                mbar_wait(&full[i % stages], (i / stages) & 1, &never);
        }
    } else if (STAGE == 0 && warp >= 6) {
        // ---------------- gathered rows: thread t copies chunk t % 8 of rows t / 8, + 16, ... ----------------
        const int t = tid - 192, chunk = t & 7, row0 = t >> 3;
        const char* base = (const char*)p.in + chunk * 16;
        const uint32_t dst0 = smem_u32(ring) + kMuABytes + swz(row0, chunk);     // + i * 2048: row0 + 16 i
        RingPos pos;
        bool alive = true;
        int next[kPer];                                      // bucket entries of the next item, fetched one item ahead
        auto fetch = [&](int w) {
            Item it;
            it.n = it.m = 0;
            while (w < work && (it = item(w)).n <= 0) w += num_units;
#pragma unroll
            for (int i = 0; i < kPer; ++i) {
                const int r = row0 + 16 * i;
                next[i] = r < it.m ? p.bucket[(int64_t)it.e * p.rows + it.r0 + it.m0 + r] : -1;
            }
        };
        fetch(unit);
        for (int w = unit; w < work && alive; w += num_units) {
            const Item it = item(w);
            if (it.n <= 0) continue;
            uint32_t off[kPer];                              // 16-byte pieces from `base`; rows outside: zeros
            uint32_t bytes[kPer];
#pragma unroll
            for (int i = 0; i < kPer; ++i) {
                off[i] = 0u;
                bytes[i] = 0u;
                if (16 * i < it.m && next[i] >= 0) {
                    off[i] = (uint32_t)(next[i] / p.m.top) * (uint32_t)(K / 8);
                    bytes[i] = 16u;
                }
            }
            fetch(w + num_units);
            for (int k = 0; k < steps; ++k, pos.next(stages)) {
                const int s = pos.stage;
                bool ok = true;
                if (pos.round > 0) ok = mbar_wait_fast(&empty[s], (pos.round - 1) & 1, &abort_flag);
                if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
                const uint32_t dst = dst0 + s * stage_bytes;
                const bool in_row = k * kMuK + chunk * 8 < K;
                const char* from = in_row ? base + (int64_t)k * (kMuK * 2) : base;
                const uint32_t on = in_row ? 16u : 0u;
#pragma unroll
                for (int i = 0; i < kPer; ++i)
                    if (16 * i < it.m)                       // uniform
                        cp_async16(dst + i * 2048, from + (uint64_t)off[i] * 16, bytes[i] & on);
                cp_async_arrive(&full[s]);
            }
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
    } else if (warp == 4) {
        // ---------------- tensor cores ----------------
        RingPos pos;
        bool alive = true;
        auto landed = [&](uint64_t* bar) {
            return __all_sync(0xffffffffu, mbar_wait_fast(bar, pos.round & 1, &abort_flag)) != 0;
        };
        if (PAIR && rank == 1) {
            // the second CTA of a pair only reports what has landed
            for (int w = unit; w < work && alive; w += num_units) {
                if (item(w).n <= 0) continue;
                for (int k = 0; k < steps; ++k, pos.next(stages)) {
                    if (!landed(&full[pos.stage])) { alive = false; break; }
                    if (STAGE == 0) fence_proxy_async();
                    if (elect_one()) mbar_arrive_at(&peer_full[pos.stage], 0);
                    __syncwarp();
                }
            }
        } else {
            int j = 0;
            const uint64_t a0 = umma_desc(smem_u32(ring), 0, 1024), b0 = umma_desc(smem_u32(ring) + kMuABytes, 0, 1024);
            for (int w = unit; w < work && alive; w += num_units) {
                const Item it = item(w);
                if (it.n <= 0) continue;
                const int cols = (it.n + kStep - 1) / kStep * kStep;
                const uint32_t idesc = PAIR ? umma_idesc_pair(cols) : umma_idesc(cols, false);
                const int buf = j & 1;
                const uint32_t d = tmem + buf * 256;
                if (j >= 2 && !__all_sync(0xffffffffu, mbar_wait_fast(&acc_free[buf], ((j >> 1) - 1) & 1, &abort_flag)))
                    break;
                tc_fence_after();
                for (int k = 0; k < steps; ++k, pos.next(stages)) {
                    const int s = pos.stage;
                    if (!landed(&full[s]) || (PAIR && !landed(&peer_full[s]))) { alive = false; break; }
                    if (STAGE == 0) fence_proxy_async();     // the gathered rows came through the generic proxy
                    tc_fence_after();
                    const uint64_t a = umma_desc_at(a0, s * stage_bytes), b = umma_desc_at(b0, s * stage_bytes);
                    if (elect_one()) {
#pragma unroll
                        for (int q = 0; q < kMuK / 16; ++q) {
                            const uint32_t more = (k > 0 || q > 0) ? 1u : 0u;
                            if (PAIR) umma_f16_pair(d, umma_desc_at(a, q * 32), umma_desc_at(b, q * 32), idesc, more);
                            else umma_f16(d, umma_desc_at(a, q * 32), umma_desc_at(b, q * 32), idesc, more);
                        }
                        if (PAIR) umma_commit_pair(&empty[s]);
                        else umma_commit(&empty[s]);
                        if (k + 1 == steps) {
                            if (PAIR) umma_commit_pair(&acc_full[buf]);
                            else umma_commit(&acc_full[buf]);
                        }
                    }
                    __syncwarp();
                }
                ++j;
            }
        }
    } else if (warp < 4) {
        // ---------------- epilogue ----------------
        const uint32_t lanes = tmem + ((uint32_t)(warp * 32) << 16);
        __nv_bfloat16* out = (__nv_bfloat16*)p.out;
        const bool odd = lane & 1;
        int j = 0;
        for (int w = unit; w < work; w += num_units) {
            const Item it = item(w);
            if (it.n <= 0) continue;
            const int buf = j & 1;
            int entry[kMuRows / 32];
            float weight[kMuRows / 32];
            if (STAGE == 1) {                                // in flight while the tensor cores work on the item
#pragma unroll
                for (int c = 0; c < kMuRows / 32; ++c) {
                    const int r = c * 32 + lane;
                    entry[c] = r < it.n ? p.bucket[(int64_t)it.e * p.rows + it.r0 + r] : 0;
                }
#pragma unroll
                for (int c = 0; c < kMuRows / 32; ++c) weight[c] = c * 32 < it.n ? p.weights[entry[c]] : 0.0f;
            }
            const bool ok = mbar_wait_fast(&acc_full[buf], (j >> 1) & 1, &abort_flag);
            if (!__all_sync(0xffffffffu, ok)) break;
            tc_fence_after();
            const int wrow = it.wrow + warp * 32 + (lane & ~1);              // weight row of the even lane of the two
#pragma unroll
            for (int ch = 0; ch < kMuRows / 32; ++ch) {
                const int c0 = ch * 32;
                if (c0 >= it.n) break;                       // uniform for the CTA
                float v[32];
                tmem_ld32(lanes + buf * 256 + c0, v);
                // neighbouring lanes hold neighbouring weight rows: the even lane takes row i of the tile, the odd i + 1
#pragma unroll
                for (int i = 0; i < 32; i += 2) {
                    const float got = __shfl_xor_sync(0xffffffffu, odd ? v[i] : v[i + 1], 1);
                    const float first = odd ? got : v[i], second = odd ? v[i + 1] : got;
                    const int row = c0 + i + odd;
                    if (STAGE == 0) {                        // gate and up of inner column wrow / 2
                        const float act = gated<true>(first, second, p.m.limit, p.m.slope, p.m.shift);
                        if (row < it.n && wrow < N)
                            out[(int64_t)(plan.first_row[it.e] + it.r0 + row) * p.m.ff_stride + (wrow >> 1)] =
                                __float2bfloat16_rn(act);
                    } else {
                        const int64_t dst = __shfl_sync(0xffffffffu, entry[ch], i + odd);
                        const float f = __shfl_sync(0xffffffffu, weight[ch], i + odd);
                        if (row < it.n && wrow < N)
                            *reinterpret_cast<uint32_t*>(out + dst * N + wrow) = pack_bf16(first * f, second * f);
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
                if (PAIR) mbar_arrive_at(&acc_free[buf], 0);
                else mbar_arrive(&acc_free[buf]);
            }
            ++j;
        }
    }
    tc_fence_before();
    __syncthreads();
    if (PAIR) cluster_sync();                                // neither CTA leaves while the other may use its memory
    if (abort_flag && tid == 0) report(p.status, KTK_STATUS_TIMEOUT);
    if (warp == 4) {
        __syncwarp();
        if (PAIR) tmem_free_pair(tmem, kMuTmemCols);
        else tmem_free(tmem, kMuTmemCols);
    }
}

bool moe_umma_supported(const ktk_moe& m) { return m.dtype == KTK_BF16; }

template <int STAGE> static int moe_umma(const MoeParams& p, cudaStream_t st) {
    const char* who = "ktk_moe_gemm";
    const uint64_t N = STAGE == 0 ? 2 * p.m.ff_stride : p.m.width_stride;
    const uint64_t K = STAGE == 0 ? p.m.width_stride : p.m.ff_stride;
    const int64_t routed = p.rows * p.m.top;
    CUtensorMap w_map, in_map;
    const uint64_t wd[3] = {K, N, (uint64_t)p.m.experts}, ws[2] = {K * 2, K * N * 2};
    const uint32_t wb[3] = {kMuK, kUmRows, 1};
    int rc = make_tensor_map_3d(&w_map, p.w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, wd, ws, wb, CU_TENSOR_MAP_SWIZZLE_128B,
                                who);
    if (rc != KTK_OK) return rc;
    const uint64_t id[3] = {K, (uint64_t)(STAGE == 0 ? p.rows : routed), 1}, is[2] = {K * 2, K * id[1] * 2};
    const uint32_t ib[3] = {kMuK, kMuBox, 1};
    rc = make_tensor_map_3d(&in_map, p.in, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, id, is, ib, CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc != KTK_OK) return rc;
    // tiles for twice the rows that an expert has on average (and never more than all of them): the ring's stages are
    // no larger than they have to be
    int64_t most = 2 * ((routed + p.m.experts - 1) / p.m.experts);
    if (most > p.rows) most = p.rows;
    const int tile_rows = (int)(most >= kMuRows ? kMuRows : (most + kMuBox - 1) / kMuBox * kMuBox);
    const bool pair = tile_rows == kMuRows;
    const int cta_rows = pair ? tile_rows / 2 : tile_rows;
    const int stage_bytes = kMuABytes + cta_rows * 128;
    const int stages = kMuRing / stage_bytes < kMuMaxStages ? kMuRing / stage_bytes : kMuMaxStages;
    const int ctas = pair ? 2 : 1;
    const int64_t per = (N + ctas * kUmRows - 1) / (ctas * kUmRows);
    const int64_t tiles = routed / tile_rows + (routed < p.m.experts ? routed : p.m.experts);
    if (tiles * per > 2147483647LL || p.rows * (int64_t)(K / 8) > 4294967295LL) {
        set_error("%s: too many rows", who);
        return KTK_ERR_TOO_LARGE;
    }
    const int64_t units = tiles * per < sm_count() / ctas ? tiles * per : sm_count() / ctas;
    auto kernel = pair ? moe_umma_kernel<STAGE, true> : moe_umma_kernel<STAGE, false>;
    KTK_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMuRing + 1024), who);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3((unsigned)(units * ctas));
    cfg.blockDim = dim3(STAGE == 0 ? 320 : 192);
    cfg.dynamicSmemBytes = (size_t)stages * stage_bytes + 1024;
    cfg.stream = st;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeClusterDimension;
    attr.val.clusterDim.x = ctas;
    attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = pair ? 1 : 0;
    KTK_CUDA_TRY(cudaLaunchKernelEx(&cfg, kernel, p, tile_rows, cta_rows, stages, w_map, in_map), who);
    return KTK_OK;
}

int launch_moe_umma(int stage, const MoeParams& p, cudaStream_t st) {
    return stage == 0 ? moe_umma<0>(p, st) : moe_umma<1>(p, st);
}

}  // namespace ktk
