// Router of a mixture of experts: fp32 logits of every row against every expert, the best `top` of them, the softmax
// over those, and each row's place in its experts' buckets -- one launch.
//
// Many rows of bf16: tiles on the tensor cores; few rows, and fp32: a CTA per row with FMA.  Then a warp per row picks the
// experts.
#include "../ktk_pipeline.cuh"
#include "ktl_common.cuh"

namespace ktk {

constexpr int kRtThreads = 256;
constexpr int kRtWarps = kRtThreads / 32;
constexpr int kRtRows = 32;          // rows of a CTA, tensor-core variant
constexpr int kRtCols = 64;          // experts per pass
constexpr int kRtByRow = 256;        // up to this many rows: a CTA per row
constexpr int kRtRowThreads = 512;
static_assert(kMaxExperts * 2 * 4 <= 4 * (kRtRows + kRtCols) * 72 * 2, "the expert counters fit the ring");

struct RouteParams {
    ktk_moe m;
    const void *h, *w;
    const float* b;
    int32_t* ids;
    float* weights;
    int32_t* counts;
    int32_t* bucket;
    int64_t rows;
};

// One warp: the `top` largest of z[0 .. experts) (ties to the lower index), weighted by the softmax over them or over all.
// z is overwritten.
// ids_s [top], shared memory of the warp: the choice, for the caller.
__device__ __forceinline__ void pick_experts(const RouteParams& p, float* z, int64_t row, int32_t* ids_s) {
    const int lane = threadIdx.x & 31;
    const int E = p.m.experts, top = p.m.top;
    float best0 = 0.0f, denom = 0.0f, denom_all = 0.0f;
    if (p.m.scoring == 1) {
        float mx = -INFINITY;
        for (int i = lane; i < E; i += 32) mx = fmaxf(mx, z[i]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        for (int i = lane; i < E; i += 32) denom_all += expf(z[i] - mx);
        denom_all = warp_sum_f(denom_all);
    }
    for (int j = 0; j < top; ++j) {
        uint32_t key = 0;
        int e = E - 1;
        for (int i = lane; i < E; i += 32) {
            const uint32_t k = score_to_key(z[i]);
            if (k > key) { key = k; e = i; }
        }
        const uint32_t best = __reduce_max_sync(0xffffffffu, key);
        e = (int)__reduce_min_sync(0xffffffffu, key == best ? (uint32_t)e : 0x7fffffffu);
        const float v = z[e];
        if (j == 0) best0 = v;
        const float ex = expf(v - best0);
        denom += ex;
        __syncwarp();
        if (lane == 0) {
            z[e] = -INFINITY;
            ids_s[j] = e;
            p.ids[row * top + j] = e;
            p.weights[row * top + j] = ex;
        }
        __syncwarp();
    }
    if (p.m.scoring == 1) denom = denom_all;
    for (int j = lane; j < top; j += 32) p.weights[row * top + j] /= denom;
}

// One CTA per row: warp w takes experts w, w + 16, ..., two at a time; lanes share the width, 8 elements per load and up
// to 16 loads in flight.  For fp32 and for the few rows of a decode step (the weights stay in L2).
template <typename T>
__global__ void __launch_bounds__(kRtRowThreads) route_row_kernel(const RouteParams p) {
    extern __shared__ float rt_z[];                       // [experts] | the row [width_stride] | ids [top]
    constexpr int kWarps = kRtRowThreads / 32, kUnroll = 8;
    const int64_t row = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int K = p.m.width_stride, E = p.m.experts, top = p.m.top;
    float* hs = rt_z + (E + 3) / 4 * 4;
    int32_t* ids_s = reinterpret_cast<int32_t*>(hs + K);
    for (int i = threadIdx.x * 8; i < K; i += kRtRowThreads * 8) {
        float v[8];
        load8((const T*)p.h + row * K + i, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) hs[i + e] = v[e];
    }
    __syncthreads();
    for (int e0 = warp; e0 < E; e0 += 2 * kWarps) {
        const int e1 = e0 + kWarps < E ? e0 + kWarps : e0;
        const T* w0 = (const T*)p.w + (int64_t)e0 * K;
        const T* w1 = (const T*)p.w + (int64_t)e1 * K;
        float s0 = 0.0f, s1 = 0.0f;
        for (int i0 = lane * 8; i0 < K; i0 += 256 * kUnroll) {
#pragma unroll
            for (int u = 0; u < kUnroll; ++u) {
                const int i = i0 + u * 256;
                if (i < K) {
                    float hv[8], a[8], b[8];
                    load8(w0 + i, a);
                    load8(w1 + i, b);
                    Vec8<float>::load(hs + i, hv);
#pragma unroll
                    for (int x = 0; x < 8; ++x) { s0 = fmaf(hv[x], a[x], s0); s1 = fmaf(hv[x], b[x], s1); }
                }
            }
        }
        s0 = warp_sum_f(s0);
        s1 = warp_sum_f(s1);
        if (lane == 0) {
            rt_z[e0] = p.b ? s0 + p.b[e0] : s0;
            if (e1 != e0) rt_z[e1] = p.b ? s1 + p.b[e1] : s1;
        }
    }
    __syncthreads();
    if (warp == 0) {
        pick_experts(p, rt_z, row, ids_s);
        for (int j = lane; j < top; j += 32) {
            const int e = ids_s[j], at = atomicAdd(p.counts + e, 1);
            if (at < p.rows) p.bucket[(int64_t)e * p.rows + at] = (int32_t)(row * top + j);
        }
    }
}

// A CTA takes 32 rows.  Columns 64 at a time: h [32 x 64] and W [64 experts x 64] through a ring of cp.async stages; warp
// w accumulates experts 8 w .. 8 w + 7 of the pass for all 32 rows with mma.m16n8k16 (exact products, fp32 sums).
constexpr int kRtK = 64, kRtStages = 4, kRtLd = kRtK + 8;        // padded rows: no bank conflicts
constexpr int kRtStageElems = (kRtRows + kRtCols) * kRtLd;

__global__ void __launch_bounds__(kRtThreads) route_mma_kernel(const RouteParams p) {
    extern __shared__ __align__(16) uint8_t rt_raw[];     // ring | logits [32][experts padded to 64] | ids, places [32][top]
    __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(rt_raw);
    float* rt_z = reinterpret_cast<float*>(rt_raw + kRtStages * kRtStageElems * 2);
    int32_t* ids_s = reinterpret_cast<int32_t*>(rt_z + kRtRows * ((p.m.experts + kRtCols - 1) / kRtCols * kRtCols));
    int32_t* place_s = ids_s + kRtRows * p.m.top;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int gid = lane >> 2, tig = lane & 3;
    const int E = p.m.experts, ld = (E + kRtCols - 1) / kRtCols * kRtCols;
    const int64_t row0 = (int64_t)blockIdx.x * kRtRows;
    const int K = p.m.width_stride, steps = (K + kRtK - 1) / kRtK;
    const __nv_bfloat16* hp = (const __nv_bfloat16*)p.h;
    const __nv_bfloat16* wp = (const __nv_bfloat16*)p.w;
    for (int c0 = 0; c0 < E; c0 += kRtCols) {
        auto load = [&](int s) {
            __nv_bfloat16* st = ring + (s % kRtStages) * kRtStageElems;
            for (int i = tid; i < (kRtRows + kRtCols) * (kRtK / 8); i += kRtThreads) {
                const int r = i / (kRtK / 8), c = i % (kRtK / 8) * 8, k = s * kRtK + c;
                const bool is_h = r < kRtRows;
                const int64_t src_row = is_h ? row0 + r : c0 + r - kRtRows;
                const bool on = k < K && src_row < (is_h ? p.rows : (int64_t)E);
                const __nv_bfloat16* src = (is_h ? hp : wp) + (on ? src_row * K + k : 0);
                const uint32_t bytes = on ? 16u : 0u;
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(st + r * kRtLd + c)), "l"(src),
                             "r"(bytes) : "memory");
            }
        };
        float acc[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][e] = 0.0f;
        for (int s = 0; s < kRtStages - 1; ++s) {
            if (s < steps) load(s);
            asm volatile("cp.async.commit_group;" ::: "memory");
        }
        for (int s = 0; s < steps; ++s) {
            asm volatile("cp.async.wait_group %0;" ::"n"(kRtStages - 2) : "memory");
            __syncthreads();                              // stage s is in place; everyone is done with stage s - 1
            if (s + kRtStages - 1 < steps) load(s + kRtStages - 1);
            asm volatile("cp.async.commit_group;" ::: "memory");
            const __nv_bfloat16* st = ring + (s % kRtStages) * kRtStageElems;
            const __nv_bfloat16* w = st + (kRtRows + warp * 8 + gid) * kRtLd + 2 * tig;
#pragma unroll
            for (int k = 0; k < kRtK; k += 16) {
                const uint32_t b0 = *reinterpret_cast<const uint32_t*>(w + k), b1 = *reinterpret_cast<const uint32_t*>(w + k + 8);
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const __nv_bfloat16* h = st + (16 * i + gid) * kRtLd + 2 * tig + k;
                    uint32_t a[4];
                    a[0] = *reinterpret_cast<const uint32_t*>(h);
                    a[1] = *reinterpret_cast<const uint32_t*>(h + 8 * kRtLd);
                    a[2] = *reinterpret_cast<const uint32_t*>(h + 8);
                    a[3] = *reinterpret_cast<const uint32_t*>(h + 8 * kRtLd + 8);
                    mma_bf16(acc[i], a, b0, b1);
                }
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        const int e = c0 + warp * 8 + 2 * tig;
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int col = e + (x & 1);
                rt_z[(16 * i + gid + (x >= 2 ? 8 : 0)) * ld + col] = acc[i][x] + (p.b && col < E ? p.b[col] : 0.0f);
            }
        __syncthreads();
    }
    for (int r = warp; r < kRtRows; r += kRtWarps)
        if (row0 + r < p.rows) pick_experts(p, rt_z + r * ld, row0 + r, ids_s + r * p.m.top);
    // places in the buckets: counted in shared memory, one global addition per expert and CTA
    int32_t* count = reinterpret_cast<int32_t*>(ring);    // [experts] | [experts] first place
    for (int e = tid; e < E; e += kRtThreads) count[e] = 0;
    __syncthreads();
    const int left = p.rows - row0 < kRtRows ? (int)(p.rows - row0) : kRtRows;
    for (int i = tid; i < left * p.m.top; i += kRtThreads) place_s[i] = atomicAdd(count + ids_s[i], 1);
    __syncthreads();
    for (int e = tid; e < E; e += kRtThreads)
        if (count[e] > 0) count[E + e] = atomicAdd(p.counts + e, count[e]);
    __syncthreads();
    for (int i = tid; i < left * p.m.top; i += kRtThreads) {
        const int e = ids_s[i], at = count[E + e] + place_s[i];
        if (at < p.rows) p.bucket[(int64_t)e * p.rows + at] = (int32_t)(row0 * p.m.top + i);
    }
}

}  // namespace ktk

using namespace ktk;

static int check_moe(const ktk_moe* m, int64_t rows, const char* who) {
    if (m == nullptr || rows < 0 || m->experts <= 0 || m->top <= 0 || m->top > m->experts || m->width <= 0 ||
        m->ff <= 0 || m->width_stride < m->width || m->ff_stride < m->ff || m->width_stride % 8 != 0 ||
        m->ff_stride % 8 != 0 || (m->dtype != KTK_F32 && m->dtype != KTK_BF16) ||
        m->scoring < 0 || m->scoring > 1 || !(m->limit > 0.0f)) {
        set_error("%s: bad sizes", who);
        return KTK_ERR_ARG;
    }
    if (m->experts > kMaxExperts || rows > 2147483647LL / m->top || rows > 65535LL * 1024) {
        set_error("%s: at most %d experts; %lld rows", who, kMaxExperts, (long long)rows);
        return KTK_ERR_TOO_LARGE;
    }
    return KTK_OK;
}

extern "C" int ktk_moe_route(const void* h, const void* w, const float* b, int32_t* ids, float* weights,
                             int32_t* counts, int32_t* bucket, int64_t rows, const ktk_moe* shape, int32_t variant,
                             void* stream) {
    const char* who = "ktk_moe_route";
    const int rc = check_moe(shape, rows, who);
    if (rc != KTK_OK) return rc;
    if (rows == 0) return KTK_OK;
    if (!h || !w || !ids || !weights || !counts || !bucket || (((uintptr_t)h | (uintptr_t)w) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    const RouteParams p{*shape, h, w, b, ids, weights, counts, bucket, rows};
    cudaStream_t st = (cudaStream_t)stream;
    const bool by_row = shape->dtype == KTK_F32 || variant == KTK_VARIANT_SIMT ||
                        (variant == KTK_VARIANT_AUTO && (rows <= kRtByRow || shape->top > 64));
    if (by_row) {
        const size_t smem = ((shape->experts + 3) / 4 * 4 + shape->width_stride + shape->top) * sizeof(float);
        if (smem > 200 * 1024) { set_error("%s: rows of %d columns", who, shape->width); return KTK_ERR_UNSUPPORTED; }
        auto kernel = shape->dtype == KTK_F32 ? route_row_kernel<float> : route_row_kernel<__nv_bfloat16>;
        KTK_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem), who);
        kernel<<<(unsigned)rows, kRtRowThreads, smem, st>>>(p);
    } else {
        const size_t smem = (size_t)kRtStages * kRtStageElems * 2 +
                            (size_t)kRtRows * ((shape->experts + kRtCols - 1) / kRtCols * kRtCols) * sizeof(float) +
                            (size_t)2 * kRtRows * shape->top * sizeof(int32_t);
        if (smem > 227 * 1024) {
            set_error("%s: top %d of %d experts", who, shape->top, shape->experts);
            return KTK_ERR_UNSUPPORTED;
        }
        KTK_CUDA_TRY(cudaFuncSetAttribute(route_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem),
                     who);
        route_mma_kernel<<<(unsigned)((rows + kRtRows - 1) / kRtRows), kRtThreads, smem, st>>>(p);
    }
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}

extern "C" int ktk_moe_gemm(int32_t stage, const void* in, const void* w, void* out, const float* weights,
                            const int32_t* counts, const int32_t* bucket, int64_t rows, const ktk_moe* shape,
                            int32_t variant, int32_t* status, void* stream) {
    const char* who = "ktk_moe_gemm";
    const int rc = check_moe(shape, rows, who);
    if (rc != KTK_OK) return rc;
    if (stage != 0 && stage != 1) { set_error("%s: stage %d", who, stage); return KTK_ERR_ARG; }
    if (rows == 0) return KTK_OK;
    if (!in || !w || !out || !counts || !bucket || (stage == 1 && !weights) ||
        (((uintptr_t)in | (uintptr_t)w | (uintptr_t)out) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    if (variant == KTK_VARIANT_UMMA && !moe_umma_supported(*shape)) {
        set_error("%s: variant %d is not built for this case", who, variant);
        return KTK_ERR_UNSUPPORTED;
    }
    const MoeParams p{*shape, in, w, out, weights, counts, bucket, rows, status};
    return variant != KTK_VARIANT_SIMT && moe_umma_supported(*shape) ? launch_moe_umma(stage, p, (cudaStream_t)stream)
                                                                     : launch_moe_simt(stage, p, (cudaStream_t)stream);
}
