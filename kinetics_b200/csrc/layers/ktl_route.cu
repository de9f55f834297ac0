// Router of a mixture of experts: fp32 logits of every row against every expert, the best `top` of them, the softmax
// over those, and each row's place in its experts' buckets -- one launch.
//
// bf16: a CTA takes 32 rows; its 8 warps share the width, each accumulating [32 x 64 experts] with mma.m16n8k16 (fp32
// accumulators, exact products), and add their parts up in shared memory in a fixed order.  fp32: FMA, a warp per
// (row, expert) pair at a time.  Then a warp per row picks the experts.
#include "../ktk_pipeline.cuh"
#include "ktl_common.cuh"

namespace ktk {

constexpr int kRtThreads = 256;
constexpr int kRtWarps = kRtThreads / 32;
constexpr int kRtRows = 32;          // rows of a CTA, tensor-core variant
constexpr int kRtCols = 64;          // experts per pass

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

// One warp: the `top` largest of z[0 .. experts) (ties to the lower index), softmax over them, bucket entries.
// z is overwritten.
__device__ __forceinline__ void pick_experts(const RouteParams& p, float* z, int64_t row) {
    const int lane = threadIdx.x & 31;
    const int E = p.m.experts, top = p.m.top;
    float best0 = 0.0f, denom = 0.0f;
    for (int j = 0; j < top; ++j) {
        float v = -INFINITY;
        int e = 0x7fffffff;
        for (int i = lane; i < E; i += 32)
            if (z[i] > v || e == 0x7fffffff) { v = z[i]; e = i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, v, o);
            const int oe = __shfl_xor_sync(0xffffffffu, e, o);
            if (oe != 0x7fffffff && (e == 0x7fffffff || ov > v || (ov == v && oe < e))) { v = ov; e = oe; }
        }
        if (j == 0) best0 = v;
        const float ex = expf(v - best0);
        denom += ex;
        __syncwarp();
        if (lane == 0) {
            z[e] = -INFINITY;
            p.ids[row * top + j] = e;
            p.weights[row * top + j] = ex;
            const int at = atomicAdd(p.counts + e, 1);
            if (at < p.rows) p.bucket[(int64_t)e * p.rows + at] = (int32_t)(row * top + j);
        }
        __syncwarp();
    }
    for (int j = lane; j < top; j += 32) p.weights[row * top + j] /= denom;
}

__global__ void __launch_bounds__(kRtThreads) route_simt_kernel(const RouteParams p) {
    extern __shared__ float rt_z[];                       // [experts]
    const int64_t row = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float* h = (const float*)p.h + row * p.m.width_stride;
    for (int e = warp; e < p.m.experts; e += kRtWarps) {
        const float* w = (const float*)p.w + (int64_t)e * p.m.width_stride;
        float s = 0.0f;
        for (int i = lane; i < p.m.width; i += 32) s = fmaf(h[i], w[i], s);
        s = warp_sum_f(s);
        if (lane == 0) rt_z[e] = s + p.b[e];
    }
    __syncthreads();
    if (warp == 0) pick_experts(p, rt_z, row);
}

__global__ void __launch_bounds__(kRtThreads) route_mma_kernel(const RouteParams p) {
    extern __shared__ float rt_z[];                       // [kRtRows][experts padded to kRtCols]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int gid = lane >> 2, tig = lane & 3;
    const int E = p.m.experts, ld = (E + kRtCols - 1) / kRtCols * kRtCols;
    const int64_t row0 = (int64_t)blockIdx.x * kRtRows;
    const int K = p.m.width_stride;
    const int steps = (K + 15) / 16;
    const __nv_bfloat16* hp = (const __nv_bfloat16*)p.h;
    const __nv_bfloat16* wp = (const __nv_bfloat16*)p.w;
    // two neighbouring elements of a row, zero outside (columns beyond `width` are zero in memory)
    auto pair = [&](const __nv_bfloat16* base, int64_t r, int64_t r_end, int c) -> uint32_t {
        return r < r_end && c < K ? __ldg(reinterpret_cast<const uint32_t*>(base + r * K + c)) : 0u;
    };
    for (int c0 = 0; c0 < E; c0 += kRtCols) {
        float acc[2][kRtCols / 8][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int n = 0; n < kRtCols / 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[i][n][e] = 0.0f;
        const int n_tiles = (E - c0 + 7) / 8 < kRtCols / 8 ? (E - c0 + 7) / 8 : kRtCols / 8;
#pragma unroll 2
        for (int s = warp; s < steps; s += kRtWarps) {
            const int k = s * 16 + 2 * tig;
            uint32_t a[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int64_t r = row0 + 16 * i + gid;
                a[i][0] = pair(hp, r, p.rows, k);
                a[i][1] = pair(hp, r + 8, p.rows, k);
                a[i][2] = pair(hp, r, p.rows, k + 8);
                a[i][3] = pair(hp, r + 8, p.rows, k + 8);
            }
#pragma unroll
            for (int n = 0; n < kRtCols / 8; ++n) {
                if (n < n_tiles) {
                    const int64_t e = c0 + n * 8 + gid;
                    const uint32_t b0 = pair(wp, e, E, k), b1 = pair(wp, e, E, k + 8);
                    mma_bf16(acc[0][n], a[0], b0, b1);
                    mma_bf16(acc[1][n], a[1], b0, b1);
                }
            }
        }
        // the warps add their parts one after the other: a fixed order
        for (int w = 0; w < kRtWarps; ++w) {
            if (warp == w) {
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int n = 0; n < kRtCols / 8; ++n)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            float* z = rt_z + (16 * i + gid + (e >= 2 ? 8 : 0)) * ld + c0 + n * 8 + 2 * tig + (e & 1);
                            *z = (w == 0 ? 0.0f : *z) + acc[i][n][e];
                        }
            }
            __syncthreads();
        }
    }
    for (int r = warp; r < kRtRows; r += kRtWarps) {
        if (row0 + r >= p.rows) break;
        for (int e = lane; e < E; e += 32) rt_z[r * ld + e] += p.b[e];
        __syncwarp();
        pick_experts(p, rt_z + r * ld, row0 + r);
    }
}

}  // namespace ktk

using namespace ktk;

static int check_moe(const ktk_moe* m, int64_t rows, const char* who) {
    if (m == nullptr || rows < 0 || m->experts <= 0 || m->top <= 0 || m->top > m->experts || m->width <= 0 ||
        m->ff <= 0 || m->width_stride < m->width || m->ff_stride < m->ff || m->width_stride % 8 != 0 ||
        m->ff_stride % 8 != 0 || (m->dtype != KTK_F32 && m->dtype != KTK_BF16)) {
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
    if (!h || !w || !b || !ids || !weights || !counts || !bucket || (((uintptr_t)h | (uintptr_t)w) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    (void)variant;
    const RouteParams p{*shape, h, w, b, ids, weights, counts, bucket, rows};
    cudaStream_t st = (cudaStream_t)stream;
    if (shape->dtype == KTK_F32) {
        route_simt_kernel<<<(unsigned)rows, kRtThreads, shape->experts * sizeof(float), st>>>(p);
    } else {
        const size_t smem = (size_t)kRtRows * ((shape->experts + kRtCols - 1) / kRtCols * kRtCols) * sizeof(float);
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
