// The experts' matrix products in fp32 math: tiles of 64 rows of one expert x 64 output columns, operands staged in
// shared memory 16 columns at a time, 4 x 4 results per thread.  Serves the fp32 models.
#include "ktl_common.cuh"

namespace ktk {

constexpr int kMsTile = 64, kMsK = 16, kMsThreads = 256;

template <typename T, int STAGE>
__global__ void __launch_bounds__(kMsThreads) moe_simt_kernel(const MoeParams p) {
    __shared__ ExpertPlan plan;
    __shared__ float sa[kMsK][kMsTile + 1], sb[2][kMsK][kMsTile + 1];
    __shared__ int64_t src_row[kMsTile], dst_row[kMsTile];
    __shared__ float wt[kMsTile];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int N = STAGE == 0 ? p.m.ff_stride : p.m.width_stride, K = STAGE == 0 ? p.m.width_stride : p.m.ff_stride;
    if (tid < 32) plan_experts(plan, p.counts, p.m.experts, p.rows, kMsTile);
    __syncthreads();
    const int tiles = plan.first_tile[p.m.experts], cols = (N + kMsTile - 1) / kMsTile;
    for (int64_t w = blockIdx.x; w < (int64_t)tiles * cols; w += gridDim.x) {
        const int t = (int)(w / cols), n0 = (int)(w % cols) * kMsTile;
        const int e = expert_of_tile(plan, p.m.experts, t);
        const int r0 = (t - plan.first_tile[e]) * kMsTile;
        const int n_e = plan.first_row[e + 1] - plan.first_row[e];
        if (tid < kMsTile) {
            const int r = r0 + tid;
            int64_t s = -1, d = -1;
            float f = 1.0f;
            if (r < n_e) {
                const int64_t at = plan.first_row[e] + r;
                const int entry = p.bucket[(int64_t)e * p.rows + r];
                if (STAGE == 0) { s = entry / p.m.top; d = at; }
                else { s = at; d = entry; f = p.weights[entry]; }
            }
            src_row[tid] = s; dst_row[tid] = d; wt[tid] = f;
        }
        __syncthreads();
        float acc[2][4][4];
#pragma unroll
        for (int g = 0; g < 2; ++g)
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[g][i][j] = 0.0f;
        for (int k0 = 0; k0 < K; k0 += kMsK) {
            for (int i = tid; i < kMsTile * kMsK; i += kMsThreads) {
                const int rr = i / kMsK, kk = i % kMsK;
                const int64_t s = src_row[rr];
                sa[kk][rr] = s >= 0 && k0 + kk < K ? to_f32(((const T*)p.in)[s * K + k0 + kk]) : 0.0f;
#pragma unroll
                for (int g = 0; g < (STAGE == 0 ? 2 : 1); ++g) {
                    const int64_t wr = STAGE == 0 ? ((int64_t)e * N + n0 + rr) * 2 + g : (int64_t)e * N + n0 + rr;
                    sb[g][kk][rr] = n0 + rr < N && k0 + kk < K ? to_f32(((const T*)p.w)[wr * K + k0 + kk]) : 0.0f;
                }
            }
            __syncthreads();
#pragma unroll
            for (int kk = 0; kk < kMsK; ++kk) {
                float av[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) av[i] = sa[kk][ty + 16 * i];
#pragma unroll
                for (int g = 0; g < (STAGE == 0 ? 2 : 1); ++g)
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float bv = sb[g][kk][tx + 16 * j];
#pragma unroll
                        for (int i = 0; i < 4; ++i) acc[g][i][j] = fmaf(av[i], bv, acc[g][i][j]);
                    }
            }
            __syncthreads();
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int64_t d = dst_row[ty + 16 * i];
            if (d < 0) continue;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int n = n0 + tx + 16 * j;
                if (n >= N) continue;
                float v = acc[0][i][j];
                if (STAGE == 0) v = gated<false>(v, acc[1][i][j], p.m.limit, p.m.slope, p.m.shift);
                else v *= wt[ty + 16 * i];
                ((T*)p.out)[d * N + n] = from_f32<T>(v);
            }
        }
        __syncthreads();
    }
}

template <typename T, int STAGE> static int moe_simt(const MoeParams& p, cudaStream_t st) {
    const int N = STAGE == 0 ? p.m.ff_stride : p.m.width_stride;
    int64_t work = ((p.rows * p.m.top + kMsTile - 1) / kMsTile + p.m.experts) * ((N + kMsTile - 1) / kMsTile);
    const int64_t cap = (int64_t)sm_count() * 8;
    if (work > cap) work = cap;
    moe_simt_kernel<T, STAGE><<<(unsigned)work, kMsThreads, 0, st>>>(p);
    KTK_CUDA_TRY(cudaGetLastError(), "ktk_moe_gemm");
    return KTK_OK;
}

int launch_moe_simt(int stage, const MoeParams& p, cudaStream_t st) {
    if (p.m.dtype == KTK_F32) return stage == 0 ? moe_simt<float, 0>(p, st) : moe_simt<float, 1>(p, st);
    return stage == 0 ? moe_simt<__nv_bfloat16, 0>(p, st) : moe_simt<__nv_bfloat16, 1>(p, st);
}

}  // namespace ktk
