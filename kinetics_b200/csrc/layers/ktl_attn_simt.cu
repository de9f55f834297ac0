// Paged causal attention in fp32 math, any head sizes: one CTA per (query row, query head).  Both maps of the head
// walk the keys in tiles of 128 -- thread t scores key t of the tile, then owns columns t, t + 128, ... of the output.
// Serves the fp32 models, and bf16 sizes that the tensor-core kernels are not built for.
#include "ktl_common.cuh"

namespace ktk {

constexpr int kSaThreads = 128;
constexpr int kSaCols = 8;         // value columns per thread: vdim <= 1024

__device__ __forceinline__ float cta_max(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    v = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    __syncthreads();
    return v;
}
__device__ __forceinline__ float cta_sum(float v, float* red) {
    v = warp_sum_f(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    v = (red[0] + red[1]) + (red[2] + red[3]);
    __syncthreads();
    return v;
}

template <typename T, int MAPS>
__global__ void __launch_bounds__(kSaThreads) attn_simt_kernel(const AttnParams p) {
    extern __shared__ float sa_q[];                       // [MAPS][dim_stride]
    __shared__ float prob[MAPS][kSaThreads];
    __shared__ int64_t key_slot[kSaThreads];              // page * page_size + slot
    __shared__ float red[4];
    const ktk_attn& a = p.a;
    const int64_t r = blockIdx.x;
    const int head = blockIdx.y, tid = threadIdx.x;
    const int kvh = head / (a.heads / a.kv_heads);
    const int b = p.new_indptr ? sequence_of_row(p.new_indptr, p.t.batch, r) : (int)r;
    const Span s = span_of(p.t, b);
    const int pos = p.new_indptr ? s.total - (p.new_indptr[b + 1] - (int)r) : s.total - 1;
    if (s.bad || pos < 0 || pos >= s.total) {             // uniform for the CTA
        if (tid == 0) report(p.status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const T* qrow = (const T*)p.q + r * p.q_stride + (int64_t)head * MAPS * a.dim_stride;
    const float factor = a.scale * query_temperature(a.temp_coef, a.temp_every, pos);
    for (int i = tid; i < MAPS * a.dim_stride; i += kSaThreads) sa_q[i] = to_f32(qrow[i]) * factor;
    float m[MAPS], l[MAPS], acc[MAPS][kSaCols];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
        m[mp] = -INFINITY; l[mp] = 0.0f;
#pragma unroll
        for (int c = 0; c < kSaCols; ++c) acc[mp][c] = 0.0f;
    }
    __syncthreads();
    for (int j0 = 0; j0 <= pos; j0 += kSaThreads) {
        const int j = j0 + tid;
        int64_t slot = -1;
        if (j <= pos) {
            const int64_t page = p.t.kv_indices[s.start + j / p.t.page_size];
            if (page < 0 || page >= p.t.num_pages) report(p.status, KTK_STATUS_BAD_PAGE);
            else slot = page * p.t.page_size + j % p.t.page_size;
        }
        key_slot[tid] = slot;
#pragma unroll
        for (int mp = 0; mp < MAPS; ++mp) {
            float sc = -INFINITY;
            if (slot >= 0) {
                const T* krow = (const T*)p.k + row_in_pages(slot, p.t.page_size, a.kv_heads * MAPS, kvh * MAPS + mp) * a.dim_stride;
                const float* qm = sa_q + mp * a.dim_stride;
                float d = 0.0f;
                for (int i = 0; i < a.dim_stride; i += 8) {
                    float kv[8];
                    load8(krow + i, kv);
#pragma unroll
                    for (int e = 0; e < 8; ++e) d = fmaf(qm[i + e], kv[e], d);
                }
                sc = a.softcap > 0.0f ? a.softcap * tanhf(d / a.softcap) : d;
            }
            const float mn = fmaxf(m[mp], cta_max(sc, red));
            const float ref = mn == -INFINITY ? 0.0f : mn;
            const float pr = expf(sc - ref);
            const float old = expf(m[mp] - ref);
            l[mp] = l[mp] * old + cta_sum(pr, red);
            m[mp] = mn;
#pragma unroll
            for (int c = 0; c < kSaCols; ++c) acc[mp][c] *= old;
            prob[mp][tid] = pr;
        }
        __syncthreads();
        const int n = pos + 1 - j0 < kSaThreads ? pos + 1 - j0 : kSaThreads;
        for (int i = 0; i < n; ++i) {
            const int64_t sl = key_slot[i];
            if (sl < 0) continue;
            const T* vrow = (const T*)p.v + row_in_pages(sl, p.t.page_size, a.kv_heads, kvh) * value_row(a);
#pragma unroll
            for (int c = 0; c < kSaCols; ++c) {
                const int col = tid + c * kSaThreads;
                if (col < a.vdim) {
                    const float v = to_f32(vrow[col]);
#pragma unroll
                    for (int mp = 0; mp < MAPS; ++mp) acc[mp][c] = fmaf(prob[mp][i], v, acc[mp][c]);
                }
            }
        }
        __syncthreads();
    }
    if (MAPS == 1 && p.sink != nullptr) {
        const float sk = p.sink[head], mn = fmaxf(m[0], sk);
        const float old = expf(m[0] - mn);
        l[0] = l[0] * old + expf(sk - mn);
#pragma unroll
        for (int c = 0; c < kSaCols; ++c) acc[0][c] *= old;
    }
    T* dst = (T*)p.o + (r * a.heads + head) * a.vdim_stride;
    float o[kSaCols], ss = 0.0f;
#pragma unroll
    for (int c = 0; c < kSaCols; ++c) {
        o[c] = acc[0][c] / l[0];
        if (MAPS == 2) o[c] -= a.lambda * (acc[MAPS - 1][c] / l[MAPS - 1]);
        if (tid + c * kSaThreads < a.vdim) ss += o[c] * o[c];
    }
    float f = 1.0f;
    if (MAPS == 1 && p.gate != nullptr) f = sigmoid_f(to_f32(((const T*)p.gate)[r * p.gate_stride + head]));
    if (MAPS == 2) f = a.out_scale / sqrtf(cta_sum(ss, red) / (float)a.vdim + a.eps);
#pragma unroll
    for (int c = 0; c < kSaCols; ++c) {
        const int col = tid + c * kSaThreads;
        if (col < a.vdim_stride) dst[col] = from_f32<T>(col < a.vdim ? o[c] * f : 0.0f);
    }
}

template <typename T>
static int simt_launch(const AttnParams& p, cudaStream_t st) {
    const size_t smem = (size_t)p.a.maps * p.a.dim_stride * sizeof(float);
    const dim3 grid((unsigned)p.rows, (unsigned)p.a.heads);
    if (p.a.maps == 2) attn_simt_kernel<T, 2><<<grid, kSaThreads, smem, st>>>(p);
    else attn_simt_kernel<T, 1><<<grid, kSaThreads, smem, st>>>(p);
    KTK_CUDA_TRY(cudaGetLastError(), "ktk_paged_attention");
    return KTK_OK;
}

int launch_attn_simt(const AttnParams& p, cudaStream_t st) {
    if (p.a.vdim_stride > kSaThreads * kSaCols || p.a.dim_stride > 2048 || p.a.heads > 65535) {
        set_error("ktk_paged_attention: dim %d (at most 2048), vdim %d (at most %d), heads %d", p.a.dim, p.a.vdim,
                  kSaThreads * kSaCols, p.a.heads);
        return KTK_ERR_UNSUPPORTED;
    }
    return p.a.dtype == KTK_F32 ? simt_launch<float>(p, st) : simt_launch<__nv_bfloat16>(p, st);
}

}  // namespace ktk
