// Decode attention of one new token per sequence over a paged cache with free head sizes (up to 128), two softmax maps
// per head over shared values: bf16 tensor cores (mma.m16n8k16), TMA-staged pages.
//
// One CTA per (sequence, kv head and up to 8 of its query heads, split of the keys).  A producer warp streams units of
// 16 tokens -- the keys of both maps and the values -- into a ring in shared memory; four consumer warps take units in
// turn.  The heads are the 8 columns:
//     S_m^T[16 keys x 8 heads] = K_m[16 x dim] . Q_m^T           per map m
//     O_m^T[vdim x 8 heads]   += V^T[vdim x 16] . P_m^T          V fragments shared by the two maps
// At the end the warps add up, and either the head is finished here (one split: difference of the maps, unit norm) or
// the un-normalised partials go to the workspace for the combine kernel.
#include "ktl_score.cuh"

namespace ktk {

constexpr int kAdConsumers = 4;
constexpr int kAdThreads = (kAdConsumers + 1) * 32;
constexpr int kAdStages = 8;          // a multiple of the consumers: a stage belongs to one warp
constexpr int kAdUnit = 16;           // tokens per stage
constexpr int kAdTile = kAdUnit * 128;
constexpr int kAdMinKeys = 256;       // a split is not worth less
constexpr int kAdMaxSplits = 256;
static_assert(kAdStages % kAdConsumers == 0, "a stage must belong to one consumer warp");

template <int DC, int VC> constexpr int ad_stage_bytes() { return (2 * DC + VC) * kAdTile; }
template <int DC, int VC> constexpr int ad_smem() {
    constexpr int ring = kAdStages * ad_stage_bytes<DC, VC>(), merge = kAdConsumers * 8 * VC * 64 * 4;
    return (ring > merge ? ring : merge) + 1024;
}

__device__ __forceinline__ uint32_t ad_off(int tok, int c16) {
    return (uint32_t)((c16 >> 3) * kAdTile + tok * 128 + (((c16 & 7) ^ (tok & 7)) << 4));
}

// partial of one (row, head, split): m1, l1, m2, l2, then O_1 and O_2 [vdim_stride] each
__host__ __device__ inline int64_t ad_partial_floats(int vdim_stride) { return 4 + 2 * (int64_t)vdim_stride; }

template <int DC, int VC, bool FIXED, int CTAS>
__global__ void __launch_bounds__(kAdThreads, CTAS)
attn_decode_kernel(const AttnParams p, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map) {
    extern __shared__ uint8_t ad_raw[];
    __shared__ __align__(8) uint64_t full[kAdStages], empty[kAdStages];
    __shared__ int abort_flag, issued_total;
    __shared__ float red_m[kAdConsumers][2][8], red_l[kAdConsumers][2][8];
    constexpr int kStage = ad_stage_bytes<DC, VC>();
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ad_raw) + 1023) & ~uintptr_t(1023));
    const ktk_attn& a = p.a;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int group = a.heads / a.kv_heads, chunks = (group + 7) / 8;
    const int split = blockIdx.x, b = blockIdx.z;
    const int kvh = blockIdx.y / chunks, g0 = (blockIdx.y % chunks) * 8;
    const int heads = group - g0 < 8 ? group - g0 : 8;
    const int head0 = kvh * group + g0;
    const Span s = span_of(p.t, b);
    if (s.bad || s.total <= 0) {
        if (tid == 0) report(p.status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const int units = (s.total + kAdUnit - 1) / kAdUnit;
    const int per = (units + p.splits - 1) / p.splits;
    const int u0 = split * per, u1 = u0 + per < units ? u0 + per : units;
    const int n = u1 > u0 ? u1 - u0 : 0;

    if (tid == 0) {
        for (int i = 0; i < kAdStages; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 1); }
        abort_flag = 0;
        issued_total = 0;
        mbar_init_fence();
    }
    __syncthreads();

    const int gid = lane >> 2, tig = lane & 3;
    float m[2][2], l[2][2], acc[2][VC * 4][4];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        m[mp][0] = m[mp][1] = FIXED ? 0.0f : -INFINITY;
        l[mp][0] = l[mp][1] = 0.0f;
#pragma unroll
        for (int t = 0; t < VC * 4; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[mp][t][e] = 0.0f;
    }

    if (warp == kAdConsumers) {
        if (lane == 0) {
            prefetch_tensormap(&k_map);
            prefetch_tensormap(&v_map);
            int i = 0;
            for (; i < n; ++i) {
                const int st = i % kAdStages;
                const int tok = (u0 + i) * kAdUnit;
                const int64_t page = p.t.kv_indices[s.start + tok / p.t.page_size];
                if (i >= kAdStages && !mbar_wait(&empty[st], ((i / kAdStages) - 1) & 1, &abort_flag)) break;
                if (page < 0 || page >= p.t.num_pages) {
                    report(p.status, KTK_STATUS_BAD_PAGE);
                    mbar_arrive(&full[st]);              // stale contents: the status word says so
                    continue;
                }
                uint8_t* dst = ring + st * kStage;
                const int y = tok % p.t.page_size;
                mbar_arrive_expect_tx(&full[st], kStage);
#pragma unroll
                for (int mp = 0; mp < 2; ++mp)
#pragma unroll
                    for (int c = 0; c < DC; ++c)
                        tma_load_3d(dst + (mp * DC + c) * kAdTile, &k_map, &full[st], c * 64, y,
                                    (int)(page * (2 * a.kv_heads)) + kvh * 2 + mp);
#pragma unroll
                for (int c = 0; c < VC; ++c)
                    tma_load_3d(dst + (2 * DC + c) * kAdTile, &v_map, &full[st], c * 64, y,
                                (int)(page * a.kv_heads) + kvh);
            }
            issued_total = i;
        }
    } else {
        const float factor = a.scale * query_temperature(a.temp_coef, a.temp_every, s.total - 1);
        CapCoef cap;
        cap.set(factor, a.softcap > 0.0f ? a.softcap : 1.0f);
        const bool capped = FIXED || a.softcap > 0.0f;
        const float plain = factor * kLog2eF;
        const int ksteps = (a.dim_stride + 15) / 16, vtiles = (a.vdim_stride + 15) / 16;
        uint32_t qb[2][DC * 4][2];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            const uint32_t* qp = reinterpret_cast<const uint32_t*>(
                (const __nv_bfloat16*)p.q + b * p.q_stride + ((int64_t)(head0 + (gid < heads ? gid : 0)) * 2 + mp) * a.dim_stride);
#pragma unroll
            for (int ks = 0; ks < DC * 4; ++ks) {
                const int c = ks * 16 + 2 * tig;
                qb[mp][ks][0] = gid < heads && c < a.dim_stride ? __ldg(qp + ks * 8 + tig) : 0u;
                qb[mp][ks][1] = gid < heads && c + 8 < a.dim_stride ? __ldg(qp + ks * 8 + 4 + tig) : 0u;
            }
        }
        const int mj = lane >> 3, mr = lane & 7;
        const int k_tok = mr + 8 * (mj & 1), k_c = mj >> 1;
        const int v_tok = mr + 8 * (mj >> 1), v_c = mj & 1;
        for (int i = warp; i < n; i += kAdConsumers) {
            const int st = i % kAdStages;
            if (!__all_sync(0xffffffffu, mbar_wait(&full[st], (i / kAdStages) & 1, &abort_flag))) break;
            uint8_t* stage = ring + st * kStage;
            const int left = s.total - (u0 + i) * kAdUnit;
            const int ntok = left < kAdUnit ? left : kAdUnit;
            const uint32_t kt = smem_u32(stage), vt = kt + 2 * DC * kAdTile;
            if (ntok < kAdUnit) {
                // rows past the end may hold anything: clear them in V so that 0 * x stays 0
                for (int c = lane; c < (kAdUnit - ntok) * VC * 8; c += 32) {
                    const int t = ntok + c / (VC * 8), cc = c % (VC * 8);
                    *reinterpret_cast<uint4*>(stage + 2 * DC * kAdTile + (cc >> 3) * kAdTile + t * 128 + ((cc & 7) << 4)) =
                        make_uint4(0u, 0u, 0u, 0u);
                }
                __syncwarp();
            }
            uint32_t pb[2][2];
#pragma unroll
            for (int mp = 0; mp < 2; ++mp) {
                float sa[4] = {0.f, 0.f, 0.f, 0.f}, sb[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int ks = 0; ks < DC * 4; ks += 2) {
                    if (ks < ksteps) {
                        uint32_t ka[4];
                        ldmatrix_x4(ka, kt + mp * DC * kAdTile + ad_off(k_tok, 2 * ks + k_c));
                        mma_bf16(sa, ka, qb[mp][ks][0], qb[mp][ks][1]);
                    }
                    if (ks + 1 < ksteps) {
                        uint32_t kb[4];
                        ldmatrix_x4(kb, kt + mp * DC * kAdTile + ad_off(k_tok, 2 * ks + 2 + k_c));
                        mma_bf16(sb, kb, qb[mp][ks + 1][0], qb[mp][ks + 1][1]);
                    }
                }
                float t[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float sc = sa[e] + sb[e];
                    t[e] = capped ? cap(sc) : sc * plain;
                    if (gid + (e >= 2 ? 8 : 0) >= ntok) t[e] = -INFINITY;
                }
                float al[2] = {1.0f, 1.0f};
                if (!FIXED) {
                    float mx[2] = {fmaxf(t[0], t[2]), fmaxf(t[1], t[3])};
#pragma unroll
                    for (int o = 4; o <= 16; o <<= 1) {
                        mx[0] = fmaxf(mx[0], __shfl_xor_sync(0xffffffffu, mx[0], o));
                        mx[1] = fmaxf(mx[1], __shfl_xor_sync(0xffffffffu, mx[1], o));
                    }
#pragma unroll
                    for (int c = 0; c < 2; ++c) {        // a unit holds at least one token: the maximum is finite
                        const float mn = fmaxf(m[mp][c], mx[c]);
                        al[c] = ex2(m[mp][c] - mn);
                        m[mp][c] = mn;
                    }
                }
                const uint32_t lo = pack_bf16(ex2(t[0] - m[mp][0]), ex2(t[1] - m[mp][1]));
                const uint32_t hi = pack_bf16(ex2(t[2] - m[mp][0]), ex2(t[3] - m[mp][1]));
                float s0 = __uint_as_float(lo << 16) + __uint_as_float(hi << 16);
                float s1 = __uint_as_float(lo & 0xffff0000u) + __uint_as_float(hi & 0xffff0000u);
                if (FIXED) {                             // rows are summed up once at the end
                    l[mp][0] += s0;
                    l[mp][1] += s1;
                } else {
#pragma unroll
                    for (int o = 4; o <= 16; o <<= 1) {
                        s0 += __shfl_xor_sync(0xffffffffu, s0, o);
                        s1 += __shfl_xor_sync(0xffffffffu, s1, o);
                    }
                    l[mp][0] = l[mp][0] * al[0] + s0;
                    l[mp][1] = l[mp][1] * al[1] + s1;
#pragma unroll
                    for (int vt_ = 0; vt_ < VC * 4; ++vt_) {
                        acc[mp][vt_][0] *= al[0]; acc[mp][vt_][1] *= al[1];
                        acc[mp][vt_][2] *= al[0]; acc[mp][vt_][3] *= al[1];
                    }
                }
                pb[mp][0] = movmatrix_trans(lo);
                pb[mp][1] = movmatrix_trans(hi);
            }
#pragma unroll
            for (int t = 0; t < VC * 4; ++t) {
                if (t < vtiles) {
                    uint32_t va[4];
                    ldmatrix_x4_trans(va, vt + ad_off(v_tok, 2 * t + v_c));
                    mma_bf16(acc[0][t], va, pb[0][0], pb[0][1]);
                    mma_bf16(acc[1][t], va, pb[1][0], pb[1][1]);
                }
            }
            if (ntok < kAdUnit) fence_proxy_async();     // the cleared rows were written by ordinary stores
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[st]);
        }
        if (FIXED) {
#pragma unroll
            for (int mp = 0; mp < 2; ++mp)
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int o = 4; o <= 16; o <<= 1) l[mp][c] += __shfl_xor_sync(0xffffffffu, l[mp][c], o);
        }
        if (gid == 0) {
#pragma unroll
            for (int mp = 0; mp < 2; ++mp)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    red_m[warp][mp][2 * tig + c] = m[mp][c];
                    red_l[warp][mp][2 * tig + c] = l[mp][c];
                }
        }
    }
    __syncthreads();                                     // every unit consumed, or the CTA gave up
    if (abort_flag) {
        if (tid == 0) {
            report(p.status, KTK_STATUS_TIMEOUT);
            volatile int never = 0;
            for (int i = issued_total > kAdStages ? issued_total - kAdStages : 0; i < issued_total; ++i)
                mbar_wait(&full[i % kAdStages], (i / kAdStages) & 1, &never);
        }
        return;                                          // uniform: abort_flag is read behind the barrier
    }

    // ---- the four warps' parts, one map at a time through the ring's memory ----
    float* merge = reinterpret_cast<float*>(ring);       // [warp][8 heads][VC * 64]
    constexpr int kVt = VC * 64;
    float o[2][8 * kVt / 128];                           // thread tid (of 128): elements tid, tid + 128, ... of [heads][kVt]
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        if (warp < kAdConsumers) {
#pragma unroll
            for (int t = 0; t < VC * 4; ++t) {
                float* d = merge + (warp * 8 + 2 * tig) * kVt + 16 * t + gid;
                d[0] = acc[mp][t][0];
                d[kVt] = acc[mp][t][1];
                d[8] = acc[mp][t][2];
                d[kVt + 8] = acc[mp][t][3];
            }
        }
        __syncthreads();
        if (warp < kAdConsumers) {
#pragma unroll
            for (int i = 0; i < 8 * kVt / 128; ++i) {
                const int x = tid + i * 128, h = x / kVt;
                float M = 0.0f, v = 0.0f;
                if (!FIXED) {
                    M = red_m[0][mp][h];
                    for (int w = 1; w < kAdConsumers; ++w) M = fmaxf(M, red_m[w][mp][h]);
                    if (M == -INFINITY) M = 0.0f;
                }
#pragma unroll
                for (int w = 0; w < kAdConsumers; ++w)
                    v += (FIXED ? 1.0f : ex2(red_m[w][mp][h] - M)) * merge[w * 8 * kVt + x];
                o[mp][i] = v;
            }
        }
        __syncthreads();
    }
    if (warp >= kAdConsumers) return;
    auto merged = [&](int mp, int h, float& M, float& L) {
        M = red_m[0][mp][h];
        for (int w = 1; w < kAdConsumers; ++w) M = fmaxf(M, red_m[w][mp][h]);
        const float ref = M == -INFINITY ? 0.0f : M;
        L = 0.0f;
        for (int w = 0; w < kAdConsumers; ++w) L += (FIXED ? 1.0f : ex2(red_m[w][mp][h] - ref)) * red_l[w][mp][h];
    };
    if (p.splits > 1) {
#pragma unroll
        for (int i = 0; i < 8 * kVt / 128; ++i) {
            const int x = tid + i * 128, h = x / kVt, c = x % kVt;
            if (h >= heads) continue;
            float* w = p.ws + (((int64_t)b * a.heads + head0 + h) * p.splits + split) * ad_partial_floats(a.vdim_stride);
            if (c < a.vdim_stride) {
                w[4 + c] = o[0][i];
                w[4 + a.vdim_stride + c] = o[1][i];
            }
            if (c == 0) {
#pragma unroll
                for (int mp = 0; mp < 2; ++mp) {
                    float M, L;
                    merged(mp, h, M, L);
                    w[2 * mp] = M;
                    w[2 * mp + 1] = L;
                }
            }
        }
        return;
    }
    // one split: difference and unit norm here; a head's columns lie in consecutive threads, summed over shared memory
    float* sq = merge;                                   // [8] sums of squares by warp: [8 heads][4 warps]
    float d[8 * kVt / 128];
#pragma unroll
    for (int i = 0; i < 8 * kVt / 128; ++i) {
        const int x = tid + i * 128, h = x / kVt, c = x % kVt;
        float M, L1, L2;
        merged(0, h, M, L1);
        merged(1, h, M, L2);
        d[i] = L1 > 0.0f && L2 > 0.0f && c < a.vdim ? o[0][i] / L1 - a.lambda * (o[1][i] / L2) : 0.0f;
        const float ss = warp_sum_f(d[i] * d[i]);        // a warp's 32 columns lie in one head
        if (lane == 0) sq[i * kAdConsumers + warp] = ss;
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 8 * kVt / 128; ++i) {
        const int x = tid + i * 128, h = x / kVt, c = x % kVt;
        float ss = 0.0f;                                 // kVt / 32 warp sums of head h
        const int w0 = kVt == 128 ? 0 : (warp & ~1);
#pragma unroll
        for (int w = 0; w < kVt / 32; ++w) ss += sq[i * kAdConsumers + w0 + w];
        const float f = a.out_scale / sqrtf(ss / (float)a.vdim + a.eps);
        if (h < heads && c < a.vdim_stride)
            ((__nv_bfloat16*)p.o)[((int64_t)b * a.heads + head0 + h) * a.vdim_stride + c] = __float2bfloat16_rn(d[i] * f);
    }
}

// One CTA per (head, row): merges the splits of both maps, takes the difference, unit norm.
__global__ void __launch_bounds__(128) attn_combine_kernel(const AttnParams p, int fixed) {
    __shared__ float part[4];
    const ktk_attn& a = p.a;
    const int c = threadIdx.x;
    const int64_t row = blockIdx.y, head = blockIdx.x;
    const int64_t stride = ad_partial_floats(a.vdim_stride);
    const float* w = p.ws + (row * a.heads + head) * p.splits * stride;
    float out[2];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        float M = fixed ? 0.0f : -INFINITY, L = 0.0f, O = 0.0f;
        if (!fixed)
            for (int s = 0; s < p.splits; ++s) M = fmaxf(M, w[s * stride + 2 * mp]);
        const float ref = M == -INFINITY ? 0.0f : M;
#pragma unroll 4
        for (int s = 0; s < p.splits; ++s) {
            const float* q = w + s * stride;
            const float f = fixed ? 1.0f : ex2(q[2 * mp] - ref);
            L += f * q[2 * mp + 1];
            if (c < a.vdim_stride) O += f * q[4 + mp * a.vdim_stride + c];
        }
        out[mp] = L > 0.0f && c < a.vdim ? O / L : 0.0f;
    }
    const float d = out[0] - a.lambda * out[1];
    const float ss = warp_sum_f(d * d);
    if ((c & 31) == 0) part[c >> 5] = ss;
    __syncthreads();
    const float f = a.out_scale / sqrtf((part[0] + part[1] + part[2] + part[3]) / (float)a.vdim + a.eps);
    if (c < a.vdim_stride) ((__nv_bfloat16*)p.o)[(row * a.heads + head) * a.vdim_stride + c] = __float2bfloat16_rn(d * f);
}

bool attn_decode_supported(const ktk_attn& a) {
    return a.dtype == KTK_BF16 && a.maps == 2 && a.v_row_stride == 0 && a.dim_stride <= 128 && a.vdim_stride <= 128;
}

static int64_t decode_units(const ktk_attn& a, int64_t batch) {
    const int group = a.heads / a.kv_heads;
    return batch * a.kv_heads * ((group + 7) / 8);
}

int32_t attn_decode_splits(const ktk_attn& a, int batch, int64_t max_keys) {
    return fill_rounds(decode_units(a, batch), (int64_t)sm_count() * 3, 2, 8, (max_keys + kAdMinKeys - 1) / kAdMinKeys,
                       kAdMaxSplits);
}

size_t attn_decode_workspace(const ktk_attn& a, int64_t rows, int splits) {
    return splits <= 1 ? 0 : (size_t)rows * a.heads * splits * ad_partial_floats(a.vdim_stride) * sizeof(float);
}

int make_cache_maps(const AttnParams& p, CUtensorMap* k_map, CUtensorMap* v_map, uint32_t box_rows, const char* who) {
    const ktk_attn& a = p.a;
    const uint64_t ps = p.t.page_size, kr = (uint64_t)a.kv_heads * a.maps, vr = a.kv_heads;
    // innermost first: columns, tokens of a page, (page, head)
    const uint64_t kd[3] = {(uint64_t)a.dim_stride, ps, (uint64_t)p.t.num_pages * kr};
    const uint64_t vd[3] = {(uint64_t)a.vdim_stride, ps, (uint64_t)p.t.num_pages * vr};
    const uint64_t ks[2] = {(uint64_t)a.dim_stride * 2, ps * a.dim_stride * 2};
    const uint64_t vs[2] = {(uint64_t)a.vdim_stride * 2, ps * a.vdim_stride * 2};
    const uint32_t box[3] = {64, box_rows, 1};
    const int rc = make_tensor_map_3d(k_map, p.k, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, kd, ks, box,
                                      CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc != KTK_OK) return rc;
    return make_tensor_map_3d(v_map, p.v, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, vd, vs, box, CU_TENSOR_MAP_SWIZZLE_128B, who);
}

template <int DC, int VC, bool FIXED, int CTAS> static int decode_launch(const AttnParams& p, cudaStream_t st) {
    const char* who = "ktk_paged_attention";
    CUtensorMap km, vm;
    const int rc = make_cache_maps(p, &km, &vm, kAdUnit, who);
    if (rc != KTK_OK) return rc;
    constexpr int smem = ad_smem<DC, VC>();
    auto kernel = attn_decode_kernel<DC, VC, FIXED, CTAS>;
    KTK_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), who);
    const int group = p.a.heads / p.a.kv_heads;
    const dim3 grid((unsigned)p.splits, (unsigned)(p.a.kv_heads * ((group + 7) / 8)), (unsigned)p.t.batch);
    kernel<<<grid, kAdThreads, smem, st>>>(p, km, vm);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    if (p.splits > 1) {
        attn_combine_kernel<<<dim3((unsigned)p.a.heads, (unsigned)p.t.batch), 128, 0, st>>>(p, FIXED ? 1 : 0);
        KTK_CUDA_TRY(cudaGetLastError(), who);
    }
    return KTK_OK;
}

int launch_attn_decode(const AttnParams& p, cudaStream_t st) {
    if (p.t.batch > 65535 || (int64_t)p.a.heads > 65535) {
        set_error("ktk_paged_attention: more than 65535 sequences or heads in one launch");
        return KTK_ERR_TOO_LARGE;
    }
    const bool d1 = p.a.dim_stride <= 64, v1 = p.a.vdim_stride <= 64, fx = fixed_reference(p.a);
    if (d1 && v1) return fx ? decode_launch<1, 1, true, 3>(p, st) : decode_launch<1, 1, false, 3>(p, st);
    if (d1) return fx ? decode_launch<1, 2, true, 3>(p, st) : decode_launch<1, 2, false, 3>(p, st);
    return fx ? decode_launch<2, 2, true, 2>(p, st) : decode_launch<2, 2, false, 2>(p, st);
}

}  // namespace ktk
