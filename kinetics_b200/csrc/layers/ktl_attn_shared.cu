// Attention of many heads over one cached row per token whose first columns are also the value (attention over
// latents): bf16 on the fifth-generation tensor cores, for decode steps and for short portions of a prompt.
//
// A row is wide (up to 576 columns) and serves every head, so the tokens are the M operand and up to 64 (row, head)
// pairs the N operand; each tile of 64 tokens comes into shared memory once and is used twice:
//     S^T[64 tokens x N]  = K[64 x dim] . Q^T                  A read K-major
//     O^T[vdim x N]      += V^T[vdim x 64] . P                 A = the same tile read MN-major, 128 columns at a time
// One CTA per (split of the tokens, chunk of heads, group of rows).  Roles:
//     loading warp     TMA: tiles of 64 tokens into a ring
//     issuing warp     both products, in whatever order their inputs become ready
//     softmax warps    warp w holds tokens 16 w .., two per thread; exponentials against a reference per column, at first the largest of its sink and the first tile's scores, that moves
//                      only when a score exceeds it by 2^8
// The sum of a column's weights stays spread over the threads until the end.  Tensor memory: S of two tiles, then
// O^T in blocks of 128 columns of V.  Every wait is bounded.
#include "ktl_score.cuh"

namespace ktk {

constexpr int kAsTok = 64;
constexpr int kAsThreads = 192;               // 4 softmax warps, the issuing warp, the loading warp
constexpr int kAsChunk = kAsTok * 128;        // [64 tokens][64 columns]
constexpr int kAsMaxStages = 8, kAsMaxBars = 40;
constexpr int kAsSmem = 232448 - 2048;        // for Q, the ring and P; static arrays and alignment aside
constexpr int kAsMinTiles = 4;                // a split is not worth less
constexpr int kAsMaxSplits = 256, kAsStartTiles = 5;
constexpr int kAsMaxDim = 576, kAsMaxVdim = 512;
constexpr float kAsSlack = 8.0f;
constexpr float kAsNone = -1e30f;             // reference of a column without a sink

// (row, head) pairs of a CTA: `heads` heads of `rows` rows, N columns
struct Packing { int n, heads, rows, chunks; };
__host__ __device__ inline Packing packing_of(int heads, bool one_row) {
    Packing k;
    k.heads = heads < 64 ? heads : 64;
    k.chunks = (heads + k.heads - 1) / k.heads;
    k.heads = (heads + k.chunks - 1) / k.chunks;
    k.rows = one_row ? 1 : 64 / k.heads;
    const int cols = k.heads * k.rows;
    k.n = cols <= 16 ? 16 : cols <= 32 ? 32 : 64;
    return k;
}

// partial of one (row, head, split): reference, sum, O [vdim_stride]
__host__ __device__ inline int64_t as_partial_floats(int vdim_stride) { return 4 + (int64_t)vdim_stride; }

template <int N> __device__ __forceinline__ void tmem_ld_cols(uint32_t addr, float (&v)[N]) {
    if constexpr (N == 16) tmem_ld16(addr, v);
    else if constexpr (N == 32) tmem_ld32(addr, v);
    else tmem_ld64(addr, *reinterpret_cast<float (*)[32]>(&v[0]), *reinterpret_cast<float (*)[32]>(&v[32]));
}
template <int N> __device__ __forceinline__ void tmem_st_cols(uint32_t addr, const float (&v)[N]) {
    if constexpr (N == 16) tmem_st16(addr, v);
    else {
        tmem_st32(addr, *reinterpret_cast<const float (*)[32]>(&v[0]));
        if constexpr (N == 64) tmem_st32(addr + 32, *reinterpret_cast<const float (*)[32]>(&v[32]));
    }
}
__device__ __forceinline__ bool any_of_softmax_warps(bool x) {
    uint32_t r;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbar.red.or.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
        : "=r"(r) : "r"((uint32_t)x) : "memory");
    return r != 0;
}
__device__ __forceinline__ void softmax_warps_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

template <int N>
__global__ void __launch_bounds__(kAsThreads, 1)
attn_shared_kernel(const AttnParams p, const __grid_constant__ CUtensorMap k_map, const int kc, const int stages,
                   const uint32_t tmem_cols) {
    extern __shared__ uint8_t as_raw[];
    // a stage has landed; a pair of its chunks has been read out
    __shared__ __align__(8) uint64_t full[kAsMaxStages], free_[kAsMaxBars], bar_s[2], bar_p, bar_o, bar_q;
    __shared__ __align__(16) float ref_s[N], alpha_s[N];
    __shared__ __align__(16) int vis_s[N];
    __shared__ uint32_t tmem_base_s;
    __shared__ int abort_flag;
    uint8_t* sQ = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(as_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* sK = sQ + kc * (N * 128);                  // [stage][chunk]
    const int stage_bytes = kc * kAsChunk, pairs = (kc + 1) / 2;
    uint8_t* sP = sK + stages * stage_bytes;            // [64 tokens][N], rows of 128 bytes
    float* scratch = reinterpret_cast<float*>(sP);

    const ktk_attn& a = p.a;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool issuer = warp == 4, loader = warp == 5;
    const Packing pk = packing_of(a.heads, p.new_indptr == nullptr);
    const int groups = p.new_indptr ? (p.max_new + pk.rows - 1) / pk.rows : 1;
    const int b = blockIdx.z / groups, split = blockIdx.x;
    const int r0 = p.new_indptr ? p.new_indptr[b] : b, n_new = p.new_indptr ? p.new_indptr[b + 1] - r0 : 1;
    const int first = (int)(blockIdx.z % groups) * pk.rows;          // the CTA's first row within the sequence
    if (first >= n_new) return;                         // uniform for the CTA: nothing allocated yet
    const int rows = n_new - first < pk.rows ? n_new - first : pk.rows;
    const bool one = pk.rows == 1;
    const int head0 = blockIdx.y * pk.heads, heads = a.heads - head0 < pk.heads ? a.heads - head0 : pk.heads;
    const Span s = span_of(p.t, b);
    const int base = s.total - n_new;
    if (s.bad || base < 0 || s.total <= 0) {
        if (tid == 0) report(p.status, KTK_STATUS_BAD_TABLE);
        return;
    }
    const int seen = base + first + rows;               // tokens the CTA's last row sees
    const int tiles = (seen + kAsTok - 1) / kAsTok, per = (tiles + p.splits - 1) / p.splits;
    const int j0 = split * per, n = (j0 + per < tiles ? j0 + per : tiles) - j0;      // this split's tiles
    const int ps = p.t.page_size;

    if (tid == 0) {
        for (int i = 0; i < stages; ++i) mbar_init(&full[i], 1);
        for (int i = 0; i < stages * pairs; ++i) mbar_init(&free_[i], 1);
        mbar_init(&bar_s[0], 1); mbar_init(&bar_s[1], 1);
        mbar_init(&bar_p, 128);
        mbar_init(&bar_q, 128);
        mbar_init(&bar_o, 1);
        abort_flag = 0;
        mbar_init_fence();
    }
    if (issuer) tmem_alloc(&tmem_base_s, tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_base_s, tmem_o = tmem + 2 * N;
    const int vblocks = (a.vdim_stride + kUmRows - 1) / kUmRows;

    if (issuer) {
        const uint32_t idesc_s = umma_idesc_of(kAsTok, N, false, false), idesc_o = umma_idesc_of(kUmRows, N, true, true);
        const uint64_t q_desc = umma_desc(smem_u32(sQ), 0, 1024), k_desc = umma_desc(smem_u32(sK), 0, 1024);
        const uint64_t v_desc = umma_desc(smem_u32(sK), kAsChunk, 1024), p_desc = umma_desc(smem_u32(sP), 0, 1024);
        int s_at = 0, o_at = 0;                          // next tile of each product
        int s_st = 0, o_st = 0;                          // their stages
        uint32_t s_par = 0, idle = 0;
        const bool started = mbar_wait_all(&bar_q, 0, &abort_flag);
        while (started && o_at < n) {
            uint32_t ready = 0;
            if (o_at < s_at && __all_sync(0xffffffffu, mbar_test(&bar_p, o_at & 1))) ready |= 1u;
            if (s_at < n && s_at <= o_at + ((ready & 1u) ? 2 : 1) && __all_sync(0xffffffffu, mbar_test(&full[s_st], s_par))) ready |= 2u;
            if (ready & 1u) {
                tc_fence_after();
                if (elect_one()) {
                    uint64_t va = umma_desc_at(v_desc, o_st * stage_bytes);
                    uint32_t d = tmem_o;
                    for (int v = 0; v < vblocks; ++v, d += N, va = umma_desc_at(va, 2 * kAsChunk)) {
#pragma unroll
                        for (int k = 0; k < kAsTok / 16; ++k)
                            umma_f16(d, umma_desc_at(va, k * (16 * 128)), umma_desc_at(p_desc, k * (16 * 128)), idesc_o,
                                     (o_at > 0 || k > 0) ? 1u : 0u);
                        umma_commit(&free_[o_st * pairs + v]);
                    }
                    umma_commit(&bar_o);
                }
                __syncwarp();
                ++o_at;
                if (++o_st == stages) o_st = 0;
            }
            if (ready & 2u) {
                if (elect_one()) {
                    uint64_t ka = umma_desc_at(k_desc, s_st * stage_bytes), qa = q_desc;
                    const uint32_t d = tmem + (s_at & 1) * N;
                    for (int c = 0; c < kc; ++c) {       // columns past `dim` are zero in Q and in K
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            umma_f16(d, umma_desc_at(ka, k * 32), umma_desc_at(qa, k * 32), idesc_s, (c > 0 || k > 0) ? 1u : 0u);
                        ka = umma_desc_at(ka, kAsChunk);
                        qa = umma_desc_at(qa, N * 128);
                    }
                    umma_commit(&bar_s[s_at & 1]);
                    for (int v = vblocks; v < pairs; ++v) umma_commit(&free_[s_st * pairs + v]);       // no values in these
                }
                __syncwarp();
                ++s_at;
                if (++s_st == stages) { s_st = 0; s_par ^= 1u; }
            }
            if (ready) { idle = 0; continue; }
            if (++idle > (1u << 22) || ((idle & 63u) == 63u && *(volatile int*)&abort_flag)) {   // bounded, like every wait
                abort_flag = 1;
                break;
            }
        }
    } else if (loader) {
        if (lane == 0) {
            const int box = ps < kAsTok ? ps : kAsTok, pages = kAsTok / box;
            int st = 0, issued = 0;
            uint32_t par = 1;
            bool alive = true;
            prefetch_tensormap(&k_map);
            for (int i = 0; i < n && alive; ++i) {
                const int tok0 = (j0 + i) * kAsTok;
                int z[kAsTok / 16], have = 0;
#pragma unroll
                for (int k = 0; k < kAsTok / 16; ++k) {
                    z[k] = -1;
                    const int tok = tok0 + k * box;
                    if (k < pages && tok < s.total) {
                        const int pg = p.t.kv_indices[s.start + tok / ps];
                        if (pg < 0 || pg >= p.t.num_pages) report(p.status, KTK_STATUS_BAD_PAGE);
                        else { z[k] = pg; ++have; }
                    }
                }
                const uint32_t bytes = (uint32_t)(have * box * 128 * kc);
                uint64_t* bar = &full[st];
                for (int c = 0; c < kc && alive; ++c) {
                    if (i >= stages && (c & 1) == 0) alive = mbar_wait_fast(&free_[st * pairs + (c >> 1)], par, &abort_flag);
                    if (!alive) break;
                    if (c == 0) {
                        if (bytes) mbar_arrive_expect_tx(bar, bytes);
                        else mbar_arrive(bar);
                    }
                    uint8_t* dst = sK + st * stage_bytes + c * kAsChunk;
                    if (pages == 1) {
                        if (z[0] >= 0) tma_load_3d(dst, &k_map, bar, c * 64, 0, z[0]);
                    } else {
#pragma unroll
                        for (int k = 0; k < kAsTok / 16; ++k)
                            if (z[k] >= 0) tma_load_3d(dst + k * box * 128, &k_map, bar, c * 64, 0, z[k]);
                    }
                }
                if (alive) ++issued;
                if (++st == stages) { st = 0; par ^= 1u; }
            }
            if (abort_flag || !alive) {                  // the copies in flight still write shared memory
                volatile int never = 0;
                for (int i = issued > stages ? issued - stages : 0; i < issued; ++i)
                    mbar_wait(&full[i % stages], (i / stages) & 1, &never);
            }
        }
    } else {
        const uint32_t my = tmem + ((uint32_t)(warp * 32) << 16);
        // column c: row first + c / heads of the sequence, head head0 + c % heads.  Q comes while the first tiles are on their
        // way: 8 threads take a column, 16 bytes of every chunk each
        for (int c = tid; c < N; c += 128) {
            const int lr = one ? 0 : c / pk.heads, h = c - lr * pk.heads;
            const bool on = lr < rows && h < heads;
            ref_s[c] = on && p.sink ? p.sink[head0 + h] * kLog2eF : kAsNone;
            vis_s[c] = on ? base + first + lr + 1 : 0;
        }
        for (int c = tid >> 3; c < N; c += 16) {
            const int lr = one ? 0 : c / pk.heads, h = c - lr * pk.heads;
            const bool on = lr < rows && h < heads;
            const uint4* src = reinterpret_cast<const uint4*>(
                (const __nv_bfloat16*)p.q + (int64_t)(r0 + first + (on ? lr : 0)) * p.q_stride +
                (int64_t)(head0 + (on ? h : 0)) * a.dim_stride) + (tid & 7);
            uint4 v[kAsMaxDim / 64];
#pragma unroll
            for (int k = 0; k < kAsMaxDim / 64; ++k)
                v[k] = on && k * 64 + (tid & 7) * 8 < a.dim_stride ? __ldg(src + k * 8) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
            for (int k = 0; k < kAsMaxDim / 64; ++k)
                if (k < kc) *reinterpret_cast<uint4*>(sQ + k * (N * 128) + swz(c, tid & 7)) = v[k];
        }
        fence_proxy_async();
        mbar_arrive(&bar_q);
        softmax_warps_sync();
        // a thread holds two tokens of the tile and, of every 8 columns, the two from 2 (lane % 4) on
        const int tok = warp * 16 + (lane >> 2), col = 2 * (lane & 3);
        const float f = a.scale * kLog2eF;
        const int clean_end = base + first + 1;          // tokens before this are seen by every row of the CTA
        float l[N / 4];
#pragma unroll
        for (int c = 0; c < N / 4; ++c) l[c] = 0.0f;
        // waits that ran out raise abort_flag; the loop still runs to its end, so that no warp misses a barrier
        for (int j = 0; j < n; ++j) {
            const int at = (j0 + j) * kAsTok + tok;
            mbar_wait_all(&bar_s[j & 1], (j >> 1) & 1, &abort_flag);
            tc_fence_after();
            uint32_t raw[N / 2];
            RowPairs<N / 8>::load(my + (j & 1) * N, raw);
            float t[N / 2];
            bool over = false;
            const bool clean = (j0 + j + 1) * kAsTok <= clean_end;
#pragma unroll
            for (int k = 0; k < N / 8; ++k) {
                const float2 r = *reinterpret_cast<const float2*>(ref_s + 8 * k + col);
                const int2 v = clean ? make_int2(0x7fffffff, 0x7fffffff) : *reinterpret_cast<const int2*>(vis_s + 8 * k + col);
                t[4 * k] = at < v.x ? __uint_as_float(raw[4 * k]) * f : -INFINITY;
                t[4 * k + 1] = at < v.y ? __uint_as_float(raw[4 * k + 1]) * f : -INFINITY;
                t[4 * k + 2] = at + 8 < v.x ? __uint_as_float(raw[4 * k + 2]) * f : -INFINITY;
                t[4 * k + 3] = at + 8 < v.y ? __uint_as_float(raw[4 * k + 3]) * f : -INFINITY;
                over |= fmaxf(t[4 * k], t[4 * k + 2]) > r.x + kAsSlack || fmaxf(t[4 * k + 1], t[4 * k + 3]) > r.y + kAsSlack;
            }
            const bool move = any_of_softmax_warps(over || j == 0);
            if (j > 0) mbar_wait_all(&bar_o, (j - 1) & 1, &abort_flag);       // P and O of the previous tile are settled
            if (move) {
                // some reference moves: every column's largest score of the tile, then O and the sums are rescaled
#pragma unroll
                for (int k = 0; k < N / 8; ++k)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        float mx = fmaxf(t[4 * k + e], t[4 * k + 2 + e]);
#pragma unroll
                        for (int o = 4; o <= 16; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                        if (lane < 4) scratch[warp * N + 8 * k + col + e] = mx;
                    }
                softmax_warps_sync();
                for (int c = tid; c < N; c += 128) {
                    const float old = ref_s[c];
                    const float mx = fmaxf(fmaxf(scratch[c], scratch[N + c]), fmaxf(scratch[2 * N + c], scratch[3 * N + c]));
                    const float now = fmaxf(mx, old);
                    ref_s[c] = now;
                    alpha_s[c] = ex2(old - now);
                }
                softmax_warps_sync();
                tc_fence_after();
#pragma unroll
                for (int k = 0; k < N / 8; ++k) {
                    const float2 al = *reinterpret_cast<const float2*>(alpha_s + 8 * k + col);
                    l[2 * k] *= al.x;
                    l[2 * k + 1] *= al.y;
                }
                if (j > 0)
                    for (int v = 0; v < vblocks; ++v) {
                        float o[N];
                        tmem_ld_cols<N>(my + 2 * N + v * N, o);
#pragma unroll
                        for (int c = 0; c < N; ++c) o[c] *= alpha_s[c];
                        tmem_st_cols<N>(my + 2 * N + v * N, o);
                    }
                tmem_st_wait();
            }
#pragma unroll
            for (int k = 0; k < N / 8; ++k) {
                const float2 r = *reinterpret_cast<const float2*>(ref_s + 8 * k + col);
                const float p0 = ex2(t[4 * k] - r.x), p1 = ex2(t[4 * k + 1] - r.y);
                const float p2 = ex2(t[4 * k + 2] - r.x), p3 = ex2(t[4 * k + 3] - r.y);
                l[2 * k] += p0 + p2;
                l[2 * k + 1] += p1 + p3;
                *reinterpret_cast<uint32_t*>(sP + swz(tok, k) + 2 * col) = pack_bf16(p0, p1);
                *reinterpret_cast<uint32_t*>(sP + swz(tok + 8, k) + 2 * col) = pack_bf16(p2, p3);
            }
            const int left = s.total - (j0 + j) * kAsTok;
            if (left < kAsTok && lane < 16 && warp * 16 + lane >= left) {
                // rows behind the sequence may hold anything: 0 * x has to stay 0
                uint8_t* st = sK + (j % stages) * stage_bytes;
                for (int c = 0; c < kc * 8; ++c)
                    *reinterpret_cast<uint4*>(st + (c >> 3) * kAsChunk + swz(warp * 16 + lane, c & 7)) = make_uint4(0u, 0u, 0u, 0u);
            }
            fence_proxy_async();
            tc_fence_before();
            mbar_arrive(&bar_p);
        }
        if (n > 0) mbar_wait_all(&bar_o, (n - 1) & 1, &abort_flag);
        tc_fence_after();
        // ---- sums over the tokens, then O^T: lane = column of V, register = (row, head)
#pragma unroll
        for (int k = 0; k < N / 8; ++k)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float v = l[2 * k + e];
#pragma unroll
                for (int o = 4; o <= 16; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                if (lane < 4) scratch[warp * N + 8 * k + col + e] = v;
            }
        softmax_warps_sync();
        for (int c = tid; c < N; c += 128) {
            float L = scratch[c] + scratch[N + c] + scratch[2 * N + c] + scratch[3 * N + c];
            const int lr = one ? 0 : c / pk.heads, h = head0 + c - lr * pk.heads;
            if (c - lr * pk.heads < heads && lr < rows) {
                const int64_t row = r0 + first + lr;
                if (p.splits > 1) {
                    float* w = p.ws + ((row * a.heads + h) * p.splits + split) * as_partial_floats(a.vdim_stride);
                    w[0] = ref_s[c];
                    w[1] = L;
                } else {
                    if (p.sink) L += ex2(p.sink[h] * kLog2eF - ref_s[c]);
                    float g = L > 0.0f ? 1.0f / L : 0.0f;
                    if (p.gate) g *= sigmoid_f(to_f32(((const __nv_bfloat16*)p.gate)[row * p.gate_stride + h]));
                    alpha_s[c] = g;
                }
            }
        }
        softmax_warps_sync();
        if (n > 0 && !abort_flag) {
            for (int v = 0; v < vblocks; ++v) {
                float o[N];
                tmem_ld_cols<N>(my + 2 * N + v * N, o);
                const int col = v * kUmRows + tid;
#pragma unroll
                for (int c = 0; c < N; ++c) {
                    if (col >= a.vdim_stride) break;
                    const int lr = one ? 0 : c / pk.heads, h = head0 + c - lr * pk.heads;
                    if (c - lr * pk.heads >= heads || lr >= rows) continue;
                    const int64_t row = r0 + first + lr;
                    if (p.splits > 1)
                        p.ws[((row * a.heads + h) * p.splits + split) * as_partial_floats(a.vdim_stride) + 4 + col] = o[c];
                    else
                        ((__nv_bfloat16*)p.o)[(row * a.heads + h) * a.vdim_stride + col] =
                            __float2bfloat16_rn(col < a.vdim ? o[c] * alpha_s[c] : 0.0f);
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
        tmem_free(tmem, tmem_cols);
    }
}

// One CTA per (head, row): merges the splits, adds the sink, applies the gate.
__global__ void __launch_bounds__(128) attn_shared_combine_kernel(const AttnParams p) {
    __shared__ float weight[kAsMaxSplits];
    const ktk_attn& a = p.a;
    const int64_t row = blockIdx.y;
    const int head = blockIdx.x;
    const int64_t stride = as_partial_floats(a.vdim_stride);
    const float* w = p.ws + (row * a.heads + head) * p.splits * stride;
    const float sk = p.sink ? p.sink[head] * kLog2eF : kAsNone;
    // every warp reads all the splits' references and sums, a lane some of them
    const int lane = threadIdx.x & 31;
    float M = sk, L = 0.0f;
    for (int s = lane; s < p.splits; s += 32) {
        const float2 ml = *reinterpret_cast<const float2*>(w + s * stride);
        if (ml.y > 0.0f) M = fmaxf(M, ml.x);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    for (int s = lane; s < p.splits; s += 32) {
        const float2 ml = *reinterpret_cast<const float2*>(w + s * stride);
        const float f = ml.y > 0.0f ? ex2(ml.x - M) : 0.0f;
        L += f * ml.y;
        if (threadIdx.x < 32) weight[s] = f;
    }
    L = warp_sum_f(L);
    __syncthreads();
    if (p.sink) L += ex2(sk - M);
    float g = L > 0.0f ? 1.0f / L : 0.0f;
    if (p.gate) g *= sigmoid_f(to_f32(((const __nv_bfloat16*)p.gate)[row * p.gate_stride + head]));
    __nv_bfloat16* o = (__nv_bfloat16*)p.o + (row * a.heads + head) * a.vdim_stride;
    for (int c = threadIdx.x * 4; c < a.vdim_stride; c += 512) {
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 4
        for (int s = 0; s < p.splits; ++s) {
            const float f = weight[s];
            if (f == 0.0f) continue;                     // an empty split has written no columns
            const float4 x = *reinterpret_cast<const float4*>(w + s * stride + 4 + c);
            v.x += f * x.x; v.y += f * x.y; v.z += f * x.z; v.w += f * x.w;
        }
        uint2 r;
        r.x = pack_bf16(c < a.vdim ? v.x * g : 0.0f, c + 1 < a.vdim ? v.y * g : 0.0f);
        r.y = pack_bf16(c + 2 < a.vdim ? v.z * g : 0.0f, c + 3 < a.vdim ? v.w * g : 0.0f);
        *reinterpret_cast<uint2*>(o + c) = r;
    }
}

static int shared_stages(const ktk_attn& a, int n) {
    const int kc = (a.dim_stride + 63) / 64, fixed = kc * n * 128 + kAsTok * 128;
    int fit = (kAsSmem - fixed) / (kc * kAsChunk);
    if (fit > kAsMaxBars / kc) fit = kAsMaxBars / kc;
    return fit < kAsMaxStages ? fit : kAsMaxStages;
}

bool attn_shared_supported(const ktk_attn& a) {
    return a.dtype == KTK_BF16 && a.maps == 1 && a.kv_heads == 1 && a.v_row_stride == a.dim_stride && a.softcap == 0.0f &&
           a.temp_coef == 0.0f && a.dim_stride <= kAsMaxDim && a.vdim_stride <= kAsMaxVdim && shared_stages(a, 64) >= 2;
}

// new_rows: 0 for one row of each of `batch` sequences, else the rows of one sequence
int32_t attn_shared_splits(const ktk_attn& a, int batch, int new_rows, int64_t max_keys) {
    const Packing k = packing_of(a.heads, new_rows == 0);
    const int64_t units = (int64_t)batch * k.chunks * (new_rows == 0 ? 1 : (new_rows + k.rows - 1) / k.rows);
    const int64_t tiles = (max_keys + kAsTok - 1) / kAsTok;
    // rounds of CTAs x (tiles of each + what starting and finishing one costs, in tiles)
    int64_t most = (tiles + kAsMinTiles - 1) / kAsMinTiles, best = 1, best_cost = -1;
    if (most > kAsMaxSplits) most = kAsMaxSplits;
    for (int64_t s = 1; s <= most && units > 0; ++s) {
        const int64_t rounds = (units * s + sm_count() - 1) / sm_count();
        const int64_t cost = rounds * ((tiles + s - 1) / s + kAsStartTiles) + (s > 1 ? kAsStartTiles : 0);
        if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = s; }
        if (rounds > 8) break;
    }
    return (int32_t)best;
}

size_t attn_shared_workspace(const ktk_attn& a, int64_t rows, int splits) {
    return splits <= 1 ? 0 : (size_t)rows * a.heads * splits * as_partial_floats(a.vdim_stride) * sizeof(float);
}

template <int N> static int shared_launch(const AttnParams& p, const Packing& k, cudaStream_t st) {
    const char* who = "ktk_paged_attention";
    const ktk_attn& a = p.a;
    const uint64_t ps = p.t.page_size;
    const uint64_t kd[3] = {(uint64_t)a.dim_stride, ps, (uint64_t)p.t.num_pages};
    const uint64_t ks[2] = {(uint64_t)a.dim_stride * 2, ps * a.dim_stride * 2};
    const uint32_t box[3] = {64, (uint32_t)(ps < kAsTok ? ps : kAsTok), 1};
    CUtensorMap km;
    const int rc = make_tensor_map_3d(&km, p.k, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, kd, ks, box, CU_TENSOR_MAP_SWIZZLE_128B, who);
    if (rc != KTK_OK) return rc;
    const int kc = (a.dim_stride + 63) / 64, stages = shared_stages(a, N), vblocks = (a.vdim_stride + kUmRows - 1) / kUmRows;
    const int smem = kc * N * 128 + stages * kc * kAsChunk + kAsTok * 128 + 1024;
    uint32_t cols = 32;
    while (cols < (uint32_t)((2 + vblocks) * N)) cols *= 2;
    const int64_t groups = p.new_indptr ? (p.max_new + k.rows - 1) / k.rows : 1;
    if (groups * p.t.batch > 65535) {
        set_error("%s: more than 65535 groups of rows in one launch", who);
        return KTK_ERR_TOO_LARGE;
    }
    KTK_CUDA_TRY(cudaFuncSetAttribute(attn_shared_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), who);
    const dim3 grid((unsigned)p.splits, (unsigned)k.chunks, (unsigned)(groups * p.t.batch));
    attn_shared_kernel<N><<<grid, kAsThreads, smem, st>>>(p, km, kc, stages, cols);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    if (p.splits > 1) {
        attn_shared_combine_kernel<<<dim3((unsigned)a.heads, (unsigned)p.rows), 128, 0, st>>>(p);
        KTK_CUDA_TRY(cudaGetLastError(), who);
    }
    return KTK_OK;
}

int launch_attn_shared(const AttnParams& p, cudaStream_t st) {
    if (p.splits > kAsMaxSplits || (p.splits > 1 && p.rows > 65535)) {
        set_error("ktk_paged_attention: %d splits of %lld rows", p.splits, (long long)p.rows);
        return KTK_ERR_TOO_LARGE;
    }
    if (p.new_indptr && p.max_new <= 0) return KTK_OK;
    const Packing k = packing_of(p.a.heads, p.new_indptr == nullptr);
    return k.n == 16 ? shared_launch<16>(p, k, st) : k.n == 32 ? shared_launch<32>(p, k, st) : shared_launch<64>(p, k, st);
}

}  // namespace ktk
