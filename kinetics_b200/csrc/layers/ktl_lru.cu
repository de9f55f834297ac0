// A linear recurrence with real gates behind a short causal convolution, per channel (see ktk_layers.h), over a
// sequence's next tokens or one token of every sequence.  State, gates and decays are fp32.
//
// The convolution keeps its newest `taps` inputs in a ring by position: a step writes the place of the input that has
// just left the window, which nobody reads.  The prompt's scan is one pass over its inputs: the CTAs of a cluster take
// consecutive tiles of tokens and exchange the tiles' products and end states through distributed shared memory.
#include "../ktk_umma.cuh"
#include "ktl_common.cuh"

namespace ktk {

constexpr int kLcThreads = 64;
constexpr int kLcChunk = 16;            // tokens per thread of the convolution
constexpr int kLsWarps = 8, kLsRun = 8;  // warps of a scan CTA, tokens of a warp
constexpr int kLsThreads = kLsWarps * 32, kLsTile = kLsWarps * kLsRun, kLsMaxCluster = 8;
constexpr int kLdThreads = 128;

// what a sequence runs now: rows [row0, row0 + n), of positions base ..; false if the table or the slot is malformed
struct Run { int64_t row0; int n, base, slot; };
__device__ __forceinline__ bool run_of(const ktk_paged& t, const int32_t* new_indptr, const int32_t* slots, int64_t num_slots,
                                       int b, int32_t* status, Run& r) {
    const Span s = span_of(t, b);
    r.row0 = new_indptr ? new_indptr[b] : b;
    r.n = new_indptr ? new_indptr[b + 1] - new_indptr[b] : 1;
    r.base = s.total - r.n;
    r.slot = slots[b];
    const bool ok = !s.bad && r.base >= 0 && r.slot >= 0 && r.slot < num_slots;
    if (!ok && threadIdx.x == 0) report(status, KTK_STATUS_BAD_TABLE);
    return ok;
}

// Thread: 8 channels of `chunk` tokens.  TAPS > 0: the window stays in registers; 0: any number of taps.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kLcThreads)
lru_conv_kernel(const T* __restrict__ x, int64_t row_stride, const int32_t* __restrict__ new_indptr,
                const int32_t* __restrict__ slots, int64_t num_slots, const float* __restrict__ w, const float* __restrict__ bias,
                T* ring, T* __restrict__ u, const ktk_paged t, int width, int taps_any, int chunk, int32_t* status) {
    Run r;
    if (!run_of(t, new_indptr, slots, num_slots, blockIdx.z, status, r)) return;
    const int taps = TAPS > 0 ? TAPS : taps_any;
    const int c = (blockIdx.x * kLcThreads + threadIdx.x) * 8;
    const int t0 = blockIdx.y * chunk, t1 = t0 + chunk < r.n ? t0 + chunk : r.n;
    if (c >= width || t0 >= r.n) return;
    T* mine = ring + (int64_t)r.slot * taps * width + c;
    auto input = [&](int i, float (&v)[8]) {              // input of token i of the run (i < 0: an earlier one)
        if (i >= 0) Vec8<T>::load(x + (r.row0 + i) * row_stride + c, v);
        else if (r.base + i >= 0) Vec8<T>::load(mine + (int64_t)((r.base + i) % taps) * width, v);
        else {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = 0.0f;
        }
    };
    float b8[8];
    load8(bias + c, b8);
    if (TAPS > 0) {
        float win[TAPS > 0 ? TAPS : 1][8], wt[TAPS > 0 ? TAPS : 1][8];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) {
            load8(w + (int64_t)k * width + c, wt[k]);
            if (k + 1 < TAPS) input(t0 - (TAPS - 1) + k, win[k]);
        }
#pragma unroll 4
        for (int i = t0; i < t1; ++i) {
            input(i, win[TAPS > 0 ? TAPS - 1 : 0]);
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = b8[e];
#pragma unroll
            for (int k = 0; k < TAPS; ++k)
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    o[e] = fmaf(wt[k][e], win[k][e], o[e]);
                    if (k > 0) win[k - 1][e] = win[k][e];
                }
            Vec8<T>::store(u + (r.row0 + i) * width + c, o);
        }
    } else {
        for (int i = t0; i < t1; ++i) {
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = b8[e];
            for (int k = 0; k < taps; ++k) {
                float v[8], wk[8];
                input(i - (taps - 1) + k, v);
                load8(w + (int64_t)k * width + c, wk);
#pragma unroll
                for (int e = 0; e < 8; ++e) o[e] = fmaf(wk[e], v[e], o[e]);
            }
            Vec8<T>::store(u + (r.row0 + i) * width + c, o);
        }
    }
    // the first chunk's thread is the only one that reads this ring (a chunk has at least `taps` tokens): it also writes
    if (t0 == 0)
        for (int i = r.n > taps ? r.n - taps : 0; i < r.n; ++i) {
            float v[8];
            Vec8<T>::load(x + (r.row0 + i) * row_stride + c, v);
            Vec8<T>::store(mine + (int64_t)((r.base + i) % taps) * width, v);
        }
}

// ---- gates and the recurrence ----
// the float that CTA `cta` of the cluster keeps at the place of *p
__device__ __forceinline__ float peer_f32(const float* p, uint32_t cta) {
    uint32_t at;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"(smem_u32(p)), "r"(cta));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(at) : "memory");
    return v;
}
__device__ __forceinline__ float sqrt_approx(float x) {
    float y;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
template <bool FAST> __device__ __forceinline__ float exp_of(float x) { return FAST ? __expf(x) : expf(x); }
template <bool FAST> __device__ __forceinline__ float sigmoid_of(float x) {
    return FAST ? __fdividef(1.0f, 1.0f + __expf(-x)) : 1.0f / (1.0f + expf(-x));
}
// 1 - exp(-x), x >= 0: the series where the difference would cancel
__device__ __forceinline__ float one_minus_exp(float x, float e) {
    const float s = x * (1.0f + x * (-0.5f + x * (1.0f / 6.0f + x * (-1.0f / 24.0f + x * (1.0f / 120.0f - x * (1.0f / 720.0f))))));
    return x < 0.3f ? s : 1.0f - e;
}
// one token of one channel: S <- a S + g
template <bool FAST>
__device__ __forceinline__ void gates(float zr, float zi, float u, float rb, float ib, float decay, float& a, float& g) {
    const float x = sigmoid_of<FAST>(zr + rb) * decay;                    // -log a
    a = exp_of<FAST>(-x);
    g = (FAST ? sqrt_approx(one_minus_exp(2.0f * x, a * a)) : sqrtf(-expm1f(-2.0f * x))) * sigmoid_of<FAST>(zi + ib) * u;
}
// 0.5 y (1 + tanh z) = y / (1 + exp(-2 z)),  z = sqrt(2 / pi) (y + 0.044715 y^3)
template <bool FAST> __device__ __forceinline__ float gelu_tanh(float y) {
    const float z2 = 2.0f * 0.7978845608028654f * (y + 0.044715f * y * y * y);
    return FAST ? __fdividef(y, 1.0f + __expf(fminf(-z2, 80.0f))) : y / (1.0f + expf(-z2));
}

struct LruParams {
    ktk_lru a;
    ktk_paged t;
    const float* z;
    const void *u, *y;
    int64_t row_stride;
    const int32_t *new_indptr, *slots;
    int64_t num_slots, rows;
    int max_new;
    const float *rb, *ib, *decay;
    float* state;
    void* out;
    int32_t* status;
};

// 32 channels of one sequence: lane = channel, a warp runs 8 consecutive tokens, a CTA 64, the CTAs of a cluster consecutive
// tiles of 64.  Per round of the cluster: local products and end states, joined over the CTA's warps in shared memory and
// over the cluster's CTAs through theirs; then every warp replays its tokens from the state in front of them.
template <typename T>
__global__ void __launch_bounds__(kLsThreads, 4) lru_scan_kernel(const LruParams p) {
    constexpr bool FAST = sizeof(T) == 2;
    // by parity of the round, so that a round needs no barrier behind its last reads
    __shared__ float warp_a[2][kLsWarps][32], warp_s[2][kLsWarps][32], tile_a[2][32], tile_s[2][32], before[2][32];
    Run r;
    if (!run_of(p.t, p.new_indptr, p.slots, p.num_slots, blockIdx.z, p.status, r)) return;      // uniform for the cluster
    const int ctas = gridDim.x, rank = blockIdx.x;
    const int bs = p.a.block_stride, width = p.a.blocks * bs;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int c = blockIdx.y * 32 + lane;
    const bool on = c < width;
    const int blk = on ? c / bs : 0, cc = on ? c - blk * bs : 0;
    const float* z = p.z + ((int64_t)blk * p.rows + r.row0) * (2 * bs) + cc;
    const T* u = (const T*)p.u + r.row0 * width + (on ? c : 0);
    const T* y = (const T*)p.y + r.row0 * p.row_stride + (on ? c : 0);
    T* out = (T*)p.out + r.row0 * width + c;
    const float rb = on ? p.rb[c] : 0.0f, ib = on ? p.ib[c] : 0.0f, decay = on ? p.decay[c] : 0.0f;
    float carry = on && r.base > 0 ? p.state[(int64_t)r.slot * width + c] : 0.0f;      // behind the previous round
    const int rounds = (r.n + ctas * kLsTile - 1) / (ctas * kLsTile);
    for (int it = 0; it < rounds; ++it) {
        const int par = it & 1, i0 = (it * ctas + rank) * kLsTile + warp * kLsRun;
        float a[kLsRun], g[kLsRun], A = 1.0f, S = 0.0f;
        {
            float zr[kLsRun], zi[kLsRun];
            T uu[kLsRun];
#pragma unroll
            for (int k = 0; k < kLsRun; ++k) {
                const bool have = on && i0 + k < r.n;
                const int64_t i = have ? i0 + k : 0;
                zr[k] = have ? __ldcs(z + i * (2 * bs)) : 0.0f;
                zi[k] = have ? __ldcs(z + i * (2 * bs) + bs) : 0.0f;
                uu[k] = u[i * width];
            }
#pragma unroll
            for (int k = 0; k < kLsRun; ++k) {
                gates<FAST>(zr[k], zi[k], to_f32(uu[k]), rb, ib, decay, a[k], g[k]);
                if (!(on && i0 + k < r.n)) { a[k] = 1.0f; g[k] = 0.0f; }
                A *= a[k];
                S = fmaf(a[k], S, g[k]);
            }
        }
        warp_a[par][warp][lane] = A;
        warp_s[par][warp][lane] = S;
        T yy[kLsRun];                                      // in flight over the barriers
#pragma unroll
        for (int k = 0; k < kLsRun; ++k) yy[k] = y[(on && i0 + k < r.n ? (int64_t)(i0 + k) : 0) * p.row_stride];
        __syncthreads();
        if (warp == 0) {
            A = 1.0f; S = 0.0f;
#pragma unroll
            for (int w = 0; w < kLsWarps; ++w) {
                const float wa = warp_a[par][w][lane];
                S = fmaf(wa, S, warp_s[par][w][lane]);
                A *= wa;
            }
            tile_a[par][lane] = A;
            tile_s[par][lane] = S;
        }
        cluster_sync();
        if (warp == 0) {
            float mine = carry;
            for (int k = 0; k < ctas; ++k) {
                if (k == rank) mine = carry;
                carry = fmaf(peer_f32(&tile_a[par][lane], k), carry, peer_f32(&tile_s[par][lane], k));
            }
            before[par][lane] = mine;
        }
        __syncthreads();
        S = before[par][lane];
        for (int w = 0; w < warp; ++w) S = fmaf(warp_a[par][w][lane], S, warp_s[par][w][lane]);
#pragma unroll
        for (int k = 0; k < kLsRun; ++k) {
            S = fmaf(a[k], S, g[k]);
            if (on && i0 + k < r.n) out[(int64_t)(i0 + k) * width] = from_f32<T>(S * gelu_tanh<FAST>(to_f32(yy[k])));
        }
    }
    if (warp == 0 && rank == 0 && on) p.state[(int64_t)r.slot * width + c] = carry;
    cluster_sync();                                        // no CTA leaves while another may read its totals
}

// One token of every sequence: a thread per channel.
template <typename T>
__global__ void __launch_bounds__(kLdThreads) lru_step_kernel(const LruParams p) {
    constexpr bool FAST = sizeof(T) == 2;
    Run r;
    if (!run_of(p.t, nullptr, p.slots, p.num_slots, blockIdx.y, p.status, r)) return;
    const int bs = p.a.block_stride, width = p.a.blocks * bs;
    const int c = blockIdx.x * kLdThreads + threadIdx.x;
    if (c >= width) return;
    const int blk = c / bs, cc = c - blk * bs;
    const float* z = p.z + ((int64_t)blk * p.rows + r.row0) * (2 * bs) + cc;
    float* state = p.state + (int64_t)r.slot * width + c;
    float a, g;
    gates<FAST>(z[0], z[bs], to_f32(((const T*)p.u)[r.row0 * width + c]), p.rb[c], p.ib[c], p.decay[c], a, g);
    const float S = fmaf(a, r.base > 0 ? *state : 0.0f, g);
    *state = S;
    ((T*)p.out)[r.row0 * width + c] = from_f32<T>(S * gelu_tanh<FAST>(to_f32(((const T*)p.y)[r.row0 * p.row_stride + c])));
}

// ---- one token of every sequence in one launch: convolution, gate products on the tensor cores, recurrence, output gate ----
// A CTA takes 32 channels of a block and up to 32 rows.  It convolves all channels of the block (the products need them;
// their inputs lie in L2), multiplies u [32 x block] with the 32 + 32 gate rows by mma.m16n8k16, and finishes its channels.
// The ring's place that a step writes is read by no other CTA.
constexpr int kLfRows = 32, kLfChan = 32, kLfThreads = 256, kLfMaxBlock = 512;

__host__ __device__ inline int lf_ld(int block_stride) { return (block_stride + 15) / 16 * 16 + 8; }      // padded: no bank conflicts
__host__ __device__ inline int lf_smem(int block_stride) { return (kLfRows + 2 * kLfChan) * lf_ld(block_stride) * 2 + kLfRows * (2 * kLfChan + 1) * 4; }

struct LruDecodeParams {
    LruParams p;
    const __nv_bfloat16 *x, *gates;
    const float *conv_w, *conv_b;
    __nv_bfloat16* ring;
};

template <int TAPS> __global__ void __launch_bounds__(kLfThreads) lru_decode_kernel(const LruDecodeParams q) {
    extern __shared__ __align__(16) uint8_t lf_raw[];
    __shared__ int row_slot[kLfRows], row_pos[kLfRows];
    const LruParams& p = q.p;
    const int bs = p.a.block_stride, taps = p.a.taps, width = p.a.blocks * bs, ld = lf_ld(bs);
    __nv_bfloat16* su = reinterpret_cast<__nv_bfloat16*>(lf_raw);       // [rows][ld]
    __nv_bfloat16* sw = su + kLfRows * ld;                              // [32 rows of r, 32 of i][ld]
    float* sz = reinterpret_cast<float*>(sw + 2 * kLfChan * ld);            // [rows][32 zr | 32 zi | pad]
    constexpr int kZ = 2 * kLfChan + 1;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slices = (bs + kLfChan - 1) / kLfChan, blk = blockIdx.x / slices, n0 = (blockIdx.x - blk * slices) * kLfChan;
    const int64_t r0 = (int64_t)blockIdx.y * kLfRows;
    const int rows = p.rows - r0 < kLfRows ? (int)(p.rows - r0) : kLfRows;
    const int c0 = blk * bs, pieces = (ld - 8) / 8;                     // 16-byte pieces of a row
    // gate weights on their way; rows and columns outside are zero
    for (int i = tid; i < 2 * kLfChan * pieces; i += kLfThreads) {
        const int n = i / pieces, k = i - n * pieces, c = n0 + (n & (kLfChan - 1));
        const bool on = c < bs && k * 8 < bs;
        const __nv_bfloat16* src = q.gates + (on ? ((int64_t)(2 * blk + n / kLfChan) * bs + c) * bs + k * 8 : 0);
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(sw + n * ld + k * 8)), "l"(src),
                     "r"(on ? 16u : 0u) : "memory");
    }
    if (tid < kLfRows) {
        int slot = -1, pos = 0;
        if (tid < rows) {
            const Span s = span_of(p.t, (int)(r0 + tid));
            slot = p.slots[r0 + tid];
            pos = s.total - 1;
            if (s.bad || pos < 0 || slot < 0 || slot >= p.num_slots) {
                report(p.status, KTK_STATUS_BAD_TABLE);
                slot = -1;
            }
        }
        row_slot[tid] = slot;
        row_pos[tid] = pos;
    }
    __syncthreads();
    // u of every channel of the block: kBatch pieces per thread with all their loads in flight
    constexpr int kBatch = TAPS > 0 ? 4 : 1, kTaps = TAPS > 0 ? TAPS : 1;
    for (int i0 = tid; i0 < kLfRows * pieces; i0 += kLfThreads * kBatch) {
        uint4 raw[kBatch][kTaps];
#pragma unroll
        for (int b = 0; b < kBatch; ++b) {
            const int i = i0 + b * kLfThreads, r = i / pieces, k = i - r * pieces;
            const bool on = i < kLfRows * pieces && row_slot[r & (kLfRows - 1)] >= 0 && k * 8 < bs;
            const int slot = on ? row_slot[r] : 0, pos = on ? row_pos[r] : 0, c = c0 + k * 8;
            const __nv_bfloat16* mine = q.ring + (int64_t)slot * taps * width + c;
#pragma unroll
            for (int t = 0; t < kTaps; ++t) {                           // the last is the token's own
                const int at = pos - (kTaps - 1) + t;
                raw[b][t] = make_uint4(0u, 0u, 0u, 0u);                 // zeros before the sequence
                if (t == kTaps - 1) { if (on) raw[b][t] = *reinterpret_cast<const uint4*>(q.x + (r0 + r) * p.row_stride + c); }
                else if (on && at >= 0) raw[b][t] = *reinterpret_cast<const uint4*>(mine + (int64_t)(at % taps) * width);
            }
        }
#pragma unroll
        for (int b = 0; b < kBatch; ++b) {
            const int i = i0 + b * kLfThreads, r = i / pieces, k = i - r * pieces, c = c0 + k * 8;
            if (i >= kLfRows * pieces) continue;
            float o[8] = {0, 0, 0, 0, 0, 0, 0, 0};
            if (row_slot[r] >= 0 && k * 8 < bs) {
                __nv_bfloat16* mine = q.ring + (int64_t)row_slot[r] * taps * width + c;
                float v[8], w[8];
                load8(q.conv_b + c, o);
                if (TAPS == 0)
                    for (int t = 0; t + 1 < taps; ++t) {
                        const int at = row_pos[r] - (taps - 1) + t;
                        if (at < 0) continue;
                        Vec8<__nv_bfloat16>::load(mine + (int64_t)(at % taps) * width, v);
                        load8(q.conv_w + (int64_t)t * width + c, w);
#pragma unroll
                        for (int e = 0; e < 8; ++e) o[e] = fmaf(w[e], v[e], o[e]);
                    }
#pragma unroll
                for (int t = 0; t < kTaps; ++t) {
                    unpack8(raw[b][t], v);
                    load8(q.conv_w + (int64_t)(taps - kTaps + t) * width + c, w);
#pragma unroll
                    for (int e = 0; e < 8; ++e) o[e] = fmaf(w[e], v[e], o[e]);
                }
                if (k * 8 >= n0 && k * 8 < n0 + kLfChan)                 // this CTA's channels
                    *reinterpret_cast<uint4*>(mine + (int64_t)(row_pos[r] % taps) * width) = raw[b][kTaps - 1];
            }
            Vec8<__nv_bfloat16>::store(su + r * ld + k * 8, o);
        }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    {
        // warp: 16 rows, 16 of the 64 columns
        const int gid = lane >> 2, tig = lane & 3, m0 = (warp & 1) * 16, g0 = (warp >> 1) * 16;
        float acc[2][4] = {};
        const __nv_bfloat16* a0 = su + (m0 + gid) * ld + 2 * tig;
        const __nv_bfloat16* b0 = sw + (g0 + gid) * ld + 2 * tig;
#pragma unroll 4
        for (int k = 0; k < ld - 8; k += 16) {
            uint32_t a[4];
            a[0] = *reinterpret_cast<const uint32_t*>(a0 + k);
            a[1] = *reinterpret_cast<const uint32_t*>(a0 + 8 * ld + k);
            a[2] = *reinterpret_cast<const uint32_t*>(a0 + k + 8);
            a[3] = *reinterpret_cast<const uint32_t*>(a0 + 8 * ld + k + 8);
#pragma unroll
            for (int t = 0; t < 2; ++t)
                mma_bf16(acc[t], a, *reinterpret_cast<const uint32_t*>(b0 + t * 8 * ld + k),
                         *reinterpret_cast<const uint32_t*>(b0 + t * 8 * ld + k + 8));
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) sz[(m0 + gid + (e >= 2 ? 8 : 0)) * kZ + g0 + t * 8 + 2 * tig + (e & 1)] = acc[t][e];
    }
    __syncthreads();
    const int n = n0 + lane, c = c0 + n;
    if (n >= bs) return;
    const float rb = p.rb[c], ib = p.ib[c], decay = p.decay[c];
#pragma unroll
    for (int r = warp; r < kLfRows; r += kLfThreads / 32) {
        const int slot = row_slot[r];
        if (slot < 0) continue;
        float* state = p.state + (int64_t)slot * width + c;
        float a, g;
        gates<true>(sz[r * kZ + lane], sz[r * kZ + kLfChan + lane], __bfloat162float(su[r * ld + n]), rb, ib, decay, a, g);
        const float S = fmaf(a, row_pos[r] > 0 ? *state : 0.0f, g);
        *state = S;
        ((__nv_bfloat16*)p.out)[(r0 + r) * width + c] =
            __float2bfloat16_rn(S * gelu_tanh<true>(__bfloat162float(((const __nv_bfloat16*)p.y)[(r0 + r) * p.row_stride + c])));
    }
}

static int check_lru(const ktk_lru* a, const ktk_paged* t, const int32_t* new_indptr, int64_t rows, int32_t max_new,
                     int64_t row_stride, int64_t col, int64_t num_slots, const char* who) {
    if (a == nullptr || t == nullptr || a->blocks <= 0 || a->block <= 0 || a->block_stride < a->block ||
        a->block_stride % 8 != 0 || a->taps <= 0 || a->taps > 1024 || (a->dtype != KTK_F32 && a->dtype != KTK_BF16) ||
        (int64_t)a->blocks * a->block_stride > (1 << 20) || t->page_size <= 0 || t->batch < 0 || t->batch > 65535) {
        set_error("%s: bad sizes", who);
        return KTK_ERR_ARG;
    }
    const int width = a->blocks * a->block_stride;
    if (rows < 0 || rows > 2147483647LL || (!new_indptr && rows != t->batch) || (new_indptr && max_new < 0) || row_stride % 8 != 0 ||
        col % 8 != 0 || col < 0 || col + width > row_stride || num_slots < 0) {
        set_error("%s: %lld rows for %d sequences, columns %lld of %lld", who, (long long)rows, t->batch, (long long)col,
                  (long long)row_stride);
        return KTK_ERR_ARG;
    }
    return KTK_OK;
}

template <typename T>
static int conv_launch(const void* x, int64_t row_stride, const int32_t* ni, int max_new, const int32_t* slots, int64_t num_slots,
                       const float* w, const float* b, void* ring, void* u, const ktk_paged& t, const ktk_lru& a,
                       int32_t* status, cudaStream_t st) {
    const int width = a.blocks * a.block_stride, chunk = a.taps > kLcChunk ? a.taps : kLcChunk;
    const int n = ni ? max_new : 1;
    const dim3 grid((unsigned)((width / 8 + kLcThreads - 1) / kLcThreads), (unsigned)((n + chunk - 1) / chunk), (unsigned)t.batch);
    if (grid.y > 65535) { set_error("ktk_lru_conv: %d tokens in one call", n); return KTK_ERR_TOO_LARGE; }
    auto kernel = a.taps == 4 ? lru_conv_kernel<T, 4> : lru_conv_kernel<T, 0>;
    kernel<<<grid, kLcThreads, 0, st>>>((const T*)x, row_stride, ni, slots, num_slots, w, b, (T*)ring, (T*)u, t, width, a.taps,
                                        chunk, status);
    KTK_CUDA_TRY(cudaGetLastError(), "ktk_lru_conv");
    return KTK_OK;
}

template <typename T> static int scan_launch(const LruParams& p, cudaStream_t st) {
    const int width = p.a.blocks * p.a.block_stride;
    if (p.new_indptr) {
        // as many CTAs along the sequence as stay resident together and have tokens
        const int64_t groups = (width + 31) / 32, tiles = (p.max_new + kLsTile - 1) / kLsTile;
        int ctas = kLsMaxCluster;
        while (ctas > 1 && (ctas > tiles || groups * p.t.batch * ctas > (int64_t)sm_count() * 4)) ctas /= 2;
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = dim3((unsigned)ctas, (unsigned)groups, (unsigned)p.t.batch);
        cfg.blockDim = dim3(kLsThreads);
        cfg.stream = st;
        cudaLaunchAttribute attr{};
        attr.id = cudaLaunchAttributeClusterDimension;
        attr.val.clusterDim.x = ctas;
        attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
        cfg.attrs = &attr;
        cfg.numAttrs = 1;
        KTK_CUDA_TRY(cudaLaunchKernelEx(&cfg, lru_scan_kernel<T>, p), "ktk_lru_scan");
    }
    else
        lru_step_kernel<T><<<dim3((unsigned)((width + kLdThreads - 1) / kLdThreads), (unsigned)p.t.batch), kLdThreads, 0, st>>>(p);
    KTK_CUDA_TRY(cudaGetLastError(), "ktk_lru_scan");
    return KTK_OK;
}

}  // namespace ktk

using namespace ktk;

extern "C" int ktk_lru_conv(const void* proj, int64_t row_stride, int64_t x_col, const int32_t* new_indptr, int64_t rows,
                            int32_t max_new, const int32_t* slots, int64_t num_slots, const float* conv_w,
                            const float* conv_b, void* ring, void* u, const ktk_paged* table, const ktk_lru* shape,
                            int32_t* status, void* stream) {
    const char* who = "ktk_lru_conv";
    const int rc = check_lru(shape, table, new_indptr, rows, max_new, row_stride, x_col, num_slots, who);
    if (rc != KTK_OK) return rc;
    if (rows == 0 || max_new == 0) return KTK_OK;
    if (!proj || !slots || !conv_w || !conv_b || !ring || !u || !table->kv_indptr || !table->kv_last_page_len ||
        (((uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)conv_b | (uintptr_t)ring | (uintptr_t)u) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    cudaStream_t st = (cudaStream_t)stream;
    if (shape->dtype == KTK_F32)
        return conv_launch<float>((const float*)proj + x_col, row_stride, new_indptr, max_new, slots, num_slots, conv_w, conv_b,
                                  ring, u, *table, *shape, status, st);
    return conv_launch<__nv_bfloat16>((const __nv_bfloat16*)proj + x_col, row_stride, new_indptr, max_new, slots, num_slots,
                                      conv_w, conv_b, ring, u, *table, *shape, status, st);
}

extern "C" int ktk_lru_scan(const float* z, const void* u, const void* proj, int64_t row_stride, int64_t y_col,
                            const int32_t* new_indptr, int64_t rows, int32_t max_new, const int32_t* slots,
                            int64_t num_slots, const float* rb, const float* ib, const float* decay, float* state,
                            void* out, const ktk_paged* table, const ktk_lru* shape, int32_t* status, void* stream) {
    const char* who = "ktk_lru_scan";
    const int rc = check_lru(shape, table, new_indptr, rows, max_new, row_stride, y_col, num_slots, who);
    if (rc != KTK_OK) return rc;
    if (rows == 0 || max_new == 0) return KTK_OK;
    if (!z || !u || !proj || !slots || !rb || !ib || !decay || !state || !out || !table->kv_indptr || !table->kv_last_page_len) {
        set_error("%s: null pointer", who);
        return KTK_ERR_ARG;
    }
    const size_t size = shape->dtype == KTK_F32 ? 4 : 2;
    const LruParams p{*shape, *table, z, u, (const char*)proj + y_col * size, row_stride, new_indptr, slots, num_slots, rows,
                      max_new, rb, ib, decay, state, out, status};
    return shape->dtype == KTK_F32 ? scan_launch<float>(p, (cudaStream_t)stream) : scan_launch<__nv_bfloat16>(p, (cudaStream_t)stream);
}

extern "C" int ktk_lru_decode_supported(const ktk_lru* shape) {
    return shape && shape->dtype == KTK_BF16 && shape->block_stride > 0 && shape->block_stride <= kLfMaxBlock ? 1 : 0;
}

extern "C" int ktk_lru_decode(const void* proj, int64_t row_stride, int64_t y_col, int64_t x_col, int64_t rows,
                              const int32_t* slots, int64_t num_slots, const float* conv_w, const float* conv_b,
                              const void* gates, const float* rb, const float* ib, const float* decay, void* ring, float* state,
                              void* out, const ktk_paged* table, const ktk_lru* shape, int32_t* status, void* stream) {
    const char* who = "ktk_lru_decode";
    int rc = check_lru(shape, table, nullptr, rows, 1, row_stride, x_col, num_slots, who);
    if (rc == KTK_OK) rc = check_lru(shape, table, nullptr, rows, 1, row_stride, y_col, num_slots, who);
    if (rc != KTK_OK) return rc;
    if (!ktk_lru_decode_supported(shape)) { set_error("%s: bf16, blocks of at most %d channels", who, kLfMaxBlock); return KTK_ERR_UNSUPPORTED; }
    if (rows == 0) return KTK_OK;
    if (!proj || !slots || !conv_w || !conv_b || !gates || !rb || !ib || !decay || !ring || !state || !out || !table->kv_indptr ||
        !table->kv_last_page_len ||
        (((uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)conv_b | (uintptr_t)gates | (uintptr_t)ring) & 15u) != 0) {
        set_error("%s: null or misaligned pointer", who);
        return KTK_ERR_ARG;
    }
    const LruParams p{*shape, *table, nullptr, nullptr, (const __nv_bfloat16*)proj + y_col, row_stride, nullptr, slots, num_slots,
                      rows, 1, rb, ib, decay, state, out, status};
    const LruDecodeParams q{p, (const __nv_bfloat16*)proj + x_col, (const __nv_bfloat16*)gates, conv_w, conv_b, (__nv_bfloat16*)ring};
    const int smem = lf_smem(shape->block_stride), slices = (shape->block_stride + kLfChan - 1) / kLfChan;
    auto kernel = shape->taps == 4 ? lru_decode_kernel<4> : lru_decode_kernel<0>;
    KTK_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), who);
    kernel<<<dim3((unsigned)(shape->blocks * slices), (unsigned)((rows + kLfRows - 1) / kLfRows)), kLfThreads, smem,
             (cudaStream_t)stream>>>(q);
    KTK_CUDA_TRY(cudaGetLastError(), who);
    return KTK_OK;
}
