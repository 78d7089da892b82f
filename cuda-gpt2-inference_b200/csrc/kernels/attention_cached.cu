// Causal softmax attention of a step's rows over a per-slot key/value cache, with grouped key/value heads
// (query head h reads key/value head h / (H / G)), separate key and value head sizes, and optional RMS norms
// of queries, keys and values and a partial rotary embedding in front.
//
// Four kernels:
//   attention_prep         norms + rotation of a step's q, and of its k and v on their way into the cache
//   attention_cached_mma   prefill on tcgen05 (fp16 operands, fp32 scores and accumulators)
//   attention_cached_simt  the same on the fp32 FMA pipe: the 32-bit arithmetic, and head sizes beyond 128
//   attention_decode       one token per sequence, prep included, the positions split over CTAs
// The cache holds fp16 (values clamped to its range: 11 significant bits where bf16 has 8) or, in the 32-bit
// arithmetic, fp32.  Positions of a slot beyond the sequence are never attended to; what they hold is finite.
#include <cuda_fp16.h>
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int kMaxHead = 256;  // largest head size

__device__ __forceinline__ __half to_half(float v) { return __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }
template <typename T> __device__ __forceinline__ T to_cache(float v);
template <> __device__ __forceinline__ float to_cache<float>(float v) { return v; }
template <> __device__ __forceinline__ __half to_cache<__half>(float v) { return to_half(v); }

// One warp turns the n values at src into the normalised, rotated vector in buf (shared memory; zeros up to n_pad):
// lane's values i = lane, lane + 32, ...  Everything is requested before anything is used.
__device__ __forceinline__ void head_vector(float* buf, const float* src, int n, int n_pad, bool norm, const float* w, float eps,
                                            int rot_dims, const float2* rot, int lane) {
    constexpr int NV = kMaxHead / 32;
    const int half = rot_dims >> 1;
    float v[NV], wv[NV];
    float2 cs[NV / 2];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        v[i] = d < n ? src[d] : 0.f;
        wv[i] = (w && d < n) ? __ldg(w + d) : 1.f;
    }
#pragma unroll
    for (int i = 0; i < NV / 2; ++i) cs[i] = lane + i * 32 < half ? __ldg(rot + lane + i * 32) : make_float2(1.f, 0.f);
    float r = 1.f;
    if (norm) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) s = fmaf(v[i], v[i], s);
        r = 1.0f / sqrtf(warp_sum(s) / (float)n + eps);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        if (d < n_pad) buf[d] = v[i] * r * wv[i];
    }
    __syncwarp();
    if (half > 0) {
#pragma unroll
        for (int i = 0; i < NV / 2; ++i) {
            const int d = lane + i * 32;
            if (d < half) {
                const float u = buf[d], x = buf[d + half];
                buf[d] = u * cs[i].x - x * cs[i].y;
                buf[d + half] = x * cs[i].x + u * cs[i].y;
            }
        }
        __syncwarp();
    }
}

// ------------------------------------------------------------------ prep
// One warp per row walks its vectors (H queries, G keys, G values), four requested at a time.  V > 0: a lane holds V consecutive elements of a vector (head sizes up to 32 V, multiples of V; the
// rotation's partner is another lane's); V = 0: any size, through shared memory.
template <typename T, int V>
__device__ __forceinline__ void store_vec(T* dst, const float (&v)[V > 0 ? V : 1]);
template <> __device__ __forceinline__ void store_vec<float, 2>(float* dst, const float (&v)[2]) { *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]); }
template <> __device__ __forceinline__ void store_vec<float, 4>(float* dst, const float (&v)[4]) { *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]); }
template <> __device__ __forceinline__ void store_vec<__half, 2>(__half* dst, const float (&v)[2]) { *reinterpret_cast<__half2*>(dst) = __halves2half2(to_half(v[0]), to_half(v[1])); }
template <> __device__ __forceinline__ void store_vec<__half, 4>(__half* dst, const float (&v)[4]) {
    const __half2 a = __halves2half2(to_half(v[0]), to_half(v[1])), b = __halves2half2(to_half(v[2]), to_half(v[3]));
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
template <int V>
__device__ __forceinline__ void load_vec(float (&v)[V], const float* p) {
    if (V == 2) { const float2 x = *reinterpret_cast<const float2*>(p); v[0] = x.x; v[1] = x.y; }
    else { const float4 x = *reinterpret_cast<const float4*>(p); v[0] = x.x; v[1] = x.y; v[2 % V] = x.z; v[3 % V] = x.w; }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
attention_prep_kernel(const CachedAttention c, const float* __restrict__ proj, int ld, T* __restrict__ q_out,
                      const SeqDesc* __restrict__ seqs, const int* __restrict__ row_seq, int M) {
    __shared__ float bufs[V > 0 ? 1 : 8][V > 0 ? 1 : kMaxHead];
    griddep_wait();
    griddep_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row = blockIdx.x * 8 + warp;
    if (row >= M) return;
    const int seq = row_seq[row];
    const int row0 = seqs[seq].row0, slot = seqs[seq].slot, pos = seqs[seq].pos0 + row - row0;
    const float* src = proj + (size_t)row * ld;
    const float2* rot = c.rot + (size_t)pos * (c.rot_dims >> 1);
    const int nvec = c.H + 2 * c.G;
    auto where = [&](int j, int& n, int& n_pad, int& col) -> T* {
        if (j < c.H) { n = c.D; n_pad = c.Dp; col = c.q_col + j * c.D; return q_out + ((size_t)row * c.H + j) * c.Dp; }
        if (j < c.H + c.G) {
            n = c.D; n_pad = c.Dp; col = c.k_col + (j - c.H) * c.D;
            return static_cast<T*>(c.K) + (((size_t)slot * c.G + j - c.H) * c.Tp + pos) * c.Dp;
        }
        n = c.Dv; n_pad = c.Dvp; col = c.v_col + (j - c.H - c.G) * c.Dv;
        return static_cast<T*>(c.V) + (((size_t)slot * c.G + j - c.H - c.G) * c.Tp + pos) * c.Dvp;
    };
    if constexpr (V == 0) {
        float* buf = bufs[V > 0 ? 0 : warp];
        for (int j = 0; j < nvec; ++j) {
            int n, n_pad, col;
            T* dst = where(j, n, n_pad, col);
            const bool is_v = j >= c.H + c.G;
            const float* w = is_v ? nullptr : (j < c.H ? c.q_norm : c.k_norm);
            head_vector(buf, src + col, n, n_pad, is_v ? c.v_norm != 0 : w != nullptr, w, c.eps, is_v ? 0 : c.rot_dims, rot, lane);
            for (int d = lane; d < n_pad; d += 32) dst[d] = to_cache<T>(buf[d]);
            __syncwarp();
        }
        return;
    } else {
        constexpr int VV = V > 0 ? V : 1;
        const int e0 = lane * VV, half = c.rot_dims >> 1, hl = half / VV;  // hl: lanes per half of the rotation
        float cs[VV], sn[VV], wq[VV], wk[VV];
        const int side = e0 < half ? 0 : (e0 < c.rot_dims ? 1 : 2);
#pragma unroll
        for (int i = 0; i < VV; ++i) {
            cs[i] = 1.f;
            sn[i] = 0.f;
            if (side < 2) { const float2 r = rot[e0 + i - side * half]; cs[i] = r.x; sn[i] = side ? r.y : -r.y; }
            wq[i] = (c.q_norm && e0 + i < c.D) ? __ldg(c.q_norm + e0 + i) : 1.f;
            wk[i] = (c.k_norm && e0 + i < c.D) ? __ldg(c.k_norm + e0 + i) : 1.f;
        }
        const int partner = side == 0 ? lane + hl : (side == 1 ? lane - hl : lane);
        constexpr int U = 4;  // vectors requested at a time
        for (int j0 = 0; j0 < nvec; j0 += U) {
            float v[U][VV];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                int n = 0, n_pad, col;
#pragma unroll
                for (int i = 0; i < VV; ++i) v[u][i] = 0.f;
                if (j0 + u < nvec) where(j0 + u, n, n_pad, col);
                if (e0 < n) load_vec<VV>(v[u], src + col + e0);
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int j = j0 + u;
                if (j < nvec) {
                    int n, n_pad, col;
                    T* dst = where(j, n, n_pad, col);
                    const bool is_q = j < c.H, is_v = j >= c.H + c.G;
                    if (is_v ? c.v_norm != 0 : (is_q ? c.q_norm : c.k_norm) != nullptr) {
                        float s = 0.f;
#pragma unroll
                        for (int i = 0; i < VV; ++i) s = fmaf(v[u][i], v[u][i], s);
                        const float r = 1.0f / sqrtf(warp_sum(s) / (float)n + c.eps);
#pragma unroll
                        for (int i = 0; i < VV; ++i) v[u][i] *= is_v ? r : r * (is_q ? wq[i] : wk[i]);
                    }
                    if (!is_v && c.rot_dims > 0) {
#pragma unroll
                        for (int i = 0; i < VV; ++i) {
                            const float other = __shfl_sync(0xffffffffu, v[u][i], partner);
                            v[u][i] = fmaf(other, sn[i], v[u][i] * cs[i]);
                        }
                    }
                    if (e0 < n_pad) store_vec<T, V>(dst + e0, v[u]);  // (elements beyond the head are zero)
                }
            }
        }
    }
}

// ------------------------------------------------------------------ fp32 FMA attention
// A CTA takes 32 query rows of one (sequence, head) over key tiles of 32.
constexpr int SQ = 32, SK = 32;
template <typename T>
__device__ __forceinline__ float cache_f(const T* p);
template <> __device__ __forceinline__ float cache_f<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float cache_f<__half>(const __half* p) { return __half2float(*p); }

template <typename T, bool OF32>
__global__ void __launch_bounds__(256)
attention_simt_kernel(const CachedAttention c, const T* __restrict__ q_in, void* out, int ldo, const SeqDesc* __restrict__ seqs) {
    extern __shared__ float sm[];
    const int Dl = c.D + 1, Vl = c.Dv + 1;
    float* qs = sm;                  // [SQ][Dl]
    float* ks = qs + SQ * Dl;        // [SK][Dl]
    float* vs = ks + SK * Dl;        // [SK][Vl]
    float* ps = vs + SK * Vl;        // [SQ][SK + 1]
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = seqs[blockIdx.z];
    const int h = blockIdx.y, q0 = blockIdx.x * SQ;
    if (q0 >= sd.n) return;
    const int kvh = h / (c.H / c.G);
    const int tid = threadIdx.x, nq = min(SQ, sd.n - q0);
    const bool flat = c.ld_kv > 0;
    if (flat && sd.kv0 < 0) return;
    const int ldk = flat ? c.ld_kv : c.Dp, ldv = flat ? c.ld_kv : c.Dvp;
    const T* K = static_cast<const T*>(c.K) + (flat ? (size_t)sd.kv0 * ldk + h * c.Dp : ((size_t)sd.slot * c.G + kvh) * c.Tp * c.Dp);
    const T* V = static_cast<const T*>(c.V) + (flat ? (size_t)sd.kv0 * ldv + h * c.Dvp : ((size_t)sd.slot * c.G + kvh) * c.Tp * c.Dvp);
    for (int i = tid; i < SQ * c.D; i += 256) {
        const int r = i / c.D, d = i - r * c.D;
        qs[r * Dl + d] = r < nq ? cache_f<T>(q_in + ((size_t)(sd.row0 + q0 + r) * c.H + h) * c.Dp + d) * c.scale : 0.f;
    }
    // a thread scores row r against keys kq, kq + 8, kq + 16, kq + 24 and accumulates columns kq, kq + 8, ... of its row
    const int r = tid >> 3, kq = tid & 7;
    float o[kMaxHead / 8];
#pragma unroll
    for (int i = 0; i < kMaxHead / 8; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    const int pos = sd.pos0 + q0 + r;
    const int keys = sd.pos0 + q0 + nq;
    for (int k0 = 0; k0 < keys; k0 += SK) {
        __syncthreads();
        const int nk = min(SK, keys - k0);
        for (int i = tid; i < SK * c.D; i += 256) {
            const int t = i / c.D, d = i - t * c.D;
            ks[t * Dl + d] = t < nk ? cache_f<T>(K + (size_t)(k0 + t) * ldk + d) : 0.f;
        }
        for (int i = tid; i < SK * c.Dv; i += 256) {
            const int t = i / c.Dv, d = i - t * c.Dv;
            vs[t * Vl + d] = t < nk ? cache_f<T>(V + (size_t)(k0 + t) * ldv + d) : 0.f;
        }
        __syncthreads();
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        for (int d = 0; d < c.D; ++d) {
            const float qv = qs[r * Dl + d];
#pragma unroll
            for (int j = 0; j < 4; ++j) s[j] = fmaf(qv, ks[(kq + 8 * j) * Dl + d], s[j]);
        }
        float tm = -INFINITY;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (k0 + kq + 8 * j > pos) s[j] = -INFINITY;
            tm = fmaxf(tm, s[j]);
        }
#pragma unroll
        for (int d = 1; d < 8; d <<= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, d));
        const float mn = fmaxf(m, tm);  // finite: key 0 counts for every row
        const float corr = expf(m - mn);
        m = mn;
        float ts = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float p = expf(s[j] - mn);
            ps[r * (SK + 1) + kq + 8 * j] = p;
            ts += p;
        }
#pragma unroll
        for (int d = 1; d < 8; d <<= 1) ts += __shfl_xor_sync(0xffffffffu, ts, d);
        l = l * corr + ts;
        __syncwarp();
#pragma unroll
        for (int i = 0; i < kMaxHead / 8; ++i) {
            const int d = kq + 8 * i;
            if (d < c.Dv) {
                float acc = o[i] * corr;
                for (int t = 0; t < SK; ++t) acc = fmaf(ps[r * (SK + 1) + t], vs[t * Vl + d], acc);
                o[i] = acc;
            }
        }
    }
    if (r < nq) {
        const float f = c.out_scale / l;
#pragma unroll
        for (int i = 0; i < kMaxHead / 8; ++i) {
            const int d = kq + 8 * i;
            if (d < c.Dv) store1<OF32>(out, (size_t)(sd.row0 + q0 + r) * ldo + h * c.Dv + d, o[i] * f);
        }
    }
}

// ------------------------------------------------------------------ tcgen05 prefill
// The structure is that of attention_split.cu (see there for what was measured): a work item is a pair of
// neighbouring 128-row query tiles, one pipeline per tile, both sharing the K and V blocks of the producer; a
// query row is one softmax thread; O accumulates in tensor memory and is rescaled only when a row's maximum
// has grown by 2^8.  What differs: q, k and v come from three tensors (k and v from the cache, so a sequence
// may start anywhere in it), head sizes of 64 or 128 on either side, single products (the operands are plain
// fp16), and every block that reaches beyond the first row's position is masked, not only a diagonal one.
constexpr int BQ = 128;
constexpr int kMmaThreads = 352;
constexpr int kPipeThreads = 128;
constexpr int kWorkWord = 58;  // index of the work counter in the context's 64-word status area
constexpr float kRescaleStep = 8.0f;
constexpr int kTmemCols = 512, kPipeCols = 256;

// KD, VD: 64-column blocks of the key / value heads.  With two value blocks the key tile is 64 long, so that a
// pipeline's scores, probabilities and output still fit its 256 tensor-memory columns.
template <int KD, int VD>
struct MmaCfg {
    static constexpr int BKV = VD == 1 ? 128 : 64;
    static constexpr int QB = BQ * 128;            // bytes of a {64 x 128 rows} block of q
    static constexpr int KB = BKV * 128;           // ... of a key or value block
    static constexpr int QSLOTS = KD == 1 ? 2 : 1;
    static constexpr int Q_OFF = 0;
    static constexpr int K_OFF = Q_OFF + QSLOTS * 2 * KD * QB;
    static constexpr int V_OFF = K_OFF + 2 * KD * KB;
    static constexpr int BAR_OFF = V_OFF + 2 * VD * KB;
    static constexpr int TOTAL = 1024 + BAR_OFF + 512;
    static constexpr int PCol = BKV, OCol = BKV + BKV / 2;
    static_assert(OCol + 64 * VD <= kPipeCols, "tensor memory of a pipeline");
    static_assert(TOTAL <= 232448, "shared memory");
    static constexpr int SMEM = TOTAL > 117 * 1024 ? TOTAL : 117 * 1024;  // one CTA per SM: the tensor memory is taken whole
};

struct MmaArgs {
    CachedAttention c;
    const SeqDesc* seqs;
    const int2* pairs;
    int num_items;
    void* out;
    int ldo;
    float scale_log2;
    int* status;
};

__device__ __forceinline__ float fmax3(float a, float b, float c) {
    float y;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(y) : "f"(a), "f"(b), "f"(c));
    return y;
}
__device__ __forceinline__ bool pipe_bar_all(int id, bool ok) {
    uint32_t r;
    asm volatile(
        "{\n\t"
        ".reg .pred p, q;\n\t"
        "setp.ne.u32 q, %2, 0;\n\t"
        "bar.red.and.pred p, %1, 128, q;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t"
        "}\n"
        : "=r"(r)
        : "r"(id), "r"((uint32_t)ok)
        : "memory");
    return r != 0;
}

struct Item {
    int row0, n, q0, pos0, slot, h, kv0;
    // key blocks pipeline x works through (0: the pair has no second tile)
    template <int BKV>
    __device__ __forceinline__ int blocks(int x) const {
        const int q = q0 + x * BQ;
        if (q >= n) return 0;
        return (pos0 + min(q + BQ, n) + BKV - 1) / BKV;
    }
};
__device__ __forceinline__ Item get_item(const MmaArgs& a, int item) {
    const int2 pr = __ldg(a.pairs + item / a.c.H);
    const SeqDesc* s = a.seqs + pr.x;
    Item it;
    it.h = item % a.c.H;
    it.row0 = __ldg(&s->row0); it.n = __ldg(&s->n); it.pos0 = __ldg(&s->pos0); it.slot = __ldg(&s->slot); it.kv0 = __ldg(&s->kv0);
    it.q0 = pr.y * 2 * BQ;
    return it;
}

template <int KD, int VD>
__global__ void __launch_bounds__(kMmaThreads, 1)
attention_cached_mma_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                            const __grid_constant__ CUtensorMap tmap_v, const MmaArgs args) {
    using Cfg = MmaCfg<KD, VD>;
    constexpr int BKV = Cfg::BKV, QB = Cfg::QB, KB = Cfg::KB, QS = Cfg::QSLOTS;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* q_s = smem + Cfg::Q_OFF;  // [slot][tile][KD]
    uint8_t* k_s = smem + Cfg::K_OFF;  // [stage][KD]
    uint8_t* v_s = smem + Cfg::V_OFF;  // [stage][VD]
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Cfg::BAR_OFF);
    uint64_t* item_full = bars;        // [2]
    uint64_t* item_empty = bars + 2;   // [2]
    uint64_t* q_full = bars + 4;       // [QS]
    uint64_t* q_empty = bars + 6;      // [QS]
    uint64_t* k_full = bars + 8;       // [2]
    uint64_t* k_empty = bars + 10;     // [2]
    uint64_t* v_full = bars + 12;      // [2]
    uint64_t* v_empty = bars + 14;     // [2]
    uint64_t* s_full = bars + 16;      // [pipeline]
    uint64_t* s_free = bars + 18;      // [pipeline]
    uint64_t* p_full = bars + 20;      // [pipeline]
    uint64_t* o_full = bars + 22;      // [pipeline]
    uint64_t* drain_bar = bars + 24;   // [pipeline]
    int* item_slot = reinterpret_cast<int*>(bars + 26);  // [2]
    uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(item_slot + 2);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < 2; ++s) {
            mbar_init(&item_full[s], 1);
            mbar_init(&item_empty[s], 2 * kPipeThreads + 2);
            mbar_init(&q_full[s], 1);
            mbar_init(&q_empty[s], 2);
            mbar_init(&k_full[s], 1);
            mbar_init(&k_empty[s], 2);
            mbar_init(&v_full[s], 1);
            mbar_init(&v_empty[s], 2);
            mbar_init(&s_full[s], 1);
            mbar_init(&s_free[s], kPipeThreads);
            mbar_init(&p_full[s], kPipeThreads);
            mbar_init(&o_full[s], 1);
            mbar_init(&drain_bar[s], 1);
        }
        *abort_flag = 0;
        fence_barrier_init();
        tma_prefetch_desc(&tmap_q);
        tma_prefetch_desc(&tmap_k);
        tma_prefetch_desc(&tmap_v);
    }
    if (warp == 1) {
        tmem_alloc(tmem_holder, kTmemCols);
        tmem_relinquish();
    }
    tc_fence_before_sync();
    __syncthreads();
    tc_fence_after_sync();
    const uint32_t tmem_base = *tmem_holder;
    griddep_wait();

    // use number n of a q slot: slot n % QS, phase (n / QS) & 1
    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            uint32_t g = 0;
            for (uint32_t n = 0; ok; ++n) {
                const int slot = n & 1, qs = n % QS;
                int item = atomicAdd(args.status + kWorkWord, 1);
                if (item >= args.num_items) item = -1;
                if (!mbar_wait(&item_empty[slot], ((n >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
                item_slot[slot] = item;
                mbar_arrive(&item_full[slot]);
                if (item < 0) break;
                const Item it = get_item(args, item);
                const int n0 = it.blocks<BKV>(0), n1 = it.blocks<BKV>(1);
                const int n_item = n1 > n0 ? n1 : n0;
                const bool flat = args.c.ld_kv > 0;
                const int kv0 = flat ? it.kv0 : (it.slot * args.c.G + it.h / (args.c.H / args.c.G)) * args.c.Tp;
                const int k_x = flat ? it.h * args.c.Dp : 0, v_x = flat ? it.h * args.c.Dvp : 0;
                if (!mbar_wait(&q_empty[qs], ((n / QS) & 1) ^ 1, abort_flag)) { ok = false; break; }
                mbar_arrive_expect_tx(&q_full[qs], (n1 > 0 ? 2 : 1) * KD * QB);
                for (int x = 0; x < (n1 > 0 ? 2 : 1); ++x)
                    for (int d = 0; d < KD; ++d)
                        tma_load_2d(q_s + ((qs * 2 + x) * KD + d) * QB, &tmap_q, it.h * args.c.Dp + d * 64, it.row0 + it.q0 + x * BQ, &q_full[qs]);
                for (int j = -1; j < n_item && ok; ++j) {
                    if (j + 1 < n_item) {
                        const uint32_t gk = g + j + 1;
                        const int s = gk & 1;
                        if (!mbar_wait(&k_empty[s], ((gk >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
                        mbar_arrive_expect_tx(&k_full[s], KD * KB);
                        for (int d = 0; d < KD; ++d) tma_load_2d(k_s + (s * KD + d) * KB, &tmap_k, k_x + d * 64, kv0 + (j + 1) * BKV, &k_full[s]);
                    }
                    if (j >= 0) {
                        const uint32_t gv = g + j;
                        const int s = gv & 1;
                        if (!mbar_wait(&v_empty[s], ((gv >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
                        mbar_arrive_expect_tx(&v_full[s], VD * KB);
                        for (int d = 0; d < VD; ++d) tma_load_2d(v_s + (s * VD + d) * KB, &tmap_v, v_x + d * 64, kv0 + j * BKV, &v_full[s]);
                    }
                }
                g += n_item;
            }
            if (!ok) atomicCAS(args.status, 0, DEV_TIMEOUT_PRODUCER);
        }
    } else if (warp <= 2) {
        if (lane == 0) {
            const int x = warp - 1;
            constexpr uint32_t idesc_s = make_idesc_f16(BQ, BKV, 0);
            constexpr uint32_t idesc_o = make_idesc_f16(BQ, 64, 1);
            const uint32_t tm = tmem_base + x * kPipeCols;
            bool ok = true;
            uint32_t g0 = 0, gx = 0;
            for (uint32_t n = 0; ok; ++n) {
                const int slot = n & 1, qs = n % QS;
                if (!mbar_wait(&item_full[slot], (n >> 1) & 1, abort_flag)) { ok = false; break; }
                const int item = item_slot[slot];
                if (item < 0) break;
                const Item it = get_item(args, item);
                const int n0 = it.blocks<BKV>(0), n1 = it.blocks<BKV>(1);
                const int n_item = n1 > n0 ? n1 : n0, n_kv = x ? n1 : n0;
                if (!mbar_wait(&q_full[qs], (n / QS) & 1, abort_flag)) { ok = false; break; }
                if (n_kv == 0) mbar_arrive(&q_empty[qs]);
                const uint32_t q_addr = smem_u32(q_s + (qs * 2 + x) * KD * QB);
                for (int j = 0; j <= n_item && ok; ++j) {
                    if (j < n_item) {
                        const uint32_t g = g0 + j;
                        const int ks = g & 1;
                        if (!mbar_wait(&k_full[ks], (g >> 1) & 1, abort_flag)) { ok = false; break; }
                        if (j < n_kv) {
                            if (!mbar_wait(&s_free[x], ((gx + j) & 1) ^ 1, abort_flag)) { ok = false; break; }
                            tc_fence_after_sync();
#pragma unroll
                            for (int kk = 0; kk < 4 * KD; ++kk) {
                                const uint64_t qd = make_smem_desc_sw128(q_addr + (kk >> 2) * QB + (kk & 3) * 32, 16, 1024);
                                const uint64_t kd = make_smem_desc_sw128(smem_u32(k_s + (ks * KD + (kk >> 2)) * KB) + (kk & 3) * 32, 16, 1024);
                                umma_f16_ss(tm, qd, kd, idesc_s, kk != 0);
                            }
                            umma_commit(&s_full[x]);
                            umma_commit(&k_empty[ks]);
                            if (j == n_kv - 1) umma_commit(&q_empty[qs]);
                        } else {
                            mbar_arrive(&k_empty[ks]);
                        }
                    }
                    if (j > 0) {
                        const int i = j - 1;
                        const uint32_t g = g0 + i;
                        const int vs = g & 1;
                        if (!mbar_wait(&v_full[vs], (g >> 1) & 1, abort_flag)) { ok = false; break; }
                        if (i < n_kv) {
                            if (!mbar_wait(&p_full[x], (gx + i) & 1, abort_flag)) { ok = false; break; }
                            tc_fence_after_sync();
#pragma unroll
                            for (int d = 0; d < VD; ++d)
#pragma unroll
                                for (int ks = 0; ks < BKV / 16; ++ks) {
                                    const uint64_t vd = make_smem_desc_sw128(smem_u32(v_s + (vs * VD + d) * KB) + ks * 2048, 16, 1024);
                                    umma_f16_ts(tm + Cfg::OCol + d * 64, tm + Cfg::PCol + ks * 8, vd, idesc_o, (i | ks) != 0);
                                }
                            umma_commit(&o_full[x]);
                            umma_commit(&v_empty[vs]);
                        } else {
                            mbar_arrive(&v_empty[vs]);
                        }
                    }
                }
                g0 += n_item;
                gx += n_kv;
                mbar_arrive(&item_empty[slot]);
            }
            umma_commit(&drain_bar[x]);
            if (!mbar_wait(&drain_bar[x], 0, abort_flag)) ok = false;
            if (!ok) atomicCAS(args.status, 0, DEV_TIMEOUT_MMA);
        }
    } else {
        constexpr int NC = BKV / 32;
        const int x = (warp - 3) >> 2;
        const int qd = warp & 3;
        const int r = qd * 32 + lane;
        const uint32_t tm = tmem_base + (uint32_t(qd * 32) << 16) + x * kPipeCols;
        bool ok = true;
        uint32_t gx = 0;
        // as in attention_split.cu: the threads of a pipeline leave together, and inside an item a failed wait
        // only skips the remaining waits
        for (uint32_t n = 0;; ++n) {
            const int slot = n & 1;
            if (ok && !mbar_wait(&item_full[slot], (n >> 1) & 1, abort_flag)) ok = false;
            const bool all_ok = pipe_bar_all(1 + x, ok);
            const int item = all_ok ? item_slot[slot] : -1;
            if (item < 0) break;
            const Item it = get_item(args, item);
            const int n_kv = x ? it.blocks<BKV>(1) : it.blocks<BKV>(0);
            if (n_kv == 0) {
                mbar_arrive(&item_empty[slot]);
                continue;
            }
            const int q0 = it.q0 + x * BQ;
            const int first = it.pos0 + q0;  // position of row 0
            float m_ref = -INFINITY, l = 0.f;
            for (int j = 0; j < n_kv; ++j) {
                const uint32_t gi = gx + j;
                uint32_t t[NC][32];
                if (ok && !mbar_wait(&s_full[x], gi & 1, abort_flag)) ok = false;
                tc_fence_after_sync();
#pragma unroll
                for (int c = 0; c < NC; ++c) tmem_ld_32x32b_x32(tm + c * 32, t[c]);
                tmem_ld_wait();
                tc_fence_before_sync();
                mbar_arrive(&s_free[x]);
                if ((j + 1) * BKV - 1 > first) {  // some key of the block lies behind some row
                    const int last = first + r - j * BKV;  // last visible key of this row, counted in the block
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (c * 32 + i > last) t[c][i] = 0xff800000u;
                    }
                }
                float pm0 = -INFINITY, pm1 = -INFINITY, pm2 = -INFINITY, pm3 = -INFINITY;
#pragma unroll
                for (int c = 0; c < NC; ++c) {
#pragma unroll
                    for (int i = 0; i < 32; i += 8) {
                        pm0 = fmax3(pm0, __uint_as_float(t[c][i]), __uint_as_float(t[c][i + 1]));
                        pm1 = fmax3(pm1, __uint_as_float(t[c][i + 2]), __uint_as_float(t[c][i + 3]));
                        pm2 = fmax3(pm2, __uint_as_float(t[c][i + 4]), __uint_as_float(t[c][i + 5]));
                        pm3 = fmax3(pm3, __uint_as_float(t[c][i + 6]), __uint_as_float(t[c][i + 7]));
                    }
                }
                // finite from the first block on: every row sees key 0
                const float cand = fmaxf(m_ref, fmaxf(fmaxf(pm0, pm1), fmaxf(pm2, pm3)) * args.scale_log2);
                const bool moved = __any_sync(0xffffffffu, cand > m_ref + kRescaleStep);
                float alpha = 1.f;
                if (moved) {
                    alpha = ex2(m_ref - cand);
                    m_ref = cand;
                }
                float sum0 = 0.f, sum1 = 0.f, sum2 = 0.f, sum3 = 0.f;
                const float neg_m = -m_ref;
                uint32_t pk[NC / 2][32];
#pragma unroll
                for (int c = 0; c < NC; ++c) {
#pragma unroll
                    for (int k = 0; k < 16; k += 2) {
                        float a0 = ex2(fmaf(__uint_as_float(t[c][2 * k]), args.scale_log2, neg_m));
                        float a1 = ex2(fmaf(__uint_as_float(t[c][2 * k + 1]), args.scale_log2, neg_m));
                        float b0 = ex2(fmaf(__uint_as_float(t[c][2 * k + 2]), args.scale_log2, neg_m));
                        float b1 = ex2(fmaf(__uint_as_float(t[c][2 * k + 3]), args.scale_log2, neg_m));
                        sum0 += a0; sum1 += a1; sum2 += b0; sum3 += b1;
                        const __half2 ah = __floats2half2_rn(a0, a1), bh = __floats2half2_rn(b0, b1);
                        pk[c >> 1][(c & 1) * 16 + k] = *reinterpret_cast<const uint32_t*>(&ah);
                        pk[c >> 1][(c & 1) * 16 + k + 1] = *reinterpret_cast<const uint32_t*>(&bh);
                    }
                }
                if (j > 0) {
                    if (ok && !mbar_wait(&o_full[x], (gi - 1) & 1, abort_flag)) ok = false;
                    tc_fence_after_sync();
                    if (moved) {
#pragma unroll
                        for (int hh = 0; hh < 2 * VD; ++hh) {
                            uint32_t o[32];
                            tmem_ld_32x32b_x32(tm + Cfg::OCol + hh * 32, o);
                            tmem_ld_wait();
#pragma unroll
                            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                            tmem_st_32x32b_x32(tm + Cfg::OCol + hh * 32, o);
                        }
                    }
                }
#pragma unroll
                for (int c = 0; c < NC / 2; ++c) tmem_st_32x32b_x32(tm + Cfg::PCol + c * 32, pk[c]);
                tmem_st_wait();
                tc_fence_before_sync();
                mbar_arrive(&p_full[x]);
                l = l * alpha + ((sum0 + sum1) + (sum2 + sum3));
            }
            gx += n_kv;
            if (ok && !mbar_wait(&o_full[x], (gx - 1) & 1, abort_flag)) ok = false;
            tc_fence_after_sync();
            const float f = args.c.out_scale / l;
            const int Dv = args.c.Dv;
            const bool mine = ok && q0 + r < it.n;
            uint16_t* orow = static_cast<uint16_t*>(args.out) + (size_t)(it.row0 + q0 + r) * args.ldo + it.h * Dv;
#pragma unroll
            for (int hh = 0; hh < 2 * VD; ++hh) {
                uint32_t o[32];
                tmem_ld_32x32b_x32(tm + Cfg::OCol + hh * 32, o);
                tmem_ld_wait();
                if (!mine || hh * 32 >= Dv) continue;
                uint32_t pk[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) pk[i] = pack_bf16(__uint_as_float(o[2 * i]) * f, __uint_as_float(o[2 * i + 1]) * f);
                if ((Dv & 7) == 0) {  // 16-byte pieces of the row (rows start at multiples of 16 bytes)
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (hh * 32 + i * 8 < Dv) *reinterpret_cast<uint4*>(orow + hh * 32 + i * 8) = make_uint4(pk[4 * i], pk[4 * i + 1], pk[4 * i + 2], pk[4 * i + 3]);
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (hh * 32 + i < Dv) orow[hh * 32 + i] = (uint16_t)(i & 1 ? pk[i >> 1] >> 16 : pk[i >> 1] & 0xffffu);
                }
            }
            tc_fence_before_sync();
            mbar_arrive(&item_empty[slot]);
        }
        if (!ok && lane == 0) atomicCAS(args.status, 0, DEV_TIMEOUT_SOFTMAX);
    }

    griddep_launch_dependents();
    tc_fence_before_sync();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after_sync();
        tmem_dealloc(tmem_base, kTmemCols);
    }
    // the last CTA to finish puts the work counters back to zero for the next launch
    if (threadIdx.x == 0) {
        __threadfence();
        if (atomicAdd(args.status + kWorkWord + 1, 1) == (int)gridDim.x - 1) {
            args.status[kWorkWord] = 0;
            args.status[kWorkWord + 1] = 0;
            __threadfence();
        }
    }
}

// ------------------------------------------------------------------ decode
// A cluster of `splits` CTAs per (sequence, key/value head, chunk of GH query heads), each with its share of the
// cached positions; further CTAs in x run the minGRU step.  The query heads of a CTA share every key and value
// read.  Keys go by in tiles of 128: scores (LK lanes per key, 16 bytes of the key per lane), softmax statistics
// (a warp per head), probabilities x values (LV lanes per key); a tile's keys and first values are requested
// together, the first tile's before the queries are formed.  The splits' states are merged through the cluster's
// shared memory.
constexpr int kDecThreads = 256, kDecTile = 128;

__device__ __forceinline__ float ld_cluster_f32(const float* p, int rank) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(map_to_cta(smem_u32(p), rank)) : "memory");
    return v;
}

template <int GH, int LK>
__global__ void __launch_bounds__(kDecThreads, 2)
attention_decode_kernel(const CachedAttention c, const float* __restrict__ proj, int ld, uint8_t* __restrict__ out, int ldo,
                        const SeqDesc* __restrict__ seqs, int splits, int chunks, const MinGruArgs gru) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float ss[GH][kDecTile];
    __shared__ float stat_m[GH], stat_l[GH], stat_a[GH];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = seqs[blockIdx.y];
    const int att_blocks = c.G * chunks * splits;
    const float* row = proj + (size_t)sd.row0 * ld;
    if ((int)blockIdx.x >= att_blocks) {  // minGRU: one thread per channel
        const int ch = (blockIdx.x - att_blocks) * kDecThreads + tid;
        if (ch < gru.width) {
            const float z = sigmoidf_(row[gru.z_col + ch]), u = row[gru.x_col + ch];
            float* Sp = gru.S + (size_t)sd.slot * gru.width + ch;
            const float S = fmaf(1.f - z, sd.pos0 > 0 ? *Sp : 0.f, z * (u >= 0.f ? u + 0.5f : sigmoidf_(u)));
            *Sp = S;
            store_split(static_cast<uint8_t*>(gru.out) + (size_t)sd.row0 * gru.ldo * 4, gru.out_col + ch, S * silu(row[gru.g_col + ch]) * gru.out_scale);
        }
        return;
    }
    const int z = blockIdx.x % splits, gc = blockIdx.x / splits, g = gc / chunks, chunk = gc % chunks;
    const int per_group = c.H / c.G, h0 = g * per_group + chunk * GH, nh = min(GH, per_group - chunk * GH);
    const int Dp = c.Dp, Dvp = c.Dvp;
    float* qs = sm;               // [GH][Dp], scaled for base-2 exponentials
    float* kn = qs + GH * Dp;     // [Dp] the new key
    float* vn = kn + Dp;          // [Dvp] the new value
    float* os = vn + Dvp;         // [GH][Dvp] the sums over the key groups, at the end
    const int pos = sd.pos0;
    const float2* rot = c.rot + (size_t)pos * (c.rot_dims >> 1);
    __half* Kc = static_cast<__half*>(c.K) + ((size_t)sd.slot * c.G + g) * c.Tp * Dp;
    __half* Vc = static_cast<__half*>(c.V) + ((size_t)sd.slot * c.G + g) * c.Tp * Dvp;
    const int per = (((pos + splits - 1) / splits + kDecTile - 1) / kDecTile) * kDecTile;  // cached keys per split
    const int t_begin = min(pos, z * per), t_end = min(pos, t_begin + per);
    constexpr int KPP = kDecThreads / LK;  // keys per pass
    constexpr int PASSES = kDecTile / KPP;
    constexpr int VU = 4;                  // values per thread requested at a time
    const int sub = lane & (LK - 1);
    const int LV = Dvp >> 3, vgroups = kDecThreads / LV, vg = tid / LV, vsub = tid - vg * LV;
    const bool v_live = vg < vgroups;
    uint4 kv[PASSES], vv[VU];
    auto request = [&](int t0) {
#pragma unroll
        for (int p = 0; p < PASSES; ++p) {
            const int t = t0 + p * KPP + tid / LK;
            kv[p] = make_uint4(0u, 0u, 0u, 0u);
            if (t < t_end && sub * 8 < Dp) kv[p] = *reinterpret_cast<const uint4*>(Kc + (size_t)t * Dp + sub * 8);
        }
#pragma unroll
        for (int u = 0; u < VU; ++u) {
            const int t = t0 + vg + u * vgroups;
            vv[u] = make_uint4(0u, 0u, 0u, 0u);
            if (v_live && t < min(t_end, t0 + kDecTile)) vv[u] = *reinterpret_cast<const uint4*>(Vc + (size_t)t * Dvp + vsub * 8);
        }
    };
    request(t_begin);
    for (int j = warp; j < GH + 2; j += 8) {
        if (j < GH) {
            if (j < nh) head_vector(qs + j * Dp, row + c.q_col + (h0 + j) * c.D, c.D, Dp, c.q_norm != nullptr, c.q_norm, c.eps, c.rot_dims, rot, lane);
            else for (int d = lane; d < Dp; d += 32) qs[j * Dp + d] = 0.f;
        } else if (j == GH) head_vector(kn, row + c.k_col + g * c.D, c.D, Dp, c.k_norm != nullptr, c.k_norm, c.eps, c.rot_dims, rot, lane);
        else head_vector(vn, row + c.v_col + g * c.Dv, c.Dv, Dvp, c.v_norm != 0, nullptr, c.eps, 0, nullptr, lane);
    }
    __syncthreads();
    // the new key and value enter in the cache's precision, like the others; split 0 of the first chunk stores them
    for (int d = tid; d < Dp; d += kDecThreads) {
        const __half v = to_half(kn[d]);
        kn[d] = __half2float(v);
        if (z == 0 && chunk == 0) Kc[(size_t)pos * Dp + d] = v;
    }
    for (int d = tid; d < Dvp; d += kDecThreads) {
        const __half v = to_half(vn[d]);
        vn[d] = __half2float(v);
        if (z == 0 && chunk == 0) Vc[(size_t)pos * Dvp + d] = v;
    }
    for (int i = tid; i < GH * Dp; i += kDecThreads) qs[i] *= c.scale * 1.4426950408889634f;
    __syncthreads();
    if (warp < GH) {
        float s = 0.f;
        for (int d = lane; d < Dp; d += 32) s = fmaf(qs[warp * Dp + d], kn[d], s);
        s = warp_sum(s);
        if (lane == 0) {
            stat_m[warp] = z == 0 ? s : -INFINITY;  // the new key belongs to split 0
            stat_l[warp] = z == 0 ? 1.f : 0.f;
        }
    }
    // this lane's piece of the queries
    float q[GH][8];
#pragma unroll
    for (int j = 0; j < GH; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) q[j][e] = sub * 8 + e < Dp ? qs[j * Dp + sub * 8 + e] : 0.f;
    float acc[GH][8];
#pragma unroll
    for (int j = 0; j < GH; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[j][e] = (z == 0 && vg == 0) ? vn[vsub * 8 + e] : 0.f;
    auto add_value = [&](const uint4& x, int t) {
        const __half2* hp = reinterpret_cast<const __half2*>(&x);
        float2 f[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) f[e] = __half22float2(hp[e]);
#pragma unroll
        for (int j = 0; j < GH; ++j) {
            const float p = ss[j][t];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                acc[j][2 * e] = fmaf(p, f[e].x, acc[j][2 * e]);
                acc[j][2 * e + 1] = fmaf(p, f[e].y, acc[j][2 * e + 1]);
            }
        }
    };
    for (int t0 = t_begin; t0 < t_end; t0 += kDecTile) {
        const int nt = min(kDecTile, t_end - t0);
#pragma unroll
        for (int p = 0; p < PASSES; ++p) {
            const int kt = p * KPP + tid / LK;
            const __half2* hp = reinterpret_cast<const __half2*>(&kv[p]);
            float s[GH];
#pragma unroll
            for (int j = 0; j < GH; ++j) s[j] = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __half22float2(hp[e]);
#pragma unroll
                for (int j = 0; j < GH; ++j) s[j] = fmaf(f.x, q[j][2 * e], fmaf(f.y, q[j][2 * e + 1], s[j]));
            }
            reduce_scatter<GH, LK>(s, lane);
            constexpr int HELD = GH > LK ? GH / LK : 1;
            if (scatter_owner<GH, LK>(lane)) {
                const int first = scatter_first<GH, LK>(lane);
#pragma unroll
                for (int j = 0; j < HELD; ++j) ss[first + j][kt] = kt < nt ? s[j] : -INFINITY;
            }
        }
        __syncthreads();
        if (warp < GH) {
            float v[kDecTile / 32], m = stat_m[warp];
            const float m_old = m;
#pragma unroll
            for (int i = 0; i < kDecTile / 32; ++i) { v[i] = ss[warp][lane + 32 * i]; m = fmaxf(m, v[i]); }
#pragma unroll
            for (int d = 16; d >= 1; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < kDecTile / 32; ++i) {
                const float p = ex2(v[i] - m);
                ss[warp][lane + 32 * i] = p;
                s += p;
            }
            s = warp_sum(s);
            __syncwarp();
            if (lane == 0) {
                const float al = ex2(m_old - m);
                stat_a[warp] = al;
                stat_m[warp] = m;
                stat_l[warp] = stat_l[warp] * al + s;
            }
        }
        __syncthreads();
        if (v_live) {
#pragma unroll
            for (int j = 0; j < GH; ++j) {
                const float al = stat_a[j];
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[j][e] *= al;
            }
#pragma unroll
            for (int u = 0; u < VU; ++u)
                if (vg + u * vgroups < nt) add_value(vv[u], vg + u * vgroups);
            for (int kt = vg + VU * vgroups; kt < nt; kt += VU * vgroups) {  // value heads of more than 64
#pragma unroll
                for (int u = 0; u < VU; ++u)
                    if (kt + u * vgroups < nt) vv[u] = *reinterpret_cast<const uint4*>(Vc + (size_t)(t0 + kt + u * vgroups) * Dvp + vsub * 8);
#pragma unroll
                for (int u = 0; u < VU; ++u)
                    if (kt + u * vgroups < nt) add_value(vv[u], kt + u * vgroups);
            }
        }
        if (t0 + kDecTile < t_end) request(t0 + kDecTile);
        __syncthreads();
    }
    // sum of the key groups: each in turn adds its part (a handful of them; fixed order)
    for (int i = tid; i < GH * Dvp; i += kDecThreads) os[i] = 0.f;
    __syncthreads();
    // groups of one warp first, by shuffles, when they are whole powers of two
    const bool pow2 = (LV & (LV - 1)) == 0;
    if (pow2) {
        for (int m = LV; m < 32; m <<= 1)
#pragma unroll
            for (int j = 0; j < GH; ++j)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[j][e] += __shfl_xor_sync(0xffffffffu, acc[j][e], m);
    }
    const int parts = pow2 ? 8 : vgroups;  // LV <= 32: a warp holds one group or several
    for (int p = 0; p < parts; ++p) {
        const bool mine = pow2 ? (warp == p && lane < LV) : (v_live && vg == p);
        if (mine) {
#pragma unroll
            for (int j = 0; j < GH; ++j)
#pragma unroll
                for (int e = 0; e < 8; ++e) os[j * Dvp + vsub * 8 + e] += acc[j][e];
        }
        __syncthreads();
    }
    uint8_t* orow = out + (size_t)sd.row0 * ldo * 4;
    if (splits == 1) {
        for (int i = tid; i < nh * c.Dv; i += kDecThreads) {
            const int j = i / c.Dv, d = i - j * c.Dv;
            store_split(orow, (h0 + j) * c.Dv + d, os[j * Dvp + d] / stat_l[j] * c.out_scale);
        }
        return;
    }
    cluster_sync_all();  // every split's state is in its shared memory
    for (int i = z * kDecThreads + tid; i < nh * c.Dv; i += splits * kDecThreads) {
        const int j = i / c.Dv, d = i - j * c.Dv;
        float m = -INFINITY, L = 0.f, O = 0.f;
        for (int s = 0; s < splits; ++s) m = fmaxf(m, ld_cluster_f32(stat_m + j, s));
        for (int s = 0; s < splits; ++s) {
            const float w = ex2(ld_cluster_f32(stat_m + j, s) - m);  // 0 for a split without keys
            L = fmaf(ld_cluster_f32(stat_l + j, s), w, L);
            O = fmaf(ld_cluster_f32(os + j * Dvp + d, s), w, O);
        }
        store_split(orow, (h0 + j) * c.Dv + d, O / L * c.out_scale);
    }
    cluster_sync_all();  // nobody leaves while its state is being read
}

template <int KD, int VD>
int launch_mma_one(b200_ctx* ctx, const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const MmaArgs& a) {
    using Cfg = MmaCfg<KD, VD>;
    static bool attr_set[64] = {};
    if (!attr_set[ctx->device & 63]) {
        B200_CUDA(ctx, cudaFuncSetAttribute(attention_cached_mma_kernel<KD, VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM));
        attr_set[ctx->device & 63] = true;
    }
    const int grid = a.num_items < ctx->num_sms ? a.num_items : ctx->num_sms;
    cudaError_t le = launch_pdl(ctx, attention_cached_mma_kernel<KD, VD>, dim3(grid), dim3(kMmaThreads), Cfg::SMEM, tq, tk, tv, a);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int decode_heads_per_cta(const CachedAttention& c) {
    const int per = c.H / c.G;
    return per >= 3 ? 4 : per;  // (eight heads' queries and sums would not leave room for two CTAs per SM)
}

template <int GH, int LK>
int launch_decode_one(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, uint8_t* out, int ldo, const SeqDesc* seqs, int B,
                      const MinGruArgs& gru) {
    const int chunks = (c.H / c.G + GH - 1) / GH;
    int splits = 1;
    while (splits < 8 && B * c.G * chunks * splits * 2 <= 2 * ctx->num_sms && splits * 2 * kDecTile <= c.Tp) splits *= 2;
    const size_t smem = (size_t)(GH * c.Dp + c.Dp + c.Dvp + GH * c.Dvp) * 4;
    if (smem > 40 * 1024) return B200_ERR_LIMIT;
    int gru_blocks = gru.S ? (gru.width + kDecThreads - 1) / kDecThreads : 0;
    gru_blocks = (gru_blocks + splits - 1) / splits * splits;  // whole clusters
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(c.G * chunks * splits + gru_blocks, B);
    cfg.blockDim = dim3(kDecThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (splits > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = splits;
        attr[n].val.clusterDim.y = attr[n].val.clusterDim.z = 1;
        ++n;
    }
    if (ctx->pdl) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    const cudaError_t le = cudaLaunchKernelEx(&cfg, attention_decode_kernel<GH, LK>, c, proj, ld, out, ldo, seqs, splits, chunks, gru);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

template <int GH>
int launch_decode_lk(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, uint8_t* out, int ldo, const SeqDesc* seqs, int B,
                     const MinGruArgs& gru) {
    if (c.Dp <= 64) return launch_decode_one<GH, 8>(ctx, c, proj, ld, out, ldo, seqs, B, gru);
    if (c.Dp <= 128) return launch_decode_one<GH, 16>(ctx, c, proj, ld, out, ldo, seqs, B, gru);
    return launch_decode_one<GH, 32>(ctx, c, proj, ld, out, ldo, seqs, B, gru);
}

}  // namespace

namespace {
template <typename T>
int launch_prep(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, void* q_out, const SeqDesc* seqs, const int* row_seq, int M) {
    const dim3 grid((M + 7) / 8), block(256);
    // V consecutive elements per lane: everything in multiples of V, the padded heads within a warp's reach
    auto fits = [&](int v) {
        return c.Dp <= 32 * v && c.Dvp <= 32 * v && c.D % v == 0 && c.Dv % v == 0 && (c.rot_dims / 2) % v == 0 && c.q_col % v == 0 && c.k_col % v == 0 &&
               c.v_col % v == 0 && ld % v == 0;
    };
    cudaError_t le;
    if (fits(2)) le = launch_pdl(ctx, attention_prep_kernel<T, 2>, grid, block, 0, c, proj, ld, static_cast<T*>(q_out), seqs, row_seq, M);
    else if (fits(4)) le = launch_pdl(ctx, attention_prep_kernel<T, 4>, grid, block, 0, c, proj, ld, static_cast<T*>(q_out), seqs, row_seq, M);
    else le = launch_pdl(ctx, attention_prep_kernel<T, 0>, grid, block, 0, c, proj, ld, static_cast<T*>(q_out), seqs, row_seq, M);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}
}  // namespace

int launch_attention_prep(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, void* q_out, const SeqDesc* seqs,
                          const int* row_seq, int M, bool f32) {
    return f32 ? launch_prep<float>(ctx, c, proj, ld, q_out, seqs, row_seq, M) : launch_prep<__half>(ctx, c, proj, ld, q_out, seqs, row_seq, M);
}

bool attention_cached_has_mma(const CachedAttention& c) { return c.Dp <= 128 && c.Dvp <= 128; }

int launch_attention_cached_mma(b200_ctx* ctx, const CachedAttention& c, const void* q, void* out, int ldo, const SeqDesc* seqs,
                                const int2* pairs, int num_pairs, int M, int max_slots) {
    CUtensorMap tq, tk, tv;
    const uint64_t kv_rows = (uint64_t)max_slots * c.G * c.Tp;
    const uint32_t bkv = c.Dvp > 64 ? 64 : 128;
    // 16-bit elements: the map's number format does not matter, nothing is converted or filled but zeros
    int st = b200_get_tensor_map_bf16(ctx, &tq, q, (uint64_t)M, (uint64_t)c.H * c.Dp, (uint64_t)c.H * c.Dp, BQ, 64);
    if (c.ld_kv > 0) {
        if (st == B200_OK) st = b200_get_tensor_map_bf16(ctx, &tk, c.K, (uint64_t)c.kv_rows, (uint64_t)c.H * c.Dp, (uint64_t)c.ld_kv, bkv, 64);
        if (st == B200_OK) st = b200_get_tensor_map_bf16(ctx, &tv, c.V, (uint64_t)c.kv_rows, (uint64_t)c.H * c.Dvp, (uint64_t)c.ld_kv, bkv, 64);
    } else {
        if (st == B200_OK) st = b200_get_tensor_map_bf16(ctx, &tk, c.K, kv_rows, (uint64_t)c.Dp, (uint64_t)c.Dp, bkv, 64);
        if (st == B200_OK) st = b200_get_tensor_map_bf16(ctx, &tv, c.V, kv_rows, (uint64_t)c.Dvp, (uint64_t)c.Dvp, bkv, 64);
    }
    if (st != B200_OK) return st;
    MmaArgs a;
    a.c = c; a.seqs = seqs; a.pairs = pairs; a.num_items = num_pairs * c.H; a.out = out; a.ldo = ldo;
    a.scale_log2 = c.scale * 1.4426950408889634f;
    a.status = ctx->d_status;
    if (c.Dp <= 64) return c.Dvp <= 64 ? launch_mma_one<1, 1>(ctx, tq, tk, tv, a) : launch_mma_one<1, 2>(ctx, tq, tk, tv, a);
    return c.Dvp <= 64 ? launch_mma_one<2, 1>(ctx, tq, tk, tv, a) : launch_mma_one<2, 2>(ctx, tq, tk, tv, a);
}

int launch_attention_cached_simt(b200_ctx* ctx, const CachedAttention& c, const void* q, void* out, int ldo, const SeqDesc* seqs,
                                 int E, int max_n, bool f32) {
    if (c.D > kMaxHead || c.Dv > kMaxHead) return B200_ERR_LIMIT;
    const size_t smem = (size_t)((SQ + SK) * (c.D + 1) + SK * (c.Dv + 1) + SQ * (SK + 1)) * 4;
    static bool attr_set[64] = {};
    if (!attr_set[ctx->device & 63]) {
        B200_CUDA(ctx, cudaFuncSetAttribute(attention_simt_kernel<float, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024));
        B200_CUDA(ctx, cudaFuncSetAttribute(attention_simt_kernel<__half, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024));
        attr_set[ctx->device & 63] = true;
    }
    const dim3 grid((max_n + SQ - 1) / SQ, c.H, E);
    cudaError_t le = f32 ? launch_pdl(ctx, attention_simt_kernel<float, true>, grid, dim3(256), smem, c, static_cast<const float*>(q), out, ldo, seqs)
                         : launch_pdl(ctx, attention_simt_kernel<__half, false>, grid, dim3(256), smem, c, static_cast<const __half*>(q), out, ldo, seqs);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_attention_cached_decode(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, uint8_t* out, int ldo,
                                   const SeqDesc* seqs, int B, const MinGruArgs& gru) {
    if (c.D > kMaxHead || c.Dv > kMaxHead) return B200_ERR_LIMIT;
    switch (decode_heads_per_cta(c)) {
        case 4: return launch_decode_lk<4>(ctx, c, proj, ld, out, ldo, seqs, B, gru);
        case 2: return launch_decode_lk<2>(ctx, c, proj, ld, out, ldo, seqs, B, gru);
        default: return launch_decode_lk<1>(ctx, c, proj, ld, out, ldo, seqs, B, gru);
    }
}

}  // namespace b200
