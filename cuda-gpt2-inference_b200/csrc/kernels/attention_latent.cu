// Softmax attention whose keys and values are linear in one cached latent per token (LatentAttention, decoder_kernels.h).
//
//   latent_prep, latent_gather   the expanded form's inputs: latents of all positions side by side, rotated queries
//   latent_query                 the latent form's queries, q W_uk beside the rotated part (and, decoding, the cache append)
//   latent_attention             the latent form: all heads of a token read the same cached rows, which therefore serve as the
//                                keys and, their first R columns, as the values of a whole tile of (token, head) pairs
#include <cuda_fp16.h>
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int kMaxRow = 640;     // R + Dr
constexpr int kMaxLatent = 512;  // R

__device__ __forceinline__ __half latent_half(float v) { return __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }
template <typename T> __device__ __forceinline__ T latent_elem(float v);
template <> __device__ __forceinline__ float latent_elem<float>(float v) { return v; }
template <> __device__ __forceinline__ __half latent_elem<__half>(float v) { return latent_half(v); }

// One warp: normalised latent and rotated key part of a token (src: its columns of the projection) to dst and, if not null, dst2
template <typename T>
__device__ __forceinline__ void latent_row(const LatentAttention& c, const float* src, int pos, T* dst, T* dst2, int lane) {
    constexpr int NV = kMaxLatent / 32;
    float v[NV], s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        v[i] = d < c.R ? src[d] : 0.f;
        s = fmaf(v[i], v[i], s);
    }
    const float r = 1.0f / sqrtf(warp_sum(s) / (float)c.R + c.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = lane + i * 32;
        if (d < c.R) {
            const T x = latent_elem<T>(v[i] * r * __ldg(c.c_norm + d));
            dst[d] = x;
            if (dst2) dst2[d] = x;
        }
    }
    const float2* rot = c.rot + (size_t)pos * (c.Dr >> 1);
    for (int i = lane; i < (c.Dr >> 1); i += 32) {
        const float2 cs = __ldg(rot + i);
        const float u = src[c.R + 2 * i], w = src[c.R + 2 * i + 1];
        const T a = latent_elem<T>(u * cs.x - w * cs.y), b = latent_elem<T>(w * cs.x + u * cs.y);
        dst[c.R + 2 * i] = a;
        dst[c.R + 2 * i + 1] = b;
        if (dst2) { dst2[c.R + 2 * i] = a; dst2[c.R + 2 * i + 1] = b; }
    }
    if (dst2)  // (the cache's own padding is never written)
        for (int d = c.R + c.Dr + lane; d < c.Lp; d += 32) dst2[d] = latent_elem<T>(0.f);
}

// one warp per row
template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const LatentAttention c, const float* __restrict__ proj, int ld, T* __restrict__ q_out, T* __restrict__ lat,
                   const SeqDesc* __restrict__ seqs, const int* __restrict__ row_seq, int M) {
    griddep_wait();
    griddep_launch_dependents();
    const int lane = threadIdx.x & 31, row = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (row >= M) return;
    const SeqDesc* sd = seqs + row_seq[row];
    const int slot = sd->slot, kv0 = sd->kv0, pos = sd->pos0 + row - sd->row0;
    const float* src = proj + (size_t)row * ld;
    latent_row<T>(c, src + c.c_col, pos, static_cast<T*>(c.cache) + ((size_t)slot * c.Tp + pos) * c.Lp, kv0 >= 0 ? lat + (size_t)(kv0 + pos) * c.Lp : nullptr, lane);
    if (kv0 < 0) return;
    const float2* rot = c.rot + (size_t)pos * (c.Dr >> 1);
    const int Dq = c.D + c.Dr;
    T* q = q_out + (size_t)row * c.H * c.Dp;
    const float* qs = src + c.q_col;
    const int total = c.H * c.Dp;
    for (int i0 = lane; i0 < total; i0 += 128) {  // four requested at a time
        float v[4], w[4];
        float2 cs[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int i = i0 + u * 32, h = i / c.Dp, d = i - h * c.Dp;
            v[u] = w[u] = 0.f;
            cs[u] = make_float2(1.f, 0.f);
            if (i < total && d < Dq) {
                v[u] = qs[h * Dq + d];
                if (d >= c.D) {
                    const int e = d - c.D;
                    w[u] = qs[h * Dq + c.D + (e ^ 1)];
                    cs[u] = __ldg(rot + (e >> 1));
                    if (!(e & 1)) cs[u].y = -cs[u].y;
                }
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (i0 + u * 32 < total) q[i0 + u * 32] = latent_elem<T>(fmaf(w[u], cs[u].y, v[u] * cs[u].x));
    }
}

// 16-byte pieces of the cached rows [0, pos0) of the sequences that are expanded and have any
template <typename T>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const LatentAttention c, T* __restrict__ lat, const SeqDesc* __restrict__ seqs) {
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = seqs[blockIdx.y];
    if (sd.kv0 < 0 || sd.pos0 == 0) return;
    const size_t n = (size_t)sd.pos0 * c.Lp * sizeof(T) / 16;
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const T*>(c.cache) + (size_t)sd.slot * c.Tp * c.Lp);
    uint4* dst = reinterpret_cast<uint4*>(lat + (size_t)sd.kv0 * c.Lp);
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) dst[i] = src[i];
}

// ------------------------------------------------------------------ queries in the latent's space
// A CTA takes one head, four rows and 256 columns: lane l owns eight columns, the warps share the head's dimensions and
// meet in shared memory.  Further CTAs (blockIdx.x = H) append the rows' latents, one warp each.
constexpr int kQueryRows = 4, kQueryCols = 256;
__global__ void __launch_bounds__(256)
latent_query_kernel(const LatentAttention c, const float* __restrict__ proj, int ld, __half* __restrict__ ql, const SeqDesc* __restrict__ seqs,
                    const int* __restrict__ row_seq, const int* __restrict__ rows, int n) {
    __shared__ float qs[kQueryRows][256];
    __shared__ float part[8][kQueryRows][kQueryCols];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, i0 = blockIdx.y * kQueryRows, nr = min(kQueryRows, n - i0);
    const int col = blockIdx.z * kQueryCols + lane * 8;
    const bool live = h < c.H && col < c.Rp;
    constexpr int AHEAD = 8;  // weights on the way before the rows are there
    uint4 w[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
        w[u] = make_uint4(0u, 0u, 0u, 0u);
        const int d = warp + u * 8;
        if (live && d < c.D) w[u] = __ldg(reinterpret_cast<const uint4*>(c.Wuk + (size_t)(h * c.D + d) * c.Rp + col));
    }
    griddep_wait();
    griddep_launch_dependents();
    auto sequence = [&](int row) { return seqs + (row_seq ? row_seq[row] : row); };
    if (h == c.H) {
        if (blockIdx.z == 0 && warp < nr) {
            const int row = rows ? rows[i0 + warp] : i0 + warp;
            const SeqDesc* sd = sequence(row);
            const int pos = sd->pos0 + row - sd->row0;
            latent_row<__half>(c, proj + (size_t)row * ld + c.c_col, pos, static_cast<__half*>(c.cache) + ((size_t)sd->slot * c.Tp + pos) * c.Lp, static_cast<__half*>(nullptr), lane);
        }
        return;
    }
    const int Dq = c.D + c.Dr;
    for (int i = tid; i < kQueryRows * c.D; i += 256) {
        const int r = i / c.D, d = i - r * c.D;
        qs[r][d] = r < nr ? proj[(size_t)(rows ? rows[i0 + r] : i0 + r) * ld + c.q_col + h * Dq + d] : 0.f;
    }
    __syncthreads();
    float acc[kQueryRows][8];
#pragma unroll
    for (int r = 0; r < kQueryRows; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = 0.f;
    for (int d0 = warp; d0 < c.D; d0 += 8 * AHEAD) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int d = d0 + u * 8;
            if (d < c.D) {
                const uint32_t x[4] = {w[u].x, w[u].y, w[u].z, w[u].w};
#pragma unroll
                for (int r = 0; r < kQueryRows; ++r) {
                    const float q = qs[r][d];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        acc[r][2 * e] = fmaf(q, __uint_as_float(x[e] << 16), acc[r][2 * e]);
                        acc[r][2 * e + 1] = fmaf(q, __uint_as_float(x[e] & 0xffff0000u), acc[r][2 * e + 1]);
                    }
                }
            }
            const int dn = d + 8 * AHEAD;
            if (live && dn < c.D) w[u] = __ldg(reinterpret_cast<const uint4*>(c.Wuk + (size_t)(h * c.D + dn) * c.Rp + col));
        }
    }
#pragma unroll
    for (int r = 0; r < kQueryRows; ++r)
#pragma unroll
        for (int e = 0; e < 8; e += 4)
            *reinterpret_cast<float4*>(&part[warp][r][lane * 8 + e]) = make_float4(acc[r][e], acc[r][e + 1], acc[r][e + 2], acc[r][e + 3]);
    __syncthreads();
    for (int i = tid; i < nr * kQueryCols; i += 256) {
        const int r = i / kQueryCols, k = i - r * kQueryCols, d = blockIdx.z * kQueryCols + k;
        if (d >= c.R) continue;
        float s = 0.f;
#pragma unroll
        for (int p = 0; p < 8; ++p) s += part[p][r][k];
        ql[((size_t)(i0 + r) * c.H + h) * c.Lp + d] = latent_half(s);
    }
    if (blockIdx.z == 0 && warp < nr) {  // the rotated part, and zeros behind it
        const int row = rows ? rows[i0 + warp] : i0 + warp;
        const SeqDesc* sd = sequence(row);
        const int pos = sd->pos0 + row - sd->row0;
        const float* q = proj + (size_t)row * ld + c.q_col + h * Dq + c.D;
        const float2* rot = c.rot + (size_t)pos * (c.Dr >> 1);
        __half* out = ql + ((size_t)(i0 + warp) * c.H + h) * c.Lp + c.R;
        for (int i = lane; i < (c.Dr >> 1); i += 32) {
            const float2 cs = __ldg(rot + i);
            const float u = q[2 * i], v = q[2 * i + 1];
            out[2 * i] = latent_half(u * cs.x - v * cs.y);
            out[2 * i + 1] = latent_half(v * cs.x + u * cs.y);
        }
        for (int d = c.Dr + lane; d < c.Lp - c.R; d += 32) out[d] = __float2half_rn(0.f);
    }
}

// ------------------------------------------------------------------ attention over latents
// A cluster of `splits` CTAs per tile of 16 MT (token, head) pairs of one sequence, each with its share of the cached
// positions.  Positions go by in tiles of 64, staged two deep (cp.async): scores on m16n8k16 fp16 tensor-core instructions, a
// warp taking eight positions over the whole row; softmax by rows; then the same staged rows are the values, a warp taking
// 8 NTW columns.  (tcgen05 would want 64 rows or more of pairs and the probabilities in tensor memory or shared memory;
// a decoding token brings as many pairs as the model has heads.)  The splits' states are merged through the cluster's shared memory, each
// CTA for its share of the pairs, and goes on to the values: W_uv, a warp per output.
constexpr int kLatThreads = 256, kLatKeys = 64, kLatP = kLatKeys + 8, kLatS = kLatKeys + 4;

__device__ __forceinline__ float ld_cluster_f32(const float* p, int rank) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(map_to_cta(smem_u32(p), rank)) : "memory");
    return v;
}
__device__ __forceinline__ float4 ld_cluster_f32x4(const float* p, int rank) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(map_to_cta(smem_u32(p), rank)) : "memory");
    return v;
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t (&r)[2], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

inline size_t latent_smem(int Lp, int MT) {
    const size_t row = (size_t)(Lp + 8) * 2;
    return 2 * kLatKeys * row + 16 * MT * row + (size_t)16 * MT * (kLatS * 4 + kLatP * 2);
}

template <int MT, int NTW>
__global__ void __launch_bounds__(kLatThreads)
latent_attention_kernel(const LatentAttention c, const __half* __restrict__ ql, void* out, int ldo, const SeqDesc* __restrict__ seqs,
                        const int* __restrict__ list, int splits, bool split_rows) {
    extern __shared__ __align__(16) uint8_t raw[];
    __shared__ float stat_m[16 * MT], stat_l[16 * MT], stat_a[16 * MT], weight[16 * MT][8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c2 = (lane & 3) * 2;
    const int ld = c.Lp + 8;  // halves
    __half* ks = reinterpret_cast<__half*>(raw);           // [2][64][ld]
    __half* qs = ks + 2 * kLatKeys * ld;                   // [16 MT][ld]
    float* ss = reinterpret_cast<float*>(qs + 16 * MT * ld);  // [16 MT][kLatS]
    __half* ps = reinterpret_cast<__half*>(ss + 16 * MT * kLatS);  // [16 MT][kLatP]
    // Descriptors, lists and the rows that earlier steps cached were there before the previous kernel started (every kernel of a
    // step waits for the one before it), and weights always: they are asked for before that kernel has finished.
    const int z = blockIdx.x % splits;
    const SeqDesc sd = seqs[list ? list[blockIdx.y] : blockIdx.y];
    const int pair0 = blockIdx.x / splits * 16 * MT, np = min(16 * MT, sd.n * c.H - pair0);  // (token, head) pairs
    if (np <= 0) return;  // (the whole cluster)
    const int mine = z < np ? (np - z + splits - 1) / splits : 0;  // pairs z, z + splits, ... are this CTA's to finish
    if (tid < min(mine, c.H)) l2_prefetch_bulk(c.Wuv + (size_t)((pair0 + z + tid * splits) % c.H) * c.Dv * c.Rp, (uint32_t)c.Dv * c.Rp * 2);
    const int keys = sd.pos0 + (pair0 + np - 1) / c.H + 1;
    const int per = ((keys + splits - 1) / splits + kLatKeys - 1) / kLatKeys * kLatKeys;
    const int t_begin = min(keys, z * per), t_end = min(keys, t_begin + per);
    const __half* rows = static_cast<const __half*>(c.cache) + (size_t)sd.slot * c.Tp * c.Lp;
    const int p16 = c.Lp >> 3;  // 16-byte pieces of a row
    auto stage = [&](int t0, int buf) {
        __half* dst = ks + buf * kLatKeys * ld;
        const int nk = min(kLatKeys, t_end - t0);
        for (int p = lane; p < p16; p += 32) {  // a warp per row
#pragma unroll
            for (int i = 0; i < kLatKeys / 8; ++i) {
                const int r = warp + i * 8;
                if (r < nk) cp_async16(dst + r * ld + p * 8, rows + (size_t)(t0 + r) * c.Lp + p * 8);
                else *reinterpret_cast<uint4*>(dst + r * ld + p * 8) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
        cp_async_commit();
    };
    const bool early = t_begin < t_end && min(t_end, t_begin + kLatKeys) <= sd.pos0;  // rows of earlier steps only
    if (early) stage(t_begin, 0);
    griddep_wait();
    griddep_launch_dependents();
    {
        const __half* q = ql + ((size_t)sd.lat0 * c.H + pair0) * c.Lp;
        for (int p = lane; p < p16; p += 32) {
#pragma unroll
            for (int i = 0; i < 2 * MT; ++i) {
                const int r = warp + i * 8;
                if (r < np) cp_async16(qs + r * ld + p * 8, q + (size_t)r * c.Lp + p * 8);
                else *reinterpret_cast<uint4*>(qs + r * ld + p * 8) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
    }
    if (!early && t_begin < t_end) stage(t_begin, 0);
    else cp_async_commit();
    if (tid < 16 * MT) { stat_m[tid] = -INFINITY; stat_l[tid] = 0.f; }
    const float scale = c.scale * 1.4426950408889634f;
    float o[MT][NTW][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < NTW; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
    const int oc0 = warp * 8 * NTW;
    for (int t0 = t_begin, n = 0; t0 < t_end; t0 += kLatKeys, ++n) {
        if (t0 + kLatKeys < t_end) { stage(t0 + kLatKeys, (n + 1) & 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const __half* kt = ks + (n & 1) * kLatKeys * ld;
        {
            float s[MT][2][4];  // two chains per tile of pairs
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int x = 0; x < 2; ++x) s[m][x][0] = s[m][x][1] = s[m][x][2] = s[m][x][3] = 0.f;
            const __half* kb = kt + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;
            const __half* qa = qs + (lane & 15) * ld + (lane >> 4) * 8;
            const int steps = c.Lp >> 4;
#pragma unroll 2
            for (int k = 0; k < steps; k += 2) {
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    if (k + x >= steps) break;
                    uint32_t b[2];
                    ldmatrix_x2(b, kb + (k + x) * 16);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        uint32_t a[4];
                        ldmatrix_x4(a, qa + m * 16 * ld + (k + x) * 16);
                        mma_f16(s[m][x], a, b[0], b[1]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = m * 16 + g + (e >> 1) * 8, key = warp * 8 + c2 + (e & 1), pair = pair0 + r;
                    const int last = min(t_end - 1, sd.pos0 + pair / c.H);  // the last position the pair may see
                    ss[r * kLatS + key] = (r < np && t0 + key <= last) ? (s[m][0][e] + s[m][1][e]) * scale : -INFINITY;
                }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2 * MT; ++i) {
            const int r = warp * 2 * MT + i;
            const float v0 = ss[r * kLatS + lane], v1 = ss[r * kLatS + lane + 32], m_old = stat_m[r];
            float m = fmaxf(v0, v1);
#pragma unroll
            for (int d = 16; d >= 1; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
            m = fmaxf(m, m_old);
            const float ref = m == -INFINITY ? 0.f : m;  // (a pair that has seen nothing yet)
            const float p0 = ex2(v0 - ref), p1 = ex2(v1 - ref);
            ps[r * kLatP + lane] = __float2half_rn(p0);
            ps[r * kLatP + lane + 32] = __float2half_rn(p1);
            const float s = warp_sum(p0 + p1);
            if (lane == 0) {
                const float al = ex2(m_old - ref);
                stat_a[r] = al;
                stat_m[r] = m;
                stat_l[r] = stat_l[r] * al + s;
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float a0 = stat_a[m * 16 + g], a1 = stat_a[m * 16 + g + 8];
#pragma unroll
            for (int j = 0; j < NTW; ++j) { o[m][j][0] *= a0; o[m][j][1] *= a0; o[m][j][2] *= a1; o[m][j][3] *= a1; }
        }
#pragma unroll
        for (int k = 0; k < kLatKeys / 16; ++k) {
            uint32_t a[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) ldmatrix_x4(a[m], ps + (m * 16 + (lane & 15)) * kLatP + k * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int j = 0; j < NTW; j += 2) {
                if (oc0 + j * 8 < c.R) {  // (two blocks of eight columns: rows are whole 16s long)
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, kt + (k * 16 + (lane & 15)) * ld + oc0 + j * 8 + (lane >> 4) * 8);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_f16(o[m][j], a[m], b[0], b[1]);
                        mma_f16(o[m][j + 1], a[m], b[2], b[3]);
                    }
                }
            }
        }
        __syncthreads();  // the tile and the probabilities may be written again
    }
    cp_async_wait<0>();
    __syncthreads();
    // this split's sums, where the staged rows were; then the merged ones of this CTA's pairs behind them
    const int ldf = c.Rp + (c.Rp % 32 == 0 ? 8 : 0);  // (at most Lp + 8)
    float* os = reinterpret_cast<float*>(ks);
    float* om = reinterpret_cast<float*>(ks + kLatKeys * ld);
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < NTW; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = m * 16 + g + (e >> 1) * 8, d = oc0 + j * 8 + c2 + (e & 1);
                if (d < c.Rp) os[r * ldf + d] = o[m][j][e];
            }
    // the values: W_uv, a warp working on U outputs at a time, 256 latent columns in a step; a step's weights are on their way during
    // the step before, the first ones' during the merge
    constexpr int U = 8;
    const int outputs = mine * c.Dv, chunks = (c.Rp + 255) >> 8;
    uint4 w[U];
    auto fetch = [&](int i0, int d0) {
        const bool live = i0 < outputs && d0 < c.Rp;
        int k = min(i0, max(outputs - 1, 0)) / c.Dv, v = i0 - k * c.Dv, h = (pair0 + z + k * splits) % c.H;
#pragma unroll
        for (int u = 0; u < U; ++u) {
            w[u] = make_uint4(0u, 0u, 0u, 0u);
            if (live && i0 + u < outputs) w[u] = __ldg(reinterpret_cast<const uint4*>(c.Wuv + (size_t)(h * c.Dv + v) * c.Rp + d0));
            if (++v == c.Dv) { v = 0; ++k; h = (pair0 + z + k * splits) % c.H; }
        }
    };
    fetch(warp * U, lane * 8);
    if (splits > 1) cluster_sync_all();
    else __syncthreads();
    if (tid < mine * 8) {  // a split's share in a pair's sum
        const int k = tid >> 3, s = tid & 7, r = z + k * splits;
        float m = s < splits ? (splits > 1 ? ld_cluster_f32(stat_m + r, s) : stat_m[r]) : -INFINITY, top = m;
        const float l = s < splits ? (splits > 1 ? ld_cluster_f32(stat_l + r, s) : stat_l[r]) : 0.f;
        const uint32_t group = 0xffu << (lane & 24);
#pragma unroll
        for (int d = 1; d < 8; d <<= 1) top = fmaxf(top, __shfl_xor_sync(group, top, d));
        const float e = ex2(m - top);  // 0 for a split that saw no key of the pair's
        float sum = l * e;
#pragma unroll
        for (int d = 1; d < 8; d <<= 1) sum += __shfl_xor_sync(group, sum, d);
        weight[k][s] = e / sum;
    }
    __syncthreads();
    const int r4 = c.Rp >> 2;  // (columns R .. Rp of the sums belong to the rotated part: their weights in W_uv are zeros)
    for (int i = tid; i < mine * r4; i += kLatThreads) {
        const int k = i / r4, d = (i - k * r4) * 4;
        const float* src = os + (z + k * splits) * ldf + d;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f), x[8];
#pragma unroll
        for (int s = 0; s < 8; ++s) {
            x[s] = v;
            if (s < splits) x[s] = splits > 1 ? ld_cluster_f32x4(src, s) : *reinterpret_cast<const float4*>(src);
        }
#pragma unroll
        for (int s = 0; s < 8; ++s) {
            const float w8 = weight[k][s];
            v.x = fmaf(x[s].x, w8, v.x); v.y = fmaf(x[s].y, w8, v.y); v.z = fmaf(x[s].z, w8, v.z); v.w = fmaf(x[s].w, w8, v.w);
        }
        *reinterpret_cast<float4*>(om + k * ldf + d) = v;
    }
    __syncthreads();
    for (int i0 = warp * U; i0 < outputs; i0 += 8 * U) {
        float acc[U];
#pragma unroll
        for (int u = 0; u < U; ++u) acc[u] = 0.f;
        for (int ch = 0; ch < chunks; ++ch) {
            const int d0 = ch * 256 + lane * 8;
            uint4 x[U];
#pragma unroll
            for (int u = 0; u < U; ++u) x[u] = w[u];
            if (ch + 1 < chunks) fetch(i0, d0 + 256);
            else fetch(i0 + 8 * U, lane * 8);
            if (d0 >= c.Rp) continue;
            int k = i0 / c.Dv, v = i0 - k * c.Dv;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const float4 x0 = *reinterpret_cast<const float4*>(om + k * ldf + d0), x1 = *reinterpret_cast<const float4*>(om + k * ldf + d0 + 4);
                const float z8[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
                const uint32_t y[4] = {x[u].x, x[u].y, x[u].z, x[u].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[u] = fmaf(__uint_as_float(y[e] << 16), z8[2 * e], acc[u]);
                    acc[u] = fmaf(__uint_as_float(y[e] & 0xffff0000u), z8[2 * e + 1], acc[u]);
                }
                if (++v == c.Dv) { v = 0; k = min(k + 1, mine - 1); }  // (outputs beyond the end: weights of zero)
            }
        }
        reduce_scatter<U, 32>(acc, lane);
        const int i = i0 + scatter_first<U, 32>(lane);
        if (i < outputs && scatter_owner<U, 32>(lane)) {
            const int k = i / c.Dv, pair = pair0 + z + k * splits, h = pair % c.H, row = sd.row0 + pair / c.H, col = h * c.Dv + i - k * c.Dv;
            if (split_rows) store_split(static_cast<uint8_t*>(out) + (size_t)row * ldo * 4, col, acc[0]);
            else store1<false>(out, (size_t)row * ldo + col, acc[0]);
        }
    }
    if (splits > 1) cluster_sync_all();  // nobody leaves while its sums are being read
}

template <int MT, int NTW>
int launch_latent_one(b200_ctx* ctx, const LatentAttention& c, const void* ql, void* out, int ldo, const SeqDesc* seqs, const int* list, int n, int max_n,
                      int max_keys, bool split_rows) {
    const size_t smem = latent_smem(c.Lp, MT);
    static size_t attr_set[64] = {};
    if (attr_set[ctx->device & 63] < smem) {
        B200_CUDA(ctx, cudaFuncSetAttribute(latent_attention_kernel<MT, NTW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set[ctx->device & 63] = smem;
    }
    const int per_seq = (int)(((long)max_n * c.H + 16 * MT - 1) / (16 * MT));
    int splits = 1;
    while (splits < 8 && (long)n * per_seq * splits * 2 <= ctx->num_sms && splits * 2 * kLatKeys <= max_keys) splits *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(per_seq * splits, n);
    cfg.blockDim = dim3(kLatThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    int na = 0;
    if (splits > 1) {
        attr[na].id = cudaLaunchAttributeClusterDimension;
        attr[na].val.clusterDim.x = splits;
        attr[na].val.clusterDim.y = attr[na].val.clusterDim.z = 1;
        ++na;
    }
    if (ctx->pdl) {
        attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[na].val.programmaticStreamSerializationAllowed = 1;
        ++na;
    }
    cfg.attrs = attr;
    cfg.numAttrs = na;
    const cudaError_t le = cudaLaunchKernelEx(&cfg, latent_attention_kernel<MT, NTW>, c, static_cast<const __half*>(ql), out, ldo, seqs, list, splits, split_rows);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

template <int MT>
int launch_latent_mt(b200_ctx* ctx, const LatentAttention& c, const void* ql, void* out, int ldo, const SeqDesc* seqs, const int* list, int n, int max_n,
                     int max_keys, bool split_rows) {
    if (c.R <= 128) return launch_latent_one<MT, 2>(ctx, c, ql, out, ldo, seqs, list, n, max_n, max_keys, split_rows);
    if (c.R <= 256) return launch_latent_one<MT, 4>(ctx, c, ql, out, ldo, seqs, list, n, max_n, max_keys, split_rows);
    return launch_latent_one<MT, 8>(ctx, c, ql, out, ldo, seqs, list, n, max_n, max_keys, split_rows);
}

}  // namespace

int latent_row_pad(int r) {
    if (r > kMaxRow) return 0;
    return r < 64 ? 64 : (r + 15) & ~15;
}

int launch_latent_prep(b200_ctx* ctx, const LatentAttention& c, const float* proj, int ld, void* q_out, void* lat, const SeqDesc* seqs, const int* row_seq,
                       int M, bool f32) {
    if (c.R > kMaxLatent) return B200_ERR_LIMIT;
    const dim3 grid((M + 7) / 8), block(256);
    cudaError_t le = f32 ? launch_pdl(ctx, latent_prep_kernel<float>, grid, block, 0, c, proj, ld, static_cast<float*>(q_out), static_cast<float*>(lat), seqs, row_seq, M)
                         : launch_pdl(ctx, latent_prep_kernel<__half>, grid, block, 0, c, proj, ld, static_cast<__half*>(q_out), static_cast<__half*>(lat), seqs, row_seq, M);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_latent_gather(b200_ctx* ctx, const LatentAttention& c, void* lat, const SeqDesc* seqs, int E, int max_pos0, bool f32) {
    const size_t pieces = (size_t)max_pos0 * c.Lp * (f32 ? 4 : 2) / 16;
    const unsigned blocks = (unsigned)((pieces + 1023) / 1024);
    const dim3 grid(blocks < 256u ? blocks : 256u, E), block(256);
    cudaError_t le = f32 ? launch_pdl(ctx, latent_gather_kernel<float>, grid, block, 0, c, static_cast<float*>(lat), seqs)
                         : launch_pdl(ctx, latent_gather_kernel<__half>, grid, block, 0, c, static_cast<__half*>(lat), seqs);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_latent_query(b200_ctx* ctx, const LatentAttention& c, const float* proj, int ld, void* ql, const SeqDesc* seqs, const int* row_seq,
                        const int* rows, int n, bool append) {
    if (c.D > 256 || c.R > kMaxLatent) return B200_ERR_LIMIT;
    const dim3 grid(c.H + (append ? 1 : 0), (n + kQueryRows - 1) / kQueryRows, (c.R + kQueryCols - 1) / kQueryCols);
    cudaError_t le = launch_pdl(ctx, latent_query_kernel, grid, dim3(256), 0, c, proj, ld, static_cast<__half*>(ql), seqs, row_seq, rows, n);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_latent_attention(b200_ctx* ctx, const LatentAttention& c, const void* ql, void* out, int ldo, const SeqDesc* seqs, const int* list, int n, int max_n,
                            int max_keys, bool split_rows) {
    // tiles of 32 pairs read the rows once for twice as many, tiles of 16 take half as long
    const long pairs = (long)max_n * c.H;
    if (pairs > 16 && (pairs + 15) / 16 * n * 8 > ctx->num_sms) return launch_latent_mt<2>(ctx, c, ql, out, ldo, seqs, list, n, max_n, max_keys, split_rows);
    return launch_latent_mt<1>(ctx, c, ql, out, ldo, seqs, list, n, max_n, max_keys, split_rows);
}

}  // namespace b200
