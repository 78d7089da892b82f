// Softmax attention whose keys and values are linear in one cached latent per token (LatentAttention, decoder_kernels.h).
//
//   latent_prep, latent_gather   the expanded form's inputs: latents of all positions side by side, rotated queries
//   latent_query                 the latent form's queries, q W_uk beside the rotated part (and, decoding, the cache append)
//   latent_attention             the latent form: all heads of a token read the same cached rows, which therefore serve as the
//                                keys and, their first R columns, as the values of a whole tile of (token, head) pairs
//   latent_value                 the weighted sums of latents through W_uv
#include <cstdlib>
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
// A CTA per tile of 16 MT (token, head) pairs of one sequence and share of its cached positions.  Positions go by in tiles of
// 64, staged two deep by bulk copies (one per row, so that rows can lie 16 bytes apart from whole bank rows): scores on
// m16n8k16 fp16 tensor-core instructions, a warp taking eight positions over the whole row; softmax by rows; then the
// same staged rows are the values, a warp taking 8 NTW columns.  (tcgen05 would want 64 rows or more of pairs; a decoding token
// brings as many as the model has heads.)  latent_value merges the shares and goes on to the values.
constexpr int kLatThreads = 256, kLatKeys = 64, kLatP = kLatKeys + 8, kLatS = kLatKeys + 4;

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
latent_attention_kernel(const LatentAttention c, const __half* __restrict__ ql, const LatentParts parts, const SeqDesc* __restrict__ seqs,
                        const int* __restrict__ list, int splits, int* status) {
    extern __shared__ __align__(128) uint8_t raw[];
    __shared__ float stat_m[16 * MT], stat_l[16 * MT], stat_a[16 * MT];
    __shared__ uint64_t full[2];
    __shared__ volatile int abort_flag;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c2 = (lane & 3) * 2;
    const int ld = c.Lp + 8;  // halves
    __half* ks = reinterpret_cast<__half*>(raw);           // [2][64][ld]
    __half* qs = ks + 2 * kLatKeys * ld;                   // [16 MT][ld]
    float* ss = reinterpret_cast<float*>(qs + 16 * MT * ld);  // [16 MT][kLatS]
    __half* ps = reinterpret_cast<__half*>(ss + 16 * MT * kLatS);  // [16 MT][kLatP]
    // Descriptors, lists and the rows that earlier steps cached were there before the previous kernel started (every kernel of a
    // step waits for the one before it): they are asked for before that kernel has finished.
    const int z = blockIdx.x % splits;
    const SeqDesc sd = seqs[list ? list[blockIdx.y] : blockIdx.y];
    const int pair0 = blockIdx.x / splits * 16 * MT, np = min(16 * MT, sd.n * c.H - pair0);  // (token, head) pairs
    if (np <= 0) return;
    if (tid == 0) {
        mbar_init(&full[0], 1);
        mbar_init(&full[1], 1);
        abort_flag = 0;
        fence_barrier_init();
    }
    if (tid < 16 * MT) { stat_m[tid] = -INFINITY; stat_l[tid] = 0.f; }
    __syncthreads();
    const int keys = sd.pos0 + (pair0 + np - 1) / c.H + 1;
    const int per = ((keys + splits - 1) / splits + 15) & ~15;
    const int t_begin = min(keys, z * per), t_end = min(keys, t_begin + per);
    const __half* rows = static_cast<const __half*>(c.cache) + (size_t)sd.slot * c.Tp * c.Lp;
    const int p16 = c.Lp >> 3;  // 16-byte pieces of a row
    auto stage = [&](int t0, int buf) {
        __half* dst = ks + buf * kLatKeys * ld;
        const int nk = min(kLatKeys, t_end - t0);
        if (warp == 0) {
            if (lane == 0) mbar_arrive_expect_tx(&full[buf], (uint32_t)nk * c.Lp * 2);
            __syncwarp();
            for (int r = lane; r < nk; r += 32) bulk_load(dst + r * ld, rows + (size_t)(t0 + r) * c.Lp, (uint32_t)c.Lp * 2, &full[buf]);
        }
        for (int r = nk + warp; r < kLatKeys; r += 8)  // (the last tile: rows behind the end are zeros)
            for (int p = lane; p < p16; p += 32) *reinterpret_cast<uint4*>(dst + r * ld + p * 8) = make_uint4(0u, 0u, 0u, 0u);
    };
    const bool early = t_begin < t_end && min(t_end, t_begin + kLatKeys) <= sd.pos0;  // rows of earlier steps only
    if (early) stage(t_begin, 0);
    griddep_wait();
    griddep_launch_dependents();
    if (!early && t_begin < t_end) stage(t_begin, 0);
    {
        const __half* q = ql + ((size_t)sd.lat0 * c.H + pair0) * c.Lp;
        for (int p = lane; p < p16; p += 32) {  // a warp per row
#pragma unroll
            for (int i = 0; i < 2 * MT; ++i) {
                const int r = warp + i * 8;
                if (r < np) cp_async16(qs + r * ld + p * 8, q + (size_t)r * c.Lp + p * 8);
                else *reinterpret_cast<uint4*>(qs + r * ld + p * 8) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
        cp_async_commit();
        cp_async_wait<0>();
    }
    const float scale = c.scale * 1.4426950408889634f;
    float o[MT][NTW][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < NTW; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
    const int oc0 = warp * 8 * NTW;
    for (int t0 = t_begin, n = 0; t0 < t_end; t0 += kLatKeys, ++n) {
        const bool more = t0 + kLatKeys < t_end;
        if (more) stage(t0 + kLatKeys, (n + 1) & 1);
        if (!__syncthreads_and(mbar_wait(&full[n & 1], (n >> 1) & 1, &abort_flag))) {
            if (tid == 0) {
                atomicCAS(status, 0, DEV_TIMEOUT_PRODUCER);
                volatile int none = 0;
                if (more) mbar_wait(&full[(n + 1) & 1], ((n + 1) >> 1) & 1, &none);  // its own copies in flight
            }
            return;
        }
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
    // this share's sums (a share without keys has none)
    const size_t pair_index = (size_t)sd.lat0 * c.H + pair0;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int r = m * 16 + g + e * 8;
            if (r >= np || t_begin >= t_end) continue;
            float* dst = parts.o + ((pair_index + r) * splits + z) * c.Rp;
#pragma unroll
            for (int j = 0; j < NTW; ++j) {
                const int d = oc0 + j * 8 + c2;
                if (d < c.Rp) *reinterpret_cast<float2*>(dst + d) = make_float2(o[m][j][2 * e], o[m][j][2 * e + 1]);
            }
        }
    if (tid < np) parts.ml[(pair_index + tid) * splits + z] = make_float2(stat_m[tid], stat_l[tid]);
}

// The shares' sums of four rows' head, merged, through W_uv: a warp works on four outputs at a time, lane l on latent columns 8l .. of
// each 256.
constexpr int kValueRows = 4, kMaxSplits = 16;
__global__ void __launch_bounds__(256)
latent_value_kernel(const LatentAttention c, const LatentParts parts, int splits, const int* __restrict__ rows, int n, void* out, int ldo, bool split_rows) {
    __shared__ __align__(16) float om[kValueRows][kMaxLatent];
    __shared__ float weight[kValueRows][kMaxSplits];
    constexpr int U = 4, CH = kMaxLatent / 256;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, i0 = blockIdx.y * kValueRows, nr = min(kValueRows, n - i0);
    uint4 w[U][CH];
    auto fetch = [&](int v0) {
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int x = 0; x < CH; ++x) {
                const int v = v0 + u, d = x * 256 + lane * 8;
                w[u][x] = make_uint4(0u, 0u, 0u, 0u);
                if (v < c.Dv && d < c.Rp) w[u][x] = __ldg(reinterpret_cast<const uint4*>(c.Wuv + (size_t)(h * c.Dv + v) * c.Rp + d));
            }
    };
    fetch(warp * U);
    griddep_wait();
    griddep_launch_dependents();
    if (warp < nr) {  // a share's weight in its pair's sum
        const float2 ml = lane < splits ? parts.ml[((size_t)(i0 + warp) * c.H + h) * splits + lane] : make_float2(-INFINITY, 0.f);
        float top = ml.x;
#pragma unroll
        for (int d = 16; d >= 1; d >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, d));  // finite: every pair sees key 0
        const float e = ex2(ml.x - top);
        const float sum = warp_sum(ml.y * e);
        if (lane < splits) weight[warp][lane] = e / sum;
    }
    __syncthreads();
    const int r4 = c.Rp >> 2;  // (columns R .. Rp of the sums belong to the rotated part: their weights in W_uv are zeros)
    for (int i = tid; i < kValueRows * r4; i += 256) {
        const int r = i / r4, d = (i - r * r4) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < nr) {
            const float* src = parts.o + ((size_t)(i0 + r) * c.H + h) * splits * c.Rp + d;
            for (int s0 = 0; s0 < splits; s0 += 8) {
                float4 x[8];
#pragma unroll
                for (int s = 0; s < 8; ++s) {
                    x[s] = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (s0 + s < splits && weight[r][s0 + s] > 0.f) x[s] = *reinterpret_cast<const float4*>(src + (size_t)(s0 + s) * c.Rp);
                }
#pragma unroll
                for (int s = 0; s < 8; ++s) {
                    const float f = s0 + s < splits ? weight[r][s0 + s] : 0.f;
                    v.x = fmaf(x[s].x, f, v.x); v.y = fmaf(x[s].y, f, v.y); v.z = fmaf(x[s].z, f, v.z); v.w = fmaf(x[s].w, f, v.w);
                }
            }
        }
        *reinterpret_cast<float4*>(&om[r][d]) = v;
    }
    __syncthreads();
    for (int v0 = warp * U; v0 < c.Dv; v0 += 8 * U) {
        float acc[U * kValueRows];
#pragma unroll
        for (int i = 0; i < U * kValueRows; ++i) acc[i] = 0.f;
#pragma unroll
        for (int x = 0; x < CH; ++x) {
            const int d = x * 256 + lane * 8;
            if (d >= c.Rp) continue;
#pragma unroll
            for (int r = 0; r < kValueRows; ++r) {
                const float4 a = *reinterpret_cast<const float4*>(&om[r][d]), b = *reinterpret_cast<const float4*>(&om[r][d + 4]);
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    float s = acc[u * kValueRows + r];
                    s = fmaf(__uint_as_float(w[u][x].x << 16), a.x, s); s = fmaf(__uint_as_float(w[u][x].x & 0xffff0000u), a.y, s);
                    s = fmaf(__uint_as_float(w[u][x].y << 16), a.z, s); s = fmaf(__uint_as_float(w[u][x].y & 0xffff0000u), a.w, s);
                    s = fmaf(__uint_as_float(w[u][x].z << 16), b.x, s); s = fmaf(__uint_as_float(w[u][x].z & 0xffff0000u), b.y, s);
                    s = fmaf(__uint_as_float(w[u][x].w << 16), b.z, s); s = fmaf(__uint_as_float(w[u][x].w & 0xffff0000u), b.w, s);
                    acc[u * kValueRows + r] = s;
                }
            }
        }
        fetch(v0 + 8 * U);
        reduce_scatter<U * kValueRows, 32>(acc, lane);
        const int t = scatter_first<U * kValueRows, 32>(lane), v = v0 + t / kValueRows, r = t % kValueRows;
        if (v < c.Dv && r < nr && scatter_owner<U * kValueRows, 32>(lane)) {
            const int row = rows ? rows[i0 + r] : i0 + r, col = h * c.Dv + v;
            if (split_rows) store_split(static_cast<uint8_t*>(out) + (size_t)row * ldo * 4, col, acc[0]);
            else store1<false>(out, (size_t)row * ldo + col, acc[0]);
        }
    }
}

template <int MT, int NTW>
int launch_latent_one(b200_ctx* ctx, const LatentAttention& c, const void* ql, const LatentParts& parts, const SeqDesc* seqs, const int* list, int n, int max_n,
                      int splits) {
    const size_t smem = latent_smem(c.Lp, MT);
    static size_t attr_set[64] = {};
    if (attr_set[ctx->device & 63] < smem) {
        B200_CUDA(ctx, cudaFuncSetAttribute(latent_attention_kernel<MT, NTW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set[ctx->device & 63] = smem;
    }
    const int per_seq = (int)(((long)max_n * c.H + 16 * MT - 1) / (16 * MT));
    cudaError_t le = launch_pdl(ctx, latent_attention_kernel<MT, NTW>, dim3(per_seq * splits, n), dim3(kLatThreads), smem, c, static_cast<const __half*>(ql), parts, seqs,
                                list, splits, ctx->d_status);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

template <int MT>
int launch_latent_mt(b200_ctx* ctx, const LatentAttention& c, const void* ql, const LatentParts& parts, const SeqDesc* seqs, const int* list, int n, int max_n,
                     int splits) {
    if (c.R <= 128) return launch_latent_one<MT, 2>(ctx, c, ql, parts, seqs, list, n, max_n, splits);
    if (c.R <= 256) return launch_latent_one<MT, 4>(ctx, c, ql, parts, seqs, list, n, max_n, splits);
    return launch_latent_one<MT, 8>(ctx, c, ql, parts, seqs, list, n, max_n, splits);
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

int launch_latent_attention(b200_ctx* ctx, const LatentAttention& c, const void* ql, const LatentParts& parts, void* out, int ldo, const SeqDesc* seqs,
                            const int* list, int n, const int* rows, int n_rows, int max_n, int max_keys, bool split_rows) {
    // shares of the positions, while there is room on the SMs and a share keeps a tile
    const long pairs = (long)max_n * c.H;
    const int resident = ctx->num_sms * (latent_smem(c.Lp, 1) > 112 * 1024 ? 1 : 2);
    // tiles of 32 pairs read the rows once for twice as many, tiles of 16 take half as long
    const int mt = pairs > 16 && (pairs + 15) / 16 * n * 4 > resident ? 2 : 1;
    const long tiles = (pairs + 16 * mt - 1) / (16 * mt) * n;
    long splits = resident / tiles;
    if (splits > (max_keys + kLatKeys - 1) / kLatKeys) splits = (max_keys + kLatKeys - 1) / kLatKeys;
    if (splits > kMaxSplits) splits = kMaxSplits;
    if (splits > parts.pairs / ((long)n_rows * c.H)) splits = parts.pairs / ((long)n_rows * c.H);
    static const int forced = [] { const char* e = getenv("B200_LATENT_SPLITS"); return e ? atoi(e) : 0; }();  // tuning hook: 1 .. 16
    if (forced >= 1 && forced <= kMaxSplits && forced <= parts.pairs / ((long)n_rows * c.H)) splits = forced;
    if (splits < 1) splits = 1;
    if ((long)n_rows * c.H > parts.pairs) return B200_ERR_LIMIT;
    const int st = mt == 2 ? launch_latent_mt<2>(ctx, c, ql, parts, seqs, list, n, max_n, (int)splits) : launch_latent_mt<1>(ctx, c, ql, parts, seqs, list, n, max_n, (int)splits);
    if (st != B200_OK) return st;
    cudaError_t le = launch_pdl(ctx, latent_value_kernel, dim3(c.H, (n_rows + kValueRows - 1) / kValueRows), dim3(256), 0, c, parts, (int)splits, rows, n_rows, out, ldo,
                                split_rows);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace b200
