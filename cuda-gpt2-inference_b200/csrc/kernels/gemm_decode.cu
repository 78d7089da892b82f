// Matrix products of a decode step: B <= 16 input rows against bf16 weights [N, K].
//
// The step is bound by reading every weight once, so the kernel is built around that stream: a CTA takes 16
// rows of W, its eight warps take alternating 32-column pieces of them (16 bytes per lane and row, several
// pieces requested before any is used), and the partial sums meet in shared memory.  The arithmetic runs on
// m16n8k16 bf16 tensor-core instructions with the weights as the 16-row operand: at 8 or 16 input rows the
// FMA pipe could not keep up with HBM.  (tcgen05's smallest M is 64 rows of either operand through shared
// memory; with 8 useful columns it would move the weights twice for nothing.)  The input rows are kept as two
// bf16 terms, value = hi + lo, so activations enter with 16 significant bits and the weights exactly.
//
// Which k an instruction's register holds is free as long as both operands agree: lane (g, c) of a warp reads
// elements 8c .. 8c+7 of rows g and g + 8 of a 32-column piece in one go, and instruction s of the piece uses
// elements 8c + 4s .. + 3 of both operands.
//
// Prologues (see DecodeGemmArgs) form the input rows in every CTA for itself, as the skinny product of
// decode.cu does with its layernorm: the residual add between two RMS norms, the embedding, or a short
// convolution are a few KB per CTA and save a launch each.
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 256, kWarps = 8;
constexpr int kU = 4;               // pieces of a warp requested ahead
constexpr int kPlainChunk = 2048;   // columns of a plain input staged at a time
constexpr int kMaxSmem = 200 * 1024;

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t a0, const uint32_t a1, const uint32_t a2, const uint32_t a3,
                                         const uint32_t b0, const uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// eight fp32 values (32 bytes) -> the same 32 bytes as eight bf16 and the eight bf16 of what that dropped
__device__ __forceinline__ void split8(float4 a, float4 b, uint4& hi, uint4& lo) {
    const float v[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
    uint32_t h[4], l[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        h[i] = pack_bf16(v[2 * i], v[2 * i + 1]);
        l[i] = pack_bf16(v[2 * i] - __uint_as_float(h[i] << 16), v[2 * i + 1] - __uint_as_float(h[i] & 0xffff0000u));
    }
    hi = make_uint4(h[0], h[1], h[2], h[3]);
    lo = make_uint4(l[0], l[1], l[2], l[3]);
}

// Input rows in shared memory: row b at b * stride, groups of eight columns as 16 bytes of hi and 16 of lo.
// stride = 4 * columns + 16, so that the lanes of a quarter warp (two rows, four groups) touch all banks once.
//
// Narrow outputs: K is cut into slices computed by the CTAs of a cluster (blockIdx.x / cluster size = first tile),
// whose partial sums the first of them reads out of the others' shared memory, in rank order.
template <int NT, int PRO>  // NT: blocks of eight input rows
__global__ void __launch_bounds__(kThreads)
decode_gemm_kernel(const DecodeGemmArgs a, const int slices, const int kslice) {
    extern __shared__ __align__(16) uint8_t xs[];
    __shared__ float red[NT][kWarps][16][9];
    __shared__ float part[NT * 128];
    __shared__ float red1[kWarps];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int K = a.K, N = a.N, B = a.B;
    const int tiles = (N + 15) >> 4;
    const int rank = slices > 1 ? (int)cluster_ctarank() : 0;
    const int tile0 = blockIdx.x / slices, tile_step = gridDim.x / slices;
    const int kb = min(K, rank * kslice), ke = min(K, kb + kslice);  // this CTA's columns (may be none)
    const int chunk = PRO == DPRO_PLAIN ? min(kslice, kPlainChunk) : kslice;  // staged columns
    const int stride = chunk * 4 + 16;
    const uint16_t* __restrict__ W = a.W;
    // this warp's pieces of a chunk: 32 columns each, number warp, warp + 8, ...
    uint4 w[kU][2];
    auto request = [&](int tile, int k0, int kend, int p0) {
#pragma unroll
        for (int u = 0; u < kU; ++u) {
            const int k = k0 + (p0 + u * kWarps) * 32 + c * 8;
            const int r0 = tile * 16 + g, r1 = r0 + 8;
            w[u][0] = w[u][1] = make_uint4(0u, 0u, 0u, 0u);
            if (k < kend) {
                if (r0 < N) w[u][0] = __ldg(reinterpret_cast<const uint4*>(W + (size_t)r0 * K + k));
                if (r1 < N) w[u][1] = __ldg(reinterpret_cast<const uint4*>(W + (size_t)r1 * K + k));
            }
        }
    };
    // the weights do not depend on the previous kernel: their first pieces are on the way while it finishes
    request(tile0, kb, min(ke, kb + chunk), warp);
    griddep_wait();
    griddep_launch_dependents();

    if (PRO == DPRO_RESIDUAL) {  // (never sliced: the norms want whole rows)
        // 256 / NR threads per row, NR = rows handled at a time; x and y arrive by asynchronous copies, all at once
        const int NR = B > 4 ? 8 : (B > 2 ? 4 : B);
        const int tpr = kThreads / NR, rsub = tid / tpr, t = tid - rsub * tpr;
        const int K4 = K >> 2, K8 = K >> 3;
        const float inv_c = 1.0f / (float)a.C;
        float* ys = reinterpret_cast<float*>(xs + (size_t)NT * 8 * stride) + (size_t)rsub * K;
        auto row_sum = [&](float v) {  // over the threads of a row (32 or more of them)
            v = warp_sum(v);
            if (tpr == 32) return v;
            __syncthreads();
            if (lane == 0) red1[warp] = v;
            __syncthreads();
            float s = 0.f;
            const int w0 = rsub * (tpr >> 5);
            for (int i = 0; i < (tpr >> 5); ++i) s += red1[w0 + i];
            return s;
        };
        const int used = (B + NR - 1) / NR * NR;  // rows formed below; the rest of the operand is zero
        for (int i = tid; i < (NT * 8 - used) * (stride >> 4); i += kThreads)
            reinterpret_cast<uint4*>(xs + (size_t)used * stride)[i] = make_uint4(0u, 0u, 0u, 0u);
        for (int b0 = 0; b0 < used; b0 += NR) {
            const int b = b0 + rsub;
            const bool live = b < B;
            uint8_t* xrow = xs + (size_t)b * stride;
            int tok = 0;
            if (live) {
                if (a.tok) {
                    tok = a.tok[b];
                    if (tok < 0 || tok >= a.vocab) { if (t == 0 && blockIdx.x == 0) atomicCAS(a.status, 0, 201); tok = 0; }
                } else {
                    for (int i = t; i < K4; i += tpr) cp_async16(xrow + i * 16, a.x + (size_t)b * K + i * 4);
                }
                if (a.y) for (int i = t; i < K4; i += tpr) cp_async16(ys + i * 4, a.y + (size_t)b * K + i * 4);
            }
            cp_async_commit();
            cp_async_wait<0>();  // a thread reads back only what it has copied itself
            float rstd_y = 0.f;
            if (a.y) {
                float s = 0.f;
                if (live) {
#pragma unroll 4
                    for (int i = t; i < K4; i += tpr) s += sq4(load4(ys, i));
                }
                rstd_y = 1.0f / sqrtf(row_sum(s) * inv_c + a.eps);
            }
            float s = 0.f;
#pragma unroll 4
            for (int i = t; i < K4; i += tpr) {  // float4 number i of the row
                float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
                if (live) {
                    if (a.tok) {
                        r = load4(a.embed + (size_t)tok * K, i);
                        r.x *= a.embed_scale; r.y *= a.embed_scale; r.z *= a.embed_scale; r.w *= a.embed_scale;
                    } else r = *reinterpret_cast<const float4*>(xrow + i * 16);
                    if (a.y) {
                        const float4 yv = load4(ys, i), wv = __ldg(reinterpret_cast<const float4*>(a.wb) + i);
                        r.x += yv.x * rstd_y * wv.x; r.y += yv.y * rstd_y * wv.y; r.z += yv.z * rstd_y * wv.z; r.w += yv.w * rstd_y * wv.w;
                    }
                    if (blockIdx.x == 0) *(reinterpret_cast<float4*>(a.x_out + (size_t)b * K) + i) = r;
                }
                s += sq4(r);
                *reinterpret_cast<float4*>(xrow + i * 16) = r;
            }
            const float rstd = 1.0f / sqrtf(row_sum(s) * inv_c + a.eps);
            __syncthreads();  // a group of eight columns may have been formed by two threads
#pragma unroll 2
            for (int i = t; i < K8; i += tpr) {
                float4* p = reinterpret_cast<float4*>(xrow + i * 32);
                float4 v0 = p[0], v1 = p[1];
                const float4 w0 = __ldg(reinterpret_cast<const float4*>(a.w) + 2 * i), w1 = __ldg(reinterpret_cast<const float4*>(a.w) + 2 * i + 1);
                v0.x *= rstd * w0.x; v0.y *= rstd * w0.y; v0.z *= rstd * w0.z; v0.w *= rstd * w0.w;
                v1.x *= rstd * w1.x; v1.y *= rstd * w1.y; v1.z *= rstd * w1.z; v1.w *= rstd * w1.w;
                uint4 hi, lo;
                split8(v0, v1, hi, lo);
                reinterpret_cast<uint4*>(p)[0] = hi;
                reinterpret_cast<uint4*>(p)[1] = lo;
            }
        }
    } else if (PRO == DPRO_CONV) {
        const int hist_rows = a.taps - 1, n8 = (ke - kb) >> 3;
        const bool writer = tile0 == 0;  // the CTAs of the first tile store what they form of their columns
        for (int i = tid; i < NT * 8 * n8; i += kThreads) {
            const int b = i / n8, k = kb + (i - b * n8) * 8;
            float4 v[2] = {make_float4(0.f, 0.f, 0.f, 0.f), make_float4(0.f, 0.f, 0.f, 0.f)};
            if (b < B) {
                const SeqDesc sd = a.seqs[b];
                const float* hr = a.hist + ((size_t)sd.bank * a.max_slots + sd.slot) * hist_rows * K;
                float* hw = a.hist + ((size_t)(sd.bank ^ 1) * a.max_slots + sd.slot) * hist_rows * K;
#pragma unroll
                for (int q = 0; q < 2; ++q) {
                    const int k4 = (k >> 2) + q;
                    float4 acc = __ldg(reinterpret_cast<const float4*>(a.conv_b) + k4);
#pragma unroll 4
                    for (int j = 0; j < a.taps; ++j) {
                        const int back = a.taps - 1 - j;  // tokens before the current one
                        float4 xv = make_float4(0.f, 0.f, 0.f, 0.f);
                        if (back == 0) xv = load4(a.x + (size_t)b * a.ldx, k4);
                        else if (back <= sd.pos0) xv = load4(hr + (size_t)j * K, k4);
                        if (writer && j > 0) *(reinterpret_cast<float4*>(hw + (size_t)(j - 1) * K) + k4) = xv;
                        const float4 wv = __ldg(reinterpret_cast<const float4*>(a.conv_w + (size_t)j * K) + k4);
                        acc.x = fmaf(xv.x, wv.x, acc.x); acc.y = fmaf(xv.y, wv.y, acc.y);
                        acc.z = fmaf(xv.z, wv.z, acc.z); acc.w = fmaf(xv.w, wv.w, acc.w);
                    }
                    v[q] = make_float4(silu(acc.x), silu(acc.y), silu(acc.z), silu(acc.w));
                    if (writer) *(reinterpret_cast<float4*>(a.conv_out + (size_t)b * K) + k4) = v[q];
                }
            }
            uint4 hi, lo;
            split8(v[0], v[1], hi, lo);
            uint4* p = reinterpret_cast<uint4*>(xs + (size_t)b * stride + ((k - kb) >> 3) * 32);
            p[0] = hi;
            p[1] = lo;
        }
    }

    auto stage_plain = [&](int k0, int kend) {
        const int n8 = (kend - k0) >> 3, total = NT * 8 * n8;
        constexpr int Q = 4;  // groups of eight columns requested before any is used
        for (int i0 = tid; i0 < total; i0 += Q * kThreads) {
            float4 v[Q][2];
            int at[Q];
#pragma unroll
            for (int q = 0; q < Q; ++q) {
                const int i = i0 + q * kThreads, b = i / n8, j = i - b * n8;
                at[q] = i < total ? b * stride + j * 32 : -1;
                v[q][0] = v[q][1] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < total && b < B) {
                    const float* p = a.x + (size_t)b * a.ldx + k0 + j * 8;
                    v[q][0] = load4(p, 0);
                    v[q][1] = load4(p, 1);
                }
            }
#pragma unroll
            for (int q = 0; q < Q; ++q)
                if (at[q] >= 0) {
                    uint4 hi, lo;
                    split8(v[q][0], v[q][1], hi, lo);
                    uint4* p = reinterpret_cast<uint4*>(xs + at[q]);
                    p[0] = hi;
                    p[1] = lo;
                }
        }
    };

    bool staged = PRO != DPRO_PLAIN;  // a plain input of one chunk is staged once for all tiles
    if (staged) __syncthreads();
    for (int tile = tile0; tile < tiles; tile += tile_step) {
        float acc[NT][4];
#pragma unroll
        for (int t = 0; t < NT; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
        for (int k0 = kb; k0 < ke; k0 += chunk) {
            const int kend = min(ke, k0 + chunk);
            const int pieces = (kend - k0 + 31) >> 5;
            if (!staged) {
                if (k0 > kb || tile != tile0) __syncthreads();  // everyone is done with the previous chunk
                stage_plain(k0, kend);
                __syncthreads();
                if (kslice <= chunk) staged = true;
            }
            if (warp >= pieces) {
                // nothing of this chunk, but the first pieces of the next one still have to be requested
                if (kend < ke) request(tile, kend, min(ke, kend + chunk), warp);
                else if (tile + tile_step < tiles) request(tile + tile_step, kb, min(ke, kb + chunk), warp);
                continue;
            }
            for (int p0 = warp; p0 < pieces; p0 += kU * kWarps) {
                uint4 cur[kU][2];
#pragma unroll
                for (int u = 0; u < kU; ++u) { cur[u][0] = w[u][0]; cur[u][1] = w[u][1]; }
                if (p0 + kU * kWarps < pieces) request(tile, k0, kend, p0 + kU * kWarps);
                else if (kend < ke) request(tile, kend, min(ke, kend + chunk), warp);
                else if (tile + tile_step < tiles) request(tile + tile_step, kb, min(ke, kb + chunk), warp);
#pragma unroll
                for (int u = 0; u < kU; ++u) {
                    const int p = p0 + u * kWarps;
                    const int j = p * 4 + c;  // group of eight columns within the chunk
                    if (p < pieces) {
                        const bool in = k0 + j * 8 < kend;
#pragma unroll
                        for (int t = 0; t < NT; ++t) {
                            uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
                            if (in) {
                                const uint4* xp = reinterpret_cast<const uint4*>(xs + (size_t)(t * 8 + g) * stride + j * 32);
                                hi = xp[0];
                                lo = xp[1];
                            }
                            mma_bf16(acc[t], cur[u][0].x, cur[u][1].x, cur[u][0].y, cur[u][1].y, hi.x, hi.y);
                            mma_bf16(acc[t], cur[u][0].x, cur[u][1].x, cur[u][0].y, cur[u][1].y, lo.x, lo.y);
                            mma_bf16(acc[t], cur[u][0].z, cur[u][1].z, cur[u][0].w, cur[u][1].w, hi.z, hi.w);
                            mma_bf16(acc[t], cur[u][0].z, cur[u][1].z, cur[u][0].w, cur[u][1].w, lo.z, lo.w);
                        }
                    }
                }
            }
        }
        // accumulator element (row g / g + 8, input row 2c / 2c + 1) of every warp -> sums over the warps
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            red[t][warp][g][2 * c] = acc[t][0];
            red[t][warp][g][2 * c + 1] = acc[t][1];
            red[t][warp][g + 8][2 * c] = acc[t][2];
            red[t][warp][g + 8][2 * c + 1] = acc[t][3];
        }
        __syncthreads();
        if (slices > 1) {
            for (int i = tid; i < NT * 128; i += kThreads) {
                float v = 0.f;
#pragma unroll
                for (int q = 0; q < kWarps; ++q) v += red[i >> 7][q][i & 15][(i >> 4) & 7];
                part[i] = v;
            }
            cluster_sync_all();
        }
        if (rank == 0) {
            for (int i = tid; i < NT * 128; i += kThreads) {
                const int n = i & 15, b = i >> 4;
                const int row = tile * 16 + n;
                if (b < B && row < N) {
                    float v = 0.f;
                    if (slices > 1) {
                        for (int s = 0; s < slices; ++s) {
                            float p;
                            asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(p) : "r"(map_to_cta(smem_u32(part + i), s)) : "memory");
                            v += p;
                        }
                    } else {
#pragma unroll
                        for (int q = 0; q < kWarps; ++q) v += red[b >> 3][q][n][b & 7];
                    }
                    if (a.bias) v += __ldg(a.bias + row);
                    if (a.act == ACT_GELU_ERF) v = gelu_erf(v);
                    else if (a.act == ACT_GELU_TANH) v = gelu_tanh(v);
                    a.out[(size_t)b * a.ldo + row] = v;
                }
            }
        }
        if (slices > 1) cluster_sync_all();  // the partial sums have been read (and nobody leaves before that)
        else __syncthreads();
    }
}

template <int NT, int PRO>
int launch_one(b200_ctx* ctx, const DecodeGemmArgs& a) {
    static bool attr_set[64] = {};
    if (!attr_set[ctx->device & 63]) {
        B200_CUDA(ctx, cudaFuncSetAttribute(decode_gemm_kernel<NT, PRO>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem));
        attr_set[ctx->device & 63] = true;
    }
    const int tiles = (a.N + 15) / 16;
    // K slices while the CTAs of one wave (two per SM) are not used up and a warp keeps at least a piece
    int slices = 1;
    if (PRO != DPRO_RESIDUAL)
        while (slices < 8 && tiles * slices * 2 <= 2 * ctx->num_sms && a.K / (slices * 2) >= 256) slices *= 2;
    const int kslice = ((a.K + slices - 1) / slices + 31) / 32 * 32;
    const int chunk = PRO == DPRO_PLAIN ? (kslice < kPlainChunk ? kslice : kPlainChunk) : kslice;
    const int nr = a.B > 4 ? 8 : (a.B > 2 ? 4 : a.B);
    const size_t smem = (size_t)NT * 8 * (chunk * 4 + 16) + (PRO == DPRO_RESIDUAL && a.y ? (size_t)nr * a.K * 4 : 0);
    if (smem > (size_t)kMaxSmem) return B200_ERR_LIMIT;
    const int per_sm = smem > 100 * 1024 ? 1 : 2;
    int grid = tiles * slices;
    if (grid > per_sm * ctx->num_sms) grid = per_sm * ctx->num_sms / slices * slices;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(grid);
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (slices > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = slices;
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
    const cudaError_t le = cudaLaunchKernelEx(&cfg, decode_gemm_kernel<NT, PRO>, a, slices, kslice);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace

bool decode_gemm_fits(int K, int B) {
    return (size_t)(B <= 8 ? 8 : 16) * ((K + 31) / 32 * 128 + 16) + (size_t)(B > 8 ? 8 : B) * K * 4 + (B == 3 || (B > 4 && B < 8) ? (size_t)4 * K * 4 : 0) <= (size_t)kMaxSmem;
}

int launch_decode_gemm(b200_ctx* ctx, const DecodeGemmArgs& a, int prologue) {
    if (a.B < 1 || a.B > 16 || a.K % 8 || a.N < 1) return B200_ERR_SHAPE;
    if (a.B <= 8) {
        if (prologue == DPRO_RESIDUAL) return launch_one<1, DPRO_RESIDUAL>(ctx, a);
        if (prologue == DPRO_CONV) return launch_one<1, DPRO_CONV>(ctx, a);
        return launch_one<1, DPRO_PLAIN>(ctx, a);
    }
    if (prologue == DPRO_RESIDUAL) return launch_one<2, DPRO_RESIDUAL>(ctx, a);
    if (prologue == DPRO_CONV) return launch_one<2, DPRO_CONV>(ctx, a);
    return launch_one<2, DPRO_PLAIN>(ctx, a);
}

}  // namespace b200
