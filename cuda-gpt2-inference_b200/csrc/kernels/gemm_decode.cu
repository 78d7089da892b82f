// Matrix products of a decode step: B <= 16 input rows against bf16 weights [N, K].
//
// The step is bound by reading every weight once, so the kernel is built around that stream: a CTA takes 16
// rows of W at a time, its eight warps take alternating 32-column pieces of them (16 bytes per lane and row), and a
// warp has eight pieces on the way at any time - a register is requested anew as soon as it has been used, across
// the borders of tiles too, and the first ones before the previous kernel has finished.  The partial sums of the
// warps meet in shared memory.  The arithmetic runs on m16n8k16 bf16 tensor-core instructions with the weights as
// the 16-row operand: at 8 or 16 input rows the FMA pipe could not keep up with HBM.  (tcgen05's smallest M is
// 64 rows, both operands through shared memory; with 8 useful columns it would move the weights twice for nothing.)
// The input rows are two bf16 terms, value = hi + lo, so activations enter with 16 significant bits and the
// weights exactly; their producers write them in that form (split rows, decoder_math.cuh).
//
// Which k an instruction's register holds is free as long as both operands agree: lane (g, c) of a warp reads
// elements 8c .. 8c+7 of rows g and g + 8 of a 32-column piece in one go, and instruction s of the piece uses
// elements 8c + 4s .. + 3 of both operands.
//
// Narrow outputs: K is cut into slices computed by the CTAs of a cluster, whose partial sums the first of them
// reads out of the others' shared memory, in rank order.
//
// Gated outputs: a tile is eight gate rows and their eight linear rows, so the two meet in the same epilogue.
//
// Table-routed experts (ROUTED): the tiles of all matrices that occur, and of the shared expert, are one sequence, cut into equal
// shares of weight bytes, and a matrix is multiplied with all rows at once, of which those that did not choose it are
// dropped.  (Which ones occur is read before the previous kernel has finished: it was there before that one started.)
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 256, kWarps = 8;
constexpr int kU = 8;             // pieces of a warp on the way
constexpr int kTwoCtaSmem = 103 * 1024;  // input rows of a CTA that still leave room for a second one ...
constexpr int kOneCtaSmem = 200 * 1024;  // ... and the most a CTA can hold
constexpr int kMaxTaps = 4;       // convolution inputs requested ahead of the product (longer ones behind it)

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t a0, const uint32_t a1, const uint32_t a2, const uint32_t a3,
                                         const uint32_t b0, const uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Input rows in shared memory: row b at b * stride, as in memory.  stride = 4 * columns + 16, so that the lanes of
// a quarter warp (two rows, four groups of eight columns) touch all banks once.
template <int NT, bool ROUTED>  // blocks of eight input rows
__global__ void __launch_bounds__(kThreads, 2)
decode_gemm_kernel(const DecodeGemmArgs a, const int slices, const int kslice, const int chunk) {
    extern __shared__ __align__(16) uint8_t xs[];
    __shared__ float red[NT][kWarps][16][9];
    __shared__ float part[NT * 128];
    __shared__ uint16_t expert[ROUTED ? kMaxPairs : 1], listed[ROUTED ? kMaxPairs : 1];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int B = a.B;
    const bool gated = a.gate != GATE_NONE;
    const int rank = slices > 1 ? (int)cluster_ctarank() : 0;
    const int stride = chunk * 4 + 16;
    // the cluster's tiles: item, item + step, ...
    const int tiles = (a.N + 15) >> 4;
    int item = blockIdx.x / slices, items = tiles, step = gridDim.x / slices, matrices = 1;
    if (ROUTED) {
        const int pairs = B * a.top;
        matrices = a.route->matrices;
        if (tid < pairs) {
            expert[tid] = a.route->expert[tid];
            listed[tid] = a.route->listed[tid];
        }
        __syncthreads();
        // shares of equal cost, in units of 64 columns of a tile, cut where a tile ends
        const unsigned shared_tiles = a.shared.W ? (a.shared.N + 15) >> 4 : 0, ku = (a.K + 63) >> 6, kus = (a.shared.K + 63) >> 6;
        const unsigned routed_cost = matrices * tiles * ku, cost = routed_cost + shared_tiles * kus, whole = cost / step, rest = cost % step;
        auto cut = [&](unsigned i) {
            const unsigned at = whole * i + rest * i / step;
            return (int)(at <= routed_cost ? (at + ku - 1) / ku : matrices * tiles + (at - routed_cost + kus - 1) / kus);
        };
        const int share = item;
        item = cut(share);
        items = cut(share + 1);
        step = 1;
    }
    struct Tile { const uint16_t* W; int N, K, kb, ke, tile, matrix; };  // kb .. ke: this CTA's columns (may be none)
    // (slices: a power of two)
    const int log_slices = __ffs(slices) - 1;
    auto tile_at = [&](int matrix, int tile) {
        Tile t;
        t.N = a.N; t.K = a.K; t.W = a.W; t.tile = tile; t.matrix = matrix;
        if (ROUTED) {
            if (matrix == matrices) { t.N = a.shared.N; t.K = a.shared.K; t.W = a.shared.W; }
            else t.W += (size_t)listed[matrix] * a.N * a.K;
        }
        const int ks = ROUTED ? (((t.K + slices - 1) >> log_slices) + 31) & ~31 : kslice;
        t.kb = min(t.K, rank * ks);
        t.ke = min(t.K, t.kb + ks);
        return t;
    };
    // row of input row b's products with the matrix (-1: it did not choose it)
    auto pair_row = [&](int b, const Tile& t) {
        if (!ROUTED || t.matrix == matrices) return b;
        const int e = listed[t.matrix];
        int r = -1;
        for (int j = 0; j < a.top; ++j) if (expert[b * a.top + j] == e) r = b * a.top + j;
        return r;
    };
    // this warp's pieces of a chunk: 32 columns each, number warp, warp + 8, ...
    uint4 w[kU][2];
    auto request = [&](uint4 (&r)[2], const Tile& t, int k0, int kend, int p) {
        const int k = k0 + p * 32 + c * 8;
        const int r0 = gated ? (t.tile >> 2) * 64 + (t.tile & 3) * 8 + g : t.tile * 16 + g, r1 = r0 + (gated ? 32 : 8);
        r[0] = r[1] = make_uint4(0u, 0u, 0u, 0u);
        if (k < kend) {
            if (r0 < t.N) r[0] = __ldg(reinterpret_cast<const uint4*>(t.W + (size_t)r0 * t.K + k));
            if (r1 < t.N) r[1] = __ldg(reinterpret_cast<const uint4*>(t.W + (size_t)r1 * t.K + k));
        }
    };
    const int matrix0 = ROUTED ? min(item / tiles, matrices) : 0;
    Tile now = tile_at(matrix0, item - matrix0 * tiles);
    const int item0 = item;
    if (item < items) {
#pragma unroll
        for (int u = 0; u < kU; ++u) request(w[u], now, now.kb, min(now.ke, now.kb + chunk), warp + u * kWarps);
    }
    for (int i = tid; i < (NT * 8 - B) * (stride >> 4); i += kThreads)
        reinterpret_cast<uint4*>(xs + (size_t)B * stride)[i] = make_uint4(0u, 0u, 0u, 0u);
    griddep_wait();
    griddep_launch_dependents();

    bool staged = false;  // an input of one chunk is staged once for all tiles that share it
    for (; item < items; item += step) {
        Tile next = now;
        if (!ROUTED) next.tile += step;
        else if (item + step < items) {
            if (now.matrix < matrices && now.tile + 1 == tiles) next = tile_at(now.matrix + 1, 0);
            else next.tile++;
        }
        const int tile = now.tile, N = now.N, kb = now.kb, ke = now.ke;
        const bool shared_tile = ROUTED && now.matrix == matrices;
        // what the epilogue's convolution wants, on its way during the product (thread tid: column tid & 15, row tid >> 4)
        float cx[kMaxTaps], cw[kMaxTaps];
        const int er = tile * 16 + (tid & 15), eb = tid >> 4;
        const bool conv = er < a.conv_n && eb < B && eb < NT * 8;
        SeqDesc sd{};
        if (conv && rank == 0) {
            sd = a.seqs[eb];
            const float* hr = a.hist + ((size_t)sd.bank * a.max_slots + sd.slot) * (a.taps - 1) * a.conv_n + er;
#pragma unroll
            for (int j = 0; j < kMaxTaps; ++j) {
                cx[j] = cw[j] = 0.f;
                if (a.taps <= kMaxTaps && j < a.taps) {
                    cw[j] = __ldg(a.conv_w + (size_t)j * a.conv_n + er);
                    if (j + 1 < a.taps && a.taps - 1 - j <= sd.pos0) cx[j] = hr[(size_t)j * a.conv_n];
                }
            }
        }
        float acc[NT][4];
#pragma unroll
        for (int t = 0; t < NT; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
        int k0 = kb;
        do {  // (a CTA without columns makes one empty pass)
            const int kend = min(ke, k0 + chunk);
            const int pieces = (kend - k0 + 31) >> 5;
            if (!staged) {
                if (k0 > kb || item != item0) __syncthreads();  // everyone is done with the previous chunk
                const int n16 = (kend - k0) >> 2;               // 16-byte pieces of a row
                const uint8_t* xin = shared_tile ? a.shared.x : a.x;
                for (int b = 0; b < B; ++b) {
                    const int xr = ROUTED && a.pair_in ? pair_row(b, now) : b;
                    if (xr < 0) continue;  // (whatever the row holds stays in its own column of the product)
                    for (int i = tid; i < n16; i += kThreads)
                        cp_async16(xs + (size_t)b * stride + i * 16, xin + ((size_t)xr * now.K + k0) * 4 + i * 16);
                }
                cp_async_commit();
                cp_async_wait<0>();
                __syncthreads();
                if (ke - kb <= chunk) staged = true;
            }
            // where the pieces behind this chunk's lie
            const bool more = kend < ke;
            const Tile behind = more ? now : next;
            const int kn = more ? kend : next.kb, en = more ? min(ke, kend + chunk) : (item + step < items ? min(next.ke, next.kb + chunk) : next.kb);
            int p0 = warp;
            do {
                const bool last = p0 + kU * kWarps >= pieces;
#pragma unroll
                for (int u = 0; u < kU; ++u) {
                    const int p = p0 + u * kWarps;
                    if (p < pieces) {
                        const int j = p * 4 + c;  // group of eight columns within the chunk
                        const bool in = k0 + j * 8 < kend;
#pragma unroll
                        for (int t = 0; t < NT; ++t) {
                            uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
                            if (in) {
                                const uint4* xp = reinterpret_cast<const uint4*>(xs + (size_t)(t * 8 + g) * stride + j * 32);
                                hi = xp[0];
                                lo = xp[1];
                            }
                            mma_bf16(acc[t], w[u][0].x, w[u][1].x, w[u][0].y, w[u][1].y, hi.x, hi.y);
                            mma_bf16(acc[t], w[u][0].x, w[u][1].x, w[u][0].y, w[u][1].y, lo.x, lo.y);
                            mma_bf16(acc[t], w[u][0].z, w[u][1].z, w[u][0].w, w[u][1].w, hi.z, hi.w);
                            mma_bf16(acc[t], w[u][0].z, w[u][1].z, w[u][0].w, w[u][1].w, lo.z, lo.w);
                        }
                    }
                    if (last) request(w[u], behind, kn, en, warp + u * kWarps);
                    else request(w[u], now, k0, kend, p + kU * kWarps);
                }
                p0 += kU * kWarps;
            } while (p0 < pieces);
            k0 += chunk;
        } while (k0 < ke);
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
            if (tid < NT * 128) {
                float v = 0.f;
#pragma unroll
                for (int q = 0; q < kWarps; ++q) v += red[tid >> 7][q][tid & 15][(tid >> 4) & 7];
                part[tid] = v;
            }
            cluster_sync_all();
        }
        auto total = [&](int row) {  // of the tile, for input row eb
            float v = 0.f;
            if (slices > 1) {
                for (int s = 0; s < slices; ++s) {
                    float p;
                    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(p) : "r"(map_to_cta(smem_u32(part + (tid & ~15) + row), s)) : "memory");
                    v += p;
                }
            } else {
#pragma unroll
                for (int q = 0; q < kWarps; ++q) v += red[eb >> 3][q][row][eb & 7];
            }
            return v;
        };
        const int out_row = (eb < B && eb < NT * 8) ? pair_row(eb, now) : -1;
        if (rank == 0 && out_row >= 0 && gated) {
            if ((tid & 15) < 8) {
                const float gv = total(tid & 7), uv = total((tid & 7) + 8);
                const float v = a.gate == GATE_CLAMP ? clamped_gate(gv, uv, shared_tile ? a.shared.limit : a.limit) : gelu_tanh(gv) * uv;
                store_split((shared_tile ? a.shared.split_out : a.split_out) + (size_t)out_row * (N >> 1) * 4, (tile >> 2) * 32 + (tile & 3) * 8 + (tid & 7), v);
            }
        } else if (rank == 0 && out_row >= 0 && er < N) {
            float v = total(tid & 15);
            if (a.bias) v += __ldg(a.bias + er);
            if (conv) {
                const int hrows = a.taps - 1;
                float* hw = a.hist + ((size_t)(sd.bank ^ 1) * a.max_slots + sd.slot) * hrows * a.conv_n + er;
                float s = a.conv_b ? __ldg(a.conv_b + er) : 0.f;
                if (a.taps <= kMaxTaps) {
#pragma unroll
                    for (int j = 0; j < kMaxTaps; ++j) {
                        if (j + 1 == a.taps) cx[j] = v;
                        s = fmaf(cx[j], cw[j], s);
                        if (j > 0 && j < a.taps) hw[(size_t)(j - 1) * a.conv_n] = cx[j];
                    }
                } else {
                    const float* hr = a.hist + ((size_t)sd.bank * a.max_slots + sd.slot) * hrows * a.conv_n + er;
                    for (int j = 0; j < a.taps; ++j) {
                        const float x = j == hrows ? v : (hrows - j <= sd.pos0 ? hr[(size_t)j * a.conv_n] : 0.f);
                        s = fmaf(x, __ldg(a.conv_w + (size_t)j * a.conv_n + er), s);
                        if (j > 0) hw[(size_t)(j - 1) * a.conv_n] = x;
                    }
                }
                v = silu(s);
            } else if (a.act == ACT_GELU_ERF) v = gelu_erf(v);
            else if (a.act == ACT_GELU_TANH) v = gelu_tanh(v);
            if (conv && a.conv_out) store_split(a.conv_out + (size_t)eb * a.conv_n * 4, er, v);
            else if (a.split_out) store_split(a.split_out + (size_t)out_row * N * 4, er, v);
            else if (shared_tile) a.shared.out[(size_t)out_row * a.shared.ldo + er] = v;
            else a.out[(size_t)out_row * a.ldo + er] = v;
        }
        if (slices > 1) cluster_sync_all();  // the partial sums have been read (and nobody leaves before that)
        else __syncthreads();
        if (ROUTED && (a.pair_in || a.shared.x != a.x) && next.matrix != now.matrix) staged = false;
        now = next;
    }
}

template <int NT, bool ROUTED>
int launch_one(b200_ctx* ctx, const DecodeGemmArgs& a) {
    static bool attr_set[64] = {};
    if (!attr_set[ctx->device & 63]) {
        B200_CUDA(ctx, cudaFuncSetAttribute(decode_gemm_kernel<NT, ROUTED>, cudaFuncAttributeMaxDynamicSharedMemorySize, kOneCtaSmem));
        attr_set[ctx->device & 63] = true;
    }
    // (routed: at most as many matrices as pairs or experts; they are not known here)
    const int max_k = ROUTED && a.shared.W && a.shared.K > a.K ? a.shared.K : a.K;
    int tiles = (a.N + 15) / 16;
    if (ROUTED) tiles = tiles * (a.B * a.top < a.experts ? a.B * a.top : a.experts) + (a.shared.W ? (a.shared.N + 15) / 16 : 0);
    // K slices while the CTAs of one wave (two per SM) are not used up and a warp keeps at least a piece
    int slices = 1;
    while (slices < 8 && tiles * slices * 2 <= 2 * ctx->num_sms && max_k / (slices * 2) >= 256) slices *= 2;
    // (routed: and as many as it takes for a slice to be staged once for all of its tiles)
    const int two_ctas = (kTwoCtaSmem / (NT * 8) - 16) / 4 / 32 * 32;
    while (ROUTED && slices < 8 && (max_k + slices - 1) / slices > two_ctas) slices *= 2;
    const int kslice = ((max_k + slices - 1) / slices + 31) / 32 * 32;
    // the columns staged at a time: all of the slice, so that they are staged once for all tiles; else as many as
    // two CTAs per SM can hold
    auto columns = [](int smem) { return (smem / (NT * 8) - 16) / 4 / 32 * 32; };
    const int chunk = kslice <= columns(kOneCtaSmem) ? kslice : columns(kTwoCtaSmem);
    const int per_sm = chunk <= columns(kTwoCtaSmem) ? 2 : 1;
    int grid = tiles * slices;
    if (grid > per_sm * ctx->num_sms) grid = per_sm * ctx->num_sms / slices * slices;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(grid);
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = (size_t)NT * 8 * (chunk * 4 + 16);
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
    const cudaError_t le = cudaLaunchKernelEx(&cfg, decode_gemm_kernel<NT, ROUTED>, a, slices, kslice, chunk);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace

int launch_decode_gemm(b200_ctx* ctx, const DecodeGemmArgs& a) {
    if (a.B < 1 || a.B > 16 || a.K % 8 || a.N < 1) return B200_ERR_SHAPE;
    if (a.top < 0 || a.B * a.top > kMaxPairs || (a.top > 0 && a.conv_n > 0) || (a.gate != GATE_NONE && (a.N % 64 || !a.split_out))) return B200_ERR_SHAPE;
    if (a.shared.W && (a.top < 1 || a.shared.K % 8 || (a.gate != GATE_NONE && (a.shared.N % 64 || !a.shared.split_out)))) return B200_ERR_SHAPE;
    if (a.top > 0) return a.B <= 8 ? launch_one<1, true>(ctx, a) : launch_one<2, true>(ctx, a);
    return a.B <= 8 ? launch_one<1, false>(ctx, a) : launch_one<2, false>(ctx, a);
}

}  // namespace b200
