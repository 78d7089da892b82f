// Feed-forward layers whose experts a table picks by token id, and gated activations.
//
// General path: the (token, expert) pairs of a step are put into runs, one per expert, each padded to a multiple of the
// product's row tile (moe_route), the norm writes its rows straight into those places, and the two products
// are grouped (GemmGroups): a tile of rows has one weight matrix.  The places are handed to the next residual
// kernel, which adds the experts' outputs up.
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int kRouteThreads = 1024;

// One CTA per feed-forward layer.  place[p] = row of pair p = (token, choice); blocks: see GemmGroups.  Pairs of
// an expert are placed in the order of arrival, which no result depends on: rows do not meet.
__global__ void __launch_bounds__(kRouteThreads)
moe_route_kernel(const MoeRoute* __restrict__ routes, const int* __restrict__ tok, int M, bool f32) {
    extern __shared__ int cursor[];  // [experts]: counts, then the next free row
    __shared__ int warp_sum_s[32];
    __shared__ int base_s;
    griddep_wait();
    griddep_launch_dependents();
    const MoeRoute r = routes[blockIdx.x];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, P = M * r.top, align = moe_run_rows(P, r.experts, f32);
    for (int e = tid; e < r.experts; e += kRouteThreads) cursor[e] = 0;
    if (tid == 0) base_s = 0;
    __syncthreads();
    for (int p = tid; p < P; p += kRouteThreads) atomicAdd(cursor + __ldg(r.table + (size_t)tok[p / r.top] * r.top + p % r.top), 1);
    __syncthreads();
    // runs of the experts, 1024 of them at a time
    for (int e0 = 0; e0 < r.experts; e0 += kRouteThreads) {
        const int e = e0 + tid;
        const int runs = e < r.experts ? (cursor[e] + align - 1) / align : 0;
        int incl = runs;
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const int o = __shfl_up_sync(0xffffffffu, incl, d);
            if (lane >= d) incl += o;
        }
        if (lane == 31) warp_sum_s[warp] = incl;
        __syncthreads();
        int before = base_s, all = 0;
        for (int w = 0; w < 32; ++w) {
            if (w < warp) before += warp_sum_s[w];
            all += warp_sum_s[w];
        }
        const int first = before + incl - runs;
        if (e < r.experts) cursor[e] = first * align;
        for (int i = 0; i < runs; ++i) r.blocks[1 + first + i] = e;
        __syncthreads();
        if (tid == 0) base_s += all;
        __syncthreads();
    }
    if (tid == 0) r.blocks[0] = base_s;
    for (int p = tid; p < P; p += kRouteThreads) r.place[p] = atomicAdd(cursor + __ldg(r.table + (size_t)tok[p / r.top] * r.top + p % r.top), 1);
}

// One CTA per feed-forward layer: the experts of B <= 16 tokens and, each once, the ones that occur (in the order of the pairs)
__global__ void __launch_bounds__(kMaxPairs)
decode_routes_kernel(const MoeRoute* __restrict__ routes, const int* __restrict__ tok, int B) {
    __shared__ int expert[kMaxPairs];
    __shared__ int first[kMaxPairs];
    griddep_wait();
    griddep_launch_dependents();
    const MoeRoute r = routes[blockIdx.x];
    const int tid = threadIdx.x, pairs = B * r.top;
    if (tid < pairs) expert[tid] = __ldg(r.table + (size_t)tok[tid / r.top] * r.top + tid % r.top);
    __syncthreads();
    bool seen = false;
    if (tid < pairs) {
        for (int p = 0; p < tid; ++p) seen = seen || expert[p] == expert[tid];
        first[tid] = !seen;
    }
    const int n = __syncthreads_count(tid < pairs && !seen);
    if (tid < pairs) {
        r.decode->expert[tid] = (uint16_t)expert[tid];
        if (!seen) {
            int at = 0;
            for (int p = 0; p < tid; ++p) at += first[p];
            r.decode->listed[at] = (uint16_t)expert[tid];
        }
    }
    if (tid == 0) r.decode->matrices = n;
}

// fp32 rows of n pairs of 32 gates and 32 linear values -> n * 32 columns
__global__ void __launch_bounds__(256)
gated_act_kernel(float* __restrict__ out, const float* __restrict__ in, int F, size_t total4, int gate, float limit) {
    griddep_wait();
    griddep_launch_dependents();
    const int F4 = F >> 2;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total4; i += (size_t)gridDim.x * blockDim.x) {
        const size_t row = i / F4;
        const int c4 = (int)(i % F4);
        const float4* src = reinterpret_cast<const float4*>(in + row * 2 * F) + (c4 >> 3) * 16 + (c4 & 7);
        const float4 g = src[0], u = src[8];
        float4 v;
        if (gate == GATE_CLAMP)
            v = make_float4(clamped_gate(g.x, u.x, limit), clamped_gate(g.y, u.y, limit), clamped_gate(g.z, u.z, limit), clamped_gate(g.w, u.w, limit));
        else
            v = make_float4(gelu_tanh(g.x) * u.x, gelu_tanh(g.y) * u.y, gelu_tanh(g.z) * u.z, gelu_tanh(g.w) * u.w);
        reinterpret_cast<float4*>(out)[i] = v;
    }
}

}  // namespace

int launch_moe_route(b200_ctx* ctx, const MoeRoute* routes, int n, const int* tok, int M, bool f32, int max_experts) {
    if ((size_t)max_experts * 4 > 40 * 1024) return B200_ERR_LIMIT;
    cudaError_t le = launch_pdl(ctx, moe_route_kernel, dim3(n), dim3(kRouteThreads), (size_t)max_experts * 4, routes, tok, M, f32);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_decode_routes(b200_ctx* ctx, const MoeRoute* routes, int n, const int* tok, int B) {
    cudaError_t le = launch_pdl(ctx, decode_routes_kernel, dim3(n), dim3(kMaxPairs), 0, routes, tok, B);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_gated_act(b200_ctx* ctx, float* out, const float* in, int M, int F, int gate, float limit) {
    if (F % 32) return B200_ERR_SHAPE;
    const size_t total = (size_t)M * (F >> 2), blocks = (total + 255) / 256;
    const unsigned grid = (unsigned)(blocks < (size_t)16 * ctx->num_sms ? blocks : (size_t)16 * ctx->num_sms);
    cudaError_t le = launch_pdl(ctx, gated_act_kernel, dim3(grid), dim3(256), 0, out, in, F, total, gate, limit);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace b200
