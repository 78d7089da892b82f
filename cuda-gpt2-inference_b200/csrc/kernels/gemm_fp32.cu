// out[M,N] = act(inp[M,K] W[N,K]^T + bias[N]) with every product and sum in fp32 (FMA pipe): the matrix
// product of the 32-bit arithmetic, where the tensor-core formats (TF32 and below) would round the operands.
// 64 x 64 tiles, 16-deep K slices double-buffered in shared memory, 4 x 4 results per thread held as
// pairs so that one instruction does two multiply-adds.
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int TM = 64, TN = 64, TK = 16, kThreads = 256;
constexpr int LDT = TM + 4;  // transposed tiles [TK][LDT]

__global__ void __launch_bounds__(kThreads)
gemm_fp32_kernel(float* __restrict__ out, const float* __restrict__ inp, const float* __restrict__ W,
                 const float* __restrict__ bias, int M, int K, int N, int act, const int* __restrict__ group_blocks, int group_align) {
    __shared__ __align__(16) float as[2][TK][LDT];
    __shared__ __align__(16) float bs[2][TK][LDT];
    griddep_wait();
    griddep_launch_dependents();
    const int tid = threadIdx.x;
    const int m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
    if (group_blocks) {  // grouped: runs of group_align rows with a matrix each (GemmGroups)
        const int run = m0 / group_align;
        if (run >= group_blocks[0]) return;
        W += (size_t)group_blocks[1 + run] * N * K;
    }
    const int lr = tid >> 2, lk = (tid & 3) * 4;  // each thread stages 4 consecutive k of one row of either operand
    const int tx = tid & 15, ty = tid >> 4;
    const bool a_ok = m0 + lr < M, b_ok = n0 + lr < N;
    const float* ap = inp + (size_t)(a_ok ? m0 + lr : 0) * K;
    const float* bp = W + (size_t)(b_ok ? n0 + lr : 0) * K;
    float4 ra, rb;
    auto fetch = [&](int k0) {
        ra = rb = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k0 + lk < K) {  // K is a multiple of 4
            if (a_ok) ra = *reinterpret_cast<const float4*>(ap + k0 + lk);
            if (b_ok) rb = __ldg(reinterpret_cast<const float4*>(bp + k0 + lk));
        }
    };
    auto put = [&](int b) {
        as[b][lk][lr] = ra.x; as[b][lk + 1][lr] = ra.y; as[b][lk + 2][lr] = ra.z; as[b][lk + 3][lr] = ra.w;
        bs[b][lk][lr] = rb.x; bs[b][lk + 1][lr] = rb.y; bs[b][lk + 2][lr] = rb.z; bs[b][lk + 3][lr] = rb.w;
    };
    uint64_t acc[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = pack2(0.f, 0.f);
    fetch(0);
    put(0);
    __syncthreads();
    int buf = 0;
    for (int k0 = 0; k0 < K; k0 += TK) {
        const bool more = k0 + TK < K;
        if (more) fetch(k0 + TK);
#pragma unroll
        for (int k = 0; k < TK; ++k) {
            const float4 av = *reinterpret_cast<const float4*>(&as[buf][k][ty * 4]);
            const ulonglong2 bv = *reinterpret_cast<const ulonglong2*>(&bs[buf][k][tx * 4]);
            const float a[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint64_t aa = pack2(a[i], a[i]);
                acc[i][0] = fma2(aa, bv.x, acc[i][0]);
                acc[i][1] = fma2(aa, bv.y, acc[i][1]);
            }
        }
        if (more) put(buf ^ 1);
        __syncthreads();
        buf ^= 1;
    }
    const int n = n0 + tx * 4;
    if (n >= N) return;  // N is a multiple of 4
    float4 b4 = make_float4(0.f, 0.f, 0.f, 0.f);
    if (bias) b4 = __ldg(reinterpret_cast<const float4*>(bias + n));
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) break;
        float4 v;
        unpack2(acc[i][0], v.x, v.y);
        unpack2(acc[i][1], v.z, v.w);
        v.x += b4.x; v.y += b4.y; v.z += b4.z; v.w += b4.w;
        if (act == ACT_GELU_ERF) { v.x = gelu_erf(v.x); v.y = gelu_erf(v.y); v.z = gelu_erf(v.z); v.w = gelu_erf(v.w); }
        else if (act == ACT_GELU_TANH) { v.x = gelu_tanh(v.x); v.y = gelu_tanh(v.y); v.z = gelu_tanh(v.z); v.w = gelu_tanh(v.w); }
        *reinterpret_cast<float4*>(out + (size_t)m * N + n) = v;
    }
}

}  // namespace

int launch_gemm_fp32(b200_ctx* ctx, float* out, const float* inp, const float* W, const float* bias, int M, int K, int N, int act, const GemmGroups* groups) {
    if (K % 4 || N % 4 || (groups && groups->align % TM)) return B200_ERR_SHAPE;
    if (M <= 0) return B200_OK;
    cudaError_t le = launch_pdl(ctx, gemm_fp32_kernel, dim3((N + TN - 1) / TN, (M + TM - 1) / TM), dim3(kThreads), 0, out, inp, W, bias, M, K, N, act,
                                groups ? groups->blocks : nullptr, groups ? groups->align : 0);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace b200
