// Row-wise kernels of the layered decoders: the residual stream with an RMS norm in front of (and, if a design
// has it, behind) every sublayer, the per-head output norm of the delta rule, and a column slice.  One CTA per
// row with the row in registers; sums in fp32, eps inside the root.
#include <cuda_bf16.h>
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

constexpr int kNormThreads = 256;
constexpr int kVpt = 4;  // float4 of a row a thread keeps in registers: rows up to 4 * 4 * 256 columns

// Pass 1: r (see launch_residual_rms) into registers and x_out, sum of r^2.  Rows longer than the registers
// hold are read again from x_out.
template <int OUT>  // H_BF16, H_F32 (with an fp32 embedding table), H_SPLIT
__global__ void __launch_bounds__(kNormThreads)
residual_rms_kernel(const ResidualNormArgs a, int* status) {
    __shared__ float red[8];
    griddep_wait();
    griddep_launch_dependents();
    const int row_out = blockIdx.x;
    const int row = a.rows ? a.rows[row_out] : row_out;
    const int C4 = a.Cp >> 2;
    const float inv_c = 1.0f / (float)a.C;
    const float4* x = a.x ? reinterpret_cast<const float4*>(a.x + (size_t)row * a.Cp) : nullptr;
    const float4* y = a.y ? reinterpret_cast<const float4*>(a.y + (size_t)row * a.Cp) : nullptr;
    float4* xo = a.x_out ? reinterpret_cast<float4*>(a.x_out + (size_t)row_out * a.Cp) : nullptr;
    float4 v[kVpt];
    int tok = 0;
    if (a.tok) {
        tok = a.tok[row];
        if (tok < 0 || tok >= a.vocab) { if (threadIdx.x == 0) atomicCAS(status, 0, 201); tok = 0; }
    }
    float rstd_y = 0.f;
#pragma unroll
    for (int i = 0; i < kVpt; ++i) v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (y) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < kVpt; ++i) {
            const int c = threadIdx.x + i * blockDim.x;
            if (c < C4) { v[i] = y[c]; s += sq4(v[i]); }
        }
        if (a.wb) {
            for (int c = threadIdx.x + kVpt * blockDim.x; c < C4; c += blockDim.x) s += sq4(y[c]);
            rstd_y = 1.0f / sqrtf(block_sum(s, red) * inv_c + a.eps);
        }
    }
    const float y_scale = a.y_scale ? a.y_scale[row] : 1.f;
    auto value = [&](int c, float4 yv) {
        float4 r;
        if (a.tok) {
            r = OUT == H_F32 ? load4(static_cast<const float*>(a.embed) + (size_t)tok * a.Cp, c)
                    : load4(static_cast<const uint16_t*>(a.embed) + (size_t)tok * a.Cp, c);
            r.x *= a.embed_scale; r.y *= a.embed_scale; r.z *= a.embed_scale; r.w *= a.embed_scale;
        } else r = x[c];
        if (a.wb && y) {
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.wb) + c);
            r.x += yv.x * rstd_y * w.x; r.y += yv.y * rstd_y * w.y; r.z += yv.z * rstd_y * w.z; r.w += yv.w * rstd_y * w.w;
        } else {
            float4 b = make_float4(yv.x * y_scale, yv.y * y_scale, yv.z * y_scale, yv.w * y_scale);
            for (int j = 0; j < a.top; ++j) {  // (0: no parts)
                const int k = row * a.top + j;
                const float4 e = reinterpret_cast<const float4*>(a.parts + (size_t)(a.part_of ? a.part_of[k] : k) * a.Cp)[c];
                b.x = fmaf(e.x, a.part_scale, b.x); b.y = fmaf(e.y, a.part_scale, b.y);
                b.z = fmaf(e.z, a.part_scale, b.z); b.w = fmaf(e.w, a.part_scale, b.w);
            }
            r.x += b.x; r.y += b.y; r.z += b.z; r.w += b.w;
        }
        return r;
    };
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kVpt; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < C4) {
            v[i] = value(c, v[i]);
            s += sq4(v[i]);
            if (xo) xo[c] = v[i];
        }
    }
    for (int c = threadIdx.x + kVpt * blockDim.x; c < C4; c += blockDim.x) {
        const float4 r = value(c, y ? y[c] : make_float4(0.f, 0.f, 0.f, 0.f));
        s += sq4(r);
        if (xo) xo[c] = r;
    }
    if (!a.w) return;
    const float rstd = 1.0f / sqrtf(block_sum(s, red) * inv_c + a.eps);
    float gate = 0.f;
    auto emit = [&](int c, float4 r) {
        const float4 w = __ldg(reinterpret_cast<const float4*>(a.w) + c);
        const float4 h = make_float4(r.x * rstd * w.x, r.y * rstd * w.y, r.z * rstd * w.z, r.w * rstd * w.w);
        if (OUT == H_SPLIT) store_split4(static_cast<uint8_t*>(a.h) + (size_t)row_out * a.Cp * 4, c, h);
        else {
            store4<OUT == H_F32>(a.h, (size_t)row_out * C4 + c, h);
            for (int j = 0; j < a.copies; ++j) store4<OUT == H_F32>(a.copy, (size_t)a.copy_of[row_out * a.copies + j] * C4 + c, h);
        }
        if (a.gate_w) {
            const float4 g = __ldg(reinterpret_cast<const float4*>(a.gate_w) + c);
            gate += (h.x * g.x + h.y * g.y) + (h.z * g.z + h.w * g.w);
        }
    };
#pragma unroll
    for (int i = 0; i < kVpt; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < C4) emit(c, v[i]);
    }
    // (columns beyond the registers are formed again: x_out may alias x, whose row this thread has already replaced)
    for (int c = threadIdx.x + kVpt * blockDim.x; c < C4; c += blockDim.x)
        emit(c, xo ? xo[c] : value(c, y ? y[c] : make_float4(0.f, 0.f, 0.f, 0.f)));
    if (a.gate_w) {
        gate = block_sum(gate, red);
        if (threadIdx.x == 0) a.gate_out[row_out] = sigmoidf_(gate);
    }
}

// one warp per (row, head)
template <bool F32>
__global__ void __launch_bounds__(256)
gated_head_norm_kernel(void* out, int ld_out, const float* __restrict__ o, int ld_o, const float* __restrict__ gate, int ld_gate,
                       const float* __restrict__ w, int M, int H, int Dv, int Dvl, float eps, bool plain_sigmoid) {
    griddep_wait();
    griddep_launch_dependents();
    const int lane = threadIdx.x & 31;
    const size_t u = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (u >= (size_t)M * H) return;
    const int row = (int)(u / H), h = (int)(u % H);
    const float* oh = o + (size_t)row * ld_o + h * Dvl;
    const float* gh = gate + (size_t)row * ld_gate + h * Dvl;
    const size_t ob = (size_t)row * ld_out + (size_t)h * Dv;
    float s = 0.f;
    if (Dv <= 256) {
        float v[8], g[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int d = lane + i * 32;
            v[i] = g[i] = 0.f;
            if (d < Dv) { v[i] = oh[d]; g[i] = gh[d]; s += v[i] * v[i]; }
        }
        const float r = 1.0f / sqrtf(warp_sum(s) / (float)Dv + eps);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int d = lane + i * 32;
            if (d < Dv) store1<F32>(out, ob + d, v[i] * r * __ldg(w + d) * (plain_sigmoid ? sigmoidf_(g[i]) : silu(g[i])));
        }
        return;
    }
    for (int d = lane; d < Dv; d += 32) s += oh[d] * oh[d];
    const float r = 1.0f / sqrtf(warp_sum(s) / (float)Dv + eps);
    for (int d = lane; d < Dv; d += 32) store1<F32>(out, ob + d, oh[d] * r * __ldg(w + d) * (plain_sigmoid ? sigmoidf_(gh[d]) : silu(gh[d])));
}

template <bool F32>
__global__ void slice_kernel(void* dst, int ld_dst, const float* __restrict__ src, int ld_src, int n, int M) {
    griddep_wait();
    griddep_launch_dependents();
    const size_t total = (size_t)M * ld_dst;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int c = (int)(i % ld_dst);
        const size_t r = i / ld_dst;
        store1<F32>(dst, i, c < n ? src[r * ld_src + c] : 0.f);
    }
}

}  // namespace

int launch_residual_rms(b200_ctx* ctx, const ResidualNormArgs& a, int format) {
    if (a.M <= 0) return B200_OK;
    int threads = ((a.Cp / 4 + 31) / 32) * 32;
    if (threads > kNormThreads) threads = kNormThreads;
    cudaError_t le;
    if (format == H_F32) le = launch_pdl(ctx, residual_rms_kernel<H_F32>, dim3(a.M), dim3(threads), 0, a, ctx->d_status);
    else if (format == H_SPLIT) le = launch_pdl(ctx, residual_rms_kernel<H_SPLIT>, dim3(a.M), dim3(threads), 0, a, ctx->d_status);
    else le = launch_pdl(ctx, residual_rms_kernel<H_BF16>, dim3(a.M), dim3(threads), 0, a, ctx->d_status);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_gated_head_norm(b200_ctx* ctx, void* out, int ld_out, const float* o, int ld_o, const float* gate, int ld_gate,
                           const float* w, int M, int H, int Dv, int Dvl, float eps, bool f32, bool plain_sigmoid) {
    const unsigned grid = (unsigned)(((size_t)M * H + 7) / 8);
    cudaError_t le = f32 ? launch_pdl(ctx, gated_head_norm_kernel<true>, dim3(grid), dim3(256), 0, out, ld_out, o, ld_o, gate, ld_gate, w, M, H, Dv, Dvl, eps, plain_sigmoid)
                         : launch_pdl(ctx, gated_head_norm_kernel<false>, dim3(grid), dim3(256), 0, out, ld_out, o, ld_o, gate, ld_gate, w, M, H, Dv, Dvl, eps, plain_sigmoid);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_slice(b200_ctx* ctx, void* dst, int ld_dst, const float* src, int ld_src, int n, int M, bool f32) {
    const size_t total = (size_t)M * ld_dst, blocks = (total + 255) / 256;
    const unsigned grid = (unsigned)(blocks < (size_t)8 * ctx->num_sms ? blocks : (size_t)8 * ctx->num_sms);
    cudaError_t le = f32 ? launch_pdl(ctx, slice_kernel<true>, dim3(grid), dim3(256), 0, dst, ld_dst, src, ld_src, n, M)
                         : launch_pdl(ctx, slice_kernel<false>, dim3(grid), dim3(256), 0, dst, ld_dst, src, ld_src, n, M);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace b200
