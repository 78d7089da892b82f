// Device helpers shared by the kernels of the layered decoders.
#pragma once
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_fp16.h>

namespace b200 {

// 1 / (1 + e^-z): one exponential and one reciprocal on the special-function unit, relative error of a few 2^-22
// (an overflowing exponential gives 0)
__device__ __forceinline__ float sigmoidf_(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float silu(float z) { return z * sigmoidf_(z); }
// log(1 + e^z) = max(z, 0) + log(1 + e), e = e^-|z|; where 1 + e would drop e's digits, from the series of log
__device__ __forceinline__ float softplusf_(float z) {
    const float e = __expf(-fabsf(z));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 1.0f / 3.0f), -0.5f), 1.0f);
    return fmaxf(z, 0.f) + (e < 0.03f ? series : __logf(1.0f + e));
}
__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }
// The same for a 16-bit result: erf by the rational approximation 7.1.26 of Abramowitz and Stegun, Handbook of
// Mathematical Functions (absolute error below 1.5e-7, here and there a few rounding errors more)
__device__ __forceinline__ float gelu_erf_h(float z) {
    const float x = fabsf(z) * 0.70710678118654752f;
    const float t = __fdividef(1.0f, fmaf(0.3275911f, x, 1.0f));
    const float p = t * fmaf(t, fmaf(t, fmaf(t, fmaf(t, 1.061405429f, -1.453152027f), 1.421413741f), -0.284496736f), 0.254829592f);
    const float erfc = p * __expf(-x * x);  // of |z| / sqrt(2)
    return z >= 0.f ? z - 0.5f * z * erfc : 0.5f * z * erfc;
}
// a gate bounded above and its linear part, bounded on both sides, that counts from one: g sigmoid(1.702 g) (u + 1)
__device__ __forceinline__ float clamped_gate(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoidf_(1.702f * g) * (u + 1.0f);
}
// 2^x on the special-function unit
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int s = 16; s >= 1; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
    return v;
}
// sum over the CTA (up to 8 warps; every thread gets it); red: 8 floats of shared memory
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    const int nw = (blockDim.x + 31) >> 5;
    if (nw == 1) return v;
    __syncthreads();  // the previous sum has been read
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += red[i];
    return t;
}
__device__ __forceinline__ float sq4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

__device__ __forceinline__ float bf16_to_f(uint16_t h) { return __uint_as_float((uint32_t)h << 16); }
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&p);
}
__device__ __forceinline__ float4 load4(const float* p, int c4) { return *(reinterpret_cast<const float4*>(p) + c4); }
__device__ __forceinline__ float4 load4(const uint16_t* p, int c4) {
    const uint2 u = *(reinterpret_cast<const uint2*>(p) + c4);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
// element i4 (in units of four) / i of a buffer of fp32 or bf16
template <bool F32>
__device__ __forceinline__ void store4(void* base, size_t i4, float4 v) {
    if (F32) reinterpret_cast<float4*>(base)[i4] = v;
    else reinterpret_cast<uint2*>(base)[i4] = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
template <bool F32>
__device__ __forceinline__ void store1(void* base, size_t i, float v) {
    if (F32) reinterpret_cast<float*>(base)[i] = v;
    else reinterpret_cast<__nv_bfloat16*>(base)[i] = __float2bfloat16_rn(v);
}

// Split rows, the operand format of the decode products: eight values as 16 bytes of bf16 and 16 bytes of the
// bf16 of what that rounding dropped (four bytes per value in all).
__device__ __forceinline__ void store_split(uint8_t* row, int k, float v) {
    const __nv_bfloat16 hi = __float2bfloat16_rn(v);
    __nv_bfloat16* p = reinterpret_cast<__nv_bfloat16*>(row + (k >> 3) * 32 + (k & 7) * 2);
    p[0] = hi;
    p[8] = __float2bfloat16_rn(v - __bfloat162float(hi));
}
__device__ __forceinline__ void store_split4(uint8_t* row, int k4, float4 v) {  // values 4 k4 .. 4 k4 + 3
    const uint32_t h0 = pack_bf16(v.x, v.y), h1 = pack_bf16(v.z, v.w);
    uint2* p = reinterpret_cast<uint2*>(row + (k4 >> 1) * 32 + (k4 & 1) * 8);
    p[0] = make_uint2(h0, h1);
    p[2] = make_uint2(pack_bf16(v.x - __uint_as_float(h0 << 16), v.y - __uint_as_float(h0 & 0xffff0000u)),
                      pack_bf16(v.z - __uint_as_float(h1 << 16), v.w - __uint_as_float(h1 & 0xffff0000u)));
}
__device__ __forceinline__ float load_split(const uint8_t* row, int k) {
    const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(row + (k >> 3) * 32 + (k & 7) * 2);
    return __bfloat162float(p[0]) + __bfloat162float(p[8]);
}

__device__ __forceinline__ void cp_async16(void* smem_dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async8(void* smem_dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// which lane of a group holds total number `idx` after reduce_scatter<CNT, L>, and where in its v
template <int CNT, int L>
__device__ constexpr int scatter_lane(int idx) {
    int lane = 0, cnt = CNT;
    for (int m = 1; m < L && cnt > 1; m <<= 1) {
        cnt >>= 1;
        if (idx >= cnt) { lane |= m; idx -= cnt; }
    }
    return lane;
}
template <int CNT, int L>
__device__ constexpr int scatter_slot(int idx) {
    int cnt = CNT;
    for (int m = 1; m < L && cnt > 1; m <<= 1) {
        cnt >>= 1;
        if (idx >= cnt) idx -= cnt;
    }
    return idx;
}

// CNT values per lane, summed over the L lanes of an aligned group and spread over them: on return the
// lane holds max(1, CNT / L) of the totals in v[0 ..).  Lane bit b (mask 2^b < L) decides between the
// lower and the upper half of what is left, so the first total a lane holds is number
//   sum over the halving steps of  bit_b * (CNT >> (b + 1))
template <int CNT, int L>
__device__ __forceinline__ void reduce_scatter(float (&v)[CNT], int lane) {
    int cnt = CNT;
#pragma unroll
    for (int m = 1; m < L; m <<= 1) {
        if (cnt > 1) {
            const int half = cnt >> 1;
            const bool up = (lane & m) != 0;
#pragma unroll
            for (int i = 0; i < CNT / 2; ++i) {
                if (i < half) {
                    const float send = up ? v[i] : v[i + half], keep = up ? v[i + half] : v[i];
                    v[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
                }
            }
            cnt = half;
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], m);
        }
    }
}
template <int CNT, int L>
__device__ __forceinline__ int scatter_first(int lane) {
    int idx = 0, cnt = CNT;
#pragma unroll
    for (int m = 1; m < L; m <<= 1) {
        if (cnt > 1) { cnt >>= 1; if (lane & m) idx += cnt; }
    }
    return idx;
}
// whether this lane is the one of its group that reports the totals it holds (with more lanes than values several hold the same)
template <int CNT, int L>
__device__ __forceinline__ bool scatter_owner(int lane) {
    return L <= CNT || (lane & (L - 1) & ~(CNT - 1)) == 0;
}

// ---- pairs of fp32 (one instruction for two multiply-adds)
__device__ __forceinline__ uint64_t pack2(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

}  // namespace b200
