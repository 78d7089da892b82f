// Layers that carry a state from token to token: the short causal convolution in front of them, the
// selective scan (diagonal state per channel), the gated delta rule (matrix state per head) and the minGRU.
//
// All of them treat a step's rows as sequences (SeqDesc): a sequence that starts (pos0 = 0) begins with
// a zero state whatever its slot holds, any other continues from the slot, so a prompt may be cut anywhere
// and a slot needs no clearing.  State and everything that enters a recurrence is fp32.
#include <cstdlib>
#include <cuda_bf16.h>
#include "decoder_kernels.h"
#include "decoder_math.cuh"
#include "../prim/sm100.cuh"

namespace b200 {
namespace {

// ------------------------------------------------------------------ short convolution
// A thread computes 4 neighbouring channels of kConvTok consecutive tokens; TAPS > 0 keeps the window in registers.
constexpr int kConvTok = 16;

template <int TAPS, bool F32>
__global__ void __launch_bounds__(128)
short_conv_kernel(const ShortConvArgs a) {
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = a.seqs[blockIdx.z];
    const int t0 = blockIdx.y * kConvTok;
    const int c4 = (a.ch0 >> 2) + blockIdx.x * blockDim.x + threadIdx.x;
    if (t0 >= sd.n || c4 * 4 >= a.np) return;
    const int taps = TAPS > 0 ? TAPS : a.taps, hrows = taps - 1;
    const float* hr = a.hist + ((size_t)sd.bank * a.max_slots + sd.slot) * hrows * a.np;
    float* hw = a.hist + ((size_t)(sd.bank ^ 1) * a.max_slots + sd.slot) * hrows * a.np;
    const float* xin = a.x + (size_t)sd.row0 * a.ldx;
    auto input = [&](int i) {  // the input of token i of this step (negative: from the history)
        if (i >= 0) return load4(xin + (size_t)i * a.ldx, c4);
        if (sd.pos0 + i < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
        return load4(hr + (size_t)(hrows + i) * a.np, c4);
    };
    const float4 bias = a.bias ? __ldg(reinterpret_cast<const float4*>(a.bias) + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
    const int t1 = min(sd.n, t0 + kConvTok);
    auto emit = [&](int t, float4 s) {
        store4<F32>(a.out, (size_t)(sd.row0 + t) * (a.ld_out >> 2) + c4, make_float4(silu(s.x), silu(s.y), silu(s.z), silu(s.w)));
    };
    if (TAPS > 0) {
        constexpr int W = TAPS > 0 ? TAPS : 1;
        float4 w[W], win[W];
#pragma unroll
        for (int j = 0; j < W; ++j) w[j] = __ldg(reinterpret_cast<const float4*>(a.w + (size_t)j * a.np) + c4);
#pragma unroll
        for (int j = 0; j + 1 < W; ++j) win[j] = input(t0 - (W - 1) + j);
        for (int tb = t0; tb < t1; tb += 4) {
            float4 nx[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) nx[u] = tb + u < t1 ? input(tb + u) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                win[W - 1] = nx[u];
                float4 s = bias;
#pragma unroll
                for (int j = 0; j < W; ++j) {
                    s.x = fmaf(win[j].x, w[j].x, s.x); s.y = fmaf(win[j].y, w[j].y, s.y);
                    s.z = fmaf(win[j].z, w[j].z, s.z); s.w = fmaf(win[j].w, w[j].w, s.w);
                }
                if (tb + u < t1) emit(tb + u, s);
#pragma unroll
                for (int j = 0; j + 1 < W; ++j) win[j] = win[j + 1];
            }
        }
    } else {
        for (int t = t0; t < t1; ++t) {
            float4 s = bias;
            for (int j = 0; j < taps; ++j) {
                const float4 x = input(t - hrows + j), w = __ldg(reinterpret_cast<const float4*>(a.w + (size_t)j * a.np) + c4);
                s.x = fmaf(x.x, w.x, s.x); s.y = fmaf(x.y, w.y, s.y); s.z = fmaf(x.z, w.z, s.z); s.w = fmaf(x.w, w.w, s.w);
            }
            emit(t, s);
        }
    }
    if (t1 == sd.n)  // the last taps - 1 inputs are the history of the next step
        for (int e = 0; e < hrows; ++e) *(reinterpret_cast<float4*>(hw + (size_t)e * a.np) + c4) = input(sd.n - hrows + e);
}

// ------------------------------------------------------------------ selective scan
// A CTA walks one sequence for 32 channels; four (or eight) lanes share a channel and keep NS of its states
// each in registers.  Tiles of 32 tokens are staged in shared memory two deep (cp.async): dt_raw, x and z
// of the channels, B and C of the tokens; softplus is applied to a staged tile once, y leaves through the
// dt tile so that the gate and the store are coalesced.
constexpr int kScanCh = 32, kScanTok = 32;

template <int NS, int LPC, bool XF32, bool OF32, bool STEP>
__global__ void __launch_bounds__(kScanCh * LPC)
selective_scan_kernel(const SelectiveScanArgs a) {
    constexpr int THREADS = kScanCh * LPC, SP = NS * LPC;
    constexpr int TOK = STEP ? 1 : kScanTok;
    constexpr int XB = XF32 ? 4 : 2;
    struct Tile {
        float dt[TOK][kScanCh];
        float z[TOK][kScanCh];
        float bc[2][TOK][SP];
        uint8_t x[TOK * kScanCh * XB];
    };
    extern __shared__ __align__(16) uint8_t raw[];
    Tile* tiles = reinterpret_cast<Tile*>(raw);
    const int tid = threadIdx.x;
    const int c0 = blockIdx.x * kScanCh, ch = tid / LPC, sub = tid % LPC, c = c0 + ch;
    const bool live = c < a.inner;
    const int cc = live ? c : a.inner - 1;
    float A2[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) A2[i] = __ldg(a.A2 + (size_t)cc * SP + sub * NS + i);
    const float Dc_ch = __ldg(a.D + min(c0 + (tid & (kScanCh - 1)), a.inner - 1));  // of the channel this thread stores
    const float dtb_ch = __ldg(a.dt_b + min(c0 + (tid & (kScanCh - 1)), a.inner - 1));
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = a.seqs[blockIdx.y];
    float* Sg = a.S + ((size_t)sd.slot * a.inner + cc) * SP + sub * NS;
    float S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) S[i] = (sd.pos0 > 0) ? Sg[i] : 0.f;

    // channels beyond the end are read as the padding's zeros as far as the rows reach, else not at all
    auto stage = [&](int t0, Tile& T) {
        const int nt = min(TOK, sd.n - t0);
        for (int i = tid; i < nt * (kScanCh / 4); i += THREADS) {
            const int t = i >> 3, q = (i & 7) * 4;
            const size_t r = (size_t)(sd.row0 + t0 + t);
            if (c0 + q < a.inner) {
                if (!STEP) cp_async16(&T.dt[t][q], a.dt + r * a.lddt + c0 + q);
                cp_async16(&T.z[t][q], a.z + r * a.ldz + c0 + q);
                if (STEP) {}  // split rows: below
                else if (XF32) cp_async16(T.x + (t * kScanCh + q) * XB, static_cast<const float*>(a.x) + r * a.ldx + c0 + q);
                else cp_async8(T.x + (t * kScanCh + q) * XB, static_cast<const uint16_t*>(a.x) + r * a.ldx + c0 + q);
            }
        }
        for (int i = tid; i < nt * (SP / 4) * 2; i += THREADS) {
            const int which = i / (nt * (SP / 4)), k = i - which * nt * (SP / 4);
            const int t = k / (SP / 4), q = (k - t * (SP / 4)) * 4;
            cp_async16(&T.bc[which][t][q], a.bc + (size_t)(sd.row0 + t0 + t) * a.ldbc + (which ? a.c_col : a.b_col) + q);
        }
        cp_async_commit();
        if (STEP && tid < kScanCh && c0 + tid < a.inner)
            reinterpret_cast<float*>(T.x)[tid] = load_split(static_cast<const uint8_t*>(a.x) + (size_t)sd.row0 * a.ldx * 4, c0 + tid);
    };
    auto xval = [&](const Tile& T, int t, int k) {
        return XF32 ? reinterpret_cast<const float*>(T.x)[t * kScanCh + k] : bf16_to_f(reinterpret_cast<const uint16_t*>(T.x)[t * kScanCh + k]);
    };
    stage(0, tiles[0]);
    for (int t0 = 0, it = 0; t0 < sd.n; t0 += TOK, ++it) {
        Tile& T = tiles[STEP ? 0 : (it & 1)];
        const int nt = min(TOK, sd.n - t0);
        if (!STEP && t0 + TOK < sd.n) { stage(t0 + TOK, tiles[(it + 1) & 1]); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        if (STEP) {
            // dt_raw of the CTA's channels: the low-rank projection, LPC lanes per channel
            float s = 0.f;
            const float* lr = a.bc + (size_t)sd.row0 * a.ldbc;
            const uint16_t* wr = a.Wdt + (size_t)cc * a.ld_wdt;
            for (int r = sub * 2; r < a.rank; r += LPC * 2) {  // columns beyond the rank are zero in Wdt
                const uint32_t wp = __ldg(reinterpret_cast<const uint32_t*>(wr + r));
                s = fmaf(__uint_as_float(wp << 16), lr[r], s);
                s = fmaf(__uint_as_float(wp & 0xffff0000u), lr[r + 1], s);
            }
#pragma unroll
            for (int m = 1; m < LPC; m <<= 1) s += __shfl_xor_sync(0xffffffffu, s, m);
            if (sub == 0) T.dt[0][ch] = s;
            __syncthreads();
        }
        for (int i = tid; i < nt * kScanCh; i += THREADS) {  // THREADS is a multiple of kScanCh: always the same channel
            float& d = (&T.dt[0][0])[i];
            d = softplusf_(d + dtb_ch);
        }
        __syncthreads();
        // y of four tokens at a time: their lane sums are formed together
        for (int tb = 0; tb < nt; tb += 4) {
            float y[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                y[u] = 0.f;
                if (STEP && u > 0) continue;
                const int t = min(tb + u, TOK - 1);
                if (tb + u < nt) {
                    const float dt = T.dt[t][ch], dx = dt * xval(T, t, ch);
#pragma unroll
                    for (int i = 0; i < NS; ++i) {
                        S[i] = fmaf(ex2(dt * A2[i]), S[i], dx * T.bc[0][t][sub * NS + i]);
                        y[u] = fmaf(S[i], T.bc[1][t][sub * NS + i], y[u]);
                    }
                }
            }
            reduce_scatter<4, LPC>(y, tid);
            const int t = tb + scatter_first<4, LPC>(tid);
            __syncwarp();  // the lanes of the channel have read dt of these tokens
            if (t < nt && scatter_owner<4, LPC>(tid)) T.dt[t][ch] = y[0];
        }
        __syncthreads();
        for (int i = tid; i < nt * kScanCh; i += THREADS) {
            const int t = i / kScanCh, k = i & (kScanCh - 1);
            if (c0 + k < a.inner) {
                const float v = (T.dt[t][k] + Dc_ch * xval(T, t, k)) * silu(T.z[t][k]);
                if (STEP) store_split(static_cast<uint8_t*>(a.out) + (size_t)sd.row0 * a.ldo * 4, c0 + k, v);
                else store1<OF32>(a.out, (size_t)(sd.row0 + t0 + t) * a.ldo + c0 + k, v);
            }
        }
        __syncthreads();  // the tile may be staged again
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NS; ++i) Sg[i] = S[i];
    }
}

// ------------------------------------------------------------------ gated delta rule
// The columns of a head's state S [D, Dv] do not touch one another: with S the state before the token,
//   u = beta (v - g S^T k),   o = g S^T q + (k.q) u,   S <- g S + k u^T
// - both products read the old state, so one reduction serves them.  The decay is kept out of the state: with
// S = c R and c the product of the decays since c was last 1,
//   c <- c g,   u = beta (v - c R^T k),   o = c R^T q + (k.q) u,   R <- R + k (u / c)^T
// which is three multiply-adds per element instead of four operations; when c has become small R takes it in.
// L = D / 16 lanes share a group of NC columns and keep 16 rows of each in registers (as pairs: one instruction
// does two multiply-adds); lane l owns rows 4 (l + L i) .. + 3, so the lanes read consecutive 16-byte pieces of
// k and q.
// With a decay per key channel (CH) g is a vector over the rows of S: every row takes its decay in first, which is
// a fourth operation per element, and the products read S already decayed:
//   S <- diag(g) S,   u = beta (v - S^T k),   o = S^T q + (k.q) u,   S <- S + k u^T
constexpr int kDeltaTok = 16;
constexpr float kDeltaSmall = 1e-9f;

template <int L, int NC, bool CH = false>
struct DeltaCore {
    static constexpr int D = 16 * L, CNT = 2 * NC;            // totals per token: R^T k of the columns, then R^T q
    static constexpr int kHeld = L >= CNT ? 1 : CNT / L;      // ... of which a lane holds this many after the reduction
    static constexpr int kOut = kHeld > NC ? NC : kHeld;      // ... belonging to one of the two products
    uint64_t S[NC][8];  // R
    float c;
    __device__ __forceinline__ void zero() {
        c = 1.f;
#pragma unroll
        for (int j = 0; j < NC; ++j)
#pragma unroll
            for (int i = 0; i < 8; ++i) S[j][i] = 0ull;
    }
    // column j of this group at base + j * D; columns from ncol on are left alone
    __device__ __forceinline__ void load(const float* base, int l, int ncol) {
        c = 1.f;
#pragma unroll
        for (int j = 0; j < NC; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                ulonglong2 v = make_ulonglong2(0ull, 0ull);
                if (j < ncol) v = *reinterpret_cast<const ulonglong2*>(base + (size_t)j * D + 4 * (l + L * i));
                S[j][2 * i] = v.x;
                S[j][2 * i + 1] = v.y;
            }
    }
    __device__ __forceinline__ void absorb() {
        const uint64_t cc = pack2(c, c);
#pragma unroll
        for (int j = 0; j < NC; ++j)
#pragma unroll
            for (int i = 0; i < 8; ++i) S[j][i] = mul2(cc, S[j][i]);
        c = 1.f;
    }
    __device__ __forceinline__ void store(float* base, int l, int ncol) {
        if (!CH) absorb();
#pragma unroll
        for (int j = 0; j < NC; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (j < ncol) *reinterpret_cast<ulonglong2*>(base + (size_t)j * D + 4 * (l + L * i)) = make_ulonglong2(S[j][2 * i], S[j][2 * i + 1]);
    }
    // o[j] of token() is column ocol + j, on the lanes where owns_o holds (the reduction's first halving, by lane
    // bit 0, separates R^T k from R^T q)
    static __device__ __forceinline__ int ocol(int lane) { return scatter_first<CNT, L>(lane) & (NC - 1); }
    static __device__ __forceinline__ bool owns_o(int lane) { return (lane & 1) && scatter_owner<CNT, L>(lane); }
    struct Row { uint64_t r[8]; };  // this lane's pairs of a D-vector in shared memory
    static __device__ __forceinline__ Row row(const float* p, int l) {
        Row x;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p + 4 * (l + L * i));
            x.r[2 * i] = v.x;
            x.r[2 * i + 1] = v.y;
        }
        return x;
    }
    // One token.  kr: its key; qr: its query on entry, the row at q_next on return (requested as soon as the registers are
    // free); v: the group's values in shared memory.  CH: the decays are gr (g is not used), the row at g_next on return.
    __device__ __forceinline__ void token(const Row& kr, Row& qr, const float* q_next, const float* v, float g, float beta, float kq, int lane,
                                          float (&o)[kOut], Row* gr = nullptr, const float* g_next = nullptr) {
        float inv_c = 1.f;
        if constexpr (CH) {
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < NC; ++j) S[j][i] = mul2(gr->r[i], S[j][i]);
            *gr = row(g_next, lane & (L - 1));
        } else {
            c *= g;
            if (c < kDeltaSmall) absorb();  // (the same decay in all lanes of a head)
            inv_c = __fdividef(1.0f, c);
        }
        const float cs = CH ? 1.f : c;
        uint64_t acc[CNT];
#pragma unroll
        for (int j = 0; j < CNT; ++j) acc[j] = 0ull;
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < NC; ++j) {
                acc[j] = fma2(kr.r[i], S[j][i], acc[j]);
                acc[NC + j] = fma2(qr.r[i], S[j][i], acc[NC + j]);
            }
        qr = row(q_next, lane & (L - 1));
        float t[CNT];
#pragma unroll
        for (int j = 0; j < CNT; ++j) {
            float x, y;
            unpack2(acc[j], x, y);
            t[j] = x + y;
        }
        reduce_scatter<CNT, L>(t, lane);
        const int first = scatter_first<CNT, L>(lane);  // t[j] is total number first + j
        float um[kOut];
#pragma unroll
        for (int j = 0; j < kOut; ++j) um[j] = beta * (v[(first + j) & (NC - 1)] - cs * t[j]);
        const int base = lane & ~(L - 1);
        float u[NC];
#pragma unroll
        for (int j = 0; j < NC; ++j) u[j] = __shfl_sync(0xffffffffu, um[scatter_slot<CNT, L>(j) & (kOut - 1)], base + scatter_lane<CNT, L>(j));
#pragma unroll
        for (int j = 0; j < kOut; ++j) {
            const int col = (first + j) & (NC - 1);
            float uc = u[0];
#pragma unroll
            for (int x = 1; x < NC; ++x) uc = col == x ? u[x] : uc;
            o[j] = fmaf(cs, t[j], kq * uc);
        }
#pragma unroll
        for (int j = 0; j < NC; ++j) {
            const float us = CH ? u[j] : u[j] * inv_c;
            const uint64_t uu = pack2(us, us);
#pragma unroll
            for (int i = 0; i < 8; ++i) S[j][i] = fma2(kr.r[i], uu, S[j][i]);
        }
    }
};

// What the scan wants per token: convolved and activated q and k as unit vectors (q also times D^-1/2) and, per
// head, {decay, beta, k.q}.  One warp per (sequence, key/value head, run of 16 tokens), a lane holding channels
// lane, lane + 32, ... (V of them) of q and k; two tokens at a time.
template <int TAPS, int V>
__global__ void __launch_bounds__(128)
delta_prep_kernel(const DeltaArgs a) {
    constexpr int W = TAPS > 0 ? TAPS : 1;
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = a.seqs[blockIdx.z];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t0 = (blockIdx.y * 4 + warp) * kDeltaTok, g = blockIdx.x;
    if (t0 >= sd.n) return;
    const int t1 = min(sd.n, t0 + kDeltaTok);
    const int taps = TAPS > 0 ? TAPS : a.taps, hrows = taps - 1;
    const float* hr = a.hist + ((size_t)sd.bank * a.max_slots + sd.slot) * hrows * a.np;
    float* hw = a.hist + ((size_t)(sd.bank ^ 1) * a.max_slots + sd.slot) * hrows * a.np;
    const float* xin = a.raw + (size_t)sd.row0 * a.ld_raw;
    float* qkv = const_cast<float*>(a.qkv) + (size_t)sd.row0 * a.ld;
    const int base[2] = {g * a.Dl, a.k_col + g * a.Dl};  // first channel of q and of k
    auto input = [&](int i, int ch) {
        if (i >= 0) return xin[(size_t)i * a.ld_raw + ch];
        if (sd.pos0 + i < 0) return 0.f;
        return hr[(size_t)(hrows + i) * a.np + ch];
    };
    const float qscale = rsqrtf((float)a.D);
    const int per = a.H / a.G;
    // the gates of the run's tokens and heads, side by side
    if (a.decay) {
        const int d4 = a.Dl >> 2, n4 = per * d4;  // the group's heads are neighbours
        for (int i = lane; i < (t1 - t0) * n4; i += 32) {
            const int t = t0 + i / n4, c4 = i % n4;
            float4* dp = reinterpret_cast<float4*>(a.decay + (size_t)(sd.row0 + t) * a.ld_decay + (size_t)g * per * a.Dl) + c4;
            const float4 b = __ldg(reinterpret_cast<const float4*>(a.dt_bias + (size_t)g * per * a.Dl) + c4);
            const float A = __ldg(a.negA + g * per + c4 / d4);
            float4 x = *dp;
            x.x = expf(A * softplusf_(x.x + b.x)); x.y = expf(A * softplusf_(x.y + b.y));
            x.z = expf(A * softplusf_(x.z + b.z)); x.w = expf(A * softplusf_(x.w + b.w));
            *dp = x;
        }
    }
    for (int i = lane; i < (t1 - t0) * per; i += 32) {
        const int t = t0 + i / per, h = g * per + i % per;
        const float* gr = a.gates + (size_t)(sd.row0 + t) * a.ldg;
        const float decay = a.decay ? 1.f : expf(__ldg(a.negA + h) * softplusf_(gr[a.a_col + h] + __ldg(a.dt_bias + h)));
        *reinterpret_cast<float2*>(a.coef + (size_t)(sd.row0 + t) * a.H + h) = make_float2(decay, sigmoidf_(gr[a.b_col + h]));
    }
    float w[2][V][W], win[2][V][W];  // weights and the window of earlier inputs
    if (TAPS > 0) {
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int i = 0; i < V; ++i) {
                const int d = lane + i * 32;
#pragma unroll
                for (int j = 0; j < W; ++j) {
                    w[x][i][j] = d < a.Dl ? __ldg(a.conv_w + (size_t)j * a.np + base[x] + d) : 0.f;
                    win[x][i][j] = (d < a.Dl && j + 1 < W) ? input(t0 - (W - 1) + j, base[x] + d) : 0.f;
                }
            }
    }
    for (int tb = t0; tb < t1; tb += 2) {
        float in[2][2][V];  // [token][q, k]
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    const int d = lane + i * 32;
                    in[u][x][i] = 0.f;
                    if (d < a.Dl && tb + u < t1) {
                        if (TAPS > 0) in[u][x][i] = input(tb + u, base[x] + d);
                        else
                            for (int j = 0; j < taps; ++j)
                                in[u][x][i] = fmaf(input(tb + u - hrows + j, base[x] + d), __ldg(a.conv_w + (size_t)j * a.np + base[x] + d), in[u][x][i]);
                    }
                }
        float sum[2][3];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            sum[u][0] = sum[u][1] = sum[u][2] = 0.f;
#pragma unroll
            for (int i = 0; i < V; ++i) {
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    float y = in[u][x][i];
                    if (TAPS > 0) {
                        win[x][i][W - 1] = y;
                        y = 0.f;
#pragma unroll
                        for (int j = 0; j < W; ++j) y = fmaf(win[x][i][j], w[x][i][j], y);
#pragma unroll
                        for (int j = 0; j + 1 < W; ++j) win[x][i][j] = win[x][i][j + 1];
                    }
                    in[u][x][i] = silu(y);
                }
                sum[u][0] = fmaf(in[u][0][i], in[u][0][i], sum[u][0]);
                sum[u][1] = fmaf(in[u][1][i], in[u][1][i], sum[u][1]);
                sum[u][2] = fmaf(in[u][0][i], in[u][1][i], sum[u][2]);
            }
        }
#pragma unroll
        for (int s = 16; s >= 1; s >>= 1)
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int x = 0; x < 3; ++x) sum[u][x] += __shfl_xor_sync(0xffffffffu, sum[u][x], s);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int t = tb + u;
            if (t >= t1) break;
            const float r[2] = {qscale / sqrtf(sum[u][0] + 1e-6f), 1.0f / sqrtf(sum[u][1] + 1e-6f)};
            float* row = qkv + (size_t)t * a.ld;
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int i = 0; i < V; ++i)
                    if (lane + i * 32 < a.Dl) row[base[x] + lane + i * 32] = in[u][x][i] * r[x];
            const float kq = sum[u][2] * r[0] * r[1];
            for (int j = lane; j < per; j += 32) a.coef[(size_t)(sd.row0 + t) * a.H + g * per + j].z = kq;
        }
    }
    if (t1 == sd.n)  // the last inputs are the history of the next step
        for (int e = 0; e < hrows; ++e)
            for (int d = lane; d < a.Dl; d += 32) {
                hw[(size_t)e * a.np + base[0] + d] = input(sd.n - hrows + e, base[0] + d);
                hw[(size_t)e * a.np + base[1] + d] = input(sd.n - hrows + e, base[1] + d);
            }
}

// Prefill: a CTA walks one (sequence, head) for blockDim.x / L * NC columns of Dv, in tiles of 16 tokens (8 with a decay
// per channel) staged two deep by asynchronous copies.
__host__ __device__ constexpr int delta_tile_tokens(bool channel) { return channel ? 8 : kDeltaTok; }
// floats of a tile: q, k, decays, v, coefficients
__host__ __device__ constexpr int delta_tile_floats(int D, int cpad, bool channel) { return delta_tile_tokens(channel) * ((channel ? 3 : 2) * D + cpad + 4); }
template <int L, int NC, bool CH>
__global__ void __launch_bounds__(128)
delta_scan_kernel(const DeltaArgs a) {
    using Core = DeltaCore<L, NC, CH>;
    constexpr int D = 16 * L, TOK = delta_tile_tokens(CH), VECS = CH ? 3 : 2;
    extern __shared__ __align__(16) float sm[];
    const int tid = threadIdx.x, lane = tid & 31;
    const int cols = blockDim.x / L * NC;
    const int cpad = (cols + 3) & ~3;
    const int tile_f = delta_tile_floats(D, cpad, CH);
    const int h = blockIdx.x, c0 = blockIdx.y * cols;
    const int kvh = h / (a.H / a.G);
    // rows of k and q beyond the head's dimension and columns beyond Dv stay zero in both tiles
    for (int i = tid; i < 2 * tile_f + D; i += blockDim.x) sm[i] = 0.f;
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = a.seqs[blockIdx.z];
    const int grp = tid / L, l = tid & (L - 1);
    const int gc = c0 + grp * NC;           // first column of this group
    const int ncol = min(NC, a.Dv - gc);    // may be <= 0
    Core core;
    float* Sg = a.S + (((size_t)sd.slot * a.H + h) * a.Dv + (gc < a.Dv ? gc : 0)) * D;
    if (sd.pos0 > 0) core.load(Sg, l, ncol);
    else core.zero();
    __syncthreads();

    const int d4 = a.Dl >> 2, v4 = min(cpad, a.Dvl - c0) >> 2;  // (c0 is a multiple of 4)
    const float* src0 = a.qkv + (size_t)sd.row0 * a.ld;
    auto stage = [&](int t0, int buf) {
        float* q = sm + buf * tile_f;
        const int nt = min(TOK, sd.n - t0);
        const int per = VECS * d4 + v4;
        for (int j = tid; j < per; j += blockDim.x) {  // a 16-byte column piece of all tokens
            const float* src = src0 + (size_t)t0 * a.ld;
            float* dst;
            int step = D, ld = a.ld;
            if (j < d4) { src += kvh * a.Dl + j * 4; dst = q + j * 4; }
            else if (j < 2 * d4) { src += a.k_col + kvh * a.Dl + (j - d4) * 4; dst = q + TOK * D + (j - d4) * 4; }
            else if (CH && j < 3 * d4) {
                ld = a.ld_decay;
                src = a.decay + (size_t)(sd.row0 + t0) * ld + (size_t)h * a.Dl + (j - 2 * d4) * 4;
                dst = q + 2 * TOK * D + (j - 2 * d4) * 4;
            } else { src += a.v_col + h * a.Dvl + c0 + (j - VECS * d4) * 4; dst = q + VECS * TOK * D + (j - VECS * d4) * 4; step = cpad; }
            for (int t = 0; t < nt; ++t) cp_async16(dst + t * step, src + (size_t)t * ld);
        }
        if (tid < nt) cp_async16(q + TOK * (VECS * D + cpad) + tid * 4, a.coef + (size_t)(sd.row0 + t0 + tid) * a.H + h);
        cp_async_commit();
    };
    stage(0, 0);
    const int oc = Core::ocol(lane);
    const bool ow = Core::owns_o(lane);
    float* orow = a.out + (size_t)sd.row0 * a.ldo + h * a.Dvl + gc + oc;
    for (int t0 = 0, it = 0; t0 < sd.n; t0 += TOK, ++it) {
        const int buf = it & 1, nt = min(TOK, sd.n - t0);
        if (t0 + TOK < sd.n) { stage(t0 + TOK, buf ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const float* q = sm + buf * tile_f;
        const float* k = q + TOK * D;
        const float* gd = k + TOK * D;  // (CH)
        const float* v = q + VECS * TOK * D + grp * NC;
        const float* cf = q + TOK * (VECS * D + cpad);
        typename Core::Row qr = Core::row(q, l), kr = Core::row(k, l), gr;
        if (CH) gr = Core::row(gd, l);
#pragma unroll 2
        for (int t = 0; t < nt; ++t) {
            const float4 co = *reinterpret_cast<const float4*>(cf + t * 4);
            const int tn = min(t + 1, TOK - 1);
            const typename Core::Row kn = Core::row(k + tn * D, l);
            float o[Core::kOut];
            core.token(kr, qr, q + tn * D, v + t * cpad, co.x, co.y, co.z, lane, o, &gr, gd + tn * D);
            kr = kn;
            if (ow) {
#pragma unroll
                for (int j = 0; j < Core::kOut; ++j)
                    if (oc + j < ncol) orow[j] = o[j];
            }
            orow += a.ldo;
        }
        __syncthreads();
    }
    core.store(Sg, l, ncol);
}

// Decode: one CTA per (head, sequence) takes its token through unit norms, the rule, the output norm and the gate.  CH: the
// decays and the output gate come from low-rank projections, whose second halves are formed here (eight lanes per row).
constexpr int kDeltaStepThreads = 256, kDeltaStepCols = 4;
template <int L, bool CH>
__global__ void __launch_bounds__(kDeltaStepThreads)
delta_step_kernel(const DeltaArgs a) {
    constexpr int D = 16 * L, COLS = kDeltaStepThreads / L * kDeltaStepCols;
    using Core = DeltaCore<L, kDeltaStepCols, CH>;
    extern __shared__ __align__(16) float sm[];  // q [D], k [D], v and o [vpad each]; CH: decays [D], gate [vpad], low-rank inputs
    __shared__ float red[8];
    float* q = sm;
    float* k = q + D;
    float* v = k + D;
    const int vpad = (a.Dvl + COLS - 1) & ~3;
    float* o = v + vpad;
    const int tid = threadIdx.x, lane = tid & 31;
    const int h = blockIdx.x, per = a.H / a.G, kvh = h / per;
    const float negA = __ldg(a.negA + h), dtb = CH ? 0.f : __ldg(a.dt_bias + h);
    float* gd = o + vpad;
    float* gate = gd + D;
    float* low = gate + vpad;
    // The descriptor and the state were there before the previous kernel started (every kernel of a step waits for the one before
    // it): they are asked for before that kernel has finished, and so are weights.
    const SeqDesc sd = a.seqs[blockIdx.y];
    const int grp = tid / L, l = tid & (L - 1);
    Core core;
    float* Sh = a.S + ((size_t)sd.slot * a.H + h) * a.Dv * D;
    auto fetch = [&](int gc) {
        if (sd.pos0 > 0) core.load(Sh + (size_t)(gc < a.Dv ? gc : 0) * D, l, min(kDeltaStepCols, a.Dv - gc));
        else core.zero();
    };
    if (!CH) fetch(grp * kDeltaStepCols);
    // CH: rows r, r + 32, ... of a low-rank matrix are this group of eight lanes', columns sub * 8 .. and 64 + sub * 8 .. of each
    // this lane's (more than 128 columns: one at a time); RU rows on their way at a time
    constexpr int LR = 8, RU = 4, LROWS = kDeltaStepThreads / LR;
    const int sub = tid & (LR - 1);
    uint4 wl[RU][2];
    const uint16_t* low_w[2] = {a.w_low + (size_t)h * a.Dl * a.ld_low, a.w_low + (size_t)(a.gate_row + h * a.Dvl) * a.ld_low + a.low_a};
    auto low_fetch = [&](int half, int r0) {
        const int rows = half ? a.Dv : a.D, cols = half ? a.low_g : a.low_a;
#pragma unroll
        for (int u = 0; u < RU; ++u)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int r = r0 + u * LROWS, col = (sub + x * LR) * 8;
                wl[u][x] = make_uint4(0u, 0u, 0u, 0u);
                if (r < rows && col < cols) wl[u][x] = __ldg(reinterpret_cast<const uint4*>(low_w[half] + (size_t)r * a.ld_low + col));
            }
    };
    if (CH) {
        if (tid == 0 && sd.pos0 > 0) l2_prefetch_bulk(Sh, (uint32_t)a.Dv * D * 4);
        low_fetch(0, tid / LR);
    }
    const float norm_w = tid < a.Dv ? __ldg(a.norm_w + tid) : 0.f;
    for (int i = tid; i < (CH ? 3 * D + 3 * vpad : 2 * D + 2 * vpad); i += kDeltaStepThreads) sm[i] = 0.f;
    griddep_wait();
    griddep_launch_dependents();
    const float* row = a.qkv + (size_t)sd.row0 * a.ld;
    __syncthreads();
    for (int i = tid; i < 2 * a.Dl + a.Dvl; i += kDeltaStepThreads) {
        if (i < a.Dl) q[i] = row[kvh * a.Dl + i];
        else if (i < 2 * a.Dl) k[i - a.Dl] = row[a.k_col + kvh * a.Dl + i - a.Dl];
        else v[i - 2 * a.Dl] = row[a.v_col + h * a.Dvl + i - 2 * a.Dl];
    }
    if (CH)
        for (int i = tid; i < a.low_a + a.low_g; i += kDeltaStepThreads) low[i] = row[a.low_col + i];
    __syncthreads();
    if (CH) {
        for (int half = 0; half < 2; ++half) {
            const int rows = half ? a.Dv : a.D, cols = half ? a.low_g : a.low_a;
            const float* lo = low + (half ? a.low_a : 0);
            float4 x[2][2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int col = (sub + i * LR) * 8;
                x[i][0] = x[i][1] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (col < cols) { x[i][0] = *reinterpret_cast<const float4*>(lo + col); x[i][1] = *reinterpret_cast<const float4*>(lo + col + 4); }
            }
            auto add = [&](float s, const uint4& w, const float4& p, const float4& q4) {
                s = fmaf(__uint_as_float(w.x << 16), p.x, s); s = fmaf(__uint_as_float(w.x & 0xffff0000u), p.y, s);
                s = fmaf(__uint_as_float(w.y << 16), p.z, s); s = fmaf(__uint_as_float(w.y & 0xffff0000u), p.w, s);
                s = fmaf(__uint_as_float(w.z << 16), q4.x, s); s = fmaf(__uint_as_float(w.z & 0xffff0000u), q4.y, s);
                s = fmaf(__uint_as_float(w.w << 16), q4.z, s); s = fmaf(__uint_as_float(w.w & 0xffff0000u), q4.w, s);
                return s;
            };
            for (int r0 = tid / LR; r0 < rows; r0 += RU * LROWS) {
                float s[RU];
#pragma unroll
                for (int u = 0; u < RU; ++u) {
                    s[u] = add(add(0.f, wl[u][0], x[0][0], x[0][1]), wl[u][1], x[1][0], x[1][1]);
                    const int r = r0 + u * LROWS;
                    if (r < rows)
                        for (int col = (sub + 2 * LR) * 8; col < cols; col += LR * 8)
                            s[u] = add(s[u], __ldg(reinterpret_cast<const uint4*>(low_w[half] + (size_t)r * a.ld_low + col)),
                                       *reinterpret_cast<const float4*>(lo + col), *reinterpret_cast<const float4*>(lo + col + 4));
                }
                if (r0 + RU * LROWS < rows) low_fetch(half, r0 + RU * LROWS);
                else if (half == 0) low_fetch(1, tid / LR);
#pragma unroll
                for (int u = 0; u < RU; ++u) {
                    const int r = r0 + u * LROWS;
#pragma unroll
                    for (int m = 1; m < LR; m <<= 1) s[u] += __shfl_xor_sync(0xffu << (lane & 24), s[u], m);
                    if (sub == 0 && r < rows) {
                        if (half) gate[r] = sigmoidf_(s[u]);
                        else gd[r] = expf(negA * softplusf_(s[u] + __ldg(a.dt_bias + (size_t)h * a.Dl + r)));
                    }
                }
            }
            if (half == 0 && tid / LR >= rows) low_fetch(1, tid / LR);  // (a group without a row in the first half)
        }
        fetch(grp * kDeltaStepCols);
    }
    float sq = 0.f, sk = 0.f, dot = 0.f;  // every warp for itself
    for (int d = lane; d < D; d += 32) { sq = fmaf(q[d], q[d], sq); sk = fmaf(k[d], k[d], sk); dot = fmaf(q[d], k[d], dot); }
    sq = warp_sum(sq); sk = warp_sum(sk); dot = warp_sum(dot);
    const float rq = rsqrtf((float)a.D) / sqrtf(sq + 1e-6f), rk = 1.0f / sqrtf(sk + 1e-6f);
    const float g = CH ? 1.f : expf(negA * softplusf_(row[a.a_col + h] + dtb)), beta = sigmoidf_(row[a.b_col + h]);
    __syncthreads();
    for (int d = tid; d < D; d += kDeltaStepThreads) { q[d] *= rq; k[d] *= rk; }
    __syncthreads();
    const int oc = Core::ocol(lane);
    const bool ow = Core::owns_o(lane);
    const typename Core::Row kr = Core::row(k, l);
    typename Core::Row qr = Core::row(q, l);
    for (int c0 = 0; c0 < a.Dv; c0 += COLS) {
        const int gc = c0 + grp * kDeltaStepCols, ncol = min(kDeltaStepCols, a.Dv - gc);
        if (c0 > 0) fetch(gc);
        float ov[Core::kOut];
        typename Core::Row gr;
        if (CH) gr = Core::row(gd, l);
        core.token(kr, qr, q, v + gc, g, beta, dot * rq * rk, lane, ov, &gr, gd);
        if (ow) {
#pragma unroll
            for (int j = 0; j < Core::kOut; ++j)
                if (oc + j < ncol) o[gc + oc + j] = ov[j];
        }
        core.store(Sh + (size_t)(gc < a.Dv ? gc : 0) * D, l, ncol);
    }
    __syncthreads();
    float s = 0.f;
    for (int d = tid; d < a.Dv; d += kDeltaStepThreads) s += o[d] * o[d];
    const float r = 1.0f / sqrtf(block_sum(s, red) / (float)a.Dv + a.eps);
    for (int d = tid; d < a.Dv; d += kDeltaStepThreads)
        store_split(reinterpret_cast<uint8_t*>(a.out) + (size_t)sd.row0 * a.ldo * 4, h * a.Dv + d,
                    o[d] * r * (d < kDeltaStepThreads ? norm_w : __ldg(a.norm_w + d)) * (CH ? gate[d] : silu(row[a.gate_col + h * a.Dvl + d])));
}

// ------------------------------------------------------------------ minGRU
// A CTA walks one sequence for 32 channels, 64 tokens at a time: each of 8 warps takes 8 consecutive
// tokens (lane = channel), first as the affine map S -> A S + b that they amount to, and once the maps
// of the warps before it are known - through shared memory - as the states themselves.  The inputs of the next
// 64 tokens are requested before these are worked on.
constexpr int kGruWarps = 8, kGruTok = 8;
template <bool F32>
__global__ void __launch_bounds__(kGruWarps * 32, 3)
min_gru_kernel(const MinGruArgs a) {
    __shared__ float mapA[2][kGruWarps][32], mapB[2][kGruWarps][32];
    griddep_wait();
    griddep_launch_dependents();
    const SeqDesc sd = a.seqs[blockIdx.y];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int c = blockIdx.x * 32 + lane;
    const bool live = c < a.width;
    float* Sg = a.S + (size_t)sd.slot * a.width + c;
    float S = (live && sd.pos0 > 0) ? *Sg : 0.f;  // state before the block of tokens (the same in every warp)
    const float* base = a.zx + (size_t)sd.row0 * a.ld + c;
    float nz[kGruTok], nu[kGruTok], ng[kGruTok];
    auto request = [&](int tw) {
#pragma unroll
        for (int i = 0; i < kGruTok; ++i) {
            nz[i] = nu[i] = ng[i] = 0.f;
            if (live && tw + i < sd.n) {
                const float* r = base + (size_t)(tw + i) * a.ld;
                nz[i] = r[a.z_col];
                nu[i] = r[a.x_col];
                ng[i] = r[a.g_col];
            }
        }
    };
    request(warp * kGruTok);
    for (int t0 = 0, it = 0; t0 < sd.n; t0 += kGruWarps * kGruTok, ++it) {
        float (&mA)[kGruWarps][32] = mapA[it & 1];
        float (&mB)[kGruWarps][32] = mapB[it & 1];
        const int tw = t0 + warp * kGruTok;
        float zi[kGruTok], ui[kGruTok], gi[kGruTok];
#pragma unroll
        for (int i = 0; i < kGruTok; ++i) { zi[i] = nz[i]; ui[i] = nu[i]; gi[i] = ng[i]; }
        request(tw + kGruWarps * kGruTok);
        float A = 1.f, b = 0.f;
#pragma unroll
        for (int i = 0; i < kGruTok; ++i) {
            const float z = tw + i < sd.n ? sigmoidf_(zi[i]) : 0.f;
            const float cand = ui[i] >= 0.f ? ui[i] + 0.5f : sigmoidf_(ui[i]);
            zi[i] = 1.f - z;
            ui[i] = z * cand;
            A *= zi[i];
            b = fmaf(zi[i], b, ui[i]);
        }
        mA[warp][lane] = A;
        mB[warp][lane] = b;
        __syncthreads();  // (two sets of maps: the next block's writes do not meet this block's reads)
        float s = S;
#pragma unroll
        for (int w = 0; w < kGruWarps; ++w) {
            if (w == warp) s = S;
            S = fmaf(mA[w][lane], S, mB[w][lane]);
        }
#pragma unroll
        for (int i = 0; i < kGruTok; ++i) {
            s = fmaf(zi[i], s, ui[i]);
            if (live && tw + i < sd.n) store1<F32>(a.out, (size_t)(sd.row0 + tw + i) * a.ldo + c, s * silu(gi[i]) * a.out_scale);
        }
    }
    if (live && warp == 0) *Sg = S;
}

template <int NS, int LPC, bool XF32, bool OF32, bool STEP>
int launch_scan_one(b200_ctx* ctx, const SelectiveScanArgs& a, int E) {
    constexpr int TOK = STEP ? 1 : kScanTok;
    constexpr size_t tile = (size_t)TOK * kScanCh * 8 + (size_t)2 * TOK * NS * LPC * 4 + (size_t)TOK * kScanCh * (XF32 ? 4 : 2);
    constexpr size_t smem = ((tile + 15) & ~(size_t)15) * (STEP ? 1 : 2);
    static_assert(smem <= 227 * 1024, "tiles in shared memory");
    static bool attr_set[64] = {};
    if (!attr_set[ctx->device & 63]) {
        B200_CUDA(ctx, cudaFuncSetAttribute(selective_scan_kernel<NS, LPC, XF32, OF32, STEP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        attr_set[ctx->device & 63] = true;
    }
    cudaError_t le = launch_pdl(ctx, selective_scan_kernel<NS, LPC, XF32, OF32, STEP>, dim3((a.inner + kScanCh - 1) / kScanCh, E), dim3(kScanCh * LPC), smem, a);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

template <int NS, int LPC>
int launch_scan_types(b200_ctx* ctx, const SelectiveScanArgs& a, int E, bool x_f32, bool out_f32) {
    if (a.Wdt) return launch_scan_one<NS, LPC, true, true, true>(ctx, a, E);
    if (x_f32 && out_f32) return launch_scan_one<NS, LPC, true, true, false>(ctx, a, E);
    if (!x_f32 && !out_f32) return launch_scan_one<NS, LPC, false, false, false>(ctx, a, E);
    return B200_ERR_SHAPE;
}

template <int L, bool CH>
int launch_delta_step_one(b200_ctx* ctx, const DeltaArgs& a, int E) {
    const int vpad = (a.Dvl + kDeltaStepThreads / L * kDeltaStepCols - 1) & ~3;
    const size_t smem = (size_t)(CH ? 48 * L + 3 * vpad + a.low_a + a.low_g : 32 * L + 2 * vpad) * 4;
    if (smem > 47 * 1024) return B200_ERR_LIMIT;
    cudaError_t le = launch_pdl(ctx, delta_step_kernel<L, CH>, dim3(a.H, E), dim3(kDeltaStepThreads), smem, a);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

template <int L, int NC, bool CH>
int launch_delta_scan_one(b200_ctx* ctx, const DeltaArgs& a, int E) {
    constexpr int D = 16 * L;
    const int groups = (a.Dv + NC - 1) / NC;
    // two warps per CTA (a block of columns starts at a multiple of four columns)
    int threads = (groups * L + 31) & ~31;
    if (threads > 64) threads = 64;
    while (threads / L * NC % 4) threads += 32;
    const int cols = threads / L * NC, cpad = (cols + 3) & ~3;
    const size_t smem = (size_t)(2 * delta_tile_floats(D, cpad, CH) + D) * 4;
    if (smem > 200 * 1024) return B200_ERR_LIMIT;
    static bool attr_set[64] = {};
    if (!attr_set[ctx->device & 63]) {
        B200_CUDA(ctx, cudaFuncSetAttribute(delta_scan_kernel<L, NC, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        attr_set[ctx->device & 63] = true;
    }
    cudaError_t le = launch_pdl(ctx, delta_scan_kernel<L, NC, CH>, dim3(a.H, (a.Dv + cols - 1) / cols, E), dim3(threads), smem, a);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

// Columns per group: four are the cheapest per column, but with few sequences and heads the warps would be too
// few to hide the chain from token to token.
template <int L, bool CH>
int launch_delta_scan_ch(b200_ctx* ctx, const DeltaArgs& a, int E) {
    static const int forced = [] { const char* e = getenv("B200_DELTA_COLS"); return e ? atoi(e) : 0; }();  // tuning hook: 1, 2 or 4
    const long columns = (long)a.H * E * a.Dv;
    auto warps = [&](int nc) { return columns / nc * L / 32; };
    const int nc = forced ? forced : (warps(4) >= 6L * ctx->num_sms ? 4 : (warps(2) >= 4L * ctx->num_sms ? 2 : 1));
    if (nc == 4) return launch_delta_scan_one<L, 4, CH>(ctx, a, E);
    if (nc == 2) return launch_delta_scan_one<L, 2, CH>(ctx, a, E);
    return launch_delta_scan_one<L, 1, CH>(ctx, a, E);
}
template <int L>
int launch_delta_scan_l(b200_ctx* ctx, const DeltaArgs& a, int E) {
    return a.decay ? launch_delta_scan_ch<L, true>(ctx, a, E) : launch_delta_scan_ch<L, false>(ctx, a, E);
}
template <int L>
int launch_delta_step_l(b200_ctx* ctx, const DeltaArgs& a, int E) {
    return a.w_low ? launch_delta_step_one<L, true>(ctx, a, E) : launch_delta_step_one<L, false>(ctx, a, E);
}

}  // namespace

int launch_short_conv(b200_ctx* ctx, const ShortConvArgs& a, int E, int max_n, bool f32) {
    const dim3 grid(((a.np - a.ch0) / 4 + 127) / 128, (max_n + kConvTok - 1) / kConvTok, E), block(128);
    cudaError_t le;
    switch (a.taps) {
        case 2: le = f32 ? launch_pdl(ctx, short_conv_kernel<2, true>, grid, block, 0, a) : launch_pdl(ctx, short_conv_kernel<2, false>, grid, block, 0, a); break;
        case 3: le = f32 ? launch_pdl(ctx, short_conv_kernel<3, true>, grid, block, 0, a) : launch_pdl(ctx, short_conv_kernel<3, false>, grid, block, 0, a); break;
        case 4: le = f32 ? launch_pdl(ctx, short_conv_kernel<4, true>, grid, block, 0, a) : launch_pdl(ctx, short_conv_kernel<4, false>, grid, block, 0, a); break;
        default: le = f32 ? launch_pdl(ctx, short_conv_kernel<0, true>, grid, block, 0, a) : launch_pdl(ctx, short_conv_kernel<0, false>, grid, block, 0, a); break;
    }
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int selective_state_pad(int state) {
    for (int p = 4; p <= 256; p <<= 1)
        if (state <= p) return p;
    return 0;
}

int launch_selective_scan(b200_ctx* ctx, const SelectiveScanArgs& a, int E, int max_n, bool x_f32, bool out_f32) {
    (void)max_n;
    switch (a.state_pad) {
        case 4: return launch_scan_types<1, 4>(ctx, a, E, x_f32, out_f32);
        case 8: return launch_scan_types<2, 4>(ctx, a, E, x_f32, out_f32);
        case 16: return launch_scan_types<4, 4>(ctx, a, E, x_f32, out_f32);
        case 32: return launch_scan_types<8, 4>(ctx, a, E, x_f32, out_f32);
        case 64: return launch_scan_types<16, 4>(ctx, a, E, x_f32, out_f32);
        case 128: return launch_scan_types<16, 8>(ctx, a, E, x_f32, out_f32);
        case 256: return launch_scan_types<32, 8>(ctx, a, E, x_f32, out_f32);
        default: return B200_ERR_LIMIT;
    }
}

int delta_state_pad(int D) {
    for (int p = 32; p <= 256; p <<= 1)
        if (D <= p) return p;
    return 0;
}

namespace {
template <int V>
cudaError_t launch_delta_prep_v(b200_ctx* ctx, const DeltaArgs& a, dim3 grid) {
    switch (a.taps) {
        case 2: return launch_pdl(ctx, delta_prep_kernel<2, V>, grid, dim3(128), 0, a);
        case 3: return launch_pdl(ctx, delta_prep_kernel<3, V>, grid, dim3(128), 0, a);
        case 4: return launch_pdl(ctx, delta_prep_kernel<4, V>, grid, dim3(128), 0, a);
        default: return launch_pdl(ctx, delta_prep_kernel<0, V>, grid, dim3(128), 0, a);
    }
}
}  // namespace

int launch_delta_prep(b200_ctx* ctx, const DeltaArgs& a, int E, int max_n) {
    const dim3 grid(a.G, (max_n + 4 * kDeltaTok - 1) / (4 * kDeltaTok), E);
    cudaError_t le;
    if (a.Dl <= 32) le = launch_delta_prep_v<1>(ctx, a, grid);
    else if (a.Dl <= 64) le = launch_delta_prep_v<2>(ctx, a, grid);
    else if (a.Dl <= 128) le = launch_delta_prep_v<4>(ctx, a, grid);
    else le = launch_delta_prep_v<8>(ctx, a, grid);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

int launch_delta_scan(b200_ctx* ctx, const DeltaArgs& a, int E) {
    switch (delta_state_pad(a.D)) {
        case 32: return launch_delta_scan_l<2>(ctx, a, E);
        case 64: return launch_delta_scan_l<4>(ctx, a, E);
        case 128: return launch_delta_scan_l<8>(ctx, a, E);
        case 256: return launch_delta_scan_l<16>(ctx, a, E);
        default: return B200_ERR_LIMIT;
    }
}

int launch_delta_step(b200_ctx* ctx, const DeltaArgs& a, int E) {
    switch (delta_state_pad(a.D)) {
        case 32: return launch_delta_step_l<2>(ctx, a, E);
        case 64: return launch_delta_step_l<4>(ctx, a, E);
        case 128: return launch_delta_step_l<8>(ctx, a, E);
        case 256: return launch_delta_step_l<16>(ctx, a, E);
        default: return B200_ERR_LIMIT;
    }
}

int launch_min_gru(b200_ctx* ctx, const MinGruArgs& a, int E, bool f32) {
    const dim3 grid((a.width + 31) / 32, E);
    cudaError_t le = f32 ? launch_pdl(ctx, min_gru_kernel<true>, grid, dim3(kGruWarps * 32), 0, a)
                         : launch_pdl(ctx, min_gru_kernel<false>, grid, dim3(kGruWarps * 32), 0, a);
    ctx->launches++;
    B200_CUDA(ctx, le);
    return B200_OK;
}

}  // namespace b200
