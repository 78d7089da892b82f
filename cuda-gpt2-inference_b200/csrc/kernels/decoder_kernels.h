// Launchers of the kernels behind driver/decoder.cu (layered decoders with per-sequence state).
// As in kernels.h they validate nothing, enqueue on ctx->stream and bump ctx->launches once per
// kernel launch.
//
// A step's tokens are rows: the rows of one sequence are consecutive and described by a SeqDesc.
// Activations come in one of two element types: 16-bit (bf16 GEMM operands) or fp32 (the 32-bit
// arithmetic); `f32` selects the type of the buffers declared void*.  Every leading dimension is
// padded (pad_dim) and the padding holds zeros, so rows can be read in 16-byte pieces.
#pragma once
#include "kernels.h"

namespace b200 {

struct SeqDesc {
    int row0;  // first row of the step
    int n;     // tokens in this step
    int slot;  // where the sequence's cache and state live
    int pos0;  // position of its first token in this step
    int bank;  // short-convolution history to read (0 / 1); the other bank is written
    int kv0;   // latent attention: first row of the sequence's expanded keys and values; -1: the latents are attended to
    int lat0;  // ... and then the first of its rows among the step's queries that do so
    int pad;
};

// leading dimension of a matrix operand with n columns: whole 16-byte pieces, at least one 64-element K block
inline int pad_dim(int n) { return n < 64 ? 64 : (n + 7) & ~7; }

// ---- row-wise (rmsnorm.cu)
// Residual stream of M rows:  r = embed[tok] * scale (tok != null), or x, or x + branch with branch = rms(y) * wb (wb, y != null),
// or y * y_scale[row] (y != null; y_scale null: 1) + part_scale * sum of `top` rows of parts (part_of[row * top + j]; null: row * top + j);
// x_out = r (if not null);  h = rms(r) * w (if w) as bf16, fp32 or split rows (decoder_math.cuh).  rows != null: row i of the output
// is made from row rows[i] of the inputs.  C columns of Cp.  copies > 0 (bf16, fp32): row i of h also goes to rows copy_of[i * copies + j]
// of copy.  gate_w: gate_out[i] = sigmoid(h . gate_w).
struct ResidualNormArgs {
    const float* x; const float* y; const float* wb; const float* w;
    float* x_out; void* h;
    const int* tok; const void* embed; float embed_scale; int vocab;
    const int* rows;
    int M, C, Cp; float eps;
    const float* y_scale; const float* parts; const int* part_of; int top; float part_scale;
    void* copy; const int* copy_of; int copies;
    const float* gate_w; float* gate_out;
};
enum : int { H_BF16 = 0, H_F32 = 1, H_SPLIT = 2 };
int launch_residual_rms(b200_ctx* ctx, const ResidualNormArgs& a, int format);  // H_F32: the embedding table is fp32, else bf16
// out[r, h*Dv + d] = o / rms(o over the head) * w[d] * silu(gate) (plain_sigmoid: sigmoid(gate));  o, gate [M] rows with heads Dvl apart
int launch_gated_head_norm(b200_ctx* ctx, void* out, int ld_out, const float* o, int ld_o, const float* gate, int ld_gate,
                           const float* w, int M, int H, int Dv, int Dvl, float eps, bool f32, bool plain_sigmoid = false);
// dst[r, 0..n) = src[r, col0 ..]  (fp32 -> bf16 or fp32), columns n..ld_dst zero
int launch_slice(b200_ctx* ctx, void* dst, int ld_dst, const float* src, int ld_src, int n, int M, bool f32);

// ---- matrix products
enum : int { ACT_NONE = 0, ACT_GELU_TANH = 1, ACT_GELU_ERF = 2 };
// out[M,N] = act(inp[M,K] W[N,K]^T + bias) on the fp32 FMA pipe (no reduced precision anywhere); K, N multiples of 4
int launch_gemm_fp32(b200_ctx* ctx, float* out, const float* inp, const float* W, const float* bias, int M, int K, int N, int act,
                     const GemmGroups* groups = nullptr);

// Decode product (gemm_decode.cu): B <= 16 split rows x [B, K] against bf16 weights [N, K], + bias, then
//   columns below conv_n: short causal convolution with the history of the row's slot (+ conv_b) and silu; the new
//     history goes to the other bank
//   the others: act
// to out (fp32) and, as split rows, to split_out (all columns) or conv_out (the convolved ones, which then do not go to out).
// gate != GATE_NONE: W's rows come in blocks of 64, 32 gates and the 32 linear values that belong to them, and the output
// (split_out) has N / 2 columns.
// Table-routed experts (top > 0): input row b belongs to the `top` matrices that `route` gives it of the stack W [..][N, K],
// and its products with them are rows b * top + j of the output; pair_in: of the input too (else one row b meets
// them all).  A matrix is read once however many rows want it.  With shared.W a further matrix of its own
// height, width, input and output meets every row in the same launch.
enum : int { GATE_NONE = 0, GATE_GELU_TANH = 1, GATE_CLAMP = 2 };
constexpr int kMaxPairs = 256;  // (input row, expert) pairs
struct DecodeRoute { int matrices; uint16_t listed[kMaxPairs], expert[kMaxPairs]; };  // matrices that occur; the one of every pair
struct DecodeGemmShared { const uint8_t* x; const uint16_t* W; int N, K; float limit; float* out; int ldo; uint8_t* split_out; };
struct DecodeGemmArgs {
    const uint8_t* x;
    const uint16_t* W; const float* bias;
    int B, N, K, act;
    float* out; int ldo;
    uint8_t* split_out;   // [B] rows of N columns
    const SeqDesc* seqs; const float* conv_w; const float* conv_b; float* hist; int conv_n, taps, max_slots;
    uint8_t* conv_out;    // [B] rows of conv_n columns
    int gate; float limit;
    const DecodeRoute* route; int top, experts, pair_in;  // (route: read before the previous kernel has finished)
    DecodeGemmShared shared;
};
int launch_decode_gemm(b200_ctx* ctx, const DecodeGemmArgs& a);

// ---- experts (experts.cu)
struct MoeRoute { const int* table; int experts, top; int* place; int* blocks; DecodeRoute* decode; };  // table [vocab][top]
// decode: the routes of B tokens' pairs -> MoeRoute::decode
int launch_decode_routes(b200_ctx* ctx, const MoeRoute* routes, int n, const int* tok, int B);
// rows per run (GemmGroups::align) of P pairs
__host__ __device__ inline int moe_run_rows(int P, int experts, bool f32) { return f32 ? 64 : (P / 1024 >= experts ? 256 : 128); }
// routes: n of them in device memory
int launch_moe_route(b200_ctx* ctx, const MoeRoute* routes, int n, const int* tok, int M, bool f32, int max_experts);
// out[M,F] = act of in[M,2F], whose columns are blocks of 32 gates and their 32 linear values (fp32; F a multiple of 32)
int launch_gated_act(b200_ctx* ctx, float* out, const float* in, int M, int F, int gate, float limit);

// ---- recurrences (recurrent.cu)
// y = silu(causal depthwise convolution of columns [0, n) of x + bias); weights [taps][np]; history
// [2 banks][max_slots][taps - 1][np] fp32
struct ShortConvArgs {
    const float* x; int ldx;
    void* out; int ld_out;
    const float* w; const float* bias;
    float* hist;
    const SeqDesc* seqs;
    int np, taps, max_slots;  // np: channels rounded up to a multiple of 4 (weights zero beyond)
    int ch0;                  // first channel (a multiple of 4): the ones before are left alone
};
int launch_short_conv(b200_ctx* ctx, const ShortConvArgs& a, int E, int max_n, bool f32);

// Selective scan with a diagonal state per channel:
//   dt = softplus(dt_raw + dt_b);  S[c,:] = 2^(dt A2[c,:]) S[c,:] + dt x B;  y = (S C + D x) * silu(z)
// With Wdt (decode, one token per sequence) dt_raw is formed here: dt_raw[c] = Wdt[c,:] . bc[0..rank), and x
// and out are split rows.
struct SelectiveScanArgs {
    const void* x; int ldx;           // convolved input: bf16 (f32: fp32; decode: split rows of ldx columns)
    const float* dt; int lddt;        // dt_raw, null with Wdt
    const float* bc; int ldbc;        // per token: [dt: ..| B: at b_col | C: at c_col]
    int b_col, c_col;
    const float* z; int ldz;
    const float* A2;                  // [inner][state_pad]: -exp(A_log) * log2(e), zero beyond the state
    const float* dt_b; const float* D;
    float* S;                         // [slots][inner][state_pad]
    void* out; int ldo;
    const SeqDesc* seqs;
    int inner, state_pad;
    const uint16_t* Wdt; int rank, ld_wdt;
};
int selective_state_pad(int state);   // 0: unsupported
int launch_selective_scan(b200_ctx* ctx, const SelectiveScanArgs& a, int E, int max_n, bool x_f32, bool out_f32);

// Gated delta rule.  In a row head g's q lies at g*Dl, its k at k_col + g*Dl, head h's v at v_col + h*Dvl.
//   decay = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b)
// State [slots][H][Dv][Dpad] fp32.
//   prep   convolution + silu of raw's q and k columns -> unit vectors (q also times D^-1/2) in qkv, and coef
//          (the v columns are a plain short convolution)
//   scan   qkv, coef -> o in out [M, H*Dvl] fp32
//   step   one token per sequence, from the convolved columns (qkv, ld) to the normalised, gated output as split rows
//          of ldo columns
struct DeltaArgs {
    const float* qkv; int ld; int k_col, v_col;
    const float* raw; int ld_raw;
    float4* coef;           // [M][H] {decay, beta, k.q, -}
    const float* gates; int ldg; int a_col, b_col;  // columns of the projection holding a and b per head
    const float* negA;      // [H] -exp(A_log)
    const float* dt_bias;   // [H]
    float* S;
    float* out; int ldo;
    const SeqDesc* seqs;
    int H, G, D, Dl, Dv, Dvl;
    const float* conv_w; float* hist; int taps, np, max_slots;
    const float* norm_w; int gate_col; float eps;
    // Decay per key channel: exp(-exp(A_log) softplus(a + dt_bias)) with dt_bias [H][Dl] and a from a low-rank projection.
    //   decay: rows of ld_decay columns, head h's at h*Dl: a on entry of prep, the decay behind it
    //   step forms a, and the output gate (through a sigmoid), itself: w_low's row h*Dl + d meets columns low_col .. + low_a of the
    //   token's row, its row gate_row + h*Dvl + d columns low_a .. low_a + low_g of the same piece
    float* decay; int ld_decay;
    const uint16_t* w_low; int ld_low, low_col, low_a, low_g, gate_row;
};
int delta_state_pad(int D);  // 0: unsupported
int launch_delta_prep(b200_ctx* ctx, const DeltaArgs& a, int E, int max_n);
int launch_delta_scan(b200_ctx* ctx, const DeltaArgs& a, int E);
int launch_delta_step(b200_ctx* ctx, const DeltaArgs& a, int E);

// minGRU: z = sigmoid(zx[z_col ..]), u = zx[x_col ..], candidate = u + 1/2 (u >= 0) or sigmoid(u);
// S = (1 - z) S + z candidate;  out = S * silu(zx[g_col ..]) * out_scale
struct MinGruArgs {
    const float* zx; int ld; int z_col, x_col, g_col;
    float* S;  // [slots][width]
    void* out; int ldo;
    const SeqDesc* seqs;
    int width; float out_scale;
    int out_col;  // added to the column (the decode kernel, whose split rows cannot be offset by a pointer)
};
int launch_min_gru(b200_ctx* ctx, const MinGruArgs& a, int E, bool f32);

// ---- attention over a per-slot key/value cache (attention_cached.cu)
// Cache layout: K [slots][G][Tp][Dp], V [slots][G][Tp][Dvp], fp16 or fp32; Tp a multiple of 128.
struct CachedAttention {
    int H, G, D, Dv, Dp, Dvp, Tp;
    int q_col, k_col, v_col;     // columns of the projection; heads D / Dv apart
    int rot_dims;                // 0: no rotation
    const float2* rot;           // [Tp][rot_dims / 2] (cos, sin)
    const float* q_norm;         // weights of the per-head RMS norms of q and k (null: none)
    const float* k_norm;
    int v_norm;                  // values are divided by their root mean square
    float scale, eps;
    void* K; void* V;
    float out_scale;
    // > 0: K and V are not the cache but rows of ld_kv columns in which every head has its own Dp / Dvp columns (G = H); a
    // sequence's positions are the rows from its kv0 on (kv_rows in all)
    int ld_kv, kv_rows;
};  // (scores: (q . k) * scale)
inline int attention_pad(int d) { return d <= 64 ? 64 : (d + 63) & ~63; }
// norms and rotation of a step's q (-> q_out [M][H * Dp]) and k, v (-> cache)
int launch_attention_prep(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, void* q_out, const SeqDesc* seqs,
                          const int* row_seq, int M, bool f32);
// causal attention of a step's rows over positions 0 .. their own; out[row, h*Dv + d] (bf16 or fp32)
// pairs: (sequence, pair of query tiles) work list of the tensor-core kernel, most keys first
bool attention_cached_has_mma(const CachedAttention& c);
int launch_attention_cached_mma(b200_ctx* ctx, const CachedAttention& c, const void* q, void* out, int ldo, const SeqDesc* seqs,
                                const int2* pairs, int num_pairs, int M, int max_slots);
int launch_attention_cached_simt(b200_ctx* ctx, const CachedAttention& c, const void* q, void* out, int ldo, const SeqDesc* seqs,
                                 int E, int max_n, bool f32);
// One token per sequence: norms, rotation, cache append and attention in one kernel (fp16 cache; out: split rows of
// ldo columns); with gru.S also a minGRU step in further CTAs of the launch (gru.out: the same rows, out_col: its first column).
int launch_attention_cached_decode(b200_ctx* ctx, const CachedAttention& c, const float* proj, int ld, uint8_t* out, int ldo,
                                   const SeqDesc* seqs, int B, const MinGruArgs& gru);

// ---- latent attention (attention_latent.cu)
// Keys and values of all heads are linear in one latent per token, W_uk c and W_uv c, beside a rotated key part that the heads
// share.  The cache holds the latent and that part: rows [c: R | rotated: Dr | zeros up to Lp], [slots][Tp][Lp], fp16 or fp32.
// A sequence's step is computed in one of two ways (SeqDesc::kv0):
//   expanded   many tokens: keys and values of all positions are formed by one product over the cached rows, whose weight
//              passes the rotated part on, and attended to by the kernels of attention_cached.cu
//   latent     few tokens (16-bit arithmetic): the queries are taken into the latent's space, q W_uk, scored against the cached rows
//              themselves, and W_uv is applied to the weighted sum of latents
struct LatentAttention {
    int H, D, Dr, Dv, R;           // per head: D unrotated and Dr rotated dimensions, values of Dv
    int Lp, Tp, Dp, Dvp;           // Dp, Dvp: padded heads of the expanded keys and values
    int q_col, c_col;              // columns of the projection: heads D + Dr apart; latent, then rotated key part
    const float2* rot;             // [Tp][Dr / 2] (cos, sin); pairs are neighbouring dimensions
    const float* c_norm;
    float scale, eps;
    void* cache;
    const uint16_t* Wuk;           // [H * D][Rp] bf16, Rp = R rounded up to 8
    const uint16_t* Wuv;           // [H * Dv][Rp]
    int Rp;
};
int latent_row_pad(int r);  // Lp of rows of r values; 0: unsupported
// norm and rotation of the step's rows: -> cache, and for the expanded sequences -> lat (rows kv0 + position, Lp columns) and their
// queries -> q_out [M][H * Dp]
int launch_latent_prep(b200_ctx* ctx, const LatentAttention& c, const float* proj, int ld, void* q_out, void* lat, const SeqDesc* seqs, const int* row_seq,
                       int M, bool f32);
// cached rows of earlier steps of the expanded sequences -> lat
int launch_latent_gather(b200_ctx* ctx, const LatentAttention& c, void* lat, const SeqDesc* seqs, int E, int max_pos0, bool f32);
// queries of rows[0 .. n) (null: 0 .. n - 1) in the latent's space -> ql [n][H][Lp] fp16; append: the rows' latents go to the cache too (one
// token per sequence: row i is sequence i's)
int launch_latent_query(b200_ctx* ctx, const LatentAttention& c, const float* proj, int ld, void* ql, const SeqDesc* seqs, const int* row_seq,
                        const int* rows, int n, bool append);
// weighted sums of latents of (token, head) pairs over shares of the positions, their maxima and sums of weights; pairs: how many there is room for
struct LatentParts { float* o; float2* ml; long pairs; };
// attention of ql's n_rows rows (rows[i] of the step; null: i) over the cached latents, W_uv applied, for sequences list[0 .. n) (null:
// 0 .. n - 1) of at most max_n tokens that see at most max_keys keys.  out: bf16, or split rows, of ldo columns.  Two launches.
int launch_latent_attention(b200_ctx* ctx, const LatentAttention& c, const void* ql, const LatentParts& parts, void* out, int ldo, const SeqDesc* seqs,
                            const int* list, int n, const int* rows, int n_rows, int max_n, int max_keys, bool split_rows);

}  // namespace b200
