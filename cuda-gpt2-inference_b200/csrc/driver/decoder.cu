// Layered decoders: models whose configuration lists their layers, each with a mixer of some kind and a
// feed-forward, served from per-sequence slots that hold whatever the mixers remember (key/value or latent cache,
// recurrent state, convolution history).
//
//   configuration  ModelSpec, read from config.json; a Design (registry below) fixes what all models of an
//                  architecture share
//   weights        safetensors or single tensors -> concatenated, padded matrices on the device
//   slots          opened and closed by the caller or the generation loop; a slot carries one sequence's
//                  length and needs no clearing (a sequence at position 0 starts from zero state)
//   step           any number of tokens of any open sequences: the general path (prompts, portions), or, with one
//                  token for each of at most 16 sequences in 16-bit arithmetic, the fused decode path, replayed
//                  as a CUDA graph
//   generate       the scheduler: admits requests to slots, runs their prompts in portions, then decodes all
//                  active sequences together
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <deque>
#include <map>
#include <new>
#include <stdexcept>
#include <string>
#include <vector>
#include <cuda_fp16.h>
#include "../api/ctx.h"
#include "../kernels/decoder_kernels.h"
#include "json.h"
#include "weights.h"

using namespace b200;

namespace {

// ------------------------------------------------------------------ configuration
// What the models of one architecture have in common and config.json does not say.
struct Design {
    const char* name;
    int mlp_act;        // of a dense feed-forward: down(act(up)) ...
    int mlp_gate;       // ... or, not GATE_NONE, down(act(gate) * up)
    bool qk_norm;       // attention: per-head RMS norm of queries and keys, with weights
    bool value_norm;    // attention: values divided by their root mean square
    bool post_norm;     // an RMS norm behind every sublayer too
    float norm_offset;  // added to the stored weights of the norms in front of the sublayers and of the last one
    bool tied_head;     // the logits' matrix is the embedding table
};
const Design kDesigns[] = {
    {"Vunolorn", ACT_GELU_ERF, GATE_NONE, true, true, true, 0.f, false},
    {"Pumotar", ACT_NONE, GATE_GELU_TANH, false, false, false, 1.f, true},
};

enum MixerKind { MIX_MAMBA1, MIX_DELTA, MIX_PARALLEL, MIX_LATENT, MIX_CHANNEL_DELTA };
enum MlpKind { MLP_NONE, MLP_DENSE, MLP_EXPERTS };

struct AttentionSpec { int heads, kv_heads, dim, vdim, rot_dims; double rot_base; float scale; };
struct LayerSpec {
    MixerKind kind;
    int conv = 0, dt_rank = 0, inner = 0, state = 0;           // mamba1 (and conv of delta)
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;            // delta, channel_delta; latent_attention (no kv_heads)
    int kv_rank = 0, rot_dim = 0; double rot_base = 0; float scale = 0.f;  // latent_attention
    AttentionSpec att{};                                       // parallel, left
    int gru_width = 0;                                         // parallel, right
    float left_scale = 1.f, right_scale = 1.f;
    MlpKind mlp = MLP_NONE;
    int ff = 0;                                                // dense: its width; experts: of one of them
    int experts = 0, top = 0, shared_ff = 0;                   // (shared_ff 0: no shared expert)
    float limit = 0.f, shared_limit = 0.f;
};
struct ModelSpec {
    const Design* design = nullptr;
    int vocab = 0, width = 0;
    float embed_scale = 1.f, eps = 1e-5f;
    std::vector<LayerSpec> layers;
    std::vector<int> order;  // the layers in the order in which they run; one that is looped occurs several times
};

void positive(int v, const char* what) { if (v < 1) throw std::runtime_error(std::string("config: '") + what + "' must be positive"); }
void head_groups(int heads, int kv_heads) {
    positive(heads, "heads");
    positive(kv_heads, "kv_heads");
    if (heads % kv_heads) throw std::runtime_error("config: 'heads' must be a multiple of 'kv_heads'");
}

AttentionSpec parse_attention(const Json& m) {
    AttentionSpec a{};
    a.heads = m.integer("heads"); a.kv_heads = m.integer("kv_heads");
    head_groups(a.heads, a.kv_heads);
    a.dim = m.integer("dim"); a.vdim = m.integer("vdim");
    positive(a.dim, "dim"); positive(a.vdim, "vdim");
    if (a.dim > 256 || a.vdim > 256) throw std::runtime_error("config: attention heads of more than 256 dimensions");
    a.scale = (float)m.number("scale");
    if (!(a.scale > 0.f)) throw std::runtime_error("config: attention 'scale' must be positive");
    const Json& r = m.at("rot");
    a.rot_dims = r.integer("dims");
    a.rot_base = r.number("base");
    if (a.rot_dims < 0 || a.rot_dims % 2 || a.rot_dims > a.dim) throw std::runtime_error("config: rot.dims must be even and at most dim");
    return a;
}

void parse_delta(const Json& m, LayerSpec& l) {
    l.conv = m.integer("conv"); l.heads = m.integer("heads"); l.kv_heads = m.integer("kv_heads");
    l.dim = m.integer("dim"); l.vdim = m.integer("vdim");
    positive(l.conv, "conv"); head_groups(l.heads, l.kv_heads); positive(l.dim, "dim"); positive(l.vdim, "vdim");
    if (!delta_state_pad(l.dim)) throw std::runtime_error("config: delta 'dim' beyond 256");
    if (l.vdim > 2048) throw std::runtime_error("config: delta 'vdim' beyond 2048");
}

// mixer registry: config name -> reader of its sizes
struct MixerType {
    const char* name;
    void (*parse)(const Json&, LayerSpec&);
};
const MixerType kMixers[] = {
    {"mamba1", [](const Json& m, LayerSpec& l) {
         l.kind = MIX_MAMBA1;
         l.conv = m.integer("conv"); l.dt_rank = m.integer("dt_rank"); l.inner = m.integer("inner"); l.state = m.integer("state");
         positive(l.conv, "conv"); positive(l.dt_rank, "dt_rank"); positive(l.inner, "inner"); positive(l.state, "state");
         if (!selective_state_pad(l.state)) throw std::runtime_error("config: mamba1 'state' beyond 256");
     }},
    {"delta", [](const Json& m, LayerSpec& l) { l.kind = MIX_DELTA; parse_delta(m, l); }},
    {"channel_delta", [](const Json& m, LayerSpec& l) { l.kind = MIX_CHANNEL_DELTA; parse_delta(m, l); }},
    {"latent_attention", [](const Json& m, LayerSpec& l) {
         l.kind = MIX_LATENT;
         l.heads = m.integer("heads"); l.dim = m.integer("dim"); l.vdim = m.integer("vdim");
         l.kv_rank = m.integer("kv_rank"); l.rot_dim = m.integer("rot_dim");
         positive(l.heads, "heads"); positive(l.dim, "dim"); positive(l.vdim, "vdim"); positive(l.kv_rank, "kv_rank"); positive(l.rot_dim, "rot_dim");
         l.scale = (float)m.number("scale");
         if (!(l.scale > 0.f)) throw std::runtime_error("config: attention 'scale' must be positive");
         const Json& r = m.at("rot");
         l.rot_base = r.number("base");
         if (r.integer("dims") != l.rot_dim || l.rot_dim % 2) throw std::runtime_error("config: rot.dims must be rot_dim, and even");
         if (l.dim + l.rot_dim > 256 || l.vdim > 256) throw std::runtime_error("config: attention heads of more than 256 dimensions");
         if (l.kv_rank > 512 || !latent_row_pad(l.kv_rank + l.rot_dim)) throw std::runtime_error("config: 'kv_rank' beyond 512, or with rot_dim beyond 640");
     }},
    {"parallel", [](const Json& m, LayerSpec& l) {
         l.kind = MIX_PARALLEL;
         l.att = parse_attention(m.at("left"));
         l.gru_width = m.at("right").integer("width");
         positive(l.gru_width, "width");
         l.left_scale = (float)m.number("left_scale");
         l.right_scale = (float)m.number("right_scale");
     }},
};

// feed-forward registry
struct MlpType {
    const char* name;
    void (*parse)(const Json&, LayerSpec&);
};
float parse_limit(const Json& m) {
    const float v = (float)m.number("limit");
    if (!(v > 0.f)) throw std::runtime_error("config: 'limit' must be positive");
    return v;
}
const MlpType kMlps[] = {
    {"dense", [](const Json& m, LayerSpec& l) {
         l.mlp = MLP_DENSE;
         l.ff = m.integer("ff");
         positive(l.ff, "ff");
     }},
    {"moe", [](const Json& m, LayerSpec& l) {
         l.mlp = MLP_EXPERTS;
         const Json &e = m.at("expert"), &r = m.at("router");
         l.ff = e.integer("ff"); l.limit = parse_limit(e);
         l.experts = r.integer("experts"); l.top = r.integer("top");
         positive(l.ff, "ff"); positive(l.experts, "experts"); positive(l.top, "top");
         if (l.top > l.experts) throw std::runtime_error("config: router.top beyond router.experts");
         if (l.top > 16 || l.experts > 8192) throw std::runtime_error("config: router.top beyond 16 or router.experts beyond 8192");
         if (m.has("shared") && !m.at("shared").is_null()) {
             const Json& s = m.at("shared");
             l.shared_ff = s.integer("ff"); l.shared_limit = parse_limit(s);
             positive(l.shared_ff, "ff");
         }
     }},
};

ModelSpec parse_config(const char* text) {
    const Json j = Json::parse(text, text + strlen(text));
    ModelSpec s;
    const std::string& arch = j.string("architecture");
    for (const Design& d : kDesigns)
        if (arch == d.name) s.design = &d;
    if (!s.design) throw std::runtime_error("config: unknown architecture '" + arch + "'");
    s.vocab = j.integer("vocab"); s.width = j.integer("width");
    positive(s.vocab, "vocab"); positive(s.width, "width");
    s.embed_scale = (float)j.at("embedding").number("scale");
    s.eps = (float)j.at("norm").number("eps");
    const Json& layers = j.at("layers");
    if (layers.kind != Json::ARR || layers.arr.empty()) throw std::runtime_error("config: 'layers' must be a list");
    for (const Json& lj : layers.arr) {
        LayerSpec l;
        const std::string& type = lj.string("type");
        const MixerType* mt = nullptr;
        for (const MixerType& t : kMixers)
            if (type == t.name) mt = &t;
        if (!mt) throw std::runtime_error("config: unknown mixer '" + type + "'");
        mt->parse(lj.at("mixer"), l);
        const Json& mlp = lj.at("mlp");
        if (!mlp.is_null()) {
            const std::string& kind = mlp.string("kind");
            const MlpType* ft = nullptr;
            for (const MlpType& t : kMlps)
                if (kind == t.name) ft = &t;
            if (!ft) throw std::runtime_error("config: unknown feed-forward '" + kind + "'");
            ft->parse(mlp, l);
        }
        s.layers.push_back(l);
    }
    const int n = (int)s.layers.size();
    int start = 0, stop = 0, times = 1;
    if (j.has("loop") && !j.at("loop").is_null()) {
        const Json& lp = j.at("loop");
        start = lp.integer("start"); stop = lp.integer("stop"); times = lp.integer("times");
        if (start < 0 || stop < start || stop > n || times < 1) throw std::runtime_error("config: 'loop' must name layers start .. stop - 1 and run them at least once");
    }
    for (int i = 0; i < start; ++i) s.order.push_back(i);
    for (int t = 0; t < times; ++t)
        for (int i = start; i < stop; ++i) s.order.push_back(i);
    for (int i = stop; i < n; ++i) s.order.push_back(i);
    return s;
}

// ------------------------------------------------------------------ the model on the device
// A matrix [N, K] in the model's element type; N and K are padded with zeros.
struct Matrix { void* w = nullptr; int N = 0, K = 0; float* bias = nullptr; };

// Gated feed-forwards: up holds gates and linear parts, blocks of 32 rows of either in turn, [2 F].  Experts: up and down are
// stacks of one matrix per expert (N, K of one).
struct Mlp {
    Matrix up, down, shared_up, shared_down;
    int gate = GATE_NONE;
    float* shared_gate = nullptr;
    int* table = nullptr;
    MoeRoute route{};  // of a step's pairs
};
// a layer run: the passes of a looped layer share the weights, each has its own state
struct Layer {
    const LayerSpec* spec = nullptr;
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    Matrix in, o;            // the mixer's joint input projection and its output projection
    Mlp mlp;
    // mamba1: in = [x: np | z: np]; xp = [dt: rank_p | B: sp | C: sp]
    Matrix xp, dt;
    float *conv_w = nullptr, *conv_b = nullptr, *A2 = nullptr, *dt_b = nullptr, *D = nullptr;
    int np = 0, sp = 0, rank_p = 0;
    // delta: in = [q: G*Dl | k: G*Dl | v: H*Dvl | gate: H*Dvl | a: H | b: H]
    // channel_delta: in = [q | k | v | a1: low_a | g1: low_g | b: H], low = a2 and g2 side by side (each zero on the other's columns)
    Matrix low;
    int low_col = 0, low_a = 0, low_g = 0, gate_row = 0;
    float *negA = nullptr, *dt_bias = nullptr, *head_norm = nullptr;
    int Dl = 0, Dvl = 0, k_col = 0, v_col = 0, gate_col = 0, a_col = 0, b_col = 0;
    // parallel: in = [q | k | v | z | x | g], o over [attention: att_p | minGRU]
    CachedAttention att{};
    int z_col = 0, x_col = 0, g_col = 0, att_p = 0;
    // latent_attention: in = [q | dkv]; kv: a cached row -> its expanded keys and values, which flat addresses
    LatentAttention lat{};
    CachedAttention flat{};
    Matrix kv;
    // what the slots hold
    float *hist = nullptr, *S = nullptr;
};

struct Slot { bool open = false; int len = 0, bank = 0; };

int round4(int n) { return (n + 3) & ~3; }
int round8(int n) { return (n + 7) & ~7; }
int gate_pad(int F) { return F < 64 ? 64 : (F + 31) & ~31; }  // columns of a gated feed-forward of width F

}  // namespace

struct b200_decoder {
    b200_ctx* ctx = nullptr;
    ModelSpec spec;
    bool f32 = false;
    int max_slots = 0, max_seq = 0, max_rows = 0, Tp = 0;
    int C = 0, Cp = 0, Vp = 0;
    bool ready = false;
    bool use_graph = true;
    TensorStore* store = nullptr;
    std::vector<void*> owned;             // every device allocation
    std::vector<Layer> layers;            // in the order in which they run
    void* embed = nullptr;
    float* final_norm = nullptr;
    Matrix head;
    std::map<std::pair<int, double>, float2*> rot_tables;
    std::vector<Slot> slots;
    // activations of the general path
    float *x = nullptr, *proj = nullptr, *y = nullptr, *aux = nullptr, *wide = nullptr;
    void *h = nullptr, *conv = nullptr, *mix = nullptr, *q = nullptr, *low = nullptr;
    float *gates = nullptr;                          // low-rank decays and output gates
    void *ql = nullptr, *lat = nullptr, *kv = nullptr;  // latent queries; latents and expanded keys and values of the step (grown on demand)
    LatentParts lat_parts{};  // (pairs: set per layer)
    long lat_rows_room = 0;
    int kv_rows = 0, expand_from = 1;                // expand_from: tokens from which a sequence's step is expanded
    void *pair_h = nullptr, *pair_mix = nullptr;     // rows of (token, expert) pairs: input, activations, outputs
    float *pair_y = nullptr, *raw = nullptr, *shared_gate = nullptr;
    MoeRoute* routes = nullptr;                      // of the layers with experts
    int num_routes = 0, max_experts = 0;
    float* logits = nullptr;
    int logits_rows = 0;
    // ... and of the decode path (16 rows: fp32, or split rows of the same size)
    float *dx = nullptr, *dproj = nullptr, *dy = nullptr, *daux = nullptr, *dlogits = nullptr;
    void *dh = nullptr, *dmix = nullptr, *dconv = nullptr, *dql = nullptr, *dpair_mix = nullptr;
    float *dpair_y = nullptr, *dshared_gate = nullptr;
    // step descriptors: a ring of pinned buffers, one device buffer per path
    static constexpr int kRing = 8;
    int* pinned[kRing] = {};
    cudaEvent_t ring_ev[kRing] = {};
    int ring = 0;
    size_t desc_ints = 0;
    int* desc = nullptr;
    SeqDesc* dseqs = nullptr;   // decode path: [16] descriptors, then 16 token ids
    int* dtokens = nullptr;
    std::map<int, cudaGraphExec_t> graphs;    // decode path, by B
    std::map<int, uint64_t> graph_launches;
    int* gen_log = nullptr;
    size_t gen_log_ints = 0;
    // per-operator timing (b200_decoder_set_profile): one event pair per launch
    bool profile = false;
    std::vector<cudaEvent_t> ev_pool;
    std::vector<const char*> ev_name;
};

namespace {

size_t elem(const b200_decoder* m) { return m->f32 ? 4 : 2; }

void* device_zeros(b200_decoder* m, size_t bytes) {
    void* p = nullptr;
    if (bytes == 0) bytes = 16;
    cudaError_t e = cudaMalloc(&p, bytes);
    if (e != cudaSuccess) throw std::runtime_error(std::string("cudaMalloc: ") + cudaGetErrorString(e));
    m->owned.push_back(p);
    e = cudaMemset(p, 0, bytes);
    if (e != cudaSuccess) throw std::runtime_error(std::string("cudaMemset: ") + cudaGetErrorString(e));
    return p;
}
void* upload(b200_decoder* m, const void* src, size_t bytes) {
    void* p = device_zeros(m, bytes);
    const cudaError_t e = cudaMemcpy(p, src, bytes, cudaMemcpyHostToDevice);
    if (e != cudaSuccess) throw std::runtime_error(std::string("cudaMemcpy: ") + cudaGetErrorString(e));
    return p;
}

// ------------------------------------------------------------------ weights
// Assembles a padded matrix from blocks of tensors, then uploads it in the model's element type.
class MatrixBuilder {
   public:
    // fp16: of a 16-bit model, elements in fp16 instead of bf16
    MatrixBuilder(b200_decoder* m, size_t N, int K, bool fp16 = false) : m_(m), N_(N), K_(K), fp16_(fp16) {
        if (m->f32) f_.assign((size_t)N * K, 0.f);
        else h_.assign((size_t)N * K, 0);
    }
    // rows `rows` of t (columns [0, cols)) to (row0, col0), times scale
    void put(const HostTensor& t, int src_row0, int rows, int cols, size_t row0, int col0) {
        for (int r = 0; r < rows; ++r) {
            const size_t s = (size_t)(src_row0 + r) * cols, d = (size_t)(row0 + r) * K_ + col0;
            if (m_->f32) for (int c = 0; c < cols; ++c) f_[d + c] = t.value(s + c);
            else if (fp16_) for (int c = 0; c < cols; ++c) h_[d + c] = half_bits(t.value(s + c));
            else if (t.type == TensorType::F32) for (int c = 0; c < cols; ++c) h_[d + c] = bf16_bits(t.value(s + c));
            else memcpy(&h_[d], t.data + 2 * s, (size_t)cols * 2);
        }
    }
    void one(size_t row, int col) {
        if (m_->f32) f_[row * K_ + col] = 1.f;
        else h_[row * K_ + col] = fp16_ ? half_bits(1.f) : bf16_bits(1.f);
    }
    // gates and linear parts [F, cols], in blocks of 32 rows of either, from row0 on
    void put_gated(const HostTensor& gate, const HostTensor& up, int F, int cols, size_t row0) {
        for (int f = 0; f < F; f += 32) {
            const int n = F - f < 32 ? F - f : 32;
            put(gate, f, n, cols, row0 + 2 * f, 0);
            put(up, f, n, cols, row0 + 2 * f + 32, 0);
        }
    }
    // parts: how many matrices are stacked
    Matrix build(int parts = 1) {
        Matrix x;
        x.N = (int)(N_ / parts); x.K = K_;
        x.w = m_->f32 ? upload(m_, f_.data(), f_.size() * 4) : upload(m_, h_.data(), h_.size() * 2);
        return x;
    }

   private:
    static uint16_t half_bits(float v) { const __half h = __float2half_rn(v); uint16_t u; memcpy(&u, &h, 2); return u; }
    b200_decoder* m_;
    size_t N_;
    int K_;
    bool fp16_;
    std::vector<float> f_;
    std::vector<uint16_t> h_;
};

float* vector_f32(b200_decoder* m, const HostTensor& t, size_t padded, float offset = 0.f) {
    std::vector<float> v(padded, 0.f);
    for (size_t i = 0; i < t.count(); ++i) v[i] = t.value(i) + offset;
    return static_cast<float*>(upload(m, v.data(), padded * 4));
}

float2* rotation_table(b200_decoder* m, int dims, double base) {
    const auto key = std::make_pair(dims, base);
    auto it = m->rot_tables.find(key);
    if (it != m->rot_tables.end()) return it->second;
    const int half = dims / 2;
    std::vector<float2> t((size_t)m->Tp * half);
    for (int i = 0; i < half; ++i) {
        const double f = pow(base, -2.0 * i / dims);
        for (int p = 0; p < m->Tp; ++p) t[(size_t)p * half + i] = make_float2((float)cos(p * f), (float)sin(p * f));
    }
    return m->rot_tables[key] = static_cast<float2*>(upload(m, t.data(), t.size() * sizeof(float2)));
}

// convolution weights [channels, taps] -> [taps][np], channel c of the tensor to channel dst(c)
void put_taps(std::vector<float>& w, int np, const HostTensor& t, int channels, int taps, int head, int head_l, int base) {
    for (int c = 0; c < channels; ++c) {
        const int d = base + c / head * head_l + c % head;
        for (int j = 0; j < taps; ++j) w[(size_t)j * np + d] = t.value((size_t)c * taps + j);
    }
}

void load_mamba1(b200_decoder* m, Layer& L, const std::string& p) {
    const LayerSpec& s = *L.spec;
    const TensorStore& w = *m->store;
    const int C = m->C, n = s.inner;
    L.np = pad_dim(n); L.sp = selective_state_pad(s.state); L.rank_p = pad_dim(s.dt_rank);
    {
        const HostTensor& t = w.get(p + ".in", {2L * n, C});
        MatrixBuilder b(m, 2 * L.np, m->Cp);
        b.put(t, 0, n, C, 0, 0);
        b.put(t, n, n, C, L.np, 0);
        L.in = b.build();
    }
    {
        const HostTensor& t = w.get(p + ".x", {(long)s.dt_rank + 2L * s.state, n});
        MatrixBuilder b(m, pad_dim(L.rank_p + 2 * L.sp), L.np);
        b.put(t, 0, s.dt_rank, n, 0, 0);
        b.put(t, s.dt_rank, s.state, n, L.rank_p, 0);
        b.put(t, s.dt_rank + s.state, s.state, n, L.rank_p + L.sp, 0);
        L.xp = b.build();
    }
    {
        MatrixBuilder b(m, L.np, L.rank_p);
        b.put(w.get(p + ".dt", {n, s.dt_rank}), 0, n, s.dt_rank, 0, 0);
        L.dt = b.build();
    }
    {
        MatrixBuilder b(m, m->Cp, L.np);
        b.put(w.get(p + ".o", {C, n}), 0, C, n, 0, 0);
        L.o = b.build();
    }
    std::vector<float> taps((size_t)s.conv * L.np, 0.f);
    put_taps(taps, L.np, w.get(p + ".conv", {n, s.conv}), n, s.conv, n, n, 0);
    L.conv_w = static_cast<float*>(upload(m, taps.data(), taps.size() * 4));
    L.conv_b = vector_f32(m, w.get(p + ".conv.b", {n}), L.np);
    L.dt_b = vector_f32(m, w.get(p + ".dt.b", {n}), L.np);
    L.D = vector_f32(m, w.get(p + ".D", {n}), L.np);
    const HostTensor& a = w.get(p + ".A_log", {n, s.state});
    std::vector<float> A2((size_t)n * L.sp, 0.f);  // exponents for base 2
    for (int c = 0; c < n; ++c)
        for (int k = 0; k < s.state; ++k) A2[(size_t)c * L.sp + k] = (float)(-exp((double)a.value((size_t)c * s.state + k)) * 1.4426950408889634);
    L.A2 = static_cast<float*>(upload(m, A2.data(), A2.size() * 4));
}

void load_delta(b200_decoder* m, Layer& L, const std::string& p) {
    const LayerSpec& s = *L.spec;
    const TensorStore& w = *m->store;
    const int C = m->C, H = s.heads, G = s.kv_heads, D = s.dim, Dv = s.vdim;
    L.Dl = round4(D); L.Dvl = round4(Dv);
    L.k_col = G * L.Dl; L.v_col = 2 * G * L.Dl;
    L.np = L.v_col + H * L.Dvl;  // the convolved columns
    const bool channel = s.kind == MIX_CHANNEL_DELTA;
    int ra = 0, rg = 0;
    if (channel) {
        ra = w.rows(p + ".a1"); rg = w.rows(p + ".g1");
        L.low_a = round8(ra); L.low_g = round8(rg);
        L.low_col = round8(L.np); L.b_col = L.low_col + L.low_a + L.low_g;
    } else {
        L.gate_col = L.np; L.a_col = L.gate_col + H * L.Dvl; L.b_col = L.a_col + H;
    }
    MatrixBuilder b(m, pad_dim(L.b_col + H), m->Cp);
    std::vector<float> taps((size_t)s.conv * L.np, 0.f);
    const struct { const char* n; int heads, dim, dim_l, col; } parts[] = {{".q", G, D, L.Dl, 0}, {".k", G, D, L.Dl, L.k_col}, {".v", H, Dv, L.Dvl, L.v_col}};
    for (const auto& a : parts) {
        const HostTensor& t = w.get(p + a.n, {(long)a.heads * a.dim, C});
        for (int h = 0; h < a.heads; ++h) b.put(t, h * a.dim, a.dim, C, a.col + h * a.dim_l, 0);
        put_taps(taps, L.np, w.get(p + a.n + ".conv", {(long)a.heads * a.dim, s.conv}), a.heads * a.dim, s.conv, a.dim, a.dim_l, a.col);
    }
    if (channel) {
        b.put(w.get(p + ".a1", {ra, C}), 0, ra, C, L.low_col, 0);
        b.put(w.get(p + ".g1", {rg, C}), 0, rg, C, L.low_col + L.low_a, 0);
        L.gate_row = round8(H * L.Dl);
        MatrixBuilder low(m, pad_dim(L.gate_row + H * L.Dvl), pad_dim(L.low_a + L.low_g));
        const HostTensor &a2 = w.get(p + ".a2", {(long)H * D, ra}), &g2 = w.get(p + ".g2", {(long)H * Dv, rg});
        for (int h = 0; h < H; ++h) {
            low.put(a2, h * D, D, ra, h * L.Dl, 0);
            low.put(g2, h * Dv, Dv, rg, L.gate_row + h * L.Dvl, L.low_a);
        }
        L.low = low.build();
    } else {
        const HostTensor& g = w.get(p + ".g", {(long)H * Dv, C});
        for (int h = 0; h < H; ++h) b.put(g, h * Dv, Dv, C, L.gate_col + h * L.Dvl, 0);
        b.put(w.get(p + ".a", {H, C}), 0, H, C, L.a_col, 0);
    }
    b.put(w.get(p + ".b", {H, C}), 0, H, C, L.b_col, 0);
    L.in = b.build();
    MatrixBuilder o(m, m->Cp, pad_dim(H * Dv));
    o.put(w.get(p + ".o", {C, (long)H * Dv}), 0, C, H * Dv, 0, 0);
    L.o = o.build();
    L.conv_w = static_cast<float*>(upload(m, taps.data(), taps.size() * 4));
    const HostTensor& a = w.get(p + ".A_log", {H});
    std::vector<float> negA(H);
    for (int h = 0; h < H; ++h) negA[h] = (float)-exp((double)a.value(h));
    L.negA = static_cast<float*>(upload(m, negA.data(), negA.size() * 4));
    if (channel) {
        const HostTensor& t = w.get(p + ".dt_bias", {(long)H * D});
        std::vector<float> bias((size_t)H * L.Dl, 0.f);
        for (int h = 0; h < H; ++h)
            for (int d = 0; d < D; ++d) bias[(size_t)h * L.Dl + d] = t.value((size_t)h * D + d);
        L.dt_bias = static_cast<float*>(upload(m, bias.data(), bias.size() * 4));
    } else L.dt_bias = vector_f32(m, w.get(p + ".dt_bias", {H}), H);
    L.head_norm = vector_f32(m, w.get(p + ".norm", {Dv}), Dv);
}

void load_latent(b200_decoder* m, Layer& L, const std::string& p) {
    const LayerSpec& s = *L.spec;
    const TensorStore& w = *m->store;
    const int C = m->C, H = s.heads, D = s.dim, Dr = s.rot_dim, Dv = s.vdim, R = s.kv_rank;
    LatentAttention& c = L.lat;
    c.H = H; c.D = D; c.Dr = Dr; c.Dv = Dv; c.R = R;
    c.Lp = latent_row_pad(R + Dr); c.Tp = m->Tp; c.Dp = attention_pad(D + Dr); c.Dvp = attention_pad(Dv); c.Rp = round8(R);
    c.q_col = 0; c.c_col = round8(H * (D + Dr));
    c.rot = rotation_table(m, Dr, s.rot_base);
    c.scale = s.scale; c.eps = m->spec.eps;
    MatrixBuilder b(m, pad_dim(c.c_col + R + Dr), m->Cp);
    b.put(w.get(p + ".q", {(long)H * (D + Dr), C}), 0, H * (D + Dr), C, 0, 0);
    b.put(w.get(p + ".dkv", {(long)R + Dr, C}), 0, R + Dr, C, c.c_col, 0);
    L.in = b.build();
    c.c_norm = vector_f32(m, w.get(p + ".dkv.norm", {R}), R);
    const HostTensor &uk = w.get(p + ".uk", {(long)H * D, R}), &uv = w.get(p + ".uv", {(long)H * Dv, R});
    // expanded: per head [W_uk c | rotated part, passed on | zeros], then all heads' [W_uv c | zeros]
    MatrixBuilder kv(m, (size_t)H * (c.Dp + c.Dvp), c.Lp, true);
    for (int h = 0; h < H; ++h) {
        kv.put(uk, h * D, D, R, (size_t)h * c.Dp, 0);
        for (int j = 0; j < Dr; ++j) kv.one((size_t)h * c.Dp + D + j, R + j);
        kv.put(uv, h * Dv, Dv, R, (size_t)H * c.Dp + h * c.Dvp, 0);
    }
    L.kv = kv.build();
    CachedAttention& f = L.flat;
    f.H = f.G = H; f.D = D + Dr; f.Dv = Dv; f.Dp = c.Dp; f.Dvp = c.Dvp; f.Tp = m->Tp;
    f.scale = s.scale; f.eps = m->spec.eps; f.out_scale = 1.f; f.ld_kv = L.kv.N;
    if (!m->f32) {
        MatrixBuilder k(m, (size_t)H * D, c.Rp), v(m, (size_t)H * Dv, c.Rp);
        k.put(uk, 0, H * D, R, 0, 0);
        v.put(uv, 0, H * Dv, R, 0, 0);
        c.Wuk = static_cast<const uint16_t*>(k.build().w);
        c.Wuv = static_cast<const uint16_t*>(v.build().w);
    }
    MatrixBuilder o(m, m->Cp, pad_dim(H * Dv));
    o.put(w.get(p + ".o", {C, (long)H * Dv}), 0, C, H * Dv, 0, 0);
    L.o = o.build();
}

// what every slot holds of a layer run
void allocate_state(b200_decoder* m, Layer& L) {
    const LayerSpec& s = *L.spec;
    const size_t slots = m->max_slots;
    auto floats = [&](size_t n) { return static_cast<float*>(device_zeros(m, n * 4)); };
    switch (s.kind) {
        case MIX_MAMBA1:
            L.hist = floats(2 * slots * (s.conv - 1) * L.np);
            L.S = floats(slots * s.inner * L.sp);
            break;
        case MIX_DELTA:
        case MIX_CHANNEL_DELTA:
            L.hist = floats(2 * slots * (s.conv - 1) * L.np);
            L.S = floats(slots * s.heads * s.vdim * delta_state_pad(s.dim));
            break;
        case MIX_PARALLEL:
            L.att.K = device_zeros(m, slots * L.att.G * L.att.Tp * L.att.Dp * elem(m));
            L.att.V = device_zeros(m, slots * L.att.G * L.att.Tp * L.att.Dvp * elem(m));
            L.S = floats(slots * s.gru_width);
            break;
        case MIX_LATENT:
            L.lat.cache = device_zeros(m, slots * L.lat.Tp * L.lat.Lp * elem(m));
            break;
    }
}

void load_parallel(b200_decoder* m, Layer& L, const std::string& p) {
    const LayerSpec& s = *L.spec;
    const AttentionSpec& a = s.att;
    const TensorStore& w = *m->store;
    const int C = m->C, W = s.gru_width;
    const std::string l = p + ".left", r = p + ".right";
    CachedAttention& c = L.att;
    c.H = a.heads; c.G = a.kv_heads; c.D = a.dim; c.Dv = a.vdim;
    c.Dp = attention_pad(a.dim); c.Dvp = attention_pad(a.vdim); c.Tp = m->Tp;
    c.q_col = 0; c.k_col = a.heads * a.dim; c.v_col = c.k_col + a.kv_heads * a.dim;
    L.z_col = (c.v_col + a.kv_heads * a.vdim + 7) & ~7;
    L.x_col = L.z_col + ((W + 7) & ~7);
    L.g_col = L.x_col + ((W + 7) & ~7);
    const int N = pad_dim(L.g_col + W);
    MatrixBuilder b(m, N, m->Cp);
    b.put(w.get(l + ".q", {(long)a.heads * a.dim, C}), 0, a.heads * a.dim, C, c.q_col, 0);
    b.put(w.get(l + ".k", {(long)a.kv_heads * a.dim, C}), 0, a.kv_heads * a.dim, C, c.k_col, 0);
    b.put(w.get(l + ".v", {(long)a.kv_heads * a.vdim, C}), 0, a.kv_heads * a.vdim, C, c.v_col, 0);
    b.put(w.get(r + ".z", {W, C}), 0, W, C, L.z_col, 0);
    b.put(w.get(r + ".x", {W, C}), 0, W, C, L.x_col, 0);
    b.put(w.get(r + ".g", {W, C}), 0, W, C, L.g_col, 0);
    L.in = b.build();
    std::vector<float> bias(N, 0.f);
    const HostTensor &zb = w.get(r + ".z.b", {W}), &xb = w.get(r + ".x.b", {W});
    for (int i = 0; i < W; ++i) { bias[L.z_col + i] = zb.value(i); bias[L.x_col + i] = xb.value(i); }
    L.in.bias = static_cast<float*>(upload(m, bias.data(), bias.size() * 4));
    // one output projection over both mixers; their scales are applied to its input
    L.att_p = (a.heads * a.vdim + 7) & ~7;
    MatrixBuilder o(m, m->Cp, pad_dim(L.att_p + W));
    o.put(w.get(l + ".o", {C, (long)a.heads * a.vdim}), 0, C, a.heads * a.vdim, 0, 0);
    o.put(w.get(r + ".o", {C, W}), 0, C, W, 0, L.att_p);
    L.o = o.build();
    c.rot_dims = a.rot_dims;
    c.rot = a.rot_dims > 0 ? rotation_table(m, a.rot_dims, a.rot_base) : nullptr;
    if (m->spec.design->qk_norm) {
        c.q_norm = vector_f32(m, w.get(l + ".q.norm", {a.dim}), a.dim);
        c.k_norm = vector_f32(m, w.get(l + ".k.norm", {a.dim}), a.dim);
    }
    c.v_norm = m->spec.design->value_norm;
    c.scale = a.scale; c.eps = m->spec.eps; c.out_scale = s.left_scale;
}

Matrix gated_up(b200_decoder* m, const std::string& p, int F) {
    const TensorStore& w = *m->store;
    MatrixBuilder b(m, (size_t)2 * gate_pad(F), m->Cp);
    b.put_gated(w.get(p + ".gate", {F, m->C}), w.get(p + ".up", {F, m->C}), F, m->C, 0);
    return b.build();
}
Matrix down_matrix(b200_decoder* m, const std::string& p, int F, int Fp) {
    MatrixBuilder b(m, m->Cp, Fp);
    b.put(m->store->get(p + ".down", {m->C, F}), 0, m->C, F, 0, 0);
    return b.build();
}

void load_mlp(b200_decoder* m, Layer& L, const std::string& p) {
    const LayerSpec& s = *L.spec;
    const TensorStore& w = *m->store;
    const int C = m->C, F = s.ff;
    Mlp& f = L.mlp;
    if (s.mlp == MLP_DENSE) {
        f.gate = m->spec.design->mlp_gate;
        if (f.gate == GATE_NONE) {
            MatrixBuilder up(m, pad_dim(F), m->Cp);
            up.put(w.get(p + ".up", {F, C}), 0, F, C, 0, 0);
            f.up = up.build();
            f.down = down_matrix(m, p, F, pad_dim(F));
        } else {
            f.up = gated_up(m, p, F);
            f.down = down_matrix(m, p, F, gate_pad(F));
        }
        return;
    }
    f.gate = GATE_CLAMP;
    const int Fp = gate_pad(F), E = s.experts, V = m->spec.vocab;
    MatrixBuilder up(m, (size_t)E * 2 * Fp, m->Cp), down(m, (size_t)E * m->Cp, Fp);
    for (int e = 0; e < E; ++e) {
        const std::string q = p + ".e" + std::to_string(e);
        up.put_gated(w.get(q + ".gate", {F, C}), w.get(q + ".up", {F, C}), F, C, (size_t)e * 2 * Fp);
        down.put(w.get(q + ".down", {C, F}), 0, C, F, (size_t)e * m->Cp, 0);
    }
    f.up = up.build(E);
    f.down = down.build(E);
    const HostTensor& t = w.get(p + ".table", {V, s.top}, true);
    std::vector<int> table((size_t)V * s.top);
    for (size_t i = 0; i < table.size(); ++i) {
        table[i] = t.integer(i);
        if (table[i] < 0 || table[i] >= E) throw std::runtime_error("weights: '" + p + ".table' names an expert that is not there");
        for (size_t k = i - i % s.top; k < i; ++k)
            if (table[k] == table[i]) throw std::runtime_error("weights: '" + p + ".table' names an expert twice for one token");
    }
    f.table = static_cast<int*>(upload(m, table.data(), table.size() * 4));
    if (s.shared_ff > 0) {
        f.shared_up = gated_up(m, p + ".shared", s.shared_ff);
        f.shared_down = down_matrix(m, p + ".shared", s.shared_ff, gate_pad(s.shared_ff));
        f.shared_gate = vector_f32(m, w.get(p + ".shared.sg", {1, C}), m->Cp);
    }
}

// the most runs, and rows of padded runs, of the pairs of M tokens
int most_runs(const b200_decoder* m, const LayerSpec& s, int M, int* rows) {
    const int P = M * s.top, align = moe_run_rows(P, s.experts, m->f32), runs = (P + (s.experts < P ? s.experts : P) * (align - 1)) / align;
    if (rows) *rows = runs * align;
    return runs;
}

void load_all(b200_decoder* m) {
    const TensorStore& w = *m->store;
    const int C = m->C, V = m->spec.vocab;
    const Design& design = *m->spec.design;
    {
        MatrixBuilder b(m, m->Vp, m->Cp);
        b.put(w.get("embed", {V, C}), 0, V, C, 0, 0);
        const Matrix e = b.build();
        m->embed = e.w;
        if (design.tied_head) m->head = e;
    }
    std::vector<Layer> layers(m->spec.layers.size());
    std::vector<MoeRoute> routes;
    for (size_t i = 0; i < layers.size(); ++i) {
        Layer& L = layers[i];
        L.spec = &m->spec.layers[i];
        const std::string p = "l" + std::to_string(i);
        L.norm1 = vector_f32(m, w.get(p + ".norm1", {C}), m->Cp, design.norm_offset);
        if (design.post_norm) L.norm1b = vector_f32(m, w.get(p + ".norm1b", {C}), m->Cp);
        switch (L.spec->kind) {
            case MIX_MAMBA1: load_mamba1(m, L, p + ".mix"); break;
            case MIX_DELTA:
            case MIX_CHANNEL_DELTA: load_delta(m, L, p + ".mix"); break;
            case MIX_PARALLEL: load_parallel(m, L, p + ".mix"); break;
            case MIX_LATENT: load_latent(m, L, p + ".mix"); break;
        }
        if (L.spec->mlp != MLP_NONE) {
            L.norm2 = vector_f32(m, w.get(p + ".norm2", {C}), m->Cp, design.norm_offset);
            if (design.post_norm) L.norm2b = vector_f32(m, w.get(p + ".norm2b", {C}), m->Cp);
            load_mlp(m, L, p + ".mlp");
        }
        if (L.spec->mlp == MLP_EXPERTS) {
            MoeRoute& r = L.mlp.route;
            r.table = L.mlp.table; r.experts = L.spec->experts; r.top = L.spec->top;
            int runs = 0;
            for (int M = 1; M <= m->max_rows; ++M) { const int n = most_runs(m, *L.spec, M, nullptr); if (n > runs) runs = n; }
            r.place = static_cast<int*>(device_zeros(m, (size_t)m->max_rows * r.top * 4));
            r.blocks = static_cast<int*>(device_zeros(m, (size_t)(1 + runs) * 4));
            r.decode = static_cast<DecodeRoute*>(device_zeros(m, sizeof(DecodeRoute)));
            routes.push_back(r);
            if (r.experts > m->max_experts) m->max_experts = r.experts;
        }
    }
    m->num_routes = (int)routes.size();
    if (m->num_routes) m->routes = static_cast<MoeRoute*>(upload(m, routes.data(), routes.size() * sizeof(MoeRoute)));
    for (int i : m->spec.order) {
        m->layers.push_back(layers[i]);
        allocate_state(m, m->layers.back());
    }
    m->final_norm = vector_f32(m, w.get("final.norm", {C}), m->Cp, design.norm_offset);
    if (!design.tied_head) {
        MatrixBuilder b(m, m->Vp, m->Cp);
        b.put(w.get("head", {V, C}), 0, V, C, 0, 0);
        m->head = b.build();
    }
}

// activations, sized from the loaded layers
void allocate(b200_decoder* m) {
    size_t proj = 0, mix = 0, conv = 0, aux = 0, wide = 0, q = 0, low = 0, gates = 0, ql = 0, raw = 0, decode_pair_mix = 0, top = 0;
    size_t pair_rows = 0, pair_mix = 0;  // (pair_mix, raw: elements)
    bool shared = false;
    auto up = [](size_t& a, size_t b) { if (b > a) a = b; };
    const size_t M = m->max_rows, e = elem(m);
    for (const Layer& L : m->layers) {
        const LayerSpec& s = *L.spec;
        up(proj, L.in.N);
        up(mix, L.o.K);
        switch (s.kind) {
            case MIX_MAMBA1: up(conv, L.np); up(aux, L.xp.N); up(wide, L.np); up(low, L.rank_p); break;
            case MIX_CHANNEL_DELTA: up(low, L.low.K); up(gates, L.low.N);  // and
            case MIX_DELTA: up(conv, 2 * L.np); up(wide, s.heads * L.Dvl); up(aux, 4 * s.heads); break;  // (fp32 in either arithmetic)
            case MIX_PARALLEL: up(q, (size_t)L.att.H * L.att.Dp); break;
            case MIX_LATENT:
                up(q, (size_t)L.lat.H * L.lat.Dp);
                up(ql, (size_t)L.lat.H * L.lat.Lp);
                break;
        }
        if (s.mlp == MLP_DENSE) {
            up(mix, L.mlp.down.K);
            if (L.mlp.gate != GATE_NONE) up(raw, M * L.mlp.up.N);
        } else if (s.mlp == MLP_EXPERTS) {
            if (s.shared_ff) { shared = true; up(mix, L.mlp.shared_down.K); up(raw, M * L.mlp.shared_up.N); }
            size_t most = 0;
            for (int n = 1; n <= m->max_rows; ++n) { int rows; most_runs(m, s, n, &rows); up(most, rows); }
            up(pair_rows, most);
            up(pair_mix, most * L.mlp.down.K);
            up(raw, most * L.mlp.up.N);
            up(top, s.top);
            up(decode_pair_mix, (size_t)16 * s.top * L.mlp.down.K);
        }
    }
    m->x = static_cast<float*>(device_zeros(m, M * m->Cp * 4));
    m->h = device_zeros(m, M * m->Cp * e);
    m->y = static_cast<float*>(device_zeros(m, M * m->Cp * 4));
    m->proj = static_cast<float*>(device_zeros(m, M * proj * 4));
    m->mix = device_zeros(m, M * mix * e);
    m->conv = device_zeros(m, M * conv * (m->f32 ? 4 : 2));
    m->aux = static_cast<float*>(device_zeros(m, M * aux * 4));
    m->wide = static_cast<float*>(device_zeros(m, M * wide * 4));
    m->low = device_zeros(m, M * low * e);
    m->q = device_zeros(m, M * q * e);
    m->gates = static_cast<float*>(device_zeros(m, M * gates * 4));
    if (pair_rows) {
        m->pair_h = device_zeros(m, pair_rows * m->Cp * e);
        m->pair_mix = device_zeros(m, pair_mix * e);
        m->pair_y = static_cast<float*>(device_zeros(m, pair_rows * m->Cp * 4));
        if (shared) m->shared_gate = static_cast<float*>(device_zeros(m, M * 4));
    }
    if (m->f32) m->raw = static_cast<float*>(device_zeros(m, raw * 4));
    if (ql && !m->f32) {
        // a sequence's step is expanded if that takes less: per head and position, n (2 R + Dr) multiply-adds on mma.sync, counted
        // four times, against n (Dp + Dvp) on tcgen05 and Lp (Dp + Dvp) for the expansion
        const Layer* first = nullptr;
        for (const Layer& L : m->layers) if (!first && L.spec->kind == MIX_LATENT) first = &L;
        const LatentAttention& c = first->lat;
        const long slow = 4L * (2 * c.R + c.Dr), fast = c.Dp + c.Dvp;
        m->expand_from = slow > fast ? (int)(c.Lp * fast / (slow - fast)) + 1 : m->max_rows + 1;
        // rows in the latent form: sequences below that many tokens, and decoding ones
        long rows = (long)m->max_slots * (m->expand_from - 1), pairs = 0, values = 0;
        if (rows > (long)M) rows = (long)M;
        if (rows < 16) rows = 16;
        m->ql = device_zeros(m, rows * ql * 2);
        for (const Layer& L : m->layers) {
            if (L.spec->kind != MIX_LATENT) continue;
            const long most = (rows > 256 ? rows : 256) * L.lat.H;  // 16 decoding rows in up to 16 shares
            if (most > pairs) pairs = most;
            if (most * L.lat.Rp > values) values = most * L.lat.Rp;
        }
        m->lat_parts.o = static_cast<float*>(device_zeros(m, values * 4));
        m->lat_parts.ml = static_cast<float2*>(device_zeros(m, pairs * sizeof(float2)));
        m->lat_rows_room = rows > 256 ? rows : 256;
    }
    if (!m->f32) {
        m->dx = static_cast<float*>(device_zeros(m, (size_t)16 * m->Cp * 4));
        m->dy = static_cast<float*>(device_zeros(m, (size_t)16 * m->Cp * 4));
        m->dh = device_zeros(m, (size_t)16 * m->Cp * 4);
        m->dproj = static_cast<float*>(device_zeros(m, (size_t)16 * proj * 4));
        m->dmix = device_zeros(m, (size_t)16 * mix * 4);
        m->dconv = device_zeros(m, (size_t)16 * conv * 4);
        m->daux = static_cast<float*>(device_zeros(m, (size_t)16 * aux * 4));
        m->dql = device_zeros(m, (size_t)16 * ql * 2);
        if (pair_rows) {
            m->dpair_mix = device_zeros(m, decode_pair_mix * 4);
            m->dpair_y = static_cast<float*>(device_zeros(m, 16 * top * m->Cp * 4));
            m->dshared_gate = static_cast<float*>(device_zeros(m, 16 * 4));
        }
        m->dlogits = static_cast<float*>(device_zeros(m, (size_t)16 * m->Vp * 4));
    }
    // descriptors: sequences, tokens, the sequence of every row, wanted rows, rows and sequences in the latent form, query-tile
    // pairs of all sequences and of the expanded ones
    m->desc_ints = (size_t)m->max_slots * 9 + 4 * M + 4 * (M / 256 + m->max_slots + 1) + 64;
    if (m->desc_ints < 16 * 9) m->desc_ints = 16 * 9;
    m->desc = static_cast<int*>(device_zeros(m, m->desc_ints * 4));
    m->dseqs = static_cast<SeqDesc*>(device_zeros(m, 16 * (sizeof(SeqDesc) + 4)));
    m->dtokens = reinterpret_cast<int*>(m->dseqs + 16);
    for (int i = 0; i < b200_decoder::kRing; ++i) {
        if (cudaHostAlloc(&m->pinned[i], m->desc_ints * 4, cudaHostAllocDefault) != cudaSuccess ||
            cudaEventCreateWithFlags(&m->ring_ev[i], cudaEventDisableTiming) != cudaSuccess)
            throw std::runtime_error("pinned descriptor buffers");
    }
}

int finish_load(b200_decoder* m) {
    b200_device_guard guard(m->ctx);
    try {
        load_all(m);
        allocate(m);
    } catch (const std::exception& e) {
        m->ctx->last_error = e.what();
        return B200_ERR_STATE;
    }
    delete m->store;
    m->store = nullptr;
    const cudaError_t e = cudaDeviceSynchronize();  // the fills above ran on the default stream
    if (e != cudaSuccess) return b200_fail_cuda(m->ctx, e, "loading weights");
    m->ready = true;
    return B200_OK;
}

#define TRY(call) do { const int st__ = (call); if (st__ != B200_OK) return st__; } while (0)

int prof_mark(b200_decoder* m, const char* name) {
    const size_t used = 2 * m->ev_name.size() - (name ? 0 : 1);  // a start, or the stop of the last start
    while (m->ev_pool.size() <= used) {
        cudaEvent_t e;
        B200_CUDA(m->ctx, cudaEventCreate(&e));
        m->ev_pool.push_back(e);
    }
    B200_CUDA(m->ctx, cudaEventRecord(m->ev_pool[used], m->ctx->stream));
    if (name) m->ev_name.push_back(name);
    return B200_OK;
}
// an operator of a step, timed under its name when profiling is on
#define OP(name, call)                            \
    do {                                          \
        if (m->profile) TRY(prof_mark(m, name));  \
        TRY(call);                                \
        if (m->profile) TRY(prof_mark(m, nullptr)); \
    } while (0)

// ------------------------------------------------------------------ general path
// out = act(in W^T + bias); out is fp32, or with elem_out the model's element type
int product(b200_decoder* m, void* out, const void* in, const Matrix& w, int M, int act = ACT_NONE, bool elem_out = false) {
    b200_ctx* ctx = m->ctx;
    if (m->f32) {
        if (M <= 16 && act == ACT_NONE && (size_t)(M <= 8 ? 8 : 16) * w.K * 4 <= (size_t)160 * 1024)
            return launch_skinny_gemm(ctx, static_cast<float*>(out), static_cast<const float*>(in), static_cast<const float*>(w.w), w.bias, M, w.K, w.N, 0);
        return launch_gemm_fp32(ctx, static_cast<float*>(out), static_cast<const float*>(in), static_cast<const float*>(w.w), w.bias, M, w.K, w.N, act);
    }
    const int flags = act == ACT_GELU_ERF ? GEMM_GELU_ERF : (act == ACT_GELU_TANH ? GEMM_GELU : 0);
    return launch_gemm_bf16(ctx, elem_out ? nullptr : static_cast<float*>(out), elem_out ? static_cast<uint16_t*>(out) : nullptr,
                            static_cast<const uint16_t*>(in), static_cast<const uint16_t*>(w.w), w.bias, M, w.K, w.N, flags);
}

// down-projection's input: act(gate) * linear part; groups: per run of rows with a matrix of its own
int gated_product(b200_decoder* m, void* out, const void* in, const Matrix& w, int M, int gate, float limit, const GemmGroups* groups = nullptr) {
    b200_ctx* ctx = m->ctx;
    if (m->f32) {
        TRY(launch_gemm_fp32(ctx, m->raw, static_cast<const float*>(in), static_cast<const float*>(w.w), nullptr, M, w.K, w.N, ACT_NONE, groups));
        return launch_gated_act(ctx, static_cast<float*>(out), m->raw, M, w.N / 2, gate, limit);
    }
    return launch_gemm_bf16(ctx, nullptr, static_cast<uint16_t*>(out), static_cast<const uint16_t*>(in), static_cast<const uint16_t*>(w.w), nullptr, M, w.K, w.N,
                            gate == GATE_CLAMP ? GEMM_GATED_CLAMP : GEMM_GATED_GELU, nullptr, 0, 0, limit, groups);
}
int grouped_product(b200_decoder* m, float* out, const void* in, const Matrix& w, int M, const GemmGroups* groups) {
    b200_ctx* ctx = m->ctx;
    if (m->f32) return launch_gemm_fp32(ctx, out, static_cast<const float*>(in), static_cast<const float*>(w.w), nullptr, M, w.K, w.N, ACT_NONE, groups);
    return launch_gemm_bf16(ctx, out, nullptr, static_cast<const uint16_t*>(in), static_cast<const uint16_t*>(w.w), nullptr, M, w.K, w.N, 0, nullptr, 0, 0, 0.f, groups);
}

struct StepView {
    const SeqDesc* seqs; const int* tokens; const int* row_seq; const int* want; const int2* pairs;
    int E, M, max_n, n_want, num_pairs;
    // latent attention: rows and sequences in the latent form, query-tile pairs of the expanded sequences, whose positions are kv_rows rows
    const int* lat_rows; const int* lat_seqs; const int2* kv_pairs;
    int num_lat_rows, num_lat_seqs, lat_max_n, lat_max_keys, num_kv_pairs, kv_rows, kv_max_pos0;
};

int mixer_mamba1(b200_decoder* m, const Layer& L, const StepView& v) {
    b200_ctx* ctx = m->ctx;
    const LayerSpec& s = *L.spec;
    OP("gemm mamba1 in", product(m, m->proj, m->h, L.in, v.M));
    ShortConvArgs c{};
    c.x = m->proj; c.ldx = L.in.N; c.out = m->conv; c.ld_out = L.np; c.w = L.conv_w; c.bias = L.conv_b; c.hist = L.hist; c.seqs = v.seqs;
    c.np = L.np; c.taps = s.conv; c.max_slots = m->max_slots;
    OP("conv mamba1", launch_short_conv(ctx, c, v.E, v.max_n, m->f32));
    OP("gemm mamba1 x", product(m, m->aux, m->conv, L.xp, v.M));
    OP("slice", launch_slice(ctx, m->low, L.rank_p, m->aux, L.xp.N, s.dt_rank, v.M, m->f32));
    OP("gemm mamba1 dt", product(m, m->wide, m->low, L.dt, v.M));
    SelectiveScanArgs a{};
    a.x = m->conv; a.ldx = L.np; a.dt = m->wide; a.lddt = L.np; a.bc = m->aux; a.ldbc = L.xp.N; a.b_col = L.rank_p; a.c_col = L.rank_p + L.sp;
    a.z = m->proj + L.np; a.ldz = L.in.N; a.A2 = L.A2; a.dt_b = L.dt_b; a.D = L.D; a.S = L.S; a.out = m->mix; a.ldo = L.o.K; a.seqs = v.seqs;
    a.inner = s.inner; a.state_pad = L.sp;
    OP("selective scan", launch_selective_scan(ctx, a, v.E, v.max_n, m->f32, m->f32));
    return B200_OK;
}

DeltaArgs delta_args(const b200_decoder* m, const Layer& L, const SeqDesc* seqs, const float* proj) {
    const LayerSpec& s = *L.spec;
    DeltaArgs a{};
    a.ld = L.np; a.k_col = L.k_col; a.v_col = L.v_col;
    a.gates = proj; a.ldg = L.in.N; a.a_col = L.a_col; a.b_col = L.b_col;
    a.negA = L.negA; a.dt_bias = L.dt_bias; a.S = L.S; a.seqs = seqs;
    a.H = s.heads; a.G = s.kv_heads; a.D = s.dim; a.Dl = L.Dl; a.Dv = s.vdim; a.Dvl = L.Dvl;
    a.conv_w = L.conv_w; a.hist = L.hist; a.taps = s.conv; a.np = L.np; a.max_slots = m->max_slots;
    a.norm_w = L.head_norm; a.gate_col = L.gate_col; a.eps = m->spec.eps;
    if (s.kind == MIX_CHANNEL_DELTA) {
        a.w_low = static_cast<const uint16_t*>(L.low.w); a.ld_low = L.low.K; a.low_col = L.low_col; a.low_a = L.low_a; a.low_g = L.low_g; a.gate_row = L.gate_row;
    }
    return a;
}

int mixer_delta(b200_decoder* m, const Layer& L, const StepView& v) {
    b200_ctx* ctx = m->ctx;
    const LayerSpec& s = *L.spec;
    const bool channel = s.kind == MIX_CHANNEL_DELTA;
    OP("gemm delta in", product(m, m->proj, m->h, L.in, v.M));
    if (channel) {
        OP("slice", launch_slice(ctx, m->low, L.low.K, m->proj + L.low_col, L.in.N, L.low_a + L.low_g, v.M, m->f32));
        OP("gemm delta low rank", product(m, m->gates, m->low, L.low, v.M));
    }
    ShortConvArgs c{};
    c.x = m->proj; c.ldx = L.in.N; c.out = m->conv; c.ld_out = L.np; c.w = L.conv_w; c.hist = L.hist; c.seqs = v.seqs;
    c.np = L.np; c.taps = s.conv; c.max_slots = m->max_slots;
    c.ch0 = L.v_col;
    OP("conv delta v", launch_short_conv(ctx, c, v.E, v.max_n, true));
    DeltaArgs a = delta_args(m, L, v.seqs, m->proj);
    a.qkv = static_cast<const float*>(m->conv);
    a.raw = m->proj; a.ld_raw = L.in.N;
    a.coef = reinterpret_cast<float4*>(m->aux);
    if (channel) { a.decay = m->gates; a.ld_decay = L.low.N; }
    OP("delta prep", launch_delta_prep(ctx, a, v.E, v.max_n));
    a.out = m->wide; a.ldo = s.heads * L.Dvl;
    OP("delta scan", launch_delta_scan(ctx, a, v.E));
    OP("head norm", launch_gated_head_norm(ctx, m->mix, L.o.K, m->wide, a.ldo, channel ? m->gates + L.gate_row : m->proj + L.gate_col, channel ? L.low.N : L.in.N,
                                           L.head_norm, v.M, s.heads, s.vdim, L.Dvl, m->spec.eps, m->f32, channel));
    return B200_OK;
}

LatentParts latent_parts(const b200_decoder* m, const Layer& L) {
    LatentParts p = m->lat_parts;
    p.pairs = m->lat_rows_room * L.lat.H;
    return p;
}

int mixer_latent(b200_decoder* m, const Layer& L, const StepView& v) {
    b200_ctx* ctx = m->ctx;
    const LatentAttention& c = L.lat;
    OP("gemm latent in", product(m, m->proj, m->h, L.in, v.M));
    OP("latent prep", launch_latent_prep(ctx, c, m->proj, L.in.N, m->q, m->lat, v.seqs, v.row_seq, v.M, m->f32));
    if (v.kv_rows > 0) {
        if (v.kv_max_pos0 > 0) OP("latent gather", launch_latent_gather(ctx, c, m->lat, v.seqs, v.E, v.kv_max_pos0, m->f32));
        CachedAttention f = L.flat;
        f.K = m->kv; f.V = static_cast<char*>(m->kv) + (size_t)c.H * c.Dp * elem(m); f.kv_rows = v.kv_rows;
        if (m->f32) OP("gemm latent kv", product(m, m->kv, m->lat, L.kv, v.kv_rows));
        else OP("gemm latent kv", launch_gemm_bf16(ctx, nullptr, static_cast<uint16_t*>(m->kv), static_cast<const uint16_t*>(m->lat), static_cast<const uint16_t*>(L.kv.w),
                                                   nullptr, v.kv_rows, L.kv.K, L.kv.N, GEMM_FP16));
        if (!m->f32 && attention_cached_has_mma(f))
            OP("attention", launch_attention_cached_mma(ctx, f, m->q, m->mix, L.o.K, v.seqs, v.kv_pairs, v.num_kv_pairs, v.M, m->max_slots));
        else
            OP("attention", launch_attention_cached_simt(ctx, f, m->q, m->mix, L.o.K, v.seqs, v.E, v.max_n, m->f32));
    }
    if (v.num_lat_rows > 0) {
        OP("latent query", launch_latent_query(ctx, c, m->proj, L.in.N, m->ql, v.seqs, v.row_seq, v.lat_rows, v.num_lat_rows, false));
        OP("latent attention", launch_latent_attention(ctx, c, m->ql, latent_parts(m, L), m->mix, L.o.K, v.seqs, v.lat_seqs, v.num_lat_seqs, v.lat_rows, v.num_lat_rows, v.lat_max_n,
                                                       v.lat_max_keys, false));
    }
    return B200_OK;
}

MinGruArgs gru_args(const Layer& L, const SeqDesc* seqs, const float* proj, void* out) {
    MinGruArgs g{};
    g.zx = proj; g.ld = L.in.N; g.z_col = L.z_col; g.x_col = L.x_col; g.g_col = L.g_col; g.S = L.S;
    g.out = out; g.ldo = L.o.K; g.seqs = seqs; g.width = L.spec->gru_width; g.out_scale = L.spec->right_scale;
    return g;
}

int mixer_parallel(b200_decoder* m, const Layer& L, const StepView& v) {
    b200_ctx* ctx = m->ctx;
    OP("gemm parallel in", product(m, m->proj, m->h, L.in, v.M));
    OP("attention prep", launch_attention_prep(ctx, L.att, m->proj, L.in.N, m->q, v.seqs, v.row_seq, v.M, m->f32));
    if (!m->f32 && attention_cached_has_mma(L.att))
        OP("attention", launch_attention_cached_mma(ctx, L.att, m->q, m->mix, L.o.K, v.seqs, v.pairs, v.num_pairs, v.M, m->max_slots));
    else
        OP("attention", launch_attention_cached_simt(ctx, L.att, m->q, m->mix, L.o.K, v.seqs, v.E, v.max_n, m->f32));
    OP("min gru", launch_min_gru(ctx, gru_args(L, v.seqs, m->proj, static_cast<char*>(m->mix) + L.att_p * elem(m)), v.E, m->f32));
    return B200_OK;
}

// what the next residual kernel adds: a mixer's (or dense feed-forward's) output ...
void branch_of_mixer(ResidualNormArgs& n, const Layer& L, const float* y) {
    n.y = y; n.wb = L.norm1b; n.y_scale = nullptr;
    n.parts = nullptr; n.part_of = nullptr; n.top = 0;
}
// ... or the experts' outputs
void branch_of_experts(ResidualNormArgs& n, const Layer& L, const float* shared, const float* shared_gate, const float* parts, const int* part_of) {
    n.y = shared; n.wb = nullptr; n.y_scale = shared ? shared_gate : nullptr;
    n.parts = parts; n.part_of = part_of; n.top = L.spec->top; n.part_scale = 1.0f / (float)L.spec->top;
}

// rows of the step -> logits of the wanted rows in m->logits
int enqueue_general(b200_decoder* m, const StepView& v) {
    b200_ctx* ctx = m->ctx;
    ResidualNormArgs n{};
    n.C = m->C; n.Cp = m->Cp; n.eps = m->spec.eps; n.vocab = m->spec.vocab;
    n.x_out = m->x; n.h = m->h; n.M = v.M;
    n.tok = v.tokens; n.embed = m->embed; n.embed_scale = m->spec.embed_scale;
    n.w = m->layers[0].norm1;
    if (m->num_routes) OP("expert routes", launch_moe_route(ctx, m->routes, m->num_routes, v.tokens, v.M, m->f32, m->max_experts));
    OP("embed norm", launch_residual_rms(ctx, n, m->f32 ? H_F32 : H_BF16));
    n.tok = nullptr;
    n.x = m->x;
    for (size_t i = 0; i < m->layers.size(); ++i) {
        const Layer& L = m->layers[i];
        const Mlp& f = L.mlp;
        const char* o_name = "";
        switch (L.spec->kind) {
            case MIX_MAMBA1: TRY(mixer_mamba1(m, L, v)); o_name = "gemm mamba1 o"; break;
            case MIX_DELTA:
            case MIX_CHANNEL_DELTA: TRY(mixer_delta(m, L, v)); o_name = "gemm delta o"; break;
            case MIX_PARALLEL: TRY(mixer_parallel(m, L, v)); o_name = "gemm parallel o"; break;
            case MIX_LATENT: TRY(mixer_latent(m, L, v)); o_name = "gemm latent o"; break;
        }
        OP(o_name, product(m, m->y, m->mix, L.o, v.M));
        const bool last = i + 1 == m->layers.size();
        branch_of_mixer(n, L, m->y);
        if (L.spec->mlp == MLP_DENSE) {
            n.w = L.norm2;
            OP("residual norms", launch_residual_rms(ctx, n, m->f32 ? H_F32 : H_BF16));
            if (f.gate == GATE_NONE) OP("gemm mlp up", product(m, m->mix, m->h, f.up, v.M, m->spec.design->mlp_act, true));
            else OP("gemm mlp up", gated_product(m, m->mix, m->h, f.up, v.M, f.gate, 0.f));
            OP("gemm mlp down", product(m, m->y, m->mix, f.down, v.M));
            n.wb = L.norm2b;
        } else if (L.spec->mlp == MLP_EXPERTS) {
            const LayerSpec& s = *L.spec;
            int rows;
            most_runs(m, s, v.M, &rows);
            const GemmGroups groups{f.route.blocks, moe_run_rows(v.M * s.top, s.experts, m->f32), s.experts};
            n.w = L.norm2;
            n.copy = m->pair_h; n.copy_of = f.route.place; n.copies = s.top;
            n.gate_w = f.shared_gate; n.gate_out = m->shared_gate;
            OP("residual norms experts", launch_residual_rms(ctx, n, m->f32 ? H_F32 : H_BF16));
            n.copies = 0;
            n.gate_w = nullptr;
            OP("gemm experts up", gated_product(m, m->pair_mix, m->pair_h, f.up, rows, f.gate, s.limit, &groups));
            OP("gemm experts down", grouped_product(m, m->pair_y, m->pair_mix, f.down, rows, &groups));
            if (s.shared_ff) {
                OP("gemm shared up", gated_product(m, m->mix, m->h, f.shared_up, v.M, f.gate, s.shared_limit));
                OP("gemm shared down", product(m, m->y, m->mix, f.shared_down, v.M));
            }
            branch_of_experts(n, L, s.shared_ff ? m->y : nullptr, m->shared_gate, m->pair_y, f.route.place);
        }
        if (!last) {
            n.w = m->layers[i + 1].norm1;
            OP(n.top ? "residual norms parts" : "residual norms", launch_residual_rms(ctx, n, m->f32 ? H_F32 : H_BF16));
        }
    }
    if (v.n_want == 0) return B200_OK;
    n.w = m->final_norm;  // only the wanted rows go on
    n.rows = v.want;
    n.M = v.n_want;
    n.x_out = nullptr;
    OP("final norm", launch_residual_rms(ctx, n, m->f32 ? H_F32 : H_BF16));
    OP("gemm head", product(m, m->logits, m->h, m->head, v.n_want));
    return B200_OK;
}

// ------------------------------------------------------------------ decode path
// One token for each of B <= 16 sequences: descriptors and tokens come from dseqs / dtokens, the logits go to
// dlogits.  The inputs of the products are split rows (decoder_math.cuh), written so by whatever produces them; the
// short convolutions run in the epilogue of the projection in front of them.
int enqueue_decode(b200_decoder* m, int B) {
    b200_ctx* ctx = m->ctx;
    ResidualNormArgs n{};
    n.C = m->C; n.Cp = m->Cp; n.eps = m->spec.eps; n.vocab = m->spec.vocab; n.M = B;
    n.x_out = m->dx; n.h = m->dh;
    n.tok = m->dtokens; n.embed = m->embed; n.embed_scale = m->spec.embed_scale;
    auto norm = [&](const float* w) {
        n.w = w;
        const int st = launch_residual_rms(ctx, n, H_SPLIT);
        n.tok = nullptr;
        n.x = m->dx;
        return st;
    };
    auto product_args = [&](const void* x, const Matrix& w) {
        DecodeGemmArgs a{};
        a.x = static_cast<const uint8_t*>(x); a.W = static_cast<const uint16_t*>(w.w); a.bias = w.bias; a.B = B; a.N = w.N; a.K = w.K;
        return a;
    };
    auto plain = [&](float* out, const void* x, const Matrix& w) {
        DecodeGemmArgs a = product_args(x, w);
        a.out = out; a.ldo = w.N;
        return launch_decode_gemm(ctx, a);
    };
    if (m->num_routes) TRY(launch_decode_routes(ctx, m->routes, m->num_routes, m->dtokens, B));
    for (const Layer& L : m->layers) {
        const LayerSpec& s = *L.spec;
        TRY(norm(L.norm1));
        DecodeGemmArgs in = product_args(m->dh, L.in);
        in.out = m->dproj; in.ldo = L.in.N;
        if (s.kind != MIX_PARALLEL && s.kind != MIX_LATENT) {
            in.seqs = m->dseqs; in.conv_w = L.conv_w; in.conv_b = L.conv_b; in.hist = L.hist; in.conv_n = L.np; in.taps = s.conv; in.max_slots = m->max_slots;
            if (s.kind == MIX_MAMBA1) in.conv_out = static_cast<uint8_t*>(m->dconv);
        }
        TRY(launch_decode_gemm(ctx, in));
        if (s.kind == MIX_MAMBA1) {
            TRY(plain(m->daux, m->dconv, L.xp));
            SelectiveScanArgs c{};
            c.x = m->dconv; c.ldx = L.np; c.bc = m->daux; c.ldbc = L.xp.N; c.b_col = L.rank_p; c.c_col = L.rank_p + L.sp;
            c.z = m->dproj + L.np; c.ldz = L.in.N; c.A2 = L.A2; c.dt_b = L.dt_b; c.D = L.D; c.S = L.S; c.out = m->dmix; c.ldo = L.o.K; c.seqs = m->dseqs;
            c.inner = s.inner; c.state_pad = L.sp;
            c.Wdt = static_cast<const uint16_t*>(L.dt.w); c.rank = s.dt_rank; c.ld_wdt = L.rank_p;
            TRY(launch_selective_scan(ctx, c, B, 1, true, true));
        } else if (s.kind == MIX_LATENT) {
            TRY(launch_latent_query(ctx, L.lat, m->dproj, L.in.N, m->dql, m->dseqs, nullptr, nullptr, B, true));
            TRY(launch_latent_attention(ctx, L.lat, m->dql, latent_parts(m, L), m->dmix, L.o.K, m->dseqs, nullptr, B, nullptr, B, 1, m->Tp, true));
        } else if (s.kind == MIX_DELTA || s.kind == MIX_CHANNEL_DELTA) {
            DeltaArgs a = delta_args(m, L, m->dseqs, m->dproj);
            a.qkv = m->dproj; a.ld = L.in.N;
            a.out = static_cast<float*>(m->dmix); a.ldo = L.o.K;
            TRY(launch_delta_step(ctx, a, B));
        } else {
            MinGruArgs gru = gru_args(L, m->dseqs, m->dproj, m->dmix);
            gru.out_col = L.att_p;
            TRY(launch_attention_cached_decode(ctx, L.att, m->dproj, L.in.N, static_cast<uint8_t*>(m->dmix), L.o.K, m->dseqs, B, gru));
        }
        TRY(plain(m->dy, m->dmix, L.o));
        branch_of_mixer(n, L, m->dy);
        const Mlp& f = L.mlp;
        if (s.mlp == MLP_DENSE) {
            TRY(norm(L.norm2));
            DecodeGemmArgs up = product_args(m->dh, f.up);
            up.act = m->spec.design->mlp_act;
            up.gate = f.gate;
            up.split_out = static_cast<uint8_t*>(m->dmix);
            TRY(launch_decode_gemm(ctx, up));
            TRY(plain(m->dy, m->dmix, f.down));
            n.wb = L.norm2b;
        } else if (s.mlp == MLP_EXPERTS) {
            n.gate_w = f.shared_gate; n.gate_out = m->dshared_gate;
            TRY(norm(L.norm2));
            n.gate_w = nullptr;
            DecodeGemmArgs up = product_args(m->dh, f.up), down = product_args(m->dpair_mix, f.down);
            up.route = down.route = f.route.decode; up.top = down.top = s.top; up.experts = down.experts = s.experts;
            up.gate = f.gate; up.limit = s.limit; up.split_out = static_cast<uint8_t*>(m->dpair_mix);
            down.pair_in = 1; down.out = m->dpair_y; down.ldo = f.down.N;
            if (s.shared_ff) {
                up.shared = {static_cast<const uint8_t*>(m->dh), static_cast<const uint16_t*>(f.shared_up.w), f.shared_up.N, f.shared_up.K, s.shared_limit, nullptr, 0,
                             static_cast<uint8_t*>(m->dmix)};
                down.shared = {static_cast<const uint8_t*>(m->dmix), static_cast<const uint16_t*>(f.shared_down.w), f.shared_down.N, f.shared_down.K, 0.f, m->dy,
                               f.shared_down.N, nullptr};
            }
            TRY(launch_decode_gemm(ctx, up));
            TRY(launch_decode_gemm(ctx, down));
            branch_of_experts(n, L, s.shared_ff ? m->dy : nullptr, m->dshared_gate, m->dpair_y, nullptr);
        }
    }
    TRY(norm(m->final_norm));
    return plain(m->dlogits, m->dh, m->head);
}

// ------------------------------------------------------------------ steps
// the next pinned descriptor buffer, free to be written
int ring_buffer(b200_decoder* m, int** out) {
    m->ring = (m->ring + 1) % b200_decoder::kRing;
    B200_CUDA(m->ctx, cudaEventSynchronize(m->ring_ev[m->ring]));
    *out = m->pinned[m->ring];
    return B200_OK;
}

struct Entry { int slot; const int* tokens; int n; };

SeqDesc describe(b200_decoder* m, int slot, int row0, int n) {
    Slot& s = m->slots[slot];
    SeqDesc d{};
    d.row0 = row0; d.n = n; d.slot = slot; d.pos0 = s.len; d.bank = s.bank; d.kv0 = -1; d.lat0 = row0;
    s.len += n;
    s.bank ^= 1;
    return d;
}

// decode path: tokens == nullptr keeps the ids that are in dtokens already
int decode_step(b200_decoder* m, const std::vector<int>& slots, const int* tokens) {
    b200_ctx* ctx = m->ctx;
    const int B = (int)slots.size();
    int* host;
    TRY(ring_buffer(m, &host));
    SeqDesc* sd = reinterpret_cast<SeqDesc*>(host);
    for (int b = 0; b < B; ++b) sd[b] = describe(m, slots[b], b, 1);
    B200_CUDA(ctx, cudaMemcpyAsync(m->dseqs, sd, B * sizeof(SeqDesc), cudaMemcpyHostToDevice, ctx->stream));
    if (tokens) {
        int* t = host + 16 * 8;
        for (int b = 0; b < B; ++b) t[b] = tokens[b];
        B200_CUDA(ctx, cudaMemcpyAsync(m->dtokens, t, B * 4, cudaMemcpyHostToDevice, ctx->stream));
    }
    B200_CUDA(ctx, cudaEventRecord(m->ring_ev[m->ring], ctx->stream));
    if (!m->use_graph || ctx->stream == nullptr) return enqueue_decode(m, B);
    auto it = m->graphs.find(B);
    if (it == m->graphs.end()) {
        // The first step of a batch size runs eagerly (kernel attributes are set outside of capture) and is
        // captured behind that, for the following ones.
        TRY(enqueue_decode(m, B));
        B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        const uint64_t before = ctx->launches;
        cudaGraph_t graph = nullptr;
        B200_CUDA(ctx, cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal));
        const int st = enqueue_decode(m, B);
        const cudaError_t e = cudaStreamEndCapture(ctx->stream, &graph);
        m->graph_launches[B] = ctx->launches - before;
        ctx->launches = before;
        if (st != B200_OK) { if (graph) cudaGraphDestroy(graph); return st; }
        if (e != cudaSuccess) return b200_fail_cuda(ctx, e, "cudaStreamEndCapture");
        cudaGraphExec_t exec = nullptr;
        const cudaError_t ie = cudaGraphInstantiate(&exec, graph, 0);
        cudaGraphDestroy(graph);
        if (ie != cudaSuccess) return b200_fail_cuda(ctx, ie, "cudaGraphInstantiate");
        m->graphs.emplace(B, exec);
        return B200_OK;
    }
    B200_CUDA(ctx, cudaGraphLaunch(it->second, ctx->stream));
    ctx->launches += m->graph_launches[B];
    return B200_OK;
}

// latents and expanded keys and values of `rows` positions
int reserve_expanded(b200_decoder* m, int rows) {
    if (rows <= m->kv_rows) return B200_OK;
    b200_ctx* ctx = m->ctx;
    size_t lat = 0, kv = 0;
    for (const Layer& L : m->layers)
        if (L.spec->kind == MIX_LATENT) { if ((size_t)L.kv.K > lat) lat = L.kv.K; if ((size_t)L.kv.N > kv) kv = L.kv.N; }
    if (rows < 2 * m->kv_rows) rows = 2 * m->kv_rows;
    B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    if (m->lat) cudaFree(m->lat);
    if (m->kv) cudaFree(m->kv);
    m->lat = m->kv = nullptr;
    m->kv_rows = 0;
    B200_CUDA(ctx, cudaMalloc(&m->lat, rows * lat * elem(m)));
    B200_CUDA(ctx, cudaMalloc(&m->kv, rows * kv * elem(m)));
    m->kv_rows = rows;
    return B200_OK;
}

int general_step(b200_decoder* m, const std::vector<Entry>& entries, const std::vector<int>& want) {
    b200_ctx* ctx = m->ctx;
    int M = 0, max_n = 0, expanded = 0;
    bool latent = false;
    for (const Layer& L : m->layers) latent = latent || L.spec->kind == MIX_LATENT;
    for (const Entry& e : entries) {
        M += e.n;
        if (e.n > max_n) max_n = e.n;
        if (latent && e.n >= m->expand_from) expanded += m->slots[e.slot].len + e.n;
    }
    if (expanded) TRY(reserve_expanded(m, expanded));
    const int E = (int)entries.size(), nw = (int)want.size();
    if (nw > m->logits_rows) {
        B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        if (m->logits) cudaFree(m->logits);
        m->logits = nullptr;
        m->logits_rows = 0;
        B200_CUDA(ctx, cudaMalloc(&m->logits, (size_t)nw * m->Vp * 4));
        m->logits_rows = nw;
    }
    int* host;
    TRY(ring_buffer(m, &host));
    SeqDesc* sd = reinterpret_cast<SeqDesc*>(host);
    int* tok = host + 8 * E;
    int* row_seq = tok + M;
    int* w = row_seq + M;
    int* lat_rows = w + nw;
    int* lat_seqs = lat_rows + M;
    int* pr = lat_seqs + E;
    if ((pr - host) & 1) ++pr;  // int2
    struct Pair { int seq, pair, keys; };
    std::vector<Pair> pairs;
    StepView v{};
    int row = 0;
    for (int i = 0; i < E; ++i) {
        const Entry& e = entries[i];
        sd[i] = describe(m, e.slot, row, e.n);
        if (latent && e.n >= m->expand_from) {
            sd[i].kv0 = v.kv_rows;
            v.kv_rows += sd[i].pos0 + e.n;
            if (sd[i].pos0 > v.kv_max_pos0) v.kv_max_pos0 = sd[i].pos0;
        } else if (latent) {
            sd[i].lat0 = v.num_lat_rows;
            for (int t = 0; t < e.n; ++t) lat_rows[v.num_lat_rows++] = row + t;
            lat_seqs[v.num_lat_seqs++] = i;
            if (e.n > v.lat_max_n) v.lat_max_n = e.n;
            if (sd[i].pos0 + e.n > v.lat_max_keys) v.lat_max_keys = sd[i].pos0 + e.n;
        }
        for (int t = 0; t < e.n; ++t) { tok[row + t] = e.tokens[t]; row_seq[row + t] = i; }
        for (int p = 0; p * 256 < e.n; ++p) pairs.push_back({i, p, sd[i].pos0 + (e.n < (p + 1) * 256 ? e.n : (p + 1) * 256)});
        row += e.n;
    }
    for (int i = 0; i < nw; ++i) w[i] = want[i];
    // most keys first (stable, so the list is the same for the same step)
    for (size_t i = 1; i < pairs.size(); ++i)
        for (size_t j = i; j > 0 && pairs[j - 1].keys < pairs[j].keys; --j) std::swap(pairs[j - 1], pairs[j]);
    for (size_t i = 0; i < pairs.size(); ++i) { pr[2 * i] = pairs[i].seq; pr[2 * i + 1] = pairs[i].pair; }
    int* kpr = pr + 2 * pairs.size();
    for (const Pair& p : pairs)
        if (sd[p.seq].kv0 >= 0) { kpr[2 * v.num_kv_pairs] = p.seq; kpr[2 * v.num_kv_pairs + 1] = p.pair; v.num_kv_pairs++; }
    const size_t used = (kpr - host) + 2 * (size_t)v.num_kv_pairs;
    if (used > m->desc_ints) return B200_ERR_LIMIT;
    B200_CUDA(ctx, cudaMemcpyAsync(m->desc, host, used * 4, cudaMemcpyHostToDevice, ctx->stream));
    B200_CUDA(ctx, cudaEventRecord(m->ring_ev[m->ring], ctx->stream));
    v.seqs = reinterpret_cast<const SeqDesc*>(m->desc);
    v.tokens = m->desc + (tok - host);
    v.row_seq = m->desc + (row_seq - host);
    v.want = m->desc + (w - host);
    v.pairs = reinterpret_cast<const int2*>(m->desc + (pr - host));
    v.kv_pairs = reinterpret_cast<const int2*>(m->desc + (kpr - host));
    v.lat_rows = m->desc + (lat_rows - host);
    v.lat_seqs = m->desc + (lat_seqs - host);
    v.E = E; v.M = M; v.max_n = max_n; v.n_want = nw; v.num_pairs = (int)pairs.size();
    return enqueue_general(m, v);
}

}  // namespace

extern "C" {

int b200_decoder_create(b200_decoder** out, b200_ctx* ctx, const char* config_json, int arithmetic, int max_slots, int max_seq, int max_rows) {
    if (!out || !ctx || !config_json) return B200_ERR_NULL;
    *out = nullptr;
    if (arithmetic != B200_DECODER_BF16 && arithmetic != B200_DECODER_FP32) return B200_ERR_SHAPE;
    if (max_slots < 1 || max_seq < 1 || max_rows < 1) return B200_ERR_SHAPE;
    b200_decoder* m = new (std::nothrow) b200_decoder();
    if (!m) return B200_ERR_CUDA;
    try {
        m->spec = parse_config(config_json);
    } catch (const std::exception& e) {
        ctx->last_error = e.what();
        delete m;
        return B200_ERR_SHAPE;
    }
    m->ctx = ctx;
    m->f32 = arithmetic == B200_DECODER_FP32;
    m->max_slots = max_slots; m->max_seq = max_seq; m->max_rows = max_rows;
    m->Tp = (max_seq + 127) / 128 * 128;
    m->C = m->spec.width; m->Cp = pad_dim(m->C); m->Vp = pad_dim(m->spec.vocab);
    m->slots.assign(max_slots, Slot());
    m->store = new TensorStore();
    *out = m;
    return B200_OK;
}

int b200_decoder_destroy(b200_decoder* m) {
    if (!m) return B200_ERR_NULL;
    b200_device_guard guard(m->ctx);
    cudaStreamSynchronize(m->ctx->stream);
    for (auto& g : m->graphs) cudaGraphExecDestroy(g.second);
    for (cudaEvent_t e : m->ev_pool) cudaEventDestroy(e);
    for (void* p : m->owned) cudaFree(p);
    if (m->logits) cudaFree(m->logits);
    if (m->lat) cudaFree(m->lat);
    if (m->kv) cudaFree(m->kv);
    if (m->gen_log) cudaFree(m->gen_log);
    for (int i = 0; i < b200_decoder::kRing; ++i) {
        if (m->pinned[i]) cudaFreeHost(m->pinned[i]);
        if (m->ring_ev[i]) cudaEventDestroy(m->ring_ev[i]);
    }
    m->ctx->tmap_cache.clear();  // the addresses may come back with other shapes
    delete m->store;
    delete m;
    return B200_OK;
}

int b200_decoder_check_config(const char* config_json, char* message, int message_bytes) {
    if (!config_json) return B200_ERR_NULL;
    if (message && message_bytes > 0) message[0] = 0;
    try {
        parse_config(config_json);
    } catch (const std::exception& e) {
        if (message && message_bytes > 0) snprintf(message, message_bytes, "%s", e.what());
        return B200_ERR_SHAPE;
    }
    return B200_OK;
}

int b200_decoder_vocab(const b200_decoder* m) { return m ? m->spec.vocab : 0; }

int b200_decoder_set_tensor(b200_decoder* m, const char* name, const void* data, int type, const long* shape, int ndim) {
    if (!m || !name || !data || !shape) return B200_ERR_NULL;
    if (type < 0 || type > 2) return B200_ERR_SHAPE;
    if (m->ready) return B200_ERR_STATE;
    m->store->set(name, data, static_cast<TensorType>(type), std::vector<long>(shape, shape + ndim));
    return B200_OK;
}

int b200_decoder_finish_load(b200_decoder* m) {
    if (!m) return B200_ERR_NULL;
    if (m->ready) return B200_ERR_STATE;
    return finish_load(m);
}

int b200_decoder_load_safetensors(b200_decoder* m, const char* path) {
    if (!m || !path) return B200_ERR_NULL;
    if (m->ready) return B200_ERR_STATE;
    try {
        m->store->open_safetensors(path);
    } catch (const std::exception& e) {
        m->ctx->last_error = e.what();
        return B200_ERR_STATE;
    }
    return finish_load(m);
}

int b200_decoder_set_graph(b200_decoder* m, int use_graph) {
    if (!m) return B200_ERR_NULL;
    m->use_graph = use_graph != 0;
    return B200_OK;
}

int b200_decoder_open(b200_decoder* m, int* slot) {
    if (!m || !slot) return B200_ERR_NULL;
    for (int i = 0; i < m->max_slots; ++i)
        if (!m->slots[i].open) {
            m->slots[i] = Slot();
            m->slots[i].open = true;
            *slot = i;
            return B200_OK;
        }
    m->ctx->last_error = "no free slot";
    return B200_ERR_LIMIT;
}

int b200_decoder_close(b200_decoder* m, int slot) {
    if (!m) return B200_ERR_NULL;
    if (slot < 0 || slot >= m->max_slots || !m->slots[slot].open) return B200_ERR_STATE;
    m->slots[slot].open = false;
    return B200_OK;
}

int b200_decoder_length(const b200_decoder* m, int slot) {
    return (m && slot >= 0 && slot < m->max_slots && m->slots[slot].open) ? m->slots[slot].len : -1;
}

int b200_decoder_step(b200_decoder* m, int n_entries, const int* slots, const int* counts, const int* tokens, int n_want, const int* want_rows,
                      float* logits_host) {
    if (!m || !slots || !counts || !tokens) return B200_ERR_NULL;
    if (n_want < 0 || (n_want > 0 && !want_rows)) return B200_ERR_NULL;
    if (!m->ready) return B200_ERR_STATE;
    b200_ctx* ctx = m->ctx;
    if (n_entries < 1 || n_entries > m->max_slots) return B200_ERR_SHAPE;
    long total = 0;
    bool single = true;
    std::vector<char> seen(m->max_slots, 0);
    for (int i = 0; i < n_entries; ++i) {
        const int s = slots[i];
        if (s < 0 || s >= m->max_slots || !m->slots[s].open || seen[s]) { ctx->last_error = "step: slot not open, or named twice"; return B200_ERR_STATE; }
        seen[s] = 1;
        if (counts[i] < 1) { ctx->last_error = "step: an entry without tokens"; return B200_ERR_SHAPE; }
        if ((long)m->slots[s].len + counts[i] > m->max_seq) { ctx->last_error = "step: sequence beyond max_seq"; return B200_ERR_LIMIT; }
        total += counts[i];
        single = single && counts[i] == 1;
    }
    for (long i = 0; i < total; ++i)
        if (tokens[i] < 0 || tokens[i] >= m->spec.vocab) { ctx->last_error = "step: token id outside the vocabulary"; return B200_ERR_SHAPE; }
    for (int i = 0; i < n_want; ++i)
        if (want_rows[i] < 0 || want_rows[i] >= total) { ctx->last_error = "step: wanted row outside the step"; return B200_ERR_SHAPE; }
    b200_device_guard guard(ctx);
    const size_t V = m->spec.vocab;
    if (single && !m->f32 && n_entries <= 16) {
        TRY(decode_step(m, std::vector<int>(slots, slots + n_entries), tokens));
        if (logits_host)
            for (int i = 0; i < n_want; ++i)
                B200_CUDA(ctx, cudaMemcpyAsync(logits_host + i * V, m->dlogits + (size_t)want_rows[i] * m->Vp, V * 4, cudaMemcpyDeviceToHost, ctx->stream));
        return b200_ctx_sync_check(ctx);
    }
    // more rows than the activation buffers hold: in portions, each with its share of the wanted rows
    std::vector<int> done(n_entries, 0), row0(n_entries, 0);
    for (int i = 1; i < n_entries; ++i) row0[i] = row0[i - 1] + counts[i - 1];
    int first = 0;
    while (first < n_entries) {
        std::vector<Entry> part;
        std::vector<int> rows_of;  // the step's row of every row of this portion
        int room = m->max_rows;
        for (int i = first; i < n_entries && room > 0; ++i) {
            const int left = counts[i] - done[i], n = left < room ? left : room;
            if (n == 0) continue;
            part.push_back({slots[i], tokens + row0[i] + done[i], n});
            for (int t = 0; t < n; ++t) rows_of.push_back(row0[i] + done[i] + t);
            done[i] += n;
            room -= n;
        }
        while (first < n_entries && done[first] == counts[first]) ++first;
        std::vector<int> want, dst;
        std::map<int, int> at;
        if (n_want > 0) for (size_t r = 0; r < rows_of.size(); ++r) at[rows_of[r]] = (int)r;
        for (int i = 0; i < n_want; ++i) {
            auto it = at.find(want_rows[i]);
            if (it != at.end()) { want.push_back(it->second); dst.push_back(i); }
        }
        // the logits' product takes as many rows as the activation buffers hold
        std::vector<int> head(want.begin(), want.size() > (size_t)m->max_rows ? want.begin() + m->max_rows : want.end());
        if (head.size() < want.size()) { ctx->last_error = "step: more wanted rows than max_rows"; return B200_ERR_LIMIT; }
        TRY(general_step(m, part, want));
        if (logits_host)
            for (size_t i = 0; i < dst.size(); ++i)
                B200_CUDA(ctx, cudaMemcpyAsync(logits_host + dst[i] * V, m->logits + i * m->Vp, V * 4, cudaMemcpyDeviceToHost, ctx->stream));
    }
    return b200_ctx_sync_check(ctx);
}

int b200_decoder_decode_device(b200_decoder* m, int n, const int* slots) {
    if (!m || !slots) return B200_ERR_NULL;
    if (!m->ready || m->f32) return B200_ERR_STATE;
    if (n < 1 || n > 16 || n > m->max_slots) return B200_ERR_SHAPE;
    for (int i = 0; i < n; ++i) {
        if (slots[i] < 0 || slots[i] >= m->max_slots || !m->slots[slots[i]].open) return B200_ERR_STATE;
        if (m->slots[slots[i]].len + 1 > m->max_seq) return B200_ERR_LIMIT;
    }
    b200_device_guard guard(m->ctx);
    return decode_step(m, std::vector<int>(slots, slots + n), nullptr);
}

int b200_decoder_prefill_device(b200_decoder* m, int n_entries, const int* slots, const int* counts, const int* tokens, int n_want, const int* want_rows) {
    if (!m || !slots || !counts || !tokens || (n_want > 0 && !want_rows)) return B200_ERR_NULL;
    if (!m->ready) return B200_ERR_STATE;
    long total = 0;
    std::vector<Entry> e;
    for (int i = 0; i < n_entries; ++i) {
        if (slots[i] < 0 || slots[i] >= m->max_slots || !m->slots[slots[i]].open || counts[i] < 1) return B200_ERR_STATE;
        if (m->slots[slots[i]].len + counts[i] > m->max_seq) return B200_ERR_LIMIT;
        e.push_back({slots[i], tokens + total, counts[i]});
        total += counts[i];
    }
    if (n_entries < 1 || n_entries > m->max_slots || total > m->max_rows || n_want > m->max_rows) return B200_ERR_LIMIT;
    for (int i = 0; i < n_want; ++i)
        if (want_rows[i] < 0 || want_rows[i] >= total) return B200_ERR_SHAPE;
    b200_device_guard guard(m->ctx);
    return general_step(m, e, std::vector<int>(want_rows, want_rows + n_want));
}

// Requests of unequal lengths, greedy (temperature <= 0) or sampled.  As many requests as there are slots (at most
// 16) are active; a request that has its n_new tokens makes room for the next one.
int b200_decoder_generate(b200_decoder* m, int n_req, const int* const* prompts, const int* lens, int n_new, float temperature, int top_k, float top_p,
                          unsigned int seed, int* out_host) {
    if (!m || !prompts || !lens || !out_host) return B200_ERR_NULL;
    if (!m->ready) return B200_ERR_STATE;
    if (n_req < 1 || n_new < 1 || top_k < 0) return B200_ERR_SHAPE;
    b200_ctx* ctx = m->ctx;
    for (int r = 0; r < n_req; ++r) {
        if (lens[r] < 1) return B200_ERR_SHAPE;
        if ((long)lens[r] + n_new - 1 > m->max_seq) { ctx->last_error = "generate: prompt and continuation beyond max_seq"; return B200_ERR_LIMIT; }
        for (int t = 0; t < lens[r]; ++t)
            if (prompts[r][t] < 0 || prompts[r][t] >= m->spec.vocab) { ctx->last_error = "generate: token id outside the vocabulary"; return B200_ERR_SHAPE; }
    }
    b200_device_guard guard(ctx);
    // sampled ids: [request][n_new] on the device; the current id of every active sequence in dtokens
    const size_t log_ints = (size_t)n_req * n_new;
    if (log_ints > m->gen_log_ints) {
        B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        if (m->gen_log) cudaFree(m->gen_log);
        m->gen_log = nullptr;
        m->gen_log_ints = 0;
        B200_CUDA(ctx, cudaMalloc(&m->gen_log, log_ints * 4));
        m->gen_log_ints = log_ints;
    }
    struct Active { int req, slot, produced; };
    std::vector<Active> act;
    std::vector<int> opened;  // slots to give back if a step fails
    const int V = m->spec.vocab;
    // the token that will stand at position p of request r uses noise stream p * 4096 + r, whatever else is in the batch
    auto draw = [&](int row, const Active& a, const float* logits) {
        return launch_sample_rows(ctx, m->dtokens + row, logits, 1, V, m->Vp, temperature, seed, (unsigned)(lens[a.req] + a.produced) * 4096u + (unsigned)a.req,
                                  top_k, top_p);
    };
    auto record = [&](int row, Active& a) -> int {
        B200_CUDA(ctx, cudaMemcpyAsync(m->gen_log + (size_t)a.req * n_new + a.produced, m->dtokens + row, 4, cudaMemcpyDeviceToDevice, ctx->stream));
        a.produced++;
        return B200_OK;
    };
    auto retire = [&]() -> int {
        for (size_t i = 0; i < act.size();) {
            if (act[i].produced < n_new) { ++i; continue; }
            b200_decoder_close(m, act[i].slot);
            const size_t last = act.size() - 1;
            if (i != last) {
                B200_CUDA(ctx, cudaMemcpyAsync(m->dtokens + i, m->dtokens + last, 4, cudaMemcpyDeviceToDevice, ctx->stream));
                act[i] = act[last];
            }
            act.pop_back();
        }
        return B200_OK;
    };
    auto run = [&]() -> int {
        int next = 0;
        while (next < n_req || !act.empty()) {
            // admit: the prompts of the new requests, together as far as they fit into a step, longer ones in portions
            std::vector<Active> fresh;
            while (next < n_req && act.size() + fresh.size() < 16) {
                int slot;
                if (b200_decoder_open(m, &slot) != B200_OK) break;
                opened.push_back(slot);
                fresh.push_back({next++, slot, 0});
            }
            if (fresh.empty() && act.empty()) { ctx->last_error = "generate: no free slot"; return B200_ERR_LIMIT; }
            size_t f = 0;
            int fed = 0;  // tokens of request fresh[f] that have been run
            while (f < fresh.size()) {
                std::vector<Entry> part;
                std::vector<int> want;
                std::vector<size_t> ends;
                int room = m->max_rows, row = 0;
                while (f < fresh.size() && room > 0) {
                    const int left = lens[fresh[f].req] - fed, n = left < room ? left : room;
                    part.push_back({fresh[f].slot, prompts[fresh[f].req] + fed, n});
                    row += n;
                    room -= n;
                    if (n < left) { fed += n; break; }
                    want.push_back(row - 1);
                    ends.push_back(f++);
                    fed = 0;
                }
                TRY(general_step(m, part, want));
                for (size_t i = 0; i < ends.size(); ++i) {
                    act.push_back(fresh[ends[i]]);
                    const int r = (int)act.size() - 1;
                    TRY(draw(r, act[r], m->logits + i * m->Vp));
                    TRY(record(r, act[r]));
                }
            }
            TRY(retire());
            if (act.empty()) continue;
            const float* logits = m->dlogits;
            std::vector<int> slots;
            for (const Active& a : act) slots.push_back(a.slot);
            if (!m->f32) {
                TRY(decode_step(m, slots, nullptr));
            } else {  // the general path wants the ids on the host
                std::vector<int> ids(act.size());
                B200_CUDA(ctx, cudaMemcpyAsync(ids.data(), m->dtokens, ids.size() * 4, cudaMemcpyDeviceToHost, ctx->stream));
                B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
                std::vector<Entry> part;
                std::vector<int> want;
                for (size_t i = 0; i < act.size(); ++i) { part.push_back({act[i].slot, &ids[i], 1}); want.push_back((int)i); }
                TRY(general_step(m, part, want));
                logits = m->logits;
            }
            if (temperature <= 0.f) TRY(launch_sample_rows(ctx, m->dtokens, logits, (int)act.size(), V, m->Vp, 0.f, seed, 0u, 0, 0.f));
            else for (size_t i = 0; i < act.size(); ++i) TRY(draw((int)i, act[i], logits + i * m->Vp));
            for (size_t i = 0; i < act.size(); ++i) TRY(record((int)i, act[i]));
            TRY(retire());
        }
        return B200_OK;
    };
    const int st = run();
    for (int s : opened) if (st != B200_OK && m->slots[s].open) b200_decoder_close(m, s);
    if (st != B200_OK) return st;
    B200_CUDA(ctx, cudaMemcpyAsync(out_host, m->gen_log, log_ints * 4, cudaMemcpyDeviceToHost, ctx->stream));
    return b200_ctx_sync_check(ctx);
}

int b200_decoder_set_profile(b200_decoder* m, int enabled) {
    if (!m) return B200_ERR_NULL;
    m->profile = enabled != 0;
    return B200_OK;
}

int b200_decoder_read_profile(b200_decoder* m, int cap, const char** names, double* ms, long* launches, int* count) {
    if (!m || !names || !ms || !launches || !count) return B200_ERR_NULL;
    b200_ctx* ctx = m->ctx;
    B200_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    *count = 0;
    for (size_t i = 0; i < m->ev_name.size(); ++i) {
        float t = 0.f;
        B200_CUDA(ctx, cudaEventElapsedTime(&t, m->ev_pool[2 * i], m->ev_pool[2 * i + 1]));
        int k = 0;
        while (k < *count && strcmp(names[k], m->ev_name[i])) ++k;
        if (k == *count) {
            if (k == cap) continue;
            names[k] = m->ev_name[i];
            ms[k] = 0.0;
            launches[k] = 0;
            ++*count;
        }
        ms[k] += t;
        launches[k]++;
    }
    m->ev_name.clear();
    return B200_OK;
}

}  // extern "C"
