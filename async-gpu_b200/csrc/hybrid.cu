// Hybrid decoders: a stack of layers given one by one in a configuration file, each a sequence mixer with an optional
// gated feed-forward, pre-norm RMS.  The architectures of this family:
//   Vivezen    gated delta rule (decay per head) and latent attention; no positions in the embedding, output tied to
//              the embedding table, tanh-GELU
//   Zufilorn   gated delta rule (decay per key channel), mLSTM and differential attention; learned positions added to
//              the embedding, an output matrix of its own, SiLU, norm weights stored around zero, and several residual
//              streams instead of one
// (any of the mixers is read in either).
//
// Two precisions: bfloat16 (weights and activations between matrix products in bfloat16, the tensor-core
// GEMM with its fused epilogues; norms, angles, scores, softmax, recurrence, state and residual f32) and f32
// (f32 FMA kernels throughout).
#include <algorithm>
#include <cmath>
#include <cstring>
#include <fstream>
#include <map>
#include <sstream>

#include "hybrid.h"
#include "json.h"

namespace {

size_t up(size_t n, size_t m) { return (n + m - 1) / m * m; }

// ---- configuration -----------------------------------------------------------------------------------
struct RotSpec { // angle table of one rotation: frequencies per pair, factor of cos and sin
    std::vector<double> freq;
    double mult = 1.0;
    bool operator==(const RotSpec &o) const { return freq == o.freq && mult == o.mult; }
};

enum MixerType { MIX_DELTA, MIX_LATENT, MIX_MLSTM, MIX_DIFF };

// What an architecture fixes.
struct Traits {
    const char *name;
    int act;               // of the gated feed-forward
    bool tied;             // output matrix = embedding table (else 'head')
    bool norm_from_one;    // norm weights are stored minus one
    bool positions;        // learned position vectors 'pos', max_positions of them
    bool streams;          // residual streams
};
const Traits TRAITS[] = {{"Vivezen", B200NN_ACT_GELU_TANH, true, false, false, false}, {"Zufilorn", B200NN_ACT_SILU, false, true, true, true}};

struct LayerSpec {
    MixerType type;
    int weights = 0; // the layer whose tensors it uses
    DeltaDims delta{};
    LatentDims lat{};
    MlstmDims mlstm{};
    DiffDims diff{};
    int dim = 0;  // differential attention: size of a map's query and key before padding
    int rope = -1, win = -1; // index into HybridConfig::rots / windows
    int ff = 0;              // 0: no feed-forward
};

struct HybridConfig {
    const Traits *traits = nullptr;
    int vocab = 0, width = 0;
    int max_positions = 0, streams = 0; // 0: none
    float eps = 0.0f;
    std::vector<LayerSpec> layers;
    std::vector<RotSpec> rots;
    std::vector<int> windows;
};

struct ConfigReader {
    std::string err;
    bool fail(const std::string &m) {
        if (err.empty()) err = m;
        return false;
    }
    bool num(const JsonValue *o, const char *key, double *v, const std::string &where) {
        const JsonValue *j = o ? o->get(key) : nullptr;
        if (!j || j->kind != JsonValue::Number) return fail("config: " + where + "." + key + " is missing or not a number");
        *v = j->num;
        return true;
    }
    bool pos(const JsonValue *o, const char *key, int *v, const std::string &where) {
        double d;
        if (!num(o, key, &d, where)) return false;
        if (d < 1 || d > 1e9 || d != std::floor(d)) return fail("config: " + where + "." + key + " must be a positive integer");
        *v = (int)d;
        return true;
    }
    bool rot(const JsonValue *o, int dims, const std::string &where, RotSpec *out) {
        double base;
        int n;
        if (!num(o, "base", &base, where) || !pos(o, "dims", &n, where)) return false;
        if (n != dims || n % 2) return fail("config: " + where + ".dims must be the (even) rotated size");
        for (int i = 0; i < n / 2; ++i) out->freq.push_back(std::pow(base, -2.0 * i / n));
        const JsonValue *s = o->get("scaling");
        if (!s || s->kind == JsonValue::Null) return true;
        double factor, original, fast, slow;
        const std::string w = where + ".scaling";
        if (!num(s, "factor", &factor, w) || !num(s, "original", &original, w) || !num(s, "fast", &fast, w) || !num(s, "slow", &slow, w))
            return false;
        // frequencies that turn often over the original length stay, slow ones are divided by the factor, with
        // a linear ramp over the pair indices in between
        auto index_of = [&](double turns) { return n * std::log(original / (2.0 * M_PI * turns)) / (2.0 * std::log(base)); };
        const double lo = std::max(std::floor(index_of(fast)), 0.0), hi = std::min(std::ceil(index_of(slow)), n - 1.0);
        for (int i = 0; i < n / 2; ++i) {
            const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            out->freq[i] = out->freq[i] / factor * ramp + out->freq[i] * (1.0 - ramp);
        }
        out->mult = 0.1 * std::log(factor) + 1.0;
        return true;
    }
    bool layer(const JsonValue &j, int i, HybridConfig *c, LayerSpec *l) {
        const std::string where = "layers[" + std::to_string(i) + "]";
        const JsonValue *t = j.get("type"), *mx = j.get("mixer"), *mlp = j.get("mlp"), *wo = j.get("weights_of");
        if (!t || !mx || mx->kind != JsonValue::Object) return fail("config: " + where + " needs 'type' and 'mixer'");
        l->weights = i;
        if (wo && wo->kind == JsonValue::Number) {
            l->weights = (int)wo->num;
            if (l->weights < 0 || l->weights >= i) return fail("config: " + where + ".weights_of must name an earlier layer");
            l->weights = c->layers[l->weights].weights;
        }
        const std::string w = where + ".mixer";
        if (t->str == "delta" || t->str == "channel_delta") {
            l->type = MIX_DELTA;
            l->delta.channel = t->str == "channel_delta";
            DeltaDims &d = l->delta;
            if (!pos(mx, "heads", &d.heads, w) || !pos(mx, "kv_heads", &d.kv_heads, w) || !pos(mx, "dim", &d.dim, w) ||
                !pos(mx, "vdim", &d.vdim, w) || !pos(mx, "conv", &d.taps, w))
                return false;
            if (d.heads % d.kv_heads) return fail("config: " + w + ".heads must be a multiple of kv_heads");
            d.dim_p = (int)up(d.dim, 16);
            d.vdim_p = (int)up(d.vdim, 16);
            d.eps = c->eps;
        } else if (t->str == "latent_attention") {
            l->type = MIX_LATENT;
            LatentDims &d = l->lat;
            int dim, vdim;
            double scale;
            if (!pos(mx, "heads", &d.heads, w) || !pos(mx, "dim", &dim, w) || !pos(mx, "rot_dim", &d.rot, w) || !pos(mx, "vdim", &vdim, w) ||
                !pos(mx, "kv_rank", &d.rank, w) || !pos(mx, "q_rank", &d.q_rank, w) || !num(mx, "scale", &scale, w))
                return false;
            d.dim_p = (int)up(dim, 16);
            d.vdim_p = (int)up(vdim, 16);
            d.rot_p = (int)up(d.rot, 16);
            d.rank_p = (int)up(d.rank, 16);
            d.q_rank_p = (int)up(d.q_rank, 8);
            d.scale = (float)scale;
            d.eps = c->eps;
            d.window = 0;
            const JsonValue *mask = mx->get("mask");
            if (mask && mask->kind == JsonValue::Object && !pos(mask, "size", &d.window, w + ".mask")) return false;
            l->win = (int)(std::find(c->windows.begin(), c->windows.end(), d.window) - c->windows.begin());
            if (l->win == (int)c->windows.size()) c->windows.push_back(d.window);
            RotSpec r;
            if (!rot(mx->get("rot"), d.rot, w + ".rot", &r)) return false;
            l->rope = (int)(std::find(c->rots.begin(), c->rots.end(), r) - c->rots.begin());
            if (l->rope == (int)c->rots.size()) c->rots.push_back(r);
        } else if (t->str == "mlstm") {
            l->type = MIX_MLSTM;
            MlstmDims &d = l->mlstm;
            double cap;
            if (!pos(mx, "heads", &d.heads, w) || !pos(mx, "dim", &d.dim, w) || !pos(mx, "vdim", &d.vdim, w) || !num(mx, "gate_cap", &cap, w)) return false;
            if (!(cap > 0)) return fail("config: " + w + ".gate_cap must be positive");
            d.dim_p = (int)up(d.dim, 16);
            d.vdim_p = (int)up(d.vdim, 16);
            d.cap = (float)cap;
            d.eps = c->eps;
        } else if (t->str == "attention") {
            l->type = MIX_DIFF;
            DiffDims &d = l->diff;
            double scale, diff, cap = 0.0, coef = 0.0;
            if (!pos(mx, "heads", &d.heads, w) || !pos(mx, "kv_heads", &d.kv_heads, w) || !pos(mx, "dim", &l->dim, w) || !pos(mx, "vdim", &d.vdim, w) ||
                !num(mx, "scale", &scale, w) || !num(mx, "diff", &diff, w))
                return false;
            if (d.heads % d.kv_heads) return fail("config: " + w + ".heads must be a multiple of kv_heads");
            const JsonValue *sc = mx->get("softcap"), *qt = mx->get("q_temp");
            if (sc && sc->kind != JsonValue::Null && !num(mx, "softcap", &cap, w)) return false;
            d.qt_every = 1;
            if (qt && qt->kind == JsonValue::Object && (!num(qt, "coef", &coef, w + ".q_temp") || !pos(qt, "every", &d.qt_every, w + ".q_temp"))) return false;
            d.dim_p = (int)up(l->dim, 16);
            d.vdim_p = (int)up(d.vdim, 16);
            d.scale = (float)scale;
            d.diff = (float)diff;
            d.cap = (float)cap;
            d.qt_coef = (float)coef;
            d.eps = c->eps;
        } else {
            return fail("config: " + where + ".type '" + t->str + "' is not a mixer of this family");
        }
        if (mlp && mlp->kind == JsonValue::Object) {
            const JsonValue *k = mlp->get("kind");
            if (!k || k->str != "dense") return fail("config: " + where + ".mlp.kind must be 'dense'");
            if (!pos(mlp, "ff", &l->ff, where + ".mlp")) return false;
        }
        return true;
    }
    bool read(const JsonValue &root, HybridConfig *c) {
        double eps;
        if (!pos(&root, "vocab", &c->vocab, "") || !pos(&root, "width", &c->width, "") || !num(root.get("norm"), "eps", &eps, "norm"))
            return false;
        c->eps = (float)eps;
        if (c->traits->positions && !pos(&root, "max_positions", &c->max_positions, "")) return false;
        if (c->traits->streams && !pos(&root, "streams", &c->streams, "")) return false;
        if (c->streams > MAX_STREAMS) return fail("config: more than " + std::to_string(MAX_STREAMS) + " residual streams");
        const JsonValue *ls = root.get("layers");
        if (!ls || ls->kind != JsonValue::Array || ls->items.empty()) return fail("config: 'layers' is missing or empty");
        for (size_t i = 0; i < ls->items.size(); ++i) {
            LayerSpec l;
            if (!layer(ls->items[i], (int)i, c, &l)) return false;
            c->layers.push_back(l);
        }
        return true;
    }
};

// ---- weights -----------------------------------------------------------------------------------------
struct TensorView {
    const float *p;
    size_t numel;
};
using TensorMap = std::map<std::string, TensorView>;

// Block-diagonal Linear in either precision.
struct GroupedLinear {
    int groups = 0, Ng = 0, Kg = 0, x_stride = 0, out_stride = 0;
    bool b16 = false;
    B16Weight b;
    std::shared_ptr<DevBuf> f;
};

struct LayerWeights {
    std::shared_ptr<DevBuf> norm1, norm2;
    LinearAny in, o, gu, down;
    // delta
    std::shared_ptr<DevBuf> conv, a_exp, dt_bias, onorm;
    // latent attention
    std::shared_ptr<DevBuf> qnorm, kvnorm;
    LinearAny uq, ukv;             // ukv: keys and values of all heads from latents (bfloat16 models)
    std::shared_ptr<DevBuf> ukv_rows; // the same as [features][rank_p] f32 (f32 models)
    GroupedLinear uk, uv;
    // delta rule with a decay per channel: second step of the decay and gate projections
    GroupedLinear ext;
    // mLSTM (onorm as above)
    std::shared_ptr<DevBuf> i_bias, f_bias;
    float lambda = 0.0f; // differential attention
    std::shared_ptr<DevBuf> hc[2]; // per sublayer: in [n], out [n], mix [n][n]
};

// Row-major host matrix being assembled, zero where nothing is written.
struct HostMat {
    size_t rows, cols;
    std::vector<float> a;
    HostMat(size_t r, size_t c) : rows(r), cols(c), a(r * c, 0.0f) {}
    float *row(size_t r) { return a.data() + r * cols; }
    void put(size_t r, const float *src, size_t n) { std::copy(src, src + n, row(r)); }
};

}  // namespace

struct b200nn_hybrid : b200nn_lm {
    HybridConfig cfg;
    bool b16 = true;
    size_t d = 0, dp = 0, es = 2; // width, width padded to 8, bytes per activation
    std::vector<std::shared_ptr<LayerWeights>> w; // by layer; shared entries for weights_of
    std::shared_ptr<DevBuf> table, pos_table, final_norm; // tables in the activation type, rows dp apart; tied bfloat16 models read lm_head's
    LinearAny lm_head;
    struct Sublayer {
        const float *norm;
        StreamCoef hc;
    };
    std::vector<Sublayer> subs; // every mixer and feed-forward in order (models with residual streams)
    // largest sizes over the layers, for the workspace
    size_t max_proj = 0, max_gate = 0, max_cq = 0, max_q = 0, max_att = 0, max_ff = 0, max_conv = 0, max_heads = 0, max_low = 0, max_ext = 0,
           max_mgate = 0;

    const char *family() const override { return "hybrid"; }
    int vocab() const override { return cfg.vocab; }
    int width() const override { return cfg.width; }
    int n_layer() const override { return (int)cfg.layers.size(); }
    size_t max_positions() const override { return (size_t)cfg.max_positions; }
    int cache_init(size_t batch, size_t cap, b200nn_kvcache *c) override;
    int workspace_init(size_t rows, size_t logit_rows, Workspace *ws) override;
    int pass_prompt(Workspace &ws, b200nn_kvcache &kv, const std::vector<PassEntry> &entries, const uint32_t *ids_host) override;
    int pass_decode(Workspace &ws, b200nn_kvcache &kv, const int *pos_ptr, StepProfile *prof) override;
    int head(Workspace &ws, const float *x, int rows, StepProfile *prof) override;
    int head_pick(Workspace &ws, const float *x, int rows, bool keep_last, bool tokens_only, uint32_t *tok_out,
                  StepProfile *prof) override;

    // one pass over T rows embedded in ws.x
    struct Pass {
        int T = 0;
        bool decode = false;
        RowMap rows;
        const int *row_seq = nullptr;
        std::vector<SeqMap> seqs; // per window
        SeqMap seq;
        StepProfile *prof = nullptr;
    };
    int embed(Workspace &ws, const void *ids, const RowMap &rows, int T);
    int stream_step(Workspace &ws, const Pass &p, size_t done); // streams between sublayers done - 1 and done
    int run_layers(Workspace &ws, b200nn_kvcache &kv, const Pass &p);
    int delta_layer(Workspace &ws, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p);
    int latent_layer(Workspace &ws, b200nn_kvcache &kv, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p);
    int mlstm_layer(Workspace &ws, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p);
    int diff_layer(Workspace &ws, b200nn_kvcache &kv, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p);
    int feed_forward(Workspace &ws, const LayerSpec &l, const LayerWeights &lw, const Pass &p);

    int act_type() const { return b16 ? OUT_BF16 : OUT_F32; }
    int upload_f32(const float *h, size_t n, std::shared_ptr<DevBuf> *out) {
        TRY(dev_alloc(ctx, n * 4, out));
        CK(ctx, cudaMemcpy((*out)->p, h, n * 4, cudaMemcpyHostToDevice));
        return B200NN_OK;
    }
    int linear(HostMat &m, LinearAny *l) {
        l->K = (int)m.cols;
        l->N = (int)m.rows;
        l->b16 = b16;
        if (b16) return b16_weight_upload(ctx, m.a.data(), m.cols, m.rows, &l->b);
        return f32_weight_upload(ctx, m.a.data(), true, nullptr, m.cols, m.rows, &l->f, true);
    }
    int grouped(const std::vector<float> &gnk, int groups, int Ng, int Kg, int x_stride, int out_stride, GroupedLinear *g) {
        g->groups = groups;
        g->Ng = Ng;
        g->Kg = Kg;
        g->x_stride = x_stride;
        g->out_stride = out_stride;
        g->b16 = b16;
        if (b16) return b16_grouped_weight_upload(ctx, gnk.data(), groups, Ng, Kg, x_stride, out_stride, &g->b);
        return upload_f32(gnk.data(), gnk.size(), &g->f);
    }
    int run_grouped(const GroupedLinear &g, const void *x, int ldx, int M, const Epilogue &e) {
        if (g.b16) return launch_b16_linear(ctx, g.b, (const __nv_bfloat16 *)x, ldx, M, e);
        return launch_grouped_f32(ctx, (const float *)g.f->p, g.groups, g.Ng, g.Kg, (const float *)x, ldx, g.x_stride, M, e, g.out_stride);
    }
    int store_linear(const LinearAny &l, const void *x, int M, void *out, int ldo, int out_type, int ldx = 0) {
        Epilogue e;
        e.out = out;
        e.ldo = ldo;
        e.out_half = out_type;
        return linear_forward(ctx, l, x, b16, M, e, ldx);
    }
    // A sublayer's last Linear: into the residual, or to ws.y for the streams' update.
    int out_linear(const LinearAny &l, const void *x, int M, Workspace &ws) {
        if (cfg.streams) return store_linear(l, x, M, ws.y->p, (int)d, OUT_F32);
        Epilogue e;
        e.mode = EPI_RESID;
        e.resid = (float *)ws.x->p;
        e.ldo = (int)d;
        return linear_forward(ctx, l, x, b16, M, e);
    }
    // A buffer of at least `bytes`, zeroed when it is (re)allocated: padding columns are never written and
    // must hold finite values.
    int need(std::shared_ptr<DevBuf> *b, size_t bytes) {
        if (*b && (*b)->bytes >= bytes) return B200NN_OK;
        if (ctx->capturing) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "activation buffer cannot grow during graph capture");
        b->reset();
        TRY(dev_alloc(ctx, bytes, b));
        CK(ctx, cudaMemsetAsync((*b)->p, 0, (*b)->bytes, ctx->stream));
        return B200NN_OK;
    }
    int build(const TensorMap &t);
    // A norm's weight as the kernels multiply with it.
    int norm_weight(const TensorMap &t, const std::string &name, std::shared_ptr<DevBuf> *out) {
        const float *n;
        TRY(take(t, name, d, &n));
        std::vector<float> v(n, n + d);
        if (cfg.traits->norm_from_one)
            for (float &x : v) x += 1.0f;
        return upload_f32(v.data(), d, out);
    }
    // [rows][dp] in the activation type
    int upload_table(const HostMat &m, std::shared_ptr<DevBuf> *out) {
        if (!b16) return upload_f32(m.a.data(), m.a.size(), out);
        B16Weight w;
        TRY(b16_weight_upload(ctx, m.a.data(), m.cols, m.rows, &w));
        *out = w.w_nk;
        return B200NN_OK;
    }
    int table_of(const TensorMap &t, const std::string &name, size_t rows, HostMat *m) {
        const float *e;
        TRY(take(t, name, rows * d, &e));
        for (size_t r = 0; r < rows; ++r) m->put(r, e + r * d, d);
        return B200NN_OK;
    }
    int build_mlstm(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw);
    int build_diff(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw);
    int build_delta(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw);
    int build_latent(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw);
    size_t rows_of(const TensorMap &t, const std::string &name) { // rows of a [., width] matrix; 0: absent or of another width
        auto it = t.find(name);
        return it == t.end() || it->second.numel % d ? 0 : it->second.numel / d;
    }
    int take(const TensorMap &t, const std::string &name, size_t numel, const float **out) {
        auto it = t.find(name);
        if (it == t.end()) return set_error(ctx, B200NN_ERR_MISSING, "missing tensor " + name);
        if (it->second.numel != numel)
            return set_error(ctx, B200NN_ERR_SHAPE, "tensor " + name + ": expected " + std::to_string(numel) + " elements, got " +
                                                        std::to_string(it->second.numel));
        *out = it->second.p;
        return B200NN_OK;
    }
};

int b200nn_hybrid::build_delta(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw) {
    const DeltaDims &D = l.delta;
    const size_t KH = D.kv_heads, H = D.heads;
    HostMat in(D.proj_w(), dp), conv(D.taps, D.conv_w());
    struct Part { const char *name; size_t heads, dim, dim_p, at; bool conv; };
    const int C = D.channel;
    std::vector<Part> parts = {{"q", KH, (size_t)D.dim, (size_t)D.dim_p, (size_t)D.q_at(), true},
                               {"k", KH, (size_t)D.dim, (size_t)D.dim_p, (size_t)D.k_at(), true},
                               {"v", H, (size_t)D.vdim, (size_t)D.vdim_p, (size_t)D.v_at(), true},
                               {"b", H, 1, 1, (size_t)D.b_at(), false}};
    const size_t ra = C ? rows_of(t, p + "a1") : 0, rg = C ? rows_of(t, p + "g1") : 0; // inner sizes of the two-step projections
    if (C) {
        parts.push_back({"a1", 1, ra, ra, (size_t)D.low_at(), false});
        parts.push_back({"g1", 1, rg, rg, (size_t)(D.low_at() + D.low), false});
    } else {
        parts.push_back({"g", H, (size_t)D.vdim, (size_t)D.vdim_p, (size_t)D.g_at(), false});
        parts.push_back({"a", H, 1, 1, (size_t)D.a_at(), false});
    }
    for (const Part &q : parts) {
        const float *m, *c = nullptr;
        TRY(take(t, p + q.name, q.heads * q.dim * d, &m));
        if (q.conv) TRY(take(t, p + q.name + ".conv", q.heads * q.dim * D.taps, &c));
        for (size_t h = 0; h < q.heads; ++h)
            for (size_t j = 0; j < q.dim; ++j) {
                in.put(q.at + h * q.dim_p + j, m + (h * q.dim + j) * d, d);
                for (int t = 0; c && t < D.taps; ++t) conv.row(t)[q.at + h * q.dim_p + j] = c[(h * q.dim + j) * D.taps + t];
            }
    }
    TRY(linear(in, &lw->in));
    TRY(upload_f32(conv.a.data(), conv.a.size(), &lw->conv));
    const float *a, *b, *n, *o;
    TRY(take(t, p + "A_log", H, &a));
    TRY(take(t, p + "dt_bias", C ? H * D.dim : H, &b));
    TRY(take(t, p + "norm", D.vdim, &n));
    TRY(take(t, p + "o", d * H * D.vdim, &o));
    std::vector<float> ae(H);
    for (size_t h = 0; h < H; ++h) ae[h] = (float)std::exp((double)a[h]);
    TRY(upload_f32(ae.data(), H, &lw->a_exp));
    std::vector<float> bias(D.decays(), 0.0f);
    if (!C) std::copy(b, b + H, bias.begin());
    else {
        for (size_t h = 0; h < H; ++h) std::copy_n(b + h * D.dim, D.dim, bias.begin() + h * D.dim_p);
        const size_t E = D.ext(), L = D.low;
        const float *a2, *g2;
        TRY(take(t, p + "a2", H * D.dim * ra, &a2));
        TRY(take(t, p + "g2", H * D.vdim * rg, &g2));
        std::vector<float> m(2 * E * L, 0.0f);
        for (size_t h = 0; h < H; ++h) {
            for (int j = 0; j < D.dim; ++j) std::copy_n(a2 + (h * D.dim + j) * ra, ra, m.begin() + (h * D.dim_p + j) * L);
            for (int j = 0; j < D.vdim; ++j) std::copy_n(g2 + (h * D.vdim + j) * rg, rg, m.begin() + (E + h * D.vdim_p + j) * L);
        }
        TRY(grouped(m, 2, (int)E, (int)L, (int)L, (int)E, &lw->ext));
    }
    TRY(upload_f32(bias.data(), bias.size(), &lw->dt_bias));
    TRY(upload_f32(n, D.vdim, &lw->onorm));
    HostMat om(d, H * D.vdim_p);
    for (size_t r = 0; r < d; ++r)
        for (size_t h = 0; h < H; ++h) std::copy_n(o + (r * H + h) * D.vdim, D.vdim, om.row(r) + h * D.vdim_p);
    return linear(om, &lw->o);
}

int b200nn_hybrid::build_mlstm(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw) {
    const MlstmDims &D = l.mlstm;
    const size_t H = D.heads;
    HostMat in(D.proj_w(), dp);
    struct Part { const char *name; size_t dim, dim_p, at; };
    const Part parts[] = {{"q", (size_t)D.dim, (size_t)D.dim_p, (size_t)D.q_at()},    {"k", (size_t)D.dim, (size_t)D.dim_p, (size_t)D.k_at()},
                          {"v", (size_t)D.vdim, (size_t)D.vdim_p, (size_t)D.v_at()}, {"g", (size_t)D.vdim, (size_t)D.vdim_p, (size_t)D.g_at()},
                          {"i", 1, 1, (size_t)D.i_at()},                             {"f", 1, 1, (size_t)D.f_at()}};
    for (const Part &q : parts) {
        const float *m;
        TRY(take(t, p + q.name, H * q.dim * d, &m));
        for (size_t h = 0; h < H; ++h)
            for (size_t j = 0; j < q.dim; ++j) in.put(q.at + h * q.dim_p + j, m + (h * q.dim + j) * d, d);
    }
    TRY(linear(in, &lw->in));
    const float *ib, *fb, *n, *o;
    TRY(take(t, p + "i.b", H, &ib));
    TRY(take(t, p + "f.b", H, &fb));
    TRY(take(t, p + "norm", H * D.vdim, &n));
    TRY(take(t, p + "o", d * H * D.vdim, &o));
    TRY(upload_f32(ib, H, &lw->i_bias));
    TRY(upload_f32(fb, H, &lw->f_bias));
    std::vector<float> nw(H * D.vdim_p, 0.0f);
    for (size_t h = 0; h < H; ++h) std::copy_n(n + h * D.vdim, D.vdim, nw.begin() + h * D.vdim_p);
    TRY(upload_f32(nw.data(), nw.size(), &lw->onorm));
    HostMat om(d, H * D.vdim_p);
    for (size_t r = 0; r < d; ++r)
        for (size_t h = 0; h < H; ++h) std::copy_n(o + (r * H + h) * D.vdim, D.vdim, om.row(r) + h * D.vdim_p);
    return linear(om, &lw->o);
}

int b200nn_hybrid::build_diff(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw) {
    const DiffDims &D = l.diff;
    const size_t H = D.heads, G = D.kv_heads, dim = l.dim, kw = D.kv_w(), kv_at = D.q_w(), g_at = kv_at + D.cache_w();
    const float *q, *k, *v, *g, *o, *lam[4];
    TRY(take(t, p + "q", H * 2 * dim * d, &q));
    TRY(take(t, p + "k", G * 2 * dim * d, &k));
    TRY(take(t, p + "v", G * D.vdim * d, &v));
    TRY(take(t, p + "g", H * d, &g));
    TRY(take(t, p + "o", d * H * D.vdim, &o));
    const char *const names[] = {"lq1", "lk1", "lq2", "lk2"};
    for (int i = 0; i < 4; ++i) TRY(take(t, p + names[i], dim, &lam[i]));
    double dot[2] = {0.0, 0.0};
    for (size_t j = 0; j < dim; ++j)
        for (int x = 0; x < 2; ++x) dot[x] += (double)lam[2 * x][j] * lam[2 * x + 1][j];
    lw->lambda = (float)(std::exp(dot[0]) - std::exp(dot[1]) + D.diff);
    // queries, then per key / value head a cache row's columns, then the gates
    HostMat in(g_at + H, dp);
    for (size_t h = 0; h < 2 * H; ++h) // heads of both maps
        for (size_t j = 0; j < dim; ++j) in.put(h * D.dim_p + j, q + (h * dim + j) * d, d);
    for (size_t h = 0; h < G; ++h) {
        for (size_t x = 0; x < 2; ++x)
            for (size_t j = 0; j < dim; ++j) in.put(kv_at + h * kw + x * D.dim_p + j, k + ((h * 2 + x) * dim + j) * d, d);
        for (int j = 0; j < D.vdim; ++j) in.put(kv_at + h * kw + 2 * D.dim_p + j, v + (h * D.vdim + j) * d, d);
    }
    for (size_t h = 0; h < H; ++h) in.put(g_at + h, g + h * d, d);
    TRY(linear(in, &lw->in));
    HostMat om(d, H * D.vdim_p);
    for (size_t r = 0; r < d; ++r)
        for (size_t h = 0; h < H; ++h) std::copy_n(o + (r * H + h) * D.vdim, D.vdim, om.row(r) + h * D.vdim_p);
    return linear(om, &lw->o);
}

int b200nn_hybrid::build_latent(const std::string &p, const LayerSpec &l, const TensorMap &t, LayerWeights *lw) {
    const LatentDims &L = l.lat;
    const size_t H = L.heads, R = L.rank, Q = L.q_rank, rd = L.rot, half = rd / 2;
    // sizes before padding: from the tensors themselves, checked against the padded ones
    auto numel = [&](const char *n) { auto it = t.find(p + n); return it == t.end() ? (size_t)0 : it->second.numel; };
    const size_t dim = numel("uk") / (H * R), vdim = numel("uv") / (H * R);
    if (up(dim, 16) != (size_t)L.dim_p || up(vdim, 16) != (size_t)L.vdim_p)
        return set_error(ctx, numel("uk") && numel("uv") ? B200NN_ERR_SHAPE : B200NN_ERR_MISSING, "tensors " + p + "uk / uv do not fit the configuration");
    const float *dq, *dqn, *uq, *dkv, *dkvn, *uk, *uv, *g, *o;
    TRY(take(t, p + "dq", Q * d, &dq));
    TRY(take(t, p + "dq.norm", Q, &dqn));
    TRY(take(t, p + "uq", H * (dim + rd) * Q, &uq));
    TRY(take(t, p + "dkv", (R + rd) * d, &dkv));
    TRY(take(t, p + "dkv.norm", R, &dkvn));
    TRY(take(t, p + "uk", H * dim * R, &uk));
    TRY(take(t, p + "uv", H * vdim * R, &uv));
    TRY(take(t, p + "g", H * d, &g));
    TRY(take(t, p + "o", d * H * vdim, &o));
    HostMat in(Q + R + rd + H, dp);
    for (size_t r = 0; r < Q; ++r) in.put(r, dq + r * d, d);
    for (size_t r = 0; r < R + rd; ++r) in.put(Q + r, dkv + r * d, d);
    for (size_t r = 0; r < H; ++r) in.put(Q + R + rd + r, g + r * d, d);
    TRY(linear(in, &lw->in));
    TRY(upload_f32(dqn, Q, &lw->qnorm));
    TRY(upload_f32(dkvn, R, &lw->kvnorm));
    // query rows: rotated entries i and i + half side by side (the key part is stored in the same order)
    const size_t hw = L.head_w();
    HostMat uqm(H * hw, L.q_rank_p);
    for (size_t h = 0; h < H; ++h) {
        for (size_t j = 0; j < dim; ++j) uqm.put(h * hw + j, uq + (h * (dim + rd) + j) * Q, Q);
        for (size_t j = 0; j < rd; ++j) {
            const size_t to = j < half ? 2 * j : 2 * (j - half) + 1;
            uqm.put(h * hw + L.dim_p + to, uq + (h * (dim + rd) + dim + j) * Q, Q);
        }
    }
    TRY(linear(uqm, &lw->uq));
    HostMat kv(L.kv_w(), L.rank_p);
    std::vector<float> ukt(H * L.rank_p * L.dim_p, 0.0f), uvm(H * L.vdim_p * L.rank_p, 0.0f);
    for (size_t h = 0; h < H; ++h) {
        for (size_t j = 0; j < dim; ++j) {
            const float *s = uk + (h * dim + j) * R;
            kv.put(h * L.dim_p + j, s, R);
            for (size_t r = 0; r < R; ++r) ukt[(h * L.rank_p + r) * L.dim_p + j] = s[r];
        }
        for (size_t j = 0; j < vdim; ++j) {
            const float *s = uv + (h * vdim + j) * R;
            kv.put(H * L.dim_p + h * L.vdim_p + j, s, R);
            std::copy_n(s, R, uvm.begin() + (h * L.vdim_p + j) * L.rank_p);
        }
    }
    if (b16) TRY(linear(kv, &lw->ukv));
    else TRY(upload_f32(kv.a.data(), kv.a.size(), &lw->ukv_rows));
    TRY(grouped(ukt, (int)H, L.rank_p, L.dim_p, (int)hw, L.rank_p, &lw->uk));
    TRY(grouped(uvm, (int)H, L.vdim_p, L.rank_p, L.rank_p, L.vdim_p, &lw->uv));
    HostMat om(d, H * L.vdim_p);
    for (size_t r = 0; r < d; ++r)
        for (size_t h = 0; h < H; ++h) std::copy_n(o + (r * H + h) * vdim, vdim, om.row(r) + h * L.vdim_p);
    return linear(om, &lw->o);
}

int b200nn_hybrid::build(const TensorMap &t) {
    d = cfg.width;
    dp = up(d, 8);
    es = b16 ? 2 : 4;
    TRY(norm_weight(t, "final.norm", &final_norm));
    HostMat em(cfg.vocab, dp);
    TRY(table_of(t, "embed", cfg.vocab, &em));
    if (cfg.traits->tied) TRY(linear(em, &lm_head));
    if (!cfg.traits->tied || !b16) TRY(upload_table(em, &table));
    if (!cfg.traits->tied) {
        TRY(table_of(t, "head", cfg.vocab, &em));
        TRY(linear(em, &lm_head));
    }
    if (cfg.max_positions) {
        HostMat pm(cfg.max_positions, dp);
        TRY(table_of(t, "pos", cfg.max_positions, &pm));
        TRY(upload_table(pm, &pos_table));
    }
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
        LayerSpec &l = cfg.layers[i];
        if (l.type == MIX_DELTA) {
            if (l.delta.channel) {
                const std::string m = "l" + std::to_string(l.weights) + ".mix.";
                const size_t ra = rows_of(t, m + "a1"), rg = rows_of(t, m + "g1");
                if (!ra || !rg) return set_error(ctx, B200NN_ERR_MISSING, "tensors " + m + "a1 / g1 are missing or do not fit the width");
                l.delta.low = (int)up(std::max(ra, rg), 16);
                max_low = std::max(max_low, (size_t)2 * l.delta.low);
                max_ext = std::max(max_ext, (size_t)2 * l.delta.ext());
            }
            max_proj = std::max(max_proj, (size_t)l.delta.proj_w());
            max_att = std::max(max_att, (size_t)l.delta.heads * l.delta.vdim_p);
            max_conv = std::max(max_conv, (size_t)l.delta.conv_ld());
            max_heads = std::max(max_heads, (size_t)l.delta.heads * l.delta.vdim_p);
        } else if (l.type == MIX_LATENT) {
            max_proj = std::max(max_proj, up((size_t)l.lat.q_rank + l.lat.rank + l.lat.rot + l.lat.heads, 4));
            max_att = std::max(max_att, (size_t)l.lat.heads * l.lat.vdim_p);
            max_gate = std::max(max_gate, (size_t)l.lat.heads);
            max_cq = std::max(max_cq, (size_t)l.lat.q_rank_p);
            max_q = std::max(max_q, (size_t)l.lat.heads * l.lat.head_w());
        } else if (l.type == MIX_MLSTM) {
            max_proj = std::max(max_proj, (size_t)l.mlstm.proj_w());
            max_att = std::max(max_att, (size_t)l.mlstm.heads * l.mlstm.vdim_p);
            max_heads = std::max(max_heads, (size_t)l.mlstm.heads * l.mlstm.vdim_p);
            max_mgate = std::max(max_mgate, (size_t)l.mlstm.heads * 4);
        } else {
            max_att = std::max(max_att, (size_t)l.diff.heads * l.diff.vdim_p);
            if (b16) {
                max_gate = std::max(max_gate, (size_t)l.diff.heads);
                max_q = std::max(max_q, (size_t)l.diff.q_w());
            } else {
                max_proj = std::max(max_proj, up((size_t)l.diff.q_w() + l.diff.cache_w() + l.diff.heads, 4));
            }
        }
        max_ff = std::max(max_ff, up(l.ff, 8));
        if (l.weights != (int)i) { // the rest of its entry must describe the tensors it shares
            if (cfg.layers[l.weights].type != l.type || cfg.layers[l.weights].ff != l.ff)
                return set_error(ctx, B200NN_ERR_SHAPE, "config: layer " + std::to_string(i) + " differs from the layer whose weights it uses");
            w.push_back(w[l.weights]);
            continue;
        }
        auto lw = std::make_shared<LayerWeights>();
        const std::string p = "l" + std::to_string(i) + ".";
        TRY(norm_weight(t, p + "norm1", &lw->norm1));
        for (int q = 0; cfg.streams && q < (l.ff ? 2 : 1); ++q) {
            const size_t S = cfg.streams;
            const std::string hc = p + "hc" + std::to_string(q + 1) + ".";
            const float *ci, *co, *mx;
            TRY(take(t, hc + "in", S, &ci));
            TRY(take(t, hc + "out", S, &co));
            TRY(take(t, hc + "mix", S * S, &mx));
            std::vector<float> v(ci, ci + S);
            v.insert(v.end(), co, co + S);
            v.insert(v.end(), mx, mx + S * S);
            TRY(upload_f32(v.data(), v.size(), &lw->hc[q]));
        }
        if (l.type == MIX_DELTA) TRY(build_delta(p + "mix.", l, t, lw.get()));
        else if (l.type == MIX_MLSTM) TRY(build_mlstm(p + "mix.", l, t, lw.get()));
        else if (l.type == MIX_DIFF) TRY(build_diff(p + "mix.", l, t, lw.get()));
        else TRY(build_latent(p + "mix.", l, t, lw.get()));
        if (l.ff) {
            const size_t ff = l.ff, ffp = up(ff, 8);
            const float *g, *u, *dn;
            TRY(norm_weight(t, p + "norm2", &lw->norm2));
            TRY(take(t, p + "mlp.gate", ff * d, &g));
            TRY(take(t, p + "mlp.up", ff * d, &u));
            TRY(take(t, p + "mlp.down", d * ff, &dn));
            HostMat gu(2 * ffp, dp), dm(d, ffp); // rows in fours: two gates, their two ups
            for (size_t j = 0; j < ff; ++j) {
                gu.put((j >> 1) * 4 + (j & 1), g + j * d, d);
                gu.put((j >> 1) * 4 + 2 + (j & 1), u + j * d, d);
            }
            for (size_t r = 0; r < d; ++r) dm.put(r, dn + r * ff, ff);
            TRY(linear(gu, &lw->gu));
            TRY(linear(dm, &lw->down));
        }
        w.push_back(lw);
    }
    for (size_t i = 0; cfg.streams && i < w.size(); ++i)
        for (int q = 0; q < (cfg.layers[i].ff ? 2 : 1); ++q) {
            const float *c = (const float *)w[i]->hc[q]->p;
            subs.push_back(Sublayer{(const float *)(q ? w[i]->norm2 : w[i]->norm1)->p, StreamCoef{c, c + cfg.streams, c + 2 * cfg.streams}});
        }
    return B200NN_OK;
}

// ---- cache and workspace -----------------------------------------------------------------------------
__global__ void rope_table_kernel(const double *__restrict__ freq, int pairs, double mult, int cap, float2 *__restrict__ out) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)cap * pairs) return;
    double s, c;
    sincos((double)(i / pairs) * freq[i % pairs], &s, &c);
    out[i] = make_float2((float)(c * mult), (float)(s * mult));
}

int b200nn_hybrid::cache_init(size_t batch, size_t cap, b200nn_kvcache *c) {
    if (cfg.max_positions && cap > (size_t)cfg.max_positions)
        return set_error(ctx, B200NN_ERR_DIM, "KvCache: capacity beyond the model's " + std::to_string(cfg.max_positions) + " positions");
    c->portion = std::min(cap, (size_t)(ctx->lm_portion > 0 ? ctx->lm_portion : 2048));
    auto zeroed = [&](size_t bytes, std::shared_ptr<DevBuf> *b) -> int {
        TRY(dev_alloc(ctx, bytes, b));
        CK(ctx, cudaMemsetAsync((*b)->p, 0, bytes, ctx->stream));
        return B200NN_OK;
    };
    for (const RotSpec &r : cfg.rots) {
        std::shared_ptr<DevBuf> f, t;
        const int pairs = (int)r.freq.size();
        TRY(dev_alloc(ctx, pairs * sizeof(double), &f));
        CK(ctx, cudaMemcpy(f->p, r.freq.data(), pairs * sizeof(double), cudaMemcpyHostToDevice));
        TRY(dev_alloc(ctx, cap * pairs * sizeof(float2), &t));
        rope_table_kernel<<<(unsigned)((cap * pairs + 255) / 256), 256, 0, ctx->stream>>>((const double *)f->p, pairs, r.mult, (int)cap, (float2 *)t->p);
        CK_LAUNCH(ctx, "rope_table_kernel");
        CK(ctx, cudaStreamSynchronize(ctx->stream)); // f goes out of scope
        c->rope.push_back(t);
    }
    for (const LayerSpec &l : cfg.layers) {
        LayerState st;
        if (l.type == MIX_LATENT) {
            size_t ring = up(cap, 128);
            if (l.lat.window) ring = std::min(ring, up(l.lat.window - 1 + c->portion, 128));
            st.ring = (int)ring;
            TRY(zeroed(batch * ring * l.lat.ld() * es, &st.latent));
        } else if (l.type == MIX_DIFF) {
            TRY(zeroed(batch * cap * l.diff.cache_w() * es, &st.kv));
        } else if (l.type == MIX_MLSTM) {
            TRY(zeroed(batch * l.mlstm.heads * l.mlstm.dim_p * l.mlstm.vdim_p * 4, &st.state));
            TRY(zeroed(batch * l.mlstm.heads * l.mlstm.dim_p * 4, &st.normaliser));
            TRY(zeroed(batch * l.mlstm.heads * 4, &st.maximum));
        } else {
            TRY(zeroed(batch * l.delta.heads * l.delta.dim_p * l.delta.vdim_p * 4, &st.state));
            TRY(zeroed(batch * l.delta.taps * l.delta.conv_w() * 4, &st.conv));
        }
        c->layers.push_back(st);
    }
    return B200NN_OK;
}

int b200nn_hybrid::workspace_init(size_t rows, size_t logit_rows, Workspace *ws) {
    ws->rows = rows;
    ws->logit_rows = logit_rows;
    const size_t V = cfg.vocab, R = std::max<size_t>(rows, 1), LR = std::max<size_t>(logit_rows, 1);
    TRY(need(&ws->x, R * d * 4));
    TRY(need(&ws->ln, R * dp * es));
    TRY(need(&ws->proj, R * std::max(max_proj, b16 ? 0 : 2 * max_ff) * 4)); // f32 models: gate and up before their product
    TRY(need(&ws->att, R * max_att * es));
    if (max_gate) TRY(need(&ws->gate, R * max_gate * 4));
    if (max_cq) TRY(need(&ws->cq, R * max_cq * es));
    if (max_q) TRY(need(&ws->q, R * max_q * es));
    if (max_low && b16) TRY(need(&ws->low, R * max_low * es));
    if (max_ext) TRY(need(&ws->ext, R * max_ext * 4));
    if (cfg.streams) {
        TRY(need(&ws->xs, R * cfg.streams * d * 4));
        TRY(need(&ws->y, R * d * 4));
    }
    if (max_ff) TRY(need(&ws->fc, R * max_ff * es));
    TRY(need(&ws->last_x, LR * d * 4));
    TRY(need(&ws->last_ln, LR * dp * es));
    TRY(need(&ws->logits, LR * V * 4));
    TRY(need(&ws->ids, R * 4));
    TRY(need(&ws->tok, std::max(R, LR) * 4));
    ws->amax_entries = (int)((V + 127) / 128) * 4;
    TRY(need(&ws->amax_val, LR * ws->amax_entries * 4));
    return need(&ws->amax_idx, LR * ws->amax_entries * 4);
}

// ---- passes ------------------------------------------------------------------------------------------
int b200nn_hybrid::embed(Workspace &ws, const void *ids, const RowMap &rows, int T) {
    return launch_embedding_rows(ctx, (const uint32_t *)ids, table ? table->p : lm_head.b.w_nk->p, b16, (int)dp, T, (int)d, cfg.vocab,
                                 pos_table ? pos_table->p : nullptr, cfg.max_positions, rows, (float *)ws.x->p);
}

int b200nn_hybrid::pass_prompt(Workspace &ws, b200nn_kvcache &kv, const std::vector<PassEntry> &entries, const uint32_t *ids_host) {
    const size_t E = entries.size(), W = cfg.windows.size();
    size_t T = 0;
    bool one = true;
    int max_n = 0;
    for (const PassEntry &e : entries) {
        if (e.n <= 0 || (size_t)e.n > kv.portion) return set_error(ctx, B200NN_ERR_SHAPE, "a pass takes 1 .. portion tokens per sequence");
        if ((size_t)e.past + e.n > kv.cap) return set_error(ctx, B200NN_ERR_DIM, "KV cache capacity exceeded");
        T += e.n;
        one &= e.n == 1;
        max_n = std::max(max_n, e.n);
    }
    if (T > ws.rows) return set_error(ctx, B200NN_ERR_SHAPE, "workspace too small");
    // row tables: position, slot, sequence; sequence tables: slot, first row, rows, past; per window: first gathered
    // key row, key rows, position of the first
    std::vector<int> h(3 * T + 4 * E + 3 * E * W);
    int *hp = h.data(), *hs = hp + T, *hq = hs + T, *sq = hq + T;
    size_t row = 0;
    for (size_t i = 0; i < E; ++i) {
        const PassEntry &e = entries[i];
        sq[i] = e.slot;
        sq[E + i] = (int)row;
        sq[2 * E + i] = e.n;
        sq[3 * E + i] = e.past;
        for (int j = 0; j < e.n; ++j, ++row) {
            hp[row] = e.past + j;
            hs[row] = e.slot;
            hq[row] = (int)i;
        }
    }
    std::vector<int> k_rows(W, 0), max_k(W, 0);
    for (size_t v = 0; v < W; ++v) {
        int *kt = sq + 4 * E + 3 * E * v;
        for (size_t i = 0; i < E; ++i) {
            const PassEntry &e = entries[i];
            const int first = cfg.windows[v] ? std::max(0, e.past - (cfg.windows[v] - 1)) : 0, n = e.past + e.n - first;
            kt[i] = k_rows[v];
            kt[E + i] = n;
            kt[2 * E + i] = first;
            k_rows[v] += n;
            max_k[v] = std::max(max_k[v], n);
        }
    }
    TRY(need(&ws.meta, h.size() * 4));
    CK(ctx, cudaMemcpyAsync(ws.meta->p, h.data(), h.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
    CK(ctx, cudaMemcpyAsync(ws.ids->p, ids_host, T * 4, cudaMemcpyHostToDevice, ctx->stream));
    const int *m = (const int *)ws.meta->p, *ms = m + 3 * T;
    Pass p;
    p.T = (int)T;
    p.decode = one;
    p.rows = RowMap{m, 1, m + T};
    p.row_seq = m + 2 * T;
    p.seq.n_seq = (int)E;
    p.seq.max_n = max_n;
    p.seq.slot = ms;
    p.seq.row0 = ms + E;
    p.seq.n = ms + 2 * E;
    p.seq.past = ms + 3 * E;
    for (size_t v = 0; v < W; ++v) {
        SeqMap s = p.seq;
        const int *kt = ms + 4 * E + 3 * E * v;
        s.krow0 = kt;
        s.klen = kt + E;
        s.kpos0 = kt + 2 * E;
        s.k_rows = k_rows[v];
        s.max_k = max_k[v];
        p.seqs.push_back(s);
    }
    TRY(embed(ws, ws.ids->p, p.rows, (int)T));
    return run_layers(ws, kv, p);
}

int b200nn_hybrid::pass_decode(Workspace &ws, b200nn_kvcache &kv, const int *pos_ptr, StepProfile *prof) {
    Pass p;
    p.T = (int)kv.batch;
    p.decode = true;
    p.rows = RowMap{pos_ptr, 0, nullptr};
    p.prof = prof;
    TRY(embed(ws, ws.tok->p, p.rows, p.T));
    prof_mark(ctx, prof, B200NN_PROF_EMBED);
    return run_layers(ws, kv, p);
}

int b200nn_hybrid::stream_step(Workspace &ws, const Pass &p, size_t done) {
    StreamStep a{};
    a.rows = p.T;
    a.n = cfg.streams;
    a.d = (int)d;
    a.ldo = (int)dp;
    a.xs = (float *)ws.xs->p;
    a.x0 = (const float *)ws.x->p;
    if (done) {
        a.y = (const float *)ws.y->p;
        a.prev = subs[done - 1].hc;
    }
    if (done < subs.size()) {
        a.next = subs[done].hc;
        a.norm = subs[done].norm;
        a.eps = cfg.eps;
        a.out = ws.ln->p;
    } else {
        a.x_sum = (float *)ws.x->p;
    }
    TRY(launch_stream_step(ctx, a, b16));
    prof_mark(ctx, p.prof, B200NN_PROF_LAYERNORM);
    return B200NN_OK;
}

int b200nn_hybrid::run_layers(Workspace &ws, b200nn_kvcache &kv, const Pass &p) {
    size_t done = 0; // sublayers
    if (cfg.streams) TRY(stream_step(ws, p, 0));
    for (size_t i = 0; i < cfg.layers.size(); ++i) {
        const LayerSpec &l = cfg.layers[i];
        const LayerWeights &lw = *w[i];
        if (!cfg.streams) {
            TRY(launch_rmsnorm(ctx, (const float *)ws.x->p, (const float *)lw.norm1->p, cfg.eps, p.T, (int)d, (int)dp, ws.ln->p, act_type()));
            prof_mark(ctx, p.prof, B200NN_PROF_LAYERNORM);
        }
        if (l.type == MIX_DELTA) TRY(delta_layer(ws, kv.layers[i], l, lw, p));
        else if (l.type == MIX_MLSTM) TRY(mlstm_layer(ws, kv.layers[i], l, lw, p));
        else if (l.type == MIX_DIFF) TRY(diff_layer(ws, kv, kv.layers[i], l, lw, p));
        else TRY(latent_layer(ws, kv, kv.layers[i], l, lw, p));
        if (cfg.streams) TRY(stream_step(ws, p, ++done));
        if (!l.ff) continue;
        if (!cfg.streams) {
            TRY(launch_rmsnorm(ctx, (const float *)ws.x->p, (const float *)lw.norm2->p, cfg.eps, p.T, (int)d, (int)dp, ws.ln->p, act_type()));
            prof_mark(ctx, p.prof, B200NN_PROF_LAYERNORM);
        }
        TRY(feed_forward(ws, l, lw, p));
        if (cfg.streams) TRY(stream_step(ws, p, ++done));
    }
    return B200NN_OK;
}

int b200nn_hybrid::delta_layer(Workspace &ws, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p) {
    const DeltaDims &D = l.delta;
    const int ldp = D.proj_w();
    const float *ext = nullptr;
    if (D.channel) { // the first steps of the decay and gate projections leave in the activation type, the second follows
        Epilogue e;
        e.out = ws.proj->p;
        e.ldo = ldp;
        if (b16) {
            e.tail_out = ws.low->p;
            e.tail_at = D.low_at();
            e.tail_ld = 2 * D.low;
            e.tail_type = OUT_BF16;
        }
        TRY(linear_forward(ctx, lw.in, ws.ln->p, b16, p.T, e));
        Epilogue x;
        x.out = ws.ext->p;
        x.ldo = 2 * D.ext();
        TRY(run_grouped(lw.ext, b16 ? ws.low->p : (const void *)((const float *)ws.proj->p + D.low_at()), b16 ? 2 * D.low : ldp, p.T, x));
        ext = (const float *)ws.ext->p;
    } else {
        TRY(store_linear(lw.in, ws.ln->p, p.T, ws.proj->p, ldp, OUT_F32));
    }
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    const DeltaWeights dw{(const float *)lw.conv->p, (const float *)lw.a_exp->p, (const float *)lw.dt_bias->p, (const float *)lw.onorm->p};
    if (p.decode) {
        TRY(launch_delta_step(ctx, D, b16, (const float *)ws.proj->p, ldp, ext, dw, (float *)st.conv->p, (float *)st.state->p, p.rows, p.T,
                              ws.att->p));
    } else {
        TRY(need(&ws.dstep, ws.rows * max_conv * 4));
        TRY(need(&ws.heads, ws.rows * max_heads * 4));
        TRY(launch_delta_prompt(ctx, D, b16, (const float *)ws.proj->p, ldp, ext, dw, (float *)st.conv->p, (float *)st.state->p, p.rows, p.seq, p.T,
                                p.row_seq, (float *)ws.dstep->p, (float *)ws.heads->p, ws.att->p));
    }
    prof_mark(ctx, p.prof, B200NN_PROF_RECURRENCE);
    TRY(out_linear(lw.o, ws.att->p, p.T, ws));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    return B200NN_OK;
}

int b200nn_hybrid::mlstm_layer(Workspace &ws, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p) {
    const MlstmDims &D = l.mlstm;
    const int ldp = D.proj_w();
    TRY(store_linear(lw.in, ws.ln->p, p.T, ws.proj->p, ldp, OUT_F32));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    const MlstmWeights mw{(const float *)lw.i_bias->p, (const float *)lw.f_bias->p, (const float *)lw.onorm->p};
    const MlstmState ms{(float *)st.state->p, (float *)st.normaliser->p, (float *)st.maximum->p};
    if (p.decode) {
        TRY(launch_mlstm_step(ctx, D, b16, (const float *)ws.proj->p, ldp, mw, ms, p.rows, p.T, ws.att->p));
    } else {
        TRY(need(&ws.gate, ws.rows * std::max(max_gate, max_mgate) * 4));
        TRY(need(&ws.heads, ws.rows * max_heads * 4));
        TRY(launch_mlstm_prompt(ctx, D, b16, (const float *)ws.proj->p, ldp, mw, ms, p.seq, p.T, (float *)ws.gate->p, (float *)ws.heads->p, ws.att->p));
    }
    prof_mark(ctx, p.prof, B200NN_PROF_RECURRENCE);
    TRY(out_linear(lw.o, ws.att->p, p.T, ws));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    return B200NN_OK;
}

int b200nn_hybrid::diff_layer(Workspace &ws, b200nn_kvcache &kv, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p) {
    DiffDims D = l.diff;
    D.lambda = lw.lambda;
    const int cap = (int)kv.cap, g_at = D.q_w() + D.cache_w();
    const size_t cache_rows = kv.batch * D.kv_heads * kv.cap;
    const void *q;
    const float *gate;
    int ldq, ldg;
    if (b16) { // queries to ws.q, keys and values into the cache, gates to ws.gate
        Epilogue e;
        e.out = ws.q->p;
        e.ldo = ldq = D.q_w();
        e.out_half = OUT_BF16;
        e.kv_cache = (__nv_bfloat16 *)st.kv->p;
        e.kv_at = D.q_w();
        e.kv_w = D.kv_w();
        e.kv_heads = D.kv_heads;
        e.kv_cap = cap;
        e.rows = p.rows;
        e.tail_out = ws.gate->p;
        e.tail_at = g_at;
        e.tail_ld = ldg = D.heads;
        e.tail_type = OUT_F32;
        TRY(linear_forward(ctx, lw.in, ws.ln->p, true, p.T, e));
        q = ws.q->p;
        gate = (const float *)ws.gate->p;
    } else {
        ldq = ldg = (int)up(lw.in.N, 4);
        TRY(store_linear(lw.in, ws.ln->p, p.T, ws.proj->p, ldq, OUT_F32));
        TRY(launch_kv_store_f32(ctx, (const float *)ws.proj->p, ldq, D.q_w(), D.kv_heads, D.kv_w(), cap, p.rows, p.T, (float *)st.kv->p));
        q = ws.proj->p;
        gate = (const float *)ws.proj->p + g_at;
    }
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    if (p.decode) TRY(need(&ws.part, diff_part_floats(ctx, D, b16, p.T, cap) * 4));
    TRY(launch_diff_attention(ctx, D, b16, q, ldq, st.kv->p, cap, cache_rows, p.rows, p.decode ? SeqMap() : p.seq, p.T, gate, ldg,
                              ws.part ? (float *)ws.part->p : nullptr, ws.att->p));
    prof_mark(ctx, p.prof, B200NN_PROF_ATTENTION);
    TRY(out_linear(lw.o, ws.att->p, p.T, ws));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    return B200NN_OK;
}

int b200nn_hybrid::latent_layer(Workspace &ws, b200nn_kvcache &kv, LayerState &st, const LayerSpec &l, const LayerWeights &lw, const Pass &p) {
    const LatentDims &L = l.lat;
    const int ldp = (int)up(lw.in.N, 4), H = L.heads;
    const float2 *tab = (const float2 *)kv.rope[l.rope]->p;
    TRY(store_linear(lw.in, ws.ln->p, p.T, ws.proj->p, ldp, OUT_F32));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    TRY(launch_latent_prep(ctx, L, b16, (const float *)ws.proj->p, ldp, (const float *)lw.qnorm->p, (const float *)lw.kvnorm->p, tab, p.rows,
                           p.T, ws.cq->p, st.latent->p, st.ring, (float *)ws.gate->p));
    prof_mark(ctx, p.prof, B200NN_PROF_LAYERNORM);
    if (b16) {
        Epilogue e;
        e.mode = EPI_ROPE;
        e.out = ws.q->p;
        e.ldo = H * L.head_w();
        e.out_half = OUT_BF16;
        e.rope_head = L.head_w();
        e.rope_at = L.dim_p;
        e.rope_pairs = L.rot / 2;
        e.rope_tab = tab;
        e.rows = p.rows;
        TRY(linear_forward(ctx, lw.uq, ws.cq->p, true, p.T, e));
    } else {
        TRY(store_linear(lw.uq, ws.cq->p, p.T, ws.q->p, H * L.head_w(), OUT_F32));
        TRY(launch_rope_heads(ctx, (float *)ws.q->p, p.T, H, L.head_w(), L.dim_p, L.rot / 2, tab, p.rows));
    }
    if (p.decode) {
        TRY(need(&ws.qlat, (size_t)p.T * H * L.rank_p * es));
        TRY(need(&ws.olat, (size_t)p.T * H * L.rank_p * es));
        TRY(need(&ws.part, latent_decode_part_floats(ctx, L, b16, p.T, (int)kv.cap) * 4));
        Epilogue e;
        e.out = ws.qlat->p;
        e.ldo = H * L.rank_p;
        e.out_half = act_type();
        TRY(run_grouped(lw.uk, ws.q->p, H * L.head_w(), p.T, e));
        prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
        TRY(launch_latent_decode(ctx, L, b16, ws.q->p, ws.qlat->p, st.latent->p, st.ring, kv.batch * st.ring, p.rows, p.T, (int)kv.cap, ws.olat->p,
                                 (float *)ws.part->p));
        prof_mark(ctx, p.prof, B200NN_PROF_ATTENTION);
        Epilogue v;
        v.out = ws.att->p;
        v.ldo = H * L.vdim_p;
        v.out_half = act_type();
        v.row_scale = (const float *)ws.gate->p;
        v.rs_ld = H;
        v.rs_cols = L.vdim_p;
        TRY(run_grouped(lw.uv, ws.olat->p, H * L.rank_p, p.T, v));
    } else {
        const SeqMap &sm = p.seqs[l.win];
        TRY(need(&ws.lin, (size_t)sm.k_rows * L.ld() * es));
        TRY(need(&ws.kvx, (size_t)sm.k_rows * L.kv_w() * es));
        TRY(launch_latent_gather(ctx, L, b16, st.latent->p, st.ring, sm, ws.lin->p));
        if (b16) {
            TRY(store_linear(lw.ukv, ws.lin->p, sm.k_rows, ws.kvx->p, L.kv_w(), OUT_BF16, L.ld()));
        } else { // block diagonal with one group: takes a row stride
            Epilogue e;
            e.out = ws.kvx->p;
            e.ldo = L.kv_w();
            TRY(launch_grouped_f32(ctx, (const float *)lw.ukv_rows->p, 1, L.kv_w(), L.rank_p, (const float *)ws.lin->p, L.ld(), 0, sm.k_rows, e, 0));
        }
        prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
        TRY(launch_latent_prefill(ctx, L, b16, p.T, ws.q->p, ws.kvx->p, ws.lin->p, sm, (const float *)ws.gate->p, ws.att->p));
        prof_mark(ctx, p.prof, B200NN_PROF_ATTENTION);
    }
    TRY(out_linear(lw.o, ws.att->p, p.T, ws));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    return B200NN_OK;
}

int b200nn_hybrid::feed_forward(Workspace &ws, const LayerSpec &l, const LayerWeights &lw, const Pass &p) {
    const int ffp = (int)up(l.ff, 8);
    if (b16) {
        Epilogue e;
        e.mode = EPI_GLU;
        e.act = cfg.traits->act;
        e.out = ws.fc->p;
        e.ldo = ffp;
        e.out_half = OUT_BF16;
        TRY(linear_forward(ctx, lw.gu, ws.ln->p, true, p.T, e));
    } else {
        TRY(store_linear(lw.gu, ws.ln->p, p.T, ws.proj->p, 2 * ffp, OUT_F32));
        TRY(launch_glu(ctx, (const float *)ws.proj->p, p.T, 2 * ffp, cfg.traits->act, (float *)ws.fc->p));
    }
    TRY(out_linear(lw.down, ws.fc->p, p.T, ws));
    prof_mark(ctx, p.prof, B200NN_PROF_LINEAR);
    return B200NN_OK;
}

int b200nn_hybrid::head(Workspace &ws, const float *x, int rows, StepProfile *prof) {
    TRY(launch_rmsnorm(ctx, x, (const float *)final_norm->p, cfg.eps, rows, (int)d, (int)dp, ws.last_ln->p, act_type()));
    prof_mark(ctx, prof, B200NN_PROF_LAYERNORM);
    TRY(store_linear(lm_head, ws.last_ln->p, rows, ws.logits->p, cfg.vocab, OUT_F32));
    prof_mark(ctx, prof, B200NN_PROF_LM_HEAD);
    return B200NN_OK;
}

int b200nn_hybrid::head_pick(Workspace &ws, const float *x, int rows, bool keep_last, bool tokens_only, uint32_t *tok_out,
                             StepProfile *prof) {
    if (!b16 || !ctx->fused_argmax) {
        TRY(head(ws, x, rows, prof));
        return launch_argmax(ctx, (const float *)ws.logits->p, rows, cfg.vocab, cfg.vocab, keep_last, tok_out);
    }
    TRY(launch_rmsnorm(ctx, x, (const float *)final_norm->p, cfg.eps, rows, (int)d, (int)dp, ws.last_ln->p, act_type()));
    prof_mark(ctx, prof, B200NN_PROF_LAYERNORM);
    Epilogue e;
    e.out = ws.logits->p;
    e.ldo = cfg.vocab;
    e.no_store = tokens_only ? 1 : 0;
    e.amax_val = (float *)ws.amax_val->p;
    e.amax_idx = (int *)ws.amax_idx->p;
    e.amax_entries = ws.amax_entries;
    e.amax_keep_last = keep_last ? 1 : 0;
    TRY(linear_forward(ctx, lm_head, ws.last_ln->p, true, rows, e));
    prof_mark(ctx, prof, B200NN_PROF_LM_HEAD);
    return launch_argmax_entries(ctx, e.amax_val, e.amax_idx, rows, e.amax_entries, cfg.vocab, keep_last, tok_out);
}

bool hybrid_architecture(const std::string &arch) {
    for (const Traits &t : TRAITS)
        if (arch == t.name) return true;
    return false;
}

int hybrid_create(b200nn_ctx *ctx, const std::string &arch, const JsonValue &root, size_t n, const char *const *names, const float *const *data, const size_t *numels,
                  uint32_t flags, b200nn_lm **out) {
    CK(ctx, cudaSetDevice(ctx->device));
    auto m = std::unique_ptr<b200nn_hybrid>(new b200nn_hybrid());
    m->ctx = ctx;
    m->b16 = !(flags & B200NN_LM_F32);
    for (const Traits &t : TRAITS)
        if (arch == t.name) m->cfg.traits = &t;
    if (!m->cfg.traits) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "no hybrid decoder of architecture '" + arch + "'");
    ConfigReader r;
    if (!r.read(root, &m->cfg)) return set_error(ctx, B200NN_ERR_UNSUPPORTED, r.err);
    TensorMap t;
    for (size_t i = 0; i < n; ++i) t[names[i]] = TensorView{data[i], numels[i]};
    TRY(m->build(t));
    CK(ctx, cudaStreamSynchronize(ctx->stream));
    *out = m.release();
    return B200NN_OK;
}
