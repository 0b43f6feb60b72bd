// Model registry and serving step: a checkpoint folder becomes a model of the family its config.json names, and
// a step feeds the next tokens of any number of requests, each in its own slot of one cache.
#include <algorithm>
#include <cstring>
#include <fstream>
#include <sstream>

#include "hybrid.h"
#include "json.h"

int hybrid_create(b200nn_ctx *ctx, const std::string &arch, const JsonValue &root, size_t n, const char *const *names, const float *const *data, const size_t *numels,
                  uint32_t flags, b200nn_lm **out);
bool hybrid_architecture(const std::string &arch);

namespace {

constexpr size_t PASS_ROWS = 8192;  // rows per pass
constexpr size_t HEAD_ROWS = 1024;  // rows per LM-head launch

int parse_config(b200nn_ctx *ctx, const std::string &text, JsonValue *root) {
    Json j{text.data(), text.data() + text.size()};
    if (!j.value(*root) || root->kind != JsonValue::Object) return set_error(ctx, B200NN_ERR_IO, "config.json is not a JSON object");
    return B200NN_OK;
}

std::string architecture_of(const JsonValue &root) {
    const JsonValue *a = root.get("architecture"), *l = root.get("architectures"), *t = root.get("model_type");
    if (a && a->kind == JsonValue::String) return a->str;
    if (l && l->kind == JsonValue::Array && !l->items.empty()) return l->items[0].str;
    return t ? t->str : std::string();
}

// BF16, F16 or F32 tensor bytes -> f32
bool to_f32(const std::string &dtype, const std::vector<char> &raw, std::vector<float> *out) {
    if (dtype == "F32") {
        out->resize(raw.size() / 4);
        memcpy(out->data(), raw.data(), raw.size());
    } else if (dtype == "BF16" || dtype == "F16") {
        out->resize(raw.size() / 2);
        const uint16_t *s = reinterpret_cast<const uint16_t *>(raw.data());
        for (size_t i = 0; i < out->size(); ++i) {
            if (dtype == "BF16") {
                const uint32_t u = (uint32_t)s[i] << 16;
                memcpy(&(*out)[i], &u, 4);
            } else {
                __half h;
                memcpy(&h, &s[i], 2);
                (*out)[i] = __half2float(h);
            }
        }
    } else {
        return false;
    }
    return true;
}

// Which builder serves an architecture name.
enum Family { FAM_NONE, FAM_GPT2, FAM_HYBRID };
struct { const char *name; Family family; } const REGISTRY[] = {
    {"GPT2LMHeadModel", FAM_GPT2}, {"GPT2Model", FAM_GPT2}, {"gpt2", FAM_GPT2}};
Family family_of(const std::string &arch) {
    for (const auto &e : REGISTRY)
        if (arch == e.name) return e.family;
    return hybrid_architecture(arch) ? FAM_HYBRID : FAM_NONE;
}

}  // namespace

extern "C" int32_t b200nn_lm_create(b200nn_ctx *ctx, const char *config_json, size_t n_tensors, const char *const *names,
                                    const float *const *data, const size_t *numels, uint32_t flags, b200nn_lm **out) {
    if (!ctx || !config_json || !names || !data || !numels || !out) return B200NN_ERR_ARG;
    *out = nullptr;
    JsonValue root;
    TRY(parse_config(ctx, config_json, &root));
    const std::string arch = architecture_of(root);
    if (family_of(arch) != FAM_HYBRID)
        return set_error(ctx, B200NN_ERR_UNSUPPORTED, "no model family builds architecture '" + arch + "' from host tensors");
    return hybrid_create(ctx, arch, root, n_tensors, names, data, numels, flags, out);
}

extern "C" int32_t b200nn_lm_load(b200nn_ctx *ctx, const char *dir, uint32_t flags, b200nn_lm **out) {
    if (!ctx || !dir || !out) return B200NN_ERR_ARG;
    *out = nullptr;
    const std::string base(dir), cfg_path = base + "/config.json", st_path = base + "/model.safetensors";
    std::ifstream f(cfg_path);
    if (!f) return set_error(ctx, B200NN_ERR_IO, "cannot open " + cfg_path);
    std::stringstream text;
    text << f.rdbuf();
    JsonValue root;
    TRY(parse_config(ctx, text.str(), &root));
    const std::string arch = architecture_of(root);
    const Family fam = family_of(arch);
    if (fam == FAM_GPT2) {
        if (flags & B200NN_LM_F32) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "GPT-2 runs its Linears with 16-bit activations");
        b200nn_gpt2 *g = nullptr;
        TRY(b200nn_gpt2_load_safetensors(ctx, st_path.c_str(), nullptr, 0, flags, &g));
        *out = g;
        return B200NN_OK;
    }
    if (fam != FAM_HYBRID) return set_error(ctx, B200NN_ERR_UNSUPPORTED, "config.json: unknown architecture '" + arch + "'");
    b200nn_safetensors *raw = nullptr;
    int rc = b200nn_safetensors_open(st_path.c_str(), &raw);
    if (rc != B200NN_OK) return set_error(ctx, rc, b200nn_safetensors_last_error());
    std::unique_ptr<b200nn_safetensors, void (*)(b200nn_safetensors *)> st(raw, b200nn_safetensors_close);
    const int n = b200nn_safetensors_count(raw);
    std::vector<std::vector<float>> store((size_t)n);
    std::vector<const char *> names;
    std::vector<const float *> data;
    std::vector<size_t> numels;
    for (int i = 0; i < n; ++i) {
        const char *name, *dtype;
        size_t nbytes;
        b200nn_safetensors_info(raw, i, &name, &dtype, nullptr, 0, nullptr, &nbytes);
        std::vector<char> bytes(nbytes);
        rc = b200nn_safetensors_read(raw, i, bytes.data(), nbytes);
        if (rc != B200NN_OK) return set_error(ctx, rc, b200nn_safetensors_last_error());
        if (!to_f32(dtype, bytes, &store[i])) continue; // integer tables are not weights of this family
        names.push_back(name);
        data.push_back(store[i].data());
        numels.push_back(store[i].size());
    }
    return hybrid_create(ctx, arch, root, names.size(), names.data(), data.data(), numels.data(), flags, out);
}

extern "C" b200nn_lm *b200nn_gpt2_as_lm(b200nn_gpt2 *m) { return m; }
extern "C" void b200nn_lm_destroy(b200nn_lm *m) { delete m; }
extern "C" int32_t b200nn_lm_get_info(const b200nn_lm *m, b200nn_lm_info *out) {
    if (!m || !out) return B200NN_ERR_ARG;
    out->n_layer = m->n_layer();
    out->width = m->width();
    out->vocab_size = m->vocab();
    out->n_positions = (int32_t)m->max_positions();
    out->eos_token = (int32_t)m->eos();
    return B200NN_OK;
}
extern "C" const char *b200nn_lm_family(const b200nn_lm *m) { return m ? m->family() : ""; }

// ---- slots -------------------------------------------------------------------------------------------
extern "C" int32_t b200nn_kvcache_acquire(b200nn_kvcache *c, int32_t *slot) {
    if (!c || !slot) return B200NN_ERR_ARG;
    for (size_t i = 0; i < c->batch; ++i)
        if (!c->slot_used[i]) {
            c->slot_used[i] = 1;
            c->slot_len[i] = 0; // a sequence that starts at position 0 reads nothing of what the slot held
            *slot = (int32_t)i;
            return B200NN_OK;
        }
    return set_error(c->m->ctx, B200NN_ERR_DIM, "every sequence slot of the cache is in use");
}
extern "C" int32_t b200nn_kvcache_release(b200nn_kvcache *c, int32_t slot) {
    if (!c || slot < 0 || (size_t)slot >= c->batch) return B200NN_ERR_ARG;
    c->slot_used[slot] = 0;
    c->slot_len[slot] = 0;
    return B200NN_OK;
}
extern "C" size_t b200nn_kvcache_slot_len(const b200nn_kvcache *c, int32_t slot) {
    return c && slot >= 0 && (size_t)slot < c->batch ? c->slot_len[slot] : 0;
}

// ---- serving step ------------------------------------------------------------------------------------
extern "C" int32_t b200nn_lm_step(b200nn_kvcache *c, size_t n_entries, const int32_t *slots, const size_t *counts,
                                  const uint32_t *tokens, size_t n_want, const size_t *want, float *logits) {
    if (!c || !slots || !counts || !tokens || (n_want && (!want || !logits))) return B200NN_ERR_ARG;
    b200nn_lm *m = c->m;
    b200nn_ctx *ctx = m->ctx;
    CK(ctx, cudaSetDevice(ctx->device));
    size_t total = 0;
    std::vector<char> seen(c->batch, 0);
    for (size_t i = 0; i < n_entries; ++i) {
        if (slots[i] < 0 || (size_t)slots[i] >= c->batch || !c->slot_used[slots[i]] || seen[slots[i]])
            return set_error(ctx, B200NN_ERR_ARG, "step: a slot is not acquired or appears twice");
        seen[slots[i]] = 1;
        if (counts[i] == 0) return set_error(ctx, B200NN_ERR_SHAPE, "step: an entry brings no token");
        if (c->slot_len[slots[i]] + counts[i] > c->cap) return set_error(ctx, B200NN_ERR_DIM, "step: cache capacity exceeded");
        total += counts[i];
    }
    for (size_t i = 0; i < total; ++i)
        if (tokens[i] >= (uint32_t)m->vocab()) return set_error(ctx, B200NN_ERR_DIM, "token id out of range for vocab_size");
    for (size_t i = 0; i < n_want; ++i)
        if (want[i] >= total) return set_error(ctx, B200NN_ERR_DIM, "step: a wanted row is not in the step");
    if (!c->ws) c->ws.reset(new Workspace());
    Workspace &ws = *c->ws;
    const size_t rows_max = std::min(total, PASS_ROWS), head_max = std::min(std::max<size_t>(n_want, 1), HEAD_ROWS);
    if (ws.rows < rows_max || ws.logit_rows < head_max) {
        const size_t r = std::max(ws.rows, rows_max), lr = std::max(ws.logit_rows, head_max);
        CK(ctx, cudaStreamSynchronize(ctx->stream));
        c->ws.reset(new Workspace());
        TRY(m->workspace_init(r, lr, c->ws.get()));
        return b200nn_lm_step(c, n_entries, slots, counts, tokens, n_want, want, logits);
    }
    std::vector<size_t> done(n_entries, 0), first(n_entries, 0);
    for (size_t i = 1; i < n_entries; ++i) first[i] = first[i - 1] + counts[i - 1];
    std::vector<int> where(total, -1); // step row -> row of the pass
    std::shared_ptr<DevBuf> idx_dev;
    TRY(dev_alloc(ctx, HEAD_ROWS * sizeof(int), &idx_dev));
    for (size_t left = total; left;) {
        // a pass: of every request its next tokens, at most a portion each
        std::vector<PassEntry> entries;
        std::vector<uint32_t> ids;
        std::vector<size_t> step_rows;
        for (size_t i = 0; i < n_entries; ++i) {
            size_t n = std::min(counts[i] - done[i], rows_max - ids.size());
            if (c->portion) n = std::min(n, c->portion);
            if (!n) continue;
            entries.push_back(PassEntry{slots[i], (int)c->slot_len[slots[i]], (int)n});
            for (size_t j = 0; j < n; ++j) {
                step_rows.push_back(first[i] + done[i] + j);
                ids.push_back(tokens[first[i] + done[i] + j]);
            }
            done[i] += n;
            c->slot_len[slots[i]] += n;
        }
        TRY(m->pass_prompt(ws, *c, entries, ids.data()));
        for (size_t r = 0; r < step_rows.size(); ++r) where[step_rows[r]] = (int)r;
        std::vector<size_t> mine;
        for (size_t i = 0; i < n_want; ++i)
            if (where[want[i]] >= 0) mine.push_back(i);
        for (size_t a = 0; a < mine.size(); a += head_max) {
            const size_t n = std::min(head_max, mine.size() - a);
            std::vector<int> idx(n);
            for (size_t i = 0; i < n; ++i) idx[i] = where[want[mine[a + i]]];
            CK(ctx, cudaMemcpyAsync(idx_dev->p, idx.data(), n * sizeof(int), cudaMemcpyHostToDevice, ctx->stream));
            TRY(launch_gather_rows(ctx, (const float *)ws.x->p, (const int *)idx_dev->p, (int)n, m->width(), (float *)ws.last_x->p));
            TRY(m->head(ws, (const float *)ws.last_x->p, (int)n, nullptr));
            const size_t V = (size_t)m->vocab();
            for (size_t i = 0; i < n;) { // consecutive wanted rows leave in one copy
                size_t j = i + 1;
                while (j < n && mine[a + j] == mine[a + j - 1] + 1) ++j;
                CK(ctx, cudaMemcpyAsync(logits + mine[a + i] * V, (const float *)ws.logits->p + i * V, (j - i) * V * 4,
                                        cudaMemcpyDeviceToHost, ctx->stream));
                i = j;
            }
        }
        for (size_t r : step_rows) where[r] = -1;
        left -= ids.size();
    }
    return stream_sync_check(ctx);
}
