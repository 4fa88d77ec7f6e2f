// host_mafuzen.cu -- the Mafuzen architecture for the decoder of host_llama.cu: where its tensors go and the graph of one batch
// step.  The decoder owns the model object, the sequence cache, the inputs and the step; this file adds no loop of its own.
//
// The stream starts as  x = scale * embed[token].  A layer has a layer norm in front of and behind each sublayer,
//     x <- x + N1b(mixer(N1(x)));   x <- x + N2b(ff(N2(x))),
// and then takes in a second embedding of the token, e = the layer's slice of side.embed[token]:
//     x <- x + RMS(proj(gelu(gate x) * e)) * w_side.
// Mixers (b200_layer_params):
//   * attention: grouped-query softmax attention without rotation; slope_h * distance is taken off the score; a layer with kv_from
//     has queries only and reads the cache rows of that earlier layer;
//   * retention: q and k rotated (entry i with i + dims / 2), k scaled by dim^(-1/2), a state per head with a fixed decay, every
//     head's read-out divided by its root mean square, times silu(W_g h), projected;
//   * window attention beside time mixing: the left side divides q and k by their root mean square per head, caches the keys as
//     projected as its values, sees a window and the first tokens, and has a sigmoid gate per value; the right side mixes every
//     token's input with the previous token's (five mixes), decays its state per token and key channel and gives the current token
//     a bonus.  The two results are scaled and added.
// The feed-forward is dense and gated, or a mixture of experts down(max(up h, 0)^2) that a table names by token id, plus a shared
// expert.  The output is the norm and the embedding table.
//
// Graph choices: everything a mixer projects from one input is ONE product over row-concatenated weights (rows padded to a multiple of
// 8); r, k, v and the gate of the time mixing, which read four different mixes, are one batched product; the two output matrices of a
// parallel mixer lie side by side along K, so that the left result (scaled in the attention's epilogue) and the right one (scaled
// through its norm weight) meet in one product; a sublayer's norm, the residual sum and the next sublayer's input norm are one launch
// (norm_chain), which also takes the experts' mean and the shared expert; the expert numbers and the second embedding of all layers
// are gathered once per step; the experts' and the shared expert's activations share one launch.
#include "host_fused.h"

namespace {

struct MfLayer {
    ggml_tensor *n1 = nullptr, *n1_b = nullptr, *n1b = nullptr, *n1b_b = nullptr, *n2 = nullptr, *n2_b = nullptr, *n2b = nullptr, *n2b_b = nullptr;
    ggml_tensor *proj1 = nullptr, *wo = nullptr;
    int64_t proj1_rows = 0;
    ggml_tensor *slope = nullptr;                                                       // attention: minus the slope per head, [1, heads]
    ggml_tensor *decay = nullptr, *freqs = nullptr;                                     // retention
    ggml_tensor *mu = nullptr, *rkvg = nullptr, *w1 = nullptr, *w2 = nullptr, *w0 = nullptr, *u = nullptr, *mnorm = nullptr;  // time mixing
    ggml_tensor *gate_up = nullptr, *up = nullptr, *down = nullptr, *sh_up = nullptr, *sh_down = nullptr;
    int64_t table_col = 0;                                                              // first column of this layer in the gathered expert numbers
    ggml_tensor *side_gate = nullptr, *side_proj = nullptr, *side_norm = nullptr;
    ggml_tensor *k_cache = nullptr, *v_cache = nullptr;                                 // [kv_heads * dim, n_ctx], [kv_heads * vdim, n_ctx] f32
    ggml_tensor *state = nullptr, *prev = nullptr;                                      // retention / time mixing: S per slot; the previous token's input
};
struct HostMat { int type; int64_t ne0, ne1; std::vector<char> data; };
struct MfData {
    std::map<std::string, std::vector<int32_t>> tables;  // expert numbers by token id, as uploaded
    std::map<std::string, HostMat> mats;                 // matrices that finalize joins along K
    std::map<std::string, std::vector<float>> vecs;      // vectors that finalize scales
    std::vector<MfLayer> layers;
    ggml_tensor *embed = nullptr, *head = nullptr, *final_norm = nullptr, *final_norm_b = nullptr, *table = nullptr, *side_embed = nullptr;
};
MfData *mf(b200_llama *m) {
    if (!m->arch_data) m->arch_data = std::shared_ptr<void>(new MfData(), [](void *p) { delete (MfData *)p; });
    return (MfData *)m->arch_data.get();
}

int64_t pad8(int64_t v) { return (v + 7) / 8 * 8; }
bool is_parallel(const b200_layer_params &lp) { return lp.mixer == B200_MIXER_WINDOW_ATTENTION_TIME_MIX; }
bool own_kv(const b200_layer_params &lp) { return lp.mixer == B200_MIXER_ATTENTION && lp.kv_from < 0; }
// everything the mixer projects from its input, in the order of the rows of the fused matrix
int parts_proj1(const b200_layer_params &lp, Part out[4]) {
    int n = 0;
    const int64_t H = lp.heads, G = lp.kv_heads, D = lp.dim, V = lp.vdim;
    if (lp.mixer == B200_MIXER_RETENTION) {
        out[n++] = {"mix.q", H * D}; out[n++] = {"mix.k", H * D}; out[n++] = {"mix.v", H * V}; out[n++] = {"mix.g", H * V};
    } else if (is_parallel(lp)) {
        out[n++] = {"mix.left.q", H * D}; out[n++] = {"mix.left.k", G * D}; out[n++] = {"mix.left.g", H * V};
    } else {
        out[n++] = {"mix.q", H * D};
        if (own_kv(lp)) { out[n++] = {"mix.k", G * D}; out[n++] = {"mix.v", G * V}; }
    }
    return n;
}
// the mixes of the time mixing in the order of the batched product; the decay's mix comes last
constexpr const char *kMix[5] = {"mix.right.r", "mix.right.k", "mix.right.v", "mix.right.g", "mix.right.w"};
constexpr const char *kMu[5] = {"mix.right.mu.r", "mix.right.mu.k", "mix.right.mu.v", "mix.right.mu.g", "mix.right.mu.w"};

int mf_place_tensor(b200_llama *m, const char *name, int type, int64_t ne0, int64_t ne1, int64_t ne2, const void *data) {
    const b200_llama_params &hp = m->hp;
    const int64_t W = hp.n_embd;
    if (!strcmp(name, "embed")) {  // the scale of the embedding is part of the table
        LL_REQUIRE(type == GGML_TYPE_F32 && ne0 == W && ne1 == hp.n_vocab && ne2 == 1, B200_ERR_INVALID, "b200_llama_set_tensor: embed must be f32 [%d, %d]", hp.n_vocab, hp.n_embd);
        const float sc = hp.embed_scale == 0.0f ? 1.0f : hp.embed_scale;
        std::vector<float> t((size_t)(ne0 * ne1));
        for (size_t i = 0; i < t.size(); i++) t[i] = ((const float *)data)[i] * sc;
        return upload_tensor(m, name, type, ne0, ne1, ne2, t.data());
    }
    int il = -1;
    const char *leaf = nullptr;
    if (!split_name(name, &il, &leaf)) return upload_tensor(m, name, type, ne0, ne1, ne2, data);
    LL_REQUIRE(il >= 0 && il < hp.n_layer, B200_ERR_INVALID, "b200_llama_set_tensor: %s names a layer outside 0..%d", name, hp.n_layer - 1);
    const b200_layer_params &lp = m->layer_hp[(size_t)il];
    LL_REQUIRE(lp.mixer != 0, B200_ERR_INVALID, "b200_llama_set_tensor: %s before b200_llama_set_layer(%d)", name, il);
    const TypeTraits tt = type_traits(type);
    LL_REQUIRE(tt.blck == 1 && ne2 == 1, B200_ERR_UNSUPPORTED, "b200_llama_set_tensor: %s: dense 1-D / 2-D tensors only", name);
    const std::string pre = "l" + std::to_string(il) + ".";
    const size_t es = (size_t)tt.size;
#define MF_SHAPE(rows, cols) LL_REQUIRE(ne0 == (cols) && ne1 == (rows), B200_ERR_INVALID, "b200_llama_set_tensor: %s is [%lld, %lld], expected [%lld, %lld]", name, (long long)ne1, (long long)ne0, \
                                        (long long)(rows), (long long)(cols))
    if (!strcmp(leaf, "mlp.table")) {
        LL_REQUIRE(type == GGML_TYPE_I32 && lp.mlp == B200_MLP_MOE_TABLE, B200_ERR_INVALID, "b200_llama_set_tensor: %s must be i32 and belong to a layer with experts", name);
        MF_SHAPE(hp.n_vocab, lp.n_expert_used);
        mf(m)->tables[name].assign((const int32_t *)data, (const int32_t *)data + ne0 * ne1);
        return B200_OK;
    }
    int e = -1;
    const char *which = nullptr;
    if (lp.mlp == B200_MLP_MOE_TABLE && split_expert(leaf, &e, &which)) {
        LL_REQUIRE(e >= 0 && e < lp.n_expert, B200_ERR_INVALID, "b200_llama_set_tensor: %s names an expert outside 0..%d", name, lp.n_expert - 1);
        const int64_t F = lp.ff;
        const size_t bytes = (size_t)(F * W) * es;
        if (!strcmp(which, "up")) { MF_SHAPE(F, W); return place_into(m, pre + "mlp.up", name, type, W, F, lp.n_expert, (size_t)e * bytes, bytes, data); }
        if (!strcmp(which, "down")) { MF_SHAPE(W, F); return place_into(m, pre + "mlp.down", name, type, F, W, lp.n_expert, (size_t)e * bytes, bytes, data); }
    }
    if (lp.mlp == B200_MLP_DENSE_GATED && (!strcmp(leaf, "mlp.gate") || !strcmp(leaf, "mlp.up"))) {
        MF_SHAPE(lp.ff, W);
        const size_t bytes = (size_t)((int64_t)lp.ff * W) * es;
        return place_into(m, pre + "mlp.gate_up", name, type, W, 2 * (int64_t)lp.ff, 1, leaf[4] == 'u' ? bytes : 0, bytes, data);
    }
    Part parts[4];
    int64_t total = 0, rows = 0;
    const int64_t off = part_offset(parts, parts_proj1(lp, parts), leaf, &total, &rows);
    if (off >= 0) {  // rows padded to a multiple of 8 with zero weights (their results are zeros nobody reads)
        MF_SHAPE(rows, W);
        const std::string fused = pre + "proj1";
        const bool first = find_w(m, fused) == nullptr;
        const int rc = place_into(m, fused, name, type, W, pad8(total), 1, (size_t)(off * W) * es, (size_t)(rows * W) * es, data);
        if (rc == B200_OK && first && pad8(total) > total) {
            ggml_tensor *f = find_w(m, fused);
            const std::vector<char> z((size_t)((pad8(total) - total) * W) * es, 0);
            f->buffer->iface.set_tensor(f->buffer, f, z.data(), (size_t)(total * W) * es, z.size());
        }
        return rc;
    }
    if (is_parallel(lp)) {
        const int64_t HD = (int64_t)lp.mix_heads * lp.mix_dim;
        for (int i = 0; i < 4; i++) {
            if (strcmp(leaf, kMix[i]) != 0) continue;
            MF_SHAPE(HD, W);
            const size_t bytes = (size_t)(HD * W) * es;
            return place_into(m, pre + "mix.rkvg", name, type, W, HD, 4, (size_t)i * bytes, bytes, data);
        }
        for (int i = 0; i < 5; i++) {
            if (strcmp(leaf, kMu[i]) != 0) continue;
            LL_REQUIRE(type == GGML_TYPE_F32, B200_ERR_INVALID, "b200_llama_set_tensor: %s must be uploaded as f32", name);
            MF_SHAPE(1, W);
            return place_into(m, pre + "mix.mu", name, type, W, 5, 1, (size_t)(i * W) * 4, (size_t)W * 4, data);
        }
        if (!strcmp(leaf, "mix.left.o") || !strcmp(leaf, "mix.right.o")) {
            LL_REQUIRE(!mf(m)->mats.count(name), B200_ERR_INVALID, "b200_llama_set_tensor: duplicate tensor %s", name);
            MF_SHAPE(W, leaf[4] == 'l' ? (int64_t)lp.heads * lp.vdim : HD);
            mf(m)->mats[name] = HostMat{type, ne0, ne1, std::vector<char>((const char *)data, (const char *)data + (size_t)(ne0 * ne1) * es)};
            return B200_OK;
        }
        if (!strcmp(leaf, "mix.right.norm")) {
            LL_REQUIRE(type == GGML_TYPE_F32, B200_ERR_INVALID, "b200_llama_set_tensor: %s must be uploaded as f32", name);
            MF_SHAPE(1, HD);
            mf(m)->vecs[name].assign((const float *)data, (const float *)data + HD);
            return B200_OK;
        }
    }
#undef MF_SHAPE
    return upload_tensor(m, name, type, ne0, ne1, ne2, data);
}

int mf_finalize(b200_llama *m) {
    const b200_llama_params &hp = m->hp;
    MfData *g = mf(m);
    g->layers.assign((size_t)hp.n_layer, MfLayer());
    const int64_t W = hp.n_embd;
    LL_REQUIRE(W <= 16384, B200_ERR_UNSUPPORTED, "b200_llama_finalize: width %d (at most 16384)", hp.n_embd);
    LL_REQUIRE(m->run_layer.empty(), B200_ERR_UNSUPPORTED, "b200_llama_finalize: this architecture runs every layer once, in order");
    auto need_at = [&](const std::string &nm, int64_t ne0, int64_t ne1, int64_t ne2 = 1) -> ggml_tensor * {
        ggml_tensor *t = find_w(m, nm);
        if (!t) { b200::set_error("b200_llama_finalize: tensor %s missing", nm.c_str()); return nullptr; }
        if (t->ne[0] != ne0 || t->ne[1] != ne1 || t->ne[2] != ne2) {
            b200::set_error("b200_llama_finalize: tensor %s has shape [%lld, %lld, %lld], the model's sizes give [%lld, %lld, %lld]", nm.c_str(), (long long)t->ne[2], (long long)t->ne[1],
                            (long long)t->ne[0], (long long)ne2, (long long)ne1, (long long)ne0);
            return nullptr;
        }
        return t;
    };
#define MF_NEED(dst, ...) do { dst = need_at(__VA_ARGS__); if (!(dst)) return B200_ERR_INVALID; } while (0)
    MF_NEED(g->embed, "embed", W, hp.n_vocab); MF_NEED(g->head, "head", W, hp.n_vocab);
    MF_NEED(g->final_norm, "final.norm", W, 1); MF_NEED(g->final_norm_b, "final.norm.b", W, 1);
    const int64_t ES = hp.n_layer > 0 ? m->layer_hp[0].token_side : 0;
    if (ES > 0) {
        MF_NEED(g->side_embed, "side.embed", ES * hp.n_layer, hp.n_vocab);
        LL_REQUIRE(g->side_embed->type == GGML_TYPE_F32, B200_ERR_INVALID, "b200_llama_finalize: side.embed must be uploaded as f32");
    }
    int64_t table_cols = 0;
    for (int il = 0; il < hp.n_layer; il++) {
        const b200_layer_params &lp = m->layer_hp[(size_t)il];
        MfLayer &L = g->layers[(size_t)il];
        const std::string pre = "l" + std::to_string(il) + ".";
        const int64_t H = lp.heads, G = lp.kv_heads, D = lp.dim, V = lp.vdim;
        int rc = B200_OK;
        LL_REQUIRE(lp.mixer == B200_MIXER_ATTENTION || lp.mixer == B200_MIXER_RETENTION || is_parallel(lp), B200_ERR_INVALID, "b200_llama_finalize: layer %d has no mixer of this architecture", il);
        LL_REQUIRE(H > 0 && D > 0 && D <= 256 && V > 0 && (V <= 256 || lp.mixer == B200_MIXER_RETENTION), B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: heads %d, dim %d and vdim %d (<= 256)", il,
                   lp.heads, lp.dim, lp.vdim);
        LL_REQUIRE(lp.token_side == ES, B200_ERR_INVALID, "b200_llama_finalize: layer %d: every layer takes a token input of one size", il);
        MF_NEED(L.n1, pre + "norm1", W, 1); MF_NEED(L.n1_b, pre + "norm1.b", W, 1); MF_NEED(L.n1b, pre + "norm1b", W, 1); MF_NEED(L.n1b_b, pre + "norm1b.b", W, 1);
        Part parts[4];
        const int np = parts_proj1(lp, parts);
        int64_t total = 0;
        part_offset(parts, np, "", &total);
        for (int i = 0; i < np; i++) LL_REQUIRE(find_w(m, pre + parts[i].leaf), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), parts[i].leaf);
        L.proj1_rows = pad8(total);
        MF_NEED(L.proj1, pre + "proj1", W, L.proj1_rows);
        if (lp.mixer == B200_MIXER_RETENTION) {
            LL_REQUIRE(lp.rope_dims >= 0 && lp.rope_dims % 2 == 0 && lp.rope_dims <= D && (lp.rope_dims == 0 || lp.rope_base > 0.0f), B200_ERR_INVALID, "b200_llama_finalize: layer %d: rotation does not fit dim", il);
            MF_NEED(L.wo, pre + "mix.o", H * V, W);
            MF_NEED(L.decay, pre + "mix.decay", H, 1);
            if (lp.rope_dims > 0) {
                std::vector<float> f;
                rope_freqs(lp, f);
                rc = upload_tensor(m, (pre + "rope_freqs").c_str(), GGML_TYPE_F32, (int64_t)f.size(), 1, 1, f.data());
                if (rc != B200_OK) return rc;
                L.freqs = find_w(m, pre + "rope_freqs");
            }
            L.state = new_device_tensor(m, (pre + "state").c_str(), GGML_TYPE_F32, H * D * V, hp.n_seq_max, true);
            LL_REQUIRE(L.state, B200_ERR_NOMEM, "b200_llama_finalize: out of device memory for the state of layer %d", il);
            m->kv_bytes += (int64_t)nbytes(L.state);
        } else {
            LL_REQUIRE(G > 0 && H % G == 0 && lp.window >= 0 && lp.keep_first >= 0, B200_ERR_INVALID, "b200_llama_finalize: layer %d: heads %d over %d kv heads, window and kept first tokens", il, lp.heads, lp.kv_heads);
            if (lp.dist_slope_exp > 0.0f) {
                std::vector<float> sl((size_t)H);
                for (int64_t h = 0; h < H; h++) sl[(size_t)h] = (float)-exp2(-(double)lp.dist_slope_exp * (double)(h + 1) / (double)H);
                rc = upload_tensor(m, (pre + "mix.slope").c_str(), GGML_TYPE_F32, 1, H, 1, sl.data());
                if (rc != B200_OK) return rc;
                L.slope = find_w(m, pre + "mix.slope");
            }
            if (lp.mixer == B200_MIXER_ATTENTION) MF_NEED(L.wo, pre + "mix.o", H * V, W);
            if (lp.mixer == B200_MIXER_ATTENTION && lp.kv_from >= 0) {
                LL_REQUIRE(lp.kv_from < il && own_kv(m->layer_hp[(size_t)lp.kv_from]), B200_ERR_INVALID, "b200_llama_finalize: layer %d reads the cache of layer %d, which keeps none before it", il, lp.kv_from);
                const b200_layer_params &src = m->layer_hp[(size_t)lp.kv_from];
                LL_REQUIRE(src.kv_heads == G && src.dim == D && src.vdim == V, B200_ERR_INVALID, "b200_llama_finalize: layer %d: the cache of layer %d has other head sizes", il, lp.kv_from);
                L.k_cache = g->layers[(size_t)lp.kv_from].k_cache; L.v_cache = g->layers[(size_t)lp.kv_from].v_cache;
            } else {
                L.k_cache = new_device_tensor(m, (pre + "k").c_str(), GGML_TYPE_F32, G * D, hp.n_ctx, true);
                L.v_cache = new_device_tensor(m, (pre + "v").c_str(), GGML_TYPE_F32, G * V, hp.n_ctx, true);
                LL_REQUIRE(L.k_cache && L.v_cache, B200_ERR_NOMEM, "b200_llama_finalize: out of device memory for the cache of layer %d", il);
                m->kv_bytes += (int64_t)(nbytes(L.k_cache) + nbytes(L.v_cache));
            }
        }
        if (is_parallel(lp)) {
            LL_REQUIRE(V == D, B200_ERR_INVALID, "b200_llama_finalize: layer %d: the values are the keys, so vdim must be dim", il);
            LL_REQUIRE(lp.mix_heads > 0 && lp.mix_dim > 0 && lp.mix_dim <= 256, B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: time mixing with %d heads of %d (<= 256)", il, lp.mix_heads, lp.mix_dim);
            const int64_t HD = (int64_t)lp.mix_heads * lp.mix_dim;
            for (int i = 0; i < 5; i++) {
                LL_REQUIRE(i == 4 || find_w(m, pre + kMix[i]), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), kMix[i]);
                LL_REQUIRE(find_w(m, pre + kMu[i]), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), kMu[i]);
            }
            MF_NEED(L.rkvg, pre + "mix.rkvg", W, HD, 4); MF_NEED(L.mu, pre + "mix.mu", W, 5);
            L.w1 = find_w(m, pre + "mix.right.w1");
            LL_REQUIRE(L.w1 && L.w1->ne[0] == W, B200_ERR_INVALID, "b200_llama_finalize: %smix.right.w1 missing or not as wide as the model", pre.c_str());
            MF_NEED(L.w2, pre + "mix.right.w2", L.w1->ne[1], HD);
            MF_NEED(L.w0, pre + "mix.right.w0", HD, 1); MF_NEED(L.u, pre + "mix.right.u", lp.mix_dim, lp.mix_heads);
            LL_REQUIRE(L.u->type == GGML_TYPE_F32, B200_ERR_INVALID, "b200_llama_finalize: %smix.right.u must be uploaded as f32", pre.c_str());
            // the right side's factor joins the weight of its head norm; the two output matrices lie side by side along K
            auto nv = g->vecs.find(pre + "mix.right.norm");
            LL_REQUIRE(nv != g->vecs.end(), B200_ERR_INVALID, "b200_llama_finalize: tensor %smix.right.norm missing", pre.c_str());
            for (float &v : nv->second) v *= lp.right_scale;
            rc = upload_tensor(m, (pre + "mix.right.scaled_norm").c_str(), GGML_TYPE_F32, HD, 1, 1, nv->second.data());
            if (rc != B200_OK) return rc;
            L.mnorm = find_w(m, pre + "mix.right.scaled_norm");
            auto ol = g->mats.find(pre + "mix.left.o"), orr = g->mats.find(pre + "mix.right.o");
            LL_REQUIRE(ol != g->mats.end() && orr != g->mats.end() && ol->second.type == orr->second.type, B200_ERR_INVALID, "b200_llama_finalize: %smix.left.o / right.o missing or of two types", pre.c_str());
            const size_t es = (size_t)type_traits(ol->second.type).size, bl = (size_t)(H * V) * es, br = (size_t)HD * es;
            std::vector<char> joined((bl + br) * (size_t)W);
            for (int64_t r = 0; r < W; r++) {
                memcpy(joined.data() + (size_t)r * (bl + br), ol->second.data.data() + (size_t)r * bl, bl);
                memcpy(joined.data() + (size_t)r * (bl + br) + bl, orr->second.data.data() + (size_t)r * br, br);
            }
            rc = upload_tensor(m, (pre + "mix.o").c_str(), ol->second.type, H * V + HD, W, 1, joined.data());
            if (rc != B200_OK) return rc;
            L.wo = find_w(m, pre + "mix.o");
            g->mats.erase(ol); g->mats.erase(orr);
            L.state = new_device_tensor(m, (pre + "state").c_str(), GGML_TYPE_F32, HD * lp.mix_dim, hp.n_seq_max, true);
            L.prev = new_device_tensor(m, (pre + "prev").c_str(), GGML_TYPE_F32, W, hp.n_seq_max, true);
            LL_REQUIRE(L.state && L.prev, B200_ERR_NOMEM, "b200_llama_finalize: out of device memory for the state of layer %d", il);
            m->kv_bytes += (int64_t)(nbytes(L.state) + nbytes(L.prev));
        }
        if (ES > 0) { MF_NEED(L.side_gate, pre + "side.gate", W, ES); MF_NEED(L.side_proj, pre + "side.proj", ES, W); MF_NEED(L.side_norm, pre + "side.norm", W, 1); }
        if (lp.mlp == B200_MLP_NONE) continue;
        MF_NEED(L.n2, pre + "norm2", W, 1); MF_NEED(L.n2_b, pre + "norm2.b", W, 1); MF_NEED(L.n2b, pre + "norm2b", W, 1); MF_NEED(L.n2b_b, pre + "norm2b.b", W, 1);
        LL_REQUIRE((lp.mlp == B200_MLP_DENSE_GATED || lp.mlp == B200_MLP_MOE_TABLE) && lp.ff > 0, B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: feed-forward kind %d", il, lp.mlp);
        if (lp.mlp == B200_MLP_DENSE_GATED) {
            for (const char *w : {"mlp.gate", "mlp.up"}) LL_REQUIRE(find_w(m, pre + w), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), w);
            MF_NEED(L.gate_up, pre + "mlp.gate_up", W, 2 * (int64_t)lp.ff); MF_NEED(L.down, pre + "mlp.down", lp.ff, W);
            continue;
        }
        LL_REQUIRE(lp.n_expert > 0 && lp.n_expert_used > 0 && lp.n_expert_used <= lp.n_expert, B200_ERR_INVALID, "b200_llama_finalize: layer %d: %d of %d experts per token", il, lp.n_expert_used, lp.n_expert);
        for (int e = 0; e < lp.n_expert; e++)
            for (const char *w : {"up", "down"}) {
                const std::string nm = pre + "mlp.e" + std::to_string(e) + "." + w;
                LL_REQUIRE(find_w(m, nm), B200_ERR_INVALID, "b200_llama_finalize: tensor %s missing", nm.c_str());
            }
        MF_NEED(L.up, pre + "mlp.up", W, lp.ff, lp.n_expert); MF_NEED(L.down, pre + "mlp.down", lp.ff, W, lp.n_expert);
        if (lp.shared_ff > 0) { MF_NEED(L.sh_up, pre + "mlp.shared.up", W, lp.shared_ff); MF_NEED(L.sh_down, pre + "mlp.shared.down", lp.shared_ff, W); }
        auto tb = g->tables.find(pre + "mlp.table");
        LL_REQUIRE(tb != g->tables.end(), B200_ERR_INVALID, "b200_llama_finalize: tensor %smlp.table missing", pre.c_str());
        for (int32_t v : tb->second) LL_REQUIRE(v >= 0 && v < lp.n_expert, B200_ERR_INVALID, "b200_llama_finalize: %smlp.table names expert %d of %d", pre.c_str(), v, lp.n_expert);
        L.table_col = table_cols;
        table_cols += lp.n_expert_used;
    }
#undef MF_NEED
    if (table_cols > 0) {  // the tables of all layers side by side: one gather per step
        std::vector<int32_t> all((size_t)(table_cols * hp.n_vocab));
        for (int il = 0; il < hp.n_layer; il++) {
            const b200_layer_params &lp = m->layer_hp[(size_t)il];
            if (lp.mlp != B200_MLP_MOE_TABLE) continue;
            const std::vector<int32_t> &t = g->tables["l" + std::to_string(il) + ".mlp.table"];
            for (int64_t v = 0; v < hp.n_vocab; v++)
                for (int k = 0; k < lp.n_expert_used; k++) all[(size_t)(v * table_cols + g->layers[(size_t)il].table_col + k)] = t[(size_t)(v * lp.n_expert_used + k)];
        }
        const int rc = upload_tensor(m, "mlp.tables", GGML_TYPE_I32, table_cols, hp.n_vocab, 1, all.data());
        if (rc != B200_OK) return rc;
        g->table = find_w(m, "mlp.tables");
    }
    g->tables.clear(); g->vecs.clear();
    return B200_OK;
}

// ------------------------------------------------------------------------------------------------ graph of one batch step
enum { R_HEAD = 0, R_EVEN = 1, R_ODD = 2, R_TAIL = 3 };
// up to this many tokens the scan of a retention layer turns q and k itself (every CTA of a head its own copy); longer prompts get one
// launch that turns them in place
constexpr int64_t kRotateInScan = 64;

int mf_build(b200_llama *m, const BatchShape &bs) {
    const b200_llama_params &hp = m->hp;
    MfData *g = mf(m);
    const int64_t T = bs.n_tokens, W = hp.n_embd;
    const float eps = hp.rms_eps;
    m->arena.reset();
    Builder b;
    b.arena = &m->arena;
    for (Bump &r : m->regions) r.off = 0;
    auto input_view = [&](const ggml_tensor &base, int64_t ne0, int64_t ne1 = 1) {
        ggml_tensor *t = m->arena.get();
        *t = base;
        set_shape(t, base.type, ne0, ne1, 1, 1);
        return t;
    };
    ggml_tensor *tokens = input_view(m->inp_tokens, T), *pos = input_view(m->inp_pos, T), *cells = input_view(m->inp_cells, T), *tok_seq = input_view(m->inp_tok_seq, T);
    ggml_tensor *cell_seq = input_view(m->inp_cell_seq, bs.n_kv), *cell_pos = input_view(m->inp_cell_pos, bs.n_kv), *seq_info = input_view(m->inp_seq_info, bs.n_seq, 4);

    auto layer_norm = [&](ggml_tensor *x, ggml_tensor *w, ggml_tensor *bias) {
        ggml_tensor *dst = b.alloc_result(GGML_TYPE_F32, x->ne[0], x->ne[1]);
        b.ext(dst, B200_EXT_NORM, {x, w, nullptr, nullptr, nullptr, bias});
        dst->op_params[2] = B200_NORM_LAYER; Builder::set_f(dst, 3, eps); dst->op_params[4] = 1; dst->op_params[5] = 0;
        return dst;
    };
    // x' = res + N1(y) and, when w2 is given, h' = the layer norm of x' that the next sublayer reads
    struct Chained { ggml_tensor *x, *h; };
    auto chain = [&](ggml_tensor *y3, float y_scale, ggml_tensor *shared, ggml_tensor *res, int kind1, ggml_tensor *w1, ggml_tensor *b1, ggml_tensor *w2, ggml_tensor *b2) {
        ggml_tensor *dst = b.alloc_result(GGML_TYPE_F32, W, T, w2 ? 2 : 1);
        b.ext(dst, B200_EXT_NORM_CHAIN, {y3, nullptr, shared, res, w1, b1, w2, b2});
        dst->op_params[2] = kind1; Builder::set_f(dst, 3, eps); dst->op_params[4] = B200_NORM_LAYER; Builder::set_f(dst, 5, y_scale);
        Chained c = {b.view_2d(dst, W, T, dst->nb[1], 0), w2 ? b.view_2d(dst, W, T, dst->nb[1], dst->nb[2]) : nullptr};
        return c;
    };
    auto one_result = [&](ggml_tensor *y) { return b.view_3d(y, W, 1, T, y->nb[1], y->nb[1], 0); };

    b.bump = &m->regions[R_HEAD];
    ggml_tensor *x = b.op(b.alloc_result(GGML_TYPE_F32, W, T), GGML_OP_GET_ROWS, g->embed, tokens);
    ggml_tensor *side_rows = g->side_embed ? b.op(b.alloc_result(GGML_TYPE_F32, g->side_embed->ne[0], T), GGML_OP_GET_ROWS, g->side_embed, tokens) : nullptr;
    ggml_tensor *expert_ids = g->table ? b.op(b.alloc_result(GGML_TYPE_I32, g->table->ne[0], T), GGML_OP_GET_ROWS, g->table, tokens) : nullptr;
    ggml_tensor *h = layer_norm(x, g->layers[0].n1, g->layers[0].n1_b);

    for (int il = 0; il < hp.n_layer; il++) {
        const b200_layer_params &lp = m->layer_hp[(size_t)il];
        MfLayer &L = g->layers[(size_t)il];
        const MfLayer *next = il + 1 < hp.n_layer ? &g->layers[(size_t)il + 1] : nullptr;
        b.bump = &m->regions[(il & 1) ? R_ODD : R_EVEN];
        b.bump->off = 0;
        const int64_t H = lp.heads, G = lp.kv_heads, D = lp.dim, V = lp.vdim;
        ggml_tensor *P = b.mul_mat(L.proj1, h);
        Part parts[4];
        const int np = parts_proj1(lp, parts);
        auto part_at = [&](const char *leaf) { return (size_t)part_offset(parts, np, leaf, nullptr) * 4; };
        auto part = [&](const char *leaf) {
            int64_t rows = 0;
            const int64_t off = part_offset(parts, np, leaf, nullptr, &rows);
            return b.view_2d(P, rows, T, P->nb[1], (size_t)off * 4);
        };
        // every head's row divided by its root mean square, optionally times a weight, times silu of a gate
        auto head_norm = [&](ggml_tensor *o, ggml_tensor *dst, ggml_tensor *w, int64_t w_period, ggml_tensor *gate) {
            b.ext(dst, B200_EXT_NORM, {o, w, gate, nullptr, nullptr, nullptr});
            dst->op_params[2] = B200_NORM_RMS; Builder::set_f(dst, 3, eps); dst->op_params[4] = (int32_t)w_period; dst->op_params[5] = 2;
            return dst;
        };
        auto attention = [&](ggml_tensor *o, ggml_tensor *q, ggml_tensor *gate, float out_scale) {
            b.ext(o, B200_EXT_SINK_ATTN, {q, b.view_2d(L.k_cache, G * D, bs.n_kv, L.k_cache->nb[1], 0), b.view_2d(L.v_cache, G * V, bs.n_kv, L.v_cache->nb[1], 0), nullptr, tok_seq, pos,
                                           cell_seq, cell_pos, gate, L.slope});
            o->op_params[2] = (int32_t)D; Builder::set_f(o, 3, lp.scale); o->op_params[4] = lp.window; o->op_params[5] = lp.keep_first;
            // bf16 weights: the attention products of a prompt batch may be bf16 as well (B200_ATTN_F32=1 keeps them in f32)
            static const bool attn_f32 = getenv("B200_ATTN_F32") != nullptr;
            o->op_params[6] = L.proj1->type == GGML_TYPE_BF16 && !attn_f32;
            o->op_params[7] = (int32_t)V; o->op_params[8] = 0; o->op_params[9] = B200_ATTN_SOFTMAX; o->op_params[10] = L.slope ? 1 : 0; Builder::set_f(o, 11, out_scale);
            return o;
        };
        // k and v to the tokens' cells (q is rewritten in place where the layer normalises it)
        auto store = [&](const char *ql, const char *kl, const char *vl, int norm_kind) {
            ggml_tensor *q = part(ql), *qo = part(ql);
            b.ext(qo, B200_EXT_QKV_STORE, {q, part(kl), part(vl), nullptr, pos, nullptr, cells, b.view_2d(L.k_cache, G * D, hp.n_ctx, L.k_cache->nb[1], 0),
                                            b.view_2d(L.v_cache, G * V, hp.n_ctx, L.v_cache->nb[1], 0)});
            qo->op_params[2] = (int32_t)D; qo->op_params[3] = (int32_t)V; qo->op_params[4] = 0; Builder::set_f(qo, 5, eps);
            qo->op_params[6] = 0; qo->op_params[7] = norm_kind; qo->op_params[8] = 0; qo->op_params[9] = 0; Builder::set_f(qo, 10, 0.0f); qo->op_params[11] = 1;
            return qo;
        };
        ggml_tensor *y;  // the mixer's result [W, T]
        if (lp.mixer == B200_MIXER_RETENTION) {
            ggml_tensor *q = part("mix.q"), *k = part("mix.k");
            const bool in_scan = lp.rope_dims > 0 && T <= kRotateInScan;
            if (lp.rope_dims > 0 && !in_scan) {  // q and k are neighbours: all their heads in one launch, in place
                ggml_tensor *qk = b.view_3d(P, D, 2 * H, T, (size_t)D * 4, P->nb[1], 0);
                ggml_tensor *r = b.view_3d(P, D, 2 * H, T, (size_t)D * 4, P->nb[1], 0);
                b.ext(r, B200_EXT_ROPE_TABLE, {qk, pos, L.freqs});
                r->op_params[2] = lp.rope_dims; Builder::set_f(r, 3, 1.0f); r->op_params[4] = 1;
                q = b.view_2d(r, H * D, T, P->nb[1], 0);
                k = b.view_2d(r, H * D, T, P->nb[1], (size_t)(H * D) * 4);
            }
            ggml_tensor *o = b.alloc_result(GGML_TYPE_F32, H * V, T);
            b.ext(o, B200_EXT_LINEAR_ATTN_SCAN, {q, k, part("mix.v"), L.decay, seq_info, L.state, pos, L.freqs});
            o->op_params[2] = (int32_t)H; o->op_params[3] = (int32_t)D; o->op_params[4] = (int32_t)V; o->op_params[5] = 0;
            Builder::set_f(o, 6, 1.0f / sqrtf((float)D)); o->op_params[7] = in_scan ? lp.rope_dims : 0;
            ggml_tensor *gate = b.view_3d(P, V, H, T, (size_t)V * 4, P->nb[1], part_at("mix.g"));
            ggml_tensor *on = head_norm(b.reshape(o, V, H, T), b.alloc_result(GGML_TYPE_F32, V, H, T), nullptr, 1, gate);
            y = b.mul_mat(L.wo, b.reshape(on, H * V, T));
        } else if (lp.mixer == B200_MIXER_ATTENTION) {
            ggml_tensor *q = own_kv(lp) ? store("mix.q", "mix.k", "mix.v", 0) : part("mix.q");
            y = b.mul_mat(L.wo, attention(b.alloc_result(GGML_TYPE_F32, H * V, T), q, nullptr, 1.0f));
        } else {
            const int64_t HR = lp.mix_heads, DR = lp.mix_dim, HD = HR * DR, KO = H * V + HD;
            ggml_tensor *both = b.alloc_result(GGML_TYPE_F32, KO, T);  // [left | right], the input of the joined output product
            // left
            ggml_tensor *ol = b.result_at(both, 0, GGML_TYPE_F32, H * V, T);
            ol->nb[1] = both->nb[1]; ol->nb[2] = ol->nb[3] = ol->nb[1] * (size_t)T;
            attention(ol, store("mix.left.q", "mix.left.k", "mix.left.k", 3), part("mix.left.g"), lp.left_scale);
            // right: five mixes with the previous token, four products, the decay's two small products
            ggml_tensor *mix = b.alloc_result(GGML_TYPE_F32, W, T, 5);
            b.ext(mix, B200_EXT_TOKEN_SHIFT, {h, L.mu, seq_info, L.prev});
            ggml_tensor *rkvg = b.mul_mat(L.rkvg, b.view_3d(mix, W, T, 4, mix->nb[1], mix->nb[2], 0));
            ggml_tensor *z1 = b.mul_mat(L.w1, b.view_2d(mix, W, T, mix->nb[1], 4 * mix->nb[2]));
            ggml_tensor *zt = b.ext(b.alloc_result(GGML_TYPE_F32, z1->ne[0], T), B200_EXT_UNARY, {z1});
            zt->op_params[2] = B200_UN_TANH;
            ggml_tensor *z = b.mul_mat(L.w2, zt);
            auto plane = [&](int i) { return b.view_2d(rkvg, HD, T, rkvg->nb[1], (size_t)i * rkvg->nb[2]); };
            ggml_tensor *o = b.alloc_result(GGML_TYPE_F32, HD, T);
            b.ext(o, B200_EXT_TIME_MIX_SCAN, {plane(0), plane(1), plane(2), z, L.w0, L.u, seq_info, L.state});
            o->op_params[2] = (int32_t)HR; o->op_params[3] = (int32_t)DR;
            ggml_tensor *orr = b.result_at(both, (size_t)(H * V) * 4, GGML_TYPE_F32, DR, HR, T);
            orr->nb[2] = both->nb[1]; orr->nb[3] = orr->nb[2] * (size_t)T;
            head_norm(b.reshape(o, DR, HR, T), orr, L.mnorm, HR, b.view_3d(rkvg, DR, HR, T, (size_t)DR * 4, rkvg->nb[1], 3 * rkvg->nb[2]));
            // the joined product waits for both sides: the view names the right one as its source, the left one hangs on as a further source
            ggml_tensor *in = b.view_of(orr, GGML_OP_VIEW, 0);
            set_shape(in, GGML_TYPE_F32, KO, T, 1, 1);
            in->data = both->data; in->view_src = both; in->view_offs = 0; in->src[1] = ol;
            y = b.mul_mat(L.wo, in);
        }
        const bool side = side_rows != nullptr, last = next == nullptr;
        auto next_w = [&](bool ends_layer) { return ends_layer && !last ? next->n1 : nullptr; };
        auto next_b = [&](bool ends_layer) { return ends_layer && !last ? next->n1_b : nullptr; };
        if (lp.mlp == B200_MLP_NONE) {
            const Chained c = chain(one_result(y), 1.0f, nullptr, x, B200_NORM_LAYER, L.n1b, L.n1b_b, next_w(!side), next_b(!side));
            x = c.x; h = c.h;
        } else {
            Chained c = chain(one_result(y), 1.0f, nullptr, x, B200_NORM_LAYER, L.n1b, L.n1b_b, L.n2, L.n2_b);
            x = c.x; h = c.h;
            const int64_t F = lp.ff;
            if (lp.mlp == B200_MLP_DENSE_GATED) {
                ggml_tensor *gu = b.mul_mat(L.gate_up, h);
                ggml_tensor *act = b.ext(b.alloc_result(GGML_TYPE_F32, F, T), B200_EXT_SILU_MUL, {b.view_2d(gu, F, T, gu->nb[1], 0), b.view_2d(gu, F, T, gu->nb[1], (size_t)F * 4)});
                act->op_params[2] = lp.glu_kind;
                c = chain(one_result(b.mul_mat(L.down, act)), 1.0f, nullptr, x, B200_NORM_LAYER, L.n2b, L.n2b_b, next_w(!side), next_b(!side));
            } else {
                const int64_t NU = lp.n_expert_used, FS = lp.shared_ff, n_exp = (F * NU * T + 3) / 4 * 4;
                ggml_tensor *ids = b.view_2d(expert_ids, NU, T, expert_ids->nb[1], (size_t)L.table_col * 4);
                // the experts' and the shared expert's hidden rows share one buffer, so that one launch activates both
                ggml_tensor *hid = b.alloc_result(GGML_TYPE_F32, n_exp + FS * T);
                ggml_tensor *eu = b.ext(b.result_at(hid, 0, GGML_TYPE_F32, F, NU, T), B200_EXT_MUL_MAT_ID, {L.up, b.reshape(h, W, 1, T), ids});
                ggml_tensor *su = FS > 0 ? b.op(b.result_at(hid, (size_t)n_exp * 4, GGML_TYPE_F32, FS, T), GGML_OP_MUL_MAT, L.sh_up, h) : nullptr;
                ggml_tensor *act = b.ext(b.alloc_result(GGML_TYPE_F32, n_exp + FS * T), B200_EXT_UNARY, {hid, eu, su});
                act->op_params[2] = B200_UN_RELU_SQR;
                ggml_tensor *dn = b.ext(b.alloc_result(GGML_TYPE_F32, W, NU, T), B200_EXT_MUL_MAT_ID, {L.down, b.view_3d(act, F, NU, T, (size_t)F * 4, (size_t)(F * NU) * 4, 0), ids});
                ggml_tensor *sd = FS > 0 ? b.mul_mat(L.sh_down, b.view_2d(act, FS, T, (size_t)FS * 4, (size_t)n_exp * 4)) : nullptr;
                c = chain(dn, 1.0f / (float)NU, sd, x, B200_NORM_LAYER, L.n2b, L.n2b_b, next_w(!side), next_b(!side));
            }
            x = c.x; h = c.h;
        }
        if (side) {
            const int64_t ES = lp.token_side;
            ggml_tensor *a = b.mul_mat(L.side_gate, x);
            ggml_tensor *e = b.view_2d(side_rows, ES, T, side_rows->nb[1], (size_t)(il * ES) * 4);
            ggml_tensor *ge = b.ext(b.alloc_result(GGML_TYPE_F32, ES, T), B200_EXT_SILU_MUL, {a, e});
            ge->op_params[2] = B200_GLU_GELU_TANH;
            const Chained c = chain(one_result(b.mul_mat(L.side_proj, ge)), 1.0f, nullptr, x, B200_NORM_RMS, L.side_norm, nullptr, next_w(true), next_b(true));
            x = c.x; h = c.h;
        }
    }
    b.bump = &m->regions[R_TAIL];
    ggml_tensor *out = x;
    if (bs.n_outputs > 0) {
        if (bs.n_outputs < T) out = b.get_rows(out, input_view(m->inp_out_ids, bs.n_outputs));
        out = b.mul_mat(g->head, layer_norm(out, g->final_norm, g->final_norm_b));
    }
    b.expand(out);
    for (Bump &r : m->regions) LL_REQUIRE(m->measuring || r.off <= r.size, B200_ERR_NOMEM, "b200_llama_decode_batch: compute buffer too small for this batch");
    LL_REQUIRE(!b.oom, B200_ERR_NOMEM, "b200_llama_decode_batch: compute buffer too small for this batch");
    m->logits_t = bs.n_outputs > 0 ? out : nullptr;
    m->graph_nodes.swap(b.nodes);
    memset(&m->graph, 0, sizeof(m->graph));
    m->graph.size = m->graph.n_nodes = (int)m->graph_nodes.size();
    m->graph.nodes = m->graph_nodes.data();
    return B200_OK;
}

const Arch k_mafuzen = {"mafuzen", mf_place_tensor, mf_finalize, nullptr, mf_build, nullptr};

}  // namespace

const Arch *b200::host::mafuzen_arch() { return &k_mafuzen; }
