// host_tugezen.cu -- the Tugezen architecture for the decoder of host_llama.cu: where its tensors go and the graph of one batch
// step.  The decoder owns the model object, the sequence cache, the inputs and the step; this file adds no loop of its own.
//
// The stream starts as the embedding row.  A layer is pre-norm (RMS):  x <- x + mixer(N1(x));  x <- x + down(gelu(gate h) * up h) with
// h = N2(x)  (the second step may be absent).  Mixers (b200_layer_params):
//   * latent attention: queries through a normed latent, one normed latent per token from which every head's keys and values come, no
//     positions, a window, a sigmoid gate per head;
//   * attention beside the gated delta rule: the left side is grouped-query attention with (YaRN-scaled) rotation and soft-capped scores;
//     on the right q, k, v pass a short causal convolution and silu, q and k become unit vectors per head, and a state per head forgets
//     by a decay per token and key channel and is corrected towards v along k; every read-out is RMS-normed and gated by a sigmoid per
//     value.  The two results are scaled and added;
//   * gated linear attention: a state per head that forgets by sigmoid(z)^(1 / tau) per token and key channel; every read-out is
//     RMS-normed and gated by silu.
// The logits are logit_scale * head N(x).
//
// Graph choices: everything a mixer projects from its input is ONE product over row-concatenated weights; the first matrices of the
// low-rank projections stand at its front, padded with zero rows to a multiple of 64, so that their second matrices (decay and gate,
// one block each of one matrix) are one more product whose K fits the tensor-core tiles; the key up-projection is folded into the
// query and the value up-projection follows the attention, so that the cache holds and the attention reads the latents only, and it
// writes its heads side by side into the output product's input; the query latent's norm shares the launch of the cache store; the two
// output matrices of a parallel mixer lie side by side along K (left scale in the attention's epilogue, right scale in the norm
// weight); a residual sum and the norm that reads it are one launch (norm_chain), the model's last norm included, whose weight carries
// the logit scale.
#include <cfloat>

#include "host_fused.h"

namespace {

constexpr float kUnitEps = 1e-6f;  // q and k of the delta rule: x / sqrt(sum(x^2) + 1e-6)

struct TzLayer {
    ggml_tensor *n1 = nullptr, *n2 = nullptr, *proj1 = nullptr, *wo = nullptr;
    int64_t proj1_rows = 0;
    ggml_tensor *dq_norm = nullptr, *uq = nullptr, *dkv_norm = nullptr, *uk_t = nullptr, *uv = nullptr;      // latent attention
    ggml_tensor *low = nullptr;                                                                              // second matrices of the low-rank projections, [padded ranks, rows]
    ggml_tensor *convw = nullptr, *a_log = nullptr, *dt_bias = nullptr, *head_norm = nullptr, *freqs = nullptr;  // parallel
    float mscale = 1.0f;
    ggml_tensor *decay_bias = nullptr;                                                                       // gated linear attention
    ggml_tensor *gate_up = nullptr, *down = nullptr;
    ggml_tensor *cache = nullptr, *k_cache = nullptr, *v_cache = nullptr;                                    // rows by cell: latents; keys and values of the left side
    ggml_tensor *state = nullptr, *tail = nullptr;                                                           // per slot: S; the convolution's last inputs
};
struct HostMat { int type; int64_t ne0, ne1; std::vector<char> data; };
struct TzData {
    std::map<std::string, HostMat> mats;              // matrices that finalize joins
    std::map<std::string, std::vector<float>> vecs;   // vectors that finalize scales
    std::vector<TzLayer> layers;
    ggml_tensor *embed = nullptr, *head = nullptr, *final_norm = nullptr;
};
TzData *tz(b200_llama *m) {
    if (!m->arch_data) m->arch_data = std::shared_ptr<void>(new TzData(), [](void *p) { delete (TzData *)p; });
    return (TzData *)m->arch_data.get();
}

int64_t pad_to(int64_t v, int64_t to) { return (v + to - 1) / to * to; }
bool is_latent(const b200_layer_params &lp) { return lp.mixer == B200_MIXER_LATENT_ATTENTION; }
bool is_parallel(const b200_layer_params &lp) { return lp.mixer == B200_MIXER_ATTENTION_DELTA; }
bool is_gla(const b200_layer_params &lp) { return lp.mixer == B200_MIXER_GATED_LINEAR_ATTENTION; }
int64_t low_ranks(const b200_layer_params &lp) { return (int64_t)lp.decay_rank + (is_parallel(lp) ? lp.gate_rank : 0); }
int64_t conv_channels(const b200_layer_params &lp) { return 2 * (int64_t)lp.mix_kv_heads * lp.mix_dim + (int64_t)lp.mix_heads * lp.mix_vdim; }

// everything the mixer projects from its input, in the order of the rows of the fused matrix; parts named "" are zero rows
constexpr int kMaxParts = 12;
int parts_proj1(const b200_layer_params &lp, Part out[kMaxParts]) {
    int n = 0;
    int64_t total = 0;
    auto add = [&](const char *leaf, int64_t rows) { if (rows > 0) out[n++] = {leaf, rows}; total += rows; };
    const int64_t H = lp.heads, G = lp.kv_heads, D = lp.dim, V = lp.vdim;
    if (is_latent(lp)) {
        add("mix.dq", lp.q_rank); add("mix.dkv", lp.kv_rank); add("mix.g", H);
    } else if (is_parallel(lp)) {
        add("mix.right.a1", lp.decay_rank); add("mix.right.g1", lp.gate_rank); add("", pad_to(low_ranks(lp), 64) - low_ranks(lp));
        add("mix.left.q", H * D); add("mix.left.k", G * D); add("mix.left.v", G * V);
        // q, k, v of the right side are neighbours: one convolution covers them
        const int64_t GD = (int64_t)lp.mix_kv_heads * lp.mix_dim;
        add("mix.right.q", GD); add("mix.right.k", GD); add("mix.right.v", (int64_t)lp.mix_heads * lp.mix_vdim); add("mix.right.b", lp.mix_heads);
    } else {
        add("mix.a1", lp.decay_rank); add("", pad_to(low_ranks(lp), 64) - low_ranks(lp));
        add("mix.q", H * D); add("mix.k", H * D); add("mix.v", H * V); add("mix.g", H * V);
    }
    add("", pad_to(total, 8) - total);
    return n;
}
// the convolution weights of the right side's q, k, v as rows of one tensor
int parts_conv(const b200_layer_params &lp, Part out[3]) {
    const int64_t GD = (int64_t)lp.mix_kv_heads * lp.mix_dim;
    out[0] = {"mix.right.q.conv", GD}; out[1] = {"mix.right.k.conv", GD}; out[2] = {"mix.right.v.conv", (int64_t)lp.mix_heads * lp.mix_vdim};
    return 3;
}

int tz_place_tensor(b200_llama *m, const char *name, int type, int64_t ne0, int64_t ne1, int64_t ne2, const void *data) {
    const b200_llama_params &hp = m->hp;
    const int64_t W = hp.n_embd;
    auto keep_vec = [&](int64_t n) -> int {
        LL_REQUIRE(type == GGML_TYPE_F32 && ne0 == n && ne1 == 1 && ne2 == 1, B200_ERR_INVALID, "b200_llama_set_tensor: %s must be %lld f32 values", name, (long long)n);
        LL_REQUIRE(!tz(m)->vecs.count(name), B200_ERR_INVALID, "b200_llama_set_tensor: duplicate tensor %s", name);
        tz(m)->vecs[name].assign((const float *)data, (const float *)data + n);
        return B200_OK;
    };
    if (!strcmp(name, "final.norm")) return keep_vec(W);
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
#define TZ_SHAPE(rows, cols) LL_REQUIRE(ne0 == (cols) && ne1 == (rows), B200_ERR_INVALID, "b200_llama_set_tensor: %s is [%lld, %lld], expected [%lld, %lld]", name, (long long)ne1, (long long)ne0, \
                                        (long long)(rows), (long long)(cols))
    auto keep_mat = [&]() -> int {
        LL_REQUIRE(!tz(m)->mats.count(name), B200_ERR_INVALID, "b200_llama_set_tensor: duplicate tensor %s", name);
        tz(m)->mats[name] = HostMat{type, ne0, ne1, std::vector<char>((const char *)data, (const char *)data + (size_t)(ne0 * ne1) * es)};
        return B200_OK;
    };
    if (lp.mlp == B200_MLP_DENSE_GATED && (!strcmp(leaf, "mlp.gate") || !strcmp(leaf, "mlp.up"))) {
        TZ_SHAPE(lp.ff, W);
        const size_t bytes = (size_t)((int64_t)lp.ff * W) * es;
        return place_into(m, pre + "mlp.gate_up", name, type, W, 2 * (int64_t)lp.ff, 1, leaf[4] == 'u' ? bytes : 0, bytes, data);
    }
    Part parts[kMaxParts];
    const int np = parts_proj1(lp, parts);
    int64_t total = 0, rows = 0;
    const int64_t off = part_offset(parts, np, leaf, &total, &rows);
    if (off >= 0) {
        TZ_SHAPE(rows, W);
        const std::string fused = pre + "proj1";
        const bool first = find_w(m, fused) == nullptr;
        const int rc = place_into(m, fused, name, type, W, total, 1, (size_t)(off * W) * es, (size_t)(rows * W) * es, data);
        if (rc == B200_OK && first) {  // the rows between and behind the parts are zero weights: their results are zeros
            ggml_tensor *f = find_w(m, fused);
            int64_t at = 0;
            for (int i = 0; i < np; at += parts[i].rows, i++) {
                if (parts[i].leaf[0]) continue;
                const std::vector<char> z((size_t)(parts[i].rows * W) * es, 0);
                f->buffer->iface.set_tensor(f->buffer, f, z.data(), (size_t)(at * W) * es, z.size());
            }
        }
        return rc;
    }
    if (is_latent(lp) && !strcmp(leaf, "mix.uk")) {
        // [kv_rank, heads * dim] -> per head the transpose [dim, kv_rank]: the contraction with the query runs over dim
        const int64_t KR = lp.kv_rank, D = lp.dim, H = lp.heads;
        TZ_SHAPE(H * D, KR);
        std::vector<char> t((size_t)(KR * D * H) * es);
        const char *src = (const char *)data;
        for (int64_t h = 0; h < H; h++)
            for (int64_t d = 0; d < D; d++)
                for (int64_t r = 0; r < KR; r++) memcpy(&t[(size_t)((h * KR + r) * D + d) * es], src + (size_t)((h * D + d) * KR + r) * es, es);
        return upload_tensor(m, (pre + "mix.uk_t").c_str(), type, D, KR, H, t.data());
    }
    if (is_gla(lp) && !strcmp(leaf, "mix.a2")) { TZ_SHAPE((int64_t)lp.heads * lp.dim, lp.decay_rank); return keep_mat(); }
    if (is_parallel(lp)) {
        const int64_t HV = (int64_t)lp.mix_heads * lp.mix_vdim;
        if (!strcmp(leaf, "mix.right.a2")) { TZ_SHAPE((int64_t)lp.mix_heads * lp.mix_dim, lp.decay_rank); return keep_mat(); }
        if (!strcmp(leaf, "mix.right.g2")) { TZ_SHAPE(HV, lp.gate_rank); return keep_mat(); }
        if (!strcmp(leaf, "mix.left.o")) { TZ_SHAPE(W, (int64_t)lp.heads * lp.vdim); return keep_mat(); }
        if (!strcmp(leaf, "mix.right.o")) { TZ_SHAPE(W, HV); return keep_mat(); }
        if (!strcmp(leaf, "mix.right.norm")) return keep_vec(lp.mix_vdim);
        Part conv[3];
        const int64_t coff = part_offset(conv, parts_conv(lp, conv), leaf, &total, &rows);
        if (coff >= 0) {
            LL_REQUIRE(type == GGML_TYPE_F32, B200_ERR_INVALID, "b200_llama_set_tensor: %s must be uploaded as f32", name);
            TZ_SHAPE(rows, lp.conv_taps);
            return place_into(m, pre + "mix.convw", name, type, lp.conv_taps, total, 1, (size_t)(coff * lp.conv_taps) * 4, (size_t)(rows * lp.conv_taps) * 4, data);
        }
    }
#undef TZ_SHAPE
    return upload_tensor(m, name, type, ne0, ne1, ne2, data);
}

// blocks of one matrix: block b's rows stand below those of the blocks before it, its columns behind theirs (diagonal) or all blocks share the
// rows and stand side by side; everything else is zero.  `cols` >= the columns the blocks need.
struct Block { const HostMat *m; int64_t row, col; };
std::vector<char> join_blocks(const std::vector<Block> &blocks, int64_t rows, int64_t cols, size_t es) {
    std::vector<char> out((size_t)(rows * cols) * es, 0);
    for (const Block &b : blocks)
        for (int64_t r = 0; r < b.m->ne1; r++) memcpy(&out[(size_t)((b.row + r) * cols + b.col) * es], &b.m->data[(size_t)(r * b.m->ne0) * es], (size_t)b.m->ne0 * es);
    return out;
}

int tz_finalize(b200_llama *m) {
    const b200_llama_params &hp = m->hp;
    TzData *g = tz(m);
    g->layers.assign((size_t)hp.n_layer, TzLayer());
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
    // a tensor made here from uploaded ones
    auto make = [&](const std::string &nm, int type, int64_t ne0, int64_t ne1, const void *data) -> ggml_tensor * {
        return upload_tensor(m, nm.c_str(), type, ne0, ne1, 1, data) == B200_OK ? find_w(m, nm) : nullptr;
    };
    auto scaled_vec = [&](const std::string &out, const std::string &src, float factor) -> ggml_tensor * {
        auto it = g->vecs.find(src);
        if (it == g->vecs.end()) { b200::set_error("b200_llama_finalize: tensor %s missing", src.c_str()); return nullptr; }
        for (float &v : it->second) v *= factor;
        return make(out, GGML_TYPE_F32, (int64_t)it->second.size(), 1, it->second.data());
    };
    auto state = [&](const std::string &nm, int64_t floats, int64_t rows) -> ggml_tensor * {
        ggml_tensor *t = new_device_tensor(m, nm.c_str(), GGML_TYPE_F32, floats > 0 ? floats : 1, rows, true);
        if (t) m->kv_bytes += (int64_t)nbytes(t);
        else b200::set_error("b200_llama_finalize: out of device memory for %s", nm.c_str());
        return t;
    };
#define TZ_NEED(dst, ...) do { dst = need_at(__VA_ARGS__); if (!(dst)) return B200_ERR_INVALID; } while (0)
#define TZ_MAKE(dst, code, expr) do { dst = (expr); if (!(dst)) return code; } while (0)
    TZ_NEED(g->embed, "embed", W, hp.n_vocab); TZ_NEED(g->head, "head", W, hp.n_vocab);
    TZ_MAKE(g->final_norm, B200_ERR_INVALID, scaled_vec("final.scaled_norm", "final.norm", hp.logit_scale == 0.0f ? 1.0f : hp.logit_scale));
    for (int il = 0; il < hp.n_layer; il++) {
        const b200_layer_params &lp = m->layer_hp[(size_t)il];
        TzLayer &L = g->layers[(size_t)il];
        const std::string pre = "l" + std::to_string(il) + ".";
        const int64_t H = lp.heads, G = lp.kv_heads, D = lp.dim, V = lp.vdim;
        LL_REQUIRE(is_latent(lp) || is_parallel(lp) || is_gla(lp), B200_ERR_INVALID, "b200_llama_finalize: layer %d has no mixer of this architecture", il);
        LL_REQUIRE(H > 0 && D > 0 && V > 0 && (is_latent(lp) || D <= 256) && (!is_parallel(lp) || V <= 256), B200_ERR_UNSUPPORTED,
                   "b200_llama_finalize: layer %d: heads %d, dim %d and vdim %d (<= 256)", il, lp.heads, lp.dim, lp.vdim);
        TZ_NEED(L.n1, pre + "norm1", W, 1);
        Part parts[kMaxParts];
        const int np = parts_proj1(lp, parts);
        part_offset(parts, np, "?", &L.proj1_rows);
        for (int i = 0; i < np; i++) LL_REQUIRE(!parts[i].leaf[0] || find_w(m, pre + parts[i].leaf), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), parts[i].leaf);
        TZ_NEED(L.proj1, pre + "proj1", W, L.proj1_rows);
        auto mat = [&](const char *leaf) -> const HostMat * {
            auto it = g->mats.find(pre + leaf);
            if (it == g->mats.end()) { b200::set_error("b200_llama_finalize: tensor %s%s missing", pre.c_str(), leaf); return nullptr; }
            return &it->second;
        };
        const int64_t LR = pad_to(low_ranks(lp), 64);
        if (is_latent(lp)) {
            const int64_t KR = lp.kv_rank, QR = lp.q_rank;
            LL_REQUIRE(KR > 0 && KR <= 1024 && QR > 0 && lp.window >= 0, B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: latent sizes %d (<= 1024) and %d", il, lp.kv_rank, lp.q_rank);
            TZ_NEED(L.dq_norm, pre + "mix.dq.norm", QR, 1); TZ_NEED(L.uq, pre + "mix.uq", QR, H * D); TZ_NEED(L.dkv_norm, pre + "mix.dkv.norm", KR, 1);
            TZ_NEED(L.uk_t, pre + "mix.uk_t", D, KR, H); TZ_NEED(L.uv, pre + "mix.uv", KR, H * V); TZ_NEED(L.wo, pre + "mix.o", H * V, W);
            TZ_MAKE(L.cache, B200_ERR_NOMEM, state(pre + "cache", KR, hp.n_ctx));
        } else if (is_gla(lp)) {
            LL_REQUIRE(lp.decay_rank > 0 && lp.decay_tau > 0.0f, B200_ERR_INVALID, "b200_llama_finalize: layer %d: the decay needs a rank and a positive tau", il);
            TZ_NEED(L.wo, pre + "mix.o", H * V, W); TZ_NEED(L.head_norm, pre + "mix.norm", V, 1); TZ_NEED(L.decay_bias, pre + "mix.a2.b", H * D, 1);
            const HostMat *a2;
            TZ_MAKE(a2, B200_ERR_INVALID, mat("mix.a2"));
            const std::vector<char> low = join_blocks({{a2, 0, 0}}, H * D, LR, (size_t)type_traits(a2->type).size);
            TZ_MAKE(L.low, B200_ERR_NOMEM, make(pre + "mix.low", a2->type, LR, H * D, low.data()));
            TZ_MAKE(L.state, B200_ERR_NOMEM, state(pre + "state", H * D * V, hp.n_seq_max));
        } else {
            const int64_t HR = lp.mix_heads, GR = lp.mix_kv_heads, DR = lp.mix_dim, VR = lp.mix_vdim;
            LL_REQUIRE(G > 0 && H % G == 0 && lp.rope_dims >= 0 && lp.rope_dims % 2 == 0 && lp.rope_dims <= D && (lp.rope_dims == 0 || lp.rope_base > 0.0f) && lp.attn_softcap >= 0.0f,
                       B200_ERR_INVALID, "b200_llama_finalize: layer %d: heads %d over %d kv heads, rotation of %d of %d values, soft cap", il, lp.heads, lp.kv_heads, lp.rope_dims, lp.dim);
            LL_REQUIRE(lp.rope_scaling == B200_ROPE_SCALING_NONE || (lp.rope_scaling == B200_ROPE_SCALING_YARN && lp.yarn_factor > 0.0f && lp.yarn_original > 0 && lp.yarn_fast > 0.0f &&
                       lp.yarn_slow > 0.0f && lp.rope_base != 1.0f), B200_ERR_INVALID, "b200_llama_finalize: layer %d: frequency scaling", il);
            LL_REQUIRE(HR > 0 && GR > 0 && HR % GR == 0 && DR > 0 && DR <= 256 && VR > 0, B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: delta rule with %d heads over %d of %d (<= 256)", il,
                       lp.mix_heads, lp.mix_kv_heads, lp.mix_dim);
            LL_REQUIRE(lp.conv_taps >= 1 && lp.conv_taps <= 17, B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: a convolution of 1 to 17 taps", il);
            LL_REQUIRE(lp.decay_rank > 0 && lp.gate_rank > 0, B200_ERR_INVALID, "b200_llama_finalize: layer %d: decay and gate need ranks", il);
            TZ_NEED(L.a_log, pre + "mix.right.A_log", HR, 1); TZ_NEED(L.dt_bias, pre + "mix.right.dt_bias", HR * DR, 1);
            Part conv[3];
            for (int i = 0; i < parts_conv(lp, conv); i++) LL_REQUIRE(find_w(m, pre + conv[i].leaf), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), conv[i].leaf);
            TZ_NEED(L.convw, pre + "mix.convw", lp.conv_taps, conv_channels(lp));
            TZ_MAKE(L.head_norm, B200_ERR_INVALID, scaled_vec(pre + "mix.right.scaled_norm", pre + "mix.right.norm", lp.right_scale));
            const HostMat *a2, *g2, *ol, *orr;
            TZ_MAKE(a2, B200_ERR_INVALID, mat("mix.right.a2")); TZ_MAKE(g2, B200_ERR_INVALID, mat("mix.right.g2"));
            TZ_MAKE(ol, B200_ERR_INVALID, mat("mix.left.o")); TZ_MAKE(orr, B200_ERR_INVALID, mat("mix.right.o"));
            LL_REQUIRE(a2->type == g2->type && ol->type == orr->type, B200_ERR_INVALID, "b200_llama_finalize: layer %d: joined matrices of two types", il);
            const std::vector<char> low = join_blocks({{a2, 0, 0}, {g2, HR * DR, lp.decay_rank}}, HR * (DR + VR), LR, (size_t)type_traits(a2->type).size);
            TZ_MAKE(L.low, B200_ERR_NOMEM, make(pre + "mix.low", a2->type, LR, HR * (DR + VR), low.data()));
            const std::vector<char> o = join_blocks({{ol, 0, 0}, {orr, 0, H * V}}, W, H * V + HR * VR, (size_t)type_traits(ol->type).size);
            TZ_MAKE(L.wo, B200_ERR_NOMEM, make(pre + "mix.o", ol->type, H * V + HR * VR, W, o.data()));
            if (lp.rope_dims > 0) {
                std::vector<float> f;
                rope_freqs(lp, f, &L.mscale);
                TZ_MAKE(L.freqs, B200_ERR_NOMEM, make(pre + "rope_freqs", GGML_TYPE_F32, (int64_t)f.size(), 1, f.data()));
            }
            TZ_MAKE(L.k_cache, B200_ERR_NOMEM, state(pre + "k", G * D, hp.n_ctx)); TZ_MAKE(L.v_cache, B200_ERR_NOMEM, state(pre + "v", G * V, hp.n_ctx));
            TZ_MAKE(L.state, B200_ERR_NOMEM, state(pre + "state", HR * DR * VR, hp.n_seq_max));
            TZ_MAKE(L.tail, B200_ERR_NOMEM, state(pre + "tail", (int64_t)(lp.conv_taps - 1) * conv_channels(lp), hp.n_seq_max));
        }
        if (lp.mlp == B200_MLP_NONE) continue;
        LL_REQUIRE(lp.mlp == B200_MLP_DENSE_GATED && lp.ff > 0, B200_ERR_UNSUPPORTED, "b200_llama_finalize: layer %d: feed-forward kind %d", il, lp.mlp);
        TZ_NEED(L.n2, pre + "norm2", W, 1);
        for (const char *w : {"mlp.gate", "mlp.up"}) LL_REQUIRE(find_w(m, pre + w), B200_ERR_INVALID, "b200_llama_finalize: tensor %s%s missing", pre.c_str(), w);
        TZ_NEED(L.gate_up, pre + "mlp.gate_up", W, 2 * (int64_t)lp.ff); TZ_NEED(L.down, pre + "mlp.down", lp.ff, W);
    }
#undef TZ_NEED
#undef TZ_MAKE
    g->mats.clear(); g->vecs.clear();
    return B200_OK;
}

// ------------------------------------------------------------------------------------------------ graph of one batch step
enum { R_HEAD = 0, R_EVEN = 1, R_ODD = 2, R_TAIL = 3 };

int tz_build(b200_llama *m, const BatchShape &bs) {
    const b200_llama_params &hp = m->hp;
    TzData *g = tz(m);
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
    // bf16 weights: the attention products of a prompt batch may be bf16 as well (B200_ATTN_F32=1 keeps them in f32)
    static const bool attn_f32 = getenv("B200_ATTN_F32") != nullptr;

    // x' = x + y and the norm of x' that comes next, one launch
    struct Chained { ggml_tensor *x, *h; };
    auto chain = [&](ggml_tensor *y, ggml_tensor *x, ggml_tensor *w) {
        ggml_tensor *dst = b.alloc_result(GGML_TYPE_F32, W, T, 2);
        b.ext(dst, B200_EXT_NORM_CHAIN, {b.view_3d(y, W, 1, T, y->nb[1], y->nb[1], 0), nullptr, nullptr, x, nullptr, nullptr, w, nullptr});
        dst->op_params[2] = B200_NORM_NONE; Builder::set_f(dst, 3, eps); dst->op_params[4] = B200_NORM_RMS; Builder::set_f(dst, 5, 1.0f);
        return Chained{b.view_2d(dst, W, T, dst->nb[1], 0), b.view_2d(dst, W, T, dst->nb[1], dst->nb[2])};
    };
    // every head's read-out: RMS norm over its values, the weight all heads share, times f of a gate per value (f: 1 sigmoid, 2 silu)
    auto head_norm = [&](ggml_tensor *o, ggml_tensor *dst, ggml_tensor *w, ggml_tensor *gate, int gate_kind) {
        b.ext(dst, B200_EXT_NORM, {o, w, gate, nullptr, nullptr, nullptr});
        dst->op_params[2] = B200_NORM_RMS; Builder::set_f(dst, 3, eps); dst->op_params[4] = 1; dst->op_params[5] = gate_kind;
        return dst;
    };
    // the rows [cols, T] of `whole` once `part`, and with it whatever `also` stands for, has been written
    auto written = [&](ggml_tensor *whole, ggml_tensor *part, ggml_tensor *also = nullptr) {
        ggml_tensor *t = b.view_of(part, GGML_OP_VIEW, 0);
        set_shape(t, GGML_TYPE_F32, whole->ne[0], T, 1, 1);
        t->nb[1] = whole->nb[1]; t->nb[2] = t->nb[3] = t->nb[1] * (size_t)T;
        t->data = whole->data; t->view_src = whole; t->view_offs = 0; t->src[1] = also;
        return t;
    };

    b.bump = &m->regions[R_HEAD];
    ggml_tensor *x = b.op(b.alloc_result(GGML_TYPE_F32, W, T), GGML_OP_GET_ROWS, g->embed, tokens);
    ggml_tensor *h = b.ext(b.alloc_result(GGML_TYPE_F32, W, T), B200_EXT_NORM, {x, g->layers[0].n1, nullptr, nullptr, nullptr, nullptr});
    h->op_params[2] = B200_NORM_RMS; Builder::set_f(h, 3, eps); h->op_params[4] = 1;

    for (int il = 0; il < hp.n_layer; il++) {
        const b200_layer_params &lp = m->layer_hp[(size_t)il];
        TzLayer &L = g->layers[(size_t)il];
        ggml_tensor *next_norm = il + 1 < hp.n_layer ? g->layers[(size_t)il + 1].n1 : g->final_norm;
        b.bump = &m->regions[(il & 1) ? R_ODD : R_EVEN];
        b.bump->off = 0;
        const int64_t H = lp.heads, G = lp.kv_heads, D = lp.dim, V = lp.vdim;
        const bool bf16 = L.proj1->type == GGML_TYPE_BF16 && !attn_f32;
        ggml_tensor *P = b.mul_mat(L.proj1, h);
        Part parts[kMaxParts];
        const int np = parts_proj1(lp, parts);
        auto part_at = [&](const char *leaf) { return (size_t)part_offset(parts, np, leaf, nullptr) * 4; };
        auto part = [&](const char *leaf) {
            int64_t rows = 0;
            const int64_t off = part_offset(parts, np, leaf, nullptr, &rows);
            return b.view_2d(P, rows, T, P->nb[1], (size_t)off * 4);
        };
        ggml_tensor *y;  // the mixer's result [W, T]
        if (is_latent(lp)) {
            const int64_t KR = lp.kv_rank;
            // one launch norms the latents: the tokens' own into their cache rows, the queries' where they lie
            ggml_tensor *st = b.view_2d(L.cache, KR, hp.n_ctx, L.cache->nb[1], 0);
            b.ext(st, B200_EXT_LATENT_KV_STORE, {part("mix.dkv"), L.dkv_norm, pos, nullptr, cells, L.cache, part("mix.dq"), L.dq_norm});
            st->op_params[2] = (int32_t)KR; Builder::set_f(st, 3, eps); Builder::set_f(st, 4, 1.0f); st->op_params[5] = 0;
            ggml_tensor *cq = part("mix.dq");
            cq->src[0] = st;
            ggml_tensor *q = b.mul_mat(L.uq, cq);                                                                    // [H * D, T]
            ggml_tensor *q_lat = b.permute(b.mul_mat(L.uk_t, b.view_3d(q, D, T, H, q->nb[1], (size_t)D * 4, 0)), 0, 2, 1, 3);  // [KR, T, H] seen as [KR, H, T]
            ggml_tensor *o_lat = b.alloc_result(GGML_TYPE_F32, KR, T, H);
            b.ext(o_lat, B200_EXT_LATENT_ATTN, {q_lat, nullptr, st, nullptr, tok_seq, pos, cell_seq, cell_pos, part("mix.g")});
            o_lat->op_params[2] = (int32_t)KR; Builder::set_f(o_lat, 3, lp.scale); o_lat->op_params[4] = lp.window; o_lat->op_params[5] = bf16;
            // every head's values land in its own columns of the output product's input
            ggml_tensor *o = b.alloc_result(GGML_TYPE_F32, H * V, T);
            ggml_tensor *oh = b.result_at(o, 0, GGML_TYPE_F32, V, T, H);
            oh->nb[1] = o->nb[1]; oh->nb[2] = (size_t)V * 4; oh->nb[3] = oh->nb[2] * (size_t)H;
            b.op(oh, GGML_OP_MUL_MAT, b.view_3d(L.uv, KR, V, H, L.uv->nb[1], L.uv->nb[1] * (size_t)V, 0), o_lat);
            y = b.mul_mat(L.wo, written(o, oh));
        } else if (is_gla(lp)) {
            ggml_tensor *z = b.mul_mat(L.low, b.view_2d(P, L.low->ne[0], T, P->nb[1], 0));
            ggml_tensor *o = b.alloc_result(GGML_TYPE_F32, H * V, T);
            b.ext(o, B200_EXT_LINEAR_ATTN_SCAN, {part("mix.q"), part("mix.k"), part("mix.v"), nullptr, seq_info, L.state, nullptr, nullptr, z, L.decay_bias});
            o->op_params[2] = (int32_t)H; o->op_params[3] = (int32_t)D; o->op_params[4] = (int32_t)V; o->op_params[5] = 0;
            Builder::set_f(o, 6, 1.0f / sqrtf((float)D)); o->op_params[7] = 0; Builder::set_f(o, 8, lp.decay_tau);  // the factor of the queries, taken on the keys
            ggml_tensor *on = head_norm(b.reshape(o, V, H, T), b.alloc_result(GGML_TYPE_F32, V, H, T), L.head_norm, b.view_3d(P, V, H, T, (size_t)V * 4, P->nb[1], part_at("mix.g")), 2);
            y = b.mul_mat(L.wo, b.reshape(on, H * V, T));
        } else {
            const int64_t HR = lp.mix_heads, GR = lp.mix_kv_heads, DR = lp.mix_dim, VR = lp.mix_vdim, CC = conv_channels(lp);
            ggml_tensor *both = b.alloc_result(GGML_TYPE_F32, H * V + HR * VR, T);  // [left | right], the input of the joined output product
            // left: rotate, store, attend
            ggml_tensor *q = part("mix.left.q"), *qo = part("mix.left.q");  // the store rewrites q in place
            b.ext(qo, B200_EXT_QKV_STORE, {q, part("mix.left.k"), part("mix.left.v"), nullptr, pos, L.freqs, cells, b.view_2d(L.k_cache, G * D, hp.n_ctx, L.k_cache->nb[1], 0),
                                            b.view_2d(L.v_cache, G * V, hp.n_ctx, L.v_cache->nb[1], 0)});
            qo->op_params[2] = (int32_t)D; qo->op_params[3] = (int32_t)V; qo->op_params[4] = lp.rope_dims; Builder::set_f(qo, 5, eps);
            qo->op_params[6] = qo->op_params[7] = qo->op_params[8] = qo->op_params[9] = 0; Builder::set_f(qo, 10, 0.0f); qo->op_params[11] = 1; Builder::set_f(qo, 12, L.mscale);
            ggml_tensor *ol = b.result_at(both, 0, GGML_TYPE_F32, H * V, T);
            ol->nb[1] = both->nb[1]; ol->nb[2] = ol->nb[3] = ol->nb[1] * (size_t)T;
            b.ext(ol, B200_EXT_SINK_ATTN, {qo, b.view_2d(L.k_cache, G * D, bs.n_kv, L.k_cache->nb[1], 0), b.view_2d(L.v_cache, G * V, bs.n_kv, L.v_cache->nb[1], 0), nullptr, tok_seq, pos,
                                           cell_seq, cell_pos, nullptr, nullptr});
            ol->op_params[2] = (int32_t)D; Builder::set_f(ol, 3, lp.scale); ol->op_params[4] = ol->op_params[5] = 0; ol->op_params[6] = bf16;
            ol->op_params[7] = (int32_t)V; ol->op_params[8] = 0; ol->op_params[9] = B200_ATTN_SOFTMAX; ol->op_params[10] = 0;
            Builder::set_f(ol, 11, lp.left_scale == 0.0f ? FLT_MIN : lp.left_scale); Builder::set_f(ol, 12, lp.attn_softcap);
            // right: q, k, v are neighbours in P: one convolution, and the same offsets hold in its result
            const size_t q_at = part_at("mix.right.q");
            ggml_tensor *C = b.ext(b.alloc_result(GGML_TYPE_F32, CC, T), B200_EXT_SHORT_CONV, {b.view_2d(P, CC, T, P->nb[1], q_at), L.convw, nullptr, seq_info, L.tail});
            C->op_params[2] = 1;
            ggml_tensor *z = b.mul_mat(L.low, b.view_2d(P, L.low->ne[0], T, P->nb[1], 0));  // per token the decays' and the gates' pre-activations
            ggml_tensor *o = b.alloc_result(GGML_TYPE_F32, HR * VR, T);
            b.ext(o, B200_EXT_DELTA_RULE_SCAN, {b.view_2d(C, GR * DR, T, C->nb[1], 0), b.view_2d(C, GR * DR, T, C->nb[1], (size_t)(GR * DR) * 4), b.view_2d(C, HR * VR, T, C->nb[1], (size_t)(2 * GR * DR) * 4),
                                                b.view_2d(z, HR * DR, T, z->nb[1], 0), part("mix.right.b"), L.a_log, L.dt_bias, seq_info, L.state});
            o->op_params[2] = (int32_t)HR; o->op_params[3] = (int32_t)GR; o->op_params[4] = (int32_t)DR; o->op_params[5] = (int32_t)VR; o->op_params[6] = 1;
            Builder::set_f(o, 7, kUnitEps); Builder::set_f(o, 8, 1.0f / sqrtf((float)DR));
            ggml_tensor *orr = b.result_at(both, (size_t)(H * V) * 4, GGML_TYPE_F32, VR, HR, T);
            orr->nb[2] = both->nb[1]; orr->nb[3] = orr->nb[2] * (size_t)T;
            head_norm(b.reshape(o, VR, HR, T), orr, L.head_norm, b.view_3d(z, VR, HR, T, (size_t)VR * 4, z->nb[1], (size_t)(HR * DR) * 4), 1);
            y = b.mul_mat(L.wo, written(both, orr, ol));
        }
        const bool mlp = lp.mlp != B200_MLP_NONE;
        Chained c = chain(y, x, mlp ? L.n2 : next_norm);
        x = c.x; h = c.h;
        if (!mlp) continue;
        const int64_t F = lp.ff;
        ggml_tensor *gu = b.mul_mat(L.gate_up, h);
        ggml_tensor *act = b.ext(b.alloc_result(GGML_TYPE_F32, F, T), B200_EXT_SILU_MUL, {b.view_2d(gu, F, T, gu->nb[1], 0), b.view_2d(gu, F, T, gu->nb[1], (size_t)F * 4)});
        act->op_params[2] = lp.glu_kind;
        c = chain(b.mul_mat(L.down, act), x, next_norm);
        x = c.x; h = c.h;
    }
    b.bump = &m->regions[R_TAIL];
    ggml_tensor *out = h;  // the last step's norm is the model's
    if (bs.n_outputs > 0) {
        if (bs.n_outputs < T) out = b.get_rows(out, input_view(m->inp_out_ids, bs.n_outputs));
        out = b.mul_mat(g->head, out);
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

const Arch k_tugezen = {"tugezen", tz_place_tensor, tz_finalize, nullptr, tz_build, nullptr};

}  // namespace

const Arch *b200::host::tugezen_arch() { return &k_tugezen; }
