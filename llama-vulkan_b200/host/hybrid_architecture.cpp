#include "hybrid_architecture.h"

#include <algorithm>
#include <cmath>
#include <iostream>

#include "hybrid_session_state.h"
#include "llava_buffer.h"
#include "llava_command_buffer.h"
#include "llava_context.h"
#include "llava_device_memory.h"
#include "llava_session.h"
#include "model_folder.h"

using namespace std;

// ---- configuration ---------------------------------------------------------------------------

namespace {
bool need_u32(const json_value* at, const char* key, u32* out, string* error, u32 least = 1) {
    const json_value* v = at ? at->find(key) : nullptr;
    if (v && v->as_u32(out) && *out >= least) return true;
    *error = string(key) + " missing or out of range";
    return false;
}

bool need_float(const json_value* at, const char* key, float* out, string* error) {
    const json_value* v = at ? at->find(key) : nullptr;
    if (v && v->as_float(out)) return true;
    *error = string(key) + " missing or not a number";
    return false;
}

bool need_double(const json_value* at, const char* key, double* out, string* error) {
    const json_value* v = at ? at->find(key) : nullptr;
    if (v && v->is_number() && isfinite(v->number())) {
        *out = v->number();
        return true;
    }
    *error = string(key) + " missing or not a number";
    return false;
}

bool given(const json_value* v) { return v != nullptr && !v->is_null(); }

const json_value* need_layers(const json_value& config, string* error) {
    const json_value* layers = config.find("layers");
    if (layers && layers->is_array() && !layers->items().empty()) return layers;
    *error = "layers missing";
    return nullptr;
}
}  // namespace

hybrid_rotation make_rotation(u32 dims, double base, const rotary_scaling* s) {
    hybrid_rotation r;
    for (u32 i = 0; i < dims / 2; ++i) r.freqs.push_back(pow(base, -2.0 * i / dims));
    if (s == nullptr) return r;
    auto pair_of = [&](double turns) { return dims * log(s->original / (2 * M_PI * turns)) / (2 * log(base)); };
    const double lo = max(floor(pair_of(s->fast)), 0.0), hi = min(ceil(pair_of(s->slow)), double(dims) - 1);
    for (u32 i = 0; i < dims / 2; ++i) {
        const double ramp = clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0);
        r.freqs[i] = r.freqs[i] / s->factor * ramp + r.freqs[i] * (1 - ramp);
    }
    r.mult = float(0.1 * log(s->factor) + 1);
    return r;
}

bool parse_sonuzen_config(const json_value& config, hybrid_config* out, string* error) {
    hybrid_config& c = *out;
    if (!need_u32(&config, "width", &c.width, error) || !need_u32(&config, "vocab", &c.vocab, error) ||
        !need_float(config.find("norm"), "eps", &c.eps, error) || !need_float(&config, "residual_mult", &c.residual_mult, error) ||
        !need_float(&config, "logit_scale", &c.logit_scale, error) || !need_u32(config.find("canon"), "taps", &c.taps, error))
        return false;
    const json_value* layers = need_layers(config, error);
    if (!layers) return false;
    for (const json_value& l : layers->items()) {
        hybrid_layer_spec spec;
        const json_value *type = l.find("type"), *mixer = l.find("mixer"), *mlp = l.find("mlp");
        hybrid_mixer& m = spec.mixer;
        if (type && type->text() == "attention") {
            m.type = hybrid_mixer::kind::attention;
            m.sink = true;
            if (!need_u32(mixer, "heads", &m.heads, error) || !need_u32(mixer, "kv_heads", &m.kv_heads, error) || !need_u32(mixer, "dim", &m.dim, error) ||
                !need_u32(mixer, "vdim", &m.vdim, error) || !need_float(mixer, "scale", &m.scale, error))
                return false;
            if (m.heads % m.kv_heads != 0) {
                *error = "heads must be a multiple of kv_heads";
                return false;
            }
        } else if (type && type->text() == "mingru") {
            m.type = hybrid_mixer::kind::mingru;
            if (!need_u32(mixer, "width", &m.width, error)) return false;
        } else {
            *error = "unknown layer type";
            return false;
        }
        if (given(mlp)) {
            const json_value* kind = mlp->find("kind");
            if (kind && kind->text() != "moe") {
                *error = "unknown feed-forward " + kind->text();
                return false;
            }
            const json_value* router = mlp->find("router");
            if (!need_u32(mlp->find("expert"), "ff", &spec.mlp.ff, error) || !need_u32(router, "experts", &spec.mlp.experts, error) ||
                !need_u32(router, "top", &spec.mlp.top, error))
                return false;
            if (spec.mlp.top > spec.mlp.experts) {
                *error = "top exceeds experts";
                return false;
            }
        }
        c.layers.push_back(spec);
    }
    if (const json_value* loop = config.find("loop"); loop && !loop->is_null()) {
        if (!need_u32(loop, "start", &c.loop_start, error, 0) || !need_u32(loop, "stop", &c.loop_stop, error) || !need_u32(loop, "times", &c.loop_times, error)) return false;
        if (c.loop_start >= c.loop_stop || c.loop_stop > c.layers.size()) {
            *error = "loop outside the layers";
            return false;
        }
    }
    return true;
}

// Nuforax: attention over latent caches and Mamba-2 layers with dense feed-forwards, norms on the outputs of the sublayers only,
// an embedding of token pairs, the embedding table as the output matrix.
bool parse_nuforax_config(const json_value& config, hybrid_config* out, string* error) {
    hybrid_config& c = *out;
    c.pre_norm = false;
    c.plain_norm = c.tied_head = true;
    const json_value *embedding = config.find("embedding"), *bigram = embedding ? embedding->find("bigram") : nullptr;
    if (!need_u32(&config, "width", &c.width, error) || !need_u32(&config, "vocab", &c.vocab, error) ||
        !need_float(config.find("norm"), "eps", &c.eps, error) || !need_float(embedding, "scale", &c.embed_scale, error) ||
        !need_u32(bigram, "buckets", &c.pair_buckets, error) || !need_u32(bigram, "mul_prev", &c.pair_mul_prev, error, 0) ||
        !need_u32(bigram, "mul_cur", &c.pair_mul_cur, error, 0))
        return false;
    const json_value* layers = need_layers(config, error);
    if (!layers) return false;
    auto bad = [&](const char* why) {
        *error = why;
        return false;
    };
    for (const json_value& l : layers->items()) {
        hybrid_layer_spec spec;
        const json_value *type = l.find("type"), *mixer = l.find("mixer"), *mlp = l.find("mlp");
        hybrid_mixer& m = spec.mixer;
        if (type && type->text() == "latent_attention") {
            m.type = hybrid_mixer::kind::latent;
            m.sink = true;
            const json_value *rot = mixer ? mixer->find("rot") : nullptr, *scaling = rot ? rot->find("scaling") : nullptr, *from = mixer ? mixer->find("kv_from") : nullptr;
            u32 dims = 0;
            double base = 0;
            if (!need_u32(mixer, "heads", &m.heads, error) || !need_u32(mixer, "dim", &m.dim, error) || !need_u32(mixer, "rot_dim", &m.rot, error) ||
                !need_u32(mixer, "vdim", &m.vdim, error) || !need_u32(mixer, "kv_rank", &m.kv_rank, error) || !need_float(mixer, "scale", &m.scale, error) ||
                !need_u32(mixer->find("mask"), "size", &m.window, error) || !need_u32(rot, "dims", &dims, error) || !need_double(rot, "base", &base, error))
                return false;
            if (dims % 2 != 0 || dims > m.rot || base <= 0) return bad("rot.dims must be even and at most rot_dim");
            rotary_scaling s{};
            if (given(scaling)) {
                if (!need_double(scaling, "factor", &s.factor, error) || !need_double(scaling, "original", &s.original, error) ||
                    !need_double(scaling, "fast", &s.fast, error) || !need_double(scaling, "slow", &s.slow, error))
                    return false;
                if (s.factor <= 0 || s.original <= 0 || s.fast <= 0 || s.slow <= 0 || base == 1) return bad("rot.scaling out of range");
            }
            hybrid_rotation r = make_rotation(dims, base, given(scaling) ? &s : nullptr);
            m.rot_pairs = dims / 2;
            while (m.rotation < c.rotations.size() && (c.rotations[m.rotation].freqs != r.freqs || c.rotations[m.rotation].mult != r.mult)) ++m.rotation;
            if (m.rotation == c.rotations.size()) {
                r.first = c.rotation_pairs();
                c.rotations.push_back(r);
            }
            if (given(from)) {
                u32 source = 0;
                if (!from->as_u32(&source) || source >= c.layers.size()) return bad("kv_from is not an earlier layer");
                const hybrid_mixer& o = c.layers[source].mixer;
                if (!o.has_own_cache() || o.kv_rank != m.kv_rank || o.rot != m.rot || o.rotation != m.rotation) return bad("kv_from names a layer without such a cache");
                m.kv_from = int(source);
            }
        } else if (type && type->text() == "mamba2") {
            m.type = hybrid_mixer::kind::ssm;
            if (!need_u32(mixer, "heads", &m.heads, error) || !need_u32(mixer, "vdim", &m.vdim, error) || !need_u32(mixer, "state", &m.state, error) ||
                !need_u32(mixer, "groups", &m.groups, error) || !need_u32(mixer, "conv", &m.taps, error) || !need_u32(mixer, "norm_groups", &m.norm_groups, error))
                return false;
            if (m.heads % m.groups != 0) return bad("heads must be a multiple of groups");
            if (u64(m.heads) * m.vdim % m.norm_groups != 0) return bad("norm_groups must divide the inner width");
        } else {
            return bad("unknown layer type");
        }
        if (given(mlp)) {
            const json_value* kind = mlp->find("kind");
            if (kind && kind->text() != "dense") {
                *error = "unknown feed-forward " + kind->text();
                return false;
            }
            if (!need_u32(mlp, "ff", &spec.dense.ff, error)) return false;
            spec.dense.act = LV_ACT_RELU2;
        }
        c.layers.push_back(spec);
    }
    return true;
}

// ---- model -----------------------------------------------------------------------------------

hybrid_architecture::~hybrid_architecture() {
    for (llava_buffer* b : tensors) delete b;
    delete rot_freqs;
    delete rot_mults;
}

bool hybrid_architecture::check(const model_file& model, u32 n_ranks) {
    string error;
    const auto* folder = dynamic_cast<const model_folder*>(&model);
    if (folder == nullptr || !parse_(folder->get_config(), &cfg, &error)) {
        cerr << "[!] " << name_ << ": bad configuration: " << error << endl;
        return false;
    }
    if (n_ranks != 1) {
        cerr << "[!] " << name_ << " models run on one GPU" << endl;
        return false;
    }
    for (const hybrid_layer_spec& l : cfg.layers) {
        const hybrid_mixer& m = l.mixer;
        const char* why = nullptr;
        if (m.type == hybrid_mixer::kind::attention && (m.dim > 256 || m.vdim > 256)) why = "heads of more than 256 values";
        if (m.type == hybrid_mixer::kind::latent && m.kv_rank > 1024) why = "latents of more than 1024 values";
        if (m.type == hybrid_mixer::kind::ssm && (m.state > 256 || m.taps > 16)) why = "states of more than 256 rows or convolutions of more than 16 taps";
        if (why) {
            cerr << "[!] " << name_ << ": " << why << " are not supported" << endl;
            return false;
        }
    }
    if (cfg.width > 16384 || cfg.taps > 16) {
        cerr << "[!] " << name_ << ": width above 16384 or more than 16 taps" << endl;
        return false;
    }
    const u32 n = u32(cfg.layers.size());
    const u32 first = cfg.loop_times ? cfg.loop_start : n, last = cfg.loop_times ? cfg.loop_stop : n;
    for (u32 i = 0; i < first; ++i) runs.push_back({i, -1});
    for (u32 t = 0; t < cfg.loop_times; ++t)
        for (u32 i = first; i < last; ++i) runs.push_back({i, i == first ? int(t) : -1});
    for (u32 i = last; i < n; ++i) runs.push_back({i, -1});
    vector<u32> latest(n, 0);            // last run of each layer so far
    for (u32 r = 0; r < runs.size(); ++r) {
        const hybrid_mixer& m = cfg.layers[runs[r].layer].mixer;
        runs[r].cache_run = m.kv_from < 0 ? r : latest[m.kv_from];
        latest[runs[r].layer] = r;
    }
    return true;
}

bool hybrid_architecture::build(llava_context* ctx) {
    const model_file* model = ctx->get_model();
    bool ok = true;
    auto find = [&](const string& name, u32 rows, u32 cols, weight_form form) -> const ggml_data_descriptor* {
        const ggml_data_descriptor* d = model->find_buffer_descriptor(name);
        const bool ints = form == weight_form::ids_u32, matrix = form == weight_form::rows_bf16;
        if (d && d->shape1 == rows && d->shape2 == cols &&
            (ints ? d->ftype == ggml_value_type::i32 : d->ftype == ggml_value_type::bf16 || (!matrix && d->ftype == ggml_value_type::f32)))
            return d;
        cerr << "[!] tensor " << name << (d ? " has another shape or type" : " missing") << endl;
        ok = false;
        return nullptr;
    };
    auto stack = [&](const vector<pair<string, u32>>& names_rows, u32 cols, weight_form form) -> llava_buffer* {
        vector<const ggml_data_descriptor*> parts;
        for (const auto& [name, rows] : names_rows)
            if (const ggml_data_descriptor* d = find(name, rows, cols, form)) parts.push_back(d);
        if (parts.size() != names_rows.size()) return nullptr;
        tensors.push_back(new llava_buffer(ctx, parts, form, ctx->weights_memory()));
        return tensors.back();
    };
    auto matrix = [&](const string& name, u32 rows, u32 cols) { return stack({{name, rows}}, cols, weight_form::rows_bf16); };
    auto values = [&](const string& name, u32 rows, u32 cols = 1) { return stack({{name, rows}}, cols, weight_form::vector_f32); };

    embed = matrix("embed", cfg.vocab, cfg.width);
    head = cfg.tied_head ? embed : matrix("head", cfg.vocab, cfg.width);
    if (cfg.pair_buckets) pair_embed = matrix("bigram", cfg.pair_buckets + 1, cfg.width);
    final_norm = values("final.norm", cfg.width);
    if (cfg.loop_times) loop_step = values("loop.step", cfg.loop_times, cfg.width);
    if (const u32 pairs = cfg.rotation_pairs()) {
        rot_freqs = new llava_buffer(ctx, ggml_value_type::f32, 2, pairs, ctx->weights_memory());
        rot_mults = new llava_buffer(ctx, ggml_value_type::f32, pairs, 1, ctx->weights_memory());
    }
    for (u32 i = 0; i < cfg.layers.size(); ++i) {
        const hybrid_layer_spec& spec = cfg.layers[i];
        const hybrid_mixer& m = spec.mixer;
        const string p = "l" + to_string(i) + ".", mix = p + "mix.", mlp = p + "mlp.";
        hybrid_layer l;
        auto taps = [&](const string& name, u32 channels, u32 n) { return stack({{name, channels}}, n, weight_form::columns_f32); };
        // "norm1" is the norm in front where there are two, and the one on the output where that is all
        auto sublayer = [&](const string& n, llava_buffer** pre, llava_buffer** post, llava_buffer** conv) {
            if (cfg.pre_norm) *pre = values(p + "norm" + n, cfg.width);
            *post = values(p + "norm" + n + (cfg.pre_norm ? "b" : ""), cfg.width);
            if (cfg.taps) *conv = taps(p + "canon" + n, cfg.width, cfg.taps);
        };
        sublayer("1", &l.pre1, &l.post1, &l.canon1);
        l.out = matrix(mix + "o", cfg.width, m.out_size());
        switch (m.type) {
            case hybrid_mixer::kind::attention:
                l.in = stack({{mix + "q", m.heads * m.dim}, {mix + "k", m.kv_heads * m.dim}, {mix + "v", m.kv_heads * m.vdim}}, cfg.width, weight_form::rows_bf16);
                l.q_norm = values(mix + "q.norm", m.dim);
                l.k_norm = values(mix + "k.norm", m.dim);
                l.r1 = values(mix + "r1", m.heads);
                l.r2 = values(mix + "r2", m.heads);
                break;
            case hybrid_mixer::kind::mingru:
                l.in = stack({{mix + "z", m.width}, {mix + "x", m.width}, {mix + "g", m.width}}, cfg.width, weight_form::rows_bf16);
                l.z_bias = values(mix + "z.b", m.width);
                l.x_bias = values(mix + "x.b", m.width);
                break;
            case hybrid_mixer::kind::latent: {
                vector<pair<string, u32>> in = {{mix + "q", m.heads * (m.dim + m.rot)}};
                if (m.has_own_cache()) {
                    in.emplace_back(mix + "dkv", m.kv_rank + m.rot);
                    l.kv_norm = values(mix + "dkv.norm", m.kv_rank);
                }
                l.in = stack(in, cfg.width, weight_form::rows_bf16);
                l.kv_up = stack({{mix + "uk", m.heads * m.dim}, {mix + "uv", m.heads * m.vdim}}, m.kv_rank, weight_form::rows_bf16);
                l.sink = values(mix + "sink", m.heads);
                break;
            }
            case hybrid_mixer::kind::ssm:
                l.in = matrix(mix + "in", m.raw_size(), cfg.width);
                l.conv_w = taps(mix + "conv", m.conv_channels(), m.taps);
                l.conv_b = values(mix + "conv.b", m.conv_channels());
                l.dt_bias = values(mix + "dt_bias", m.heads);
                l.A_log = values(mix + "A_log", m.heads);
                l.D = values(mix + "D", m.heads);
                l.norm = values(mix + "norm", m.out_size());
                break;
        }
        if (spec.has_feed_forward()) sublayer("2", &l.pre2, &l.post2, &l.canon2);
        if (spec.dense.ff) {
            l.up = matrix(mlp + "up", spec.dense.ff, cfg.width);
            l.down = matrix(mlp + "down", cfg.width, spec.dense.ff);
        }
        if (spec.mlp.experts) {
            vector<pair<string, u32>> gate, up, down;
            for (u32 e = 0; e < spec.mlp.experts; ++e) {
                const string x = mlp + "e" + to_string(e) + ".";
                gate.emplace_back(x + "gate", spec.mlp.ff);
                up.emplace_back(x + "up", spec.mlp.ff);
                down.emplace_back(x + "down", cfg.width);
            }
            l.gate = stack(gate, cfg.width, weight_form::rows_bf16);
            l.up = stack(up, cfg.width, weight_form::rows_bf16);
            l.down = stack(down, spec.mlp.ff, weight_form::rows_bf16);
            l.table = stack({{mlp + "table", cfg.vocab}}, spec.mlp.top, weight_form::ids_u32);
        }
        layers.push_back(l);
    }
    return ok;
}

bool hybrid_architecture::upload(llava_context* ctx) {
    for (llava_buffer* b : tensors)
        if (ctx->pop_signal() || !b->load_to_gpu()) {
            cerr << "[!] cannot upload " << b->backing_buffer_name << ": " << lv_last_error_string() << endl;
            return false;
        }
    if (rot_freqs == nullptr) return true;
    vector<double> freqs;
    vector<float> mults;
    for (const hybrid_rotation& r : cfg.rotations) {
        freqs.insert(freqs.end(), r.freqs.begin(), r.freqs.end());
        mults.insert(mults.end(), r.freqs.size(), r.mult);
    }
    return rot_freqs->write_raw(0, freqs.data(), freqs.size() * sizeof(double)) && rot_mults->write_raw(0, mults.data(), mults.size() * sizeof(float));
}

unique_ptr<session_state> hybrid_architecture::make_session_state(llava_session* session) { return make_unique<hybrid_session_state>(session, this); }

// ---- one step --------------------------------------------------------------------------------

// Records the operations of a step.  The output of a sublayer is added to the residual stream by the launch that begins the
// next one (lv_norm_conv), which therefore carries the finished sublayer's norm along.
struct hybrid_recorder {
    const hybrid_architecture& arch;
    const hybrid_config& cfg;
    llava_command_buffer* cb;
    llava_session* s;
    hybrid_session_state* st;
    lv_ctx* lv;
    u32 T;
    bool batched;                        // tensor-core products on bfloat16 activations
    const u32* pos;
    const u32* log;
    // residual stream; null until the embedding rows have been read
    float* x = nullptr;
    // the sublayer that the next norm_conv finishes
    const float* y = nullptr;
    const u32* y_index = nullptr;
    u32 y_rows = 1;
    const llava_buffer* post = nullptr;
    int finished_run = -1;               // the layer run that ends with it, for traces

    static float* f32(const llava_buffer* b) { return b ? static_cast<float*>(b->device_ptr()) : nullptr; }
    static u32 pad8(u32 n) { return (n + 7) / 8 * 8; }
    int act_type() const { return batched ? LV_TYPE_BF16 : LV_TYPE_F32; }

    // rows: destination rows of every token (experts), null for one row per token
    void norm_conv(const llava_buffer* pre, const llava_buffer* conv, llava_buffer* history, const float* step, const llava_buffer* rows = nullptr,
                   u32 copies = 1, bool last_only = false) {
        lv_norm_conv_args a{};
        a.x = x;
        a.embed = arch.embed->device_ptr();
        a.embed_ld = arch.embed->leading();
        a.vocab = cfg.vocab;
        a.token_log = log;
        a.pos = pos;
        a.y = y;
        a.y_index = y_index;
        a.y_rows = y_rows;
        a.mult = cfg.residual_mult;
        a.eps = cfg.eps;
        a.post_w = f32(post);
        a.step = step;
        if (finished_run >= 0 && !st->trace.empty()) a.trace = f32(st->trace[finished_run]);
        a.x_out = f32(st->stream);
        a.row_factor = f32(st->row_factor);
        a.pre_w = f32(pre);
        if (conv) {
            a.conv_w = f32(conv);
            a.taps = cfg.taps;
            a.history = f32(history);
        }
        a.out = f32(st->normed);
        a.out_type = last_only ? LV_TYPE_F32 : act_type();
        a.out_ld = pad8(cfg.width);
        a.out_index = rows ? static_cast<const u32*>(rows->device_ptr()) : nullptr;
        a.out_copies = copies;
        a.plain_w = cfg.plain_norm;
        a.embed_scale = cfg.embed_scale;
        if (arch.pair_embed) {
            a.pair_embed = arch.pair_embed->device_ptr();
            a.pair_ld = arch.pair_embed->leading();
            a.pair_buckets = cfg.pair_buckets;
            a.pair_mul_prev = cfg.pair_mul_prev;
            a.pair_mul_cur = cfg.pair_mul_cur;
        }
        a.width = cfg.width;
        a.first = last_only ? T - 1 : 0;
        a.batch = T;
        cb->note(lv_norm_conv(lv, &a));
        x = a.x_out;
        y = nullptr;
        y_index = nullptr;
        y_rows = 1;
        post = nullptr;
        finished_run = -1;
    }

    void product(llava_buffer* out, const llava_buffer* w, llava_buffer* in, u32 in_ld, float factor = 1.0f) {
        const u32 rows = w->shape.first;
        if (batched) cb->note(lv_gemm_bf16(lv, f32(out), LV_TYPE_F32, rows, w->device_ptr(), rows, w->leading(), w->shape.second, f32(in), in_ld, T, factor, LV_ACT_NONE));
        else cb->note(lv_gemv_bf16(lv, f32(out), rows, w->device_ptr(), rows, w->leading(), w->shape.second, f32(in), in_ld, T, factor, LV_ACT_NONE));
    }

    void dense(const hybrid_layer& l, const hybrid_dense& d) {
        const u32 ld = pad8(cfg.width), act_ld = pad8(d.ff);
        if (batched) cb->note(lv_gemm_bf16(lv, f32(st->act), LV_TYPE_BF16, act_ld, l.up->device_ptr(), d.ff, l.up->leading(), cfg.width, f32(st->normed), ld, T, 1.0f, d.act));
        else cb->note(lv_gemv_bf16(lv, f32(st->act), act_ld, l.up->device_ptr(), d.ff, l.up->leading(), cfg.width, f32(st->normed), ld, T, 1.0f, d.act));
        product(st->sub, l.down, st->act, act_ld);
    }

    void latent(const hybrid_layer& l, const hybrid_mixer& m, const hybrid_run& run) {
        product(st->raw, l.in, st->normed, pad8(cfg.width));
        lv_latent_args a = st->latent_args(m);
        a.q = f32(st->raw);
        a.q_ld = m.raw_size();
        if (m.has_own_cache()) {
            a.dkv = a.q + m.heads * (m.dim + m.rot);
            a.dkv_ld = a.q_ld;
            a.kv_norm = f32(l.kv_norm);
        }
        a.angles = f32(st->angles) + 2 * cfg.rotations[m.rotation].first;
        a.angle_ld = 2 * cfg.rotation_pairs();
        a.w = l.kv_up->device_ptr();
        a.w_ld = l.kv_up->leading();
        a.sink = f32(l.sink);
        a.cache = st->runs[run.cache_run].latent_cache->device_ptr();
        a.pos = pos;
        a.out = f32(st->mixed);
        a.out_type = act_type();
        a.out_ld = pad8(m.out_size());
        cb->note(lv_latent_attention(lv, &a, st->mix_scratch->device_ptr(), st->mix_scratch->byte_size(), T, cb->backlog_size));
        product(st->sub, l.out, st->mixed, a.out_ld);
    }

    void ssm(const hybrid_layer& l, const hybrid_mixer& m, const hybrid_run_state& r) {
        product(st->raw, l.in, st->normed, pad8(cfg.width));
        lv_ssm_args a = st->ssm_args(m);
        a.raw = f32(st->raw);
        a.raw_ld = m.raw_size();
        a.conv_w = f32(l.conv_w);
        a.conv_b = f32(l.conv_b);
        a.dt_bias = f32(l.dt_bias);
        a.A_log = f32(l.A_log);
        a.D = f32(l.D);
        a.norm_w = f32(l.norm);
        a.history = f32(r.conv_history);
        a.S = f32(r.ssm_state);
        a.pos = pos;
        a.out = f32(st->mixed);
        a.out_type = act_type();
        a.out_ld = pad8(m.out_size());
        cb->note(lv_ssm(lv, &a, st->mix_scratch->device_ptr(), st->mix_scratch->byte_size(), T));
        product(st->sub, l.out, st->mixed, a.out_ld);
    }

    void attention(const hybrid_layer& l, const hybrid_mixer& m, const hybrid_run_state& r) {
        product(st->raw, l.in, st->normed, pad8(cfg.width));
        lv_gqa_args a{};
        a.qkv = f32(st->raw);
        a.qkv_ld = m.raw_size();
        a.heads = m.heads;
        a.kv_heads = m.kv_heads;
        a.dim = m.dim;
        a.vdim = m.vdim;
        a.scale = m.scale;
        a.eps = cfg.eps;
        a.q_norm = f32(l.q_norm);
        a.k_norm = f32(l.k_norm);
        a.r1 = f32(l.r1);
        a.r2 = f32(l.r2);
        a.sink = m.sink;
        a.k_cache = r.k_cache->device_ptr();
        a.v_cache = r.v_cache->device_ptr();
        a.cache_type = st->f32 ? LV_TYPE_F32 : LV_TYPE_BF16;
        a.ctx_rows = s->max_context;
        a.pos = pos;
        a.out = f32(st->mixed);
        a.out_type = act_type();
        a.out_ld = pad8(m.out_size());
        if (T > 1) cb->note(lv_qk_norm_append(lv, &a, T));
        cb->note(lv_attention_gqa(lv, &a, st->attn_scratch->device_ptr(), st->attn_scratch->byte_size(), T, cb->backlog_size, T == 1));
        product(st->sub, l.out, st->mixed, a.out_ld);
    }

    void mingru(const hybrid_layer& l, const hybrid_mixer& m, const hybrid_run_state& r) {
        if (T == 1) {
            const u16* w = static_cast<const u16*>(l.in->device_ptr());
            const size_t each = size_t(m.width) * l.in->leading();
            cb->note(lv_gemv_bf16_mingru(lv, f32(st->mixed), w, w + each, w + 2 * each, l.in->leading(), m.width, cfg.width, f32(l.z_bias), f32(l.x_bias),
                                         f32(st->normed), f32(r.gru_state), pos));
        } else {
            product(st->raw, l.in, st->normed, pad8(cfg.width));
            cb->note(lv_mingru_scan(lv, f32(st->mixed), act_type(), pad8(m.width), f32(st->raw), m.raw_size(), m.width, f32(l.z_bias), f32(l.x_bias),
                                    f32(r.gru_state), pos, T));
        }
        product(st->sub, l.out, st->mixed, pad8(m.width));
    }

    void experts(u32 layer, const hybrid_layer& l, const hybrid_experts& e) {
        const u32 ld = pad8(cfg.width), act_ld = pad8(e.ff);
        lv_expert_args gate_up{}, down{};
        gate_up.w0 = l.gate->device_ptr();
        gate_up.w1 = l.up->device_ptr();
        gate_up.ld = l.gate->leading();
        gate_up.rows = e.ff;
        gate_up.cols = cfg.width;
        gate_up.experts = e.experts;
        gate_up.top = e.top;
        gate_up.vocab = cfg.vocab;
        gate_up.table = static_cast<const u32*>(l.table->device_ptr());
        gate_up.token_log = log;
        gate_up.pos = pos;
        down = gate_up;
        down.w0 = l.down->device_ptr();
        down.w1 = nullptr;
        down.ld = l.down->leading();
        down.rows = cfg.width;
        down.cols = e.ff;
        if (batched) {
            const auto* tiles = static_cast<const lv_expert_tile*>(st->route_tiles[layer]->device_ptr());
            cb->note(lv_gemm_bf16_expert_gate_up(lv, f32(st->act), act_ld, &gate_up, tiles, f32(st->normed), ld, T));
            cb->note(lv_gemm_bf16_expert_down(lv, f32(st->sub), cfg.width, &down, tiles, f32(st->act), act_ld, T));
            y_index = static_cast<const u32*>(st->route_index[layer]->device_ptr());      // the next norm_conv averages the choices
            y_rows = e.top;
        } else {
            cb->note(lv_gemv_bf16_expert_gate_up(lv, f32(st->act), act_ld, &gate_up, f32(st->normed), ld, T));
            cb->note(lv_gemv_bf16_expert_down(lv, f32(st->sub), cfg.width, &down, f32(st->act), act_ld, T));
        }
    }

    void finish_sublayer(const llava_buffer* norm) {
        y = f32(st->sub);
        post = norm;
    }

    void step() {
        const auto& runs = arch.runs_in_order();
        if (batched && st->n_route_jobs)
            cb->note(lv_expert_route(lv, static_cast<const lv_route_job*>(st->route_jobs->device_ptr()), st->n_route_jobs, st->max_experts, log, pos, cfg.vocab, T));
        if (st->angles)
            cb->note(lv_rotary_table(lv, f32(st->angles), static_cast<const double*>(arch.rot_freqs->device_ptr()), f32(arch.rot_mults), cfg.rotation_pairs(), pos, T));
        for (size_t i = 0; i < runs.size(); ++i) {
            const u32 layer = runs[i].layer;
            const hybrid_layer& l = arch.layer(layer);
            const hybrid_layer_spec& spec = cfg.layers[layer];
            const hybrid_run_state& r = st->runs[i];
            norm_conv(l.pre1, l.canon1, r.history1, runs[i].begins_pass >= 0 ? f32(arch.loop_step) + size_t(runs[i].begins_pass) * cfg.width : nullptr);
            switch (spec.mixer.type) {
                case hybrid_mixer::kind::attention: attention(l, spec.mixer, r); break;
                case hybrid_mixer::kind::mingru: mingru(l, spec.mixer, r); break;
                case hybrid_mixer::kind::latent: latent(l, spec.mixer, runs[i]); break;
                case hybrid_mixer::kind::ssm: ssm(l, spec.mixer, r); break;
            }
            finish_sublayer(l.post1);
            if (spec.dense.ff) {
                norm_conv(l.pre2, l.canon2, r.history2, nullptr);
                dense(l, spec.dense);
                finish_sublayer(l.post2);
            } else if (spec.mlp.experts) {
                norm_conv(l.pre2, l.canon2, r.history2, nullptr, batched ? st->route_index[layer] : nullptr, spec.mlp.top);
                experts(layer, l, spec.mlp);
                finish_sublayer(l.post2);
            }
            finished_run = int(i);
        }
        if (cb->row_logits) {
            norm_conv(arch.final_norm, nullptr, nullptr, nullptr);
            product(st->logits_rows, arch.head, st->normed, pad8(cfg.width), cfg.logit_scale);
        } else if (cb->with_head) {
            // only the last row's logits are wanted; a trace wants the last layer's stream of every row as well
            if (!st->trace.empty() && T > 1) norm_conv(arch.final_norm, nullptr, nullptr, nullptr);      // (finishes the last sublayer for all rows)
            norm_conv(arch.final_norm, nullptr, nullptr, nullptr, nullptr, 1, true);
            cb->note(lv_gemv_bf16(lv, f32(s->output_probs), cfg.vocab, arch.head->device_ptr(), cfg.vocab, arch.head->leading(), cfg.width,
                                  f32(st->normed), pad8(cfg.width), 1, cfg.logit_scale, LV_ACT_NONE));
        }
        cb->finish_step();
    }
};

void hybrid_architecture::record(llava_command_buffer* cb) {
    llava_session* s = cb->session;
    auto* st = static_cast<hybrid_session_state*>(s->state.get());
    if (!cb->expect(st != nullptr && cb->batch_size <= s->max_batch, "session state")) return;
    hybrid_recorder r{*this, cfg, cb, s, st, s->ctx->lv(), cb->batch_size, st->batched(cb->batch_size), static_cast<const u32*>(s->config_buffer->device_ptr()),
                      static_cast<const u32*>(s->token_log->device_ptr())};
    r.step();
}
