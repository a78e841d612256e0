#include "hybrid_session_state.h"

#include <algorithm>
#include <cstring>
#include <string>

#include "llava_buffer.h"
#include "llava_context.h"
#include "llava_device_memory.h"
#include "llava_session.h"

using namespace std;

namespace {
u32 pad8(u32 n) { return (n + 7) / 8 * 8; }
}  // namespace

hybrid_session_state::hybrid_session_state(llava_session* _session, const hybrid_architecture* _arch)
    : session(_session), arch(_arch), f32(_session->ctx->get_compute_type() == compute_type::f32) {
    const hybrid_config& c = arch->config();
    llava_context* ctx = session->ctx;
    const auto F = ggml_value_type::f32, C = f32 ? ggml_value_type::f32 : ggml_value_type::bf16;
    lasting = new llava_device_memory(ctx);
    for (const hybrid_run& r : arch->runs_in_order()) {
        const hybrid_layer_spec& spec = c.layers[r.layer];
        hybrid_run_state s;
        const hybrid_mixer& m = spec.mixer;
        switch (m.type) {
            case hybrid_mixer::kind::attention:
                s.k_cache = new llava_buffer(ctx, C, m.kv_heads * session->max_context, pad8(m.dim), lasting, "k_cache");
                s.v_cache = new llava_buffer(ctx, C, m.kv_heads * session->max_context, pad8(m.vdim), lasting, "v_cache");
                break;
            case hybrid_mixer::kind::mingru:
                s.gru_state = new llava_buffer(ctx, F, m.width, 1, lasting, "gru_state");
                break;
            case hybrid_mixer::kind::latent:
                if (m.has_own_cache()) s.latent_cache = new llava_buffer(ctx, C, session->max_context, pad8(m.kv_rank) + pad8(m.rot), lasting, "latent_cache");
                break;
            case hybrid_mixer::kind::ssm:
                s.ssm_state = new llava_buffer(ctx, F, m.heads * m.vdim, lv_ssm_state_rows(m.state), lasting, "ssm_state");
                s.conv_history = new llava_buffer(ctx, F, m.conv_channels(), m.taps, lasting, "conv_history");
                break;
        }
        if (c.taps > 1) {
            s.history1 = new llava_buffer(ctx, F, c.width, c.taps - 1, lasting, "history1");
            if (spec.has_feed_forward()) s.history2 = new llava_buffer(ctx, F, c.width, c.taps - 1, lasting, "history2");
        }
        runs.push_back(s);
    }
    lasting->freeze();
}

hybrid_session_state::~hybrid_session_state() {
    drop_scratch();
    for (hybrid_run_state& s : runs)
        for (llava_buffer* b : {s.k_cache, s.v_cache, s.latent_cache, s.gru_state, s.ssm_state, s.conv_history, s.history1, s.history2}) delete b;
    delete lasting;
}

void hybrid_session_state::drop_scratch() {
    for (llava_buffer** b : {&stream, &row_factor, &normed, &raw, &mixed, &act, &sub, &attn_scratch, &mix_scratch, &angles, &logits_rows, &route_jobs}) {
        delete *b;
        *b = nullptr;
    }
    for (auto* list : {&trace, &route_index, &route_tiles}) {
        for (llava_buffer* b : *list) delete b;
        list->clear();
    }
    n_route_jobs = max_experts = 0;
    delete scratch;
    scratch = nullptr;
    scratch_batch = 0;
}

lv_latent_args hybrid_session_state::latent_args(const hybrid_mixer& m) const {
    lv_latent_args a{};
    a.heads = m.heads;
    a.dim = m.dim;
    a.rot = m.rot;
    a.vdim = m.vdim;
    a.kv_rank = m.kv_rank;
    a.angle_pairs = m.rot_pairs;
    a.scale = m.scale;
    a.eps = arch->config().eps;
    a.window = m.window;
    a.cache_type = f32 ? LV_TYPE_F32 : LV_TYPE_BF16;
    a.ctx_rows = session->max_context;
    a.form = LV_LATENT_AUTO;
    return a;
}

lv_ssm_args hybrid_session_state::ssm_args(const hybrid_mixer& m) const {
    lv_ssm_args a{};
    a.heads = m.heads;
    a.vdim = m.vdim;
    a.state = m.state;
    a.groups = m.groups;
    a.taps = m.taps;
    a.norm_groups = m.norm_groups;
    a.eps = arch->config().eps;
    return a;
}

bool hybrid_session_state::resize() {
    if (!lasting->is_frozen()) return false;
    const u32 B = session->max_batch;
    const bool want_trace = session->is_tracing_enabled(), want_rows = session->want_row_logits;
    if (scratch_batch == B && scratch_trace == want_trace && scratch_rows == want_rows) return true;
    drop_scratch();
    const hybrid_config& c = arch->config();
    llava_context* ctx = session->ctx;
    u32 raw_size = 8, mixed_size = 8, act_size = 8, copies = 1;
    size_t attention_bytes = 0, mix_bytes = 0;
    for (const hybrid_layer_spec& l : c.layers) {
        raw_size = max(raw_size, l.mixer.raw_size());
        mixed_size = max(mixed_size, pad8(l.mixer.out_size()));
        if (l.mlp.experts) {
            act_size = max(act_size, l.mlp.top * pad8(l.mlp.ff));
            copies = max(copies, l.mlp.top);
        }
        act_size = max(act_size, pad8(l.dense.ff));
        if (l.mixer.type == hybrid_mixer::kind::latent) {
            const lv_latent_args a = latent_args(l.mixer);         // its form follows the batch, every batch must fit
            for (u32 n = 1; n <= B; ++n) mix_bytes = max(mix_bytes, lv_latent_scratch_bytes(ctx->lv(), &a, n, session->max_context));
        }
        if (l.mixer.type == hybrid_mixer::kind::ssm) {
            const lv_ssm_args a = ssm_args(l.mixer);
            mix_bytes = max(mix_bytes, lv_ssm_scratch_bytes(&a, B));
        }
        if (l.mixer.type == hybrid_mixer::kind::attention) {
            lv_gqa_args a{};
            a.heads = l.mixer.heads;
            a.kv_heads = l.mixer.kv_heads;
            a.dim = l.mixer.dim;
            a.vdim = l.mixer.vdim;
            attention_bytes = max(attention_bytes, lv_gqa_scratch_bytes(ctx->lv(), &a, B, session->max_context));
        }
    }
    const auto F = ggml_value_type::f32;
    scratch = new llava_device_memory(ctx);
    stream = new llava_buffer(ctx, F, c.width, B, scratch);
    row_factor = new llava_buffer(ctx, F, 1, B, scratch);
    normed = new llava_buffer(ctx, F, pad8(c.width) * copies, B, scratch);
    raw = new llava_buffer(ctx, F, raw_size, B, scratch);
    mixed = new llava_buffer(ctx, F, mixed_size, B, scratch);
    act = new llava_buffer(ctx, F, act_size, B, scratch);
    sub = new llava_buffer(ctx, F, c.width * copies, B, scratch);
    if (attention_bytes) attn_scratch = new llava_buffer(ctx, F, u32((attention_bytes + 3) / 4), 1, scratch);
    if (mix_bytes) mix_scratch = new llava_buffer(ctx, F, u32((mix_bytes + 3) / 4), 1, scratch);
    if (c.rotation_pairs()) angles = new llava_buffer(ctx, F, 2 * c.rotation_pairs(), B, scratch);
    for (const hybrid_layer_spec& l : c.layers) {
        const hybrid_experts& e = l.mlp;
        if (f32 || e.experts == 0) {
            route_index.push_back(nullptr);
            route_tiles.push_back(nullptr);
            continue;
        }
        u32 tiles = 0;                                         // the tile size follows the batch, every batch must fit
        for (u32 n = 2; n <= max(B, 2u); ++n) tiles = max(tiles, lv_expert_max_tiles(n, e.top, e.experts));
        route_index.push_back(new llava_buffer(ctx, F, e.top, B, scratch));
        route_tiles.push_back(new llava_buffer(ctx, F, u32(sizeof(lv_expert_tile) / 4), tiles, scratch));
        max_experts = max(max_experts, e.experts);
        ++n_route_jobs;
    }
    if (n_route_jobs) route_jobs = new llava_buffer(ctx, F, u32(sizeof(lv_route_job) / 4), n_route_jobs, scratch);
    if (want_rows) logits_rows = new llava_buffer(ctx, F, c.vocab, B, scratch);
    if (want_trace)
        for (size_t r = 0; r < runs.size(); ++r) {            // numbered so that frames list them in order
            const string n = to_string(r);
            trace.push_back(new llava_buffer(ctx, F, c.width, B, scratch, "run." + string(4 - min<size_t>(4, n.size()), '0') + n + ".residual"));
        }
    if (!scratch->freeze() || !scratch->zero(0, scratch->get_size()) || !upload_route_jobs()) return false;
    scratch_batch = B;
    scratch_trace = want_trace;
    scratch_rows = want_rows;
    return true;
}

bool hybrid_session_state::upload_route_jobs() {
    if (n_route_jobs == 0) return true;
    vector<lv_route_job> jobs;
    for (size_t i = 0; i < route_index.size(); ++i) {
        if (route_index[i] == nullptr) continue;
        const hybrid_experts& e = arch->config().layers[i].mlp;
        lv_route_job j{};
        j.table = static_cast<const u32*>(arch->layer(u32(i)).table->device_ptr());
        j.experts = e.experts;
        j.top = e.top;
        j.index = static_cast<u32*>(route_index[i]->device_ptr());
        j.tiles = static_cast<lv_expert_tile*>(route_tiles[i]->device_ptr());
        j.max_tiles = route_tiles[i]->shape.second;
        jobs.push_back(j);
    }
    return route_jobs->write_raw(0, jobs.data(), jobs.size() * sizeof(lv_route_job));
}

void hybrid_session_state::dump_frame(int fd) {
    if (scratch) scratch->dump_buffers(fd, "step");
}

// Per layer run: the first n rows of every key head, then of every value head, or of the latent cache, or the recurrent state; then
// the histories.
size_t hybrid_session_state::snapshot_bytes(u32 n) const {
    size_t total = 0;
    for (const hybrid_run_state& s : runs) {
        for (const llava_buffer* b : {s.k_cache, s.v_cache, s.latent_cache})
            if (b) total += size_t(b->shape.first / session->max_context) * n * b->shape.second * cache_bytes();
        for (const llava_buffer* b : {s.gru_state, s.ssm_state, s.conv_history, s.history1, s.history2})
            if (b) total += b->byte_size();
    }
    return total;
}

bool hybrid_session_state::transfer(u8* dst, const u8* src, u32 n) {
    size_t at = 0;
    bool ok = true;
    auto move = [&](llava_buffer* b, size_t offset, size_t bytes) {
        if (bytes != 0) ok = ok && (dst ? b->read_raw(offset, dst + at, bytes) : b->write_raw(offset, src + at, bytes));
        at += bytes;
    };
    for (hybrid_run_state& s : runs) {
        for (llava_buffer* b : {s.k_cache, s.v_cache, s.latent_cache}) {
            if (b == nullptr) continue;
            const size_t row = size_t(b->shape.second) * cache_bytes();
            for (u32 g = 0; g < b->shape.first / session->max_context; ++g) move(b, size_t(g) * session->max_context * row, n * row);
        }
        for (llava_buffer* b : {s.gru_state, s.ssm_state, s.conv_history, s.history1, s.history2})
            if (b) move(b, 0, b->byte_size());
    }
    return ok;
}

bool hybrid_session_state::read_snapshot(u8* dst, u32 n) { return transfer(dst, nullptr, n); }
bool hybrid_session_state::write_snapshot(const u8* src, u32 n) { return transfer(nullptr, src, n); }
