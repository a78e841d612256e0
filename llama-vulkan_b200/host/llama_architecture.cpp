#include "llama_architecture.h"

#include <algorithm>
#include <iostream>

#include "llava_buffer.h"
#include "llava_command_buffer.h"
#include "llava_context.h"
#include "llava_device_memory.h"
#include "llava_layer.h"
#include "llava_layer_session_data.h"
#include "llava_session.h"

using namespace std;

bool llama_architecture::check(const model_file& model, u32 n_ranks) {
    const ggml_header& h = model.get_header();
    const u32 ff = model.get_ff_size();
    if (h.n_heads % n_ranks != 0 || (h.dim / 32) % n_ranks != 0 || (ff / 32) % n_ranks != 0 || ff % (2 * n_ranks) != 0) {
        cerr << "[!] heads, dim and ff must divide evenly over " << n_ranks << " ranks" << endl;
        return false;
    }
    // the kernels are specialised for the reference's geometries (llava_session.cpp:357-375:
    // dim 4096 or 5120, ff 11008 or 13824) and for heads of 128
    if (h.rot != 128 || h.dim % 256 != 0 || ff % 256 != 0) {
        cerr << "[!] unsupported geometry: need head size 128 and dim, ff multiples of 256" << endl;
        return false;
    }
    return true;
}

bool llama_architecture::build(llava_context* ctx) {
    const model_file* model = ctx->get_model();
    const ggml_header& h = model->get_header();
    const ggml_data_descriptor* emb = model->find_buffer_descriptor("tok_embeddings");
    const ggml_data_descriptor* norm = model->find_buffer_descriptor("norm");
    const ggml_data_descriptor* out = model->find_buffer_descriptor("output");
    if (!emb || !norm || !out) {
        cerr << "[!] tok_embeddings / norm / output missing from the model" << endl;
        return false;
    }
    llava_device_memory* memory = ctx->weights_memory();
    ctx->tok_embeddings = new llava_buffer(ctx, *emb, memory);
    ctx->norm_w = new llava_buffer(ctx, *norm, memory);
    ctx->output_w = new llava_buffer(ctx, *out, memory);
    if (ctx->norm_w->type != ggml_value_type::f32 || !ctx->output_w->weight_buffer_is_quantised() || emb->shape1 != h.vocab_size ||
        !(ctx->tok_embeddings->weight_buffer_is_quantised() || ctx->tok_embeddings->type == ggml_value_type::f32)) {
        cerr << "[!] unsupported tensor types for tok_embeddings / norm / output" << endl;
        return false;
    }

    void* table = nullptr;
    if (lv_arena_create(ctx->lv(), size_t(max_backlog_size) * h.rot * sizeof(float), &table) != LV_OK) return false;
    ctx->rope_table = static_cast<float*>(table);
    if (lv_rope_table_build(ctx->lv(), ctx->rope_table, max_backlog_size, h.rot) != LV_OK) return false;

    auto& layers = ctx->get_layers();
    layers.reserve(h.n_layers);
    for (u32 i = 0; i < h.n_layers; ++i) {
        layers.push_back(new llava_layer(ctx, i));
        if (!layers.back()->is_valid()) return false;
    }
    return true;
}

bool llama_architecture::upload(llava_context* ctx) {
    if (!ctx->tok_embeddings->load_to_gpu() || !ctx->norm_w->load_to_gpu() || !ctx->output_w->load_to_gpu()) return false;
    for (llava_layer* l : ctx->get_layers()) {
        if (ctx->pop_signal()) return false;
        if (!l->freeze_storage() || !l->load_to_gpu()) {
            cerr << "[!] cannot upload layer " << l->layer_id << ": " << lv_last_error_string() << endl;
            return false;
        }
    }
    return true;
}

bool llama_architecture::make_scratch(llava_session* s) {
    llava_context* ctx = s->ctx;
    const ggml_header& h = s->model->get_header();
    const u32 dim = h.dim, ff = s->model->get_ff_size(), B = s->max_batch;
    const u32 ranks = ctx->tp_size(), rank = ctx->tp_rank();
    // per-rank sizes: heads (and with them Q, K, V, the attention output) and the FFN width are
    // split; the inputs of the column-sharded wo and w2 are padded like their shards
    const u32 local_dim = dim / ranks;
    const auto Wt = ctx->output_w->type;
    const u32 vout_len = ranks == 1 ? dim : tp_shape(Wt, dim, dim, tp_split::columns, rank, ranks).cols;
    const u32 ff_len = ranks == 1 ? ff : tp_shape(Wt, dim, ff, tp_split::columns, rank, ranks).cols;
    const auto F = ggml_value_type::f32;
    llava_device_memory* m = s->main_buffer_memory;
    s->current_thought = new llava_buffer(ctx, F, dim, B, m);
    s->current_thought_sublayer = new llava_buffer(ctx, F, dim, B, m);
    s->current_thought_middle_normd = new llava_buffer(ctx, F, dim, B, m);
    s->main_ff_result = new llava_buffer(ctx, F, ff_len, B, m);
    s->current_Q = new llava_buffer(ctx, F, local_dim, B, m);
    s->current_K = new llava_buffer(ctx, F, local_dim, B, m);
    s->current_V = new llava_buffer(ctx, F, local_dim, B, m);
    s->current_Vout = new llava_buffer(ctx, F, vout_len, B, m);
    if (ranks > 1) s->tp_partial = new llava_buffer(ctx, F, dim, B, m);
    if (s->is_tracing_enabled()) s->main_attn_result = new llava_buffer(ctx, F, s->backlog_size, h.n_heads * B, m);
    const size_t scratch = lv_attention_scratch_bytes(h.n_heads / ranks, h.rot, max_backlog_size, B);
    if (scratch == 0) return false;
    s->attn_scratch = new llava_buffer(ctx, F, u32((scratch + 3) / 4), 1, m);
    if (B >= llava_command_buffer::kTensorCoreMinBatch)
        s->act_split = new llava_buffer(ctx, F, u32(lv_act_split_bytes(max(max(dim, ff_len), vout_len), B) / 4), 1, m);
    return true;
}

void llama_architecture::record(llava_command_buffer* cb) {
    llava_session* s = cb->session;
    llava_context* c = s->ctx;
    const ggml_header& h = s->model->get_header();
    if (!cb->expect(s->get_layer_data().size() == c->get_layers().size(), "one layer data per layer")) return;
    u32* config = static_cast<u32*>(s->config_buffer->device_ptr());
    u32* log = static_cast<u32*>(s->token_log->device_ptr());
    if (cb->batch_size == 1 && s->step_plan != nullptr && !s->is_tracing_enabled()) {
        // a single token: the whole list below as one persistent kernel
        cb->note(lv_decode_step(c->lv(), s->step_plan, config, log, s->log_capacity(), static_cast<float*>(s->output_probs->device_ptr()),
                                static_cast<u32*>(s->argmax_result->device_ptr()), s->argmax_word(), cb->with_head ? 1 : 0));
        if (cb->sample) cb->record_sampler();
        return;
    }
    // embedding rows of the tokens at positions config.token_count .. + batch (the reference
    // dequantises them on the host, llava_session.cpp:219-223)
    cb->note(lv_dequant_rows(c->lv(), static_cast<float*>(s->current_thought->device_ptr()), c->tok_embeddings->device_ptr(),
                             c->tok_embeddings->kernel_type(), log, config, h.dim, h.vocab_size, cb->batch_size));
    llava_buffer* current = s->current_thought;
    for (u32 i = 0; i < c->get_layers().size(); ++i) current = c->get_layers()[i]->execute(cb, s->get_layer_data()[i], current);
    if (cb->with_head) {
        // final norm + output matrix on the last row only (llava_command_buffer.cpp:38-39; the
        // reference computes every row and reads the last, llava_session.cpp:129-135)
        const float* last = static_cast<const float*>(current->device_ptr()) + size_t(cb->batch_size - 1) * h.dim;
        float* logits = static_cast<float*>(s->output_probs->device_ptr());
        // sharded with fused exchanges: the last layer's w2 pushed its partial rows; the head's
        // normalisation takes residual + the ranks' sum
        if (c->tp_size() > 1 && c->fused_exchange() && !cb->use_tensor_cores(c->get_layers()[0]->wq()))
            cb->tp_arm_pull(2 * u32(c->get_layers().size()) - 1, h.dim, current == s->current_thought ? s->current_thought_sublayer : s->current_thought);
        cb->note(lv_norm_gemv(c->lv(), logits, c->output_w->device_ptr(), c->output_w->kernel_type(), last,
                              static_cast<const float*>(c->norm_w->device_ptr()), h.vocab_size, h.dim, 1));
    }
    cb->finish_step();
}
