// What a session of a hybrid decoder keeps on the device: per layer run the key/value or latent caches or the recurrent state and
// the histories of its convolutions, which live as long as the session, and scratch for a step, which follows max_batch.
// No cache or state needs clearing: kernels take a state before position 0 as zero and read cache rows up to the position.
#ifndef LLAVA_B200_HYBRID_SESSION_STATE_H
#define LLAVA_B200_HYBRID_SESSION_STATE_H

#include <vector>

#include "hybrid_architecture.h"

struct hybrid_run_state {
    llava_buffer *k_cache = nullptr, *v_cache = nullptr;      // attention: [kv_heads][max_context][padded dim]
    llava_buffer *latent_cache = nullptr;                     // latent: [max_context][padded kv_rank + padded rot], none when another run's is read
    llava_buffer *gru_state = nullptr;                        // mingru: f32 [width]
    llava_buffer *ssm_state = nullptr, *conv_history = nullptr;      // ssm: f32 [heads][vdim][padded state], [taps][channels]
    llava_buffer *history1 = nullptr, *history2 = nullptr;    // f32 [taps - 1][width]
};

class hybrid_session_state : public session_state {
public:
    hybrid_session_state(llava_session* session, const hybrid_architecture* arch);
    ~hybrid_session_state() override;
    bool resize() override;
    size_t snapshot_bytes(u32 n) const override;
    bool read_snapshot(u8* dst, u32 n) override;
    bool write_snapshot(const u8* src, u32 n) override;
    void dump_frame(int fd) override;
    llava_buffer* row_logits() const override { return logits_rows; }

    llava_session* const session;
    const hybrid_architecture* const arch;
    std::vector<hybrid_run_state> runs;
    // sizes and constants of a mixer; buffers are left to the recorder
    lv_latent_args latent_args(const hybrid_mixer& m) const;
    lv_ssm_args ssm_args(const hybrid_mixer& m) const;
    // scratch of one step
    llava_buffer *stream = nullptr;                           // residual stream, f32 [batch][width]
    llava_buffer *row_factor = nullptr;                       // one word per token between the two launches of lv_norm_conv
    llava_buffer *normed = nullptr;                           // input of a sublayer, one row per token or per chosen expert
    llava_buffer *raw = nullptr;                              // input projections, f32
    llava_buffer *mixed = nullptr;                            // mixer output before its output projection
    llava_buffer *act = nullptr;                              // activations between the products of a feed-forward
    llava_buffer *sub = nullptr;                              // output of a sublayer, f32
    llava_buffer *attn_scratch = nullptr;
    llava_buffer *mix_scratch = nullptr;                      // of latent attention and state spaces
    llava_buffer *angles = nullptr;                           // {cos, sin} of all rotations of the model, f32 [batch][pairs][2]
    llava_buffer *route_jobs = nullptr;                       // lv_route_job per layer with experts, in layer order
    std::vector<llava_buffer*> route_index, route_tiles;      // per layer; null without experts
    u32 n_route_jobs = 0, max_experts = 0;
    llava_buffer *logits_rows = nullptr;                      // f32 [batch][vocab], only for evaluate_pending
    std::vector<llava_buffer*> trace;                         // per layer run: the residual stream after it, only when tracing
    u32 cache_bytes() const { return f32 ? 4 : 2; }
    // several tokens go through the tensor-core products (bfloat16 activations), one token through f32 activations
    bool batched(u32 tokens) const { return !f32 && tokens > 1; }
    bool const f32;                                           // 32-bit arithmetic: activations and caches are f32

private:
    void drop_scratch();
    bool transfer(u8* dst, const u8* src, u32 n);
    llava_device_memory* lasting = nullptr;
    llava_device_memory* scratch = nullptr;
    bool upload_route_jobs();
    u32 scratch_batch = 0;
    bool scratch_trace = false, scratch_rows = false;
};

#endif
