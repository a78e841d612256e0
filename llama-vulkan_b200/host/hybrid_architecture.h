// Decoders put together from a list of layers, each with a mixer (attention, attention over a latent cache, a gated recurrence or
// a selective state space) and an optional feed-forward (dense or a mixture of experts), read from a model folder.  A design is one parse function from config.json to
// hybrid_config; everything it fixes (norm placement, sink, convolution) is a field here, so that another design can
// combine the same mechanisms differently.
#ifndef LLAVA_B200_HYBRID_ARCHITECTURE_H
#define LLAVA_B200_HYBRID_ARCHITECTURE_H

#include <string>
#include <vector>

#include "../../include/lv_b200.h"
#include "json.h"
#include "model_architecture.h"

struct hybrid_mixer {
    enum class kind { attention, mingru, latent, ssm };
    kind type = kind::attention;
    // attention: grouped heads, query/key norm, distance bias r1 ln(1 + r2 d), softmax with `sink` added to the denominator
    u32 heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1;
    bool sink = false;
    // mingru
    u32 width = 0;
    // latent: heads, dim (unrotated), vdim, scale and sink (a learned logit per head) as above; rot rotated dimensions, the leading
    // 2 * rot_pairs of which turn; rotation: entry of hybrid_config::rotations
    u32 rot = 0, rot_pairs = 0, rotation = 0, kv_rank = 0, window = 0;
    int kv_from = -1;                    // layer whose cache it reads; -1: its own
    // ssm: heads, vdim
    u32 state = 0, groups = 0, taps = 0, norm_groups = 0;
    bool has_own_cache() const { return type == kind::latent && kv_from < 0; }
    u32 conv_channels() const { return heads * vdim + 2 * groups * state; }
    u32 raw_size() const {
        switch (type) {
            case kind::attention: return (heads + kv_heads) * dim + kv_heads * vdim;
            case kind::mingru: return 3 * width;
            case kind::latent: return heads * (dim + rot) + (has_own_cache() ? kv_rank + rot : 0);
            case kind::ssm: return heads * vdim + conv_channels() + heads;
        }
        return 0;
    }
    u32 out_size() const { return type == kind::mingru ? width : heads * vdim; }
};

struct hybrid_experts {                  // feed-forward experts chosen by token id; experts == 0: no feed-forward
    u32 ff = 0, experts = 0, top = 0;
};

struct hybrid_dense {                    // act(x up) down; ff == 0: none
    u32 ff = 0;
    int act = LV_ACT_NONE;
};

struct hybrid_layer_spec {
    hybrid_mixer mixer;
    hybrid_experts mlp;
    hybrid_dense dense;
    bool has_feed_forward() const { return mlp.experts != 0 || dense.ff != 0; }
};

// Rotary positions: angle = position * freqs[i] for pair i, cos and sin times mult
struct hybrid_rotation {
    std::vector<double> freqs;
    float mult = 1;
    u32 first = 0;                       // of its pairs among all pairs of the model
};
// Frequencies base^(-2 i / dims); with scaling, frequencies that turn less than `slow` times within `original` positions are divided by
// `factor`, those that turn more than `fast` times stay, a linear ramp lies between, and cos and sin grow by 0.1 ln(factor) + 1.
struct rotary_scaling { double factor, original, fast, slow; };
hybrid_rotation make_rotation(u32 dims, double base, const rotary_scaling* scaling);

struct hybrid_config {
    u32 width = 0, vocab = 0;
    float eps = 0, residual_mult = 1, logit_scale = 1;
    u32 taps = 0;                        // of the convolution in front of every sublayer
    bool pre_norm = true;                // a norm in front of every sublayer, besides the one on its output
    bool plain_norm = false;             // norms multiply by w instead of 1 + w
    bool tied_head = false;              // logits from the embedding table
    float embed_scale = 1;
    u32 pair_buckets = 0, pair_mul_prev = 0, pair_mul_cur = 0;      // embedding of pairs of tokens; 0 buckets: none
    std::vector<hybrid_rotation> rotations;
    std::vector<hybrid_layer_spec> layers;
    u32 rotation_pairs() const { return rotations.empty() ? 0 : rotations.back().first + u32(rotations.back().freqs.size()); }
    // layers loop_start .. loop_stop - 1 run loop_times times in a row; 0: no loop
    u32 loop_start = 0, loop_stop = 0, loop_times = 0;
};

// false with a message when the configuration is incomplete or inconsistent
bool parse_sonuzen_config(const json_value& config, hybrid_config* out, std::string* error);
bool parse_nuforax_config(const json_value& config, hybrid_config* out, std::string* error);

// one layer's tensors
struct hybrid_layer {
    // norms in front of (pre) and behind (post) the mixer (1) and the feed-forward (2); convolutions in front of them
    llava_buffer *pre1 = nullptr, *post1 = nullptr, *pre2 = nullptr, *post2 = nullptr, *canon1 = nullptr, *canon2 = nullptr;
    llava_buffer *in = nullptr;          // stacked input projections: q, k, v or z, x, g or q, dkv or the one of a state space
    llava_buffer *out = nullptr;
    llava_buffer *q_norm = nullptr, *k_norm = nullptr, *r1 = nullptr, *r2 = nullptr;      // attention
    llava_buffer *z_bias = nullptr, *x_bias = nullptr;                                    // mingru
    llava_buffer *kv_norm = nullptr, *kv_up = nullptr, *sink = nullptr;                   // latent; kv_up: W_uk, then W_uv
    llava_buffer *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *A_log = nullptr, *D = nullptr, *norm = nullptr;      // ssm
    llava_buffer *gate = nullptr, *up = nullptr, *down = nullptr, *table = nullptr;       // feed-forward; experts are stacked
};

// one execution of a layer in a step: looped layers appear once per pass, each with its own cache or state
struct hybrid_run {
    u32 layer = 0;
    int begins_pass = -1;                // number of the pass that this run begins
    u32 cache_run = 0;                   // latent: the run whose cache it reads
};

class hybrid_architecture : public model_architecture {
public:
    using parser = bool (*)(const json_value&, hybrid_config*, std::string*);
    hybrid_architecture(const char* name, parser parse) : name_(name), parse_(parse) {}
    ~hybrid_architecture() override;
    const char* name() const override { return name_; }
    bool check(const model_file& model, u32 n_ranks) override;
    bool build(llava_context* ctx) override;
    bool upload(llava_context* ctx) override;
    std::unique_ptr<session_state> make_session_state(llava_session* session) override;
    bool has_session_state() const override { return true; }
    void record(llava_command_buffer* cb) override;
    u32 max_context_limit() const override { return 1u << 20; }
    u32 max_batch_limit() const override { return 2048; }
    u32 default_batch() const override { return 512; }
    bool can_rewind() const override { return false; }
    bool has_row_logits() const override { return true; }

    const hybrid_config& config() const { return cfg; }
    const std::vector<hybrid_run>& runs_in_order() const { return runs; }
    const hybrid_layer& layer(u32 i) const { return layers[i]; }

private:
    const char* name_;
    parser parse_;
    hybrid_config cfg;
    std::vector<hybrid_layer> layers;
    std::vector<hybrid_run> runs;
    std::vector<llava_buffer*> tensors;              // everything from the model folder, in upload order
    llava_buffer *embed = nullptr, *final_norm = nullptr, *head = nullptr, *loop_step = nullptr, *pair_embed = nullptr;
    llava_buffer *rot_freqs = nullptr, *rot_mults = nullptr;      // f64 and f32, of all rotations in a row
    friend struct hybrid_recorder;
};

#endif
