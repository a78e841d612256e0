// Decoders put together from a list of layers, each with a mixer (attention or a gated recurrence) and an optional
// mixture-of-experts feed-forward, read from a model folder.  A design is one parse function from config.json to
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
    enum class kind { attention, mingru };
    kind type = kind::attention;
    // attention: grouped heads, query/key norm, distance bias r1 ln(1 + r2 d), softmax with `sink` added to the denominator
    u32 heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1;
    bool sink = false;
    // mingru
    u32 width = 0;
    u32 raw_size() const { return type == kind::attention ? (heads + kv_heads) * dim + kv_heads * vdim : 3 * width; }
    u32 out_size() const { return type == kind::attention ? heads * vdim : width; }
};

struct hybrid_experts {                  // feed-forward experts chosen by token id; experts == 0: no feed-forward
    u32 ff = 0, experts = 0, top = 0;
};

struct hybrid_layer_spec {
    hybrid_mixer mixer;
    hybrid_experts mlp;
};

struct hybrid_config {
    u32 width = 0, vocab = 0;
    float eps = 0, residual_mult = 1, logit_scale = 1;
    u32 taps = 0;                        // of the convolution in front of every sublayer
    std::vector<hybrid_layer_spec> layers;
    // layers loop_start .. loop_stop - 1 run loop_times times in a row; 0: no loop
    u32 loop_start = 0, loop_stop = 0, loop_times = 0;
};

// false with a message when the configuration is incomplete or inconsistent
bool parse_sonuzen_config(const json_value& config, hybrid_config* out, std::string* error);

// one layer's tensors
struct hybrid_layer {
    llava_buffer *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *canon1 = nullptr, *canon2 = nullptr;
    llava_buffer *in = nullptr;          // stacked input projections: q, k, v or z, x, g
    llava_buffer *out = nullptr;
    llava_buffer *q_norm = nullptr, *k_norm = nullptr, *r1 = nullptr, *r2 = nullptr;      // attention
    llava_buffer *z_bias = nullptr, *x_bias = nullptr;                                    // mingru
    llava_buffer *gate = nullptr, *up = nullptr, *down = nullptr, *table = nullptr;       // experts, stacked
};

// one execution of a layer in a step: looped layers appear once per pass, each with its own cache or state
struct hybrid_run {
    u32 layer = 0;
    int begins_pass = -1;                // number of the pass that this run begins
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
    std::vector<llava_buffer*> tensors;              // everything below, in upload order
    llava_buffer *embed = nullptr, *final_norm = nullptr, *head = nullptr, *loop_step = nullptr;
    friend struct hybrid_recorder;
};

#endif
