// The reference's model: LLaMA decoder layers from a ggjt file (llava_layer.h).
#ifndef LLAVA_B200_LLAMA_ARCHITECTURE_H
#define LLAVA_B200_LLAMA_ARCHITECTURE_H

#include "model_architecture.h"

class llama_architecture : public model_architecture {
public:
    const char* name() const override { return "LLaMA (ggjt)"; }
    bool check(const model_file& model, u32 n_ranks) override;
    bool build(llava_context* ctx) override;
    bool upload(llava_context* ctx) override;
    bool make_scratch(llava_session* session) override;
    void record(llava_command_buffer* cb) override;
    u32 max_context_limit() const override { return 2048; }        // llava_session.cpp:24
    u32 max_batch_limit() const override { return 64; }
    bool can_group() const override { return true; }
};

#endif
