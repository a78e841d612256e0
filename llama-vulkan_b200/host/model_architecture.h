// What differs between model designs, behind one interface: which tensors a model has, what a session keeps on the device
// for it, and the operations of one evaluation step.  Everything else -- token buffers, positions, recorded steps, greedy
// and sampled decoding, the server, the command line -- is shared.
//
// make_architecture() is the registry: the key is "ggjt" for ggjt files and config.json's "architecture" for model folders.
#ifndef LLAVA_B200_MODEL_ARCHITECTURE_H
#define LLAVA_B200_MODEL_ARCHITECTURE_H

#include <memory>
#include <string>
#include <vector>

#include "types.h"

// Arithmetic of matrix products, activations and caches of models that leave the choice: bfloat16 with 32-bit sums, or 32-bit
// throughout.  (ggjt models have one arithmetic, given by their block formats.)
enum class compute_type : u32 { bf16 = 0, f32 = 1 };

// Device memory that a design keeps per session beyond llava_session's common buffers.
class session_state {
public:
    virtual ~session_state() = default;
    // called when the batch, the tracing option or the row-logits option changed; what earlier tokens left survives
    virtual bool resize() = 0;
    // bytes that describe the session after its first n tokens (n = evaluated tokens), and their transfer
    virtual size_t snapshot_bytes(u32 n) const = 0;
    virtual bool read_snapshot(u8* dst, u32 n) = 0;
    virtual bool write_snapshot(const u8* src, u32 n) = 0;
    virtual void dump_frame(int fd) = 0;              // trace buffers (llava_session::save_frame)
    virtual llava_buffer* row_logits() const { return nullptr; }
};

class model_architecture {
public:
    virtual ~model_architecture() = default;
    virtual const char* name() const = 0;
    // refuses (with a message) a model or rank count that it cannot run; no device yet
    virtual bool check(const model_file& model, u32 n_ranks) = 0;
    // registers the tensors in ctx->weights_memory() / uploads them once that is allocated
    virtual bool build(llava_context* ctx) = 0;
    virtual bool upload(llava_context* ctx) = 0;
    // the session's memory; null for designs that use llava_session's own layer data
    virtual std::unique_ptr<session_state> make_session_state(llava_session*) { return nullptr; }
    virtual bool has_session_state() const { return false; }
    // scratch buffers that follow max_batch, registered before the session's arena is allocated
    virtual bool make_scratch(llava_session*) { return true; }
    // records the operations of one step up to the logits and the position words
    virtual void record(llava_command_buffer* cb) = 0;

    virtual u32 max_context_limit() const = 0;          // tokens of a session
    virtual u32 max_batch_limit() const = 0;            // tokens of a recorded step
    virtual u32 default_batch() const { return 1; }
    // false: the state cannot be taken back to an earlier position, a rewound session evaluates its tokens again
    virtual bool can_rewind() const { return true; }
    virtual bool can_group() const { return false; }    // llava_session_group
    virtual bool has_row_logits() const { return false; }   // a step can produce the logits of all its rows
    virtual bool runs(compute_type) const { return true; }
};

std::unique_ptr<model_architecture> make_architecture(const std::string& key);      // null: unknown
std::vector<std::string> known_architectures();

#endif
