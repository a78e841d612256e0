// A model on disk: header, vocabulary and tensor table over a memory mapping.  Two kinds exist: ggjt files (ggml_file) and
// folders with config.json and model.safetensors (model_folder); open_model() picks by looking at the path.
#ifndef LLAVA_B200_MODEL_FILE_H
#define LLAVA_B200_MODEL_FILE_H

#include <map>
#include <memory>
#include <string>
#include <vector>

#include "types.h"

struct ggml_header {               // ggml_file.h:12-22; model folders fill vocab_size, dim and n_layers
    u32 magic;
    u32 file_version;
    u32 vocab_size;
    u32 dim;
    u32 multiple_of;
    u32 n_heads;
    u32 n_layers;
    u32 rot;
    u32 ftype;
} __attribute__((__packed__));

struct ggml_token {
    std::string text;
    float score;
};

class ggml_data_descriptor {       // ggml_file.h:29-41
public:
    ggml_data_descriptor(std::string name, ggml_value_type ftype, u32 model_version, size_t offset, u32 shape1, u32 shape2);
    std::string name;
    ggml_value_type ftype;
    u32 model_version;
    size_t offset;     // of the data in the file
    u32 shape1;        // rows (length for 1-D tensors)
    u32 shape2;        // columns (1 for 1-D tensors)
    size_t size;       // bytes in the file; 0 for an unsupported type
    static size_t size_in_file(ggml_value_type ftype, u32 model_version, u64 elements);
};

class model_file {
public:
    virtual ~model_file();
    model_file(const model_file&) = delete;
    model_file& operator=(const model_file&) = delete;

    // key of the architecture registry (model_architecture.h)
    virtual std::string architecture() const = 0;
    virtual void print_info() const = 0;
    virtual void tokenize(std::vector<uint32_t>& output, const std::string& text, bool bos) const = 0;
    std::string tokens_to_text(u32 const* tokens, u32 count) const;
    // looks up `s`, then `s + ".weight"`; nullptr when absent
    const ggml_data_descriptor* find_buffer_descriptor(const std::string& s) const;
    // as the reference's accessor: the tensor must exist (aborts otherwise)
    const ggml_data_descriptor& get_buffer_descriptor(const std::string& s) const;
    const std::vector<ggml_token>& get_tokens() const { return tokens; }
    const std::vector<ggml_data_descriptor>& get_tables() const { return tables; }
    // id that ends a generation; ~0U when the model has none
    virtual u32 eos_token() const { return ~0U; }

    bool is_open() const { return mapping != nullptr; }
    const std::string& error() const { return error_text; }
    const ggml_header& get_header() const { return header; }
    u32 get_ff_size() const { return ff_size; }
    const u8* data() const { return mapping; }
    size_t data_size() const { return mapping_size; }

protected:
    model_file() = default;
    bool map_file(const char* path);     // sets error_text on failure
    void close_mapping();
    u8* mapping = nullptr;
    size_t mapping_size = 0;
    ggml_header header{};
    u32 ff_size = 0;
    std::vector<ggml_token> tokens;
    std::vector<ggml_data_descriptor> tables;
    std::map<std::string, u32> name_to_index;
    std::string error_text;
};

// a folder -> model_folder, anything else -> ggml_file; check is_open()
std::unique_ptr<model_file> open_model(const std::string& path);

#endif
