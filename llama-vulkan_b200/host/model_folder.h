// A model kept as a folder with config.json and model.safetensors (an 8-byte little-endian length, that many bytes of
// JSON {name: {dtype, shape, data_offsets}}, the data).  Tensors are bfloat16, f32 or 32-bit integers of one or two
// dimensions.  Such a folder brings no vocabulary: a token's text is its id in angle brackets ("<17>"), which tokenize()
// reads back.
#ifndef LLAVA_B200_MODEL_FOLDER_H
#define LLAVA_B200_MODEL_FOLDER_H

#include "json.h"
#include "model_file.h"

class model_folder : public model_file {
public:
    explicit model_folder(const std::string& path);
    std::string architecture() const override { return architecture_name; }
    void print_info() const override;
    void tokenize(std::vector<uint32_t>& output, const std::string& text, bool bos) const override;
    const json_value& get_config() const { return config; }

private:
    bool read_config(const std::string& path);
    bool read_tensor_table();
    json_value config;
    std::string architecture_name;
};

#endif
