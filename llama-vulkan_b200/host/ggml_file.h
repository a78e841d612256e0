// ggjt model file: memory-mapped header, vocabulary and tensor table, plus the
// SentencePiece-style tokenizer.  Same public surface as the reference's
// ggml_file (ggml_file.h:51-57); malformed files make is_open() false instead
// of tripping asserts.
#ifndef LLAVA_B200_GGML_FILE_H
#define LLAVA_B200_GGML_FILE_H

#include <string>
#include <unordered_map>
#include <vector>

#include "model_file.h"
#include "types.h"

class ggml_file : public model_file {
public:
    explicit ggml_file(const char* filepath);

    std::string architecture() const override { return "ggjt"; }
    void print_info() const override;
    void tokenize(std::vector<uint32_t>& output, const std::string& text, bool bos) const override;
    u32 eos_token() const override { return 2; }

private:
    bool parse();
    // token text -> lowest id with that text (what the reference's linear scan returns)
    std::unordered_map<std::string, u32> text_to_id;
};

#endif
