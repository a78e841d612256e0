#include "model_folder.h"

#include <cstring>
#include <fstream>
#include <iostream>
#include <sstream>

using namespace std;

model_folder::model_folder(const string& path) {
    if (!read_config(path + "/config.json") || !map_file((path + "/model.safetensors").c_str())) {
        cerr << error_text << endl;
        return;
    }
    if (!read_tensor_table()) {
        cerr << "Bad model folder " << path << ": " << error_text << endl;
        close_mapping();
    }
}

bool model_folder::read_config(const string& path) {
    ifstream in(path, ios::binary);
    stringstream text;
    text << in.rdbuf();
    if (!in) {
        error_text = "Cannot read " + path;
        return false;
    }
    string why;
    if (!json_value::parse(text.str(), &config, &why)) {
        error_text = path + ": " + why;
        return false;
    }
    const json_value* name = config.find("architecture");
    const json_value* vocab = config.find("vocab");
    const json_value* width = config.find("width");
    const json_value* layers = config.find("layers");
    u32 vocab_size = 0, dim = 0;
    if (!name || !name->is_text() || !vocab || !vocab->as_u32(&vocab_size) || vocab_size == 0 || !width || !width->as_u32(&dim) || dim == 0 ||
        !layers || !layers->is_array()) {
        error_text = path + ": architecture, vocab, width or layers missing";
        return false;
    }
    architecture_name = name->text();
    header.vocab_size = vocab_size;
    header.dim = dim;
    header.n_layers = u32(layers->items().size());
    tokens.reserve(header.vocab_size);
    for (u32 i = 0; i < header.vocab_size; ++i) tokens.push_back({"<" + to_string(i) + ">", 0.0f});
    return true;
}

bool model_folder::read_tensor_table() {
    u64 head = 0;
    if (mapping_size < 8) { error_text = "file shorter than its header"; return false; }
    memcpy(&head, mapping, 8);
    if (head > mapping_size - 8) { error_text = "file shorter than its header"; return false; }
    json_value table;
    if (!json_value::parse(reinterpret_cast<const char*>(mapping) + 8, size_t(head), &table, &error_text)) return false;
    const size_t data_at = 8 + size_t(head), data_bytes = mapping_size - data_at;
    for (const auto& [name, t] : table.members()) {
        if (name == "__metadata__") continue;
        const json_value *dtype = t.find("dtype"), *shape = t.find("shape"), *offsets = t.find("data_offsets");
        u64 lo = 0, hi = 0;
        if (!dtype || !dtype->is_text() || !shape || !shape->is_array() || !offsets || offsets->items().size() != 2 ||
            !offsets->items()[0].as_u64(&lo) || !offsets->items()[1].as_u64(&hi) || lo > hi || hi > data_bytes) {
            error_text = "bad record of tensor " + name;
            return false;
        }
        u32 dims[2] = {1, 1};
        const auto& s = shape->items();
        bool ok = s.size() <= 2;
        for (size_t i = 0; ok && i < s.size(); ++i) ok = s[i].as_u32(&dims[i]);
        ggml_value_type type{};
        if (dtype->text() == "BF16") type = ggml_value_type::bf16;
        else if (dtype->text() == "F32") type = ggml_value_type::f32;
        else if (dtype->text() == "I32") type = ggml_value_type::i32;
        else ok = false;
        if (!ok) {
            error_text = "tensor " + name + ": unsupported type or shape";
            return false;
        }
        ggml_data_descriptor d(name, type, 0, data_at + size_t(lo), dims[0], dims[1]);
        if (d.size != hi - lo || !name_to_index.emplace(name, u32(tables.size())).second) {
            error_text = "tensor " + name + ": size and shape disagree, or it appears twice";
            return false;
        }
        tables.push_back(std::move(d));
    }
    return true;
}

void model_folder::print_info() const {
    cout << "architecture: " << architecture_name << "\n"
         << "  vocab_size: " << header.vocab_size << "\n"
         << "       width: " << header.dim << "\n"
         << "    n_layers: " << header.n_layers << "\n"
         << "     tensors: " << tables.size() << endl;
}

// "<5><17>" -> {5, 17}; text outside such brackets and ids beyond the vocabulary are skipped, bos does not exist
void model_folder::tokenize(vector<uint32_t>& output, const string& text, bool) const {
    for (size_t at = text.find('<'); at != string::npos; at = text.find('<', at + 1)) {
        u64 id = 0;
        size_t p = at + 1;
        while (p < text.size() && text[p] >= '0' && text[p] <= '9' && id < header.vocab_size) id = id * 10 + u64(text[p++] - '0');
        if (p > at + 1 && p < text.size() && text[p] == '>' && id < header.vocab_size) output.push_back(u32(id));
    }
}
