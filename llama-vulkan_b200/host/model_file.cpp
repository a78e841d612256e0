#include "model_file.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstdlib>
#include <cstring>
#include <iostream>

#include "ggml_file.h"
#include "model_folder.h"

using namespace std;

ggml_data_descriptor::ggml_data_descriptor(string _name, ggml_value_type _ftype, u32 _model_version, size_t _offset,
                                           u32 _shape1, u32 _shape2)
    : name(std::move(_name)), ftype(_ftype), model_version(_model_version), offset(_offset), shape1(_shape1),
      shape2(_shape2), size(size_in_file(_ftype, _model_version, u64(_shape1) * _shape2)) {}

// Bytes of a tensor in the file (ggml_file.cpp:162-186 of the reference): f32 4 B and
// f16 2 B per element; quantised blocks of 32 elements take 20/36 B (f32 scale) in
// version-1 files and 18/34 B (f16 scale) otherwise.
size_t ggml_data_descriptor::size_in_file(ggml_value_type ftype, u32 model_version, u64 elements) {
    switch (ftype) {
        case ggml_value_type::f32: return elements * 4;
        case ggml_value_type::i32: return elements * 4;
        case ggml_value_type::f16: case ggml_value_type::bf16: return elements * 2;
        case ggml_value_type::q4_0: return elements % 32 ? 0 : elements / 32 * (model_version == 1 ? 20 : 18);
        case ggml_value_type::q8_0: return elements % 32 ? 0 : elements / 32 * (model_version == 1 ? 36 : 34);
        default: return 0;
    }
}

model_file::~model_file() { close_mapping(); }

bool model_file::map_file(const char* path) {
    const int fd = ::open(path, O_RDONLY);
    if (fd < 0) {
        error_text = string("Cannot open ") + path + ": " + strerror(errno);
        return false;
    }
    struct stat st {};
    if (::fstat(fd, &st) < 0 || st.st_size <= 0) {
        error_text = string("Cannot stat ") + path;
        ::close(fd);
        return false;
    }
    mapping_size = static_cast<size_t>(st.st_size);
    void* m = ::mmap(nullptr, mapping_size, PROT_READ, MAP_SHARED, fd, 0);
    ::close(fd);
    if (m == MAP_FAILED) {
        error_text = string("Cannot mmap ") + path + ": " + strerror(errno);
        mapping_size = 0;
        return false;
    }
    mapping = static_cast<u8*>(m);
    return true;
}

void model_file::close_mapping() {
    if (mapping) ::munmap(mapping, mapping_size);
    mapping = nullptr;
    mapping_size = 0;
}

const ggml_data_descriptor* model_file::find_buffer_descriptor(const string& s) const {      // ggml_file.cpp:337-344
    auto it = name_to_index.find(s);
    if (it == name_to_index.end()) it = name_to_index.find(s + ".weight");
    return it == name_to_index.end() ? nullptr : &tables[it->second];
}

const ggml_data_descriptor& model_file::get_buffer_descriptor(const string& s) const {
    const ggml_data_descriptor* d = find_buffer_descriptor(s);
    if (!d) {
        cerr << "[!] tensor " << s << " not found in the model file" << endl;
        abort();
    }
    return *d;
}

string model_file::tokens_to_text(const u32* ids, u32 count) const {                         // ggml_file.cpp:346-357
    string res;
    for (u32 j = 0; j < count; ++j) res += tokens.at(ids[j]).text;
    return res;
}

unique_ptr<model_file> open_model(const string& path) {
    struct stat st {};
    if (::stat(path.c_str(), &st) == 0 && S_ISDIR(st.st_mode)) return make_unique<model_folder>(path);
    return make_unique<ggml_file>(path.c_str());
}
