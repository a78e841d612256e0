#include "model_architecture.h"

#include "hybrid_architecture.h"
#include "llama_architecture.h"

using namespace std;

namespace {
struct entry {
    const char* key;
    unique_ptr<model_architecture> (*make)();
};
const entry kRegistry[] = {
    {"ggjt", []() -> unique_ptr<model_architecture> { return make_unique<llama_architecture>(); }},
    {"Sonuzen", []() -> unique_ptr<model_architecture> { return make_unique<hybrid_architecture>("Sonuzen", parse_sonuzen_config); }},
    {"Nuforax", []() -> unique_ptr<model_architecture> { return make_unique<hybrid_architecture>("Nuforax", parse_nuforax_config); }},
};
}  // namespace

unique_ptr<model_architecture> make_architecture(const string& key) {
    for (const entry& e : kRegistry)
        if (key == e.key) return e.make();
    return nullptr;
}

vector<string> known_architectures() {
    vector<string> out;
    for (const entry& e : kRegistry) out.push_back(e.key);
    return out;
}
