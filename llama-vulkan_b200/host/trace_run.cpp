// Replays given token ids through a model, step by step, and writes logits: a session per request, evaluated by
// llava_session::evaluate_pending, i.e. by the recorded steps that generation uses.
//
//   trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps
//
// A step is one line {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [0]}], "end": ["a"]}: the next tokens of
// each request, the places among them whose logits are wanted, and the requests that end after the step.  The wanted
// logits go to DIR/<step>.f32 (little-endian f32, [wanted][vocab], in the order of entries and wants), and "done <step>" is
// printed when a step is finished.  Exit code 3: the model does not run in the requested arithmetic.
#include <cstring>
#include <fstream>
#include <iostream>
#include <map>
#include <memory>
#include <string>

#include "json.h"
#include "llava_context.h"
#include "llava_session.h"

using namespace std;

namespace {
int fail(const string& what) {
    cerr << "[!] trace_run: " << what << endl;
    return 1;
}
}  // namespace

int main(int argc, char** argv) {
    string model, out;
    u32 max_tokens = 0;
    int device = 0;
    compute_type compute = compute_type::bf16;
    for (int i = 1; i + 1 < argc; i += 2) {
        const string key = argv[i], value = argv[i + 1];
        if (key == "--model") model = value;
        else if (key == "--out") out = value;
        else if (key == "--max-tokens") max_tokens = u32(strtoul(value.c_str(), nullptr, 10));
        else if (key == "--device") device = atoi(value.c_str());
        else if (key == "--dtype" && (value == "bfloat16" || value == "float32")) compute = value == "float32" ? compute_type::f32 : compute_type::bf16;
        else return fail("unexpected " + key + " " + value);
    }
    if (model.empty() || out.empty() || argc % 2 == 0) return fail("--model DIR --dtype bfloat16|float32 --out DIR --max-tokens N");

    llava_context context;
    context.set_compute_type(compute);
    if (!context.open(model, device)) return fail("cannot open " + model);
    if (!context.architecture()->runs(compute)) return 3;
    map<string, unique_ptr<llava_session>> sessions;
    string line;
    while (getline(cin, line)) {
        if (line.find_first_not_of(" \t\r") == string::npos) continue;
        json_value step;
        string why;
        u64 number = 0;
        if (!json_value::parse(line, &step, &why)) return fail("bad step: " + why);
        const json_value *n = step.find("step"), *entries = step.find("entries"), *end = step.find("end");
        if (!n || !n->as_u64(&number) || !entries || !entries->is_array()) return fail("a step needs 'step' and 'entries'");
        vector<float> rows;
        for (const json_value& e : entries->items()) {
            const json_value *id = e.find("id"), *tokens = e.find("tokens"), *want = e.find("want");
            if (!id || !id->is_text() || !tokens || !tokens->is_array()) return fail("an entry needs 'id' and 'tokens'");
            auto& session = sessions[id->text()];
            if (!session) {
                session = make_unique<llava_session>(&context, max_tokens);
                session->set_deterministic(true);
                if (!session->is_valid()) return fail("cannot create a session of " + to_string(max_tokens) + " tokens");
            }
            const u32 first = session->get_token_count();
            for (const json_value& t : tokens->items()) {
                u32 v = 0;
                if (!t.as_u32(&v) || !session->push_token(v)) return fail("token out of range or session full");
            }
            vector<u32> wanted;
            if (want)
                for (const json_value& w : want->items()) {
                    u32 v = 0;
                    if (!w.as_u32(&v) || v >= tokens->items().size()) return fail("wanted place out of range");
                    wanted.push_back(first + v);
                }
            vector<float> logits;
            if (!session->evaluate_pending(wanted, &logits)) return fail(string("evaluation failed: ") + lv_last_error_string());
            rows.insert(rows.end(), logits.begin(), logits.end());
        }
        if (!rows.empty()) {
            ofstream f(out + "/" + to_string(number) + ".f32", ios::binary);
            f.write(reinterpret_cast<const char*>(rows.data()), streamsize(rows.size() * sizeof(float)));
            f.close();
            if (!f) return fail("cannot write to " + out);
        }
        if (end)
            for (const json_value& id : end->items()) sessions.erase(id.text());
        cout << "done " << number << endl;
    }
    sessions.clear();
    return 0;
}
