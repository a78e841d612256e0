// Pieces shared by the two forms of the state-space recurrence.
#pragma once

#include "../../include/lv_b200.h"
#include "common.cuh"

namespace lv {

constexpr uint32_t kSsMaxTaps = 16, kSsMaxState = 256;
constexpr float kSsMinLog = -200.f;          // a decay below e^-200 is zero in f32

struct SsmParams {
    lv_ssm_args a;
    uint32_t batch, inner, channels, state_p;    // state_p: state rounded up to a power of two, at least 16
    // what the convolution leaves: x, B and C (state_p per group), f32 or bfloat16; in f32 dt and log a per head
    uint32_t b_at, c_at, conv_ld;
    void* conv;                                  // [batch][conv_ld]
    float* rates;                                // [batch][heads][2]
    float* gated;                                // [batch][inner]
};

// state_space_tc.cu: several tokens on the tensor cores, from a bfloat16 `conv`
bool ssm_tc_supported(const lv_ssm_args& a);
int ssm_tc_launch(lv_ctx* ctx, const SsmParams& p);

}  // namespace lv
