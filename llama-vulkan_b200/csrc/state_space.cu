// Selective state spaces (lv_ssm_args): a short causal convolution, a linear recurrence with one decay per head and token, gate and
// grouped norm.
//
//   several tokens   ssm_conv_kernel   convolution, silu, step sizes and logarithms of the decays
//                    ssm_scan_kernel   the recurrence, D x and the gate
//   one token        ssm_step_kernel   all of that
//   both             ssm_norm_kernel   RMS norm of each part
//
// The recurrence S_t = a_t S_(t-1) + dt_t B_t x_t^T is carried in f32 registers: a CTA has some columns of one head's state, a thread two
// columns and up to sixteen of the state's rows.  Tokens come in chunks of 32 through shared memory.  Within a chunk the state is
// kept relative to its decay, S_t = exp(L_t - R) Z_t with L the running sum of log a and R its value at a reference token, so
// that a token costs one multiply-add per element for Z += (dt exp(R - L)) B x^T and one for y = exp(L - R) C Z; a new reference is
// taken whenever L has moved on by 16, which bounds every factor.  L is summed in f64.
#include <cuda_bf16.h>
#include <math.h>

#include "common.cuh"
#include "ctx.h"

namespace lv {

constexpr uint32_t kSsMaxTaps = 16, kSsMaxState = 256;
constexpr int kSsThreads = 128;
constexpr int kSsChunk = 32;                 // tokens
constexpr double kSsReference = 16.0;
constexpr float kSsMinLog = -200.f;          // a decay below e^-200 is zero in f32

struct SsmParams {
    lv_ssm_args a;
    uint32_t batch, inner, channels, state_p;    // state_p: state rounded up to 16
    uint32_t x_at, b_at, c_at, dt_at, log_at, conv_ld;      // columns of `conv`: x, B and C (state_p per group), dt and log a per head
    uint32_t tokens_per_block, columns;          // columns of a head per CTA
    float* conv;                                 // [batch][conv_ld]
    float* gated;                                // [batch][inner]
};

__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ss_log_decay(float A_log, float dt) { return fmaxf(-expf(A_log) * dt, kSsMinLog); }

// two f32 in one register pair
__device__ __forceinline__ uint64_t ss_pack(float lo, float hi) { return uint64_t(__float_as_uint(lo)) | (uint64_t(__float_as_uint(hi)) << 32); }
__device__ __forceinline__ uint64_t ss_fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ float ss_sum2(uint64_t v) { return __uint_as_float(uint32_t(v)) + __uint_as_float(uint32_t(v >> 32)); }

// Columns of `conv`: a thread owns one and slides over its tokens.  Block row 0 alone reads the history, whose successor it writes.
template <int MAXT>
__global__ void __launch_bounds__(kSsThreads) ssm_conv_kernel(const SsmParams p) {
    pdl_launch_dependents();
    const lv_ssm_args& a = p.a;
    const uint32_t col = blockIdx.x * kSsThreads + threadIdx.x, T = p.batch;
    const uint32_t t0 = blockIdx.y * p.tokens_per_block, t1 = min(T, t0 + p.tokens_per_block);
    if (col >= p.conv_ld) return;
    uint32_t channel = ~0u;                      // of the convolution
    if (col < p.inner) channel = col;
    else if (col >= p.b_at && col < p.dt_at) {
        const bool second = col >= p.c_at;
        const uint32_t g = (col - (second ? p.c_at : p.b_at)) / p.state_p, n = (col - (second ? p.c_at : p.b_at)) - g * p.state_p;
        if (g < a.groups && n < a.state) channel = p.inner + (second ? a.groups * a.state : 0) + g * a.state + n;
    }
    float w[MAXT], win[MAXT], bias = 0.f;        // taps right-aligned: index MAXT - 1 is the current token
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
        const int s = j - (MAXT - int(a.taps));
        w[j] = channel != ~0u && s >= 0 ? a.conv_w[size_t(s) * p.channels + channel] : 0.f;
        win[j] = 0.f;
    }
    if (channel != ~0u) bias = a.conv_b[channel];
    pdl_wait();
    float* out = p.conv + col;
    if (channel == ~0u) {
        const bool is_dt = col >= p.dt_at && col < p.dt_at + a.heads, is_log = col >= p.log_at && col < p.log_at + a.heads;
        const uint32_t h = is_dt ? col - p.dt_at : col - p.log_at;
        for (uint32_t t = t0; t < t1; ++t) {
            float v = 0.f;                       // padding
            if (is_dt || is_log) {
                v = softplus_f32(a.raw[size_t(t) * a.raw_ld + p.inner + p.channels + h] + a.dt_bias[h]);
                if (is_log) v = ss_log_decay(a.A_log[h], v);
            }
            out[size_t(t) * p.conv_ld] = v;
        }
        return;
    }
    const uint32_t pos = *a.pos;
    const float* raw = a.raw + p.inner + channel;
    float* history = a.history + channel;
#pragma unroll
    for (int j = 1; j < MAXT; ++j) {             // the window before t0
        const uint32_t back = MAXT - j;
        if (back >= a.taps) continue;
        if (t0 >= back) win[j] = raw[size_t(t0 - back) * a.raw_ld];
        else if (pos + t0 >= back) win[j] = history[size_t((pos + t0 - back) % a.taps) * p.channels];
    }
#pragma unroll 4
    for (uint32_t t = t0; t < t1; ++t) {
#pragma unroll
        for (int j = 0; j + 1 < MAXT; ++j) win[j] = win[j + 1];
        win[MAXT - 1] = raw[size_t(t) * a.raw_ld];
        float v = bias;
#pragma unroll
        for (int j = 0; j < MAXT; ++j) v = fmaf(w[j], win[j], v);
        out[size_t(t) * p.conv_ld] = silu_f32(v);
    }
    if (blockIdx.y != 0) return;
    for (uint32_t t = T > a.taps ? T - a.taps : 0; t < T; ++t) history[size_t((pos + t) % a.taps) * p.channels] = raw[size_t(t) * a.raw_ld];
}

// Sums a thread's two columns over the NL lanes that share them; afterwards lane 0 of the NL holds the first column's sum and lane
// NL / 2 the second's (NL = 1: both stay).
template <int NL>
__device__ __forceinline__ void ss_reduce(float& y0, float& y1) {
    if constexpr (NL > 1) {
        const bool upper = (threadIdx.x & (NL / 2)) != 0;
        const float keep = upper ? y1 : y0, give = upper ? y0 : y1;
        y0 = keep + __shfl_xor_sync(0xffffffffu, give, NL / 2);
#pragma unroll
        for (int o = NL / 4; o > 0; o /= 2) y0 += __shfl_xor_sync(0xffffffffu, y0, o);
    }
}

// State rows of a thread: four at a time, 4 (q NL + slice) .. + 3 for q < 4 (conflict-free in shared memory, contiguous over lanes).
template <int NL>
__global__ void __launch_bounds__(kSsThreads) ssm_scan_kernel(const SsmParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_ssm_args& a = p.a;
    const uint32_t blocks = (a.vdim + p.columns - 1) / p.columns, h = blockIdx.x / blocks, c0 = (blockIdx.x - h * blocks) * p.columns;
    const uint32_t cols = min(p.columns, a.vdim - c0), g = h / (a.heads / a.groups), N = p.state_p;
    const uint32_t slice = threadIdx.x % NL, pc = threadIdx.x / NL * 2;       // columns pc, pc + 1 of the CTA's
    float* s_b = reinterpret_cast<float*>(smem_raw);       // [2][chunk][N]
    float* s_c = s_b + 2 * kSsChunk * N;
    float* s_x = s_c + 2 * kSsChunk * N;                   // [2][chunk][columns]
    float* s_y = s_x + 2 * kSsChunk * p.columns;           // [chunk][columns]
    float* s_raw = s_y + kSsChunk * p.columns;             // [2][chunk][2]: dt, log a
    __shared__ __align__(16) float4 s_f[kSsChunk];         // {dt exp(R - L), exp(L - R), factor of Z, -}
    const bool live0 = pc < cols, live1 = pc + 1 < cols;
    const float Dh = a.D[h];
    pdl_wait();
    const uint32_t T = p.batch;
    auto fetch = [&](uint32_t chunk, uint32_t buffer) {
        const uint32_t t0 = chunk * kSsChunk, n = min(uint32_t(kSsChunk), T - t0);
        const float* src = p.conv + size_t(t0) * p.conv_ld;
        const uint32_t n4 = N / 4, b = smem_u32(s_b + buffer * kSsChunk * N), c = smem_u32(s_c + buffer * kSsChunk * N);
        for (uint32_t i = threadIdx.x; i < n * n4; i += kSsThreads) {
            const uint32_t t = i / n4, q = i - t * n4;
            const float* at = src + size_t(t) * p.conv_ld + g * N + q * 4;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(b + i * 16u), "l"(at + p.b_at) : "memory");
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(c + i * 16u), "l"(at + p.c_at) : "memory");
        }
        const uint32_t x = smem_u32(s_x + buffer * kSsChunk * p.columns);
        for (uint32_t i = threadIdx.x; i < n * cols; i += kSsThreads) {
            const uint32_t t = i / cols, q = i - t * cols;
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(x + (t * p.columns + q) * 4u), "l"(src + size_t(t) * p.conv_ld + h * a.vdim + c0 + q) : "memory");
        }
        const uint32_t r = smem_u32(s_raw + buffer * kSsChunk * 2);
        for (uint32_t i = threadIdx.x; i < n * 2; i += kSsThreads)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(r + i * 4u), "l"(src + size_t(i >> 1) * p.conv_ld + ((i & 1u) ? p.log_at : p.dt_at) + h) : "memory");
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    uint64_t Z[2][8];                                      // pairs of state rows
    float* state = a.S + (size_t(h) * a.vdim + c0 + pc) * N;
    const bool fresh = *a.pos == 0;
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const uint32_t n = 4 * (q * NL + slice);
            const bool live = !fresh && (c ? live1 : live0) && n < N;
            const float4 v = live ? *reinterpret_cast<const float4*>(state + c * N + n) : make_float4(0.f, 0.f, 0.f, 0.f);
            Z[c][2 * q] = ss_pack(v.x, v.y);
            Z[c][2 * q + 1] = ss_pack(v.z, v.w);
        }
    const uint32_t chunks = (T + kSsChunk - 1) / kSsChunk;
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        const uint32_t buffer = chunk & 1u, t0 = chunk * kSsChunk, n = min(uint32_t(kSsChunk), T - t0);
        if (chunk + 1 < chunks) {
            fetch(chunk + 1, buffer ^ 1u);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if (threadIdx.x < 32) {
            const uint32_t t = threadIdx.x;
            const float dt = t < n ? s_raw[buffer * kSsChunk * 2 + 2 * t] : 0.f;
            double L = t < n ? double(s_raw[buffer * kSsChunk * 2 + 2 * t + 1]) : 0.0;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double v = __shfl_up_sync(0xffffffffu, L, o);
                if (t >= uint32_t(o)) L += v;
            }
            const int band = int(-L / kSsReference);
            const int before = __shfl_up_sync(0xffffffffu, band, 1);
            const bool starts = t == 0 || band != before;
            const uint32_t upto = __ballot_sync(0xffffffffu, starts) & (0xffffffffu >> (31u - t));      // reference tokens up to this one
            const uint32_t ref = 31u - __clz(upto), rest = upto & ~(1u << ref), earlier = rest ? 31u - __clz(rest) : 0u;
            const double R = __shfl_sync(0xffffffffu, L, ref), R_before = __shfl_sync(0xffffffffu, L, earlier);
            s_f[t] = make_float4(dt * expf(float(R - L)), expf(float(L - R)), starts ? expf(float(t == 0 ? L : L - R_before)) : 1.f, 0.f);
        }
        __syncthreads();
        const float* xs = s_x + buffer * kSsChunk * p.columns + pc;
        const float* bs = s_b + buffer * kSsChunk * N + 4 * slice;
        const float* cs = s_c + buffer * kSsChunk * N + 4 * slice;
        auto token = [&](uint32_t t) {
            const float4 f = s_f[t];
            if (f.z != 1.f) {
                const uint64_t k = ss_pack(f.z, f.z);
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 8; ++i) Z[c][i] = ss_fma2(Z[c][i], k, 0ull);
            }
            const float x0 = live0 ? xs[t * p.columns] * f.x : 0.f, x1 = live1 ? xs[t * p.columns + 1] * f.x : 0.f;
            const uint64_t u0 = ss_pack(x0, x0), u1 = ss_pack(x1, x1);
            uint64_t y0[2] = {0ull, 0ull}, y1[2] = {0ull, 0ull};
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                if (uint32_t(4 * q * NL) >= N) continue;   // (uniform: N is a multiple of 4 NL or NL is all it needs)
                const bool in = 4 * (q * NL + slice) < N;
                const ulonglong2 b = in ? *reinterpret_cast<const ulonglong2*>(bs + t * N + 4 * q * NL) : make_ulonglong2(0ull, 0ull);
                const ulonglong2 c = in ? *reinterpret_cast<const ulonglong2*>(cs + t * N + 4 * q * NL) : make_ulonglong2(0ull, 0ull);
                Z[0][2 * q] = ss_fma2(b.x, u0, Z[0][2 * q]);
                Z[1][2 * q] = ss_fma2(b.x, u1, Z[1][2 * q]);
                Z[0][2 * q + 1] = ss_fma2(b.y, u0, Z[0][2 * q + 1]);
                Z[1][2 * q + 1] = ss_fma2(b.y, u1, Z[1][2 * q + 1]);
                y0[0] = ss_fma2(c.x, Z[0][2 * q], y0[0]);
                y1[0] = ss_fma2(c.x, Z[1][2 * q], y1[0]);
                y0[1] = ss_fma2(c.y, Z[0][2 * q + 1], y0[1]);
                y1[1] = ss_fma2(c.y, Z[1][2 * q + 1], y1[1]);
            }
            float a0 = ss_sum2(y0[0]) + ss_sum2(y0[1]), a1 = ss_sum2(y1[0]) + ss_sum2(y1[1]);
            ss_reduce<NL>(a0, a1);
            float* ys = s_y + t * p.columns + pc;
            if constexpr (NL == 1) {
                if (live0) ys[0] = a0 * f.y;
                if (live1) ys[1] = a1 * f.y;
            } else {
                if (slice == 0 && live0) ys[0] = a0 * f.y;
                if (slice == NL / 2 && live1) ys[1] = a0 * f.y;
            }
        };
        if (n == kSsChunk) {
#pragma unroll 4
            for (uint32_t t = 0; t < uint32_t(kSsChunk); ++t) token(t);
        } else {
            for (uint32_t t = 0; t < n; ++t) token(t);
        }
        const float end = s_f[n - 1].y;                    // back to the state itself
        const uint64_t k = ss_pack(end, end);
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 8; ++i) Z[c][i] = ss_fma2(Z[c][i], k, 0ull);
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < n * cols; i += kSsThreads) {
            const uint32_t t = i / cols, q = i - t * cols;
            const float z = a.raw[size_t(t0 + t) * a.raw_ld + h * a.vdim + c0 + q];
            const float y = fmaf(Dh, s_x[buffer * kSsChunk * p.columns + t * p.columns + q], s_y[t * p.columns + q]);
            p.gated[size_t(t0 + t) * p.inner + h * a.vdim + c0 + q] = y * silu_f32(z);
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const uint32_t n = 4 * (q * NL + slice);
            if (!(c ? live1 : live0) || n >= N) continue;
            float4 v;
            v.x = __uint_as_float(uint32_t(Z[c][2 * q])); v.y = __uint_as_float(uint32_t(Z[c][2 * q] >> 32));
            v.z = __uint_as_float(uint32_t(Z[c][2 * q + 1])); v.w = __uint_as_float(uint32_t(Z[c][2 * q + 1] >> 32));
            *reinterpret_cast<float4*>(state + c * N + n) = v;
        }
}

// One token.  The same split of a head's state; the CTA convolves the channels that it needs itself.
template <int NL>
__global__ void __launch_bounds__(kSsThreads) ssm_step_kernel(const SsmParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_ssm_args& a = p.a;
    const uint32_t blocks = (a.vdim + p.columns - 1) / p.columns, h = blockIdx.x / blocks, c0 = (blockIdx.x - h * blocks) * p.columns;
    const uint32_t cols = min(p.columns, a.vdim - c0), per_group = a.heads / a.groups, g = h / per_group, N = p.state_p;
    const uint32_t slice = threadIdx.x % NL, pc = threadIdx.x / NL * 2;
    float* s_b = reinterpret_cast<float*>(smem_raw);       // [N]
    float* s_c = s_b + N;
    float* s_x = s_c + N;                                  // [columns]
    const bool live0 = pc < cols, live1 = pc + 1 < cols;
    const float Dh = a.D[h], bias = a.dt_bias[h], A_log = a.A_log[h];
    pdl_wait();
    const uint32_t pos = *a.pos;
    float* state = a.S + (size_t(h) * a.vdim + c0 + pc) * N;
    float4 S[2][4];
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const uint32_t n = 4 * (q * NL + slice);
            S[c][q] = pos != 0 && (c ? live1 : live0) && n < N ? *reinterpret_cast<const float4*>(state + c * N + n) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    const float z0 = live0 ? a.raw[h * a.vdim + c0 + pc] : 0.f, z1 = live1 ? a.raw[h * a.vdim + c0 + pc + 1] : 0.f;
    const float dt = softplus_f32(a.raw[p.inner + p.channels + h] + bias), decay = expf(ss_log_decay(A_log, dt));
    for (uint32_t i = threadIdx.x; i < 2 * N + cols; i += kSsThreads) {
        uint32_t channel = ~0u;
        bool mine = true;                                  // one CTA writes a channel's history
        if (i < 2 * N) {
            const uint32_t n = i < N ? i : i - N;
            if (n < a.state) channel = p.inner + (i < N ? 0 : a.groups * a.state) + g * a.state + n;
            mine = h == g * per_group && c0 == 0;
        } else {
            channel = h * a.vdim + c0 + i - 2 * N;
        }
        float v = 0.f;
        if (channel != ~0u) {
            const float now = a.raw[p.inner + channel];
            v = fmaf(a.conv_w[size_t(a.taps - 1) * p.channels + channel], now, a.conv_b[channel]);
            for (uint32_t back = 1; back < a.taps && back <= pos; ++back)
                v = fmaf(a.conv_w[size_t(a.taps - 1 - back) * p.channels + channel], a.history[size_t((pos - back) % a.taps) * p.channels + channel], v);
            v = silu_f32(v);
            if (mine) a.history[size_t(pos % a.taps) * p.channels + channel] = now;      // (a row that no token of this step reads)
        }
        s_b[i] = v;                                        // s_b, s_c and s_x lie in a row
    }
    __syncthreads();
    const float x0 = live0 ? s_x[pc] : 0.f, x1 = live1 ? s_x[pc + 1] : 0.f;
    float y0 = 0.f, y1 = 0.f;
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const uint32_t n = 4 * (q * NL + slice);
        if (n >= N) continue;
        const float4 b = *reinterpret_cast<const float4*>(s_b + n), c = *reinterpret_cast<const float4*>(s_c + n);
        auto column = [&](float4& s, float u, float& y) {
            s.x = fmaf(decay, s.x, u * b.x); s.y = fmaf(decay, s.y, u * b.y); s.z = fmaf(decay, s.z, u * b.z); s.w = fmaf(decay, s.w, u * b.w);
            y = fmaf(c.x, s.x, y); y = fmaf(c.y, s.y, y); y = fmaf(c.z, s.z, y); y = fmaf(c.w, s.w, y);
        };
        column(S[0][q], dt * x0, y0);
        column(S[1][q], dt * x1, y1);
        if (live0) *reinterpret_cast<float4*>(state + n) = S[0][q];
        if (live1) *reinterpret_cast<float4*>(state + N + n) = S[1][q];
    }
    ss_reduce<NL>(y0, y1);
    float* out = p.gated + h * a.vdim + c0 + pc;
    if constexpr (NL == 1) {
        if (live0) out[0] = fmaf(Dh, x0, y0) * silu_f32(z0);
        if (live1) out[1] = fmaf(Dh, x1, y1) * silu_f32(z1);
    } else {
        if (slice == 0 && live0) out[0] = fmaf(Dh, x0, y0) * silu_f32(z0);
        if (slice == NL / 2 && live1) out[1] = fmaf(Dh, x1, y0) * silu_f32(z1);
    }
}

// CTA: one part of one token
template <typename OutT>
__global__ void __launch_bounds__(256) ssm_norm_kernel(const SsmParams p) {
    pdl_launch_dependents();
    __shared__ float scratch[64];
    const lv_ssm_args& a = p.a;
    const uint32_t t = blockIdx.y, n = p.inner / a.norm_groups, at = blockIdx.x * n;
    constexpr int kPer = 16;                               // values kept in registers
    float v[kPer], part = 0.f;
    pdl_wait();
    const float* src = p.gated + size_t(t) * p.inner + at;
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = threadIdx.x + k * blockDim.x;
        v[k] = i < n ? src[i] : 0.f;
        part = fmaf(v[k], v[k], part);
    }
    for (uint32_t i = threadIdx.x + kPer * blockDim.x; i < n; i += blockDim.x) part = fmaf(src[i], src[i], part);
    const float r = 1.f / sqrtf(block_sum(part, scratch) / float(n) + a.eps);
    OutT* out = static_cast<OutT*>(a.out) + size_t(t) * a.out_ld + at;
    auto store = [&](uint32_t i, float x) {
        const float y = x * r * a.norm_w[at + i];
        if constexpr (sizeof(OutT) == 2) out[i] = __float2bfloat16_rn(y);
        else out[i] = y;
    };
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = threadIdx.x + k * blockDim.x;
        if (i < n) store(i, v[k]);
    }
    for (uint32_t i = threadIdx.x + kPer * blockDim.x; i < n; i += blockDim.x) store(i, src[i]);
}

static void ssm_layout(SsmParams& p) {
    const lv_ssm_args& a = p.a;
    auto pad = [](uint32_t n, uint32_t to) { return (n + to - 1) / to * to; };
    p.inner = a.heads * a.vdim;
    p.channels = p.inner + 2 * a.groups * a.state;
    p.state_p = pad(a.state, 16);
    p.x_at = 0;
    p.b_at = pad(p.inner, 4);
    p.c_at = p.b_at + a.groups * p.state_p;
    p.dt_at = p.c_at + a.groups * p.state_p;
    p.log_at = p.dt_at + a.heads;
    p.conv_ld = pad(p.log_at + a.heads, 4);
}

template <int NL>
static int ssm_launch(lv_ctx* ctx, SsmParams& p) {
    const lv_ssm_args& a = p.a;
    p.columns = 2 * kSsThreads / NL;
    const dim3 grid(a.heads * ((a.vdim + p.columns - 1) / p.columns));
    if (p.batch == 1) {
        const size_t smem = sizeof(float) * (2 * p.state_p + p.columns);
        LV_CUDA(launch_pdl(ctx, ssm_step_kernel<NL>, grid, dim3(kSsThreads), smem, p));
        return LV_OK;
    }
    const size_t smem = sizeof(float) * kSsChunk * (4 * size_t(p.state_p) + 3 * p.columns + 4);
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "ssm: state needs too much shared memory");
    LV_CUDA(cudaFuncSetAttribute(ssm_scan_kernel<NL>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, ssm_scan_kernel<NL>, grid, dim3(kSsThreads), smem, p));
    return LV_OK;
}

}  // namespace lv

using namespace lv;

extern "C" size_t lv_ssm_scratch_bytes(const lv_ssm_args* a, uint32_t batch) {
    if (!a || !batch) return 0;
    SsmParams p{};
    p.a = *a;
    ssm_layout(p);
    return sizeof(float) * size_t(batch) * (p.conv_ld + (p.inner + 3) / 4 * 4);
}

extern "C" int lv_ssm(lv_ctx* ctx, const lv_ssm_args* a, void* scratch, size_t scratch_bytes, uint32_t batch) {
    LV_ENTER(ctx);
    LV_REQUIRE(a && a->raw && a->conv_w && a->conv_b && a->dt_bias && a->A_log && a->D && a->norm_w && a->history && a->S && a->pos && a->out && batch && batch <= 65535,
               "bad ssm arguments");
    LV_REQUIRE(a->heads && a->vdim && a->groups && a->heads % a->groups == 0 && a->norm_groups && (a->heads * a->vdim) % a->norm_groups == 0, "ssm: groups do not divide the heads");
    LV_REQUIRE(a->state && a->state <= kSsMaxState && a->taps && a->taps <= kSsMaxTaps, "ssm: more than 256 state rows or 16 taps");
    SsmParams p{};
    p.a = *a;
    ssm_layout(p);
    p.batch = batch;
    LV_REQUIRE(a->raw_ld >= p.inner + p.channels + a->heads && a->out_ld >= p.inner && (a->out_type == LV_TYPE_F32 || a->out_type == LV_TYPE_BF16), "ssm: bad strides");
    LV_REQUIRE((reinterpret_cast<uintptr_t>(a->S) & 15u) == 0 && scratch && (reinterpret_cast<uintptr_t>(scratch) & 15u) == 0 &&
               scratch_bytes >= lv_ssm_scratch_bytes(a, batch), "ssm: bad scratch or state");
    p.conv = static_cast<float*>(scratch);
    p.gated = p.conv + size_t(batch) * p.conv_ld;
    if (batch > 1) {
        const uint32_t cta_columns = (p.conv_ld + kSsThreads - 1) / kSsThreads;
        p.tokens_per_block = 32;
        while (p.tokens_per_block > 8 && cta_columns * ((batch + p.tokens_per_block - 1) / p.tokens_per_block) < 4u * uint32_t(ctx->sm_count)) p.tokens_per_block /= 2;
        if (p.tokens_per_block < a->taps) p.tokens_per_block = a->taps;
        const dim3 grid(cta_columns, (batch + p.tokens_per_block - 1) / p.tokens_per_block);
        auto* conv = a->taps <= 4 ? ssm_conv_kernel<4> : a->taps <= 8 ? ssm_conv_kernel<8> : ssm_conv_kernel<16>;
        LV_CUDA(launch_pdl(ctx, conv, grid, dim3(kSsThreads), 0, p));
    }
    // lanes that share a column: sixteen state rows each
    int rc = LV_OK;
    if (p.state_p <= 16) rc = ssm_launch<1>(ctx, p);
    else if (p.state_p <= 32) rc = ssm_launch<2>(ctx, p);
    else if (p.state_p <= 64) rc = ssm_launch<4>(ctx, p);
    else if (p.state_p <= 128) rc = ssm_launch<8>(ctx, p);
    else rc = ssm_launch<16>(ctx, p);
    if (rc != LV_OK) return rc;
    const uint32_t part = p.inner / a->norm_groups, threads = part >= 2048 ? 256 : part >= 512 ? 128 : 64;
    const dim3 grid(a->norm_groups, batch);
    if (a->out_type == LV_TYPE_BF16) LV_CUDA(launch_pdl(ctx, ssm_norm_kernel<__nv_bfloat16>, grid, dim3(threads), 0, p));
    else LV_CUDA(launch_pdl(ctx, ssm_norm_kernel<float>, grid, dim3(threads), 0, p));
    return LV_OK;
}
