// Selective state spaces (lv_ssm_args): a short causal convolution, a linear recurrence with one decay per head and token, gate and
// grouped norm.
//
//   several tokens   ssm_conv_kernel   convolution, silu, step sizes and logarithms of the decays
//                    ssm_scan_kernel   the recurrence, D x and the gate; for bfloat16 models chunks of tokens as matrix products
//                                      instead (state_space_tc.cu)
//   one token        ssm_step_kernel   all of that
//   both             ssm_norm_kernel   RMS norm of each part
//
// The recurrence S_t = a_t S_(t-1) + dt_t B_t x_t^T is carried in f32 registers: a CTA has some columns of one head's state, a thread two
// columns and sixteen of the state's rows.  Tokens come in chunks of 32 through shared memory.  Within a chunk the state is
// kept relative to its decay, S_t = exp(L_t - R) Z_t with L the running sum of log a and R its value at a reference token, so
// that a token costs one multiply-add per element for Z += (dt exp(R - L)) B x^T and one for y = exp(L - R) C Z (two elements per
// instruction); a new reference is taken whenever L has moved on by 32, which bounds every factor.  L is summed in f64.  The lanes
// that share a column exchange the sums of four tokens at a time.
#include <cuda_bf16.h>
#include <math.h>

#include "common.cuh"
#include "ctx.h"
#include "state_space.cuh"

namespace lv {

constexpr int kSsThreads = 128;              // of the convolution; at most of the others
// columns of a head per CTA and threads of it when NL lanes share a column
__host__ __device__ constexpr int ss_columns(int NL) { return NL <= 4 ? 64 : 256 / NL; }
__host__ __device__ constexpr int ss_threads(int NL) { return ss_columns(NL) / 2 * NL; }
constexpr int kSsChunk = 32;                 // tokens
constexpr double kSsReference = 32.0;
constexpr int kSsConvTokens = 16;            // tokens of a block of the convolution; at least the taps - 1 before them

__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ss_log_decay(float A_log, float dt) { return fmaxf(-expf(A_log) * dt, kSsMinLog); }

// two f32 in one register pair
__device__ __forceinline__ uint64_t ss_pack(float lo, float hi) { return uint64_t(__float_as_uint(lo)) | (uint64_t(__float_as_uint(hi)) << 32); }
__device__ __forceinline__ uint64_t ss_fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t ss_mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t ss_add2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float ss_sum2(uint64_t v) { return __uint_as_float(uint32_t(v)) + __uint_as_float(uint32_t(v >> 32)); }

// Columns of `conv`, then dt and log a of the heads: a thread owns one column and kSsConvTokens tokens, all loads before the first use.
// Block row 0 alone reads the history, whose successor it writes.
template <typename OutT, int MAXT>
__global__ void __launch_bounds__(kSsThreads) ssm_conv_kernel(const SsmParams p) {
    pdl_launch_dependents();
    const lv_ssm_args& a = p.a;
    const uint32_t col = blockIdx.x * kSsThreads + threadIdx.x, T = p.batch, t0 = blockIdx.y * kSsConvTokens;
    if (col >= p.conv_ld + 2 * a.heads) return;
    const bool rate = col >= p.conv_ld;
    const uint32_t h = rate ? (col - p.conv_ld) >> 1 : 0;
    uint32_t channel = ~0u;                      // of the convolution; none: padding, or a rate
    if (col < p.inner) {
        channel = col;
    } else if (!rate && col >= p.b_at) {
        const bool second = col >= p.c_at;
        const uint32_t g = (col - (second ? p.c_at : p.b_at)) / p.state_p, n = (col - (second ? p.c_at : p.b_at)) - g * p.state_p;
        if (g < a.groups && n < a.state) channel = p.inner + (second ? a.groups * a.state : 0) + g * a.state + n;
    }
    const bool conv = channel != ~0u;
    float w[MAXT], bias = 0.f, A_log = 0.f;      // taps right-aligned: index MAXT - 1 is the current token
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
        const int s = j - (MAXT - int(a.taps));
        w[j] = conv && s >= 0 ? a.conv_w[size_t(s) * p.channels + channel] : 0.f;
    }
    if (conv) bias = a.conv_b[channel];
    if (rate) {
        bias = a.dt_bias[h];
        A_log = a.A_log[h];
    }
    pdl_wait();
    const uint32_t pos = *a.pos;
    const float* raw = a.raw + p.inner + (conv ? channel : p.channels + h);
    float* history = a.history + channel;
    float v[MAXT - 1 + kSsConvTokens];           // v[MAXT - 1 + i]: token t0 + i
#pragma unroll
    for (int i = 0; i < MAXT - 1 + kSsConvTokens; ++i) {
        const int t = int(t0) + i - (MAXT - 1), back = -t;
        v[i] = 0.f;
        if (t >= 0 && t < int(T) && (conv || (rate && i >= MAXT - 1))) v[i] = raw[size_t(t) * a.raw_ld];
        else if (t < 0 && conv && back < int(a.taps) && pos >= uint32_t(back)) v[i] = history[size_t((pos - back) % a.taps) * p.channels];
    }
    if (rate) {
        float* out = p.rates + size_t(t0) * a.heads * 2 + (col - p.conv_ld);
#pragma unroll
        for (int i = 0; i < kSsConvTokens; ++i) {
            const float dt = softplus_f32(v[MAXT - 1 + i] + bias);
            if (t0 + i < T) out[size_t(i) * a.heads * 2] = (col - p.conv_ld) & 1u ? ss_log_decay(A_log, dt) : dt;
        }
        return;
    }
    OutT* out = static_cast<OutT*>(p.conv) + size_t(t0) * p.conv_ld + col;
#pragma unroll
    for (int i = 0; i < kSsConvTokens; ++i) {
        float y = bias;
#pragma unroll
        for (int j = 0; j < MAXT; ++j) y = fmaf(w[j], v[i + j], y);
        if (t0 + i >= T) continue;               // (padding: zero)
        if constexpr (sizeof(OutT) == 2) out[size_t(i) * p.conv_ld] = __float2bfloat16_rn(silu_fast(y));
        else out[size_t(i) * p.conv_ld] = silu_f32(y);
    }
    if (blockIdx.y != 0 || !conv) return;
    for (uint32_t t = T > a.taps ? T - a.taps : 0; t < T; ++t) history[size_t((pos + t) % a.taps) * p.channels] = raw[size_t(t) * a.raw_ld];
}

template <int NL> __host__ __device__ constexpr size_t ss_scan_floats() {
    constexpr int N = 16 * NL, cols = ss_columns(NL);
    return size_t(kSsChunk) * (4 * N + 4 * cols + 3 * cols + 4);
}

// NL lanes share a column, sixteen state rows each: four at a time, 4 (q NL + slice) .. + 3 for q < 4 (conflict-free in shared memory,
// contiguous over lanes).
template <int NL>
__global__ void __launch_bounds__(ss_threads(NL)) ssm_scan_kernel(const SsmParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const lv_ssm_args& a = p.a;
    constexpr uint32_t N = 16 * NL, kCols = ss_columns(NL), kThreads = ss_threads(NL);
    constexpr int kGroup = 4, V = 2 * kGroup;              // tokens whose sums are exchanged together
    const uint32_t blocks = (a.vdim + kCols - 1) / kCols, h = blockIdx.x / blocks, c0 = (blockIdx.x - h * blocks) * kCols;
    const uint32_t cols = min(kCols, a.vdim - c0), g = h / (a.heads / a.groups);
    const uint32_t slice = threadIdx.x % NL, pc = threadIdx.x / NL * 2;       // columns pc, pc + 1 of the CTA's
    float* s_b = reinterpret_cast<float*>(smem_raw);       // [2][chunk][N]
    float* s_c = s_b + 2 * kSsChunk * N;
    float* s_x = s_c + 2 * kSsChunk * N;                   // [2][chunk][columns]
    float* s_z = s_x + 2 * kSsChunk * kCols;               // the same
    float2* s_u = reinterpret_cast<float2*>(s_z + 2 * kSsChunk * kCols);      // [chunk][columns]: x dt exp(R - L), twice
    float* s_y = reinterpret_cast<float*>(s_u + kSsChunk * kCols);            // [chunk][columns]
    float* s_raw = s_y + kSsChunk * kCols;                 // [2][chunk][2]: dt, log a
    __shared__ float s_in[kSsChunk], s_out[kSsChunk], s_turn[kSsChunk];       // dt exp(R - L), exp(L - R), factor of Z at a new reference
    __shared__ uint32_t s_refs;                            // tokens that are references
    const bool live0 = pc < cols, live1 = pc + 1 < cols;
    const float Dh = a.D[h];
    pdl_wait();
    const uint32_t T = p.batch;
    auto copy4 = [](const float* dst, const float* src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory"); };
    auto fetch = [&](uint32_t chunk, uint32_t buffer) {
        const uint32_t t0 = chunk * kSsChunk, n = min(uint32_t(kSsChunk), T - t0);
        const float* src = static_cast<const float*>(p.conv) + size_t(t0) * p.conv_ld;
        const float* z = a.raw + size_t(t0) * a.raw_ld + h * a.vdim + c0;
#pragma unroll 4
        for (uint32_t i = threadIdx.x; i < n * (N / 4); i += kThreads) {
            const uint32_t t = i / (N / 4), q = i % (N / 4);
            const float* at = src + size_t(t) * p.conv_ld + g * N + q * 4;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(s_b + buffer * kSsChunk * N + i * 4)), "l"(at + p.b_at) : "memory");
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(s_c + buffer * kSsChunk * N + i * 4)), "l"(at + p.c_at) : "memory");
        }
#pragma unroll 4
        for (uint32_t i = threadIdx.x; i < n * kCols; i += kThreads) {
            const uint32_t t = i / kCols, q = i % kCols;
            if (q >= cols) continue;
            copy4(s_x + buffer * kSsChunk * kCols + i, src + size_t(t) * p.conv_ld + h * a.vdim + c0 + q);
            copy4(s_z + buffer * kSsChunk * kCols + i, z + size_t(t) * a.raw_ld + q);
        }
        // the rows that complete the last group of tokens
        for (uint32_t i = n * N + threadIdx.x; i < (n + kGroup - 1) / kGroup * kGroup * N; i += kThreads) s_b[buffer * kSsChunk * N + i] = 0.f;
        for (uint32_t i = threadIdx.x; i < n * 2; i += kThreads) copy4(s_raw + buffer * kSsChunk * 2 + i, p.rates + (size_t(t0 + (i >> 1)) * a.heads + h) * 2 + (i & 1u));
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    uint64_t Z[2][8];                                      // pairs of state rows
    float* state = a.S + (size_t(h) * a.vdim + c0 + pc) * N + 4 * slice;
    const bool fresh = *a.pos == 0;
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const float4 v = !fresh && (c ? live1 : live0) ? *reinterpret_cast<const float4*>(state + c * N + 4 * q * NL) : make_float4(0.f, 0.f, 0.f, 0.f);
            Z[c][2 * q] = ss_pack(v.x, v.y);
            Z[c][2 * q + 1] = ss_pack(v.z, v.w);
        }
    auto scale = [&](float f) {
        const uint64_t k = ss_pack(f, f);
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 8; ++i) Z[c][i] = ss_mul2(Z[c][i], k);
    };
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
            const int band = int(-L * (1.0 / kSsReference));
            const int before = __shfl_up_sync(0xffffffffu, band, 1);
            const uint32_t refs = __ballot_sync(0xffffffffu, t == 0 || band != before);
            const uint32_t upto = refs & (0xffffffffu >> (31u - t));          // reference tokens up to this one
            const uint32_t ref = 31u - __clz(upto), rest = upto & ~(1u << ref), earlier = rest ? 31u - __clz(rest) : 0u;
            const double R = __shfl_sync(0xffffffffu, L, ref), R_before = __shfl_sync(0xffffffffu, L, earlier);
            s_in[t] = dt * expf(float(R - L));
            s_out[t] = expf(float(L - R));
            s_turn[t] = expf(float(t == 0 ? L : L - R_before));               // (read at references only)
            if (t == 0) s_refs = refs;
        }
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < uint32_t(kSsChunk) * kCols; i += kThreads) {
            const uint32_t t = i / kCols, q = i % kCols;
            const float u = t < n && q < cols ? s_x[buffer * kSsChunk * kCols + i] * s_in[t] : 0.f;
            s_u[i] = make_float2(u, u);
        }
        __syncthreads();
        const float* bs = s_b + buffer * kSsChunk * N + 4 * slice;
        const float* cs = s_c + buffer * kSsChunk * N + 4 * slice;
        const uint32_t refs = s_refs;
        // (tokens behind the last one of a short chunk add nothing, and their sums are not used)
        // a token's operands are requested while the one before it is worked on (behind the chunk: rows that are not used)
        ulonglong2 bq[2][4], cq[2][4], uq[2];
        auto load = [&](uint32_t t, int into) {
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                bq[into][q] = *reinterpret_cast<const ulonglong2*>(bs + t * N + 4 * q * NL);
                cq[into][q] = *reinterpret_cast<const ulonglong2*>(cs + t * N + 4 * q * NL);
            }
            uq[into] = *reinterpret_cast<const ulonglong2*>(s_u + t * kCols + pc);
        };
        load(0, 0);
#pragma unroll 1
        for (uint32_t first = 0; first < n; first += kGroup) {
            float y[V];
            const bool turns = __any_sync(0xffffffffu, (refs >> first & ((1u << kGroup) - 1u)) != 0);
#pragma unroll
            for (int i = 0; i < kGroup; ++i) {
                const uint32_t t = first + i;
                load(t + 1, (i + 1) & 1);
                if (turns)
                    if (refs >> t & 1u) scale(s_turn[t]);
                const ulonglong2 u = uq[i & 1];
                uint64_t y0[2], y1[2];
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const ulonglong2 b = bq[i & 1][q];
                    Z[0][2 * q] = ss_fma2(b.x, u.x, Z[0][2 * q]);
                    Z[1][2 * q] = ss_fma2(b.x, u.y, Z[1][2 * q]);
                    Z[0][2 * q + 1] = ss_fma2(b.y, u.x, Z[0][2 * q + 1]);
                    Z[1][2 * q + 1] = ss_fma2(b.y, u.y, Z[1][2 * q + 1]);
                }
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const ulonglong2 c = cq[i & 1][q];
                    y0[0] = q ? ss_fma2(c.x, Z[0][2 * q], y0[0]) : ss_mul2(c.x, Z[0][2 * q]);
                    y1[0] = q ? ss_fma2(c.x, Z[1][2 * q], y1[0]) : ss_mul2(c.x, Z[1][2 * q]);
                    y0[1] = q ? ss_fma2(c.y, Z[0][2 * q + 1], y0[1]) : ss_mul2(c.y, Z[0][2 * q + 1]);
                    y1[1] = q ? ss_fma2(c.y, Z[1][2 * q + 1], y1[1]) : ss_mul2(c.y, Z[1][2 * q + 1]);
                }
                y[2 * i] = ss_sum2(ss_add2(y0[0], y0[1]));
                y[2 * i + 1] = ss_sum2(ss_add2(y1[0], y1[1]));
            }
            lanes_reduce<NL, V>(y);
            constexpr int kKeep = V >= NL ? V / NL : 1;
            if (V >= NL || slice % (NL / V > 0 ? NL / V : 1) == 0) {
                const uint32_t at = V >= NL ? slice * kKeep : slice / (NL / V > 0 ? NL / V : 1);
#pragma unroll
                for (int k = 0; k < kKeep; ++k) s_y[(first + (at + k) / 2) * kCols + pc + ((at + k) & 1u)] = y[k];
            }
        }
        scale(s_out[n - 1]);                               // back to the state itself
        __syncthreads();
#pragma unroll 2
        for (uint32_t i = threadIdx.x; i < n * kCols; i += kThreads) {
            const uint32_t t = i / kCols, q = i % kCols;
            if (q >= cols) continue;
            const float y = fmaf(Dh, s_x[buffer * kSsChunk * kCols + i], s_y[i] * s_out[t]);
            p.gated[size_t(t0 + t) * p.inner + h * a.vdim + c0 + q] = y * silu_f32(s_z[buffer * kSsChunk * kCols + i]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            if (!(c ? live1 : live0)) continue;
            float4 v;
            v.x = __uint_as_float(uint32_t(Z[c][2 * q])); v.y = __uint_as_float(uint32_t(Z[c][2 * q] >> 32));
            v.z = __uint_as_float(uint32_t(Z[c][2 * q + 1])); v.w = __uint_as_float(uint32_t(Z[c][2 * q + 1] >> 32));
            *reinterpret_cast<float4*>(state + c * N + 4 * q * NL) = v;
        }
}

// One token.  The same split of a head's state; the CTA convolves the channels that it needs itself.
template <int NL, int MAXT>
__global__ void __launch_bounds__(ss_threads(NL)) ssm_step_kernel(const SsmParams p) {
    pdl_launch_dependents();
    const lv_ssm_args& a = p.a;
    constexpr uint32_t N = 16 * NL, kCols = ss_columns(NL), kThreads = ss_threads(NL);
    const uint32_t blocks = (a.vdim + kCols - 1) / kCols, h = blockIdx.x / blocks, c0 = (blockIdx.x - h * blocks) * kCols;
    const uint32_t cols = min(kCols, a.vdim - c0), per_group = a.heads / a.groups, g = h / per_group;
    const uint32_t slice = threadIdx.x % NL, pc = threadIdx.x / NL * 2;
    __shared__ __align__(16) float s_conv[2 * N + kCols];  // B, C, x
    const float *s_b = s_conv, *s_c = s_b + N, *s_x = s_c + N;
    const bool live0 = pc < cols, live1 = pc + 1 < cols;
    const float Dh = a.D[h], bias = a.dt_bias[h], A_log = a.A_log[h];
    // the channels that this thread convolves, with their taps
    constexpr int kPer = (2 * N + kCols + kThreads - 1) / kThreads;
    uint32_t channel[kPer];
    float w[kPer][MAXT], b[kPer];
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = threadIdx.x + k * kThreads;
        channel[k] = ~0u;
        if (i < 2 * N) {
            if (i % N < a.state) channel[k] = p.inner + (i < N ? 0 : a.groups * a.state) + g * a.state + i % N;
        } else if (i < 2 * N + cols) {
            channel[k] = h * a.vdim + c0 + i - 2 * N;
        }
        b[k] = channel[k] != ~0u ? a.conv_b[channel[k]] : 0.f;
#pragma unroll
        for (int j = 0; j < MAXT; ++j) w[k][j] = channel[k] != ~0u && j < int(a.taps) ? a.conv_w[size_t(a.taps - 1 - j) * p.channels + channel[k]] : 0.f;
    }
    pdl_wait();
    const uint32_t pos = *a.pos;
    // all loads before the first use
    float now[kPer], old[kPer][MAXT];
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        now[k] = channel[k] != ~0u ? a.raw[p.inner + channel[k]] : 0.f;
#pragma unroll
        for (int j = 1; j < MAXT; ++j)
            old[k][j] = channel[k] != ~0u && j < int(a.taps) && uint32_t(j) <= pos ? a.history[size_t((pos - j) % a.taps) * p.channels + channel[k]] : 0.f;
    }
    float* state = a.S + (size_t(h) * a.vdim + c0 + pc) * N + 4 * slice;
    float4 S[2][4];
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q)
            S[c][q] = pos != 0 && (c ? live1 : live0) ? *reinterpret_cast<const float4*>(state + c * N + 4 * q * NL) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float z0 = live0 ? a.raw[h * a.vdim + c0 + pc] : 0.f, z1 = live1 ? a.raw[h * a.vdim + c0 + pc + 1] : 0.f;
    const float dt = softplus_f32(a.raw[p.inner + p.channels + h] + bias), decay = expf(ss_log_decay(A_log, dt));
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = threadIdx.x + k * kThreads;
        float v = fmaf(w[k][0], now[k], b[k]);
#pragma unroll
        for (int j = 1; j < MAXT; ++j) v = fmaf(w[k][j], old[k][j], v);
        if (i < 2 * N + kCols) s_conv[i] = silu_f32(v);    // (padding: zero)
        // one CTA writes a channel's history, to a row that no token of this step reads
        if (channel[k] != ~0u && (i >= 2 * N || (h == g * per_group && c0 == 0))) a.history[size_t(pos % a.taps) * p.channels + channel[k]] = now[k];
    }
    __syncthreads();
    const float x0 = live0 ? s_x[pc] : 0.f, x1 = live1 ? s_x[pc + 1] : 0.f;
    float y[2] = {0.f, 0.f};
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const float4 bq = *reinterpret_cast<const float4*>(s_b + 4 * (q * NL + slice)), cq = *reinterpret_cast<const float4*>(s_c + 4 * (q * NL + slice));
        auto column = [&](float4& s, float u, float& sum) {
            s.x = fmaf(decay, s.x, u * bq.x); s.y = fmaf(decay, s.y, u * bq.y); s.z = fmaf(decay, s.z, u * bq.z); s.w = fmaf(decay, s.w, u * bq.w);
            sum = fmaf(cq.x, s.x, sum); sum = fmaf(cq.y, s.y, sum); sum = fmaf(cq.z, s.z, sum); sum = fmaf(cq.w, s.w, sum);
        };
        column(S[0][q], dt * x0, y[0]);
        column(S[1][q], dt * x1, y[1]);
        if (live0) *reinterpret_cast<float4*>(state + 4 * q * NL) = S[0][q];
        if (live1) *reinterpret_cast<float4*>(state + N + 4 * q * NL) = S[1][q];
    }
    lanes_reduce<NL, 2>(y);
    float* out = p.gated + h * a.vdim + c0 + pc;
    if constexpr (NL == 1) {
        if (live0) out[0] = fmaf(Dh, x0, y[0]) * silu_f32(z0);
        if (live1) out[1] = fmaf(Dh, x1, y[1]) * silu_f32(z1);
    } else {
        if (slice == 0 && live0) out[0] = fmaf(Dh, x0, y[0]) * silu_f32(z0);
        if (slice == NL / 2 && live1) out[1] = fmaf(Dh, x1, y[0]) * silu_f32(z1);
    }
}

// CTA: one part of one token; VEC values per access
template <typename OutT, int VEC>
__global__ void __launch_bounds__(256) ssm_norm_kernel(const SsmParams p) {
    pdl_launch_dependents();
    __shared__ float scratch[64];
    const lv_ssm_args& a = p.a;
    const uint32_t t = blockIdx.y, n = p.inner / a.norm_groups, at = blockIdx.x * n;
    constexpr int kPer = VEC == 4 ? 4 : 16;                // accesses kept in registers
    struct alignas(4 * VEC) Vec { float v[VEC]; };
    Vec x[kPer], w[kPer];
    const float* src = p.gated + size_t(t) * p.inner + at;
    auto weight = [&](uint32_t i) { return *reinterpret_cast<const Vec*>(a.norm_w + at + i); };
    auto value = [&](uint32_t i) { return *reinterpret_cast<const Vec*>(src + i); };
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
        if (i < n) w[k] = weight(i);
    }
    pdl_wait();
    float part = 0.f;
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
        if (i < n) x[k] = value(i);
    }
    auto add = [&](const Vec& v) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) part = fmaf(v.v[e], v.v[e], part);
    };
#pragma unroll
    for (int k = 0; k < kPer; ++k)
        if ((threadIdx.x + k * blockDim.x) * VEC < n) add(x[k]);
    for (uint32_t i = (threadIdx.x + kPer * blockDim.x) * VEC; i < n; i += blockDim.x * VEC) add(value(i));
    const float r = 1.f / sqrtf(block_sum(part, scratch) / float(n) + a.eps);
    OutT* out = static_cast<OutT*>(a.out) + size_t(t) * a.out_ld + at;
    auto store = [&](uint32_t i, const Vec& v, const Vec& f) {
        struct alignas(sizeof(OutT) * VEC) Out { OutT v[VEC]; } o;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float y = v.v[e] * r * f.v[e];
            if constexpr (sizeof(OutT) == 2) o.v[e] = __float2bfloat16_rn(y);
            else o.v[e] = y;
        }
        *reinterpret_cast<Out*>(out + i) = o;
    };
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
        const uint32_t i = (threadIdx.x + k * blockDim.x) * VEC;
        if (i < n) store(i, x[k], w[k]);
    }
    for (uint32_t i = (threadIdx.x + kPer * blockDim.x) * VEC; i < n; i += blockDim.x * VEC) store(i, value(i), weight(i));
}

static bool ssm_tc(const lv_ssm_args& a, uint32_t batch) {
    return batch > 1 && a.form != LV_SSM_SCAN && (a.form == LV_SSM_TENSOR || a.out_type == LV_TYPE_BF16) && ssm_tc_supported(a);
}

static void ssm_layout(SsmParams& p) {
    const lv_ssm_args& a = p.a;
    auto pad8 = [](uint32_t n) { return (n + 7) / 8 * 8; };
    p.inner = a.heads * a.vdim;
    p.channels = p.inner + 2 * a.groups * a.state;
    p.state_p = lv_ssm_state_rows(a.state);
    p.b_at = pad8(p.inner);
    p.c_at = p.b_at + a.groups * p.state_p;
    p.conv_ld = p.c_at + a.groups * p.state_p;
}

template <typename OutT>
static int ssm_conv_launch(lv_ctx* ctx, const SsmParams& p) {
    const dim3 grid((p.conv_ld + 2 * p.a.heads + kSsThreads - 1) / kSsThreads, (p.batch + kSsConvTokens - 1) / kSsConvTokens);
    auto* conv = p.a.taps <= 4 ? ssm_conv_kernel<OutT, 4> : p.a.taps <= 8 ? ssm_conv_kernel<OutT, 8> : ssm_conv_kernel<OutT, 16>;
    LV_CUDA(launch_pdl(ctx, conv, grid, dim3(kSsThreads), 0, p));
    return LV_OK;
}

template <int NL>
static int ssm_launch(lv_ctx* ctx, SsmParams& p) {
    const lv_ssm_args& a = p.a;
    constexpr uint32_t kCols = ss_columns(NL);
    const dim3 grid(a.heads * ((a.vdim + kCols - 1) / kCols));
    if (p.batch == 1) {
        LV_CUDA(launch_pdl(ctx, a.taps <= 4 ? ssm_step_kernel<NL, 4> : ssm_step_kernel<NL, 16>, grid, dim3(ss_threads(NL)), 0, p));
        return LV_OK;
    }
    constexpr size_t smem = sizeof(float) * ss_scan_floats<NL>();
    LV_REQUIRE(smem <= size_t(ctx->max_smem_optin), "ssm: state needs too much shared memory");
    LV_CUDA(cudaFuncSetAttribute(ssm_scan_kernel<NL>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    LV_CUDA(launch_pdl(ctx, ssm_scan_kernel<NL>, grid, dim3(ss_threads(NL)), smem, p));
    return LV_OK;
}

template <typename OutT>
static int ssm_norm_launch(lv_ctx* ctx, const SsmParams& p) {
    const lv_ssm_args& a = p.a;
    auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
    const uint32_t part = p.inner / a.norm_groups;
    const bool vec = part % 4 == 0 && p.inner % 4 == 0 && a.out_ld % 4 == 0 && aligned(a.out) && aligned(a.norm_w);
    const uint32_t units = vec ? part / 4 : part, threads = units > 512 ? 256 : units > 128 ? 128 : units > 32 ? 64 : 32;
    LV_CUDA(launch_pdl(ctx, vec ? ssm_norm_kernel<OutT, 4> : ssm_norm_kernel<OutT, 1>, dim3(a.norm_groups, p.batch), dim3(threads), 0, p));
    return LV_OK;
}

}  // namespace lv

using namespace lv;

extern "C" uint32_t lv_ssm_state_rows(uint32_t state) {
    uint32_t n = 16;
    while (n < state && n < kSsMaxState) n *= 2;
    return n;
}

extern "C" size_t lv_ssm_scratch_bytes(const lv_ssm_args* a, uint32_t batch) {
    if (!a || !batch) return 0;
    SsmParams p{};
    p.a = *a;
    ssm_layout(p);
    return sizeof(float) * size_t(batch) * (p.conv_ld + (p.inner + 3) / 4 * 4 + 2 * a->heads);
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
    LV_REQUIRE(a->form != LV_SSM_TENSOR || batch == 1 || ssm_tc_supported(*a), "ssm: the tensor-core form does not take these sizes");
    p.conv = scratch;
    p.gated = static_cast<float*>(scratch) + size_t(batch) * p.conv_ld;
    p.rates = p.gated + size_t(batch) * ((p.inner + 3) / 4 * 4);
    const bool tensor = ssm_tc(*a, batch);
    int rc = LV_OK;
    if (batch > 1) rc = tensor ? ssm_conv_launch<__nv_bfloat16>(ctx, p) : ssm_conv_launch<float>(ctx, p);
    if (rc != LV_OK) return rc;
    // lanes that share a column: sixteen state rows each
    if (tensor) rc = ssm_tc_launch(ctx, p);
    else if (p.state_p <= 16) rc = ssm_launch<1>(ctx, p);
    else if (p.state_p <= 32) rc = ssm_launch<2>(ctx, p);
    else if (p.state_p <= 64) rc = ssm_launch<4>(ctx, p);
    else if (p.state_p <= 128) rc = ssm_launch<8>(ctx, p);
    else rc = ssm_launch<16>(ctx, p);
    if (rc != LV_OK) return rc;
    return a->out_type == LV_TYPE_BF16 ? ssm_norm_launch<__nv_bfloat16>(ctx, p) : ssm_norm_launch<float>(ctx, p);
}
