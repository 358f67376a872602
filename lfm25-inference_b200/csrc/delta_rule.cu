// The generalised delta rule with a decay per key channel:
//     u_t = k_t / sqrt(|k_t|^2 + 1e-6)
//     S_t = diag(w_t) S_(t-1) - (a_t * u_t) (u_t^T S_(t-1)) + k_t v_t^T          o_t = S_t^T r_t
// per head, with w_t = exp(-exp(-1/2) sigmoid(W2 tanh(z_t) + w0)) and a_t = sigmoid(a_t' + bias), followed by the
// head's RMS norm, the norm weight and the output gate.
//
// A column of S (one value channel) never meets another one, so a CTA takes the columns of one head of one sequence and
// keeps them in registers over the whole segment: the state is read from and written to memory once per step however
// long the segment is.  Four kernels:
//   decode    one token per sequence: every load is issued up front, then three barriers
//   chunk     bf16 segments, heads up to 64: tiles of 16 tokens as matrix products on the tensor cores
//   prompt    bf16 segments, larger heads: half of the warps prepare a tile of 16 tokens (decays with one small tensor-core product,
//             removal rates, unit scales) and finish the previous one (norm, gate), the others run the recurrence over
//             the tile between them; projections arrive through cp.async two tiles ahead
//   general   any activation type and head size
// Outside the chunk kernel (see there) all arithmetic on the state is f32 multiply-adds, two-wide where the sm_100 packed instructions take it (each half
// rounds like the scalar one).
#include <math.h>

#include <type_traits>

#include "launch.h"
#include "options.h"
#include "stack_common.cuh"

namespace lfm25 {

namespace {

using Pair = unsigned long long;     // two f32 values

__device__ __forceinline__ Pair pair_of(float low, float high) {
    Pair out;
    asm("mov.b64 %0, {%1, %2};" : "=l"(out) : "f"(low), "f"(high));
    return out;
}
__device__ __forceinline__ float pair_sum(Pair value) {
    float low, high;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(low), "=f"(high) : "l"(value));
    return low + high;
}
__device__ __forceinline__ float low_of(Pair value) { return __uint_as_float(static_cast<uint32_t>(value)); }
__device__ __forceinline__ float high_of(Pair value) { return __uint_as_float(static_cast<uint32_t>(value >> 32)); }
__device__ __forceinline__ Pair fma_pair(Pair a, Pair b, Pair c) {
    Pair out;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(out) : "l"(a), "l"(b), "l"(c));
    return out;
}
__device__ __forceinline__ Pair add_pair(Pair a, Pair b) {
    Pair out;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(out) : "l"(a), "l"(b));
    return out;
}
__device__ __forceinline__ Pair mul_pair(Pair a, Pair b) {
    Pair out;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(out) : "l"(a), "l"(b));
    return out;
}

constexpr float kUnitEps = 1e-6f;
constexpr float kDecayScale = 0.60653065971263342f;    // exp(-1/2)

template <typename T>
struct DeltaArgs {
    StackSegments segments;
    uint32_t heads, dim, rank;
    const T* projected;
    size_t pitch;
    const __nv_bfloat16* decay_up;
    const __nv_bfloat16* decay_base;
    const __nv_bfloat16* removal_bias;
    const __nv_bfloat16* norm;
    StackRecord record;
    float* raw;
    T* out;
    size_t out_pitch;
    float eps;
    uint32_t splits;         // CTAs per head, each with COLUMNS value channels
};

constexpr uint32_t kTileTokens = 16;
// per token in shared memory: r, w, -(a * u), u, k over the padded key channels, then v over them as well
constexpr uint32_t kVectors = 6;

inline uint32_t padded_rank(uint32_t rank) { return (rank + 3) / 4 * 4; }

template <uint32_t DP>
size_t delta_shared_bytes(uint32_t tokens, uint32_t rank, bool staged) {
    const size_t padded = padded_rank(rank);
    size_t floats = static_cast<size_t>(tokens) * (kVectors + 1) * DP + tokens * padded + 2 * tokens;
    floats = (floats + 3) / 4 * 4;
    return floats * sizeof(float) + (staged ? padded * DP * sizeof(__nv_bfloat16) : 0);
}

// What one token's projections turn into for one key channel.
struct Prepared {
    float r, w, removal, u, k, v;
};
template <typename T>
__device__ __forceinline__ Prepared prepare(const DeltaArgs<T>& args, const T* row, size_t width, size_t channel,
                                            float logit, float unit_scale) {
    Prepared p;
    p.r = to_float<T>(row[channel]);
    p.k = to_float<T>(row[width + channel]);
    p.v = to_float<T>(row[2 * width + channel]);
    const float removal = sigmoidf(to_float<T>(row[4 * width + channel]) + __bfloat162float(args.removal_bias[channel]));
    p.w = expf(-kDecayScale * sigmoidf(logit + __bfloat162float(args.decay_base[channel])));
    p.u = p.k * unit_scale;
    p.removal = -removal * p.u;
    return p;
}

// ------------------------------------------------------------------------------------------------ general kernel

// LANES threads a column.  Everything a token contributes is prepared for a tile of tokens in shared memory (all in f32)
// and then consumed token by token: per token a thread forms its share of u^T S, LANES threads add theirs up, and the
// same pass over its rows updates S and accumulates r^T S.
// TOKENS: tokens per tile (1 = decode steps).  STAGED: the head's rows of W2 sit in shared memory.
template <typename T, uint32_t DP, uint32_t LANES, uint32_t COLUMNS, uint32_t TOKENS, bool STAGED>
__global__ void __launch_bounds__(LANES * COLUMNS)
delta_rule_kernel(const DeltaArgs<T> args) {
    constexpr uint32_t kThreads = LANES * COLUMNS;
    constexpr uint32_t kWarps = kThreads / 32;
    constexpr uint32_t kRows = DP / LANES;              // key channels per thread, in groups of four
    constexpr uint32_t kGroups = kRows / 4;
    static_assert(kRows % 4 == 0, "four consecutive key channels per access");
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float shared[];
    const uint32_t dim = args.dim;
    const uint32_t padded_z = (args.rank + 3) / 4 * 4;
    float* vectors = shared;                                          // [TOKENS][kVectors][DP]
    float* produced = vectors + TOKENS * kVectors * DP;               // [TOKENS][DP]
    float* z_values = produced + TOKENS * DP;                         // [TOKENS][padded_z], tanh applied
    float* unit_scale = z_values + TOKENS * padded_z;                 // [TOKENS]
    __nv_bfloat162* w2 = reinterpret_cast<__nv_bfloat162*>(
        shared + (TOKENS * ((kVectors + 1) * DP + padded_z + 2) + 3) / 4 * 4);   // [padded_z / 2][DP]

    const uint32_t split = blockIdx.x % args.splits;
    const uint32_t head = blockIdx.x / args.splits % args.heads;
    const uint32_t segment = blockIdx.x / args.splits / args.heads;
    uint32_t begin = segment, end = segment + 1;
    if (args.segments.offsets != nullptr) {
        begin = args.segments.offsets[segment];
        end = args.segments.offsets[segment + 1];
        end = end < args.segments.num_tokens ? end : static_cast<uint32_t>(args.segments.num_tokens);
    }
    const size_t slot = args.segments.slots[segment];
    if (begin >= end || slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t lane = threadIdx.x % LANES;
    const uint32_t column = split * COLUMNS + threadIdx.x / LANES;
    const size_t width = static_cast<size_t>(args.heads) * dim;
    const size_t head_base = static_cast<size_t>(head) * dim;
    float* state_column = reinterpret_cast<float*>(static_cast<unsigned char*>(args.record.base) +
                                                   slot * args.record.stride + args.record.offset) +
                          (head_base + column) * dim;
    const bool live = column < dim;
    const bool vector_state = dim % 4 == 0;

    Pair state[kRows / 2];
#pragma unroll
    for (uint32_t g = 0; g < kGroups; ++g) {
        const uint32_t row = (g * LANES + lane) * 4;
        float4 value = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (live && row < dim) {
            if (vector_state) {
                value = *reinterpret_cast<const float4*>(state_column + row);
            } else {
                value.x = state_column[row];
                if (row + 1 < dim) value.y = state_column[row + 1];
                if (row + 2 < dim) value.z = state_column[row + 2];
                if (row + 3 < dim) value.w = state_column[row + 3];
            }
        }
        state[2 * g] = pair_of(value.x, value.y);
        state[2 * g + 1] = pair_of(value.z, value.w);
    }
    if (STAGED) {
        for (uint32_t item = threadIdx.x; item < padded_z / 2 * DP; item += kThreads) {
            const uint32_t channel = item % DP;
            const uint32_t z = item / DP * 2;
            const __nv_bfloat16 zero = __float2bfloat16_rn(0.0f);
            const __nv_bfloat16* source = args.decay_up + (head_base + channel) * args.rank;
            w2[item] = __halves2bfloat162(channel < dim && z < args.rank ? source[z] : zero,
                                          channel < dim && z + 1 < args.rank ? source[z + 1] : zero);
        }
    }

    const uint32_t warp = threadIdx.x / 32;
    const uint32_t warp_lane = threadIdx.x % 32;
    for (uint32_t tile = begin; tile < end; tile += TOKENS) {
        const uint32_t tokens = end - tile < TOKENS ? end - tile : TOKENS;
        for (uint32_t t = warp; t < tokens; t += kWarps) {
            const T* row = args.projected + static_cast<size_t>(tile + t) * args.pitch;
            float sum = 0.0f;
            for (uint32_t channel = warp_lane; channel < dim; channel += 32) {
                const float value = to_float<T>(row[width + head_base + channel]);
                sum = fmaf(value, value, sum);
            }
            sum = warp_sum(sum);
            if (warp_lane == 0) unit_scale[t] = 1.0f / sqrtf(sum + kUnitEps);
        }
        for (uint32_t item = threadIdx.x; item < tokens * padded_z; item += kThreads) {
            const uint32_t t = item / padded_z;
            const uint32_t z = item % padded_z;
            z_values[item] = z < args.rank ? tanhf(to_float<T>(args.projected[static_cast<size_t>(tile + t) * args.pitch +
                                                                             5 * width + z]))
                                           : 0.0f;
        }
        __syncthreads();
        // one key channel and every (kThreads / DP)-th group of four tokens per thread, so that a W2 value serves four
        constexpr uint32_t kShared = TOKENS < 4 ? TOKENS : 4;
        constexpr uint32_t kStride = kThreads >= DP ? kThreads / DP : 1;
        for (uint32_t channel = threadIdx.x % DP; channel < DP; channel += kThreads >= DP ? DP : kThreads) {
            for (uint32_t t0 = threadIdx.x / DP * kShared; t0 < tokens; t0 += kStride * kShared) {
                float logit[kShared];
#pragma unroll
                for (uint32_t i = 0; i < kShared; ++i) logit[i] = 0.0f;
                if (channel < dim) {
                    if (STAGED) {
                        for (uint32_t z = 0; z < padded_z; z += 4) {
                            const float2 low = __bfloat1622float2(w2[z / 2 * DP + channel]);
                            const float2 high = __bfloat1622float2(w2[(z / 2 + 1) * DP + channel]);
#pragma unroll
                            for (uint32_t i = 0; i < kShared; ++i) {
                                const float4 value =
                                    *reinterpret_cast<const float4*>(z_values + (t0 + i) * padded_z + z);
                                logit[i] = fmaf(low.x, value.x, logit[i]);
                                logit[i] = fmaf(low.y, value.y, logit[i]);
                                logit[i] = fmaf(high.x, value.z, logit[i]);
                                logit[i] = fmaf(high.y, value.w, logit[i]);
                            }
                        }
                    } else {
                        const __nv_bfloat16* source = args.decay_up + (head_base + channel) * args.rank;
                        for (uint32_t z = 0; z < args.rank; ++z) {
                            const float weight = __bfloat162float(source[z]);
#pragma unroll
                            for (uint32_t i = 0; i < kShared; ++i) {
                                logit[i] = fmaf(weight, z_values[(t0 + i) * padded_z + z], logit[i]);
                            }
                        }
                    }
                }
#pragma unroll
                for (uint32_t i = 0; i < kShared; ++i) {
                    const uint32_t t = t0 + i;
                    if (t >= tokens) break;
                    Prepared p = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
                    if (channel < dim) {
                        p = prepare<T>(args, args.projected + static_cast<size_t>(tile + t) * args.pitch, width,
                                       head_base + channel, logit[i], unit_scale[t]);
                    }
                    float* target = vectors + t * kVectors * DP + channel;
                    target[0 * DP] = p.r;
                    target[1 * DP] = p.w;
                    target[2 * DP] = p.removal;
                    target[3 * DP] = p.u;
                    target[4 * DP] = p.k;
                    target[5 * DP] = p.v;
                }
            }
        }
        __syncthreads();

        for (uint32_t t = 0; t < tokens; ++t) {
            const float* token = vectors + t * kVectors * DP;
            const float value = token[5 * DP + (column < DP ? column : 0)];
            Pair dot0 = 0, dot1 = 0;                                // bit pattern of (0.0f, 0.0f)
#pragma unroll
            for (uint32_t g = 0; g < kGroups; ++g) {
                const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(token + 3 * DP + (g * LANES + lane) * 4);
                dot0 = fma_pair(u.x, state[2 * g], dot0);
                dot1 = fma_pair(u.y, state[2 * g + 1], dot1);
            }
            float dot = pair_sum(dot0) + pair_sum(dot1);
#pragma unroll
            for (uint32_t delta = 1; delta < LANES; delta <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, delta);
            const Pair recalled = pair_of(dot, dot);
            const Pair values = pair_of(value, value);
            Pair sum0 = 0, sum1 = 0;
#pragma unroll
            for (uint32_t g = 0; g < kGroups; ++g) {
                const uint32_t row = (g * LANES + lane) * 4;
                const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(token + row);
                const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(token + 1 * DP + row);
                const ulonglong2 removal = *reinterpret_cast<const ulonglong2*>(token + 2 * DP + row);
                const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(token + 4 * DP + row);
                state[2 * g] = fma_pair(k.x, values, fma_pair(removal.x, recalled, mul_pair(w.x, state[2 * g])));
                state[2 * g + 1] =
                    fma_pair(k.y, values, fma_pair(removal.y, recalled, mul_pair(w.y, state[2 * g + 1])));
                sum0 = fma_pair(r.x, state[2 * g], sum0);
                sum1 = fma_pair(r.y, state[2 * g + 1], sum1);
            }
            float result = pair_sum(sum0) + pair_sum(sum1);
#pragma unroll
            for (uint32_t delta = 1; delta < LANES; delta <<= 1) result += __shfl_xor_sync(0xffffffffu, result, delta);
            if (lane == 0 && live) {
                if (args.raw != nullptr) {
                    args.raw[static_cast<size_t>(tile + t) * width + head_base + column] = result;
                } else {
                    produced[t * DP + column] = result;
                }
            }
        }
        __syncthreads();
        if (args.raw == nullptr) {
            for (uint32_t t = warp; t < tokens; t += kWarps) {
                const size_t token = tile + t;
                const T* gate = args.projected + token * args.pitch + 3 * width + head_base;
                float sum = 0.0f;
                for (uint32_t channel = warp_lane; channel < dim; channel += 32) {
                    sum = fmaf(produced[t * DP + channel], produced[t * DP + channel], sum);
                }
                const float scale = inverse_rms(warp_sum(sum), dim, args.eps);
                for (uint32_t channel = warp_lane; channel < dim; channel += 32) {
                    const float normalised =
                        produced[t * DP + channel] * scale * __bfloat162float(args.norm[head_base + channel]);
                    args.out[token * args.out_pitch + head_base + channel] =
                        from_float<T>(normalised * sigmoidf(to_float<T>(gate[channel])));
                }
            }
        }
        // the next tile's first barrier lies behind writes to unit_scale and z_values only, which nobody reads now
    }

#pragma unroll
    for (uint32_t g = 0; g < kGroups; ++g) {
        const uint32_t row = (g * LANES + lane) * 4;
        if (live && row < dim) {
            float4 value;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(value.x), "=f"(value.y) : "l"(state[2 * g]));
            asm("mov.b64 {%0, %1}, %2;" : "=f"(value.z), "=f"(value.w) : "l"(state[2 * g + 1]));
            if (vector_state) {
                *reinterpret_cast<float4*>(state_column + row) = value;
            } else {
                state_column[row] = value.x;
                if (row + 1 < dim) state_column[row + 1] = value.y;
                if (row + 2 < dim) state_column[row + 2] = value.z;
                if (row + 3 < dim) state_column[row + 3] = value.w;
            }
        }
    }
}

// Norm and gate of heads whose columns were spread over several CTAs: one warp per token and head.
template <typename T>
__global__ void __launch_bounds__(128)
delta_output_kernel(const DeltaArgs<T> args) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t item = static_cast<size_t>(blockIdx.x) * 4 + threadIdx.x / 32;
    const size_t token = item / args.heads;
    if (token >= args.segments.num_tokens) {
        return;
    }
    const size_t width = static_cast<size_t>(args.heads) * args.dim;
    const size_t head_base = item % args.heads * args.dim;
    const uint32_t lane = threadIdx.x & 31;
    const float* raw = args.raw + token * width + head_base;
    const T* gate = args.projected + token * args.pitch + 3 * width + head_base;
    float sum = 0.0f;
    for (uint32_t channel = lane; channel < args.dim; channel += 32) sum = fmaf(raw[channel], raw[channel], sum);
    const float scale = inverse_rms(warp_sum(sum), args.dim, args.eps);
    for (uint32_t channel = lane; channel < args.dim; channel += 32) {
        const float normalised = raw[channel] * scale * __bfloat162float(args.norm[head_base + channel]);
        args.out[token * args.out_pitch + head_base + channel] =
            from_float<T>(normalised * sigmoidf(to_float<T>(gate[channel])));
    }
}


// ------------------------------------------------------------------------------------------------ decode kernel

// One token per sequence, one CTA per sequence and head; four threads per value column (for the state) and per key
// channel (for what the token contributes).
template <typename T, uint32_t DP>
__global__ void __launch_bounds__(DP * 4)
delta_decode_kernel(const DeltaArgs<T> args) {
    constexpr uint32_t kThreads = DP * 4;
    constexpr uint32_t kGroups = DP / 16;              // groups of four key channels per thread
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float shared[];
    float* r_values = shared;                          // [DP] each
    float* w_values = r_values + DP;
    float* removal_values = w_values + DP;
    float* u_values = removal_values + DP;
    float* k_values = u_values + DP;
    float* partial = k_values + DP;                    // [warps] twice: |k|^2, |o|^2
    float* z_values = partial + 2 * (kThreads / 32);   // [rank]
    const uint32_t dim = args.dim;
    const uint32_t head = blockIdx.x % args.heads;
    const size_t token = blockIdx.x / args.heads;
    const size_t slot = args.segments.slots[token];
    if (slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t channel = threadIdx.x / 4;          // value column and key channel
    const uint32_t lane = threadIdx.x % 4;
    const bool live = channel < dim;
    const size_t width = static_cast<size_t>(args.heads) * dim;
    const size_t head_base = static_cast<size_t>(head) * dim;
    float* state_column = reinterpret_cast<float*>(static_cast<unsigned char*>(args.record.base) +
                                                   slot * args.record.stride + args.record.offset) +
                          (head_base + channel) * dim;
    const bool vector_state = dim % 4 == 0;
    Pair state[kGroups * 2];
#pragma unroll
    for (uint32_t g = 0; g < kGroups; ++g) {
        const uint32_t row = (g * 4 + lane) * 4;
        float4 value = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (live && row < dim) {
            if (vector_state) {
                value = __ldcs(reinterpret_cast<const float4*>(state_column + row));
            } else {
                value.x = state_column[row];
                if (row + 1 < dim) value.y = state_column[row + 1];
                if (row + 2 < dim) value.z = state_column[row + 2];
                if (row + 3 < dim) value.w = state_column[row + 3];
            }
        }
        state[2 * g] = pair_of(value.x, value.y);
        state[2 * g + 1] = pair_of(value.z, value.w);
    }
    const T* row = args.projected + token * args.pitch;
    float r = 0.0f, k = 0.0f, v = 0.0f, gate = 0.0f, removal = 0.0f, base = 0.0f, weight = 0.0f;
    if (live) {
        const size_t index = head_base + channel;
        r = to_float<T>(row[index]);
        k = to_float<T>(row[width + index]);
        v = to_float<T>(row[2 * width + index]);
        gate = to_float<T>(row[3 * width + index]);
        removal = to_float<T>(row[4 * width + index]) + __bfloat162float(args.removal_bias[index]);
        base = __bfloat162float(args.decay_base[index]);
        weight = __bfloat162float(args.norm[index]);
    }
    for (uint32_t z = threadIdx.x; z < args.rank; z += kThreads) z_values[z] = tanhf(to_float<T>(row[5 * width + z]));
    // this thread's quarter of the channel's row of W2, its first 16 values in registers before the barrier
    const uint32_t part = (args.rank / 4 + 7) / 8 * 8;
    const uint32_t from = min(lane * part, args.rank);
    const uint32_t to = lane == 3 ? args.rank : min(from + part, args.rank);
    const __nv_bfloat16* decay_row = args.decay_up + (head_base + (live ? channel : 0)) * args.rank;
    const bool vector_rank = args.rank % 8 == 0;
    uint4 early[2] = {};
    if (live && vector_rank) {
#pragma unroll
        for (uint32_t i = 0; i < 2; ++i) {
            if (from + 8 * i < to) early[i] = *reinterpret_cast<const uint4*>(decay_row + from + 8 * i);
        }
    }
    // every channel is held by four threads
    const float k_squares = warp_sum(lane == 0 ? k * k : 0.0f);
    const uint32_t warp = threadIdx.x / 32;
    if (threadIdx.x % 32 == 0) partial[warp] = k_squares;
    __syncthreads();
    float logit = 0.0f;
    if (live) {
        if (vector_rank) {
            for (uint32_t z = from; z < to; z += 8) {
                const uint4 raw = z < from + 16 ? (z == from ? early[0] : early[1])
                                                : *reinterpret_cast<const uint4*>(decay_row + z);
                const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) {
                    const float2 both = __bfloat1622float2(pairs[i]);
                    logit = fmaf(both.x, z_values[z + 2 * i], logit);
                    logit = fmaf(both.y, z_values[z + 2 * i + 1], logit);
                }
            }
        } else {
            for (uint32_t z = from; z < to; ++z) logit = fmaf(__bfloat162float(decay_row[z]), z_values[z], logit);
        }
    }
    logit += __shfl_xor_sync(0xffffffffu, logit, 1);
    logit += __shfl_xor_sync(0xffffffffu, logit, 2);
    float squares = 0.0f;
#pragma unroll
    for (uint32_t w = 0; w < kThreads / 32; ++w) squares += partial[w];
    const float u = k / sqrtf(squares + kUnitEps);
    if (lane == 0) {
        w_values[channel] = expf(-kDecayScale * sigmoidf(logit + base));
    } else if (lane == 1) {
        removal_values[channel] = -sigmoidf(removal) * u;
    } else if (lane == 2) {
        u_values[channel] = u;
        r_values[channel] = r;
    } else {
        k_values[channel] = k;
    }
    __syncthreads();
    Pair dot0 = 0, dot1 = 0;                           // bit pattern of (0.0f, 0.0f)
#pragma unroll
    for (uint32_t g = 0; g < kGroups; ++g) {
        const ulonglong2 unit = *reinterpret_cast<const ulonglong2*>(u_values + (g * 4 + lane) * 4);
        dot0 = fma_pair(unit.x, state[2 * g], dot0);
        dot1 = fma_pair(unit.y, state[2 * g + 1], dot1);
    }
    float dot = pair_sum(dot0) + pair_sum(dot1);
    dot += __shfl_xor_sync(0xffffffffu, dot, 1);
    dot += __shfl_xor_sync(0xffffffffu, dot, 2);
    const Pair recalled = pair_of(dot, dot);
    const Pair values = pair_of(v, v);
    Pair sum0 = 0, sum1 = 0;
#pragma unroll
    for (uint32_t g = 0; g < kGroups; ++g) {
        const uint32_t at = (g * 4 + lane) * 4;
        const ulonglong2 rr = *reinterpret_cast<const ulonglong2*>(r_values + at);
        const ulonglong2 ww = *reinterpret_cast<const ulonglong2*>(w_values + at);
        const ulonglong2 aa = *reinterpret_cast<const ulonglong2*>(removal_values + at);
        const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(k_values + at);
        state[2 * g] = fma_pair(kk.x, values, fma_pair(aa.x, recalled, mul_pair(ww.x, state[2 * g])));
        state[2 * g + 1] = fma_pair(kk.y, values, fma_pair(aa.y, recalled, mul_pair(ww.y, state[2 * g + 1])));
        sum0 = fma_pair(rr.x, state[2 * g], sum0);
        sum1 = fma_pair(rr.y, state[2 * g + 1], sum1);
        if (live && at < dim) {
            const float4 value = {low_of(state[2 * g]), high_of(state[2 * g]), low_of(state[2 * g + 1]),
                                  high_of(state[2 * g + 1])};
            if (vector_state) {
                __stcs(reinterpret_cast<float4*>(state_column + at), value);
            } else {
                state_column[at] = value.x;
                if (at + 1 < dim) state_column[at + 1] = value.y;
                if (at + 2 < dim) state_column[at + 2] = value.z;
                if (at + 3 < dim) state_column[at + 3] = value.w;
            }
        }
    }
    float result = pair_sum(sum0) + pair_sum(sum1);
    result += __shfl_xor_sync(0xffffffffu, result, 1);
    result += __shfl_xor_sync(0xffffffffu, result, 2);
    const float o_squares = warp_sum(lane == 0 && live ? result * result : 0.0f);
    if (threadIdx.x % 32 == 0) partial[kThreads / 32 + warp] = o_squares;
    __syncthreads();
    squares = 0.0f;
#pragma unroll
    for (uint32_t w = 0; w < kThreads / 32; ++w) squares += partial[kThreads / 32 + w];
    if (lane == 0 && live) {
        args.out[token * args.out_pitch + head_base + channel] =
            from_float<T>(result * inverse_rms(squares, dim, args.eps) * weight * sigmoidf(gate));
    }
}

// ------------------------------------------------------------------------------------------------ prompt kernel

// 16-byte copy global -> shared without registers
__device__ __forceinline__ void copy_async_16(void* target, const void* source) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(target)), "l"(source) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int PENDING>
__device__ __forceinline__ void copy_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(PENDING) : "memory");
}
__device__ __forceinline__ void named_barrier(uint32_t id, uint32_t threads) {
    asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory");
}

// The prompt kernel's decays and rates: the fast f32 exponential and division, a few units in the last place from the
// correctly rounded ones.
__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float fast_tanh(float z) { return 1.0f - __fdividef(2.0f, 1.0f + __expf(2.0f * z)); }

constexpr uint32_t kPromptTokens = 16;       // tokens per tile = rows of one MMA tile
constexpr uint32_t kRawStages = 4;           // being finished, in the recurrence, being prepared, arriving
constexpr uint32_t kPromptMaxRank = 256;

template <uint32_t DP>
struct PromptLayout {
    uint32_t rank_pad;        // multiple of 32
    uint32_t z_stride;        // bf16 elements between rows of z / W2 in shared memory: 16-byte rows, no bank conflicts
    uint32_t raw_row;         // bf16 elements per token: r | k | v | g | a (DP each) | z
    size_t raw, vectors, produced, tanh_parts, w2, constants, scale, total;
    __host__ __device__ explicit PromptLayout(uint32_t rank) {
        rank_pad = (rank + 31) / 32 * 32;
        z_stride = rank_pad + 8;
        raw_row = 5 * DP + rank_pad;
        size_t at = 0;
        raw = at;
        at += static_cast<size_t>(kRawStages) * kPromptTokens * raw_row * 2;
        vectors = at;                                             // [2][tokens][2][DP] f32: w, removal / |k|^2
        at += 2 * kPromptTokens * 2 * DP * 4;
        produced = at;                                            // [2][tokens][DP] f32
        at += 2 * kPromptTokens * DP * 4;
        tanh_parts = at;                                          // [2][tokens][z_stride] bf16: high and low parts
        at += 2 * kPromptTokens * z_stride * 2;
        w2 = at;                                                  // [DP][z_stride] bf16
        at += static_cast<size_t>(DP) * z_stride * 2;
        constants = at;                                           // [3][DP] f32: w0, removal bias, norm weight
        at += 3 * DP * 4;
        scale = at;                                               // [2][tokens] f32: 1 / |k|^2
        at += 2 * kPromptTokens * 4;
        total = at;
    }
};

// Where key channel `row` of a prepared f32 vector lies: the 4-channel groups of the eight threads that share a column
// are interleaved, so that their 16-byte reads are consecutive.
template <uint32_t DP>
__device__ __forceinline__ uint32_t interleaved(uint32_t row) {
    constexpr uint32_t kRows = DP / 8;
    return row % kRows / 4 * 32 + row / kRows * 4 + row % 4;
}

// Eight threads per group of COLUMNS value columns run the recurrence, DP / 8 consecutive key channels each; HELPERS
// threads prepare and finish.
template <uint32_t DP, uint32_t COLUMNS, uint32_t HELPERS>
__global__ void __launch_bounds__(DP / COLUMNS * 8 + HELPERS)
delta_prompt_kernel(const DeltaArgs<__nv_bfloat16> args) {
    constexpr uint32_t kRows = DP / 8;
    constexpr uint32_t kScanThreads = DP / COLUMNS * 8;
    constexpr uint32_t kHelpers = HELPERS;
    constexpr uint32_t kHelperWarps = kHelpers / 32;
    constexpr uint32_t kTokensPerHelper = kPromptTokens / kHelperWarps;   // tokens per helper warp
    static_assert(COLUMNS == 2 || COLUMNS == 4, "columns per thread");
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char prompt_shared[];
    const PromptLayout<DP> layout(args.rank);
    const uint32_t dim = args.dim;
    const uint32_t head = blockIdx.x % args.heads;
    const uint32_t segment = blockIdx.x / args.heads;
    const uint32_t begin = args.segments.offsets[segment];
    uint32_t end = args.segments.offsets[segment + 1];
    end = end < args.segments.num_tokens ? end : static_cast<uint32_t>(args.segments.num_tokens);
    const size_t slot = args.segments.slots[segment];
    if (begin >= end || slot >= args.segments.num_request_slots) {
        return;
    }
    const uint32_t tiles = (end - begin + kPromptTokens - 1) / kPromptTokens;
    const size_t width = static_cast<size_t>(args.heads) * dim;
    const size_t head_base = static_cast<size_t>(head) * dim;
    auto* raw = reinterpret_cast<__nv_bfloat16*>(prompt_shared + layout.raw);
    auto* vectors = reinterpret_cast<float*>(prompt_shared + layout.vectors);
    auto* produced = reinterpret_cast<float*>(prompt_shared + layout.produced);
    auto* tanh_parts = reinterpret_cast<__nv_bfloat16*>(prompt_shared + layout.tanh_parts);
    auto* w2 = reinterpret_cast<__nv_bfloat16*>(prompt_shared + layout.w2);
    auto* constants = reinterpret_cast<float*>(prompt_shared + layout.constants);
    auto* scale = reinterpret_cast<float*>(prompt_shared + layout.scale);
    float* state_base = reinterpret_cast<float*>(static_cast<unsigned char*>(args.record.base) +
                                                 slot * args.record.stride + args.record.offset) +
                        head_base * dim;

    // padding channels and tokens that never arrive stay zero
    for (uint32_t item = threadIdx.x; item < kRawStages * kPromptTokens * layout.raw_row / 8;
         item += kScanThreads + kHelpers) {
        reinterpret_cast<uint4*>(raw)[item] = make_uint4(0, 0, 0, 0);
    }
    for (uint32_t item = threadIdx.x; item < DP * layout.z_stride; item += kScanThreads + kHelpers) {
        const uint32_t channel = item / layout.z_stride;
        const uint32_t z = item % layout.z_stride;
        w2[item] = channel < dim && z < args.rank ? args.decay_up[(head_base + channel) * args.rank + z]
                                                  : __float2bfloat16_rn(0.0f);
    }
    for (uint32_t channel = threadIdx.x; channel < DP; channel += kScanThreads + kHelpers) {
        const bool live = channel < dim;
        constants[channel] = live ? __bfloat162float(args.decay_base[head_base + channel]) : 0.0f;
        constants[DP + channel] = live ? __bfloat162float(args.removal_bias[head_base + channel]) : 0.0f;
        constants[2 * DP + channel] = live ? __bfloat162float(args.norm[head_base + channel]) : 0.0f;
    }
    __syncthreads();

    const bool scanner = threadIdx.x < kScanThreads;
    const uint32_t helper = threadIdx.x - kScanThreads;
    const uint32_t helper_warp = helper / 32;
    const uint32_t warp_lane = threadIdx.x % 32;

    // the 16-byte pieces of a token's row that this lane copies: offsets in the row and in the stage
    constexpr uint32_t kPieces = (5 * DP / 8 + kPromptMaxRank / 8 + 31) / 32;
    const uint32_t per_vector = dim / 8;
    const uint32_t pieces = 5 * per_vector + (args.rank + 7) / 8;
    auto piece_offsets = [&](uint32_t piece, uint32_t& source, uint32_t& target) {
        if (piece < 5 * per_vector) {
            const uint32_t vector = piece / per_vector;
            const uint32_t chunk = piece - vector * per_vector;
            source = static_cast<uint32_t>(vector * width + head_base) + chunk * 8;
            target = vector * DP + chunk * 8;
        } else {
            const uint32_t chunk = piece - 5 * per_vector;
            source = static_cast<uint32_t>(5 * width) + chunk * 8;
            target = 5 * DP + chunk * 8;
        }
    };
    uint32_t first_source = 0, first_target = 0, second_source = 0, second_target = 0;
    piece_offsets(warp_lane, first_source, first_target);
    piece_offsets(warp_lane + 32, second_source, second_target);
    auto load_tile = [&](uint32_t tile) {             // helpers only; always one group per call
        const uint32_t first = begin + tile * kPromptTokens;
#pragma unroll
        for (uint32_t i = 0; i < kTokensPerHelper; ++i) {
            const uint32_t t = helper_warp * kTokensPerHelper + i;
            if (tile < tiles && first + t < end) {
                const __nv_bfloat16* source = args.projected + static_cast<size_t>(first + t) * args.pitch;
                __nv_bfloat16* target = raw + (tile % kRawStages * kPromptTokens + t) * layout.raw_row;
                if (warp_lane < pieces) copy_async_16(target + first_target, source + first_source);
                if (warp_lane + 32 < pieces) copy_async_16(target + second_target, source + second_source);
                for (uint32_t piece = warp_lane + 64; kPieces > 2 && piece < pieces; piece += 32) {
                    uint32_t from, to;
                    piece_offsets(piece, from, to);
                    copy_async_16(target + to, source + from);
                }
            }
        }
        copy_async_commit();
    };

    auto prepare_tile = [&](uint32_t tile) {          // helpers only; the tile's copies have arrived for all of them
        const __nv_bfloat16* stage = raw + tile % kRawStages * kPromptTokens * layout.raw_row;
        float* target = vectors + tile % 2 * kPromptTokens * 2 * DP;
        float* unit = scale + tile % 2 * kPromptTokens;
        float squares[kTokensPerHelper];
#pragma unroll
        for (uint32_t i = 0; i < kTokensPerHelper; ++i) {
            const __nv_bfloat16* row = stage + (helper_warp * kTokensPerHelper + i) * layout.raw_row;
            squares[i] = 0.0f;
#pragma unroll
            for (uint32_t part = 0; part < DP / 64; ++part) {
                const float2 both =
                    __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row + DP + part * 64 + warp_lane * 2));
                squares[i] = fmaf(both.x, both.x, fmaf(both.y, both.y, squares[i]));
            }
        }
        for (uint32_t z = warp_lane * 2; z < layout.rank_pad; z += 64) {
#pragma unroll
            for (uint32_t i = 0; i < kTokensPerHelper; ++i) {
                const uint32_t t = helper_warp * kTokensPerHelper + i;
                const float2 both = __bfloat1622float2(
                    *reinterpret_cast<const __nv_bfloat162*>(stage + t * layout.raw_row + 5 * DP + z));
                // columns between rank and the end of its last copy belong to nobody
                const float a = z < args.rank ? fast_tanh(both.x) : 0.0f;
                const float b = z + 1 < args.rank ? fast_tanh(both.y) : 0.0f;
                const __nv_bfloat162 high = __floats2bfloat162_rn(a, b);
                const float2 rounded = __bfloat1622float2(high);
                *reinterpret_cast<__nv_bfloat162*>(tanh_parts + t * layout.z_stride + z) = high;
                *reinterpret_cast<__nv_bfloat162*>(tanh_parts + (kPromptTokens + t) * layout.z_stride + z) =
                    __floats2bfloat162_rn(a - rounded.x, b - rounded.y);
            }
        }
#pragma unroll
        for (uint32_t i = 0; i < kTokensPerHelper; ++i) squares[i] = warp_sum(squares[i]);
        if (warp_lane == 0) {
#pragma unroll
            for (uint32_t i = 0; i < kTokensPerHelper; ++i) {
                unit[helper_warp * kTokensPerHelper + i] = 1.0f / (squares[i] + kUnitEps);
            }
        }
        named_barrier(1, kHelpers);
        // decay logits of 16 tokens x 8 channels at a time: tanh(z) W2^T with tanh(z) as a sum of two bf16 values
#pragma unroll
        for (uint32_t n = 0; n < DP / 8 / kHelperWarps; ++n) {
            const uint32_t channel0 = (n * kHelperWarps + helper_warp) * 8;
            float logits[4] = {};
            const uint32_t z_row = warp_lane % 16, z_part = warp_lane / 16 * 8;
            for (uint32_t step = 0; step < layout.rank_pad; step += 32) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(smem_u32(w2 + (channel0 + warp_lane % 8) * layout.z_stride + step + warp_lane / 8 * 8), b0, b1,
                            b2, b3);
#pragma unroll
                for (uint32_t part = 0; part < 2; ++part) {
                    uint32_t high[4], low[4];
                    const __nv_bfloat16* source = tanh_parts + z_row * layout.z_stride + step + part * 16 + z_part;
                    ldmatrix_x4(smem_u32(source), high[0], high[1], high[2], high[3]);
                    ldmatrix_x4(smem_u32(source + kPromptTokens * layout.z_stride), low[0], low[1], low[2], low[3]);
                    mma_bf16_16816(logits, high[0], high[1], high[2], high[3], part ? b2 : b0, part ? b3 : b1);
                    mma_bf16_16816(logits, low[0], low[1], low[2], low[3], part ? b2 : b0, part ? b3 : b1);
                }
            }
            const uint32_t channel = channel0 + warp_lane % 4 * 2;
            const uint32_t t0 = warp_lane / 4;
            const float2 base = *reinterpret_cast<const float2*>(constants + channel);
            const float2 bias = *reinterpret_cast<const float2*>(constants + DP + channel);
            float2 rate[2];
            float factor[2];
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                rate[half] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(
                    stage + (t0 + half * 8) * layout.raw_row + 4 * DP + channel));
                factor[half] = unit[t0 + half * 8];
            }
            float2 w[2], removal[2];
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                w[half].x = __expf(-kDecayScale * fast_sigmoid(logits[2 * half] + base.x));
                w[half].y = __expf(-kDecayScale * fast_sigmoid(logits[2 * half + 1] + base.y));
                // -(a * u) (u^T S) = -(a / |k|^2) * k * (k^T S): the recurrence multiplies by k anyway
                removal[half].x = -fast_sigmoid(rate[half].x + bias.x) * factor[half];
                removal[half].y = -fast_sigmoid(rate[half].y + bias.y) * factor[half];
            }
            const uint32_t at = interleaved<DP>(channel);
#pragma unroll
            for (uint32_t half = 0; half < 2; ++half) {
                float* row = target + (t0 + half * 8) * 2 * DP + at;
                *reinterpret_cast<float2*>(row) = w[half];
                *reinterpret_cast<float2*>(row + DP) = removal[half];
            }
        }
    };

    auto finish_tile = [&](uint32_t tile) {           // helpers only
        const __nv_bfloat16* stage = raw + tile % kRawStages * kPromptTokens * layout.raw_row;
        const float* source = produced + tile % 2 * kPromptTokens * DP;
        const uint32_t first = begin + tile * kPromptTokens;
        float2 value[kTokensPerHelper][DP / 64], gate[kTokensPerHelper][DP / 64];
        float squares[kTokensPerHelper];
#pragma unroll
        for (uint32_t i = 0; i < kTokensPerHelper; ++i) {
            const uint32_t t = helper_warp * kTokensPerHelper + i;
            squares[i] = 0.0f;
#pragma unroll
            for (uint32_t part = 0; part < DP / 64; ++part) {
                const uint32_t channel = part * 64 + warp_lane * 2;
                value[i][part] = *reinterpret_cast<const float2*>(source + t * DP + channel);
                gate[i][part] = __bfloat1622float2(
                    *reinterpret_cast<const __nv_bfloat162*>(stage + t * layout.raw_row + 3 * DP + channel));
                squares[i] = fmaf(value[i][part].x, value[i][part].x,
                                  fmaf(value[i][part].y, value[i][part].y, squares[i]));
            }
        }
#pragma unroll
        for (uint32_t i = 0; i < kTokensPerHelper; ++i) squares[i] = warp_sum(squares[i]);
#pragma unroll
        for (uint32_t i = 0; i < kTokensPerHelper; ++i) {
            const uint32_t t = helper_warp * kTokensPerHelper + i;
            const float factor = rsqrtf(squares[i] / static_cast<float>(dim) + args.eps);
#pragma unroll
            for (uint32_t part = 0; part < DP / 64; ++part) {
                const uint32_t channel = part * 64 + warp_lane * 2;
                const float2 weight = *reinterpret_cast<const float2*>(constants + 2 * DP + channel);
                const uint32_t both =
                    pack_bf16x2(value[i][part].x * factor * weight.x * fast_sigmoid(gate[i][part].x),
                                value[i][part].y * factor * weight.y * fast_sigmoid(gate[i][part].y));
                if (channel < dim && first + t < end) {
                    *reinterpret_cast<uint32_t*>(args.out + static_cast<size_t>(first + t) * args.out_pitch + head_base +
                                                 channel) = both;
                }
            }
        }
    };

    // ---- the state: columns COLUMNS * group .. + COLUMNS - 1, key channels lane * kRows .. + kRows - 1
    const uint32_t lane = threadIdx.x % 8;
    const uint32_t column0 = threadIdx.x / 8 * COLUMNS;
    Pair state[COLUMNS][kRows / 2];
    if (scanner) {
#pragma unroll
        for (uint32_t c = 0; c < COLUMNS; ++c) {
#pragma unroll
            for (uint32_t g = 0; g < kRows / 4; ++g) {
                const uint32_t row = lane * kRows + g * 4;
                float4 value = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (column0 + c < dim && row < dim) {          // dim is a multiple of 8
                    value = *reinterpret_cast<const float4*>(state_base + static_cast<size_t>(column0 + c) * dim + row);
                }
                state[c][2 * g] = pair_of(value.x, value.y);
                state[c][2 * g + 1] = pair_of(value.z, value.w);
            }
        }
    } else {
        load_tile(0);
        load_tile(1);
        copy_async_wait<1>();
        named_barrier(1, kHelpers);
        prepare_tile(0);
    }
    __syncthreads();

    for (uint32_t tile = 0; tile < tiles; ++tile) {
        if (scanner) {
            const uint32_t tokens = min(kPromptTokens, end - begin - tile * kPromptTokens);
            const __nv_bfloat16* stage = raw + tile % kRawStages * kPromptTokens * layout.raw_row;
            const float* prepared = vectors + tile % 2 * kPromptTokens * 2 * DP;
            float* target = produced + tile % 2 * kPromptTokens * DP;
            // software pipeline: a token's vectors are read one token ahead, and the sums over the eight threads of a
            // column group run for o of the previous token beside those for u^T S of this one
            struct Vectors {
                uint4 k[kRows / 8], r[kRows / 8];
                uint32_t v[COLUMNS / 2];
            };
            auto read = [&](uint32_t t) {
                Vectors out;
                const __nv_bfloat16* row = stage + t * layout.raw_row;
#pragma unroll
                for (uint32_t part = 0; part < kRows / 8; ++part) {
                    out.k[part] = *reinterpret_cast<const uint4*>(row + DP + lane * kRows + part * 8);
                    out.r[part] = *reinterpret_cast<const uint4*>(row + lane * kRows + part * 8);
                }
                if constexpr (COLUMNS == 4) {
                    const uint2 both = *reinterpret_cast<const uint2*>(row + 2 * DP + column0);
                    out.v[0] = both.x;
                    out.v[1] = both.y;
                } else {
                    out.v[0] = *reinterpret_cast<const uint32_t*>(row + 2 * DP + column0);
                }
                return out;
            };
            Vectors next = read(0);
            float result[COLUMNS] = {};
            const bool upper1 = lane & 1, upper2 = lane & 2;
            float* slot_of_lane = target + column0 + (COLUMNS == 4 ? (lane & 1) * 2 + (lane >> 1 & 1) : (lane & 1));
            // column sums of o over the eight threads, each pair of threads keeping half of the columns
            auto total_of = [&](const float (&share)[COLUMNS]) {
                if constexpr (COLUMNS == 2) {
                    float total = (upper1 ? share[1] : share[0]) +
                                  __shfl_xor_sync(0xffffffffu, upper1 ? share[0] : share[1], 1);
                    total += __shfl_xor_sync(0xffffffffu, total, 2);
                    return total + __shfl_xor_sync(0xffffffffu, total, 4);
                } else {
                const float keep0 = upper1 ? share[2] : share[0], keep1 = upper1 ? share[3] : share[1];
                const float give0 = upper1 ? share[0] : share[2], give1 = upper1 ? share[1] : share[3];
                const float half0 = keep0 + __shfl_xor_sync(0xffffffffu, give0, 1);
                const float half1 = keep1 + __shfl_xor_sync(0xffffffffu, give1, 1);
                float total = (upper2 ? half1 : half0) + __shfl_xor_sync(0xffffffffu, upper2 ? half0 : half1, 2);
                return total + __shfl_xor_sync(0xffffffffu, total, 4);
                }
            };
            for (uint32_t t = 0; t < tokens; ++t) {
                const Vectors now = next;
                next = read(t + 1 < tokens ? t + 1 : t);
                Pair w[kRows / 2], removal[kRows / 2];
#pragma unroll
                for (uint32_t g = 0; g < kRows / 4; ++g) {
                    const float* token = prepared + t * 2 * DP + g * 32 + lane * 4;
                    const ulonglong2 w_pair = *reinterpret_cast<const ulonglong2*>(token);
                    const ulonglong2 removal_pair = *reinterpret_cast<const ulonglong2*>(token + DP);
                    w[2 * g] = w_pair.x;
                    w[2 * g + 1] = w_pair.y;
                    removal[2 * g] = removal_pair.x;
                    removal[2 * g + 1] = removal_pair.y;
                }
                Pair k[kRows / 2], r[kRows / 2];
#pragma unroll
                for (uint32_t part = 0; part < kRows / 8; ++part) {
                    const uint32_t k_words[4] = {now.k[part].x, now.k[part].y, now.k[part].z, now.k[part].w};
                    const uint32_t r_words[4] = {now.r[part].x, now.r[part].y, now.r[part].z, now.r[part].w};
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {       // bf16 -> f32 is a shift
                        k[part * 4 + i] = pair_of(__uint_as_float(k_words[i] << 16),
                                                  __uint_as_float(k_words[i] & 0xffff0000u));
                        r[part * 4 + i] = pair_of(__uint_as_float(r_words[i] << 16),
                                                  __uint_as_float(r_words[i] & 0xffff0000u));
                    }
                }
                float v[COLUMNS], dot[COLUMNS];
#pragma unroll
                for (uint32_t c = 0; c < COLUMNS; c += 2) {
                    v[c] = __uint_as_float(now.v[c / 2] << 16);
                    v[c + 1] = __uint_as_float(now.v[c / 2] & 0xffff0000u);
                }
#pragma unroll
                for (uint32_t c = 0; c < COLUMNS; ++c) {
                    Pair even = mul_pair(k[0], state[c][0]);
                    Pair odd = mul_pair(k[1], state[c][1]);
#pragma unroll
                    for (uint32_t i = 2; i < kRows / 2; i += 2) {
                        even = fma_pair(k[i], state[c][i], even);
                        odd = fma_pair(k[i + 1], state[c][i + 1], odd);
                    }
                    dot[c] = pair_sum(add_pair(even, odd));
                }
#pragma unroll
                for (uint32_t delta = 1; delta < 8; delta <<= 1) {
#pragma unroll
                    for (uint32_t c = 0; c < COLUMNS; ++c) dot[c] += __shfl_xor_sync(0xffffffffu, dot[c], delta);
                }
                const float before = total_of(result);
                Pair sums[COLUMNS];
                // w S does not depend on the sums above
#pragma unroll
                for (uint32_t c = 0; c < COLUMNS; ++c) {
#pragma unroll
                    for (uint32_t i = 0; i < kRows / 2; ++i) state[c][i] = mul_pair(w[i], state[c][i]);
                }
#pragma unroll
                for (uint32_t c = 0; c < COLUMNS; ++c) {
                    const Pair recalled = pair_of(dot[c], dot[c]);
                    const Pair values = pair_of(v[c], v[c]);
                    Pair even = 0, odd = 0;
#pragma unroll
                    for (uint32_t i = 0; i < kRows / 2; i += 2) {      // w S + k (v - (a / |k|^2) (k^T S))
                        state[c][i] = fma_pair(k[i], fma_pair(removal[i], recalled, values), state[c][i]);
                        state[c][i + 1] = fma_pair(k[i + 1], fma_pair(removal[i + 1], recalled, values), state[c][i + 1]);
                        even = fma_pair(r[i], state[c][i], even);
                        odd = fma_pair(r[i + 1], state[c][i + 1], odd);
                    }
                    sums[c] = add_pair(even, odd);
                }
#pragma unroll
                for (uint32_t c = 0; c < COLUMNS; ++c) result[c] = pair_sum(sums[c]);
                if (lane < COLUMNS && t > 0) slot_of_lane[(t - 1) * DP] = before;
            }
            const float last = total_of(result);
            if (lane < COLUMNS) slot_of_lane[(tokens - 1) * DP] = last;
        } else {
            load_tile(tile + 2);
            if (tile > 0) finish_tile(tile - 1);
            copy_async_wait<1>();                     // tile + 1 has arrived for this thread ...
            named_barrier(1, kHelpers);               // ... and for all helpers
            if (tile + 1 < tiles) prepare_tile(tile + 1);
        }
        __syncthreads();
    }
    if (scanner) {
#pragma unroll
        for (uint32_t c = 0; c < COLUMNS; ++c) {
#pragma unroll
            for (uint32_t g = 0; g < kRows / 4; ++g) {
                const uint32_t row = lane * kRows + g * 4;
                if (column0 + c < dim && row < dim) {
                    *reinterpret_cast<float4*>(state_base + static_cast<size_t>(column0 + c) * dim + row) =
                        make_float4(low_of(state[c][2 * g]), high_of(state[c][2 * g]), low_of(state[c][2 * g + 1]),
                                    high_of(state[c][2 * g + 1]));
                }
            }
        }
    } else {
        finish_tile(tiles - 1);
    }
}


// ------------------------------------------------------------------------------------------------ chunk kernel
//
// The recurrence over a tile of 16 tokens as matrix products.  With P_t the product of the decays of the tile's tokens
// up to t, S_t = diag(P_t) Q_t, and
//     U_t = u_t P_(t-1),   R_t = r_t P_t,   K_t = k_t / P_t,   B_t = -(a_t u_t) / P_t          (per key channel)
// the update is Q_t = Q_(t-1) + B_t (U_t^T Q_(t-1)) + K_t v_t^T, so with Y_t = Q_(t-1)^T U_t
//     (I - tril(U B^T, -1)) Y = U Q_0 + tril(U K^T, -1) V
//     O = R Q_0 + tril(R B^T) Y + tril(R K^T) V,      Q_16 = Q_0 + B^T Y + K^T V.
// A decay is at least exp(-exp(-1/2)), so 1 / P_t stays below 17000 and every product keeps its relative accuracy.
// The products run on the tensor cores in TF32 with both operands split into two parts (three products), which
// leaves errors of the size of f32 rounding; v is bf16 and needs no second part.
//
// A CTA owns one head of one segment and works as a pipeline over tiles, one barrier per step; in step i
//     copies       load tile i + 4, finish tile i - 1 (norm, gate, output), tanh(z) and |k| of tile i + 3
//     elements     decay logits (a small product), prefix sums over the tokens, U, R, K, B of tile i + 2
//     triangles    the four masked 16 x 16 products and the inverse of the unit triangle of tile i + 1
//     matrices     everything that meets the state, for tile i; a warp owns 16 value columns and their state

constexpr uint32_t kChunkDim = 64;                // padded head size
constexpr uint32_t kChunkStages = 6;              // tiles i - 1 .. i + 4 of raw projections
constexpr uint32_t kRowStride = kChunkDim + 4;    // U, R: A operands, [token][channel]
constexpr uint32_t kTransposedStride = kChunkDim + 8;   // K, B: also read as [channel][token]
constexpr uint32_t kProducedStride = kChunkDim + 8;
constexpr uint32_t kTriangleStride = 20;
constexpr uint32_t kColumnStride = 24;            // a warp's 16 columns: state, right-hand side, Y

struct ChunkLayout {
    uint32_t rank_pad, z_stride, raw_row;
    size_t raw, operands, triangles, decay_end, tanh_parts, w2, constants, scale, produced, state, columns, total;
    __host__ __device__ explicit ChunkLayout(uint32_t rank) {
        rank_pad = (rank + 31) / 32 * 32;
        z_stride = rank_pad + 8;
        raw_row = 5 * kChunkDim + rank_pad;
        size_t at = 0;
        raw = at;
        at += static_cast<size_t>(kChunkStages) * kPromptTokens * raw_row * 2;
        operands = at;                            // [3][U | R | K | B]
        at += 3 * kPromptTokens * 2 * (kRowStride + kTransposedStride) * 4;
        triangles = at;                           // [2][inverse | U K^T | R B^T | R K^T | U B^T]
        at += 2 * 5 * kPromptTokens * kTriangleStride * 4;
        decay_end = at;                           // [3][channel]: P of the tile's last token
        at += 3 * kChunkDim * 4;
        tanh_parts = at;                          // [2][high | low][token][z_stride]
        at += 2 * 2 * kPromptTokens * z_stride * 2;
        w2 = at;
        at += kChunkDim * z_stride * 2;
        constants = at;                           // w0, removal bias, norm weight
        at += 3 * kChunkDim * 4;
        scale = at;                               // [2][token]: 1 / |k|
        at += 2 * kPromptTokens * 4;
        produced = at;                            // [2][token][kProducedStride]
        at += 2 * kPromptTokens * kProducedStride * 4;
        state = at;                               // [warp][channel][kColumnStride]
        at += 4 * kChunkDim * kColumnStride * 4;
        columns = at;                             // [warp][token][kColumnStride]
        at += 4 * kPromptTokens * kColumnStride * 4;
        total = at;
    }
};

// D(16x8) += A(16x8, tf32) * B(8x8, tf32), f32 accumulation
__device__ __forceinline__ void mma_tf32(float (&d)[4], const float (&a)[4], const float (&b)[2]) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
        "{%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])),
          "r"(__float_as_uint(b[0])), "r"(__float_as_uint(b[1])));
}

// An operand fragment as high + low: the high part is what TF32 keeps of the value (10 mantissa bits), the low part the
// rest, of which TF32 keeps another 10.
template <int N>
struct SplitFragment {
    float high[N], low[N];
    __device__ __forceinline__ void set(int index, float value) {
        high[index] = __uint_as_float(__float_as_uint(value) & 0xffffe000u);
        low[index] = value - high[index];
    }
};
using FragmentA = SplitFragment<4>;
using FragmentB = SplitFragment<2>;

__device__ __forceinline__ void mma_split(float (&d)[4], const FragmentA& a, const FragmentB& b) {
    mma_tf32(d, a.low, b.high);
    mma_tf32(d, a.high, b.low);
    mma_tf32(d, a.high, b.high);
}
// B is exact in TF32
__device__ __forceinline__ void mma_split(float (&d)[4], const FragmentA& a, const float (&b)[2]) {
    mma_tf32(d, a.low, b);
    mma_tf32(d, a.high, b);
}
// The same for two accumulators, whose products alternate so that none waits for the one before it.
__device__ __forceinline__ void mma_split(float (&d)[2][4], const FragmentA& a, const FragmentB& b0, const FragmentB& b1) {
    mma_tf32(d[0], a.low, b0.high);
    mma_tf32(d[1], a.low, b1.high);
    mma_tf32(d[0], a.high, b0.low);
    mma_tf32(d[1], a.high, b1.low);
    mma_tf32(d[0], a.high, b0.high);
    mma_tf32(d[1], a.high, b1.high);
}
__device__ __forceinline__ void mma_split(float (&d)[2][4], const FragmentA& a, const float (&b0)[2], const float (&b1)[2]) {
    mma_tf32(d[0], a.low, b0);
    mma_tf32(d[1], a.low, b1);
    mma_tf32(d[0], a.high, b0);
    mma_tf32(d[1], a.high, b1);
}

// rows `source[row * stride + column]` of a 16 x 8 operand
__device__ __forceinline__ FragmentA load_a(const float* source, uint32_t stride, uint32_t lane) {
    FragmentA out;
    const float* at = source + (lane >> 2) * stride + (lane & 3);
    out.set(0, at[0]);
    out.set(1, at[8 * stride]);
    out.set(2, at[4]);
    out.set(3, at[8 * stride + 4]);
    return out;
}
// the same operand stored transposed: `source[column * stride + row]`
__device__ __forceinline__ FragmentA load_a_transposed(const float* source, uint32_t stride, uint32_t lane) {
    FragmentA out;
    const float* at = source + (lane & 3) * stride + (lane >> 2);
    out.set(0, at[0]);
    out.set(1, at[8]);
    out.set(2, at[4 * stride]);
    out.set(3, at[4 * stride + 8]);
    return out;
}
// an 8 x 8 operand B[k][n] stored as `source[k * stride + n]`, or transposed as `source[n * stride + k]`
__device__ __forceinline__ FragmentB load_b(const float* source, uint32_t stride, uint32_t lane) {
    FragmentB out;
    const float* at = source + (lane & 3) * stride + (lane >> 2);
    out.set(0, at[0]);
    out.set(1, at[4 * stride]);
    return out;
}
__device__ __forceinline__ FragmentB load_b_transposed(const float* source, uint32_t stride, uint32_t lane) {
    FragmentB out;
    const float* at = source + (lane >> 2) * stride + (lane & 3);
    out.set(0, at[0]);
    out.set(1, at[4]);
    return out;
}
// a 16 x 8 result to `target[row * stride + column]`
__device__ __forceinline__ void store_c(float* target, uint32_t stride, uint32_t lane, const float (&c)[4]) {
    float* at = target + (lane >> 2) * stride + (lane & 3) * 2;
    *reinterpret_cast<float2*>(at) = make_float2(c[0], c[1]);
    *reinterpret_cast<float2*>(at + 8 * stride) = make_float2(c[2], c[3]);
}

constexpr uint32_t kChunkThreads = 512;           // four groups of four warps
static_assert(kChunkThreads == 8 * kChunkDim, "eight threads per channel stage W2");

__global__ void __launch_bounds__(kChunkThreads)
delta_chunk_kernel(const DeltaArgs<__nv_bfloat16> args) {
    constexpr uint32_t DP = kChunkDim;
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char chunk_shared[];
    const ChunkLayout layout(args.rank);
    const uint32_t dim = args.dim;
    const uint32_t head = blockIdx.x % args.heads;
    const uint32_t segment = blockIdx.x / args.heads;
    const uint32_t begin = args.segments.offsets[segment];
    uint32_t end = args.segments.offsets[segment + 1];
    end = end < args.segments.num_tokens ? end : static_cast<uint32_t>(args.segments.num_tokens);
    const size_t slot = args.segments.slots[segment];
    if (begin >= end || slot >= args.segments.num_request_slots) {
        return;
    }
    const int tiles = static_cast<int>((end - begin + kPromptTokens - 1) / kPromptTokens);
    const size_t width = static_cast<size_t>(args.heads) * dim;
    const size_t head_base = static_cast<size_t>(head) * dim;
    auto* raw = reinterpret_cast<__nv_bfloat16*>(chunk_shared + layout.raw);
    auto* tanh_parts = reinterpret_cast<__nv_bfloat16*>(chunk_shared + layout.tanh_parts);
    auto* w2 = reinterpret_cast<__nv_bfloat16*>(chunk_shared + layout.w2);
    auto* constants = reinterpret_cast<float*>(chunk_shared + layout.constants);
    float* state_base = reinterpret_cast<float*>(static_cast<unsigned char*>(args.record.base) +
                                                 slot * args.record.stride + args.record.offset) +
                        head_base * dim;
    auto stage_of = [&](int tile) { return raw + tile % kChunkStages * kPromptTokens * layout.raw_row; };
    auto unit_of = [&](int tile) {
        return reinterpret_cast<float*>(chunk_shared + layout.scale) + tile % 2 * kPromptTokens;
    };
    auto tanh_of = [&](int tile) { return tanh_parts + tile % 2 * 2 * kPromptTokens * layout.z_stride; };
    auto operands_of = [&](int tile) {
        return reinterpret_cast<float*>(chunk_shared + layout.operands) +
               tile % 3 * kPromptTokens * 2 * (kRowStride + kTransposedStride);
    };
    constexpr uint32_t kOperandR = kPromptTokens * kRowStride, kOperandK = 2 * kPromptTokens * kRowStride,
                       kOperandB = kOperandK + kPromptTokens * kTransposedStride;
    auto decay_end_of = [&](int tile) {
        return reinterpret_cast<float*>(chunk_shared + layout.decay_end) + tile % 3 * DP;
    };
    constexpr uint32_t kTriangle = kPromptTokens * kTriangleStride;
    auto triangles_of = [&](int tile) {
        return reinterpret_cast<float*>(chunk_shared + layout.triangles) + tile % 2 * 5 * kTriangle;
    };
    auto produced_of = [&](int tile) {
        return reinterpret_cast<float*>(chunk_shared + layout.produced) + tile % 2 * kPromptTokens * kProducedStride;
    };

    for (uint32_t item = threadIdx.x; item < kChunkStages * kPromptTokens * layout.raw_row / 8; item += kChunkThreads) {
        reinterpret_cast<uint4*>(raw)[item] = make_uint4(0, 0, 0, 0);
    }
    {
        // eight threads per channel
        const uint32_t channel = threadIdx.x / 8;
        const __nv_bfloat16* source = args.decay_up + (head_base + channel) * args.rank;
        const bool vector_rank = args.rank % 8 == 0;
        for (uint32_t z = threadIdx.x % 8 * 8; z < layout.z_stride; z += 64) {
            uint4 value = make_uint4(0, 0, 0, 0);
            if (channel < dim && z < args.rank) {
                if (vector_rank) {
                    value = *reinterpret_cast<const uint4*>(source + z);
                } else {
                    auto* elements = reinterpret_cast<__nv_bfloat16*>(&value);
                    for (uint32_t i = 0; i < 8 && z + i < args.rank; ++i) elements[i] = source[z + i];
                }
            }
            *reinterpret_cast<uint4*>(w2 + channel * layout.z_stride + z) = value;
        }
    }
    if (threadIdx.x < DP) {
        const uint32_t channel = threadIdx.x;
        const bool live = channel < dim;
        constants[channel] = live ? __bfloat162float(args.decay_base[head_base + channel]) : 0.0f;
        constants[DP + channel] = live ? __bfloat162float(args.removal_bias[head_base + channel]) : 0.0f;
        constants[2 * DP + channel] = live ? __bfloat162float(args.norm[head_base + channel]) : 0.0f;
    }

    const uint32_t group = threadIdx.x / 128;          // 0 matrices, 1 copies, 2 elements, 3 triangles
    const uint32_t warp = threadIdx.x / 32 % 4;        // of the group
    const uint32_t lane = threadIdx.x % 32;

    // ---- matrices: state of 16 value columns, as the accumulators of the update product
    const uint32_t column0 = warp * 16;
    float* state = reinterpret_cast<float*>(chunk_shared + layout.state) + warp * DP * kColumnStride;
    float* columns = reinterpret_cast<float*>(chunk_shared + layout.columns) + warp * kPromptTokens * kColumnStride;
    float accumulator[4][2][4];                        // [16 key channels][8 columns]
    if (group == 0) {
#pragma unroll
        for (uint32_t m = 0; m < 4; ++m) {
#pragma unroll
            for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) {
                    const uint32_t row = m * 16 + (lane >> 2) + (i >> 1) * 8;
                    const uint32_t column = column0 + n * 8 + (lane & 3) * 2 + (i & 1);
                    accumulator[m][n][i] =
                        row < dim && column < dim ? state_base[static_cast<size_t>(column) * dim + row] : 0.0f;
                }
                store_c(state + m * 16 * kColumnStride + n * 8, kColumnStride, lane, accumulator[m][n]);
            }
        }
    }
    // ---- copies: the 16-byte pieces of a token's row that this lane moves
    const uint32_t per_vector = dim / 8;
    const uint32_t pieces = 5 * per_vector + (args.rank + 7) / 8;
    auto piece_offsets = [&](uint32_t piece, uint32_t& source, uint32_t& target) {
        if (piece < 5 * per_vector) {
            const uint32_t vector = piece / per_vector;
            const uint32_t chunk = piece - vector * per_vector;
            source = static_cast<uint32_t>(vector * width + head_base) + chunk * 8;
            target = vector * DP + chunk * 8;
        } else {
            const uint32_t chunk = piece - 5 * per_vector;
            source = static_cast<uint32_t>(5 * width) + chunk * 8;
            target = 5 * DP + chunk * 8;
        }
    };
    uint32_t first_source = 0, first_target = 0, second_source = 0, second_target = 0;
    piece_offsets(lane, first_source, first_target);
    piece_offsets(lane + 32, second_source, second_target);
    __syncthreads();

    for (int step = -4; step <= tiles; ++step) {
        if (group == 0) {
            const int tile = step;
            if (tile >= 0 && tile < tiles) {
                const float* operands = operands_of(tile);
                const float* triangles = triangles_of(tile);
                // U Q_0 and R Q_0
                float from_state[2][2][4] = {};        // [U, R][8 columns]
#pragma unroll
                for (uint32_t k = 0; k < DP / 8; ++k) {
                    const FragmentB b0 = load_b(state + k * 8 * kColumnStride, kColumnStride, lane);
                    const FragmentB b1 = load_b(state + k * 8 * kColumnStride + 8, kColumnStride, lane);
#pragma unroll
                    for (uint32_t m = 0; m < 2; ++m) {
                        const FragmentA a = load_a(operands + m * kOperandR + k * 8, kRowStride, lane);
                        mma_split(from_state[m], a, b0, b1);
                    }
                }
                // v of the tile: B operand [token][column], exact in TF32
                float v[2][2][2];                      // [8 tokens][8 columns]
                const __nv_bfloat16* values = stage_of(tile) + 2 * DP + column0;
#pragma unroll
                for (uint32_t k = 0; k < 2; ++k) {
#pragma unroll
                    for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                        for (uint32_t i = 0; i < 2; ++i) {
                            v[k][n][i] = __bfloat162float(
                                values[(k * 8 + (lane & 3) + i * 4) * layout.raw_row + n * 8 + (lane >> 2)]);
                        }
                    }
                }
                // right-hand side, then Y
#pragma unroll
                for (uint32_t k = 0; k < 2; ++k) {
                    const FragmentA a = load_a(triangles + 1 * kTriangle + k * 8, kTriangleStride, lane);
                    mma_split(from_state[0], a, v[k][0], v[k][1]);
                }
                store_c(columns, kColumnStride, lane, from_state[0][0]);
                store_c(columns + 8, kColumnStride, lane, from_state[0][1]);
                __syncwarp();
                float solved[2][4] = {};
#pragma unroll
                for (uint32_t k = 0; k < 2; ++k) {
                    const FragmentA a = load_a(triangles + k * 8, kTriangleStride, lane);
                    mma_split(solved, a, load_b(columns + k * 8 * kColumnStride, kColumnStride, lane),
                              load_b(columns + k * 8 * kColumnStride + 8, kColumnStride, lane));
                }
                __syncwarp();
                store_c(columns, kColumnStride, lane, solved[0]);
                store_c(columns + 8, kColumnStride, lane, solved[1]);
                __syncwarp();
                FragmentB y[2][2];
#pragma unroll
                for (uint32_t k = 0; k < 2; ++k) {
#pragma unroll
                    for (uint32_t n = 0; n < 2; ++n) {
                        y[k][n] = load_b(columns + k * 8 * kColumnStride + n * 8, kColumnStride, lane);
                    }
                }
                // O
#pragma unroll
                for (uint32_t k = 0; k < 2; ++k) {
                    const FragmentA with_y = load_a(triangles + 2 * kTriangle + k * 8, kTriangleStride, lane);
                    const FragmentA with_v = load_a(triangles + 3 * kTriangle + k * 8, kTriangleStride, lane);
                    mma_split(from_state[1], with_v, v[k][0], v[k][1]);
                    mma_split(from_state[1], with_y, y[k][0], y[k][1]);
                }
                store_c(produced_of(tile) + column0, kProducedStride, lane, from_state[1][0]);
                store_c(produced_of(tile) + column0 + 8, kProducedStride, lane, from_state[1][1]);
                // the state behind the tile
                const float* decay = decay_end_of(tile);
#pragma unroll
                for (uint32_t m = 0; m < 4; ++m) {
#pragma unroll
                    for (uint32_t k = 0; k < 2; ++k) {
                        const uint32_t at = k * 8 * kTransposedStride + m * 16;
                        const FragmentA with_v = load_a_transposed(operands + kOperandK + at, kTransposedStride, lane);
                        const FragmentA with_y = load_a_transposed(operands + kOperandB + at, kTransposedStride, lane);
                        mma_split(accumulator[m], with_v, v[k][0], v[k][1]);
                        mma_split(accumulator[m], with_y, y[k][0], y[k][1]);
                    }
                    const float upper = decay[m * 16 + (lane >> 2)], lower = decay[m * 16 + (lane >> 2) + 8];
#pragma unroll
                    for (uint32_t n = 0; n < 2; ++n) {
                        accumulator[m][n][0] *= upper;
                        accumulator[m][n][1] *= upper;
                        accumulator[m][n][2] *= lower;
                        accumulator[m][n][3] *= lower;
                        store_c(state + m * 16 * kColumnStride + n * 8, kColumnStride, lane, accumulator[m][n]);
                    }
                }
            }
        } else if (group == 1) {
            // ---- load tile step + 4
            {
                const int tile = step + 4;
                const uint32_t first = begin + static_cast<uint32_t>(tile) * kPromptTokens;
                if (tile < tiles) {
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {
                        const uint32_t t = warp * 4 + i;
                        if (first + t < end) {
                            const __nv_bfloat16* source = args.projected + static_cast<size_t>(first + t) * args.pitch;
                            __nv_bfloat16* target = stage_of(tile) + t * layout.raw_row;
                            if (lane < pieces) copy_async_16(target + first_target, source + first_source);
                            if (lane + 32 < pieces) copy_async_16(target + second_target, source + second_source);
                            for (uint32_t piece = lane + 64; piece < pieces; piece += 32) {
                                uint32_t from, to;
                                piece_offsets(piece, from, to);
                                copy_async_16(target + to, source + from);
                            }
                        }
                    }
                }
                copy_async_commit();
            }
            // ---- finish tile step - 1
            if (step >= 1) {
                const int tile = step - 1;
                const __nv_bfloat16* stage = stage_of(tile);
                const float* source = produced_of(tile);
                const uint32_t first = begin + static_cast<uint32_t>(tile) * kPromptTokens;
                float2 value[4], gate[4];
                float squares[4];
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) {
                    const uint32_t t = warp * 4 + i;
                    value[i] = *reinterpret_cast<const float2*>(source + t * kProducedStride + lane * 2);
                    gate[i] = __bfloat1622float2(
                        *reinterpret_cast<const __nv_bfloat162*>(stage + t * layout.raw_row + 3 * DP + lane * 2));
                    squares[i] = fmaf(value[i].x, value[i].x, value[i].y * value[i].y);
                }
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) squares[i] = warp_sum(squares[i]);
                const float2 weight = *reinterpret_cast<const float2*>(constants + 2 * DP + lane * 2);
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) {
                    const uint32_t t = warp * 4 + i;
                    const float factor = rsqrtf(squares[i] / static_cast<float>(dim) + args.eps);
                    const uint32_t both = pack_bf16x2(value[i].x * factor * weight.x * fast_sigmoid(gate[i].x),
                                                      value[i].y * factor * weight.y * fast_sigmoid(gate[i].y));
                    if (lane * 2 < dim && first + t < end) {
                        *reinterpret_cast<uint32_t*>(args.out + static_cast<size_t>(first + t) * args.out_pitch +
                                                     head_base + lane * 2) = both;
                    }
                }
            }
            // ---- tanh(z) and 1 / |k| of tile step + 3, whose copies were issued one step ago
            copy_async_wait<1>();
            named_barrier(1, 128);
            const int tile = step + 3;
            if (tile >= 0 && tile < tiles) {
                const __nv_bfloat16* stage = stage_of(tile);
                __nv_bfloat16* parts = tanh_of(tile);
                float squares[4];
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) {
                    const float2 both = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(
                        stage + (warp * 4 + i) * layout.raw_row + DP + lane * 2));
                    squares[i] = fmaf(both.x, both.x, both.y * both.y);
                }
                for (uint32_t z = lane * 2; z < layout.rank_pad; z += 64) {
                    float2 both[4];
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {
                        both[i] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(
                            stage + (warp * 4 + i) * layout.raw_row + 5 * DP + z));
                        // columns between rank and the end of its last copy belong to nobody
                        both[i].x = z < args.rank ? fast_tanh(both[i].x) : 0.0f;
                        both[i].y = z + 1 < args.rank ? fast_tanh(both[i].y) : 0.0f;
                    }
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {
                        const __nv_bfloat162 high = __floats2bfloat162_rn(both[i].x, both[i].y);
                        const float2 rounded = __bfloat1622float2(high);
                        __nv_bfloat16* target = parts + (warp * 4 + i) * layout.z_stride + z;
                        *reinterpret_cast<__nv_bfloat162*>(target) = high;
                        *reinterpret_cast<__nv_bfloat162*>(target + kPromptTokens * layout.z_stride) =
                            __floats2bfloat162_rn(both[i].x - rounded.x, both[i].y - rounded.y);
                    }
                }
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) squares[i] = warp_sum(squares[i]);
                if (lane < 4) {
                    const float mine = lane == 0 ? squares[0] : (lane == 1 ? squares[1] : (lane == 2 ? squares[2] : squares[3]));
                    unit_of(tile)[warp * 4 + lane] = rsqrtf(mine + kUnitEps);
                }
            }
        } else if (group == 2) {
            const int tile = step + 2;
            if (tile >= 0 && tile < tiles) {
                const uint32_t tokens = min(kPromptTokens, end - begin - static_cast<uint32_t>(tile) * kPromptTokens);
                const __nv_bfloat16* stage = stage_of(tile);
                const __nv_bfloat16* parts = tanh_of(tile);
                const float* unit = unit_of(tile);
                float* operands = operands_of(tile);
                // decay logits of 16 tokens x 16 channels per warp
                float logits[2][4] = {};
                const uint32_t z_row = lane % 16, z_part = lane / 16 * 8;
                for (uint32_t z = 0; z < layout.rank_pad; z += 16) {
                    uint32_t b0, b1, b2, b3, high[4], low[4];
                    const uint32_t channel = warp * 16 + lane / 16 * 8 + lane % 8;
                    ldmatrix_x4(smem_u32(w2 + channel * layout.z_stride + z + lane / 8 % 2 * 8), b0, b1, b2, b3);
                    const __nv_bfloat16* source = parts + z_row * layout.z_stride + z + z_part;
                    ldmatrix_x4(smem_u32(source), high[0], high[1], high[2], high[3]);
                    ldmatrix_x4(smem_u32(source + kPromptTokens * layout.z_stride), low[0], low[1], low[2], low[3]);
                    mma_bf16_16816(logits[0], high[0], high[1], high[2], high[3], b0, b1);
                    mma_bf16_16816(logits[1], high[0], high[1], high[2], high[3], b2, b3);
                    mma_bf16_16816(logits[0], low[0], low[1], low[2], low[3], b0, b1);
                    mma_bf16_16816(logits[1], low[0], low[1], low[2], low[3], b2, b3);
                }
                const uint32_t t0 = lane >> 2;
                // log decay per token, then its prefix sums: over the eight lanes that hold tokens 0..7, and over
                // those that hold 8..15 in the other half of the fragment
                float own[2][4], prefix[2][4];
#pragma unroll
                for (uint32_t n = 0; n < 2; ++n) {
                    const uint32_t channel = warp * 16 + n * 8 + (lane & 3) * 2;
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {
                        own[n][i] = t0 + (i >> 1) * 8 < tokens
                                        ? -kDecayScale * fast_sigmoid(logits[n][i] + constants[channel + (i & 1)])
                                        : 0.0f;
                        prefix[n][i] = own[n][i];
                    }
                }
#pragma unroll
                for (uint32_t delta = 4; delta < 32; delta <<= 1) {
#pragma unroll
                    for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                        for (uint32_t i = 0; i < 4; ++i) {
                            const float other = __shfl_up_sync(0xffffffffu, prefix[n][i], delta);
                            if (lane >= delta) prefix[n][i] += other;
                        }
                    }
                }
#pragma unroll
                for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                    for (uint32_t i = 0; i < 2; ++i) {
                        prefix[n][2 + i] += __shfl_sync(0xffffffffu, prefix[n][i], 28 + (lane & 3));
                    }
                }
#pragma unroll
                for (uint32_t n = 0; n < 2; ++n) {
                    const uint32_t channel = warp * 16 + n * 8 + (lane & 3) * 2;
                    const float2 bias = *reinterpret_cast<const float2*>(constants + DP + channel);
#pragma unroll
                    for (uint32_t half = 0; half < 2; ++half) {
                        const uint32_t t = t0 + half * 8;
                        const __nv_bfloat16* row = stage + t * layout.raw_row + channel;
                        float2 r = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row));
                        float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row + DP));
                        const float2 rate = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row + 4 * DP));
                        if (t >= tokens) r = k = make_float2(0.0f, 0.0f);      // left over from an earlier tile
                        const float scale = unit[t];
                        const float px = __expf(prefix[n][2 * half]), py = __expf(prefix[n][2 * half + 1]);
                        const float bx = __expf(prefix[n][2 * half] - own[n][2 * half]);
                        const float by = __expf(prefix[n][2 * half + 1] - own[n][2 * half + 1]);
                        const float ix = __expf(-prefix[n][2 * half]), iy = __expf(-prefix[n][2 * half + 1]);
                        float* row_target = operands + t * kRowStride + channel;
                        *reinterpret_cast<float2*>(row_target) = make_float2(k.x * scale * bx, k.y * scale * by);
                        *reinterpret_cast<float2*>(row_target + kOperandR) = make_float2(r.x * px, r.y * py);
                        float* transposed_target = operands + kOperandK + t * kTransposedStride + channel;
                        *reinterpret_cast<float2*>(transposed_target) = make_float2(k.x * ix, k.y * iy);
                        *reinterpret_cast<float2*>(transposed_target + kOperandB - kOperandK) =
                            make_float2(-fast_sigmoid(rate.x + bias.x) * k.x * scale * ix,
                                        -fast_sigmoid(rate.y + bias.y) * k.y * scale * iy);
                        if (t == kPromptTokens - 1) {
                            *reinterpret_cast<float2*>(decay_end_of(tile) + channel) = make_float2(px, py);
                        }
                    }
                }
            }
        } else {
            const int tile = step + 1;
            if (tile >= 0 && tile < tiles) {
                const float* operands = operands_of(tile);
                float* triangles = triangles_of(tile);
                // warps 0, 1: rows of U; 2, 3: rows of R; even warps against B, odd ones against K
                const float* rows = operands + (warp >> 1) * kOperandR;
                const float* against = operands + (warp & 1 ? kOperandK : kOperandB);
                float product[2][4] = {};
#pragma unroll
                for (uint32_t k = 0; k < DP / 8; ++k) {
                    const FragmentA a = load_a(rows + k * 8, kRowStride, lane);
                    mma_split(product, a, load_b_transposed(against + k * 8, kTransposedStride, lane),
                              load_b_transposed(against + 8 * kTransposedStride + k * 8, kTransposedStride, lane));
                }
                // U B^T goes behind the four results, U K^T, R B^T and R K^T to places 1, 2 and 3
                float* target = triangles + (warp == 0 ? 4 : warp) * kTriangle;
#pragma unroll
                for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                    for (uint32_t i = 0; i < 4; ++i) {
                        const uint32_t row = (lane >> 2) + (i >> 1) * 8;
                        const uint32_t column = n * 8 + (lane & 3) * 2 + (i & 1);
                        const bool kept = warp < 2 ? column < row : column <= row;     // U meets the state before s = t
                        if (!kept) product[n][i] = 0.0f;
                    }
                    store_c(target + n * 8, kTriangleStride, lane, product[n]);
                }
                if (warp == 0) {
                    __syncwarp();
                    // column `lane` of the inverse of I - L: x_t = e_t + sum over s < t of L[t][s] x_s
                    const float* lower = triangles + 4 * kTriangle;
                    float x[kPromptTokens];
#pragma unroll
                    for (uint32_t t = 0; t < kPromptTokens; ++t) {
                        float even = t == lane ? 1.0f : 0.0f, odd = 0.0f;
#pragma unroll
                        for (uint32_t s = 0; s < t; s += 2) {
                            const float2 pair = *reinterpret_cast<const float2*>(lower + t * kTriangleStride + s);
                            even = fmaf(pair.x, x[s], even);
                            if (s + 1 < t) odd = fmaf(pair.y, x[s + 1], odd);
                        }
                        x[t] = even + odd;
                        if (lane < kPromptTokens) triangles[t * kTriangleStride + lane] = x[t];
                    }
                }
            }
        }
        __syncthreads();
    }
    if (group == 0) {
#pragma unroll
        for (uint32_t m = 0; m < 4; ++m) {
#pragma unroll
            for (uint32_t n = 0; n < 2; ++n) {
#pragma unroll
                for (uint32_t i = 0; i < 4; ++i) {
                    const uint32_t row = m * 16 + (lane >> 2) + (i >> 1) * 8;
                    const uint32_t column = column0 + n * 8 + (lane & 3) * 2 + (i & 1);
                    if (row < dim && column < dim) {
                        state_base[static_cast<size_t>(column) * dim + row] = accumulator[m][n][i];
                    }
                }
            }
        }
    }
}

template <typename T, uint32_t DP>
cudaError_t launch_decode(cudaStream_t stream, const DeltaArgs<T>& args) {
    const size_t shared = (5 * DP + 2 * (DP * 4 / 32) + args.rank) * sizeof(float);
    if (shared > 48 * 1024) {
        return cudaErrorInvalidValue;
    }
    return launch_kernel(delta_decode_kernel<T, DP>,
                         static_cast<unsigned int>(args.segments.num_segments * args.heads), DP * 4, shared, stream, 1,
                         args);
}

template <uint32_t DP, uint32_t COLUMNS, uint32_t HELPERS>
cudaError_t launch_prompt(cudaStream_t stream, const DeltaArgs<__nv_bfloat16>& args) {
    const size_t shared = PromptLayout<DP>(args.rank).total;
    const auto kernel = delta_prompt_kernel<DP, COLUMNS, HELPERS>;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                    static_cast<int>(shared));
    if (status != cudaSuccess) return status;
    return launch_kernel(kernel, static_cast<unsigned int>(args.segments.num_segments * args.heads),
                         DP / COLUMNS * 8 + HELPERS, shared, stream, 1, args);
}

cudaError_t launch_chunk(cudaStream_t stream, const DeltaArgs<__nv_bfloat16>& args) {
    const size_t shared = ChunkLayout(args.rank).total;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(delta_chunk_kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                    static_cast<int>(shared));
    if (status != cudaSuccess) return status;
    return launch_kernel(delta_chunk_kernel, static_cast<unsigned int>(args.segments.num_segments * args.heads),
                         kChunkThreads, shared, stream, 1, args);
}

bool prompt_kernel_takes(const DeltaArgs<__nv_bfloat16>& args) {
    const size_t shared = args.dim <= 64 ? PromptLayout<64>(args.rank).total : PromptLayout<128>(args.rank).total;
    return args.dim % 8 == 0 && args.dim <= 128 && args.rank <= kPromptMaxRank && args.pitch % 8 == 0 &&
           args.out_pitch % 2 == 0 && aligned_to(args.projected, 16) && aligned_to(args.out, 4) &&
           aligned_to(args.decay_up, 16) &&
           shared <= 227 * 1024;
}

template <typename T, uint32_t DP, uint32_t LANES, uint32_t COLUMNS>
cudaError_t launch_sized(cudaStream_t stream, DeltaArgs<T> args) {
    args.splits = (args.dim + COLUMNS - 1) / COLUMNS;
    const bool single = args.segments.offsets == nullptr;
    const size_t staged_bytes = delta_shared_bytes<DP>(kTileTokens, args.rank, true);
    const bool staged = !single && staged_bytes <= 160 * 1024;
    const size_t shared = single ? delta_shared_bytes<DP>(1, args.rank, false)
                                 : (staged ? staged_bytes : delta_shared_bytes<DP>(kTileTokens, args.rank, false));
    void (*kernel)(const DeltaArgs<T>) =
        single ? delta_rule_kernel<T, DP, LANES, COLUMNS, 1, false>
               : (staged ? delta_rule_kernel<T, DP, LANES, COLUMNS, kTileTokens, true>
                         : delta_rule_kernel<T, DP, LANES, COLUMNS, kTileTokens, false>);
    if (shared > 227 * 1024) {
        return cudaErrorInvalidValue;
    }
    if (shared > 48 * 1024) {
        const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                        cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                        static_cast<int>(shared));
        if (status != cudaSuccess) return status;
    }
    const size_t blocks = args.segments.num_segments * args.heads * args.splits;
    const cudaError_t status =
        launch_kernel(kernel, static_cast<unsigned int>(blocks), LANES * COLUMNS, shared, stream, 1, args);
    if (status != cudaSuccess || args.raw == nullptr) {
        return status;
    }
    return launch_kernel(delta_output_kernel<T>,
                         static_cast<unsigned int>((args.segments.num_tokens * args.heads + 3) / 4), 128, 0, stream, 1,
                         args);
}

template <typename T>
cudaError_t launch_typed(cudaStream_t stream, const DeltaRuleLaunch& launch) {
    DeltaArgs<T> args;
    args.segments = launch.segments;
    args.heads = launch.heads;
    args.dim = launch.dim;
    args.rank = launch.rank;
    args.projected = static_cast<const T*>(launch.projected);
    args.pitch = launch.pitch;
    args.decay_up = static_cast<const __nv_bfloat16*>(launch.decay_up);
    args.decay_base = static_cast<const __nv_bfloat16*>(launch.decay_base);
    args.removal_bias = static_cast<const __nv_bfloat16*>(launch.removal_bias);
    args.norm = static_cast<const __nv_bfloat16*>(launch.norm);
    args.record = launch.record;
    args.raw = delta_rule_needs_scratch(launch.dim) ? launch.raw : nullptr;
    args.out = static_cast<T*>(launch.out);
    args.out_pitch = launch.out_pitch;
    args.eps = launch.eps;
    args.splits = 1;
    if (launch.segments.offsets == nullptr && launch.dim <= 128 && launch.rank <= 4096) {
        if (launch.dim <= 32) return launch_decode<T, 32>(stream, args);
        if (launch.dim <= 64) return launch_decode<T, 64>(stream, args);
        return launch_decode<T, 128>(stream, args);
    }
    if constexpr (std::is_same<T, __nv_bfloat16>::value) {
        if (launch.segments.offsets != nullptr && option(kOptDeltaPrompt) != 2 && prompt_kernel_takes(args)) {
            if (launch.dim <= kChunkDim && ChunkLayout(launch.rank).total <= 227 * 1024 && option(kOptDeltaPrompt) == 0) {
                return launch_chunk(stream, args);
            }
            return launch.dim <= 64 ? launch_prompt<64, 4, 128>(stream, args) : launch_prompt<128, 4, 128>(stream, args);
        }
    }
    if (launch.dim <= 32) return launch_sized<T, 32, 4, 32>(stream, args);
    if (launch.dim <= 64) return launch_sized<T, 64, 4, 64>(stream, args);
    if (launch.dim <= 128) return launch_sized<T, 128, 4, 128>(stream, args);
    if (launch.dim <= kDeltaMaxDim && launch.raw != nullptr) return launch_sized<T, 256, 8, 64>(stream, args);
    return cudaErrorInvalidValue;
}

}  // namespace

bool delta_rule_needs_scratch(uint32_t dim) { return dim > 128; }

cudaError_t launch_delta_rule(cudaStream_t stream, const DeltaRuleLaunch& launch) {
    const auto run = [&](const DeltaRuleLaunch& part) {
        return part.type == Activation::kF32 ? launch_typed<float>(stream, part)
                                             : launch_typed<__nv_bfloat16>(stream, part);
    };
    if (launch.segments.offsets == nullptr || launch.decode_tokens == 0) {
        return run(launch);
    }
    DeltaRuleLaunch decodes = launch;
    decodes.segments.offsets = nullptr;
    decodes.segments.num_segments = launch.decode_tokens;
    decodes.segments.num_tokens = launch.decode_tokens;
    const cudaError_t status = run(decodes);
    if (status != cudaSuccess || launch.decode_tokens == launch.segments.num_segments) {
        return status;
    }
    DeltaRuleLaunch prompts = launch;      // segment offsets are absolute token indices
    prompts.segments.offsets += launch.decode_tokens;
    prompts.segments.slots += launch.decode_tokens;
    prompts.segments.num_segments -= launch.decode_tokens;
    return run(prompts);
}

}  // namespace lfm25
