// The generalised delta rule with a decay per key channel:
//     u_t = k_t / sqrt(|k_t|^2 + 1e-6)
//     S_t = diag(w_t) S_(t-1) - (a_t * u_t) (u_t^T S_(t-1)) + k_t v_t^T          o_t = S_t^T r_t
// per head, with w_t = exp(-exp(-1/2) sigmoid(W2 tanh(z_t) + w0)) and a_t = sigmoid(a_t' + bias), followed by the
// head's RMS norm, the norm weight and the output gate.
//
// A column of S (one value channel) never meets another one, so a CTA takes the columns of one head of one sequence,
// LANES threads a column, and keeps them in registers over the whole segment: the state is read from and written to
// memory once per step however long the segment is.  Everything a token contributes is prepared for a tile of tokens
// in shared memory (all in f32) and then consumed token by token: per token a thread forms its share of u^T S, LANES
// threads add theirs up, and the same pass over its rows updates S and accumulates r^T S.  Arithmetic on the state
// uses the packed two-wide f32 instructions of sm_100 (each half rounds like the scalar one).
#include <math.h>

#include "launch.h"
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
__device__ __forceinline__ Pair fma_pair(Pair a, Pair b, Pair c) {
    Pair out;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(out) : "l"(a), "l"(b), "l"(c));
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
    if (launch.dim <= 32) return launch_sized<T, 32, 4, 32>(stream, args);
    if (launch.dim <= 64) return launch_sized<T, 64, 4, 64>(stream, args);
    if (launch.dim <= 128) return launch_sized<T, 128, 4, 128>(stream, args);
    if (launch.dim <= kDeltaMaxDim && launch.raw != nullptr) return launch_sized<T, 256, 8, 64>(stream, args);
    return cudaErrorInvalidValue;
}

}  // namespace

bool delta_rule_needs_scratch(uint32_t dim) { return dim > 128; }

cudaError_t launch_delta_rule(cudaStream_t stream, const DeltaRuleLaunch& launch) {
    return launch.type == Activation::kF32 ? launch_typed<float>(stream, launch)
                                           : launch_typed<__nv_bfloat16>(stream, launch);
}

}  // namespace lfm25
