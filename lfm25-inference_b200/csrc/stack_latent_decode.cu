// Attention against cached latents on the 5th-generation tensor cores (tcgen05 + tensor memory), for bf16 activations: one
// query token, any number of heads, latents of up to 512 and rotated parts of up to 128 dimensions.
//
// All heads read the same latent and the same rotated key, so the keys take the 64 or 128 rows of an MMA and the heads its
// columns: a CTA owns one token, up to 64 heads (16, 32 or 64 columns) and a share of the visible keys.
//   warp 0      producer: the queries once, then the keys in stages of 64 (4 pages), [latent | rotated key] in chunks of 64
//               dimensions, 128-byte swizzle
//   warp 1      tensor memory and the MMAs: S^T [64 keys, heads] = K Q^T over all chunks, then O^T [kv_rank, heads] +=
//               latent^T P^T over the same shared memory, now read with the latent dimensions as rows
//   warps 2-5   one key per thread (lanes 0 .. 15 of a quadrant): mask and softmax weights in f32.  The weights are taken
//               against a reference that follows the running maximum only when it falls more than 2^8 behind; then the
//               accumulators in tensor memory are rescaled
// The weights enter the second product as a sum of two bf16 values (16 significant bits); sums and accumulators are f32.
// The splits of a token merge through the distributed shared memory of their cluster.
#include <cooperative_groups.h>
#include <cuda.h>
#include <math.h>

#include <algorithm>

#include "launch.h"
#include "options.h"
#include "stack_latent.h"
#include "tcgen05.cuh"
#include "tensor_map.h"

namespace lfm25 {

namespace {

namespace cg = cooperative_groups;

constexpr uint32_t kThreads = 192;
constexpr uint32_t kPagesPerStage = 4;
constexpr uint32_t kKeys = kPagesPerStage * kPageSize;       // 64
constexpr uint32_t kBoxBytes = kPageSize * 128;              // one page, 64 dimensions
constexpr uint32_t kChunkBytes = kPagesPerStage * kBoxBytes; // a stage's keys, 64 dimensions
constexpr uint32_t kMaxStages = 6;
constexpr uint32_t kMaxSplits = 8;
constexpr float kSlack = 8.0f;                               // how far (log2) a score may exceed the reference
constexpr size_t kSharedLimit = 227 * 1024;

struct Params {
    uint32_t heads, kv_rank;
    float scale;
    const uint32_t* block_tables;
    size_t block_table_stride;
    size_t block_table_rows;
    size_t num_pages;
    const uint32_t* request_slots;
    const uint32_t* positions;
    __nv_bfloat16* out;
    unsigned int* status;
    uint32_t latent_chunks, chunks;      // 64-dimension chunks of a key: of the latent, altogether
    uint32_t blocks;                     // 128-dimension blocks of the latent
    uint32_t head_blocks, splits, stages;
    uint32_t tmem_columns;
    uint64_t wait_limit;
};

// Floats and barriers behind the ring
template <uint32_t N>
struct Control {
    float reference[N];      // log2 of what the weights are taken against
    float factor[N];
    float warp_max[4][N];
    float warp_sum[4][N];
    float total[N];
    uint64_t full[kMaxStages], empty[kMaxStages];
    uint64_t query, scores[2], weights[2], product[2];
    uint32_t tmem;
    volatile uint32_t abort;
    volatile uint32_t missing_page;
    volatile uint32_t failed[2];
};

template <uint32_t N>
constexpr size_t shared_bytes(uint32_t chunks, uint32_t stages) {
    return 1024 + static_cast<size_t>(chunks) * N * 128 + 4 * N * 128 + static_cast<size_t>(stages) * chunks * kChunkBytes +
           sizeof(Control<N>);
}

__device__ __forceinline__ void mma_shared(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc,
                                           uint32_t accumulate) {
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
        "}\n" ::"r"(tmem_d),
        "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
        : "memory");
}

// (dimensions, heads, tokens)
__device__ __forceinline__ void load_queries(uint32_t dst, const void* tensor_map, uint32_t bar, int32_t x, int32_t head,
                                             int32_t token) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
        ::"r"(dst), "l"(reinterpret_cast<uint64_t>(tensor_map)), "r"(bar), "r"(x), "r"(head), "r"(token)
        : "memory");
}

// MN-major operand of 128 rows, 128-byte swizzle: 64 rows (dimensions) per 128-byte line, one line per key, 8-key groups
// 1024 bytes apart, the other 64 rows `kChunkBytes` further on.
__device__ __forceinline__ uint64_t transposed_descriptor(uint32_t address) {
    uint64_t descriptor = static_cast<uint64_t>((address & 0x3ffff) >> 4);
    descriptor |= static_cast<uint64_t>(kChunkBytes >> 4) << 16;
    descriptor |= static_cast<uint64_t>(1024 >> 4) << 32;
    descriptor |= static_cast<uint64_t>(1) << 46;
    descriptor |= static_cast<uint64_t>(2) << 61;
    return descriptor;
}

// Barrier of the four softmax warps
__device__ __forceinline__ void softmax_barrier() {
    __syncwarp();
    asm volatile("bar.sync 1, 128;" ::: "memory");
}
__device__ __forceinline__ bool softmax_any(bool mine) {
    __syncwarp();
    uint32_t any;
    asm volatile(
        "{\n"
        ".reg .pred p, q;\n"
        "setp.ne.u32 p, %1, 0;\n"
        "bar.red.or.pred q, 1, 128, p;\n"
        "selp.u32 %0, 1, 0, q;\n"
        "}\n"
        : "=r"(any)
        : "r"(mine ? 1u : 0u)
        : "memory");
    return any != 0;
}

template <uint32_t N>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_umma_kernel(const __grid_constant__ CUtensorMap absorbed_map, const __grid_constant__ CUtensorMap rotated_map,
                             const __grid_constant__ CUtensorMap latent_map, const __grid_constant__ CUtensorMap key_map,
                             const Params p) {
    const uint32_t warp = threadIdx.x >> 5;
    const uint32_t lane = threadIdx.x & 31;
    extern __shared__ uint8_t latent_smem[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(latent_smem) + 1023) & ~uintptr_t(1023));
    const uint32_t stage_bytes = p.chunks * kChunkBytes;
    const uint32_t q_base = smem_u32(smem);
    const uint32_t p_base = q_base + p.chunks * N * 128;         // [buffer][high, low][head][64 keys]
    const uint32_t ring = p_base + 4 * N * 128;
    uint8_t* ring_bytes = smem + p.chunks * N * 128 + 4 * N * 128;
    Control<N>& control = *reinterpret_cast<Control<N>*>(ring_bytes + p.stages * stage_bytes);
    const uint32_t bar_full = smem_u32(control.full);
    const uint32_t bar_empty = smem_u32(control.empty);
    const uint32_t bar_query = smem_u32(&control.query);
    const uint32_t bar_scores = smem_u32(control.scores);
    const uint32_t bar_weights = smem_u32(control.weights);
    const uint32_t bar_product = smem_u32(control.product);
    pdl_launch_dependents();
    if (threadIdx.x == 0) {
        tma_prefetch_descriptor(&absorbed_map);
        tma_prefetch_descriptor(&rotated_map);
        tma_prefetch_descriptor(&latent_map);
        tma_prefetch_descriptor(&key_map);
        for (uint32_t stage = 0; stage < p.stages; ++stage) {
            mbar_init(bar_full + 8 * stage, 1);
            mbar_init(bar_empty + 8 * stage, 1);
        }
        mbar_init(bar_query, 1);
        for (uint32_t buffer = 0; buffer < 2; ++buffer) {
            mbar_init(bar_scores + 8 * buffer, 1);
            mbar_init(bar_weights + 8 * buffer, 4);
            mbar_init(bar_product + 8 * buffer, 1);
            control.failed[buffer] = 0;
        }
        control.abort = 0;
        control.missing_page = 0;
        fence_barrier_init();
        fence_proxy_async_smem();
    }
    if (threadIdx.x < N) {
        control.reference[threadIdx.x] = -INFINITY;
        control.total[threadIdx.x] = 0.0f;
    }
    if (warp == 1) {
        tmem_allocate(smem_u32(&control.tmem), p.tmem_columns);
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(&control.tmem);
    const uint32_t tmem_out = tmem_base + 2 * N;
    pdl_wait();

    const uint32_t split = blockIdx.x % p.splits;
    const uint32_t head0 = blockIdx.x / p.splits % p.head_blocks * N;
    const uint32_t token = blockIdx.x / p.splits / p.head_blocks;
    const size_t table_row = p.request_slots[token];
    const uint32_t position = p.positions[token];
    const bool valid = table_row < p.block_table_rows && position / kPageSize < p.block_table_stride;
    const uint32_t pages = valid ? position / kPageSize + 1 : 0;
    const uint32_t* __restrict__ table = p.block_tables + (valid ? table_row * p.block_table_stride : 0);
    const uint32_t all_stages = (pages + kPagesPerStage - 1) / kPagesPerStage;
    // this CTA's stages: split, split + splits, ...
    const uint32_t count = all_stages > split ? (all_stages - split + p.splits - 1) / p.splits : 0;
    auto pages_of = [&](uint32_t index) -> uint32_t {
        return min(kPagesPerStage, pages - (split + index * p.splits) * kPagesPerStage);
    };
    auto fail = [&](uint32_t where) {
        if (!control.abort) {
            control.abort = 1;
            record_wait_timeout(p.status, kTagLatentAttention, (blockIdx.x << 2) | where);
        }
    };

    if (warp == 0) {
        // ------------------------------------------------------------------------------------ producer
        if (count > 0) {
            if (lane == 0) {
                mbar_arrive_expect_tx(bar_query, p.chunks * N * 128);
                for (uint32_t chunk = 0; chunk < p.chunks; ++chunk) {
                    const bool latent = chunk < p.latent_chunks;
                    const uint32_t x = (latent ? chunk : chunk - p.latent_chunks) * 64;
                    load_queries(q_base + chunk * N * 128, latent ? &absorbed_map : &rotated_map, bar_query,
                                 static_cast<int32_t>(x), static_cast<int32_t>(head0), static_cast<int32_t>(token));
                }
            }
            __syncwarp();
            uint32_t issued = 0;
            uint32_t next_entry = lane < pages_of(0) ? __ldg(table + split * kPagesPerStage + lane) : 0;
            for (uint32_t index = 0; index < count; ++index) {
                const uint32_t stage = index % p.stages;
                const uint32_t present = pages_of(index);
                uint32_t entry = next_entry;
                if (index + 1 < count) {
                    const uint32_t first = (split + (index + 1) * p.splits) * kPagesPerStage;
                    next_entry = lane < pages_of(index + 1) ? __ldg(table + first + lane) : 0;
                }
                bool ready = control.abort == 0;
                if (ready && index >= p.stages) {
                    ready = mbar_wait_bounded(bar_empty + 8 * stage, ((index / p.stages) - 1) & 1, p.wait_limit);
                }
                if (!__all_sync(0xffffffffu, ready)) {
                    if (lane == 0) fail(1);
                    break;
                }
                // a page that does not exist is flagged and read as page 0, so that the pipeline stays uniform
                if (lane < present && entry >= p.num_pages) {
                    control.missing_page = 1;
                    entry = 0;
                }
                const uint32_t bar = bar_full + 8 * stage;
                if (lane == 0) mbar_arrive_expect_tx(bar, present * p.chunks * kBoxBytes);
                __syncwarp();
                const uint32_t target = ring + stage * stage_bytes;
                for (uint32_t first = 0; first < present * p.chunks; first += 32) {
                    const uint32_t item = first + lane;
                    const uint32_t page = item / p.chunks;          // page-major: a page's latent is contiguous in memory
                    const uint32_t chunk = item - page * p.chunks;
                    const uint32_t row = __shfl_sync(0xffffffffu, entry, page & 31) * kPageSize;
                    if (page < present) {
                        const bool latent = chunk < p.latent_chunks;
                        const uint32_t x = (latent ? chunk : chunk - p.latent_chunks) * 64;
                        tma_load_2d(target + chunk * kChunkBytes + page * kBoxBytes, latent ? &latent_map : &key_map, bar,
                                    static_cast<int32_t>(x), static_cast<int32_t>(row));
                    }
                }
                issued = index + 1;
            }
            // nobody leaves while copies are in flight
            mbar_wait_bounded(bar_query, 0, p.wait_limit);
            for (uint32_t index = issued > p.stages ? issued - p.stages : 0; index < issued; ++index) {
                mbar_wait_bounded(bar_full + 8 * (index % p.stages), (index / p.stages) & 1, p.wait_limit);
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------------------------------ MMA issuer
        if (lane == 0 && count > 0) {
            // D = f32, A = B = bf16.  S^T: M = 64, both K-major; O^T: M = 128, A (the latents) MN-major
            const uint32_t idesc_common = (1u << 4) | (1u << 7) | (1u << 10) | ((N >> 3) << 17);
            const uint32_t idesc_scores = idesc_common | ((64u >> 4) << 24);
            const uint32_t idesc_out = idesc_common | (1u << 15) | ((128u >> 4) << 24);
            bool ok = mbar_wait_bounded(bar_query, 0, p.wait_limit);
            auto issue_scores = [&](uint32_t index) -> bool {
                const uint32_t stage = index % p.stages;
                if (control.abort || !mbar_wait_bounded(bar_full + 8 * stage, (index / p.stages) & 1, p.wait_limit)) {
                    return false;
                }
                tcgen05_fence_after();
                const uint32_t target = tmem_base + (index & 1) * N;
                for (uint32_t chunk = 0; chunk < p.chunks; ++chunk) {
                    const uint64_t k_desc = smem_descriptor(ring + stage * stage_bytes + chunk * kChunkBytes);
                    const uint64_t q_desc = smem_descriptor(q_base + chunk * N * 128);
#pragma unroll
                    for (uint32_t ks = 0; ks < 4; ++ks) {   // 16 dimensions = 32 bytes inside the swizzled row per step
                        mma_shared(target, k_desc + ks * 2, q_desc + ks * 2, idesc_scores, chunk + ks);
                    }
                }
                umma_commit(bar_scores + 8 * (index & 1));
                return true;
            };
            ok = ok && issue_scores(0);
            for (uint32_t index = 0; index < count && ok; ++index) {
                const uint32_t stage = index % p.stages;
                const uint32_t buffer = index & 1;
                const uint32_t present = pages_of(index);
                // the next stage's scores first: the tensor core computes them while this stage's softmax runs
                if (index + 1 < count && !issue_scores(index + 1)) {
                    ok = false;
                    break;
                }
                if (control.abort || !mbar_wait_bounded(bar_weights + 8 * buffer, (index >> 1) & 1, p.wait_limit)) {
                    ok = false;
                    break;
                }
                tcgen05_fence_after();
                const uint64_t high = smem_descriptor(p_base + buffer * 2 * N * 128);
                const uint64_t low = smem_descriptor(p_base + (buffer * 2 + 1) * N * 128);
                for (uint32_t block = 0; block < p.blocks; ++block) {
                    const uint32_t target = tmem_out + block * N;
                    for (uint32_t step = 0; step < present; ++step) {    // one page of 16 keys
                        const uint64_t v_desc = transposed_descriptor(ring + stage * stage_bytes +
                                                                      2 * block * kChunkBytes + step * kBoxBytes);
                        mma_shared(target, v_desc, high + step * 2, idesc_out, index + step);
                        mma_shared(target, v_desc, low + step * 2, idesc_out, 1);
                    }
                }
                umma_commit(bar_product + 8 * buffer);
                umma_commit(bar_empty + 8 * stage);
            }
            if (!ok) fail(2);
        }
    } else {
        // ------------------------------------------------------------------------------------ softmax / output
        const uint32_t quadrant = warp & 3;                 // the tensor-memory lanes this warp may touch
        const uint32_t lane_address = (quadrant * 32) << 16;
        const uint32_t thread = threadIdx.x - 64;           // 0..127
        const uint32_t key = quadrant * 16 + (lane & 15);   // of the stage; lanes 16 .. 31 hold nothing
        const float scale_log2 = p.scale * kLog2e;
        float sum[N];
#pragma unroll
        for (uint32_t head = 0; head < N; ++head) sum[head] = 0.0f;
        bool ok = true;
        for (uint32_t index = 0; index < count; ++index) {
            const uint32_t stage = index % p.stages;
            const uint32_t buffer = index & 1;
            ok = ok && !control.abort && mbar_wait_bounded(bar_scores + 8 * buffer, (index >> 1) & 1, p.wait_limit);
            if (!ok) control.failed[buffer] = 1;
            tcgen05_fence_after();
            __syncwarp();
            const uint32_t stage_first = (split + index * p.splits) * kKeys;
            const bool visible = lane < 16 && stage_first + key <= position;
            float score[N];
#pragma unroll
            for (uint32_t part = 0; part < N / 16; ++part) {
                uint32_t raw[16];
                tmem_load16_nowait(tmem_base + lane_address + buffer * N + part * 16, raw);
                tmem_load_wait();
#pragma unroll
                for (uint32_t i = 0; i < 16; ++i) {
                    score[part * 16 + i] = visible ? __uint_as_float(raw[i]) * scale_log2 : -INFINITY;
                }
            }
            bool over = false;
#pragma unroll
            for (uint32_t head = 0; head < N; ++head) over |= score[head] > control.reference[head] + kSlack;
            // whatever happened above, all four warps meet here; the flag of this parity is written before the barrier
            // only, so that all of them leave the loop together
            over = softmax_any(over);
            if (control.failed[buffer]) {
                ok = false;
                break;
            }
            if (over) {
#pragma unroll
                for (uint32_t head = 0; head < N; ++head) {
                    float best = score[head];
#pragma unroll
                    for (uint32_t delta = 8; delta > 0; delta >>= 1) {
                        best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, delta));
                    }
                    if (lane == 0) control.warp_max[quadrant][head] = best;
                }
                softmax_barrier();
                if (thread < N) {
                    const float before = control.reference[thread];
                    float now = before;
#pragma unroll
                    for (uint32_t w = 0; w < 4; ++w) now = fmaxf(now, control.warp_max[w][thread]);
                    control.reference[thread] = now;
                    control.factor[thread] = now == before ? 1.0f : fast_exp2(before - now);
                }
                softmax_barrier();
#pragma unroll
                for (uint32_t head = 0; head < N; ++head) sum[head] *= control.factor[head];
                if (index > 0) {
                    ok = mbar_wait_bounded(bar_product + 8 * ((index - 1) & 1), ((index - 1) >> 1) & 1, p.wait_limit);
                    tcgen05_fence_after();
                    __syncwarp();
                    for (uint32_t block = 0; block < p.blocks; ++block) {
#pragma unroll
                        for (uint32_t part = 0; part < N / 16; ++part) {
                            const uint32_t address = tmem_out + lane_address + block * N + part * 16;
                            uint32_t raw[16];
                            tmem_load16_nowait(address, raw);
                            tmem_load_wait();
#pragma unroll
                            for (uint32_t i = 0; i < 16; ++i) {
                                raw[i] = __float_as_uint(__uint_as_float(raw[i]) * control.factor[part * 16 + i]);
                            }
                            tmem_store16(address, raw);
                        }
                    }
                    tmem_store_wait();
                }
            }
            // the weights of two stages before have been consumed
            if (index >= 2) {
                ok = mbar_wait_bounded(bar_product + 8 * buffer, ((index >> 1) - 1) & 1, p.wait_limit) && ok;
            }
            uint8_t* high_rows = smem + p.chunks * N * 128 + buffer * 2 * N * 128;
            uint8_t* low_rows = high_rows + N * 128;
#pragma unroll
            for (uint32_t head = 0; head < N; ++head) {
                const float weight = visible ? fast_exp2(score[head] - control.reference[head]) : 0.0f;
                sum[head] += weight;
                const __nv_bfloat16 high = __float2bfloat16_rn(weight);
                const __nv_bfloat16 low = __float2bfloat16_rn(weight - __bfloat162float(high));
                if (lane < 16) {
                    const uint32_t at = head * 128 + ((key * 2) ^ ((head & 7) << 4));
                    *reinterpret_cast<__nv_bfloat16*>(high_rows + at) = high;
                    *reinterpret_cast<__nv_bfloat16*>(low_rows + at) = low;
                }
            }
            // latents behind the last key may hold anything: clear them (a zero weight times a NaN pattern is NaN)
            if (stage_first + kKeys > position + 1) {
                const uint32_t exists = position + 1 - stage_first;
                const uint32_t rows = pages_of(index) * kPageSize - exists;
                for (uint32_t item = thread; item < rows * p.latent_chunks * 8; item += 128) {
                    const uint32_t chunk = item / (rows * 8);
                    const uint32_t row = exists + item / 8 % rows;
                    *reinterpret_cast<uint4*>(ring_bytes + stage * stage_bytes + chunk * kChunkBytes + row * 128 +
                                              item % 8 * 16) = make_uint4(0, 0, 0, 0);
                }
            }
            fence_proxy_async_smem();
            tcgen05_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_weights + 8 * buffer);
        }
        if (count > 0) {
            const uint32_t last = count - 1;
            ok = ok && mbar_wait_bounded(bar_product + 8 * (last & 1), (last >> 1) & 1, p.wait_limit);
            if (!__all_sync(0xffffffffu, ok)) {
                if (lane == 0) fail(3);
            }
            tcgen05_fence_after();
#pragma unroll
            for (uint32_t head = 0; head < N; ++head) {
                const float total = warp_sum(sum[head]);
                if (lane == 0) control.warp_sum[quadrant][head] = total;
            }
            softmax_barrier();
            if (thread < N) {
                float total = 0.0f;
#pragma unroll
                for (uint32_t w = 0; w < 4; ++w) total += control.warp_sum[w][thread];
                control.total[thread] = total;
            }
            softmax_barrier();
            const bool write = control.abort == 0 && control.missing_page == 0;
            float* result = reinterpret_cast<float*>(ring_bytes);        // [head][kv_rank]; every stage has been consumed
            __syncwarp();
            for (uint32_t block = 0; block < p.blocks; ++block) {
                const uint32_t dim = block * 128 + quadrant * 32 + lane;
#pragma unroll
                for (uint32_t part = 0; part < N / 16; ++part) {
                    uint32_t raw[16];
                    tmem_load16_nowait(tmem_out + lane_address + block * N + part * 16, raw);
                    tmem_load_wait();
#pragma unroll
                    for (uint32_t i = 0; i < 16; ++i) {
                        const uint32_t head = part * 16 + i;
                        const float value = __uint_as_float(raw[i]);
                        if (dim < p.kv_rank && write) {
                            if (p.splits > 1) {
                                result[head * p.kv_rank + dim] = value;
                            } else if (head0 + head < p.heads) {
                                p.out[(static_cast<size_t>(token) * p.heads + head0 + head) * p.kv_rank + dim] =
                                    __float2bfloat16_rn(value / control.total[head]);
                            }
                        }
                    }
                }
            }
        }
    }

    // the producer and MMA warps ran parts of their loops on one lane: the warp meets again here
    __syncwarp();
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tmem_free(tmem_base, p.tmem_columns);
    }
    if (p.splits == 1) {
        return;
    }
    // ---- splits of the token: every CTA of the cluster finishes a share of the outputs
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    bool usable = true;
    for (uint32_t rank = 0; rank < p.splits; ++rank) {
        const Control<N>* other = cluster.map_shared_rank(&control, rank);
        usable = usable && other->abort == 0 && other->missing_page == 0;
    }
    const uint32_t heads = min(N, p.heads - head0);
    for (uint32_t item = threadIdx.x * p.splits + split; usable && item < heads * p.kv_rank; item += kThreads * p.splits) {
        const uint32_t head = item / p.kv_rank;
        float best = -INFINITY;
        for (uint32_t rank = 0; rank < p.splits; ++rank) {
            best = fmaxf(best, cluster.map_shared_rank(&control, rank)->reference[head]);
        }
        float total = 0.0f, value = 0.0f;
        for (uint32_t rank = 0; rank < p.splits; ++rank) {
            const Control<N>* other = cluster.map_shared_rank(&control, rank);
            const float reference = other->reference[head];
            if (reference != -INFINITY) {       // the split saw keys
                const float factor = fast_exp2(reference - best);
                total = fmaf(other->total[head], factor, total);
                value = fmaf(cluster.map_shared_rank(reinterpret_cast<float*>(ring_bytes), rank)[item], factor, value);
            }
        }
        if (total > 0.0f) {
            p.out[(static_cast<size_t>(token) * p.heads + head0) * p.kv_rank + item] = __float2bfloat16_rn(value / total);
        }
    }
    cluster.sync();           // nobody leaves while its results are being read
}

// (dimensions, heads, tokens) in boxes of 64 x `heads_per_box` x 1
bool make_query_map(CUtensorMap* map, const void* base, size_t size, size_t heads, size_t tokens, size_t head_pitch,
                    size_t token_pitch, uint32_t heads_per_box) {
    EncodeTiledFn encode = encode_tiled_entry();
    if (encode == nullptr) {
        return false;
    }
    const cuuint64_t dims[3] = {size, heads, tokens};
    const cuuint64_t strides[2] = {head_pitch * 2, token_pitch * 2};
    const cuuint32_t box[3] = {64, heads_per_box, 1};
    const cuuint32_t element_strides[3] = {1, 1, 1};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, element_strides,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

uint32_t chunks_of(uint32_t size) { return (size + 63) / 64; }

// Ring slots that fit beside the queries and the weights of N heads; 0: not even two.
template <uint32_t N>
uint32_t stages_for(const LatentAttentionShape& shape) {
    const uint32_t chunks = chunks_of(shape.kv_rank) + chunks_of(shape.rot_dim);
    uint32_t stages = kMaxStages;
    while (stages >= 2 && shared_bytes<N>(chunks, stages) > kSharedLimit) --stages;
    return stages >= 2 ? stages : 0;
}

template <uint32_t N>
cudaError_t launch_heads(cudaStream_t stream, const LatentAttentionLaunch& launch) {
    const LatentAttentionShape& shape = launch.shape;
    const auto* query = static_cast<const __nv_bfloat16*>(launch.query);
    const size_t rows = launch.num_pages * kPageSize;
    CUtensorMap absorbed_map, rotated_map, latent_map, key_map;
    if (!make_query_map(&absorbed_map, launch.absorbed, shape.kv_rank, shape.heads, launch.tokens, shape.kv_rank,
                        static_cast<size_t>(shape.heads) * shape.kv_rank, N) ||
        !make_query_map(&rotated_map, query + shape.dim, shape.rot_dim, shape.heads, launch.tokens,
                        shape.dim + shape.rot_dim, launch.query_pitch, N) ||
        !make_swizzled_2d_map_width(&latent_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, launch.latent_cache, rows,
                                    shape.kv_rank, static_cast<size_t>(shape.kv_rank) * 2, kPageSize) ||
        !make_swizzled_2d_map_width(&key_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, launch.key_cache, rows, shape.rot_dim,
                                    static_cast<size_t>(shape.rot_dim) * 2, kPageSize)) {
        return cudaErrorInvalidValue;
    }
    Params params;
    params.heads = shape.heads;
    params.kv_rank = shape.kv_rank;
    params.scale = shape.scale;
    params.block_tables = launch.block_tables;
    params.block_table_stride = launch.block_table_stride;
    params.block_table_rows = launch.block_table_rows;
    params.num_pages = launch.num_pages;
    params.request_slots = launch.request_slots;
    params.positions = launch.positions;
    params.out = static_cast<__nv_bfloat16*>(launch.out);
    params.status = launch.status;
    params.latent_chunks = chunks_of(shape.kv_rank);
    params.chunks = params.latent_chunks + chunks_of(shape.rot_dim);
    params.blocks = (shape.kv_rank + 127) / 128;
    params.head_blocks = (shape.heads + N - 1) / N;
    params.splits = latent_attention_splits(launch.tokens * params.head_blocks, launch.context);
    params.stages = stages_for<N>(shape);
    params.tmem_columns = 32;
    while (params.tmem_columns < (2 + params.blocks) * N) params.tmem_columns *= 2;
    params.wait_limit = wait_limit_ns();
    const size_t shared = shared_bytes<N>(params.chunks, params.stages);
    const auto kernel = latent_attention_umma_kernel<N>;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
    if (status != cudaSuccess) return status;
    const size_t blocks = launch.tokens * params.head_blocks * params.splits;
    return launch_kernel(kernel, static_cast<unsigned int>(blocks), kThreads, shared, stream, params.splits, absorbed_map,
                         rotated_map, latent_map, key_map, params);
}

}  // namespace

// CTAs per token and block of heads over the key axis: enough to even out unequal contexts over the machine while every
// CTA keeps four stages of the longest one.
uint32_t latent_attention_splits(size_t ctas, size_t context) {
    const size_t stages = (context + kKeys - 1) / kKeys;
    uint32_t splits = 1;
    while (splits < kMaxSplits && ctas * splits * 2 <= 4 * 148 && stages >= 4 * splits * 2) splits *= 2;
    return splits;
}

bool latent_attention_umma_supports(const LatentAttentionLaunch& launch) {
    const LatentAttentionShape& shape = launch.shape;
    return launch.type == Activation::kBf16 && launch.status != nullptr && shape.scale > 0.0f && shape.kv_rank <= 512 &&
           shape.rot_dim <= 128 && shape.kv_rank % 8 == 0 && shape.rot_dim % 8 == 0 && shape.dim % 8 == 0 &&
           launch.query_pitch % 8 == 0 && aligned_to(launch.absorbed, 16) && aligned_to(launch.query, 16) &&
           aligned_to(launch.latent_cache, 16) && aligned_to(launch.key_cache, 16) &&
           launch.num_pages * kPageSize <= 0x7fffffffu && stages_for<16>(shape) > 0;
}

cudaError_t launch_latent_attention_umma(cudaStream_t stream, const LatentAttentionLaunch& launch) {
    // as many heads per CTA as there are and as fit: the cache is read once per block of heads
    if (launch.shape.heads > 32 && stages_for<64>(launch.shape) > 0 &&
        (2 + (launch.shape.kv_rank + 127) / 128) * 64 <= 512) {
        return launch_heads<64>(stream, launch);
    }
    if (launch.shape.heads > 16 && stages_for<32>(launch.shape) > 0) {
        return launch_heads<32>(stream, launch);
    }
    return launch_heads<16>(stream, launch);
}

}  // namespace lfm25
