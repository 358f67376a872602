// Attention against cached latents on the 5th-generation tensor cores (tcgen05 + tensor memory), for bf16 activations: one
// query token, any number of heads, latents of up to 512 and rotated parts of up to 128 dimensions.
//
// All heads read the same latent and the same rotated key, so the keys take the 64 or 128 rows of an MMA and the heads its
// columns: a CTA owns one token, up to 64 heads (16, 32 or 64 columns) and a share of the visible keys.
//   warp 0      producer: the queries once, then the keys in stages of 64 (4 pages).  A stage holds the latents in groups of
//               8 keys, each group in chunks of 64 dimensions (1 KiB, 128-byte swizzle), so that all whole chunks of a page
//               arrive in one copy; behind them the rotated keys, chunk by chunk
//   warp 1      tensor memory and the MMAs: S^T [64 keys, heads] = K Q^T over all chunks, then O^T [kv_rank, heads] +=
//               latent^T P^T over the same shared memory, now read with the latent dimensions as rows
//   others      one key per thread (lanes 0 .. 15; two or four warps share a quadrant of tensor memory and divide the heads
//               among them): mask and softmax weights in f32.  The weights are taken against a reference that follows the
//               running maximum only when it falls more than 2^8 behind; then the accumulators in tensor memory are rescaled
// The weights enter the second product as a sum of two bf16 values (16 significant bits), the two parts as neighbouring
// columns of one MMA; sums and accumulators are f32.  The splits of a token merge through the distributed shared memory of
// their cluster.
#include <cooperative_groups.h>
#include <cuda.h>
#include <math.h>

#include <algorithm>
#include <type_traits>

#include "launch.h"
#include "options.h"
#include "stack_latent.h"
#include "tcgen05.cuh"
#include "tensor_map.h"

namespace lfm25 {

namespace {

namespace cg = cooperative_groups;

// Warps that share a quadrant of tensor memory, by the number of heads of a CTA
constexpr __host__ __device__ uint32_t sharing_warps(uint32_t heads) { return heads <= 16 ? 2 : 4; }
constexpr __host__ __device__ uint32_t softmax_threads(uint32_t heads) { return sharing_warps(heads) * 128; }
constexpr __host__ __device__ uint32_t cta_threads(uint32_t heads) { return 64 + softmax_threads(heads); }
constexpr uint32_t kPagesPerStage = 4;
constexpr uint32_t kKeys = kPagesPerStage * kPageSize;       // 64
constexpr uint32_t kGroupKeys = 8;
constexpr uint32_t kGroups = kKeys / kGroupKeys;             // of a stage
constexpr uint32_t kChunkBytes = kGroupKeys * 128;           // one group, 64 dimensions
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
    const uint32_t* token_order;
    __nv_bfloat16* out;
    unsigned int* status;
    uint32_t whole_chunks;               // chunks of 64 latent dimensions that are full
    uint32_t latent_chunks, chunks;      // chunks of the latent, and of a key altogether
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
    // what every split of the token tells the others
    float split_reference[kMaxSplits][N], split_total[kMaxSplits][N];
    uint32_t split_unusable[kMaxSplits];
    float share[kMaxSplits][N];     // what a split's result counts for
    uint64_t full[kMaxStages], empty[kMaxStages];
    uint64_t query, scores[2], weights[2], product[2];
    uint32_t tmem;
    volatile uint32_t abort;
    volatile uint32_t missing_page;
    volatile uint32_t failed[2];
};

template <uint32_t N>
constexpr size_t shared_bytes(uint32_t chunks, uint32_t stages) {
    return 1024 + static_cast<size_t>(chunks) * N * 128 + 4 * N * 128 +
           static_cast<size_t>(stages) * chunks * kGroups * kChunkBytes + sizeof(Control<N>);
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

__device__ __forceinline__ void load_3d(uint32_t dst, const void* tensor_map, uint32_t bar, int32_t x, int32_t y,
                                        int32_t z) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
        ::"r"(dst), "l"(reinterpret_cast<uint64_t>(tensor_map)), "r"(bar), "r"(x), "r"(y), "r"(z)
        : "memory");
}

__device__ __forceinline__ void load_4d(uint32_t dst, const void* tensor_map, uint32_t bar, int32_t x, int32_t y, int32_t z,
                                        int32_t w) {
    asm volatile(
        "cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes "
        "[%0], [%1, {%3, %4, %5, %6}], [%2];"
        ::"r"(dst), "l"(reinterpret_cast<uint64_t>(tensor_map)), "r"(bar), "r"(x), "r"(y), "r"(z), "r"(w)
        : "memory");
}

// Operand with 128-byte swizzle whose 8-line groups are `group_bytes` apart.  K-major (lines are rows): `leading_bytes` is
// not used.  MN-major (a line holds 64 rows at one k): the next 64 rows lie `leading_bytes` further on.
__device__ __forceinline__ uint64_t descriptor(uint32_t address, uint32_t group_bytes, uint32_t leading_bytes) {
    uint64_t value = static_cast<uint64_t>((address & 0x3ffff) >> 4);
    value |= static_cast<uint64_t>(leading_bytes >> 4) << 16;
    value |= static_cast<uint64_t>(group_bytes >> 4) << 32;
    value |= static_cast<uint64_t>(1) << 46;
    value |= static_cast<uint64_t>(2) << 61;
    return value;
}

// Barrier of the softmax warps
template <uint32_t THREADS>
__device__ __forceinline__ void softmax_barrier() {
    __syncwarp();
    asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory");
}
template <uint32_t THREADS>
__device__ __forceinline__ bool softmax_any(bool mine) {
    __syncwarp();
    uint32_t any;
    asm volatile(
        "{\n"
        ".reg .pred p, q;\n"
        "setp.ne.u32 p, %1, 0;\n"
        "bar.red.or.pred q, 1, %2, p;\n"
        "selp.u32 %0, 1, 0, q;\n"
        "}\n"
        : "=r"(any)
        : "r"(mine ? 1u : 0u), "n"(THREADS)
        : "memory");
    return any != 0;
}

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.aligned;" ::: "memory"); }

template <uint32_t N>
__global__ void __launch_bounds__(cta_threads(N), 1)
latent_attention_umma_kernel(const __grid_constant__ CUtensorMap absorbed_map,
                             const __grid_constant__ CUtensorMap rotated_map,
                             const __grid_constant__ CUtensorMap latent_map,
                             const __grid_constant__ CUtensorMap tail_map,
                             const __grid_constant__ CUtensorMap key_map, const Params p) {
    constexpr uint32_t kSharing = sharing_warps(N);
    constexpr uint32_t kShare = N / kSharing;       // heads per softmax thread
    constexpr uint32_t kSoftmax = softmax_threads(N);
    constexpr uint32_t kThreads = cta_threads(N);
    const uint32_t warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0);     // the same value to the compiler's eye as well
    const uint32_t lane = threadIdx.x & 31;
    extern __shared__ uint8_t latent_smem[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(latent_smem) + 1023) & ~uintptr_t(1023));
    const uint32_t group_bytes = p.latent_chunks * kChunkBytes;
    const uint32_t stage_bytes = kGroups * p.chunks * kChunkBytes;
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
        for (uint32_t stage = 0; stage < p.stages; ++stage) {
            mbar_init(bar_full + 8 * stage, 1);
            mbar_init(bar_empty + 8 * stage, 1);
        }
        mbar_init(bar_query, 1);
        for (uint32_t buffer = 0; buffer < 2; ++buffer) {
            mbar_init(bar_scores + 8 * buffer, 1);
            mbar_init(bar_weights + 8 * buffer, kSoftmax / 32);
            mbar_init(bar_product + 8 * buffer, 1);
            control.failed[buffer] = 0;
        }
        control.abort = 0;
        control.missing_page = 0;
        fence_barrier_init();
        fence_proxy_async_smem();
        tma_prefetch_descriptor(&absorbed_map);
        tma_prefetch_descriptor(&rotated_map);
        tma_prefetch_descriptor(&latent_map);
        tma_prefetch_descriptor(&key_map);
    }
    if (threadIdx.x >= 64 && threadIdx.x < 64 + N) {
        control.reference[threadIdx.x - 64] = -INFINITY;
        control.total[threadIdx.x - 64] = 0.0f;
    }
    if (warp == 1) {
        tmem_allocate(smem_u32(&control.tmem), p.tmem_columns);
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    // a CTA writes into the others' shared memory at its end, which may come before they have started
    if (p.splits > 1) cluster_arrive();
    const uint32_t tmem_base = __shfl_sync(0xffffffffu, *reinterpret_cast<volatile uint32_t*>(&control.tmem), 0);
    const uint32_t tmem_out = tmem_base + 2 * N;                 // [block][high heads | low heads]
    pdl_wait();

    const uint32_t split = blockIdx.x % p.splits;
    const uint32_t head0 = blockIdx.x / p.splits % p.head_blocks * N;
    const uint32_t rank = blockIdx.x / p.splits / p.head_blocks;
    const uint32_t token = p.token_order != nullptr ? p.token_order[rank] : rank;
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
            // lane: page of the stage and what it copies of it -- the whole chunks of the latents (group by group where a
            // partial chunk follows them), that partial chunk, the rotated part (up to two chunks)
            const uint32_t page = lane & 3;
            const uint32_t part = lane >> 2;
            const bool partial = p.latent_chunks > p.whole_chunks;
            const bool copies = part < 2   ? p.whole_chunks > 0 && (part == 0 || partial)
                                : part < 4 ? partial
                                           : part - 4 < p.chunks - p.latent_chunks;
            const uint32_t offset =
                part < 2   ? (page * 2 + part) * group_bytes
                : part < 4 ? (page * 2 + part - 2) * group_bytes + p.whole_chunks * kChunkBytes
                           : kGroups * group_bytes + (part - 4) * kGroups * kChunkBytes + page * 2 * kChunkBytes;
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
                if (lane == 0) mbar_arrive_expect_tx(bar, present * 2 * p.chunks * kChunkBytes);
                const uint32_t source = __shfl_sync(0xffffffffu, entry, page);
                if (copies && page < present) {
                    const int32_t row = static_cast<int32_t>(source * kPageSize);
                    const uint32_t target = ring + stage * stage_bytes + offset;
                    if (part < 2) {
                        load_4d(target, &latent_map, bar, 0, 0, 0,
                                row / static_cast<int32_t>(kGroupKeys) + static_cast<int32_t>(part));
                    } else if (part < 4) {
                        tma_load_2d(target, &tail_map, bar, 0, row + static_cast<int32_t>((part - 2) * kGroupKeys));
                    } else {
                        tma_load_2d(target, &key_map, bar, static_cast<int32_t>((part - 4) * 64), row);
                    }
                }
                __syncwarp();
                if (index == 0 && lane == 0) {
                    mbar_arrive_expect_tx(bar_query, p.chunks * N * 128);
                    for (uint32_t chunk = 0; chunk < p.chunks; ++chunk) {
                        const bool latent = chunk < p.latent_chunks;
                        const uint32_t x = (latent ? chunk : chunk - p.latent_chunks) * 64;
                        load_3d(q_base + chunk * N * 128, latent ? &absorbed_map : &rotated_map, bar_query,
                                static_cast<int32_t>(x), static_cast<int32_t>(head0), static_cast<int32_t>(token));
                    }
                }
                issued = index + 1;
            }
            // nobody leaves while copies are in flight
            __syncwarp();
            if (issued > 0) mbar_wait_bounded(bar_query, 0, p.wait_limit);
            for (uint32_t index = issued > p.stages ? issued - p.stages : 0; index < issued; ++index) {
                mbar_wait_bounded(bar_full + 8 * (index % p.stages), (index / p.stages) & 1, p.wait_limit);
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------------------------------ MMA issuer
        if (count > 0) {
            const bool issuer = elect_one();
            // D = f32, A = B = bf16.  S^T: M = 64, both K-major; O^T: M = 128, A (the latents) MN-major, the high and low
            // parts of the weights side by side
            const uint32_t idesc_common = (1u << 4) | (1u << 7) | (1u << 10);
            const uint32_t idesc_scores = idesc_common | ((N >> 3) << 17) | ((64u >> 4) << 24);
            const uint32_t idesc_out = idesc_common | (1u << 15) | ((2 * N >> 3) << 17) | ((128u >> 4) << 24);
            bool ok = mbar_wait_bounded(bar_query, 0, p.wait_limit);
            auto issue_scores = [&](uint32_t index) {       // the stage has arrived
                tcgen05_fence_after();
                const uint32_t target = tmem_base + (index & 1) * N;
                const uint32_t stage = ring + index % p.stages * stage_bytes;
                if (issuer) {
                    uint64_t k_desc = descriptor(stage, group_bytes, 16);
                    uint64_t q_desc = descriptor(q_base, 1024, 16);
                    for (uint32_t chunk = 0; chunk < p.chunks; ++chunk) {
                        if (chunk == p.latent_chunks) k_desc = descriptor(stage + kGroups * group_bytes, kChunkBytes, 16);
#pragma unroll
                        for (uint32_t ks = 0; ks < 4; ++ks) {   // 16 dimensions = 32 bytes inside the swizzled row per step
                            mma_shared(target, k_desc + ks * 2, q_desc + ks * 2, idesc_scores, chunk + ks);
                        }
                        k_desc += (chunk < p.latent_chunks ? kChunkBytes : kGroups * kChunkBytes) >> 4;
                        q_desc += N * 128 >> 4;
                    }
                    umma_commit(bar_scores + 8 * (index & 1));
                }
                __syncwarp();
            };
            auto arrived = [&](uint32_t index) -> bool {
                return mbar_wait_bounded(bar_full + 8 * (index % p.stages), (index / p.stages) & 1, p.wait_limit);
            };
            ok = ok && arrived(0);
            ok = __all_sync(0xffffffffu, ok);
            if (ok) issue_scores(0);
            for (uint32_t index = 0; index < count && ok; ++index) {
                const uint32_t stage = index % p.stages;
                const uint32_t buffer = index & 1;
                const uint32_t present = pages_of(index);
                // the next stage's scores first if it is there: the tensor core computes them during this stage's softmax
                bool ahead = false;
                if (index + 1 < count) {
                    ahead = __all_sync(0xffffffffu, mbar_test(bar_full + 8 * ((index + 1) % p.stages),
                                                              ((index + 1) / p.stages) & 1));
                    if (ahead) issue_scores(index + 1);
                }
                ok = control.abort == 0 && mbar_wait_bounded(bar_weights + 8 * buffer, (index >> 1) & 1, p.wait_limit);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                tcgen05_fence_after();
                const uint64_t weights = descriptor(p_base + buffer * 2 * N * 128, 1024, 16);
                uint64_t v_desc = descriptor(ring + stage * stage_bytes, group_bytes, kChunkBytes);
                if (issuer) {
#pragma unroll
                    for (uint32_t step = 0; step < kPagesPerStage; ++step) {    // one page of 16 keys, block after block
                        if (step < present) {
                            for (uint32_t block = 0; block < p.blocks; ++block) {
                                mma_shared(tmem_out + block * 2 * N, v_desc + block * (2 * kChunkBytes >> 4),
                                           weights + step * 2, idesc_out, index + step);
                            }
                        }
                        v_desc += 2 * group_bytes >> 4;
                    }
                    umma_commit(bar_product + 8 * buffer);
                    umma_commit(bar_empty + 8 * stage);
                }
                __syncwarp();
                if (index + 1 < count && !ahead) {
                    ok = __all_sync(0xffffffffu, arrived(index + 1));
                    if (ok) issue_scores(index + 1);
                }
            }
            if (!ok && lane == 0) fail(2);
        }
    } else {
        // ------------------------------------------------------------------------------------ softmax / output
        const uint32_t quadrant = warp & 3;                 // the tensor-memory lanes this warp may touch
        const uint32_t lane_address = (quadrant * 32) << 16;
        const uint32_t thread = threadIdx.x - 64;
        const uint32_t share = thread / 128;                // which part of the heads
        const uint32_t first_head = share * kShare;
        const uint32_t key = quadrant * 16 + (lane & 15);   // of the stage; lanes 16 .. 31 hold nothing
        const float scale_log2 = p.scale * kLog2e;
        float sum[kShare];
#pragma unroll
        for (uint32_t head = 0; head < kShare; ++head) sum[head] = 0.0f;
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
            float score[kShare];
            bool over = false;
#pragma unroll
            for (uint32_t part = 0; part < kShare / 8; ++part) {
                uint32_t raw[8];
                tmem_load8_nowait(tmem_base + lane_address + buffer * N + first_head + part * 8, raw);
                tmem_load_wait();
#pragma unroll
                for (uint32_t i = 0; i < 8; ++i) {
                    const float value = visible ? __uint_as_float(raw[i]) * scale_log2 : -INFINITY;
                    score[part * 8 + i] = value;
                    over |= value > control.reference[first_head + part * 8 + i] + kSlack;
                }
            }
            // whatever happened above, all warps meet here; the flag of this parity is written before the barrier only, so
            // that all of them leave the loop together
            over = softmax_any<kSoftmax>(over);
            if (control.failed[buffer]) {
                ok = false;
                break;
            }
            if (over) {
#pragma unroll
                for (uint32_t head = 0; head < kShare; ++head) {
                    float best = score[head];
#pragma unroll
                    for (uint32_t delta = 8; delta > 0; delta >>= 1) {
                        best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, delta));
                    }
                    if (lane == 0) control.warp_max[quadrant][first_head + head] = best;
                }
                softmax_barrier<kSoftmax>();
                if (thread < N) {
                    const float before = control.reference[thread];
                    float now = before;
#pragma unroll
                    for (uint32_t w = 0; w < 4; ++w) now = fmaxf(now, control.warp_max[w][thread]);
                    control.reference[thread] = now;
                    control.factor[thread] = now == before ? 1.0f : fast_exp2(before - now);
                }
                softmax_barrier<kSoftmax>();
#pragma unroll
                for (uint32_t head = 0; head < kShare; ++head) sum[head] *= control.factor[first_head + head];
                if (index > 0) {
                    ok = mbar_wait_bounded(bar_product + 8 * ((index - 1) & 1), ((index - 1) >> 1) & 1, p.wait_limit);
                    tcgen05_fence_after();
                    __syncwarp();
                    // the high and the low columns of a block, divided among the warps of the quadrant
                    constexpr uint32_t kColumns = 2 * N / kSharing;
                    for (uint32_t block = 0; block < p.blocks; ++block) {
#pragma unroll 1
                        for (uint32_t part = 0; part < kColumns / 16; ++part) {
                            const uint32_t column = share * kColumns + part * 16;
                            const uint32_t address = tmem_out + lane_address + block * 2 * N + column;
                            uint32_t raw[16];
                            tmem_load16_nowait(address, raw);
                            tmem_load_wait();
#pragma unroll
                            for (uint32_t i = 0; i < 16; ++i) {
                                raw[i] = __float_as_uint(__uint_as_float(raw[i]) * control.factor[column % N + i]);
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
            uint8_t* high_rows = smem + p.chunks * N * 128 + buffer * 2 * N * 128 + first_head * 128;
#pragma unroll
            for (uint32_t part = 0; part < kShare / 8; ++part) {
                uint32_t high[4], low[4];
#pragma unroll
                for (uint32_t pair = 0; pair < 4; ++pair) {
                    const uint32_t head = part * 8 + 2 * pair;
                    const float2 reference = *reinterpret_cast<const float2*>(control.reference + first_head + head);
                    const float first = fast_exp2(score[head] - reference.x);       // keys that are not visible: exp2(-inf)
                    const float second = fast_exp2(score[head + 1] - reference.y);
                    sum[head] += first;
                    sum[head + 1] += second;
                    high[pair] = pack_bf16x2(first, second);
                    const float2 rounded = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&high[pair]));
                    low[pair] = pack_bf16x2(first - rounded.x, second - rounded.y);
                }
                if (lane < 16) {
#pragma unroll
                    for (uint32_t i = 0; i < 8; ++i) {
                        // first_head is a multiple of 8, so i is the line of its 8-line group
                        const uint32_t at = (part * 8 + i) * 128 + ((key * 2) ^ (i << 4));
                        const uint32_t shift = i % 2 * 16;
                        *reinterpret_cast<uint16_t*>(high_rows + at) = static_cast<uint16_t>(high[i / 2] >> shift);
                        *reinterpret_cast<uint16_t*>(high_rows + N * 128 + at) = static_cast<uint16_t>(low[i / 2] >> shift);
                    }
                }
            }
            // latents behind the last key may hold anything: clear them (a zero weight times a NaN pattern is NaN)
            if (stage_first + kKeys > position + 1) {
                const uint32_t exists = position + 1 - stage_first;
                const uint32_t rows = pages_of(index) * kPageSize - exists;
                for (uint32_t item = thread; item < rows * p.latent_chunks * 8; item += kSoftmax) {
                    const uint32_t chunk = item / (rows * 8);
                    const uint32_t row = exists + item / 8 % rows;
                    *reinterpret_cast<uint4*>(ring_bytes + stage * stage_bytes + row / kGroupKeys * group_bytes +
                                              chunk * kChunkBytes + row % kGroupKeys * 128 + item % 8 * 16) =
                        make_uint4(0, 0, 0, 0);
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
            __syncwarp();
            // the accumulators as f32 [head][kv_rank] in shared memory: every stage has been consumed
            float* result = reinterpret_cast<float*>(ring_bytes) + first_head * p.kv_rank;
            for (uint32_t block = 0; block < p.blocks; ++block) {
                const uint32_t dim = block * 128 + quadrant * 32 + lane;
#pragma unroll
                for (uint32_t part = 0; part < kShare / 8; ++part) {
                    uint32_t high[8], low[8];
                    const uint32_t address = tmem_out + lane_address + block * 2 * N + first_head + part * 8;
                    tmem_load8_nowait(address, high);
                    tmem_load8_nowait(address + N, low);
                    tmem_load_wait();
                    if (dim < p.kv_rank) {
#pragma unroll
                        for (uint32_t i = 0; i < 8; ++i) {
                            result[(part * 8 + i) * p.kv_rank + dim] = __uint_as_float(high[i]) + __uint_as_float(low[i]);
                        }
                    }
                }
            }
#pragma unroll
            for (uint32_t head = 0; head < kShare; ++head) {
                const float total = warp_sum(sum[head]);
                if (lane == 0) control.warp_sum[quadrant][first_head + head] = total;
            }
            softmax_barrier<kSoftmax>();
            if (thread < N) {
                float total = 0.0f;
#pragma unroll
                for (uint32_t w = 0; w < 4; ++w) total += control.warp_sum[w][thread];
                control.total[thread] = total;
            }
        }
    }

    // the warps meet again here
    __syncwarp();
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tmem_free(tmem_base, p.tmem_columns);
    }
    if (p.splits == 1) {
        const uint32_t quads = p.kv_rank / 4;
        const uint32_t items = min(N, p.heads - head0) * quads;
        const bool usable = count > 0 && control.abort == 0 && control.missing_page == 0;
        for (uint32_t item = threadIdx.x; usable && item < items; item += kThreads) {
            const float share = 1.0f / control.total[item / quads];
            const float4 value = reinterpret_cast<const float4*>(ring_bytes)[item];
            uint2 packed;
            packed.x = pack_bf16x2(value.x * share, value.y * share);
            packed.y = pack_bf16x2(value.z * share, value.w * share);
            *reinterpret_cast<uint2*>(p.out + (static_cast<size_t>(token) * p.heads + head0) * p.kv_rank + item * 4) =
                packed;
        }
        return;
    }
    // ---- splits of the token: every CTA of the cluster finishes a share of the outputs.  First what each split counts
    // for, per head, then the weighted sum of the splits' results, four columns at a time with all loads in flight.
    cg::cluster_group cluster = cg::this_cluster();
    const uint32_t heads = min(N, p.heads - head0);
    cluster_wait();           // all have started
    for (uint32_t item = threadIdx.x; item < heads * p.splits; item += kThreads) {
        const uint32_t head = item % heads;
        Control<N>* other = cluster.map_shared_rank(&control, item / heads);
        other->split_reference[split][head] = control.reference[head];
        other->split_total[split][head] = control.total[head];
        if (head == 0) other->split_unusable[split] = control.abort | control.missing_page;
    }
    cluster.sync();
    bool usable = true;
    for (uint32_t rank = 0; rank < p.splits; ++rank) usable = usable && control.split_unusable[rank] == 0;
    if (threadIdx.x < heads) {
        float reference[kMaxSplits], total[kMaxSplits];
#pragma unroll
        for (uint32_t rank = 0; rank < kMaxSplits; ++rank) {
            reference[rank] = rank < p.splits ? control.split_reference[rank][threadIdx.x] : -INFINITY;
            total[rank] = rank < p.splits ? control.split_total[rank][threadIdx.x] : 0.0f;
        }
        float best = -INFINITY, sum = 0.0f;
#pragma unroll
        for (uint32_t rank = 0; rank < kMaxSplits; ++rank) best = fmaxf(best, reference[rank]);
#pragma unroll
        for (uint32_t rank = 0; rank < kMaxSplits; ++rank) {      // a split that saw no keys counts for nothing
            reference[rank] = reference[rank] == -INFINITY ? 0.0f : fast_exp2(reference[rank] - best);
            sum = fmaf(total[rank], reference[rank], sum);
        }
#pragma unroll
        for (uint32_t rank = 0; rank < kMaxSplits; ++rank) {
            control.share[rank][threadIdx.x] = sum > 0.0f ? reference[rank] / sum : 0.0f;
        }
    }
    __syncthreads();
    const uint32_t quads = p.kv_rank / 4;
    const uint32_t items = heads * quads;
    const uint32_t mine = (items + p.splits - 1) / p.splits;
    const uint32_t last_item = min(items, (split + 1) * mine);
    __nv_bfloat16* target = p.out + (static_cast<size_t>(token) * p.heads + head0) * p.kv_rank;
    auto merge = [&](auto count_tag) {
        constexpr uint32_t kSplits = decltype(count_tag)::value;
        const float4* parts[kSplits];
#pragma unroll
        for (uint32_t rank = 0; rank < kSplits; ++rank) {
            parts[rank] =
                reinterpret_cast<const float4*>(cluster.map_shared_rank(reinterpret_cast<float*>(ring_bytes), rank));
        }
        for (uint32_t item = split * mine + threadIdx.x; item < last_item; item += kThreads) {
            const uint32_t head = item / quads;
            float4 part[kSplits];
#pragma unroll
            for (uint32_t rank = 0; rank < kSplits; ++rank) part[rank] = parts[rank][item];
            float4 value = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (uint32_t rank = 0; rank < kSplits; ++rank) {
                const float share = control.share[rank][head];
                if (share != 0.0f) {                // a split that saw no keys has no result either
                    value.x = fmaf(part[rank].x, share, value.x);
                    value.y = fmaf(part[rank].y, share, value.y);
                    value.z = fmaf(part[rank].z, share, value.z);
                    value.w = fmaf(part[rank].w, share, value.w);
                }
            }
            uint2 packed;
            packed.x = pack_bf16x2(value.x, value.y);
            packed.y = pack_bf16x2(value.z, value.w);
            *reinterpret_cast<uint2*>(target + item * 4) = packed;
        }
    };
    if (usable) {
        if (p.splits == 2) {
            merge(std::integral_constant<uint32_t, 2>());
        } else if (p.splits == 4) {
            merge(std::integral_constant<uint32_t, 4>());
        } else {
            merge(std::integral_constant<uint32_t, 8>());
        }
    }
    cluster.sync();           // nobody leaves while its results are being read
}

// Three dimensions, the innermost contiguous and cut into boxes of 64, the others with pitches in bytes
bool make_3d_map(CUtensorMap* map, const void* base, size_t inner, size_t middle, size_t outer, size_t middle_pitch,
                 size_t outer_pitch, uint32_t box_middle, uint32_t box_outer) {
    EncodeTiledFn encode = encode_tiled_entry();
    if (encode == nullptr) {
        return false;
    }
    const cuuint64_t dims[3] = {inner, middle, outer};
    const cuuint64_t strides[2] = {middle_pitch, outer_pitch};
    const cuuint32_t box[3] = {64, box_middle, box_outer};
    const cuuint32_t element_strides[3] = {1, 1, 1};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, element_strides,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// Rows of `row_bytes` of which `chunks` times 128 bytes are copied: boxes of `groups` groups of 8 rows, ordered by groups,
// then chunks, then rows
bool make_group_map(CUtensorMap* map, const void* base, size_t rows, size_t row_bytes, size_t chunks, uint32_t groups) {
    EncodeTiledFn encode = encode_tiled_entry();
    if (encode == nullptr) {
        return false;
    }
    const cuuint64_t dims[4] = {64, kGroupKeys, chunks, rows / kGroupKeys};
    const cuuint64_t strides[3] = {row_bytes, 128, kGroupKeys * row_bytes};
    const cuuint32_t box[4] = {64, kGroupKeys, static_cast<cuuint32_t>(chunks), groups};
    const cuuint32_t element_strides[4] = {1, 1, 1, 1};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, element_strides,
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
    const uint32_t whole = shape.kv_rank / 64;
    const auto* latents = static_cast<const __nv_bfloat16*>(launch.latent_cache);
    const size_t latent_bytes = static_cast<size_t>(shape.kv_rank) * 2;
    CUtensorMap absorbed_map, rotated_map, latent_map, tail_map, key_map;
    if (!make_3d_map(&absorbed_map, launch.absorbed, shape.kv_rank, shape.heads, launch.tokens, latent_bytes,
                     shape.heads * latent_bytes, N, 1) ||
        !make_3d_map(&rotated_map, query + shape.dim, shape.rot_dim, shape.heads, launch.tokens,
                     static_cast<size_t>(shape.dim + shape.rot_dim) * 2, launch.query_pitch * 2, N, 1) ||
        !make_swizzled_2d_map_width(&key_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, launch.key_cache, rows, shape.rot_dim,
                                    static_cast<size_t>(shape.rot_dim) * 2, kPageSize)) {
        return cudaErrorInvalidValue;
    }
    // the whole chunks of the latents group by group; what is left of them as a matrix of its own
    latent_map = tail_map = key_map;
    if (whole > 0 && !make_group_map(&latent_map, latents, rows, latent_bytes, whole, shape.kv_rank % 64 != 0 ? 1 : 2)) {
        return cudaErrorInvalidValue;
    }
    if (shape.kv_rank % 64 != 0 &&
        !make_swizzled_2d_map_width(&tail_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, latents + whole * 64, rows,
                                    shape.kv_rank % 64, latent_bytes, kGroupKeys)) {
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
    params.token_order = launch.token_order;
    params.out = static_cast<__nv_bfloat16*>(launch.out);
    params.status = launch.status;
    params.whole_chunks = whole;
    params.latent_chunks = chunks_of(shape.kv_rank);
    params.chunks = params.latent_chunks + chunks_of(shape.rot_dim);
    params.blocks = (shape.kv_rank + 127) / 128;
    params.head_blocks = (shape.heads + N - 1) / N;
    params.splits = latent_attention_splits(launch.tokens * params.head_blocks, launch.context, params.latent_chunks);
    params.stages = stages_for<N>(shape);
    params.tmem_columns = 32;
    while (params.tmem_columns < (2 + 2 * params.blocks) * N) params.tmem_columns *= 2;
    params.wait_limit = wait_limit_ns();
    const size_t shared = shared_bytes<N>(params.chunks, params.stages);
    const auto kernel = latent_attention_umma_kernel<N>;
    const cudaError_t status = cudaFuncSetAttribute(reinterpret_cast<const void*>(kernel),
                                                    cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
    if (status != cudaSuccess) return status;
    const size_t blocks = launch.tokens * params.head_blocks * params.splits;
    return launch_kernel(kernel, static_cast<unsigned int>(blocks), cta_threads(N), shared, stream, params.splits,
                         absorbed_map, rotated_map, latent_map, tail_map, key_map, params);
}

}  // namespace

// CTAs per token and block of heads over the key axis.  A CTA costs what several stages of keys cost before and behind its
// own, and the larger a cluster is, the fewer SMs its shape lets the machine use (one CTA per SM; cluster counts as the
// occupancy calculator reports them).  The cheapest split when contexts are half of the longest on average and handed out
// longest first.
uint32_t latent_attention_splits(size_t clusters, size_t context, uint32_t latent_chunks) {
    constexpr size_t kResident[] = {148, 74, 33, 15};            // clusters of 1, 2, 4, 8 CTAs
    const double stages = static_cast<double>((context + kKeys - 1) / kKeys);
    const double overhead = 40.0 / latent_chunks;
    uint32_t best = 1;
    double best_cost = 0.0;
    for (uint32_t step = 0; step < 4; ++step) {
        const uint32_t splits = 1u << step;
        if (splits > 1 && splits > stages) break;
        const size_t waves = (clusters + kResident[step] - 1) / kResident[step];
        const double longest = stages / splits + overhead;
        const double cost = std::max(longest, waves * (stages / (2 * splits) + overhead));
        if (splits == 1 || cost < best_cost) {
            best = splits;
            best_cost = cost;
        }
    }
    return best;
}

bool latent_attention_umma_supports(const LatentAttentionLaunch& launch) {
    const LatentAttentionShape& shape = launch.shape;
    return launch.type == Activation::kBf16 && launch.status != nullptr && shape.scale > 0.0f && shape.kv_rank <= 512 &&
           shape.rot_dim <= 128 && shape.kv_rank % 8 == 0 && shape.rot_dim % 8 == 0 && shape.dim % 8 == 0 &&
           launch.query_pitch % 8 == 0 && aligned_to(launch.absorbed, 16) && aligned_to(launch.query, 16) &&
           aligned_to(launch.latent_cache, 16) && aligned_to(launch.key_cache, 16) && aligned_to(launch.out, 16) &&
           launch.num_pages * kPageSize <= 0x7fffffffu && stages_for<16>(shape) > 0;
}

cudaError_t launch_latent_attention_umma(cudaStream_t stream, const LatentAttentionLaunch& launch) {
    // as many heads per CTA as there are and as fit: the cache is read once per block of heads
    if (launch.shape.heads > 32 && stages_for<64>(launch.shape) > 0 &&
        (2 + 2 * ((launch.shape.kv_rank + 127) / 128)) * 64 <= 512) {
        return launch_heads<64>(stream, launch);
    }
    if (launch.shape.heads > 16 && stages_for<32>(launch.shape) > 0) {
        return launch_heads<32>(stream, launch);
    }
    return launch_heads<16>(stream, launch);
}

}  // namespace lfm25
