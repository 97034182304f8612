// Prefill of a latent attention with the keys and values of every head formed, on the fifth-generation tensor cores:
// the step's sequences all start at their first token, so everything a query sees lies in the step's own packed rows
// and no page table is needed. Per head a key is [D unrotated elements of its own | R rotated ones that all heads share],
// a value V elements:
//     q    [T, ld]: head h's query in columns h (D + R) .. (rotated)
//     kv   [T, H (D + V)]: head h's unrotated key, then its value, in columns h (D + V) ..
//     rows [T, C + R]: the shared rotated key part in the last R columns
// With `sinks` (float32 [H], optional) e^sink is one more term of a head's denominator, without key or value, not scaled.
//
// One block serves 256 queries of one head of one sequence as two tiles of 128 (the rows of tensor memory), which share
// the keys and values that come by TMA in blocks of 64 tokens:
//
// * warp 0, one lane: TMA for the queries (once) and the keys; warp 3, one lane: the values. 64 x 64 boxes with the
//   128-byte swizzle, two buffers each; a buffer is requested again when the products of BOTH tiles that read it are
//   complete. The rotated piece of a key is a box of `rows` (zeros beyond R).
// * warps 1 and 2, one lane each: the products of a tile. S[128 q, 64 keys] = Q K^T over the D + R elements (steps of 16)
//   into one of two score buffers of the tile in tensor memory; O[128 q, V] += P V with P read from tensor memory (over
//   its buffer's scores, as bfloat16) and V from shared memory as an MN-major operand. The scores of the block after the
//   next are issued right behind P V of a block, so that the softmax of one buffer runs under the products of the other.
// * warps 4-7 and 8-11: a thread a query row of a tile. It reads its 64 scores once, keeps the running maximum and sum in
//   32-bit, writes the probabilities, and rescales O in place when its maximum outgrows the exponent's reference by
//   2^8. Keys beyond a query's own position are masked by value; blocks wholly above a tile's diagonal are not computed
//   (its products' lane then only releases the buffers for the other tile).
//
// All waits are bounded by a clock limit and report through the status word of this library.
#include "tc.cuh"

using namespace llmb;
using namespace llmb::tc;

LLMB_DEFINE_LAST_ERROR(llmb_latent_prefill_tc)

namespace {

constexpr int BQ = 128;                 // queries of a tile = lanes of tensor memory
constexpr int TILES = 2;                // tiles of a block
constexpr int BKV = 64;                 // keys per step
constexpr int THREADS = 384;
constexpr int Q_PIECE = BQ * 64 * 2, KV_PIECE = BKV * 64 * 2;
// tensor memory of a tile: two buffers of scores (64 columns each), then O
constexpr uint32_t S_COL = 0, O_COL = 128, TILE_COLS = 256, TMEM_COLS = TILES * TILE_COLS;

__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// D and V: 64 or 128 (one or two 64-column pieces); the rotated part is one piece of up to 64.
template <int D, int V>
__host__ __device__ constexpr size_t smem_bytes() {
    return 1024 + (size_t)TILES * (D / 64 + 1) * Q_PIECE + 2 * (D / 64 + 1) * KV_PIECE + 2 * (V / 64) * KV_PIECE + 32 * 8;
}

template <int D, int V>
__global__ void __launch_bounds__(THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                         const __grid_constant__ CUtensorMap map_r, const int* __restrict__ cu_seqlens,
                         const int* __restrict__ seq_order, __nv_bfloat16* __restrict__ out, int out_stride, int R,
                         float scale_log2, const float* __restrict__ sinks, int* status) {
    constexpr int PIECES = D / 64 + 1, V_PIECES = V / 64;
    constexpr int Q_BYTES = PIECES * Q_PIECE, K_BYTES = PIECES * KV_PIECE, V_BYTES = V_PIECES * KV_PIECE;
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* q_tile = base;                             // [TILES][pieces]
    unsigned char* k_tile = q_tile + TILES * Q_BYTES;         // two buffers
    unsigned char* v_tile = k_tile + 2 * K_BYTES;             // two buffers
    uint64_t* bars = reinterpret_cast<uint64_t*>(v_tile + 2 * V_BYTES);
    uint64_t* k_full = bars;                  // [2]
    uint64_t* k_empty = bars + 2;             // [2] both tiles' Q K^T are complete
    uint64_t* v_full = bars + 4;              // [2]
    uint64_t* v_empty = bars + 6;             // [2] both tiles' P V are complete
    uint64_t* tile_bars = bars + 8;           // per tile: q_full, s_full[2], p_full[2], o_full
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 20);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

    griddep_launch();
    griddep_wait();
    int seq = seq_order ? seq_order[blockIdx.z] : (int)blockIdx.z, head = blockIdx.x;
    int first_token = cu_seqlens[seq];
    int n_new = cu_seqlens[seq + 1] - first_token;
    int n_groups = (n_new + TILES * BQ - 1) / (TILES * BQ);
    if ((int)blockIdx.y >= n_groups) return;                  // uniform for the block: nothing is allocated yet
    int group0 = (n_groups - 1 - blockIdx.y) * TILES * BQ;    // the heaviest first
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // key blocks of a tile (none where it has no query)
    auto blocks_of = [&](int tile) {
        int first = group0 + tile * BQ;
        return first < n_new ? min(first + BQ - 1, n_new - 1) / BKV + 1 : 0;
    };
    int n_blocks = max(blocks_of(0), blocks_of(1));

    if (threadIdx.x == 0) {
        for (int i = 0; i < 8; ++i) mbar_init(smem_u32(&bars[i]), ((i >> 1) & 1) ? TILES : 1);
        for (int t = 0; t < TILES; ++t)
            for (int i = 0; i < 6; ++i) mbar_init(smem_u32(&tile_bars[t * 6 + i]), (i == 3 || i == 4) ? BQ : 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(tmem_slot)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            for (int t = 0; t < TILES; ++t) {
                if (blocks_of(t) == 0) continue;
                uint32_t bar = smem_u32(&tile_bars[t * 6]);
                mbar_expect_tx(bar, Q_BYTES);
                for (int h = 0; h < PIECES; ++h)
                    tma_load_2d(smem_u32(q_tile + t * Q_BYTES + h * Q_PIECE), &map_q, bar, head * (D + R) + h * 64,
                                first_token + group0 + t * BQ);
            }
            for (int kb = 0; kb < n_blocks; ++kb) {
                int b = kb & 1;
                if (kb >= 2 && !mbar_wait(smem_u32(&k_empty[b]), ((kb >> 1) - 1) & 1, abort_flag, status, 21)) break;
                uint32_t bar = smem_u32(&k_full[b]);
                mbar_expect_tx(bar, K_BYTES);
                int row = first_token + kb * BKV;
                for (int h = 0; h < D / 64; ++h)
                    tma_load_2d(smem_u32(k_tile + b * K_BYTES + h * KV_PIECE), &map_kv, bar, head * (D + V) + h * 64, row);
                tma_load_2d(smem_u32(k_tile + b * K_BYTES + (D / 64) * KV_PIECE), &map_r, bar, 0, row);
            }
        }
    } else if (warp == 3) {
        if (lane == 0) {
            for (int kb = 0; kb < n_blocks; ++kb) {
                int b = kb & 1;
                if (kb >= 2 && !mbar_wait(smem_u32(&v_empty[b]), ((kb >> 1) - 1) & 1, abort_flag, status, 22)) break;
                uint32_t bar = smem_u32(&v_full[b]);
                mbar_expect_tx(bar, V_BYTES);
                for (int h = 0; h < V_PIECES; ++h)
                    tma_load_2d(smem_u32(v_tile + b * V_BYTES + h * KV_PIECE), &map_kv, bar, head * (D + V) + D + h * 64,
                                first_token + kb * BKV);
            }
        }
    } else if (warp < 3) {
        if (lane == 0) {
            int t = warp - 1, mine = blocks_of(t);
            uint64_t* s_full = tile_bars + t * 6 + 1;
            uint64_t* p_full = tile_bars + t * 6 + 3;
            uint64_t* o_full = tile_bars + t * 6 + 5;
            // D 32-bit, A and B bfloat16, M = 128; S has N = 64 keys, O has N = V with B MN-major
            constexpr uint32_t idesc_qk = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BKV >> 3) << 17) | ((uint32_t)(BQ >> 4) << 24);
            constexpr uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(V >> 3) << 17) |
                                          ((uint32_t)(BQ >> 4) << 24);
            const uint64_t q_desc = smem_desc(smem_u32(q_tile + t * Q_BYTES));
            const uint64_t k_desc0 = smem_desc(smem_u32(k_tile)), v_desc0 = smem_desc_mn(smem_u32(v_tile), KV_PIECE);
            constexpr uint64_t K_BUFFER = (uint64_t)(K_BYTES >> 4), V_BUFFER = (uint64_t)(V_BYTES >> 4);
            const uint32_t tmem = tmem_base + t * TILE_COLS;
            const int rot_steps = (R + 15) >> 4;
            auto issue_qk = [&](int kb) -> bool {
                int b = kb & 1;
                if (!mbar_wait(smem_u32(&k_full[b]), (kb >> 1) & 1, abort_flag, status, 24)) return false;
                tcgen05_fence_after();
                uint64_t k_desc = k_desc0 + b * K_BUFFER;
                uint32_t to = tmem + S_COL + b * BKV;
#pragma unroll
                for (int j = 0; j < D / 16; ++j)
                    tcgen05_mma(to, q_desc + (uint64_t)(((j >> 2) * Q_PIECE + (j & 3) * 32) >> 4),
                                k_desc + (uint64_t)(((j >> 2) * KV_PIECE + (j & 3) * 32) >> 4), idesc_qk, j > 0 ? 1u : 0u);
                for (int j = 0; j < rot_steps; ++j)
                    tcgen05_mma(to, q_desc + (uint64_t)(((D / 64) * Q_PIECE + j * 32) >> 4),
                                k_desc + (uint64_t)(((D / 64) * KV_PIECE + j * 32) >> 4), idesc_qk, 1u);
                tcgen05_commit(smem_u32(&s_full[b]));
                tcgen05_commit(smem_u32(&k_empty[b]));
                return true;
            };
            bool ok = true;
            if (mine > 0) {
                ok = mbar_wait(smem_u32(&tile_bars[t * 6]), 0, abort_flag, status, 23) && issue_qk(0);
                if (ok && mine > 1) ok = issue_qk(1);
            }
            // keys of blocks beyond this tile's own: released unread (one block at a time, when it has arrived)
            int released = mine;
            for (int kb = 0; kb < mine && ok; ++kb) {
                int b = kb & 1, phase = (kb >> 1) & 1;
                ok = mbar_wait(smem_u32(&p_full[b]), phase, abort_flag, status, 25) &&
                     mbar_wait(smem_u32(&v_full[b]), phase, abort_flag, status, 26);
                if (!ok) break;
                tcgen05_fence_after();
#pragma unroll
                for (int j = 0; j < BKV / 16; ++j)        // 16 keys a step: 8 columns of P, 2048 bytes of V rows
                    tcgen05_mma_ts(tmem + O_COL, tmem + S_COL + b * BKV + j * 8,
                                   v_desc0 + b * V_BUFFER + (uint64_t)((j * 2048) >> 4), idesc_pv, (kb > 0 || j > 0) ? 1u : 0u);
                tcgen05_commit(smem_u32(o_full));
                tcgen05_commit(smem_u32(&v_empty[b]));
                if (kb + 2 < mine) ok = issue_qk(kb + 2);
            }
            for (int kb = released; kb < n_blocks && ok; ++kb) {
                int b = kb & 1, phase = (kb >> 1) & 1;
                ok = mbar_wait(smem_u32(&k_full[b]), phase, abort_flag, status, 27);
                if (!ok) break;
                mbar_arrive(smem_u32(&k_empty[b]));
                ok = mbar_wait(smem_u32(&v_full[b]), phase, abort_flag, status, 28);
                if (!ok) break;
                mbar_arrive(smem_u32(&v_empty[b]));
            }
        }
    } else {
        int t = (warp - 4) >> 2, mine = blocks_of(t);
        int quarter = warp & 3;
        int row = quarter * 32 + lane;                       // query row of the tile = lane of tensor memory
        int pos = group0 + t * BQ + row;                     // its place in the sequence
        uint64_t* s_full = tile_bars + t * 6 + 1;
        uint64_t* p_full = tile_bars + t * 6 + 3;
        uint64_t* o_full = tile_bars + t * 6 + 5;
        uint32_t lane_addr = tmem_base + t * TILE_COLS + ((uint32_t)(quarter * 32) << 16);
        float run_max = -INFINITY, run_sum = 0.f;
        bool ok = mine > 0;
        for (int kb = 0; kb < mine && ok; ++kb) {
            int b = kb & 1;
            ok = mbar_wait(smem_u32(&s_full[b]), (kb >> 1) & 1, abort_flag, status, 29);
            if (!ok) break;
            __syncwarp();
            tcgen05_fence_after();
            int key0 = kb * BKV;
            bool whole = key0 + BKV - 1 <= pos;              // no key of the block is hidden from this row
            uint32_t s_addr = lane_addr + S_COL + b * BKV;
            uint32_t ra[32], rb[32];
            tmem_ld32_start(s_addr, ra);
            tmem_ld32_start(s_addr + 32, rb);
            float block_max = -INFINITY;
            auto row_max = [&](const uint32_t (&r)[32], int c) {
                if (whole) {
#pragma unroll
                    for (int j = 0; j < 32; j += 2) block_max = max3(block_max, __uint_as_float(r[j]), __uint_as_float(r[j + 1]));
                } else {
#pragma unroll
                    for (int j = 0; j < 32; ++j)
                        if (key0 + c + j <= pos) block_max = fmaxf(block_max, __uint_as_float(r[j]));
                }
            };
            tmem_ld32_wait(ra);
            tmem_ld32_wait(rb);
            row_max(ra, 0);
            row_max(rb, 32);
            // the exponent's reference moves only when the block's maximum exceeds it by more than 2^8
            bool move = kb == 0 || (block_max - run_max) * scale_log2 > 8.f;
            float new_max = move ? block_max : run_max;      // finite: key 0 is visible to every row
            float alpha = (move && kb > 0) ? fast_exp2((run_max - new_max) * scale_log2) : 1.f;
            float shift = new_max * scale_log2;
            run_max = new_max;
            float add = 0.f;
            auto to_probabilities = [&](const uint32_t (&r)[32], int c) {
                uint32_t packed[16];
                if (whole) {
#pragma unroll
                    for (int j = 0; j < 32; j += 2) {
                        float p0 = fast_exp2(fmaf(__uint_as_float(r[j]), scale_log2, -shift));
                        float p1 = fast_exp2(fmaf(__uint_as_float(r[j + 1]), scale_log2, -shift));
                        add += p0 + p1;
                        packed[j >> 1] = pack2(p0, p1);
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j += 2) {
                        float p0 = key0 + c + j <= pos ? fast_exp2(fmaf(__uint_as_float(r[j]), scale_log2, -shift)) : 0.f;
                        float p1 = key0 + c + j + 1 <= pos ? fast_exp2(fmaf(__uint_as_float(r[j + 1]), scale_log2, -shift)) : 0.f;
                        add += p0 + p1;
                        packed[j >> 1] = pack2(p0, p1);
                    }
                }
                tmem_st16(s_addr + (c >> 1), packed);
            };
            to_probabilities(ra, 0);
            to_probabilities(rb, 32);
            run_sum = run_sum * alpha + add;
            // O is rescaled behind the exponentials: the product before this one has had their time to finish
            if (kb > 0) {
                ok = mbar_wait(smem_u32(o_full), (kb - 1) & 1, abort_flag, status, 30);
                if (!ok) break;
                __syncwarp();
                tcgen05_fence_after();
                if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
                    for (int c = 0; c < V; c += 16) {
                        uint32_t r[16];
                        tmem_ld16(lane_addr + O_COL + c, r);
#pragma unroll
                        for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * alpha);
                        tmem_st16(lane_addr + O_COL + c, r);
                    }
                }
            }
            tmem_st_wait();
            tcgen05_fence_before();
            mbar_arrive(smem_u32(&p_full[b]));
        }
        if (ok) ok = mbar_wait(smem_u32(o_full), (mine - 1) & 1, abort_flag, status, 31);
        if (ok) {
            __syncwarp();
            tcgen05_fence_after();
            // (a sink far above every score makes the denominator infinite and the result zero, as it should be)
            if (sinks) run_sum += fast_exp2(fmaf(sinks[head], 1.4426950408889634f, -run_max * scale_log2));
            float inv = 1.0f / run_sum;
            __nv_bfloat16* o = out + (size_t)(first_token + pos) * out_stride + (size_t)head * V;
#pragma unroll 1
            for (int c = 0; c < V; c += 32) {
                uint32_t r[32];
                tmem_ld32(lane_addr + O_COL + c, r);
                if (pos < n_new) {
#pragma unroll
                    for (int d = 0; d < 32; d += 8) {
                        uint4 packed;
                        packed.x = pack2(__uint_as_float(r[d]) * inv, __uint_as_float(r[d + 1]) * inv);
                        packed.y = pack2(__uint_as_float(r[d + 2]) * inv, __uint_as_float(r[d + 3]) * inv);
                        packed.z = pack2(__uint_as_float(r[d + 4]) * inv, __uint_as_float(r[d + 5]) * inv);
                        packed.w = pack2(__uint_as_float(r[d + 6]) * inv, __uint_as_float(r[d + 7]) * inv);
                        *reinterpret_cast<uint4*>(o + c + d) = packed;
                    }
                }
            }
        }
    }

    tcgen05_fence_before();
    __syncthreads();
    if (*abort_flag) {
        for (int i = 0; i < 100; ++i) __nanosleep(10000);          // copies in flight land before shared memory is given up
        __syncthreads();
    }
    if (warp == 1) {
        tcgen05_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
    }
}

}  // namespace

LLMB_EXPORT int llmb_latent_prefill_tc_status() {
    int* s = status_word();
    if (!s) return -1;
    int v = *s;
    *s = 0;
    return v;
}

namespace {
template <int D, int V>
int launch(const CUtensorMap& map_q, const CUtensorMap& map_kv, const CUtensorMap& map_r, const int* cu_seqlens,
           const int* seq_order, void* out, int out_stride, int n_seqs, int max_new, int H, int R, float scale,
           const float* sinks, cudaStream_t stream) {
    constexpr size_t smem = smem_bytes<D, V>() < 120 * 1024 ? 120 * 1024 : smem_bytes<D, V>();     // one block an SM: it takes all of tensor memory
    static bool configured = false;
    if (!configured) {
        LLMB_CUDA(cudaFuncSetAttribute(latent_prefill_tc_kernel<D, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = true;
    }
    int* status = status_word();
    int* status_dev = nullptr;
    if (status) cudaHostGetDevicePointer((void**)&status_dev, status, 0);
    dim3 grid(H, ceil_div(max_new, TILES * BQ), n_seqs);
    LLMB_CUDA(llmb::launch(latent_prefill_tc_kernel<D, V>, grid, dim3(THREADS), smem, stream, true, map_q, map_kv, map_r, cu_seqlens,
                           seq_order, (__nv_bfloat16*)out, out_stride, R, scale * 1.4426950408889634f, sinks, status_dev));
    return check_launch("latent_prefill_tc");
}
}  // namespace

// All bfloat16: q [T, ldq], kv [T, H (D + V)], rows [T, C + R], out [T, out_stride] (H V columns). Every sequence of the
// step starts at its first token.
LLMB_EXPORT int llmb_latent_prefill_tc(const void* q, int ldq, const void* kv, const void* rows, int n_tokens,
                                       const int* cu_seqlens, const int* seq_order, void* out, int out_stride, int n_seqs,
                                       int max_new, int H, int D, int R, int V, int C, float scale, const float* sinks,
                                       cudaStream_t stream) {
    if (n_seqs == 0 || max_new == 0) return LLMB_OK;
    LLMB_REQUIRE((D == 64 || D == 128) && (V == 64 || V == 128) && R > 0 && R <= 64 && R % 8 == 0 && C % 8 == 0 && H > 0,
                 "latent_prefill_tc: heads of %d + %d with values of %d over a latent of %d", D, R, V, C);
    LLMB_REQUIRE(ldq % 8 == 0 && out_stride % 8 == 0 &&
                 ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(rows) |
                   reinterpret_cast<uintptr_t>(out)) & 15) == 0,
                 "latent_prefill_tc: operands must be 16-byte aligned with row strides that are multiples of 8");
    LLMB_REQUIRE(n_seqs <= 65535 && max_new / (TILES * BQ) < 65535 && scale > 0.f, "latent_prefill_tc: bad sizes");
    CUtensorMap map_q, map_kv, map_r;
    int code;
    if ((code = make_map_2d(&map_q, q, n_tokens, (long long)H * (D + R), ldq, 64, BQ))) return code;
    if ((code = make_map_2d(&map_kv, kv, n_tokens, (long long)H * (D + V), (long long)H * (D + V), 64, BKV))) return code;
    if ((code = make_map_2d(&map_r, (const __nv_bfloat16*)rows + C, n_tokens, R, C + R, 64, BKV))) return code;
#define GO(DD, VV) return launch<DD, VV>(map_q, map_kv, map_r, cu_seqlens, seq_order, out, out_stride, n_seqs, max_new, H, R, scale, sinks, stream)
    if (D == 64 && V == 64) GO(64, 64);
    if (D == 64) GO(64, 128);
    if (V == 64) GO(128, 64);
    GO(128, 128);
#undef GO
}
LLMB_PACKED(llmb_latent_prefill_tc)
