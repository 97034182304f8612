// The scan of a recurrence whose state S [D, V] fades and is written row by row, token by token:
//     S_t = diag(f_t) S_{t-1} + w_t v_t^T,      o_t = S_t^T q_t,
// with w = 1 - f (a forget gate that also decides what is written), or one fixed decay f per head and w = k. Every column
// of S is a recurrence of its own; a warp holds several columns of one head, lane l the pairs of state rows
// 2 l, 2 l + 1, then 64 further, .. of each, as packed 32-bit values. Per token it fades, writes and sums S q over its
// rows (even and odd rows in rising order, the two added, then the lanes as a butterfly), so a token's result depends on
// nothing but the sequence before it. The state is stored [H, V, D]: the rows that a value element reads are contiguous.
#pragma once

#include "pairs.cuh"
#include "scan.cuh"

namespace llmb {

// two rows of a column: f s + w v
__device__ __forceinline__ pair_t update(pair_t s, pair_t f, pair_t write, pair_t v) { return fma2(f, s, mul2(write, v)); }
// two neighbouring rows of a column, from n on, of which `rows` exist (an even number of rows is read and written in pairs)
__device__ __forceinline__ pair_t load_rows(const float* column, int n, int rows) {
    if (n >= rows) return 0ull;
    if (rows % 2 == 0) return *reinterpret_cast<const pair_t*>(column + n);
    return pack2(column[n], n + 1 < rows ? column[n + 1] : 0.f);
}
__device__ __forceinline__ void store_rows(float* column, int n, int rows, pair_t v) {
    if (n >= rows) return;
    if (rows % 2 == 0) { *reinterpret_cast<pair_t*>(column + n) = v; return; }
    float lo, hi;
    unpack2(v, lo, hi);
    column[n] = lo;
    if (n + 1 < rows) column[n + 1] = hi;
}

// PER: pairs of state rows a lane holds of each column (D <= 64 * PER). A block: WARPS warps of COLS columns each, the columns
// [blockIdx.x * TILE, + TILE) of head blockIdx.y for sequence blockIdx.z.
// FIXED: one decay per head for all rows and tokens, and a row of the work holds what is written instead of the gate f.
template <int PER, int COLS, int WARPS, bool FIXED>
__global__ void __launch_bounds__(WARPS * 32)
row_scan_kernel(const float* __restrict__ work, int work_ld, float* __restrict__ state, long long state_stride,
                const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids, const float* __restrict__ decays,
                float* __restrict__ o, int H, int D, int V, int vectors) {
    constexpr int TILE = WARPS * COLS;         // columns a block holds
    constexpr int GROUP = 32 / COLS;           // tokens whose partial sums meet in one butterfly
    constexpr int CHUNK = GROUP > 8 ? GROUP : 8;   // tokens staged at a time
    extern __shared__ __align__(16) float staged[];      // [2][CHUNK][row]: f or k (E) | q (E) | v (TILE), E: D rounded up to even
    griddep_launch();
    griddep_wait();
    work = behind_wait(work);
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int head = blockIdx.y, seq = blockIdx.z;
    int tile0 = blockIdx.x * TILE, v0 = tile0 + warp * COLS;
    int first = cu_seqlens[seq], n_new = cu_seqlens[seq + 1] - first;
    if (n_new <= 0) return;
    const int E = (D + 1) & ~1, row = (2 * E + TILE + 3) / 4 * 4;
    const int keys = H * D, f_at = head * D, q_at = keys + head * D, v_at = 2 * keys + head * V + tile0;
    float* S = state + (long long)slot_ids[seq] * state_stride + (size_t)head * D * V;   // [V, D]
    const float decay = FIXED ? decays[head] : 1.f;
    pair_t s[PER][COLS];
#pragma unroll
    for (int i = 0; i < PER; ++i)
#pragma unroll
        for (int c = 0; c < COLS; ++c) s[i][c] = v0 + c < V ? load_rows(S + (size_t)(v0 + c) * D, 2 * lane + 64 * i, D) : 0ull;
    auto request = [&](int chunk) {
        float* to = staged + (chunk & 1) * CHUNK * row;
        int t0 = chunk * CHUNK, count = min(CHUNK, n_new - t0);
        if (vectors) {                     // 16 bytes a copy, one token a warp at a time
            const int quads = (2 * D + TILE) / 4;
            for (int t = warp; t < count; t += WARPS) {
                const float* from = work + (size_t)(first + t0 + t) * work_ld;
                float* row_to = to + t * row;
                for (int q = lane; q < quads; q += 32) {
                    int r = 4 * q;
                    if (r < 2 * D) copy16(row_to + r, from + (r < D ? f_at + r : q_at + r - D));
                    else if (tile0 + r - 2 * D < V) copy16(row_to + r, from + v_at + r - 2 * D);
                }
            }
        } else {
            for (int t = 0; t < count; ++t) {
                const float* from = work + (size_t)(first + t0 + t) * work_ld;
                float* row_to = to + t * row;
                for (int r = threadIdx.x; r < 2 * D; r += WARPS * 32)
                    copy4(row_to + (r < D ? r : E + r - D), from + (r < D ? f_at + r : q_at + r - D));
                for (int r = threadIdx.x; r < TILE; r += WARPS * 32)
                    if (tile0 + r < V) copy4(row_to + 2 * E + r, from + v_at + r);
            }
        }
        copies_commit();
    };
    // one token of a group: fade, write, and the lane's share of S q for each column
    auto token = [&](const float* tok, float (&sums)[32], int j, bool live) {
        pair_t v[COLS], acc[COLS];
#pragma unroll
        for (int c = 0; c < COLS; ++c) {
            float value = (live && v0 + c < V) ? tok[2 * E + warp * COLS + c] : 0.f;
            v[c] = pack2(value, value);
            acc[c] = 0ull;
        }
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            int n = 2 * lane + 64 * i;
            // (beyond the step or the state nothing fades, is written or read)
            float2 f = live && n < D ? *reinterpret_cast<const float2*>(tok + n) : FIXED ? make_float2(0.f, 0.f) : make_float2(1.f, 1.f);
            float2 q = live && n < D ? *reinterpret_cast<const float2*>(tok + E + n) : make_float2(0.f, 0.f);
            if (n + 1 >= D) { f.y = FIXED ? 0.f : 1.f; q.y = 0.f; }
            pair_t qq = pack2(q.x, q.y), ff, write;
            if constexpr (FIXED) {
                float fade = live ? decay : 1.f;
                ff = pack2(fade, fade);
                write = pack2(f.x, f.y);
            } else {
                ff = pack2(f.x, f.y);
                write = pack2(1.0f - f.x, 1.0f - f.y);
            }
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                s[i][c] = update(s[i][c], ff, write, v[c]);
                acc[c] = fma2(s[i][c], qq, acc[c]);
            }
        }
#pragma unroll
        for (int c = 0; c < COLS; ++c) {
            float even, odd;
            unpack2(acc[c], even, odd);
            sums[j * COLS + c] = even + odd;
        }
    };
    int n_chunks = (n_new + CHUNK - 1) / CHUNK;
    request(0);
    for (int chunk = 0; chunk < n_chunks; ++chunk) {
        if (chunk + 1 < n_chunks) { request(chunk + 1); copies_wait<1>(); }
        else copies_wait<0>();
        __syncthreads();
        const float* from = staged + (chunk & 1) * CHUNK * row;
        int t0 = chunk * CHUNK, count = min(CHUNK, n_new - t0);
        for (int g0 = 0; g0 < count; g0 += GROUP) {
            float sums[32];
            if (g0 + GROUP <= count) {
#pragma unroll
                for (int j = 0; j < GROUP; ++j) token(from + (g0 + j) * row, sums, j, true);
            } else {
#pragma unroll
                for (int j = 0; j < GROUP; ++j) token(from + (g0 + j) * row, sums, j, g0 + j < count);
            }
            fold<16, 16>(sums, lane);
            fold<8, 8>(sums, lane);
            fold<4, 4>(sums, lane);
            fold<2, 2>(sums, lane);
            fold<1, 1>(sums, lane);
            int j = lane / COLS, c = lane % COLS;           // lane l holds token l / COLS, column l % COLS of the group
            if (g0 + j < count && v0 + c < V)
                o[(size_t)(first + t0 + g0 + j) * H * V + head * V + v0 + c] = sums[0];
        }
        __syncthreads();                   // the stage is requested again two chunks on
    }
#pragma unroll
    for (int i = 0; i < PER; ++i)
#pragma unroll
        for (int c = 0; c < COLS; ++c)
            if (v0 + c < V) store_rows(S + (size_t)(v0 + c) * D, 2 * lane + 64 * i, D, s[i][c]);
}

}  // namespace llmb
