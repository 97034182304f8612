// Attention over one cached latent row per position, [c (C) | r (R)], whose first C elements serve all heads as values
// and whose last R are a rotated key part that all heads share. What lies around it is here too.
//
// latent_write    one block per token of the projection [q: H x (D | R) | c (C) | r (R)]: c / sqrt(mean(c^2) + eps) * gain, r
//                 rotated, both into the token's cache row (and, optionally, a dense row); the rotated part of every
//                 query head, either into the last R columns of its latent query [C | R] or in place. Where the queries pass
//                 a latent of their own, the launch behind the first product norms that latent and writes the cache row, and
//                 a second one, behind the queries' product, rotates the query heads.
// head_products   out[t, h, :] = W_h x[t, h, :] with a matrix per head: queries into the latent space, results out of it.
// latent_attention_tiles (bfloat16)  softmax attention of the new tokens' latent queries [T, H, C + R] over the cached
//                 rows. All heads share the row, so (token, head) pairs are the rows of the tiles: a block takes 16, 32 or 64
//                 consecutive pairs of a sequence (a decode step: its heads), brings a page of 64 rows into shared memory once
//                 (cp.async, the next page under the current), forms S = Q K^T with its warps on (row, key) parts, meets on
//                 the rows' maxima, and forms P V with every warp on a range of value columns for all rows. Long
//                 sequences of a decode step are cut into slices of pages whose partial results a second kernel merges.
//                 Shared memory rows are swizzled by 16-byte pieces (piece ^ row % 8).
// latent_decode_tc (bfloat16)  the same for a step of one token a sequence on tcgen05, with the rows by TMA: see there.
//
// `sinks` [H] (optional): e^sink[h] is one more term of a head's denominator, without key or value, not scaled.
// Norm, rotation, scores, weights and sums are 32-bit (weights are rounded as the operand of P V, whose sum is 32-bit).
// A query at position p sees the keys j <= p.
#include "common.cuh"
#include "mma.cuh"
#include "tc.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_latent_attention)

constexpr int THREADS = 256;

__device__ __forceinline__ float block_sum(float v, float* scratch) {
    v = warp_sum(v);
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += scratch[w];
    return total;
}

// ---------------------------------------------------------------------------------------------- behind the projection

// The rotated value of element d of a part x of R elements: pairs (2i, 2i + 1) or (i, i + n_rot / 2) of its first n_rot.
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int d, const float* angles, int n_rot, int interleaved) {
    float v = to_float(x[d]);
    if (d >= n_rot) return v;
    int half = n_rot / 2, pair, partner;
    bool first;
    if (interleaved) { pair = d >> 1; first = (d & 1) == 0; partner = first ? d + 1 : d - 1; }
    else { first = d < half; pair = first ? d : d - half; partner = first ? d + half : d - half; }
    float c = angles[pair], s = angles[half + pair], other = to_float(x[partner]);
    return first ? v * c - other * s : v * c + other * s;
}

// 1 / root mean square of the block's row of n elements.
template <typename T>
__device__ __forceinline__ float row_factor(const T* x, int n, float eps, float* scratch) {
    float sq = 0.f;
    for (int d = threadIdx.x; d < n; d += THREADS) {
        float v = to_float(x[d]);
        sq = fmaf(v, v, sq);
    }
    return 1.0f / sqrtf(block_sum(sq, scratch) / (float)n + eps);
}

// Three parts, each optional: the queries' latent (the first q_rank columns of u, normed, into cq), the cached row (c_at >= 0: the
// columns [c | r] of u from there on), and the rotated parts of the query heads in `heads` (which may be u).
template <typename T>
__global__ void __launch_bounds__(THREADS)
latent_write_kernel(const T* u, int ld, int c_at, int q_rank, const float* __restrict__ q_gain, T* __restrict__ cq, T* heads,
                    int heads_ld, int H, int D, int R, int C, const float* __restrict__ gain, float eps,
                    const float* __restrict__ table, int n_rot, int interleaved, const int* __restrict__ tok_pos,
                    const int* __restrict__ tok_seq, const int* __restrict__ block_table, int table_stride, int ring_pages,
                    T* __restrict__ cache, int write_cache, T* __restrict__ queries, T* __restrict__ dense) {
    __shared__ float scratch[THREADS / 32];
    griddep_launch();
    griddep_wait();
    size_t t = blockIdx.x;
    const T* row = u + t * ld;
    int pos = tok_pos[t], width = C + R;
    const float* angles = table + (size_t)pos * n_rot;
    if (q_rank > 0) {
        float factor = row_factor(row, q_rank, eps, scratch);
        for (int d = threadIdx.x; d < q_rank; d += THREADS)
            cq[t * q_rank + d] = from_float<T>(to_float(row[d]) * factor * q_gain[d]);
    }
    if (c_at >= 0) {
        const T* c_in = row + c_at;
        float factor = row_factor(c_in, C, eps, scratch);
        T* to = nullptr;
        if (write_cache) {
            size_t page = (size_t)block_table[(size_t)tok_seq[t] * table_stride + (pos / LLMB_PAGE) % ring_pages];
            to = cache + (page * LLMB_PAGE + pos % LLMB_PAGE) * width;
        }
        for (int d = threadIdx.x; d < width; d += THREADS) {
            T v = from_float<T>(d < C ? to_float(c_in[d]) * factor * gain[d] : rotated(c_in + C, d - C, angles, n_rot, interleaved));
            if (to) to[d] = v;
            if (dense) dense[t * width + d] = v;
        }
    }
    if (!heads) return;
    T* in = heads + t * heads_ld;
    if (queries) {
        for (int i = threadIdx.x; i < H * R; i += THREADS) {
            int head = i / R, d = i % R;
            queries[(t * H + head) * width + C + d] =
                from_float<T>(rotated(in + head * (D + R) + D, d, angles, n_rot, interleaved));
        }
    } else {                               // in place: a thread takes both elements of a pair
        int half = n_rot / 2;
        for (int i = threadIdx.x; i < H * half; i += THREADS) {
            int head = i / half, pair = i % half;
            T* x = in + head * (D + R) + D;
            int a = interleaved ? 2 * pair : pair, b = interleaved ? 2 * pair + 1 : pair + half;
            float c = angles[pair], s = angles[half + pair], va = to_float(x[a]), vb = to_float(x[b]);
            x[a] = from_float<T>(va * c - vb * s);
            x[b] = from_float<T>(vb * c + va * s);
        }
    }
}

// u [T, ld]: [queries' latent (q_rank) ..] and from column c_at on [c (C) | r (R)] (c_at < 0: not there); heads [T, heads_ld]: H query
// heads of D + R (null: none; it may be u); q_gain float32 [q_rank] and cq [T, q_rank] with q_rank > 0; gain float32 [C]; table
// float32 [positions, n_rot] (or null: no rotation); cache [pages, 1, 64, C + R]; queries [T, H, C + R] (or null: query heads
// rotate in place); dense [T, C + R] or null.
LLMB_EXPORT int llmb_latent_write(const void* u, int ld, int dtype, int c_at, int q_rank, const float* q_gain, void* cq, void* heads,
                                  int heads_ld, int H, int D, int R, int C, const float* gain, float eps,
                                  const float* table, int n_rot, int interleaved, const int* tok_pos, const int* tok_seq,
                                  const int* block_table, int table_stride, int ring_pages, void* cache, int write_cache,
                                  void* queries, void* dense, int n_tokens, cudaStream_t stream) {
    if (n_tokens == 0) return LLMB_OK;
    LLMB_REQUIRE(H > 0 && D > 0 && R > 0 && C > 0 && ring_pages > 0 && (c_at < 0 || (gain && u && ld >= c_at + C + R)) &&
                 (q_rank <= 0 || (q_gain && cq && u && ld >= q_rank)) && (!heads || heads_ld >= H * (D + R)), "latent_write: bad sizes");
    LLMB_REQUIRE(!table || (n_rot > 0 && n_rot % 2 == 0 && n_rot <= R), "latent_write: %d of %d elements rotate", n_rot, R);
#define LLMB_WRITE(T)                                                                                                     \
    LLMB_CUDA(llmb::launch(latent_write_kernel<T>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const T*)u, ld, c_at, q_rank, \
                           q_gain, (T*)cq, (T*)heads, heads_ld, H, D, R, C, gain, eps, table, table ? n_rot : 0, interleaved, \
                           tok_pos, tok_seq, block_table, table_stride, ring_pages, (T*)cache, write_cache, (T*)queries, (T*)dense))
    if (dtype == LLMB_DTYPE_F32) LLMB_WRITE(float);
    else if (dtype == LLMB_DTYPE_BF16) LLMB_WRITE(__nv_bfloat16);
    else return fail(LLMB_ERR_ARGUMENT, "latent_write: unknown dtype %d", dtype);
#undef LLMB_WRITE
    return check_launch("latent_write");
}
LLMB_PACKED(llmb_latent_write)

// ---------------------------------------------------------------------------------------------- a matrix per head

// CUDA cores: 16 tokens x 64 outputs a block, k in rising order whatever else is in the block.
template <typename T>
__global__ void __launch_bounds__(THREADS)
head_products_kernel(const T* __restrict__ x, int ldx, int x_head, const T* __restrict__ w, int N, int K, T* __restrict__ out,
                     int ldo, int out_head, int n_tokens) {
    __shared__ float xs[16][33], ws[64][33];
    griddep_launch();
    griddep_wait();
    x = behind_wait(x);
    int head = blockIdx.z, t0 = blockIdx.y * 16, n0 = blockIdx.x * 64;
    const T* wh = w + (size_t)head * N * K;
    int tx = threadIdx.x & 63, ty = threadIdx.x >> 6;          // output n0 + tx of the tokens ty, ty + 4, ..
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < K; k0 += 32) {
        for (int i = threadIdx.x; i < 16 * 32; i += THREADS) {
            int r = i >> 5, k = k0 + (i & 31);
            xs[r][i & 31] = (t0 + r < n_tokens && k < K) ? to_float(x[(size_t)(t0 + r) * ldx + head * x_head + k]) : 0.f;
        }
        for (int i = threadIdx.x; i < 64 * 32; i += THREADS) {
            int r = i >> 5, k = k0 + (i & 31);
            ws[r][i & 31] = (n0 + r < N && k < K) ? to_float(wh[(size_t)(n0 + r) * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            float b = ws[tx][k];
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i] = fmaf(xs[ty + 4 * i][k], b, acc[i]);
        }
        __syncthreads();
    }
    if (n0 + tx >= N) return;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        int t = t0 + ty + 4 * i;
        if (t < n_tokens) out[(size_t)t * ldo + head * out_head + n0 + tx] = from_float<T>(acc[i]);
    }
}

// Tensor cores: TM tokens x 64 outputs a block of four warps, k in steps of 64 through two buffers. TM 16: a warp takes 16
// of the outputs; TM 64: 16 of the tokens.
template <int TM>
__global__ void __launch_bounds__(128)
head_products_mma_kernel(const __nv_bfloat16* __restrict__ x, int ldx, int x_head, const __nv_bfloat16* __restrict__ w, int N,
                         int K, __nv_bfloat16* __restrict__ out, int ldo, int out_head, int n_tokens) {
    constexpr int LDS = 64 + 8;
    __shared__ __align__(16) __nv_bfloat16 xs[2][TM][LDS], ws[2][64][LDS];
    griddep_launch();
    int head = blockIdx.z, t0 = blockIdx.y * TM, n0 = blockIdx.x * 64;
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const __nv_bfloat16* wh = w + (size_t)head * N * K;
    const __nv_bfloat16* xh = x + (size_t)t0 * ldx + head * x_head;
    const __nv_bfloat16 zero = __float2bfloat16(0.f);
    // what is never loaded (rows beyond the tokens or outputs, the last step's columns beyond K) reads as zeros
    for (int i = threadIdx.x; i < 2 * TM * LDS; i += 128) (&xs[0][0][0])[i] = zero;
    for (int i = threadIdx.x; i < 2 * 64 * LDS; i += 128) (&ws[0][0][0])[i] = zero;
    __syncthreads();
    auto request_w = [&](int stage, int k0) {
        for (int i = threadIdx.x; i < 64 * 8; i += 128) {
            int r = i >> 3, c = (i & 7) * 8;
            if (n0 + r < N) {
                if (k0 + c < K) cp_async16(&ws[stage][r][c], wh + (size_t)(n0 + r) * K + k0 + c);
                else *reinterpret_cast<uint4*>(&ws[stage][r][c]) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
    };
    auto request_x = [&](int stage, int k0) {
        for (int i = threadIdx.x; i < TM * 8; i += 128) {
            int r = i >> 3, c = (i & 7) * 8;
            if (t0 + r < n_tokens) {
                if (k0 + c < K) cp_async16(&xs[stage][r][c], xh + (size_t)r * ldx + k0 + c);
                else *reinterpret_cast<uint4*>(&xs[stage][r][c]) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
    };
    constexpr int NB = TM == 16 ? 2 : 8;                  // blocks of 8 outputs a warp holds
    float acc[NB][4] = {};
    int row0 = TM == 16 ? 0 : warp * 16, col0 = TM == 16 ? warp * 16 : 0;
    int steps = (K + 63) / 64;
    request_w(0, 0);                                      // weights: no kernel of a step writes them
    griddep_wait();
    request_x(0, 0);
    cp_async_commit();
    for (int s = 0; s < steps; ++s) {
        if (s + 1 < steps) { request_w((s + 1) & 1, (s + 1) * 64); request_x((s + 1) & 1, (s + 1) * 64); cp_async_commit(); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 64; k += 16) {
            uint32_t a[4];
            ldmatrix_x4(a, &xs[s & 1][row0 + (lane & 15)][k + (lane >> 4) * 8]);
#pragma unroll
            for (int nb = 0; nb < NB; nb += 2) {
                uint32_t b[4];
                ldmatrix_x4(b, &ws[s & 1][col0 + nb * 8 + (lane & 7) + ((lane >> 4) << 3)][k + ((lane >> 3) & 1) * 8]);
                mma_bf16(acc[nb], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(acc[nb + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
#pragma unroll
        for (int f = 0; f < 2; ++f) {
            int t = t0 + row0 + (lane >> 2) + f * 8, n = n0 + col0 + nb * 8 + (lane & 3) * 2;
            if (t >= n_tokens || n >= N) continue;
            __nv_bfloat16* o = out + (size_t)t * ldo + head * out_head + n;
            if (n + 1 < N && (reinterpret_cast<uintptr_t>(o) & 3) == 0)
                *reinterpret_cast<__nv_bfloat162*>(o) = __floats2bfloat162_rn(acc[nb][2 * f], acc[nb][2 * f + 1]);
            else {
                o[0] = __float2bfloat16_rn(acc[nb][2 * f]);
                if (n + 1 < N) o[1] = __float2bfloat16_rn(acc[nb][2 * f + 1]);
            }
        }
}

// out[t * ldo + h * out_head + n] = sum_k x[t * ldx + h * x_head + k] w[h, n, k], n < N, k < K, h < H.
LLMB_EXPORT int llmb_head_products(const void* x, int ldx, int x_head, const void* w, int H, int N, int K, void* out, int ldo,
                                   int out_head, int dtype, int n_tokens, int tensor_cores, cudaStream_t stream) {
    if (n_tokens == 0) return LLMB_OK;
    LLMB_REQUIRE(H > 0 && N > 0 && K > 0 && H <= 65535 && x_head >= K && ldx >= (H - 1) * x_head + K && ldo >= (H - 1) * out_head + N,
                 "head_products: bad sizes");
    LLMB_REQUIRE(ceil_div(n_tokens, 16) <= 65535, "head_products: %d tokens", n_tokens);
    bool mma = tensor_cores && dtype == LLMB_DTYPE_BF16 && K % 8 == 0 && ldx % 8 == 0 && x_head % 8 == 0 &&
               ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
    if (mma) {
        typedef __nv_bfloat16 B;
        if (n_tokens <= 32)
            LLMB_CUDA(llmb::launch(head_products_mma_kernel<16>, dim3(ceil_div(N, 64), ceil_div(n_tokens, 16), H), dim3(128), 0,
                                   stream, true, (const B*)x, ldx, x_head, (const B*)w, N, K, (B*)out, ldo, out_head, n_tokens));
        else
            LLMB_CUDA(llmb::launch(head_products_mma_kernel<64>, dim3(ceil_div(N, 64), ceil_div(n_tokens, 64), H), dim3(128), 0,
                                   stream, true, (const B*)x, ldx, x_head, (const B*)w, N, K, (B*)out, ldo, out_head, n_tokens));
        return check_launch("head_products");
    }
    dim3 grid(ceil_div(N, 64), ceil_div(n_tokens, 16), H);
#define LLMB_HEADS(T)                                                                                                      \
    LLMB_CUDA(llmb::launch(head_products_kernel<T>, grid, dim3(THREADS), 0, stream, true, (const T*)x, ldx, x_head, (const T*)w, \
                           N, K, (T*)out, ldo, out_head, n_tokens))
    if (dtype == LLMB_DTYPE_F32) LLMB_HEADS(float);
    else if (dtype == LLMB_DTYPE_BF16) LLMB_HEADS(__nv_bfloat16);
    else return fail(LLMB_ERR_ARGUMENT, "head_products: unknown dtype %d", dtype);
#undef LLMB_HEADS
    return check_launch("head_products");
}
LLMB_PACKED(llmb_head_products)

// ---------------------------------------------------------------------------------------------- attention

__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// What a sink adds to a denominator in units of 2^m (m: the row's reference, base 2). A sink far above every score makes it
// infinite and the row's result zero, as it should be.
__device__ __forceinline__ float sink_share(float sink, float m) { return exp2f(fmaf(sink, 1.4426950408889634f, -m)); }

// MT: tiles of 16 rows ((token, head) pairs) a block holds; NT: blocks of 8 value columns a warp holds (C <= 64 NT).
// Eight warps. S: warp w works on rows [(w % MT) 16, +16) and keys [(w / MT) 8 MT, + 8 MT) of a page.
// `width` C + R, `row_elems` the elements of a row in shared memory (a multiple of 64, at least width and 64 NT).
template <int MT, int NT>
__global__ void __launch_bounds__(THREADS, 1)
latent_tiles_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache,
                    const int* __restrict__ block_table, int table_stride, int ring_pages, const int* __restrict__ cu_seqlens,
                    const int* __restrict__ seq_lens, const int* __restrict__ seq_order, __nv_bfloat16* __restrict__ out,
                    float* __restrict__ part_acc, float* __restrict__ part_stats, int H, int C, int width, int row_elems,
                    float scale_log2, const float* __restrict__ sinks) {
    constexpr int ROWS = 16 * MT, KW = 8 / MT;             // KW: warps that share a row tile's keys
    extern __shared__ __align__(128) unsigned char smem_raw[];
    const int row_bytes = row_elems * 2;
    unsigned char* k_smem = smem_raw;                                     // [2][64][row]
    unsigned char* q_smem = k_smem + 2 * LLMB_PAGE * row_bytes;           // [ROWS][row]
    unsigned char* p_smem = q_smem + ROWS * row_bytes;                    // [ROWS][64] bfloat16
    float* red = reinterpret_cast<float*>(p_smem + ROWS * 128);           // [KW][ROWS] maxima, then sums
    float* alphas = red + KW * ROWS;                                      // [ROWS]

    griddep_launch();
    int split = blockIdx.x, n_splits = gridDim.x;
    int seq = seq_order ? seq_order[blockIdx.z] : (int)blockIdx.z;
    int first_token = cu_seqlens[seq], n_new = cu_seqlens[seq + 1] - first_token;
    int n_rows = n_new * H, n_tiles = (n_rows + ROWS - 1) / ROWS;
    if ((int)blockIdx.y >= n_tiles) { griddep_wait(); return; }
    int tile = n_tiles - 1 - blockIdx.y;                   // the heaviest first
    int start = seq_lens[seq] - n_new;
    int row_first = tile * ROWS, row_last = min(row_first + ROWS, n_rows) - 1;
    int last_pos = start + row_last / H;
    int n_pages = last_pos / LLMB_PAGE + 1;
    int per_split = (n_pages + n_splits - 1) / n_splits;
    int page_begin = min(split * per_split, n_pages), page_end = min(page_begin + per_split, n_pages);
    const int* pages = block_table + (size_t)seq * table_stride;
    int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int pieces = width / 8, row_pieces = row_elems / 8;

    auto swizzled = [&](int row, int piece) { return row * row_bytes + ((piece ^ (row & 7)) << 4); };
    auto load_page = [&](int logical, int stage) {
        const __nv_bfloat16* from = cache + (size_t)pages[logical % ring_pages] * LLMB_PAGE * width;
        unsigned char* to = k_smem + stage * LLMB_PAGE * row_bytes;
        for (int i = tid; i < LLMB_PAGE * pieces; i += THREADS) {
            int r = i / pieces, c = i - r * pieces;
            cp_async16(to + swizzled(r, c), from + (size_t)r * width + c * 8);
        }
    };
    // columns that are never loaded read as zeros
    const uint4 none = make_uint4(0u, 0u, 0u, 0u);
    int tail = row_pieces - pieces;
    if (tail > 0) {
        for (int i = tid; i < 2 * LLMB_PAGE * tail; i += THREADS) {
            int r = i / tail, c = pieces + i % tail;
            *reinterpret_cast<uint4*>(k_smem + (r >> 6) * LLMB_PAGE * row_bytes + swizzled(r & 63, c)) = none;
        }
        for (int i = tid; i < ROWS * tail; i += THREADS)
            *reinterpret_cast<uint4*>(q_smem + swizzled(i / tail, pieces + i % tail)) = none;
    }
    // a page that holds none of this step's tokens is final: it may be requested before the kernel in front has ended
    bool early = page_begin < page_end && (page_begin + 1) * LLMB_PAGE <= start;
    if (early) load_page(page_begin, page_begin & 1);
    griddep_wait();
    if (!early && page_begin < page_end) load_page(page_begin, page_begin & 1);
    for (int i = tid; i < ROWS * pieces; i += THREADS) {
        int r = i / pieces, c = i - r * pieces;
        if (row_first + r < n_rows)
            cp_async16(q_smem + swizzled(r, c), q + ((size_t)first_token * H + row_first + r) * width + c * 8);
        else *reinterpret_cast<uint4*>(q_smem + swizzled(r, c)) = none;
    }
    cp_async_commit();

    float acc[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
    int m_tile = warp % MT, k_part = warp / MT;
    int row0 = m_tile * 16 + g, row1 = row0 + 8;           // this lane's rows of the score tile
    int pos0 = start + (row_first + row0) / H, pos1 = start + (row_first + row1) / H;
    float max0 = -INFINITY, max1 = -INFINITY, sum0 = 0.f, sum1 = 0.f;      // sums over this lane's keys only
    int tile_first_pos = start + row_first / H;

    for (int p = page_begin; p < page_end; ++p) {
        cp_async_wait<0>();
        __syncthreads();                                   // the page landed; everyone is done with the one before
        if (p + 1 < page_end) load_page(p + 1, (p + 1) & 1);
        cp_async_commit();
        const unsigned char* ks = k_smem + (p & 1) * LLMB_PAGE * row_bytes;
        // ---- S: 16 rows x 8 MT keys a warp; two k-steps of 16 at a time
        float s[MT][4];
#pragma unroll
        for (int n = 0; n < MT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) s[n][i] = 0.f;
        int key_part = k_part * 8 * MT;
#pragma unroll 2
        for (int c = 0; c < row_pieces; c += 4) {
            uint32_t a0[4], a1[4];
            ldmatrix_x4(a0, q_smem + swizzled(m_tile * 16 + (lane & 15), c + (lane >> 4)));
            ldmatrix_x4(a1, q_smem + swizzled(m_tile * 16 + (lane & 15), c + 2 + (lane >> 4)));
#pragma unroll
            for (int n = 0; n < MT; ++n) {
                uint32_t b[4];
                ldmatrix_x4(b, ks + swizzled(key_part + n * 8 + (lane & 7), c + (lane >> 3)));
                mma_bf16(s[n], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                mma_bf16(s[n], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
            }
        }
        int key0 = p * LLMB_PAGE + key_part;
        bool diagonal = (p + 1) * LLMB_PAGE - 1 > tile_first_pos;
        float local0 = -INFINITY, local1 = -INFINITY;
#pragma unroll
        for (int n = 0; n < MT; ++n)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                if (diagonal) {
                    int key = key0 + n * 8 + 2 * t4 + i;
                    if (key > pos0) s[n][i] = -INFINITY;
                    if (key > pos1) s[n][2 + i] = -INFINITY;
                }
                local0 = fmaxf(local0, s[n][i]);
                local1 = fmaxf(local1, s[n][2 + i]);
            }
        local0 = fmaxf(local0, __shfl_xor_sync(0xffffffffu, local0, 1));
        local0 = fmaxf(local0, __shfl_xor_sync(0xffffffffu, local0, 2));
        local1 = fmaxf(local1, __shfl_xor_sync(0xffffffffu, local1, 1));
        local1 = fmaxf(local1, __shfl_xor_sync(0xffffffffu, local1, 2));
        if (t4 == 0) { red[k_part * ROWS + row0] = local0; red[k_part * ROWS + row1] = local1; }
        __syncthreads();
        float new0 = max0, new1 = max1;
#pragma unroll
        for (int w = 0; w < KW; ++w) {
            new0 = fmaxf(new0, red[w * ROWS + row0]);
            new1 = fmaxf(new1, red[w * ROWS + row1]);
        }
        // (a row of a later tile page may have seen nothing yet: a reference of 0 keeps every term 0)
        float ref0 = new0 == -INFINITY ? 0.f : new0, ref1 = new1 == -INFINITY ? 0.f : new1;
        float alpha0 = fast_exp2((max0 - ref0) * scale_log2), alpha1 = fast_exp2((max1 - ref1) * scale_log2);
        max0 = new0;
        max1 = new1;
        float add0 = 0.f, add1 = 0.f;
#pragma unroll
        for (int n = 0; n < MT; ++n) {
            float p00 = fast_exp2((s[n][0] - ref0) * scale_log2), p01 = fast_exp2((s[n][1] - ref0) * scale_log2);
            float p10 = fast_exp2((s[n][2] - ref1) * scale_log2), p11 = fast_exp2((s[n][3] - ref1) * scale_log2);
            add0 += p00 + p01;
            add1 += p10 + p11;
            int piece = (key_part + n * 8) >> 3;
            *reinterpret_cast<uint32_t*>(p_smem + row0 * 128 + ((piece ^ (row0 & 7)) << 4) + t4 * 4) = pack_bf16(p00, p01);
            *reinterpret_cast<uint32_t*>(p_smem + row1 * 128 + ((piece ^ (row1 & 7)) << 4) + t4 * 4) = pack_bf16(p10, p11);
        }
        sum0 = sum0 * alpha0 + add0;
        sum1 = sum1 * alpha1 + add1;
        if (k_part == 0 && t4 == 0) { alphas[row0] = alpha0; alphas[row1] = alpha1; }
        __syncthreads();                                   // P and the factors are there
        // ---- O += P V: every warp all rows, its own value columns
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            float f0 = alphas[m * 16 + g], f1 = alphas[m * 16 + g + 8];
#pragma unroll
            for (int n = 0; n < NT; ++n) { acc[m][n][0] *= f0; acc[m][n][1] *= f0; acc[m][n][2] *= f1; acc[m][n][3] *= f1; }
        }
        int col_piece = warp * NT;                         // the warp's first block of 8 columns
        if constexpr (NT == 1) {
#pragma unroll
            for (int kk = 0; kk < 4; kk += 2) {            // 32 keys: four 8 x 8 blocks of the same columns
                uint32_t b[4];
                ldmatrix_x4_trans(b, ks + swizzled(kk * 16 + lane, col_piece));
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    uint32_t a[4];
                    int r = m * 16 + (lane & 15);
                    ldmatrix_x4(a, p_smem + r * 128 + (((kk * 2 + (lane >> 4)) ^ (r & 7)) << 4));
                    mma_bf16(acc[m][0], a[0], a[1], a[2], a[3], b[0], b[1]);
                    ldmatrix_x4(a, p_smem + r * 128 + (((kk * 2 + 2 + (lane >> 4)) ^ (r & 7)) << 4));
                    mma_bf16(acc[m][0], a[0], a[1], a[2], a[3], b[2], b[3]);
                }
            }
        } else {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t a[MT][4];
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    int r = m * 16 + (lane & 15);
                    ldmatrix_x4(a[m], p_smem + r * 128 + (((kk * 2 + (lane >> 4)) ^ (r & 7)) << 4));
                }
#pragma unroll
                for (int n = 0; n < NT; n += 2) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, ks + swizzled(kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), col_piece + n + (lane >> 4)));
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_bf16(acc[m][n], a[m][0], a[m][1], a[m][2], a[m][3], b[0], b[1]);
                        mma_bf16(acc[m][n + 1], a[m][0], a[m][1], a[m][2], a[m][3], b[2], b[3]);
                    }
                }
            }
        }
    }
    cp_async_wait<0>();
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
    __syncthreads();
    if (t4 == 0) {
        red[k_part * ROWS + row0] = sum0;
        red[k_part * ROWS + row1] = sum1;
        if (k_part == 0) { alphas[row0] = max0; alphas[row1] = max1; }      // (the factors have been read)
    }
    __syncthreads();
    size_t base = (size_t)first_token * H + row_first;     // the tile's first row among all rows of the step
    if (n_splits > 1 && warp < MT && t4 == 0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            int r = i ? row1 : row0;
            if (row_first + r >= n_rows) continue;
            float total = 0.f;
#pragma unroll
            for (int w = 0; w < KW; ++w) total += red[w * ROWS + r];
            float* to = part_stats + ((base + r) * n_splits + split) * 2;
            to[0] = (i ? max1 : max0) * scale_log2;
            to[1] = total;
        }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            int r = m * 16 + g + i * 8;
            if (row_first + r >= n_rows) continue;
            float total = 0.f;
#pragma unroll
            for (int w = 0; w < KW; ++w) total += red[w * ROWS + r];
            if (sinks && n_splits == 1)
                total += sink_share(sinks[(row_first + r) % H], alphas[r] * scale_log2);
            float inv = n_splits == 1 ? 1.0f / total : 1.f;
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                int col = (warp * NT + n) * 8 + 2 * t4;
                if (col >= C) continue;                    // (C is a multiple of 8)
                float lo = acc[m][n][2 * i] * inv, hi = acc[m][n][2 * i + 1] * inv;
                if (n_splits == 1)
                    *reinterpret_cast<__nv_bfloat162*>(out + (base + r) * C + col) = __floats2bfloat162_rn(lo, hi);
                else
                    *reinterpret_cast<float2*>(part_acc + ((base + r) * n_splits + split) * C + col) = make_float2(lo, hi);
            }
        }
}

// One token a sequence on the fifth-generation tensor cores: block (slice, chunk of NH heads, sequence). The cached rows
// stream through a ring of pages (boxes of 64 columns and 64 rows a piece, 128-byte swizzle; the last piece is the rotated
// part, zeros beyond it), each read once for all heads of the block, by both products:
//
// * scores: S[head, key] = Q K^T, the heads as rows of the 128-row side, with the queries in tensor memory (written there
//   once: a product that reads its 128 rows from shared memory takes twice as long, whatever its width; rows beyond NH
//   hold what tensor memory held before: their results are not looked at).
// * values: O^T[value element, head] += V^T P^T, 128 value elements a product, the rows' own bytes as an MN-major operand, P
//   from shared memory (bfloat16 [head, key]); ceil(C / 128) accumulators of NH columns. Turned this way nothing is padded:
//   with the heads on the 128-row side O alone would fill tensor memory.
//
// Warp 0: softmax, a lane a head (its 64 scores read once, and their buffer given back at once; running maximum and sum in
// 32-bit). Warp 1, one lane: TMA. Warp 2, one lane: the products, whichever is ready first. Warps 4-7: rescale O where a
// head's maximum outgrew its reference by 2^8 (a column is a head; rare), and the result. Pages of older rows than the
// step's are requested before the kernel in front has ended. Waits are bounded.
namespace decode {

using namespace llmb::tc;

constexpr int KEYS = LLMB_PAGE, PIECE = KEYS * 128, MAX_STAGES = 8;

// whether the phase is complete, without waiting for it
__device__ __forceinline__ bool mbar_test(uint32_t bar, uint32_t parity) {
    uint32_t done;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(done) : "r"(bar), "r"(parity) : "memory");
    return done != 0;
}

struct Shape { int stages; size_t smem; };

inline Shape shape_of(int C, int nh) {
    Shape s;
    size_t fixed = 1024 + 2 * (size_t)nh * 128 + 1024, stage = (size_t)(C / 64 + 1) * PIECE;
    s.stages = (int)((227 * 1024 - fixed) / stage);
    if (s.stages > MAX_STAGES) s.stages = MAX_STAGES;
    s.smem = fixed + s.stages * stage;
    if (s.smem < 120 * 1024) s.smem = 120 * 1024;           // one block an SM: it takes all of tensor memory
    return s;
}

// NH: heads of a block; C: the latent
template <int NH, int C>
__global__ void __launch_bounds__(256, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap map_rows, const __nv_bfloat16* __restrict__ q,
                        const int* __restrict__ block_table, int table_stride, int ring_pages, const int* __restrict__ seq_lens,
                        const int* __restrict__ seq_order, __nv_bfloat16* __restrict__ out, float* __restrict__ part_acc,
                        float* __restrict__ part_stats, int H, int R, int stages, float scale_log2,
                        const float* __restrict__ sinks, int* status) {
    constexpr int pieces = C / 64 + 1, values = (C + 127) / 128;         // of a row; accumulators
    // tensor memory: the queries (two elements a column), the scores, the accumulators
    constexpr uint32_t Q_COL = 0, S_COL = pieces * 32, O_COL = S_COL + KEYS, COLS = 512;
    static_assert(O_COL + values * NH <= COLS, "tensor memory");
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* ring = base;                                          // [stages][pieces][64][64]
    unsigned char* p_tile = ring + (size_t)stages * pieces * PIECE;      // [2][NH][64]
    uint64_t* full = reinterpret_cast<uint64_t*>(p_tile + 2 * NH * 128); // [8]
    uint64_t* empty = full + 8;                                          // [8]
    uint64_t* s_full = full + 16;                                        // the scores are complete
    uint64_t* s_free = full + 17;                                        // they have been read
    uint64_t* p_full = full + 18;                                        // [2] a buffer's weights are written (and O rescaled)
    uint64_t* o_full = full + 20;                                        // [2] its values have been added
    uint64_t* q_full = full + 22;
    uint64_t* go = full + 23;                                            // warps 4-7: rescale, or the end
    uint64_t* went = full + 24;                                          // they have rescaled
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(full + 25);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    float* alphas = reinterpret_cast<float*>(full + 26);                 // [NH] factors, at the end the sums
    float* maxima = alphas + NH;                                         // [NH]
    volatile int* at_end = reinterpret_cast<volatile int*>(maxima + NH);

    griddep_launch();
    int split = blockIdx.x, n_splits = gridDim.x;
    int seq = seq_order ? seq_order[blockIdx.z] : (int)blockIdx.z, head0 = blockIdx.y * NH;
    int len = seq_lens[seq];
    int n_pages = (len + KEYS - 1) / KEYS, per_split = (n_pages + n_splits - 1) / n_splits;
    int page_begin = min(split * per_split, n_pages);
    int n = min(page_begin + per_split, n_pages) - page_begin;           // pages of this slice
    const int* pages = block_table + (size_t)seq * table_stride;
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (int i = 0; i < 25; ++i) mbar_init(smem_u32(&full[i]), i == 24 ? 128 : (i == 17 || i == 18 || i == 19 || i == 22) ? 32 : 1);
        *abort_flag = 0;
        *at_end = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(tmem_slot)), "r"(COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    uint32_t tmem_base = *tmem_slot;

    if (warp == 1) {
        if (lane == 0) {
            auto request = [&](int j) {
                int s = j % stages;
                uint32_t bar = smem_u32(&full[s]);
                mbar_expect_tx(bar, pieces * PIECE);
                int row = pages[(page_begin + j) % ring_pages] * KEYS;
                for (int c = 0; c < pieces; ++c)
                    tma_load_2d(smem_u32(ring + ((size_t)s * pieces + c) * PIECE), &map_rows, bar, c * 64, row);
            };
            int j = 0;
            // pages of older positions are final: requested before the kernel in front has ended
            while (j < n && j < stages && (page_begin + j + 1) * KEYS <= len - 1) request(j++);
            griddep_wait();
            for (; j < n; ++j) {
                if (j >= stages && !mbar_wait(smem_u32(&empty[j % stages]), (j / stages - 1) & 1, abort_flag, status, 41)) break;
                request(j);
            }
        } else {
            griddep_wait();
        }
    } else if (warp == 2) {
        griddep_wait();
        if (lane == 0 && n > 0) {
            // D 32-bit, A and B bfloat16, M = 128. Scores: N = 64 keys, K-major. Values: N = NH heads, A MN-major.
            constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(KEYS >> 3) << 17) | (8u << 24);
            constexpr uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 15) | ((uint32_t)(NH >> 3) << 17) | (8u << 24);
            const uint64_t k_desc0 = smem_desc(smem_u32(ring)), v_desc0 = smem_desc_mn(smem_u32(ring), PIECE);
            const uint64_t p_desc0 = smem_desc(smem_u32(p_tile));
            int next_s = 0, next_o = 0, s_stage = 0, o_stage = 0;
            uint32_t s_phase = 0;
            long long since = 0;
            bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag, status, 42);
            tcgen05_fence_after();
            while (ok && next_o < n) {
                bool moved = false;
                if (next_s < n && mbar_test(smem_u32(&full[s_stage]), s_phase) &&
                    (next_s == 0 || mbar_test(smem_u32(s_free), (next_s - 1) & 1))) {
                    tcgen05_fence_after();
                    uint64_t k_desc = k_desc0 + (uint64_t)((s_stage * pieces * PIECE) >> 4);
                    // (all steps spelled out: the one lane that issues them sets their pace)
#pragma unroll
                    for (int k = 0; k < pieces * 4; ++k)
                        tcgen05_mma_ts(tmem_base + S_COL, tmem_base + Q_COL + k * 8,
                                       k_desc + (uint64_t)(((k >> 2) * PIECE + (k & 3) * 32) >> 4), idesc_s, k > 0 ? 1u : 0u);
                    tcgen05_commit(smem_u32(s_full));
                    ++next_s;
                    if (++s_stage == stages) { s_stage = 0; s_phase ^= 1; }
                    moved = true;
                }
                if (next_o < next_s && mbar_test(smem_u32(&p_full[next_o & 1]), (next_o >> 1) & 1)) {
                    tcgen05_fence_after();
                    uint64_t v_desc = v_desc0 + (uint64_t)((o_stage * pieces * PIECE) >> 4);
                    uint64_t p_desc = p_desc0 + (uint64_t)(((next_o & 1) * NH * 128) >> 4);
#pragma unroll
                    for (int m = 0; m < values; ++m)
#pragma unroll
                        for (int k = 0; k < KEYS / 16; ++k)           // 16 keys: 2,048 bytes of rows, 32 bytes of P
                            tcgen05_mma(tmem_base + O_COL + m * NH, v_desc + (uint64_t)((2 * m * PIECE + k * 2048) >> 4),
                                        p_desc + 2 * k, idesc_o, (next_o > 0 || k > 0) ? 1u : 0u);
                    tcgen05_commit(smem_u32(&o_full[next_o & 1]));
                    tcgen05_commit(smem_u32(&empty[o_stage]));
                    ++next_o;
                    if (++o_stage == stages) o_stage = 0;
                    moved = true;
                }
                if (moved) {
                    since = 0;
                } else {
                    if (*abort_flag) break;
                    long long now = clock64();
                    if (since == 0) since = now;
                    else if (now - since > WAIT_CYCLES) {
                        *abort_flag = 1;
                        if (status) atomicCAS(status, 0, 43);
                        break;
                    }
                }
            }
        }
    } else if (warp == 0) {
        griddep_wait();
        // the queries, a lane a head, into tensor memory (zeros beyond the head count and beyond the row)
        const bool live = lane < NH && head0 + lane < H;
        const __nv_bfloat16* row_q = behind_wait(q) + ((size_t)seq * H + head0 + (live ? lane : 0)) * (C + R);
#pragma unroll 1
        for (int c0 = 0; c0 < pieces; c0 += 3) {                     // three pieces' loads in flight
            uint4 v[3][8];
#pragma unroll
            for (int c = 0; c < 3; ++c)
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    int at = (c0 + c) * 64 + i * 8;
                    v[c][i] = live && at < C + R ? *reinterpret_cast<const uint4*>(row_q + at) : make_uint4(0u, 0u, 0u, 0u);
                }
#pragma unroll
            for (int c = 0; c < 3; ++c) {
                if (c0 + c >= pieces) break;
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t r[16];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        r[4 * i] = v[c][half * 4 + i].x; r[4 * i + 1] = v[c][half * 4 + i].y;
                        r[4 * i + 2] = v[c][half * 4 + i].z; r[4 * i + 3] = v[c][half * 4 + i].w;
                    }
                    tmem_st16(tmem_base + Q_COL + (c0 + c) * 32 + half * 16, r);
                }
            }
        }
        tmem_st_wait();
        tcgen05_fence_before();
        mbar_arrive(smem_u32(q_full));
        float run_max = -INFINITY, run_sum = 0.f;
        bool ok = true;
        int rescales = 0;
        for (int j = 0; j < n && ok; ++j) {
            int b = j & 1, phase = (j >> 1) & 1;
            ok = mbar_wait(smem_u32(s_full), j & 1, abort_flag, status, 44);
            if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
            tcgen05_fence_after();
            uint32_t ra[32], rb[32];
            tmem_ld32_start(tmem_base + S_COL, ra);
            tmem_ld32_start(tmem_base + S_COL + 32, rb);
            tmem_ld32_wait(ra);
            tmem_ld32_wait(rb);
            tcgen05_fence_before();
            mbar_arrive(smem_u32(s_free));
            int left = len - (page_begin + j) * KEYS;                // keys of this page that exist
            if (left < KEYS) {
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    if (i >= left) ra[i] = 0xff800000u;              // -inf
                    if (32 + i >= left) rb[i] = 0xff800000u;
                }
            }
            float block_max = -INFINITY;
#pragma unroll
            for (int i = 0; i < 32; ++i) block_max = max3(block_max, __uint_as_float(ra[i]), __uint_as_float(rb[i]));
            bool move = j == 0 || (block_max - run_max) * scale_log2 > 8.f;
            float new_max = move ? block_max : run_max;
            float alpha = (move && j > 0) ? fast_exp2((run_max - new_max) * scale_log2) : 1.f;
            float shift = new_max * scale_log2, add = 0.f;
            run_max = new_max;
            if (j >= 2) ok = mbar_wait(smem_u32(&o_full[b]), phase ^ 1, abort_flag, status, 45);          // P's buffer has been read
            if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
            unsigned char* row = p_tile + (b * NH + (lane < NH ? lane : 0)) * 128;
            auto weights = [&](const uint32_t (&r)[32], int half) {
#pragma unroll
                for (int c = 0; c < 4; ++c) {                        // 8 keys: 16 bytes
                    uint32_t packed[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        float p0 = fast_exp2(fmaf(__uint_as_float(r[8 * c + 2 * i]), scale_log2, -shift));
                        float p1 = fast_exp2(fmaf(__uint_as_float(r[8 * c + 2 * i + 1]), scale_log2, -shift));
                        add += p0 + p1;
                        packed[i] = pack_bf16(p0, p1);
                    }
                    if (lane < NH)
                        *reinterpret_cast<uint4*>(row + (((half * 4 + c) ^ (lane & 7)) << 4)) =
                            make_uint4(packed[0], packed[1], packed[2], packed[3]);
                }
            };
            weights(ra, 0);
            weights(rb, 1);
            run_sum = run_sum * alpha + add;
            if (!live) alpha = 1.f;                                  // (no head: whatever its scores are)
            if (j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
                ok = mbar_wait(smem_u32(&o_full[b ^ 1]), ((j - 1) >> 1) & 1, abort_flag, status, 46);     // the page before has been added
                if (lane < NH) alphas[lane] = alpha;
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(go));
                ok = ok && mbar_wait(smem_u32(went), rescales & 1, abort_flag, status, 47);
                ++rescales;
            }
            if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
            fence_async_shared();
            tcgen05_fence_before();
            mbar_arrive(smem_u32(&p_full[b]));
        }
        // what the result needs, then the signal
        if (sinks && n_splits == 1 && live) run_sum += sink_share(sinks[head0 + lane], run_max * scale_log2);
        if (lane < NH) { alphas[lane] = run_sum; maxima[lane] = run_max; }
        if (lane == 0) *at_end = 1;
        __threadfence_block();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(go));
    } else if (warp >= 4) {
        griddep_wait();
        int quarter = warp & 3;
        uint32_t lane_addr = tmem_base + O_COL + ((uint32_t)(quarter * 32) << 16);
        bool ok = true;
        for (int turn = 0;; ++turn) {
            ok = mbar_wait(smem_u32(go), turn & 1, abort_flag, status, 48);
            if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
            if (*at_end) break;
            tcgen05_fence_after();
#pragma unroll 1
            for (int c = 0; c < values * NH; c += 16) {
                uint32_t r[16];
                tmem_ld16(lane_addr + c, r);
#pragma unroll
                for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alphas[(c % NH) + i]);
                tmem_st16(lane_addr + c, r);
            }
            tmem_st_wait();
            tcgen05_fence_before();
            mbar_arrive(smem_u32(went));
        }
        if (ok && n > 0) ok = mbar_wait(smem_u32(&o_full[(n - 1) & 1]), ((n - 1) >> 1) & 1, abort_flag, status, 49);
        if (__all_sync(0xffffffffu, ok)) {
            tcgen05_fence_after();
            int heads = min(NH, H - head0);
            size_t row0 = (size_t)seq * H + head0;
            if (n_splits > 1 && warp == 4 && lane < heads) {
                float* to = part_stats + ((row0 + lane) * n_splits + split) * 2;
                to[0] = n > 0 ? maxima[lane] * scale_log2 : -INFINITY;
                to[1] = n > 0 ? alphas[lane] : 0.f;
            }
#pragma unroll 1
            for (int m = 0; m < values; ++m) {
                int d = m * 128 + quarter * 32 + lane;
#pragma unroll
                for (int c = 0; c < NH; c += 16) {
                    uint32_t r[16];
                    if (n > 0) tmem_ld16(lane_addr + m * NH + c, r);
                    if (d >= C) continue;
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        if (c + i >= heads) break;
                        float v = n > 0 ? __uint_as_float(r[i]) : 0.f;
                        if (n_splits == 1) out[(row0 + c + i) * C + d] = __float2bfloat16_rn(v / alphas[c + i]);
                        else part_acc[((row0 + c + i) * n_splits + split) * C + d] = v;
                    }
                }
            }
        }
    } else {
        griddep_wait();
    }

    tcgen05_fence_before();
    __syncthreads();
    if (*abort_flag) {
        for (int i = 0; i < 100; ++i) __nanosleep(10000);          // copies in flight land before shared memory is given up
        __syncthreads();
    }
    if (warp == 2) {
        tcgen05_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(COLS) : "memory");
    }
}

}  // namespace decode

// block (row): the slices' weighted values, maxima (base-2 units) and sums merged in slice order
constexpr int MAX_SPLITS = 32;
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_stats, __nv_bfloat16* __restrict__ out,
                      int C, int n_splits, int H, const float* __restrict__ sinks) {
    griddep_launch();
    griddep_wait();
    part_acc = behind_wait(part_acc);
    part_stats = behind_wait(part_stats);
    __shared__ float shares[MAX_SPLITS];
    size_t row = blockIdx.x;
    const float* stats = part_stats + row * n_splits * 2;
    if (threadIdx.x < 32) {                                // a lane a slice: its share of the result
        int s = threadIdx.x;
        float ms = s < n_splits ? stats[2 * s] : -INFINITY, m = warp_max(ms);
        float weight = ms == -INFINITY ? 0.f : exp2f(ms - m);
        float total = warp_sum(s < n_splits ? stats[2 * s + 1] * weight : 0.f);
        if (sinks) total += sink_share(sinks[row % H], m);
        if (s < n_splits) shares[s] = weight / total;
    }
    __syncthreads();
    for (int c = threadIdx.x * 4; c < C; c += 128 * 4) {
        float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
        for (int s = 0; s < n_splits; ++s) {
            float4 a = *reinterpret_cast<const float4*>(part_acc + (row * n_splits + s) * C + c);
            float share = shares[s];
            v[0] = fmaf(a.x, share, v[0]); v[1] = fmaf(a.y, share, v[1]);
            v[2] = fmaf(a.z, share, v[2]); v[3] = fmaf(a.w, share, v[3]);
        }
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(out + row * C + c) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    }
}

namespace {
struct TilePlan { int row_elems, mt; size_t smem; };

size_t tile_smem(int row_elems, int mt) {
    return (size_t)(2 * LLMB_PAGE + 16 * mt) * row_elems * 2 + 16 * mt * 128 + sizeof(float) * (8 / mt + 1) * 16 * mt;
}
// rows: (token, head) pairs the longest sequence of the step brings
TilePlan plan_tiles(int C, int width, int rows) {
    TilePlan p;
    int nt = C <= 64 ? 1 : C <= 128 ? 2 : C <= 256 ? 4 : 8;
    p.row_elems = (width + 63) / 64 * 64;
    if (p.row_elems < 64 * nt) p.row_elems = 64 * nt;
    p.mt = rows <= 16 ? 1 : rows <= 32 ? 2 : 4;
    while (p.mt > 1 && tile_smem(p.row_elems, p.mt) > 227 * 1024) p.mt /= 2;
    p.smem = tile_smem(p.row_elems, p.mt);
    return p;
}
}  // namespace

// Rows of a tile for a step whose longest sequence brings `rows` (token, head) pairs.
LLMB_EXPORT int llmb_latent_tile_rows(int C, int R, int rows) { return 16 * plan_tiles(C, C + R, rows).mt; }
// Whether two blocks of such a tile fit on an SM.
LLMB_EXPORT int llmb_latent_tile_pairs(int C, int R, int rows) { return plan_tiles(C, C + R, rows).smem <= 113 * 1024 ? 1 : 0; }
LLMB_EXPORT long long llmb_latent_scratch_floats(int n_tokens, int H, int C, int n_splits) {
    return (long long)n_tokens * H * n_splits * (C + 2);
}

// q [T, H, C + R] (contiguous), cache [pages, 1, 64, C + R], out [T, H, C]; all bfloat16. max_new: the most new tokens
// of a sequence. scratch: llmb_latent_scratch_floats where n_splits > 1.
LLMB_EXPORT int llmb_latent_attention(const void* q, const void* cache, const int* block_table, int table_stride,
                                      int ring_pages, const int* cu_seqlens, const int* seq_lens, const int* seq_order, void* out,
                                      float* scratch, long long scratch_floats, int n_tokens, int n_seqs, int max_new, int H,
                                      int C, int R, float scale, const float* sinks, int n_splits, cudaStream_t stream) {
    if (n_seqs == 0 || max_new == 0) return LLMB_OK;
    LLMB_REQUIRE(H > 0 && C > 0 && R > 0 && C % 8 == 0 && R % 8 == 0 && C <= 512 && C + R <= 640,
                 "latent_attention: rows of %d + %d (multiples of 8, up to 512 and 640 in all)", C, R);
    LLMB_REQUIRE(n_seqs <= 65535 && ring_pages > 0 && n_splits >= 1 && n_splits <= MAX_SPLITS && scale > 0.f, "latent_attention: bad sizes");
    LLMB_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15) == 0,
                 "latent_attention: operands must be 16-byte aligned");
    LLMB_REQUIRE(n_splits == 1 || (scratch && scratch_floats >= llmb_latent_scratch_floats(n_tokens, H, C, n_splits)),
                 "latent_attention: scratch too small");
    TilePlan p = plan_tiles(C, C + R, max_new * H);
    LLMB_REQUIRE(p.smem <= 227 * 1024, "latent_attention: %zu bytes of shared memory", p.smem);
    int tiles = ceil_div((long long)max_new * H, 16 * p.mt);
    LLMB_REQUIRE(tiles <= 65535, "latent_attention: %d tiles of a sequence", tiles);
    dim3 grid(n_splits, tiles, n_seqs);
    float* part_acc = scratch;
    float* part_stats = scratch ? scratch + (long long)n_tokens * H * n_splits * C : nullptr;
#define LLMB_TILES_AS(MT, NT)                                                                                             \
    do {                                                                                                                  \
        static size_t configured = 0;                                                                                     \
        if (configured < p.smem) {                                                                                        \
            LLMB_CUDA(cudaFuncSetAttribute(latent_tiles_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)p.smem)); \
            configured = p.smem;                                                                                          \
        }                                                                                                                 \
        LLMB_CUDA(llmb::launch(latent_tiles_kernel<MT, NT>, grid, dim3(THREADS), p.smem, stream, true,                    \
                               (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, block_table, table_stride, ring_pages, \
                               cu_seqlens, seq_lens, seq_order, (__nv_bfloat16*)out, part_acc, part_stats, H, C, C + R,   \
                               p.row_elems, scale * 1.4426950408889634f, sinks));                                         \
    } while (0)
#define LLMB_TILES(MT)                                 \
    do {                                               \
        if (C <= 64) LLMB_TILES_AS(MT, 1);             \
        else if (C <= 128) LLMB_TILES_AS(MT, 2);       \
        else if (C <= 256) LLMB_TILES_AS(MT, 4);       \
        else LLMB_TILES_AS(MT, 8);                     \
    } while (0)
    if (p.mt == 1) LLMB_TILES(1);
    else if (p.mt == 2) LLMB_TILES(2);
    else LLMB_TILES(4);
#undef LLMB_TILES
#undef LLMB_TILES_AS
    int code = check_launch("latent_attention");
    if (code || n_splits == 1) return code;
    LLMB_CUDA(llmb::launch(latent_combine_kernel, dim3(n_tokens * H), dim3(128), 0, stream, true, (const float*)part_acc,
                           (const float*)part_stats, (__nv_bfloat16*)out, C, n_splits, H, sinks));
    return check_launch("latent_attention_combine");
}
LLMB_PACKED(llmb_latent_attention)

LLMB_EXPORT int llmb_latent_attention_status() {
    int* s = llmb::tc::status_word();
    if (!s) return -1;
    int v = *s;
    *s = 0;
    return v;
}

// A step of one token a sequence: q [n_seqs, H, C + R] (contiguous), cache [n_pages, 1, 64, C + R], out [n_seqs, H, C]; all
// bfloat16. scratch as in llmb_latent_attention.
LLMB_EXPORT int llmb_latent_decode_tc(const void* q, const void* cache, int n_pages, const int* block_table, int table_stride,
                                      int ring_pages, const int* seq_lens, const int* seq_order, void* out, float* scratch,
                                      long long scratch_floats, int n_seqs, int H, int C, int R, float scale,
                                      const float* sinks, int n_splits, cudaStream_t stream) {
    if (n_seqs == 0) return LLMB_OK;
    LLMB_REQUIRE(H > 0 && (C == 64 || C == 128 || C == 256 || C == 512) && R > 0 && R <= 64 && R % 8 == 0,
                 "latent_decode_tc: rows of %d + %d (64, 128, 256 or 512, a multiple of 8 up to 64)", C, R);
    LLMB_REQUIRE(n_seqs <= 65535 && n_pages > 0 && ring_pages > 0 && n_splits >= 1 && n_splits <= MAX_SPLITS && scale > 0.f, "latent_decode_tc: bad sizes");
    LLMB_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15) == 0,
                 "latent_decode_tc: operands must be 16-byte aligned");
    LLMB_REQUIRE(n_splits == 1 || (scratch && scratch_floats >= llmb_latent_scratch_floats(n_seqs, H, C, n_splits)),
                 "latent_decode_tc: scratch too small");
    int nh = H <= 16 ? 16 : 32;
    decode::Shape s = decode::shape_of(C, nh);
    LLMB_REQUIRE(s.stages >= 2 && s.smem <= 227 * 1024, "latent_decode_tc: %zu bytes of shared memory", s.smem);
    CUtensorMap map_rows;
    int code;
    if ((code = llmb::tc::make_map_2d(&map_rows, cache, (long long)n_pages * LLMB_PAGE, C + R, C + R, 64, decode::KEYS))) return code;
    float* part_acc = scratch;
    float* part_stats = scratch ? scratch + (long long)n_seqs * H * n_splits * C : nullptr;
    int* status_dev = nullptr;
    int* status_host = llmb::tc::status_word();
    if (status_host) LLMB_CUDA(cudaHostGetDevicePointer((void**)&status_dev, status_host, 0));
#define LLMB_DECODE_AS(NH, CC)                                                                                            \
    do {                                                                                                                  \
        static bool configured = false;                                                                                   \
        if (!configured) {                                                                                                \
            LLMB_CUDA(cudaFuncSetAttribute(decode::latent_decode_tc_kernel<NH, CC>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           (int)s.smem));                                                                 \
            configured = true;                                                                                            \
        }                                                                                                                 \
        LLMB_CUDA(llmb::launch(decode::latent_decode_tc_kernel<NH, CC>, dim3(n_splits, ceil_div(H, NH), n_seqs), dim3(256), s.smem, \
                               stream, true, map_rows, (const __nv_bfloat16*)q, block_table, table_stride, ring_pages, seq_lens, seq_order, \
                               (__nv_bfloat16*)out, part_acc, part_stats, H, R, s.stages, scale * 1.4426950408889634f, sinks, status_dev)); \
    } while (0)
#define LLMB_DECODE(NH)                               \
    do {                                              \
        if (C == 64) LLMB_DECODE_AS(NH, 64);          \
        else if (C == 128) LLMB_DECODE_AS(NH, 128);   \
        else if (C == 256) LLMB_DECODE_AS(NH, 256);   \
        else LLMB_DECODE_AS(NH, 512);                 \
    } while (0)
    if (nh == 16) LLMB_DECODE(16);
    else LLMB_DECODE(32);
#undef LLMB_DECODE
#undef LLMB_DECODE_AS
    code = check_launch("latent_decode_tc");
    if (code || n_splits == 1) return code;
    LLMB_CUDA(llmb::launch(latent_combine_kernel, dim3(n_seqs * H), dim3(128), 0, stream, true, (const float*)part_acc,
                           (const float*)part_stats, (__nv_bfloat16*)out, C, n_splits, H, sinks));
    return check_launch("latent_attention_combine");
}
LLMB_PACKED(llmb_latent_decode_tc)
