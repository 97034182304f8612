// Prefill attention: the new tokens of every sequence of a step attend, causally,
// to everything their sequence has in the paged cache (their own keys included),
// bfloat16, tiled so that nothing of the size of the context is ever stored.
//
// The scheme is the flash prefill of MythEclipse/llm (attention_prefill_mma,
// apps/engine/kernels/gpu.cu:1444-1655): query tiles against key tiles with
// mma.sync, a running (max, sum) per query row and the accumulator rescaled by
// exp(m_old - m_new) (gpu.cu:1560-1613), probabilities reused as the A operand of
// the second product (gpu.cu:1615-1631), and the heaviest query tile of a
// sequence launched first (gpu.cu:1457-1461). What is different: sequences of
// unequal length in one launch, keys and values read page by page from the slot
// cache through a block table, any group size (one head per block; the heads
// of a group find their shared pages in L2), head sizes 32 to 128.
//
// * grid (query tiles, heads, sequences); tile 0 of the grid is a sequence's last
//   64 queries. A block has four warps of 16 query rows each.
// * K and V of a page (64 keys) come through shared memory with cp.async, two
//   pages in flight; S = Q K^T and O += P V are mma.sync.m16n8k16 with fragments
//   from ldmatrix / ldmatrix.trans; softmax statistics are 32-bit, exponentials
//   base 2 with the scale folded in.
// * a key at position j is visible to the query at position p iff j <= p; only
//   the pages that cross a warp's diagonal are masked element by element, and
//   pages wholly above it are skipped by that warp.
//
// * with a window w a query at position p sees the keys j with p - w < j <= p: a tile starts at the
//   page of its first query's oldest visible key (pages before it are neither read nor needed: they
//   may have left a ring of pages), the pages that cross a row's lower edge are masked element by
//   element, and a row whose first pages hold nothing it sees keeps a maximum of -inf without NaN.
// * optional, all in the epilogue and in 32-bit: `sinks` [heads] (e^sink joins the head's
//   denominator: no key, no value, not scaled), `gate` [T, heads] (the head's result times
//   sigmoid(gate)), `out_scale`. `bias` [heads, span]: bias[h, min(p - j, span - 1)] is added to the
//   scaled score of key j; a page whose keys are all span - 1 or further behind every query of a warp adds one number
//   inside the exponent's multiply-add. When the value cache IS the key cache (a mixer whose cached rows
//   serve as both), a page is fetched once and both products read the same tile.
//
// Refused (the generic kernel serves them): 32-bit caches, head sizes other than 32, 64, 96, 128.
#include "common.cuh"
#include "mma.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_attention_prefill)

constexpr int WARPS = 4;
constexpr int BQ = WARPS * 16;               // queries per block
constexpr int STAGES = 2;
constexpr int PAD = 8;

// 2^x by the hardware approximation (relative error about 2^-22; 2^-inf = 0)
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int D, bool BIAS>
__global__ void __launch_bounds__(WARPS * 32, 3)          // three blocks per SM: at most 170 registers
attention_prefill_kernel(const __nv_bfloat16* __restrict__ q, int q_stride,
                         const __nv_bfloat16* __restrict__ k_cache,
                         const __nv_bfloat16* __restrict__ v_cache,
                         const int* __restrict__ block_table, int table_stride, int ring_pages,
                         const int* __restrict__ cu_seqlens, const int* __restrict__ seq_lens,
                         __nv_bfloat16* __restrict__ out, int out_stride, int n_heads,
                         int n_kv_heads, float scale_log2, int window, const float* __restrict__ sinks,
                         const __nv_bfloat16* __restrict__ gate, int gate_stride, float out_scale,
                         float cap_raw, const float* __restrict__ bias, int span) {
    constexpr int LDS = D + PAD;
    const bool values_are_keys = k_cache == v_cache;
    constexpr int PAGE_ELEMS = LLMB_PAGE * LDS;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* smem = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // [STAGES][2][64][LDS]

    int seq = blockIdx.z, head = blockIdx.x;
    int first_token = cu_seqlens[seq];
    int n_new = cu_seqlens[seq + 1] - first_token;
    int n_tiles = (n_new + BQ - 1) / BQ;
    if ((int)blockIdx.y >= n_tiles) return;
    int tile = n_tiles - 1 - blockIdx.y;                 // the heaviest tile of every head first (x runs fastest)
    int start = seq_lens[seq] - n_new;                   // position of the sequence's first new token
    int kv_head = head / (n_heads / n_kv_heads);
    int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int* pages = block_table + (size_t)seq * table_stride;

    int row0 = tile * BQ + warp * 16 + g, row1 = row0 + 8;      // index among the new tokens
    int pos0 = start + row0, pos1 = start + row1;               // positions (also of rows beyond n_new)
    int warp_last_pos = start + min(tile * BQ + warp * 16 + 15, n_new - 1);
    if (tile * BQ + warp * 16 >= n_new) warp_last_pos = -1;    // no query in this warp: skip every page
    int tile_last_pos = start + min(tile * BQ + BQ - 1, n_new - 1);
    int n_pages = tile_last_pos / LLMB_PAGE + 1;
    // with a window: the oldest key that the tile's first query sees, and this warp's first query
    int tile_oldest = window > 0 ? max(start + tile * BQ - window + 1, 0) : 0;
    int first_page = tile_oldest / LLMB_PAGE;
    int warp_oldest = window > 0 ? max(start + tile * BQ + warp * 16 - window + 1, 0) : 0;
    int low0 = window > 0 ? pos0 - window + 1 : 0, low1 = window > 0 ? pos1 - window + 1 : 0;

    uint32_t qa[D / 16][4];
    {
        const __nv_bfloat16* q0 = q + (size_t)(first_token + row0) * q_stride + (size_t)head * D;
        const __nv_bfloat16* q1 = q + (size_t)(first_token + row1) * q_stride + (size_t)head * D;
        bool ok0 = row0 < n_new, ok1 = row1 < n_new;
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
            qa[ks][0] = ok0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 2 * t) : 0u;
            qa[ks][1] = ok1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 2 * t) : 0u;
            qa[ks][2] = ok0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 8 + 2 * t) : 0u;
            qa[ks][3] = ok1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 8 + 2 * t) : 0u;
        }
    }

    auto load_page = [&](int logical_page, int stage) {
        int page = pages[logical_page % ring_pages];
        size_t base = ((size_t)page * n_kv_heads + kv_head) * LLMB_PAGE * D;
        __nv_bfloat16* ks = smem + (size_t)stage * 2 * PAGE_ELEMS;
        __nv_bfloat16* vs = ks + PAGE_ELEMS;
        constexpr int CHUNKS_PER_ROW = D / 8;
        for (int c = tid; c < LLMB_PAGE * CHUNKS_PER_ROW; c += WARPS * 32) {
            int row = c / CHUNKS_PER_ROW, col = (c % CHUNKS_PER_ROW) * 8;
            cp_async16(ks + row * LDS + col, k_cache + base + (size_t)row * D + col);
            if (!values_are_keys) cp_async16(vs + row * LDS + col, v_cache + base + (size_t)row * D + col);
        }
    };

    float acc[D / 8][4];
#pragma unroll
    for (int n = 0; n < D / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[n][i] = 0.f;
    float max0 = -INFINITY, max1 = -INFINITY, sum0 = 0.f, sum1 = 0.f;

    load_page(first_page, first_page % STAGES);
    cp_async_commit();
    for (int p = first_page; p < n_pages; ++p) {
        cp_async_wait<0>();
        __syncthreads();                                // page p landed; everyone is done with page p - 1
        if (p + 1 < n_pages) load_page(p + 1, (p + 1) % STAGES);
        cp_async_commit();
        int key0 = p * LLMB_PAGE;
        if (key0 > warp_last_pos) continue;             // wholly above this warp's diagonal
        if (key0 + LLMB_PAGE <= warp_oldest) continue;  // wholly before this warp's windows

        const __nv_bfloat16* ks = smem + (size_t)(p % STAGES) * 2 * PAGE_ELEMS;
        const __nv_bfloat16* vs = values_are_keys ? ks : ks + PAGE_ELEMS;
        float s[8][4];
#pragma unroll
        for (int nb = 0; nb < 8; ++nb)
#pragma unroll
            for (int i = 0; i < 4; ++i) s[nb][i] = 0.f;
#pragma unroll
        for (int kstep = 0; kstep < D / 16; ++kstep) {
#pragma unroll
            for (int nb = 0; nb < 8; nb += 2) {
                uint32_t b[4];
                int row = nb * 8 + (lane >> 4) * 8 + (lane & 7);
                int col = kstep * 16 + ((lane >> 3) & 1) * 8;
                ldmatrix_x4(b, ks + row * LDS + col);
                mma_bf16(s[nb], qa[kstep][0], qa[kstep][1], qa[kstep][2], qa[kstep][3], b[0], b[1]);
                mma_bf16(s[nb + 1], qa[kstep][0], qa[kstep][1], qa[kstep][2], qa[kstep][3], b[2], b[3]);
            }
        }
        // s[nb][0..1]: row0, keys key0 + nb * 8 + 2t, +1; s[nb][2..3]: row1, the same keys.
        // A soft cap bounds the scaled score: c tanh(s * scale / c); cap_raw = c / scale keeps it in raw units.
        if (cap_raw > 0.f) {
            float inv_cap = 1.0f / cap_raw;
#pragma unroll
            for (int nb = 0; nb < 8; ++nb)
#pragma unroll
                for (int i = 0; i < 4; ++i) s[nb][i] = cap_raw * tanhf(s[nb][i] * inv_cap);
        }
        // A bias by distance: near keys take theirs here, in raw units (the scale is positive); to far ones one number
        // belongs, which enters where the maxima and the exponents are formed.
        float far_raw = 0.f;
        if constexpr (BIAS) {
            const float* mine = bias + (size_t)head * span;
            float inv_scale = 1.4426950408889634f / scale_log2;
            if (start + tile * BQ + warp * 16 - (key0 + LLMB_PAGE - 1) >= span - 1) {
                far_raw = mine[span - 1] * inv_scale;
            } else {
#pragma unroll
                for (int nb = 0; nb < 8; ++nb)
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        int key = key0 + nb * 8 + 2 * t + i;
                        s[nb][i] = fmaf(mine[max(0, min(pos0 - key, span - 1))], inv_scale, s[nb][i]);
                        s[nb][2 + i] = fmaf(mine[max(0, min(pos1 - key, span - 1))], inv_scale, s[nb][2 + i]);
                    }
            }
        }
        // Maxima are kept on the raw scores (the scale is positive); the scale and log2(e) are
        // applied inside the exponent with one fused multiply-add per score.
        bool diagonal = key0 + LLMB_PAGE - 1 > start + tile * BQ + warp * 16;   // some key may be hidden
        // with a window: some key may lie before the window of the warp's LAST row (the highest lower edge)
        bool lower = window > 0 && key0 < start + tile * BQ + warp * 16 + 15 - window + 1;
        float local0 = -INFINITY, local1 = -INFINITY;
#pragma unroll
        for (int nb = 0; nb < 8; ++nb) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                if (diagonal || lower) {
                    int key = key0 + nb * 8 + 2 * t + i;
                    if (key > pos0 || key < low0) s[nb][i] = -INFINITY;
                    if (key > pos1 || key < low1) s[nb][2 + i] = -INFINITY;
                }
                local0 = fmaxf(local0, s[nb][i]);
                local1 = fmaxf(local1, s[nb][2 + i]);
            }
        }
        local0 = fmaxf(local0, __shfl_xor_sync(0xffffffffu, local0, 1));
        local0 = fmaxf(local0, __shfl_xor_sync(0xffffffffu, local0, 2));
        local1 = fmaxf(local1, __shfl_xor_sync(0xffffffffu, local1, 1));
        local1 = fmaxf(local1, __shfl_xor_sync(0xffffffffu, local1, 2));
        // Without a window key 0 is visible to every row, so after page 0 both maxima are finite. With one, a
        // row may have seen nothing yet: its maximum stays -inf, and a reference of 0 keeps every term 0.
        if constexpr (BIAS) { local0 += far_raw; local1 += far_raw; }
        float new0 = fmaxf(max0, local0), new1 = fmaxf(max1, local1);
        float ref0 = new0 == -INFINITY ? 0.f : new0, ref1 = new1 == -INFINITY ? 0.f : new1;
        float rescale0 = fast_exp2((max0 - ref0) * scale_log2), rescale1 = fast_exp2((max1 - ref1) * scale_log2);
        max0 = new0;
        max1 = new1;
        float shift0 = (ref0 - far_raw) * scale_log2, shift1 = (ref1 - far_raw) * scale_log2;
        float add0 = 0.f, add1 = 0.f;
#pragma unroll
        for (int nb = 0; nb < 8; ++nb) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                s[nb][i] = fast_exp2(fmaf(s[nb][i], scale_log2, -shift0));
                s[nb][2 + i] = fast_exp2(fmaf(s[nb][2 + i], scale_log2, -shift1));
                add0 += s[nb][i];
                add1 += s[nb][2 + i];
            }
        }
        sum0 = sum0 * rescale0 + add0;
        sum1 = sum1 * rescale1 + add1;
#pragma unroll
        for (int n = 0; n < D / 8; ++n) {
            acc[n][0] *= rescale0; acc[n][1] *= rescale0;
            acc[n][2] *= rescale1; acc[n][3] *= rescale1;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t pa0 = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
            uint32_t pa1 = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
            uint32_t pa2 = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
            uint32_t pa3 = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
            for (int n = 0; n < D / 8; n += 2) {
                uint32_t b[4];
                int row = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
                int col = (n + (lane >> 4)) * 8;
                ldmatrix_x4_trans(b, vs + row * LDS + col);
                mma_bf16(acc[n], pa0, pa1, pa2, pa3, b[0], b[1]);
                mma_bf16(acc[n + 1], pa0, pa1, pa2, pa3, b[2], b[3]);
            }
        }
    }
    cp_async_wait<0>();

    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
    // sum and acc of a row are relative to e^(max * scale). A sink joins the denominator; where it exceeds
    // the row's maximum it becomes the reference, so that nothing overflows.
    float inv0, inv1;
    if (sinks) {
        float sink2 = sinks[head] * 1.4426950408889634f;
        float m0 = max0 * scale_log2, m1 = max1 * scale_log2;
        float r0 = fmaxf(m0, sink2), r1 = fmaxf(m1, sink2);
        float w0 = fast_exp2(m0 - r0), w1 = fast_exp2(m1 - r1);
        inv0 = w0 / (sum0 * w0 + fast_exp2(sink2 - r0));
        inv1 = w1 / (sum1 * w1 + fast_exp2(sink2 - r1));
    } else {
        inv0 = 1.0f / sum0;
        inv1 = 1.0f / sum1;
    }
    inv0 *= out_scale;
    inv1 *= out_scale;
    if (gate) {
        if (row0 < n_new) inv0 *= 1.0f / (1.0f + expf(-to_float(gate[(size_t)(first_token + row0) * gate_stride + head])));
        if (row1 < n_new) inv1 *= 1.0f / (1.0f + expf(-to_float(gate[(size_t)(first_token + row1) * gate_stride + head])));
    }
    __nv_bfloat16* o0 = out + (size_t)(first_token + row0) * out_stride + (size_t)head * D;
    __nv_bfloat16* o1 = out + (size_t)(first_token + row1) * out_stride + (size_t)head * D;
#pragma unroll
    for (int n = 0; n < D / 8; ++n) {
        if (row0 < n_new)
            *reinterpret_cast<__nv_bfloat162*>(o0 + n * 8 + 2 * t) = __floats2bfloat162_rn(acc[n][0] * inv0, acc[n][1] * inv0);
        if (row1 < n_new)
            *reinterpret_cast<__nv_bfloat162*>(o1 + n * 8 + 2 * t) = __floats2bfloat162_rn(acc[n][2] * inv1, acc[n][3] * inv1);
    }
}

template <int D>
static int launch(const void* q, int q_stride, const void* k_cache, const void* v_cache,
                  const int* block_table, int table_stride, int ring_pages, const int* cu_seqlens,
                  const int* seq_lens, void* out, int out_stride, int n_seqs, int max_new, int n_heads,
                  int n_kv_heads, float scale, int window, const float* sinks, const void* gate, int gate_stride,
                  float out_scale, float softcap, const float* bias, int span, cudaStream_t stream) {
    constexpr int LDS = D + PAD;
    size_t smem = (size_t)STAGES * 2 * LLMB_PAGE * LDS * sizeof(__nv_bfloat16);
    static bool configured = false;
    if (!configured) {
        LLMB_CUDA(cudaFuncSetAttribute(attention_prefill_kernel<D, false>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        LLMB_CUDA(cudaFuncSetAttribute(attention_prefill_kernel<D, true>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = true;
    }
    dim3 grid(n_heads, (max_new + BQ - 1) / BQ, n_seqs);
    auto kernel = bias ? attention_prefill_kernel<D, true> : attention_prefill_kernel<D, false>;
    kernel<<<grid, WARPS * 32, smem, stream>>>(
        (const __nv_bfloat16*)q, q_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache,
        block_table, table_stride, ring_pages, cu_seqlens, seq_lens, (__nv_bfloat16*)out, out_stride,
        n_heads, n_kv_heads, scale * 1.4426950408889634f, window, sinks, (const __nv_bfloat16*)gate, gate_stride,
        out_scale, softcap > 0.f ? softcap / scale : 0.f, bias, span);
    return check_launch("attention_prefill");
}

LLMB_EXPORT int llmb_attention_prefill_supports(int n_heads, int n_kv_heads, int head_dim, int window) {
    LLMB_REQUIRE(window >= 0, "attention_prefill: a window of %d", window);
    LLMB_REQUIRE(n_kv_heads > 0 && n_heads % n_kv_heads == 0,
                 "attention_prefill: %d heads are no multiple of %d kv heads", n_heads, n_kv_heads);
    LLMB_REQUIRE(head_dim == 32 || head_dim == 64 || head_dim == 96 || head_dim == 128,
                 "attention_prefill: head_dim %d (served: 32, 64, 96, 128)", head_dim);
    return LLMB_OK;
}

// q: the new tokens' queries, packed sequence after sequence [T, q_stride]; token i of sequence b
// is row cu_seqlens[b] + i and stands at position seq_lens[b] - n_new(b) + i, where seq_lens are
// the lengths after this step. max_new: the most new tokens any sequence brings.
LLMB_EXPORT int llmb_attention_prefill(const void* q, int q_stride, const void* k_cache,
                                       const void* v_cache, const int* block_table, int table_stride,
                                       int ring_pages, const int* cu_seqlens, const int* seq_lens,
                                       void* out, int out_stride, int n_seqs, int max_new,
                                       int n_heads, int n_kv_heads, int head_dim, float scale,
                                       int window, const float* sinks, const void* gate, int gate_stride,
                                       float out_scale, float softcap, const float* bias, int span,
                                       cudaStream_t stream) {
    if (n_seqs == 0 || max_new == 0) return LLMB_OK;
    LLMB_REQUIRE((softcap <= 0.f && !bias) || scale > 0.f, "attention_prefill: a soft cap or a bias needs a positive scale");
    LLMB_REQUIRE(!bias || (span > 0 && softcap <= 0.f), "attention_prefill: a bias with a soft cap, or an empty one");
    int code = llmb_attention_prefill_supports(n_heads, n_kv_heads, head_dim, window);
    if (code) return code;
    LLMB_REQUIRE(n_seqs <= 65535 && max_new / BQ < 65535 && ring_pages > 0, "attention_prefill: bad sizes");
    LLMB_REQUIRE(q_stride % 2 == 0 && out_stride % 2 == 0 && (reinterpret_cast<uintptr_t>(q) & 3) == 0 &&
                 (reinterpret_cast<uintptr_t>(out) & 3) == 0,
                 "attention_prefill: q and out must be 4-byte aligned with even row strides");
#define ARGS q, q_stride, k_cache, v_cache, block_table, table_stride, ring_pages, cu_seqlens, seq_lens, \
             out, out_stride, n_seqs, max_new, n_heads, n_kv_heads, scale, window, sinks, gate, gate_stride, \
             out_scale, softcap, bias, span, stream
    switch (head_dim) {
        case 32: return launch<32>(ARGS);
        case 64: return launch<64>(ARGS);
        case 96: return launch<96>(ARGS);
        default: return launch<128>(ARGS);
    }
#undef ARGS
}

// the packed doors of the launching entry points (common.cuh)
LLMB_PACKED(llmb_attention_prefill)
