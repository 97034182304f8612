// A residual of several streams x_1 .. x_S per token (Zhu et al., "Hyper-Connections"), X [T, S, width] in 32-bit.
//
// streams_embed   every stream of a token is its row of the embedding table. A pass's first kernel: it starts behind
//                 everything before it, so that kernels of the pass may read states of sequences before their own wait.
// streams_update  behind a part: y = the sum of a token's result rows (`terms` rows in index order), then, from the old
//                 streams, x_t <- sum_s mix[s, t] x_s + out[t] y; and in the same launch, where `read` is given, the next
//                 part's input: u = sum_s read[s] x_s (of the new streams), h = u / sqrt(mean(u^2) + eps) * gain.
// streams_read    that input alone, of the streams as they are, optionally of gathered tokens; without `read` u is
//                 the plain sum of the streams (what a model's last norm reads).
//
// All arithmetic is 32-bit; only h is rounded (to the run's dtype). A token's sums run in an order that depends on
// nothing but the width (streams in rising order; of a row a thread's elements in rising order, lanes as a
// butterfly, warps in order).
#include "common.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_streams)

constexpr int MAX_STREAMS = 16;

// The block's sum of its threads' values, HALVES each, as if HALVES * THREADS threads held one each: lanes as a butterfly, then
// the warps in order (value i of warp w counts as warp i * THREADS / 32 + w).
template <int THREADS, int HALVES>
__device__ __forceinline__ float block_sum(float (&v)[HALVES], float* scratch) {
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
    for (int i = 0; i < HALVES; ++i) {
        float sum = warp_sum(v[i]);
        if (lane == 0) scratch[i * (THREADS / 32) + warp] = sum;
    }
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < HALVES * THREADS / 32; ++w) total += scratch[w];
    return total;
}

template <int VEC> struct Pack { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Pack<VEC> load(const float* p);
template <> __device__ __forceinline__ Pack<1> load<1>(const float* p) { return {{*p}}; }
template <> __device__ __forceinline__ Pack<4> load<4>(const float* p) {
    float4 f = *reinterpret_cast<const float4*>(p);
    return {{f.x, f.y, f.z, f.w}};
}
__device__ __forceinline__ void store(float* p, const Pack<1>& a) { *p = a.v[0]; }
__device__ __forceinline__ void store(float* p, const Pack<4>& a) {
    *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
}
__device__ __forceinline__ void store(__nv_bfloat16* p, const Pack<1>& a) { *p = __float2bfloat16_rn(a.v[0]); }
__device__ __forceinline__ void store(__nv_bfloat16* p, const Pack<4>& a) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
streams_embed_kernel(const int* __restrict__ tokens, const T* __restrict__ table, float* __restrict__ X, int S, int width,
                     int vocab, float scale) {
    griddep_launch();
    griddep_wait();
    size_t t = blockIdx.x;
    int id = min(max(tokens[t], 0), vocab - 1);
    const T* row = table + (size_t)id * width;
    for (int c = threadIdx.x * VEC; c < width; c += 256 * VEC) {
        Pack<VEC> v;
        if constexpr (VEC == 4 && sizeof(T) == 2) {
            T raw[4];
            *reinterpret_cast<uint2*>(raw) = *reinterpret_cast<const uint2*>(row + c);
#pragma unroll
            for (int i = 0; i < 4; ++i) v.v[i] = to_float(raw[i]) * scale;
        } else if constexpr (VEC == 4) {
            v = load<4>(reinterpret_cast<const float*>(row) + c);
#pragma unroll
            for (int i = 0; i < 4; ++i) v.v[i] *= scale;
        } else {
            v.v[0] = to_float(row[c]) * scale;
        }
        for (int s = 0; s < S; ++s) store(X + (t * S + s) * width + c, v);
    }
}

// THREADS, HALVES: HALVES * THREADS columns' quads are a turn of the row. Two halves: few threads a block, several blocks an SM
// (many tokens); one: a token's row on more threads (few tokens). The sums are the same.
// STREAMS: the number of streams, or 0 for any number up to MAX_STREAMS (`n_streams`). `write` = [out (S) | mix (S, S)] (null:
// the streams stay), `read` [S] (null: ones). h null: no input is wanted.
template <typename TOut, int VEC, int THREADS, int HALVES, int STREAMS>
__global__ void __launch_bounds__(THREADS, HALVES == 2 ? 4 : 1)
streams_kernel(float* __restrict__ X, int n_streams, const float* __restrict__ y, int terms, const float* __restrict__ write,
               const float* __restrict__ read, const float* __restrict__ gain, float eps, const int* __restrict__ rows,
               TOut* __restrict__ h, int width) {
    constexpr int MOST = STREAMS > 0 ? STREAMS : MAX_STREAMS;
    const int S = STREAMS > 0 ? STREAMS : n_streams;
    extern __shared__ __align__(16) float row[];            // u [width]
    __shared__ float scratch[HALVES * THREADS / 32], coef[MAX_STREAMS * (MAX_STREAMS + 2)];     // read (S) | out (S) | mix (S, S)
    griddep_launch();
    for (int i = threadIdx.x; i < S; i += THREADS) coef[i] = read ? read[i] : 1.f;
    if (write)
        for (int i = threadIdx.x; i < S * (S + 1); i += THREADS) coef[S + i] = write[i];
    __syncthreads();
    griddep_wait();
    y = behind_wait(y);
    size_t r = blockIdx.x, t = rows ? (size_t)rows[r] : r;
    float* x = X + t * S * width;
    float sq[HALVES];
#pragma unroll
    for (int i = 0; i < HALVES; ++i) sq[i] = 0.f;
    auto turn = [&](int c, float& squares) {
        Pack<VEC> old[MOST], u;
#pragma unroll
        for (int s = 0; s < MOST; ++s)
            if (s < S) old[s] = load<VEC>(x + (size_t)s * width + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u.v[i] = 0.f;
        if (write) {
            const float* from = y + t * terms * width + c;
            Pack<VEC> sum = load<VEC>(from);
#pragma unroll 8
            for (int k = 1; k < terms; ++k) {
                Pack<VEC> a = load<VEC>(from + (size_t)k * width);
#pragma unroll
                for (int i = 0; i < VEC; ++i) sum.v[i] += a.v[i];
            }
#pragma unroll
            for (int to = 0; to < MOST; ++to) {
                if (to >= S) break;
                Pack<VEC> now;
#pragma unroll
                for (int i = 0; i < VEC; ++i) now.v[i] = 0.f;
#pragma unroll
                for (int s = 0; s < MOST; ++s) {
                    if (s >= S) break;
                    float m = coef[2 * S + s * S + to];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) now.v[i] = fmaf(m, old[s].v[i], now.v[i]);
                }
                float w = coef[S + to], in = coef[to];
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    now.v[i] = fmaf(w, sum.v[i], now.v[i]);
                    u.v[i] = fmaf(in, now.v[i], u.v[i]);
                }
                store(x + (size_t)to * width + c, now);
            }
        } else {
#pragma unroll
            for (int s = 0; s < MOST; ++s) {
                if (s >= S) break;
#pragma unroll
                for (int i = 0; i < VEC; ++i) u.v[i] = fmaf(coef[s], old[s].v[i], u.v[i]);
            }
        }
        if (h) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) squares = fmaf(u.v[i], u.v[i], squares);
            store(row + c, u);
        }
    };
    for (int c0 = threadIdx.x * VEC; c0 < width; c0 += HALVES * THREADS * VEC)
#pragma unroll
        for (int half = 0; half < HALVES; ++half)
            if (half == 0 || c0 + half * THREADS * VEC < width) turn(c0 + half * THREADS * VEC, sq[half]);
    if (!h) return;
    float factor = 1.0f / sqrtf(block_sum<THREADS, HALVES>(sq, scratch) / (float)width + eps);
    for (int c = threadIdx.x * VEC; c < width; c += THREADS * VEC) {
        Pack<VEC> g = load<VEC>(gain + c), a;
#pragma unroll
        for (int i = 0; i < VEC; ++i) a.v[i] = row[c + i] * factor * g.v[i];
        store(h + r * width + c, a);
    }
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// X float32 [T, S, width]; tokens int32 [T]; table [vocab, width] in `dtype`.
LLMB_EXPORT int llmb_streams_embed(const int* tokens, const void* table, int dtype, float* X, int n_tokens, int S, int width,
                                   int vocab, float scale, cudaStream_t stream) {
    if (n_tokens == 0) return LLMB_OK;
    LLMB_REQUIRE(S >= 1 && S <= MAX_STREAMS && width > 0 && vocab > 0, "streams_embed: %d streams (up to %d) of %d", S, MAX_STREAMS, width);
    bool vector = width % 4 == 0 && aligned16(table) && aligned16(X);
#define LLMB_STREAMS_EMBED(T, VEC)                                                                                         \
    LLMB_CUDA(llmb::launch(streams_embed_kernel<T, VEC>, dim3(n_tokens), dim3(256), 0, stream, false, tokens, (const T*)table, X, \
                           S, width, vocab, scale))
    if (dtype == LLMB_DTYPE_F32) { if (vector) LLMB_STREAMS_EMBED(float, 4); else LLMB_STREAMS_EMBED(float, 1); }
    else if (dtype == LLMB_DTYPE_BF16) { if (vector) LLMB_STREAMS_EMBED(__nv_bfloat16, 4); else LLMB_STREAMS_EMBED(__nv_bfloat16, 1); }
#undef LLMB_STREAMS_EMBED
    else return fail(LLMB_ERR_ARGUMENT, "streams_embed: unknown dtype %d", dtype);
    return check_launch("streams_embed");
}
LLMB_PACKED(llmb_streams_embed)

// One launch of the above: update (write given; y float32 [T * terms, width]), read (h [n_rows, width] in h_dtype and gain
// [width] given) or both. n_rows: tokens, or the gathered `rows` (read only).
LLMB_EXPORT int llmb_streams(float* X, int S, const float* y, int terms, const float* write, const float* read, const float* gain,
                             float eps, const int* rows, void* h, int h_dtype, int n_rows, int width, cudaStream_t stream) {
    if (n_rows == 0) return LLMB_OK;
    size_t smem = h ? sizeof(float) * (size_t)width : 0;
    LLMB_REQUIRE(S >= 1 && S <= MAX_STREAMS && width > 0 && smem <= 200 * 1024, "streams: %d streams (up to %d) of %d", S, MAX_STREAMS, width);
    LLMB_REQUIRE((write && y && terms > 0 && !rows) || (!write && h), "streams: an update needs a result, and gathered rows are only read");
    LLMB_REQUIRE(!h || gain, "streams: the part's input needs a gain");
    LLMB_REQUIRE(h_dtype == LLMB_DTYPE_F32 || h_dtype == LLMB_DTYPE_BF16, "streams: unknown dtype %d", h_dtype);
    bool vector = width % 4 == 0 && aligned16(X) && aligned16(y) && aligned16(gain) && aligned16(h);
    // columns a turn: a function of the width alone (sums keep one order)
#define LLMB_STREAMS_AS(T, VEC, THREADS, HALVES, STREAMS)                                                                  \
    do {                                                                                                                   \
        if (smem > 40 * 1024)                                                                                              \
            LLMB_CUDA(cudaFuncSetAttribute(streams_kernel<T, VEC, THREADS, HALVES, STREAMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        LLMB_CUDA(llmb::launch(streams_kernel<T, VEC, THREADS, HALVES, STREAMS>, dim3(n_rows), dim3(THREADS), smem, stream, true, X, S, \
                               y, terms, write, read, gain, eps, rows, (T*)h, width));                                     \
    } while (0)
#define LLMB_STREAMS_OF(T, VEC, THREADS, HALVES)                         \
    do {                                                                 \
        if (S == 1) LLMB_STREAMS_AS(T, VEC, THREADS, HALVES, 1);         \
        else if (S == 2) LLMB_STREAMS_AS(T, VEC, THREADS, HALVES, 2);    \
        else if (S == 3) LLMB_STREAMS_AS(T, VEC, THREADS, HALVES, 3);    \
        else LLMB_STREAMS_AS(T, VEC, THREADS, HALVES, 4);                \
    } while (0)
#define LLMB_STREAMS(T)                                                  \
    do {                                                                 \
        if (S > 4) LLMB_STREAMS_AS(T, 1, 256, 1, 0);                     \
        else if (!vector) LLMB_STREAMS_OF(T, 1, 256, 1);                 \
        else if (width < 2048) LLMB_STREAMS_OF(T, 4, 256, 1);            \
        else if (n_rows <= 256) LLMB_STREAMS_OF(T, 4, 512, 1);           \
        else LLMB_STREAMS_OF(T, 4, 256, 2);                              \
    } while (0)
    if (h_dtype == LLMB_DTYPE_F32) LLMB_STREAMS(float);
    else LLMB_STREAMS(__nv_bfloat16);
#undef LLMB_STREAMS
#undef LLMB_STREAMS_OF
#undef LLMB_STREAMS_AS
    return check_launch("streams");
}
LLMB_PACKED(llmb_streams)
