// Row kernels of layers that norm their parts' results only and feed a part the 32-bit stream plus a short causal
// convolution of it:  x += norm(part(x + conv(x))).
//
// layernorm        rows (optionally gathered): (x - mean) / sqrt(mean squared deviation + eps) * gain.
// output_norm_add  s = the sum of a token's result rows (`terms` rows y[t * terms + k] in index order, then, where
//                  `extra` is given, extra[t]); x[t] += norm(s), the norm a layer norm or an RMS norm. In a step of one
//                  token a sequence the same launch can convolve the new x[t] for the part that runs next (below).
// input_conv       h[t, c] = x[t, c] + sum_j taps[j, c] x[t - (K - 1) + j, c] over the tokens of a sequence; rows before
//                  the step's first token come from the sequence's state [K - 1, width] (32-bit, oldest first; zeroed
//                  when a slot is taken), which then holds the last K - 1 rows again.
//
// All arithmetic is 32-bit; only h is rounded (to the run's dtype). Every sum has one order that depends on nothing
// but the row's width (a thread's elements in rising order, lanes as a butterfly, warps in order; a convolution's
// taps from the oldest row on), so a token's values do not depend on the batch or on how a prompt was cut.
#include "common.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_output_norm)

constexpr int MAX_TAPS = 16;
constexpr int NORM_RMS = 0, NORM_LAYER = 1;

template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    v = warp_sum(v);
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __syncthreads();                       // scratch may still be read from the call before
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += scratch[w];
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

// Mean and factor of the row that the block holds in shared memory (every thread its own elements), `total` this thread's
// sum of them. RMS: mean 0.
template <int VEC, int THREADS>
__device__ __forceinline__ void row_statistics(const float* row, int width, int kind, float eps, float total, float* scratch,
                                               float& mean, float& factor) {
    mean = kind == NORM_LAYER ? block_sum<THREADS>(total, scratch) / (float)width : 0.f;
    float sq = 0.f;
    for (int c = threadIdx.x * VEC; c < width; c += THREADS * VEC)
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            float d = row[c + i] - mean;
            sq = fmaf(d, d, sq);
        }
    factor = 1.0f / sqrtf(block_sum<THREADS>(sq, scratch) / (float)width + eps);
}

template <typename TOut, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS)
layernorm_kernel(const float* __restrict__ x, const float* __restrict__ gain, const int* __restrict__ rows,
                 TOut* __restrict__ out, int width, float eps) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[THREADS / 32];
    griddep_launch();
    griddep_wait();
    x = behind_wait(x);
    size_t r = blockIdx.x;
    const float* in = x + (size_t)(rows ? rows[r] : (int)r) * width;
    float total = 0.f, mean, factor;
    for (int c = threadIdx.x * VEC; c < width; c += THREADS * VEC) {
        Pack<VEC> a = load<VEC>(in + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) total += a.v[i];
        store(row + c, a);
    }
    row_statistics<VEC, THREADS>(row, width, NORM_LAYER, eps, total, scratch, mean, factor);
    for (int c = threadIdx.x * VEC; c < width; c += THREADS * VEC) {
        Pack<VEC> g = load<VEC>(gain + c), a;
#pragma unroll
        for (int i = 0; i < VEC; ++i) a.v[i] = (row[c + i] - mean) * factor * g.v[i];
        store(out + r * width + c, a);
    }
}

// `conv`: 0 none, 1 also h[t] = x[t] + conv (one token a sequence: block t is sequence t), with taps [K, width] (K may be
// 0: h = x) and `state` (rows of width, `state_stride` floats a slot) shifted.
template <typename TOut, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS)
output_norm_add_kernel(const float* __restrict__ y, int terms, const float* __restrict__ extra, const float* __restrict__ gain,
                       float eps, int kind, float* __restrict__ x, int width, int conv, const float* __restrict__ taps, int K,
                       float* __restrict__ state, long long state_stride, const int* __restrict__ slot_ids,
                       TOut* __restrict__ h) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[THREADS / 32];
    griddep_launch();
    griddep_wait();
    y = behind_wait(y);
    extra = behind_wait(extra);
    size_t t = blockIdx.x;
    float total = 0.f, mean, factor;
    for (int c = threadIdx.x * VEC; c < width; c += THREADS * VEC) {
        Pack<VEC> s = load<VEC>(y + t * terms * width + c);
        for (int k = 1; k < terms; ++k) {
            Pack<VEC> a = load<VEC>(y + (t * terms + k) * width + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) s.v[i] += a.v[i];
        }
        if (extra) {
            Pack<VEC> a = load<VEC>(extra + t * width + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) s.v[i] += a.v[i];
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) total += s.v[i];
        store(row + c, s);
    }
    row_statistics<VEC, THREADS>(row, width, kind, eps, total, scratch, mean, factor);
    float* st = (conv && K > 1) ? state + (long long)slot_ids[t] * state_stride : nullptr;
    for (int c = threadIdx.x * VEC; c < width; c += THREADS * VEC) {
        Pack<VEC> g = load<VEC>(gain + c), v = load<VEC>(x + t * width + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v.v[i] += (row[c + i] - mean) * factor * g.v[i];
        store(x + t * width + c, v);
        if (!conv) continue;
        Pack<VEC> acc;
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc.v[i] = 0.f;
        for (int j = 0; j + 1 < K; ++j) {                    // the rows before, oldest first; each moves up by one
            Pack<VEC> old = load<VEC>(st + (size_t)j * width + c), w = load<VEC>(taps + (size_t)j * width + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc.v[i] = fmaf(w.v[i], old.v[i], acc.v[i]);
            if (j > 0) store(st + (size_t)(j - 1) * width + c, old);
        }
        if (K > 1) store(st + (size_t)(K - 2) * width + c, v);
        if (K > 0) {
            Pack<VEC> w = load<VEC>(taps + (size_t)(K - 1) * width + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc.v[i] = v.v[i] + fmaf(w.v[i], v.v[i], acc.v[i]);
        } else {
            acc = v;
        }
        store(h + t * width + c, acc);
    }
}

// Tokens [tile * TILE, + TILE) of sequence blockIdx.z, VEC channels a thread. TILE >= MAX_TAPS - 1, so only a sequence's
// first tile reads its state, and the same threads then bring it up to date. TAPS > 0: the number of taps, with the rows
// before the token in registers; 0: any number, rows read again.
constexpr int TILE = 16;
template <typename TOut, int VEC, int TAPS>
__global__ void __launch_bounds__(256)
input_conv_kernel(const float* __restrict__ x, const float* __restrict__ taps, int n_taps, float* __restrict__ state,
                  long long state_stride, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids,
                  TOut* __restrict__ h, int width) {
    griddep_launch();
    griddep_wait();
    x = behind_wait(x);
    const int K = TAPS > 0 ? TAPS : n_taps;
    int b = blockIdx.z, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    int first = cu_seqlens[b], n = cu_seqlens[b + 1] - first;
    int begin = blockIdx.x * TILE, end = min(begin + TILE, n);
    if (c >= width || begin >= end) return;
    float* st = K > 1 ? state + (long long)slot_ids[b] * state_stride : nullptr;
    // the stream's row at place i of the step's tokens (negative: before them)
    auto row_at = [&](int i) { return load<VEC>(i >= 0 ? x + (size_t)(first + i) * width + c : st + (size_t)(K - 1 + i) * width + c); };
    if constexpr (TAPS > 0) {
        Pack<VEC> held[TAPS], w[TAPS];                        // rows i - (K - 1) .. i
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = load<VEC>(taps + (size_t)j * width + c);
#pragma unroll
        for (int j = 1; j < TAPS; ++j) held[j] = row_at(begin - TAPS + j);
        for (int i0 = begin; i0 < end; i0 += 4) {
            Pack<VEC> rows[4];                                // four rows in flight
#pragma unroll
            for (int k = 0; k < 4; ++k) rows[k] = row_at(min(i0 + k, end - 1));
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                if (i0 + k >= end) break;
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) held[j] = held[j + 1];
                held[TAPS - 1] = rows[k];
                Pack<VEC> out;
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    float acc = 0.f;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j].v[e], held[j].v[e], acc);
                    out.v[e] = held[TAPS - 1].v[e] + acc;
                }
                store(h + (size_t)(first + i0 + k) * width + c, out);
            }
        }
    } else {
        for (int i = begin; i < end; ++i) {
            Pack<VEC> acc, now = row_at(i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc.v[e] = 0.f;
            for (int j = 0; j < K; ++j) {
                Pack<VEC> a = row_at(i - (K - 1) + j), w = load<VEC>(taps + (size_t)j * width + c);
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc.v[e] = fmaf(w.v[e], a.v[e], acc.v[e]);
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc.v[e] = now.v[e] + acc.v[e];
            store(h + (size_t)(first + i) * width + c, acc);
        }
    }
    if (begin > 0 || K < 2) return;
    // rows move towards the front: row r of the new state is place n - (K - 1) + r, which lies behind every row
    // written before it
    for (int r = 0; r < K - 1; ++r) store(st + (size_t)r * width + c, row_at(n - (K - 1) + r));
}

template <typename TOut>
__global__ void cast_kernel(const float* __restrict__ x, TOut* __restrict__ h, long long n) {
    griddep_launch();
    griddep_wait();
    x = behind_wait(x);
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) h[i] = from_float<TOut>(x[i]);
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// Threads of a row kernel: a function of the width alone (sums keep one order).
#define LLMB_ROW_KERNEL(KERNEL, T, VECTOR, ...)                                                                        \
    do {                                                                                                               \
        auto go = [&](auto kernel, int threads) -> int {                                                               \
            if (smem > 48 * 1024) LLMB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
            LLMB_CUDA(llmb::launch(kernel, dim3(n_rows), dim3(threads), smem, stream, true, __VA_ARGS__));              \
            return LLMB_OK;                                                                                            \
        };                                                                                                             \
        int code = !(VECTOR) ? go(KERNEL<T, 1, 256>, 256) : width >= 2048 ? go(KERNEL<T, 4, 512>, 512) : go(KERNEL<T, 4, 256>, 256); \
        if (code) return code;                                                                                         \
    } while (0)

LLMB_EXPORT int llmb_layernorm(const float* x, const float* gain, const int* rows, void* out, int out_dtype, int n_rows,
                               int width, float eps, cudaStream_t stream) {
    if (n_rows == 0) return LLMB_OK;
    size_t smem = sizeof(float) * (size_t)width;
    LLMB_REQUIRE(width > 0 && smem <= 200 * 1024, "layernorm: a row of %d values", width);
    bool vector = width % 4 == 0 && aligned16(x) && aligned16(gain) && aligned16(out);
    if (out_dtype == LLMB_DTYPE_F32) LLMB_ROW_KERNEL(layernorm_kernel, float, vector, x, gain, rows, (float*)out, width, eps);
    else if (out_dtype == LLMB_DTYPE_BF16)
        LLMB_ROW_KERNEL(layernorm_kernel, __nv_bfloat16, vector, x, gain, rows, (__nv_bfloat16*)out, width, eps);
    else return fail(LLMB_ERR_ARGUMENT, "layernorm: unknown dtype %d", out_dtype);
    return check_launch("layernorm");
}
LLMB_PACKED(llmb_layernorm)

// y [T * terms, width], extra [T, width] or null, x [T, width], gain [width]: all float32. conv: h [T, width] in h_dtype,
// taps float32 [K, width], state float32 [slots, state_stride] (K - 1 rows each).
LLMB_EXPORT int llmb_output_norm_add(const float* y, int terms, const float* extra, const float* gain, float eps, int kind,
                                     float* x, int n_rows, int width, int conv, const float* taps, int K, float* state,
                                     long long state_stride, const int* slot_ids, void* h, int h_dtype, cudaStream_t stream) {
    if (n_rows == 0) return LLMB_OK;
    size_t smem = sizeof(float) * (size_t)width;
    LLMB_REQUIRE(width > 0 && terms > 0 && smem <= 200 * 1024, "output_norm_add: %d rows of %d values", terms, width);
    LLMB_REQUIRE(kind == NORM_RMS || kind == NORM_LAYER, "output_norm_add: unknown norm %d", kind);
    LLMB_REQUIRE(!conv || (h && K >= 0 && K <= MAX_TAPS && (K == 0 || taps) && (K < 2 || (state && slot_ids && state_stride >= (long long)(K - 1) * width))),
                 "output_norm_add: a convolution of %d taps (up to %d) needs its taps, state and result", K, MAX_TAPS);
    bool vector = width % 4 == 0 && aligned16(y) && aligned16(extra) && aligned16(gain) && aligned16(x) && aligned16(taps) &&
                  aligned16(state) && state_stride % 4 == 0 && aligned16(h);
#define ARGS(T) y, terms, extra, gain, eps, kind, x, width, conv, taps, K, state, state_stride, slot_ids, (T*)h
    if (h_dtype == LLMB_DTYPE_F32) LLMB_ROW_KERNEL(output_norm_add_kernel, float, vector, ARGS(float));
    else if (h_dtype == LLMB_DTYPE_BF16) LLMB_ROW_KERNEL(output_norm_add_kernel, __nv_bfloat16, vector, ARGS(__nv_bfloat16));
    else return fail(LLMB_ERR_ARGUMENT, "output_norm_add: unknown dtype %d", h_dtype);
#undef ARGS
    return check_launch("output_norm_add");
}
LLMB_PACKED(llmb_output_norm_add)

// x float32 [T, width] -> h [T, width] in h_dtype. K == 0: h = x. max_new: the most tokens a sequence brings.
LLMB_EXPORT int llmb_input_conv(const float* x, const float* taps, int K, float* state, long long state_stride,
                                const int* cu_seqlens, const int* slot_ids, void* h, int h_dtype, int n_tokens, int n_seqs,
                                int max_new, int width, cudaStream_t stream) {
    if (n_tokens == 0) return LLMB_OK;
    LLMB_REQUIRE(width > 0 && n_seqs > 0 && n_seqs <= 65535 && max_new > 0, "input_conv: bad sizes");
    LLMB_REQUIRE(K >= 0 && K <= MAX_TAPS, "input_conv: %d taps (up to %d are built)", K, MAX_TAPS);
    LLMB_REQUIRE(h_dtype == LLMB_DTYPE_F32 || h_dtype == LLMB_DTYPE_BF16, "input_conv: unknown dtype %d", h_dtype);
    if (K == 0) {
        long long n = (long long)n_tokens * width;
        dim3 grid((unsigned)((n + 255) / 256));
        if (h_dtype == LLMB_DTYPE_F32) LLMB_CUDA(llmb::launch(cast_kernel<float>, grid, dim3(256), 0, stream, true, x, (float*)h, n));
        else LLMB_CUDA(llmb::launch(cast_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, true, x, (__nv_bfloat16*)h, n));
        return check_launch("input_conv");
    }
    LLMB_REQUIRE(taps && (K < 2 || (state && slot_ids && state_stride >= (long long)(K - 1) * width)),
                 "input_conv: %d taps need their weights and a state", K);
    bool vector = width % 4 == 0 && aligned16(x) && aligned16(taps) && aligned16(state) && state_stride % 4 == 0 && aligned16(h);
    int per = vector ? 4 : 1;
    int threads = ceil_div(width, per) < 256 ? ceil_div(ceil_div(width, per), 32) * 32 : 256;
    dim3 grid(ceil_div(max_new, TILE), ceil_div(width, per * threads), n_seqs);
    LLMB_REQUIRE(grid.y <= 65535, "input_conv: rows of %d values", width);
#define LLMB_CONV_AS(T, VEC, TAPS) \
    LLMB_CUDA(llmb::launch(input_conv_kernel<T, VEC, TAPS>, grid, dim3(threads), 0, stream, true, x, taps, K, state, state_stride, \
                           cu_seqlens, slot_ids, (T*)h, width))
#define LLMB_CONV(T)                                                         \
    do {                                                                     \
        if (!vector) LLMB_CONV_AS(T, 1, 0);                                  \
        else if (K == 2) LLMB_CONV_AS(T, 4, 2);                              \
        else if (K == 3) LLMB_CONV_AS(T, 4, 3);                              \
        else if (K == 4) LLMB_CONV_AS(T, 4, 4);                              \
        else LLMB_CONV_AS(T, 4, 0);                                          \
    } while (0)
    if (h_dtype == LLMB_DTYPE_F32) LLMB_CONV(float);
    else LLMB_CONV(__nv_bfloat16);
#undef LLMB_CONV
#undef LLMB_CONV_AS
    return check_launch("input_conv");
}
LLMB_PACKED(llmb_input_conv)
