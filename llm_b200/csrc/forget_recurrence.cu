// Linear attention whose forget gate also decides what is written (Qin et al., "HGRN2: Gated Linear RNNs with State
// Expansion"): per head a state S [D, V], token by token
//     S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,      o_t = S_t^T q_t
// with q = silu(.), f = l + (1 - l) sigmoid(. + b), l a stored lower bound per head and row; every head's o is
// divided by its root mean square over V and multiplied by a weight that the heads share.
//
// The projection row of a token is [q (H D) | f (H D) | v (H V) | ...] in the run's dtype; everything behind it is 32-bit.
// Per sequence the state is S as [H, V, D] (a column of a head's state, the D rows that one value element reads, is
// contiguous).
//
// Every column of S is a recurrence of its own, with a decay per row; a warp holds several columns of one head, lane l
// the pairs of state rows 2 l, 2 l + 1, then 64 further, .. of each, as packed 32-bit values (one instruction a pair);
// per token it fades, writes and sums S q over its rows (even and odd rows in rising order, the two added, then the lanes
// as a butterfly), so a token's result depends on nothing but the sequence before it, and is the same bits in either form:
//
// steps with more than one token a sequence: prepare (gates into a 32-bit work row [f | q | v] per token), scan (a block
//     holds 32 columns; tokens staged in shared memory a chunk at a time, the next chunk requested under the current; the
//     partial sums of several tokens meet in one butterfly), finish (the heads' norm, rounded to the run's dtype).
// steps of one token a sequence: ONE launch, a block per head and sequence: the head's state is requested before the
//     kernel in front has ended (nothing else in a step touches it), then gates, update, read-out and norm.
#include "row_scan.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_forget_recurrence)

constexpr int THREADS = 256;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float forget(float z, float bias, float low) {
    float s = 1.0f / (1.0f + expf(-(z + bias)));
    return fmaf(1.0f - low, s, low);
}
template <typename T, int VEC>
__global__ void __launch_bounds__(THREADS)
forget_prepare_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ bias, const float* __restrict__ lower,
                      float* __restrict__ work, int work_ld, int keys, int values) {
    griddep_launch();
    griddep_wait();
    proj = behind_wait(proj);
    size_t t = blockIdx.x;
    const T* in = proj + t * ld;
    float* out = work + t * work_ld;
    for (int c = threadIdx.x * VEC; c < 2 * keys + values; c += THREADS * VEC) {
        T raw[VEC];
        float r[VEC];
        if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(raw) = *reinterpret_cast<const uint2*>(in + c);
        else if constexpr (VEC == 4) *reinterpret_cast<float4*>(raw) = *reinterpret_cast<const float4*>(in + c);
        else raw[0] = in[c];
        int to = c < keys ? keys + c : c < 2 * keys ? c - keys : c;          // f in front of q
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            float z = to_float(raw[i]);
            if (c < keys) r[i] = silu(z);
            else if (c < 2 * keys) r[i] = forget(z, bias[c - keys + i], lower[c - keys + i]);
            else r[i] = z;
        }
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(out + to) = make_float4(r[0], r[1], r[2], r[3]);
        else out[to] = r[0];
    }
}

// The factor of a head's norm: a warp sums the squares, its lanes the elements in strides of 32.
__device__ __forceinline__ float head_factor(const float* o, int V, float eps) {
    float sq = 0.f;
    for (int d = threadIdx.x & 31; d < V; d += 32) sq = fmaf(o[d], o[d], sq);
    return 1.0f / sqrtf(warp_sum(sq) / (float)V + eps);
}

// one block per token, a warp a head at a time
template <typename T>
__global__ void __launch_bounds__(THREADS)
forget_finish_kernel(const float* __restrict__ o, const float* __restrict__ weight, float eps, T* __restrict__ mixed,
                     int mixed_ld, int H, int V) {
    griddep_launch();
    griddep_wait();
    o = behind_wait(o);
    size_t t = blockIdx.x;
    for (int head = threadIdx.x >> 5; head < H; head += THREADS / 32) {
        const float* row = o + t * H * V + head * V;
        float factor = head_factor(row, V, eps);
        for (int d = threadIdx.x & 31; d < V; d += 32)
            mixed[t * mixed_ld + head * V + d] = from_float<T>(row[d] * factor * weight[d]);
    }
}

// One token a sequence: block (head, sequence), a warp per 8 columns (V <= 8 * warps).
constexpr int STEP_COLS = 8;
template <typename T, int PER, int MAX_THREADS>
__global__ void __launch_bounds__(MAX_THREADS)
forget_step_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ bias, const float* __restrict__ lower,
                   float* __restrict__ state, long long state_stride, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ slot_ids, const float* __restrict__ weight, float eps, T* __restrict__ mixed,
                   int mixed_ld, int H, int D, int V) {
    extern __shared__ __align__(16) float shared[];      // f (E) | q (E) | v (V) | o (V), E: D rounded up to even
    griddep_launch();
    int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int head = blockIdx.x, seq = blockIdx.y, v0 = warp * STEP_COLS;
    size_t t = cu_seqlens[seq];
    float* S = state + (long long)slot_ids[seq] * state_stride + (size_t)head * D * V;   // [V, D]
    pair_t s[PER][STEP_COLS];
#pragma unroll
    for (int i = 0; i < PER; ++i)
#pragma unroll
        for (int c = 0; c < STEP_COLS; ++c) s[i][c] = v0 + c < V ? load_rows(S + (size_t)(v0 + c) * D, 2 * lane + 64 * i, D) : 0ull;
    griddep_wait();
    proj = behind_wait(proj);
    const T* in = proj + t * ld;
    int keys = H * D, E = (D + 1) & ~1;
    for (int c = threadIdx.x; c < 2 * D + V; c += blockDim.x) {
        if (c < D) shared[c] = forget(to_float(in[keys + head * D + c]), bias[head * D + c], lower[head * D + c]);
        else if (c < 2 * D) shared[E + c - D] = silu(to_float(in[head * D + c - D]));
        else shared[2 * E + c - 2 * D] = to_float(in[2 * keys + head * V + c - 2 * D]);
    }
    __syncthreads();
    float sums[STEP_COLS];
    pair_t v[STEP_COLS], acc[STEP_COLS];
#pragma unroll
    for (int c = 0; c < STEP_COLS; ++c) {
        float value = v0 + c < V ? shared[2 * E + v0 + c] : 0.f;
        v[c] = pack2(value, value);
        acc[c] = 0ull;
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        int n = 2 * lane + 64 * i;
        float2 f = n < D ? *reinterpret_cast<const float2*>(shared + n) : make_float2(1.f, 1.f);
        float2 q = n < D ? *reinterpret_cast<const float2*>(shared + E + n) : make_float2(0.f, 0.f);
        if (n + 1 >= D) { f.y = 1.f; q.y = 0.f; }
        pair_t ff = pack2(f.x, f.y), qq = pack2(q.x, q.y), write = pack2(1.0f - f.x, 1.0f - f.y);
#pragma unroll
        for (int c = 0; c < STEP_COLS; ++c) {
            s[i][c] = update(s[i][c], ff, write, v[c]);
            acc[c] = fma2(s[i][c], qq, acc[c]);
            if (v0 + c < V) store_rows(S + (size_t)(v0 + c) * D, n, D, s[i][c]);
        }
    }
#pragma unroll
    for (int c = 0; c < STEP_COLS; ++c) {
        float even, odd;
        unpack2(acc[c], even, odd);
        sums[c] = even + odd;
    }
    // eight sums over the lanes: the same tree of lane pairs as in the scan
    fold<4, 16>(sums, lane);
    fold<2, 8>(sums, lane);
    fold<1, 4>(sums, lane);
    float total = sums[0];
    total += __shfl_xor_sync(0xffffffffu, total, 2);
    total += __shfl_xor_sync(0xffffffffu, total, 1);
    float* o = shared + 2 * E + V;
    if ((lane & 3) == 0 && v0 + (lane >> 2) < V) o[v0 + (lane >> 2)] = total;
    __syncthreads();
    float factor = head_factor(o, V, eps);
    for (int d = threadIdx.x; d < V; d += blockDim.x)
        mixed[t * mixed_ld + head * V + d] = from_float<T>(o[d] * factor * weight[d]);
}

// Floats of a token's work row: [f | q | v], rounded up to a multiple of four.
LLMB_EXPORT int llmb_forget_recurrence_work_width(int H, int D, int V) { return (2 * H * D + H * V + 3) / 4 * 4; }

// proj [T, ld >= 2 H D + H V] in `dtype`; bias, lower float32 [H D]; state float32 [slots, state_stride >= H D V]; weight
// float32 [V]; work float32 [T, work_ld], o float32 [T, H V] (scratch; not touched where the step is one launch);
// mixed [T, mixed_ld] in `dtype` receives the H V result columns. single: every sequence brings one token.
LLMB_EXPORT int llmb_forget_recurrence(const void* proj, int ld, int dtype, const float* bias, const float* lower,
                                       float* state, long long state_stride, const int* cu_seqlens, const int* slot_ids,
                                       const float* weight, float eps, float* work, int work_ld, float* o, void* mixed,
                                       int mixed_ld, int n_tokens, int n_seqs, int H, int D, int V, int single,
                                       cudaStream_t stream) {
    if (n_tokens == 0) return LLMB_OK;
    LLMB_REQUIRE(H > 0 && D > 0 && V > 0 && D <= 512, "forget_recurrence: %d heads with states of %d x %d (up to 512 rows are built)", H, D, V);
    LLMB_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && H <= 65535, "forget_recurrence: bad sizes");
    LLMB_REQUIRE(ld >= 2 * H * D + H * V && work_ld >= 2 * H * D + H * V && state_stride >= (long long)H * D * V &&
                 (D % 2 || (state_stride % 2 == 0 && ((size_t)state % 8) == 0)),
                 "forget_recurrence: rows too short (or a state of an even number of rows off an 8-byte boundary)");
    LLMB_REQUIRE(dtype == LLMB_DTYPE_F32 || dtype == LLMB_DTYPE_BF16, "forget_recurrence: unknown dtype %d", dtype);
    typedef __nv_bfloat16 B;
    int warps = ceil_div(V, STEP_COLS);
    // (1,024 threads leave 64 registers each: wide states of many rows take the other form)
    if (single && n_tokens == n_seqs && warps <= 32 && D <= 256 && !(D > 128 && warps > 16)) {
        size_t smem = sizeof(float) * (size_t)(2 * D + 2 + 2 * V);
#define LLMB_STEP_AS(T, PER, MOST)                                                                                        \
        LLMB_CUDA(llmb::launch(forget_step_kernel<T, PER, MOST>, dim3(H, n_seqs), dim3(warps * 32), smem, stream, true,         \
                               (const T*)proj, ld, bias, lower, state, state_stride, cu_seqlens, slot_ids, weight, eps,   \
                               (T*)mixed, mixed_ld, H, D, V))
#define LLMB_STEP(T)                                  \
        do {                                          \
            if (D <= 64) LLMB_STEP_AS(T, 1, 1024);    \
            else if (D <= 128 && warps > 16) LLMB_STEP_AS(T, 2, 1024); \
            else if (D <= 128) LLMB_STEP_AS(T, 2, 512); \
            else LLMB_STEP_AS(T, 4, 512);             \
        } while (0)
        if (dtype == LLMB_DTYPE_F32) LLMB_STEP(float); else LLMB_STEP(B);
#undef LLMB_STEP
#undef LLMB_STEP_AS
        return check_launch("forget_recurrence");
    }
    int keys = H * D, values = H * V, esize = dtype == LLMB_DTYPE_F32 ? 4 : 2;
    bool wide_loads = keys % 4 == 0 && values % 4 == 0 && ld % 4 == 0 && work_ld % 4 == 0 && ((size_t)proj % (4 * esize)) == 0 &&
                      ((size_t)work % 16) == 0;
#define LLMB_PREPARE(T, VEC)                                                                                              \
    LLMB_CUDA(llmb::launch(forget_prepare_kernel<T, VEC>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const T*)proj, \
                           ld, bias, lower, work, work_ld, keys, values))
    if (dtype == LLMB_DTYPE_F32) { if (wide_loads) LLMB_PREPARE(float, 4); else LLMB_PREPARE(float, 1); }
    else { if (wide_loads) LLMB_PREPARE(B, 4); else LLMB_PREPARE(B, 1); }
#undef LLMB_PREPARE
    // steps of one token a sequence: 8 columns a warp, 4 warps; steps with more tokens: 2 columns a warp, 16 warps
    bool few = n_tokens <= n_seqs || D > 256;
    int cols = few ? 8 : 2, scan_warps = few ? 4 : 16;
    int tile = scan_warps * cols, chunk = 32 / cols > 8 ? 32 / cols : 8;
    dim3 grid(ceil_div(V, tile), H, n_seqs);
    size_t smem = sizeof(float) * 2 * chunk * ((2 * ((D + 1) & ~1) + tile + 3) / 4 * 4);
    int vectors = D % 4 == 0 && V % 4 == 0 && work_ld % 4 == 0 && ((size_t)work % 16) == 0;
#define LLMB_SCAN_AS(PER, COLS, WARPS)                                                                                    \
    do {                                                                                                                  \
        if (smem > 48 * 1024)                                                                                             \
            LLMB_CUDA(cudaFuncSetAttribute(row_scan_kernel<PER, COLS, WARPS, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           (int)smem));                                                                   \
        LLMB_CUDA(llmb::launch(row_scan_kernel<PER, COLS, WARPS, false>, grid, dim3(WARPS * 32), smem, stream, true,           \
                               (const float*)work, work_ld, state, state_stride, cu_seqlens, slot_ids, (const float*)nullptr, o, H, D, V, vectors)); \
    } while (0)
#define LLMB_SCAN(PER)                                      \
    do {                                                    \
        if (few) LLMB_SCAN_AS(PER, 8, 4);                   \
        else LLMB_SCAN_AS(PER, 2, 16);                      \
    } while (0)
    if (D <= 64) LLMB_SCAN(1);
    else if (D <= 128) LLMB_SCAN(2);
    else if (D <= 256) LLMB_SCAN(4);
    else LLMB_SCAN_AS(8, 8, 4);
#undef LLMB_SCAN
#undef LLMB_SCAN_AS
    if (dtype == LLMB_DTYPE_F32)
        LLMB_CUDA(llmb::launch(forget_finish_kernel<float>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const float*)o,
                               weight, eps, (float*)mixed, mixed_ld, H, V));
    else
        LLMB_CUDA(llmb::launch(forget_finish_kernel<B>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const float*)o, weight,
                               eps, (B*)mixed, mixed_ld, H, V));
    return check_launch("forget_recurrence");
}
LLMB_PACKED(llmb_forget_recurrence)
