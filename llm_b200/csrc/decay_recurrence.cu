// Linear attention with one fixed decay per head (Qin et al., "Lightning Attention-2"; Sun et al., "Retentive Network"):
// per head a state S [D, V], token by token
//     S_t = decay S_{t-1} + k_t v_t^T,      o_t = S_t^T q_t
// with q, k and v behind silu; the heads of a token are then divided by their common root mean square, multiplied by a
// weight per element and by sigmoid of a gate.
//
// The projection row of a token is [q (H D) | k (H D) | v (H V) | gate (H V) | ...] in the run's dtype; everything behind
// it is 32-bit. Per sequence the state is S as [H, V, D] (row_scan.cuh: how a warp holds it and in which order it sums).
//
// steps with more than one token a sequence: prepare (silu into a 32-bit work row [k | q | v] per token), scan, finish (norm,
//     weight and gate, rounded to the run's dtype).
// steps of one token a sequence: a block per head and sequence requests the head's state before the kernel in front has
//     ended (nothing else in a step touches it), then silu, update and read-out; finish.
// Both sum in the same order.
#include "row_scan.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_decay_recurrence)

constexpr int THREADS = 256;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

template <typename T, int VEC>
__global__ void __launch_bounds__(THREADS)
decay_prepare_kernel(const T* __restrict__ proj, int ld, float* __restrict__ work, int work_ld, int keys, int values) {
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
        int to = c < keys ? keys + c : c < 2 * keys ? c - keys : c;          // k in front of q
#pragma unroll
        for (int i = 0; i < VEC; ++i) r[i] = silu(to_float(raw[i]));
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(out + to) = make_float4(r[0], r[1], r[2], r[3]);
        else out[to] = r[0];
    }
}

// One block per token: the factor of the norm over all heads, then weight and gate.
template <typename T>
__global__ void __launch_bounds__(THREADS)
decay_finish_kernel(const float* __restrict__ o, const T* __restrict__ gate, int ld, const float* __restrict__ weight, float eps,
                    T* __restrict__ mixed, int mixed_ld, int values) {
    __shared__ float scratch[THREADS / 32];
    griddep_launch();
    griddep_wait();
    o = behind_wait(o);
    gate = behind_wait(gate);
    size_t t = blockIdx.x;
    const float* row = o + t * values;
    float sq = 0.f;
    for (int d = threadIdx.x; d < values; d += THREADS) sq = fmaf(row[d], row[d], sq);
    sq = warp_sum(sq);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = sq;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += scratch[w];
    float factor = 1.0f / sqrtf(total / (float)values + eps);
    for (int d = threadIdx.x; d < values; d += THREADS) {
        float g = to_float(gate[t * ld + d]);
        mixed[t * mixed_ld + d] = from_float<T>(row[d] * factor * weight[d] / (1.0f + expf(-g)));
    }
}

// One token a sequence: block (head, sequence), a warp per 8 columns (V <= 8 * warps).
constexpr int STEP_COLS = 8;
template <typename T, int PER, int MAX_THREADS>
__global__ void __launch_bounds__(MAX_THREADS)
decay_step_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ decays, float* __restrict__ state,
                  long long state_stride, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids,
                  float* __restrict__ o, int H, int D, int V) {
    extern __shared__ __align__(16) float shared[];      // k (E) | q (E) | v (V), E: D rounded up to even
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
    float decay = decays[head];
    griddep_wait();
    proj = behind_wait(proj);
    const T* in = proj + t * ld;
    int keys = H * D, E = (D + 1) & ~1;
    for (int c = threadIdx.x; c < 2 * D + V; c += blockDim.x) {
        if (c < D) shared[c] = silu(to_float(in[keys + head * D + c]));
        else if (c < 2 * D) shared[E + c - D] = silu(to_float(in[head * D + c - D]));
        else shared[2 * E + c - 2 * D] = silu(to_float(in[2 * keys + head * V + c - 2 * D]));
    }
    __syncthreads();
    float sums[STEP_COLS];
    pair_t v[STEP_COLS], acc[STEP_COLS], fade = pack2(decay, decay);
#pragma unroll
    for (int c = 0; c < STEP_COLS; ++c) {
        float value = v0 + c < V ? shared[2 * E + v0 + c] : 0.f;
        v[c] = pack2(value, value);
        acc[c] = 0ull;
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        int n = 2 * lane + 64 * i;
        float2 k = n < D ? *reinterpret_cast<const float2*>(shared + n) : make_float2(0.f, 0.f);
        float2 q = n < D ? *reinterpret_cast<const float2*>(shared + E + n) : make_float2(0.f, 0.f);
        if (n + 1 >= D) { k.y = 0.f; q.y = 0.f; }
        pair_t qq = pack2(q.x, q.y), write = pack2(k.x, k.y);
#pragma unroll
        for (int c = 0; c < STEP_COLS; ++c) {
            s[i][c] = update(s[i][c], fade, write, v[c]);
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
    if ((lane & 3) == 0 && v0 + (lane >> 2) < V) o[t * H * V + head * V + v0 + (lane >> 2)] = total;
}

// proj [T, ld >= 2 H D + 2 H V] in `dtype`; decays float32 [H]; state float32 [slots, state_stride >= H D V]; weight
// float32 [H V]; work float32 [T, work_ld >= 2 H D + H V] (scratch; not touched where the step takes its own kernel), o
// float32 [T, H V] (scratch); mixed [T, mixed_ld] in `dtype` receives the H V result columns. single: every sequence
// brings one token.
LLMB_EXPORT int llmb_decay_recurrence(const void* proj, int ld, int dtype, const float* decays, float* state,
                                      long long state_stride, const int* cu_seqlens, const int* slot_ids, const float* weight,
                                      float eps, float* work, int work_ld, float* o, void* mixed, int mixed_ld, int n_tokens,
                                      int n_seqs, int H, int D, int V, int single, cudaStream_t stream) {
    if (n_tokens == 0) return LLMB_OK;
    LLMB_REQUIRE(H > 0 && D > 0 && V > 0 && D <= 512, "decay_recurrence: %d heads with states of %d x %d (up to 512 rows are built)", H, D, V);
    LLMB_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && H <= 65535, "decay_recurrence: bad sizes");
    LLMB_REQUIRE(ld >= 2 * H * D + 2 * H * V && work_ld >= 2 * H * D + H * V && state_stride >= (long long)H * D * V &&
                 (D % 2 || (state_stride % 2 == 0 && ((size_t)state % 8) == 0)),
                 "decay_recurrence: rows too short (or a state of an even number of rows off an 8-byte boundary)");
    LLMB_REQUIRE(dtype == LLMB_DTYPE_F32 || dtype == LLMB_DTYPE_BF16, "decay_recurrence: unknown dtype %d", dtype);
    typedef __nv_bfloat16 B;
    int keys = H * D, values = H * V, esize = dtype == LLMB_DTYPE_F32 ? 4 : 2;
    int warps = ceil_div(V, STEP_COLS);
    // (1,024 threads leave 64 registers each: wide states of many rows take the other form)
    if (single && n_tokens == n_seqs && warps <= 32 && D <= 256 && !(D > 128 && warps > 16)) {
        size_t smem = sizeof(float) * (size_t)(2 * D + 2 + V);
#define LLMB_STEP_AS(T, PER, MOST)                                                                                        \
        LLMB_CUDA(llmb::launch(decay_step_kernel<T, PER, MOST>, dim3(H, n_seqs), dim3(warps * 32), smem, stream, true,          \
                               (const T*)proj, ld, decays, state, state_stride, cu_seqlens, slot_ids, o, H, D, V))
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
    } else {
        bool wide_loads = keys % 4 == 0 && values % 4 == 0 && ld % 4 == 0 && work_ld % 4 == 0 && ((size_t)proj % (4 * esize)) == 0 &&
                          ((size_t)work % 16) == 0;
#define LLMB_PREPARE(T, VEC)                                                                                              \
        LLMB_CUDA(llmb::launch(decay_prepare_kernel<T, VEC>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const T*)proj, \
                               ld, work, work_ld, keys, values))
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
        do {                                                                                                              \
            if (smem > 48 * 1024)                                                                                         \
                LLMB_CUDA(cudaFuncSetAttribute(row_scan_kernel<PER, COLS, WARPS, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                               (int)smem));                                                               \
            LLMB_CUDA(llmb::launch(row_scan_kernel<PER, COLS, WARPS, true>, grid, dim3(WARPS * 32), smem, stream, true,   \
                                   (const float*)work, work_ld, state, state_stride, cu_seqlens, slot_ids, decays, o, H, D, V, vectors)); \
        } while (0)
#define LLMB_SCAN(PER)                                      \
        do {                                                \
            if (few) LLMB_SCAN_AS(PER, 8, 4);               \
            else LLMB_SCAN_AS(PER, 2, 16);                  \
        } while (0)
        if (D <= 64) LLMB_SCAN(1);
        else if (D <= 128) LLMB_SCAN(2);
        else if (D <= 256) LLMB_SCAN(4);
        else LLMB_SCAN_AS(8, 8, 4);
#undef LLMB_SCAN
#undef LLMB_SCAN_AS
    }
    int gate_at = 2 * keys + values;
    if (dtype == LLMB_DTYPE_F32)
        LLMB_CUDA(llmb::launch(decay_finish_kernel<float>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const float*)o,
                               (const float*)proj + gate_at, ld, weight, eps, (float*)mixed, mixed_ld, values));
    else
        LLMB_CUDA(llmb::launch(decay_finish_kernel<B>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const float*)o,
                               (const B*)proj + gate_at, ld, weight, eps, (B*)mixed, mixed_ld, values));
    return check_launch("decay_recurrence");
}
LLMB_PACKED(llmb_decay_recurrence)
