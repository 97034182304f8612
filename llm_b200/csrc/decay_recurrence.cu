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
// bfloat16 steps of many tokens (sizes in llmb_decay_recurrence): with one decay per head the tokens of a chunk can be taken
//     together, and the work is matrix products (chunk_kernel below): prepare writes bfloat16 rows, the chunks replace the
//     scan, finish. The state stays 32-bit: where it, or anything else of 32 bits, is an operand of a product, it
//     enters as three bfloat16 parts that add up to its 24 bits.
#include "mma.cuh"
#include "row_scan.cuh"

using namespace llmb;

LLMB_DEFINE_LAST_ERROR(llmb_decay_recurrence)

constexpr int THREADS = 256;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

template <typename T, int VEC, typename TWork>
__global__ void __launch_bounds__(THREADS)
decay_prepare_kernel(const T* __restrict__ proj, int ld, TWork* __restrict__ work, int work_ld, int keys, int values) {
    griddep_launch();
    griddep_wait();
    proj = behind_wait(proj);
    size_t t = blockIdx.x;
    const T* in = proj + t * ld;
    TWork* out = work + t * work_ld;
    for (int c = threadIdx.x * VEC; c < 2 * keys + values; c += THREADS * VEC) {
        T raw[VEC];
        float r[VEC];
        if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(raw) = *reinterpret_cast<const uint2*>(in + c);
        else if constexpr (VEC == 4) *reinterpret_cast<float4*>(raw) = *reinterpret_cast<const float4*>(in + c);
        else raw[0] = in[c];
        int to = c < keys ? keys + c : c < 2 * keys ? c - keys : c;          // k in front of q
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            float z = to_float(raw[i]);
            // (what is rounded to bfloat16 next takes the hardware's exponential and quotient)
            r[i] = sizeof(TWork) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : silu(z);
        }
        if constexpr (VEC == 4 && sizeof(TWork) == 2) *reinterpret_cast<uint2*>(out + to) = make_uint2(pack_bf16(r[0], r[1]), pack_bf16(r[2], r[3]));
        else if constexpr (VEC == 4) *reinterpret_cast<float4*>(out + to) = make_float4(r[0], r[1], r[2], r[3]);
        else out[to] = from_float<TWork>(r[0]);
    }
}

// ---------------------------------------------------------------------------------------------- chunks of tokens

// With b = decay, for the token i of a chunk that starts from the state S:
//     o_i = b^(i + 1) S^T q_i + sum_{j <= i} b^(i - j) (q_i . k_j) v_j,      S' = b^n S + sum_j b^(n - 1 - j) k_j v_j^T
// (n tokens in the chunk). A block takes 32 columns of a head's state for one sequence, sixteen warps (mma.sync, 32-bit
// accumulation). The state lives in registers, as the 32-bit accumulators of the second formula: 16 rows and 16 columns a warp.
// q, k and v are bfloat16 as they are; the state, the weights b^(i - j) (q_i . k_j) and the faded values b^(n - 1 - j) v_j are
// split into three bfloat16 parts each in shared memory. Per chunk: first all parts (16 rows and 16 keys of the weights a
// warp), then, behind one barrier, the results (16 rows and 8 columns a warp) and the new state. The chunks' rows come by
// cp.async, the next under the current.
namespace chunk {

constexpr int C = 64, VT = 32, WARPS = 16, LDV = VT + 8, LDW = C + 8;

__device__ __forceinline__ void split3(float x, float& a, float& b, float& c) {
    a = __bfloat162float(__float2bfloat16_rn(x));
    float r = x - a;
    b = __bfloat162float(__float2bfloat16_rn(r));
    c = r - b;                                               // (rounded when it is packed)
}
// two neighbouring values as packed parts
__device__ __forceinline__ void split_pair(float lo, float hi, uint32_t (&part)[3]) {
    float a0, b0, c0, a1, b1, c1;
    split3(lo, a0, b0, c0);
    split3(hi, a1, b1, c1);
    part[0] = pack_bf16(a0, a1);
    part[1] = pack_bf16(b0, b1);
    part[2] = pack_bf16(c0, c1);
}

// bfloat16 elements in front of each part of shared memory
template <int D>
struct Place {
    static constexpr int LDD = D + 8;
    static constexpr int K = 0, Q = K + 2 * C * LDD, V = Q + 2 * C * LDD, S = V + 2 * C * LDV, F = S + 3 * D * LDV, W = F + 3 * C * LDV,
                         END = W + 3 * C * LDW;
    static constexpr size_t bytes = sizeof(__nv_bfloat16) * END + sizeof(float) * (C + 4);
};

template <int D>
__global__ void __launch_bounds__(WARPS * 32, 1)
decay_chunk_kernel(const __nv_bfloat16* __restrict__ work, int work_ld, float* __restrict__ state, long long state_stride,
                   const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids, const float* __restrict__ decays,
                   float* __restrict__ o, int H, int V) {
    typedef __nv_bfloat16 B;
    typedef Place<D> P;
    extern __shared__ __align__(16) unsigned char raw[];
    B* base = reinterpret_cast<B*>(raw);
    auto Ks = reinterpret_cast<B (*)[C][P::LDD]>(base + P::K);       // [2] stages
    auto Qs = reinterpret_cast<B (*)[C][P::LDD]>(base + P::Q);
    auto Vs = reinterpret_cast<B (*)[C][LDV]>(base + P::V);
    auto Sp = reinterpret_cast<B (*)[D][LDV]>(base + P::S);          // [3] parts: the state before the chunk,
    auto Vp = reinterpret_cast<B (*)[C][LDV]>(base + P::F);          // the faded values,
    auto Wp = reinterpret_cast<B (*)[C][LDW]>(base + P::W);          // the weights
    float* power = reinterpret_cast<float*>(base + P::END);          // [C + 1] b^n
    griddep_launch();
    int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    int head = blockIdx.y, seq = blockIdx.z, v0 = blockIdx.x * VT;
    int first = cu_seqlens[seq], n_new = cu_seqlens[seq + 1] - first;
    if (tid == 0) {
        double b = decays[head], p = 1.0;
        for (int n = 0; n <= C; ++n) { power[n] = (float)p; p *= b; }
    }
    float* S = state + (long long)slot_ids[seq] * state_stride + (size_t)head * D * V;   // [V, D]
    // this warp's part of the state: rows d0 + g, + 8; columns c0 + 8 nt + 2 t4, + 1 of the block's
    const int d0 = (warp & 7) * 16, c0 = (warp >> 3) * 16;
    const bool owns = d0 < D;
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int f = 0; f < 4; ++f) {
            int d = d0 + g + (f >> 1) * 8, v = v0 + c0 + nt * 8 + 2 * t4 + (f & 1);
            s[nt][f] = owns && n_new > 0 && v < V ? S[(size_t)v * D + d] : 0.f;
        }
    griddep_wait();
    if (n_new <= 0) return;
    work = behind_wait(work);
    const int keys = H * D;
    const B* k_from = work + (size_t)first * work_ld + head * D;
    const B* v_from = work + (size_t)first * work_ld + 2 * keys + head * V + v0;
    auto request = [&](int chunk) {                          // rows beyond the step's tokens become zeros
        int st = chunk & 1, t0 = chunk * C, count = min(C, n_new - t0);
        const uint4 none = make_uint4(0u, 0u, 0u, 0u);
        for (int i = tid; i < C * (D / 8); i += WARPS * 32) {
            int r = i / (D / 8), c = i % (D / 8) * 8;
            if (r < count) {
                cp_async16(&Ks[st][r][c], k_from + (size_t)(t0 + r) * work_ld + c);
                cp_async16(&Qs[st][r][c], k_from + (size_t)(t0 + r) * work_ld + keys + c);
            } else {
                *reinterpret_cast<uint4*>(&Ks[st][r][c]) = none;
                *reinterpret_cast<uint4*>(&Qs[st][r][c]) = none;
            }
        }
        for (int i = tid; i < C * (VT / 8); i += WARPS * 32) {
            int r = i / (VT / 8), c = i % (VT / 8) * 8;
            if (r < count && v0 + c < V) cp_async16(&Vs[st][r][c], v_from + (size_t)(t0 + r) * work_ld + c);
            else *reinterpret_cast<uint4*>(&Vs[st][r][c]) = none;
        }
        cp_async_commit();
    };
    const int n_chunks = (n_new + C - 1) / C;
    const int mt = warp & 3, nq = warp >> 2;                 // rows 16 mt .. of the results; keys 16 nq .., columns 8 nq ..
    const int row0 = mt * 16 + g, row1 = row0 + 8;
    request(0);
    for (int chunk = 0; chunk < n_chunks; ++chunk) {
        int st = chunk & 1, t0 = chunk * C, count = min(C, n_new - t0);
        cp_async_wait<0>();
        __syncthreads();                                     // the chunk landed; everyone is done with the one before and its parts
        if (chunk + 1 < n_chunks) request(chunk + 1);
        // ---- the parts
        if (owns) {
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int f = 0; f < 2; ++f) {
                    uint32_t part[3];
                    split_pair(s[nt][2 * f], s[nt][2 * f + 1], part);
#pragma unroll
                    for (int p = 0; p < 3; ++p)
                        *reinterpret_cast<uint32_t*>(&Sp[p][d0 + g + f * 8][c0 + nt * 8 + 2 * t4]) = part[p];
                }
        }
        for (int i = tid; i < C * VT / 2; i += WARPS * 32) {
            int r = i / (VT / 2), c = i % (VT / 2) * 2;
            float fade = r < count ? power[count - 1 - r] : 0.f;
            uint32_t part[3];
            split_pair(to_float(Vs[st][r][c]) * fade, to_float(Vs[st][r][c + 1]) * fade, part);
#pragma unroll
            for (int p = 0; p < 3; ++p) *reinterpret_cast<uint32_t*>(&Vp[p][r][c]) = part[p];
        }
        const bool rows_live = mt * 16 < count;
        if (rows_live && nq <= mt) {
            float w[2][4] = {};
#pragma unroll
            for (int k = 0; k < D; k += 16) {
                uint32_t a[4], b[4];
                ldmatrix_x4(a, &Qs[st][mt * 16 + (lane & 15)][k + (lane >> 4) * 8]);
                ldmatrix_x4(b, &Ks[st][nq * 16 + (lane >> 4) * 8 + (lane & 7)][k + ((lane >> 3) & 1) * 8]);
                mma_bf16(w[0], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(w[1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int f = 0; f < 2; ++f) {
                    int r = f ? row1 : row0, j = nq * 16 + n * 8 + 2 * t4, back = r - j;
                    uint32_t part[3];
                    split_pair(back >= 0 ? w[n][2 * f] * power[back] : 0.f, back >= 1 ? w[n][2 * f + 1] * power[back - 1] : 0.f, part);
#pragma unroll
                    for (int p = 0; p < 3; ++p) *reinterpret_cast<uint32_t*>(&Wp[p][r][j]) = part[p];
                }
        }
        __syncthreads();
        // ---- results: what the state gives, faded, and what the chunk's own tokens give
        if (rows_live) {
            float acc[3][4] = {};                            // a sum per part: their products do not wait for one another
#pragma unroll
            for (int k = 0; k < D; k += 32) {
                uint32_t a[2][4];
                ldmatrix_x4(a[0], &Qs[st][mt * 16 + (lane & 15)][k + (lane >> 4) * 8]);
                ldmatrix_x4(a[1], &Qs[st][mt * 16 + (lane & 15)][k + 16 + (lane >> 4) * 8]);
#pragma unroll
                for (int p = 0; p < 3; ++p) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, &Sp[p][k + lane][nq * 8]);
                    mma_bf16(acc[p], a[0][0], a[0][1], a[0][2], a[0][3], b[0], b[1]);
                    mma_bf16(acc[p], a[1][0], a[1][1], a[1][2], a[1][3], b[2], b[3]);
                }
            }
            float fade0 = power[row0 + 1], fade1 = power[row1 + 1];
#pragma unroll
            for (int p = 0; p < 3; ++p) { acc[p][0] *= fade0; acc[p][1] *= fade0; acc[p][2] *= fade1; acc[p][3] *= fade1; }
#pragma unroll
            for (int pair = 0; pair < 2; ++pair) {
                if (2 * pair > mt) break;
                uint32_t b[4];
                ldmatrix_x4_trans(b, &Vs[st][pair * 32 + lane][nq * 8]);
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    if (2 * pair + h > mt) break;
#pragma unroll
                    for (int p = 0; p < 3; ++p) {
                        uint32_t a[4];
                        ldmatrix_x4(a, &Wp[p][mt * 16 + (lane & 15)][pair * 32 + h * 16 + (lane >> 4) * 8]);
                        mma_bf16(acc[p], a[0], a[1], a[2], a[3], b[2 * h], b[2 * h + 1]);
                    }
                }
            }
            int v = v0 + nq * 8 + 2 * t4;
            float* to = o + (size_t)(first + t0) * H * V + head * V + v;
#pragma unroll
            for (int f = 0; f < 4; ++f) acc[0][f] += acc[1][f] + acc[2][f];
            if (v < V) {
                if (row0 < count) *reinterpret_cast<float2*>(to + (size_t)row0 * H * V) = make_float2(acc[0][0], acc[0][1]);
                if (row1 < count) *reinterpret_cast<float2*>(to + (size_t)row1 * H * V) = make_float2(acc[0][2], acc[0][3]);
            }
        }
        // ---- the state after the chunk
        if (owns) {
            float fade = power[count];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int f = 0; f < 4; ++f) s[nt][f] *= fade;
            float low[2][2][4] = {};                         // what the second and third parts add
#pragma unroll
            for (int k = 0; k < C; k += 16) {
                if (k >= count) break;
                uint32_t a[4];                               // rows of k as columns: the operand is K^T
                ldmatrix_x4_trans(a, &Ks[st][k + ((lane >> 4) & 1) * 8 + (lane & 7)][d0 + ((lane >> 3) & 1) * 8]);
#pragma unroll
                for (int p = 0; p < 3; ++p) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, &Vp[p][k + ((lane >> 3) & 1) * 8 + (lane & 7)][c0 + (lane >> 4) * 8]);
                    mma_bf16(p == 0 ? s[0] : low[p - 1][0], a[0], a[1], a[2], a[3], b[0], b[1]);
                    mma_bf16(p == 0 ? s[1] : low[p - 1][1], a[0], a[1], a[2], a[3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int f = 0; f < 4; ++f) s[nt][f] += low[0][nt][f] + low[1][nt][f];
        }
    }
    if (!owns) return;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int f = 0; f < 4; ++f) {
            int d = d0 + g + (f >> 1) * 8, v = v0 + c0 + nt * 8 + 2 * t4 + (f & 1);
            if (v < V) S[(size_t)v * D + d] = s[nt][f];
        }
}

}  // namespace chunk

// One block per token: the factor of the norm over all heads, then weight and gate. VEC: elements a thread takes together (a
// property of the model, so a token's sum has one order in every step).
template <typename T, int VEC>
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
#pragma unroll 4
    for (int d = threadIdx.x * VEC; d < values; d += THREADS * VEC) {
        float x[VEC];
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(row + d);
        else x[0] = row[d];
#pragma unroll
        for (int i = 0; i < VEC; ++i) sq = fmaf(x[i], x[i], sq);
    }
    sq = warp_sum(sq);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = sq;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += scratch[w];
    float factor = 1.0f / sqrtf(total / (float)values + eps);
#pragma unroll 4
    for (int d = threadIdx.x * VEC; d < values; d += THREADS * VEC) {
        float x[VEC], g[VEC], w[VEC];
        if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(row + d);
            *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(weight + d);
            if constexpr (sizeof(T) == 2) {
                T raw[4];
                *reinterpret_cast<uint2*>(raw) = *reinterpret_cast<const uint2*>(gate + t * ld + d);
#pragma unroll
                for (int i = 0; i < 4; ++i) g[i] = to_float(raw[i]);
            } else {
                *reinterpret_cast<float4*>(g) = *reinterpret_cast<const float4*>(gate + t * ld + d);
            }
        } else {
            x[0] = row[d]; w[0] = weight[d]; g[0] = to_float(gate[t * ld + d]);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] = x[i] * factor * w[i] / (1.0f + expf(-g[i]));
        T* to = mixed + t * mixed_ld + d;
        if constexpr (VEC == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(to) = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]));
        else if constexpr (VEC == 4) *reinterpret_cast<float4*>(to) = make_float4(x[0], x[1], x[2], x[3]);
        else to[0] = from_float<T>(x[0]);
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

// Whether a step of these sizes takes the chunked form.
LLMB_EXPORT int llmb_decay_recurrence_chunked(int dtype, int n_tokens, int n_seqs, int D, int V) {
    return dtype == LLMB_DTYPE_BF16 && (D == 32 || D == 64 || D == 96 || D == 128) && V % 8 == 0 && n_tokens >= 16LL * n_seqs;
}

// proj [T, ld >= 2 H D + 2 H V] in `dtype`; decays float32 [H]; state float32 [slots, state_stride >= H D V]; weight
// float32 [H V]; work float32 [T, work_ld >= 2 H D + H V] (scratch; not touched where the step takes its own kernel), o
// float32 [T, H V] (scratch); mixed [T, mixed_ld] in `dtype` receives the H V result columns. single: every sequence
// brings one token. chunks: whether steps that can may take the chunked form.
LLMB_EXPORT int llmb_decay_recurrence(const void* proj, int ld, int dtype, const float* decays, float* state,
                                      long long state_stride, const int* cu_seqlens, const int* slot_ids, const float* weight,
                                      float eps, float* work, int work_ld, float* o, void* mixed, int mixed_ld, int n_tokens,
                                      int n_seqs, int H, int D, int V, int single, int chunks, cudaStream_t stream) {
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
    } else if (chunks && llmb_decay_recurrence_chunked(dtype, n_tokens, n_seqs, D, V) && ld % 4 == 0 && work_ld % 4 == 0 &&
               (((size_t)proj | (size_t)work) % 16) == 0 && ((size_t)o % 8) == 0) {
        LLMB_CUDA(llmb::launch(decay_prepare_kernel<B, 4, B>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const B*)proj, ld,
                               (B*)work, 2 * work_ld, keys, values));
        dim3 grid(ceil_div(V, chunk::VT), H, n_seqs);
#define LLMB_CHUNK(DD)                                                                                                    \
        do {                                                                                                              \
            static bool configured = false;                                                                               \
            if (!configured) {                                                                                            \
                LLMB_CUDA(cudaFuncSetAttribute(chunk::decay_chunk_kernel<DD>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                               (int)chunk::Place<DD>::bytes));                                            \
                configured = true;                                                                                        \
            }                                                                                                             \
            LLMB_CUDA(llmb::launch(chunk::decay_chunk_kernel<DD>, grid, dim3(chunk::WARPS * 32), chunk::Place<DD>::bytes, stream, true, \
                                   (const B*)work, 2 * work_ld, state, state_stride, cu_seqlens, slot_ids, decays, o, H, V)); \
        } while (0)
        if (D == 32) LLMB_CHUNK(32);
        else if (D == 64) LLMB_CHUNK(64);
        else if (D == 96) LLMB_CHUNK(96);
        else LLMB_CHUNK(128);
#undef LLMB_CHUNK
    } else {
        bool wide_loads = keys % 4 == 0 && values % 4 == 0 && ld % 4 == 0 && work_ld % 4 == 0 && ((size_t)proj % (4 * esize)) == 0 &&
                          ((size_t)work % 16) == 0;
#define LLMB_PREPARE(T, VEC)                                                                                              \
        LLMB_CUDA(llmb::launch(decay_prepare_kernel<T, VEC, float>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const T*)proj, \
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
    const char* gate = (const char*)proj + (size_t)(2 * keys + values) * esize;
    bool wide_rows = values % 4 == 0 && ld % 4 == 0 && mixed_ld % 4 == 0 && ((size_t)gate % (4 * esize)) == 0 &&
                     ((size_t)mixed % (4 * esize)) == 0 && (((size_t)o | (size_t)weight) % 16) == 0;
#define LLMB_FINISH(T, VEC)                                                                                               \
    LLMB_CUDA(llmb::launch(decay_finish_kernel<T, VEC>, dim3(n_tokens), dim3(THREADS), 0, stream, true, (const float*)o,  \
                           (const T*)gate, ld, weight, eps, (T*)mixed, mixed_ld, values))
    if (dtype == LLMB_DTYPE_F32) { if (wide_rows) LLMB_FINISH(float, 4); else LLMB_FINISH(float, 1); }
    else { if (wide_rows) LLMB_FINISH(B, 4); else LLMB_FINISH(B, 1); }
#undef LLMB_FINISH
    return check_launch("decay_recurrence");
}
LLMB_PACKED(llmb_decay_recurrence)
