// A decoding step of the generalised delta rule (general_delta_scan.cu has the recurrence and the form for prompts): every
// request brings one token, and one block per (request, head) does everything between the input and the output projection:
// the decay's second product, decay and removal rates, the state's update and read-out (sums of the old state; rows of S are
// read and written side by side), the head's root mean square, the norm's weight and the sigmoid gate. Beside it the
// activation of a fused projection's columns on their way into a product of their own.
#include "general_delta.cuh"

namespace celeg_b200 {

struct DeltaDecodeArgs {
    const float* proj; int stride; int r_off, k_off, v_off, gate_off, a_off, low_off;
    const void* decay_up; int rank;               // [heads * dim, rank] in the matrix type
    const float* w0; const float* a_bias; const float* norm_w;
    float* state; long long slot_stride; const int* span_slot;
    int heads, dim;
    float eps, unit_eps;
    void* out;                                    // [tokens, heads * dim], activation type
};

constexpr int kDeltaDecodeThreads = 256;

// kKeep: rows of the state that a thread can hold in registers
template <typename A, int kKeep>
__global__ void __launch_bounds__(kDeltaDecodeThreads) delta_decode_kernel(const DeltaDecodeArgs p) {
    extern __shared__ __align__(16) float smem[];  // tanh [rank] | k r w b [4 dim] | o [dim] | partial sums [2 threads]
    __shared__ float scratch[4][8];
    constexpr int kThreads = kDeltaDecodeThreads, kWarps = kThreads / 32;
    chain_release();
    const int head = blockIdx.x, t = blockIdx.y;
    const int dim = p.dim, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rank_pad = (p.rank + 3) & ~3;
    float* low_s = smem;
    float* k_s = low_s + rank_pad;
    float* r_s = k_s + dim;
    float* w_s = r_s + dim;
    float* b_s = w_s + dim;
    float* o_s = b_s + dim;
    float* part_s = o_s + dim;
    chain_wait();
    const float* row = p.proj + (size_t)t * p.stride;
    float* s_head = p.state + (long long)p.span_slot[t] * p.slot_stride + (size_t)head * dim * dim;
    // The state: a warp takes 32 neighbouring columns and every `split`-th row of them; a thread's rows stay in registers
    // between the sums and the update where they fit, and their loads are under way while the vectors are made.
    const int groups = (dim + 31) >> 5;
    const int split = max(1, kWarps / groups), at_once = kWarps / split;
    const bool kept = dim <= kKeep * split && groups <= at_once;
    const int part = warp % split;
    float cells[kKeep];
    if (kept) {
        const int j = (warp / split) * 32 + lane;
        const bool active = warp / split < groups && j < dim;
#pragma unroll
        for (int i = 0; i < kKeep; ++i) {
            const int e = part + i * split;
            cells[i] = active && e < dim ? s_head[(size_t)e * dim + j] : 0.0f;
        }
    }
    for (int i = threadIdx.x; i < p.rank; i += kThreads) low_s[i] = tanhf(row[p.low_off + i]);
    __syncthreads();
    float kk = 0.0f, rb = 0.0f, rk = 0.0f;
    // four lanes an element: the decay's second product, then the element's decay, removal and shares of the sums
    for (int e0 = 0; e0 < dim; e0 += kThreads / 4) {
        const int e = e0 + (threadIdx.x >> 2), quarter = threadIdx.x & 3;
        float z = 0.0f;
        if (e < dim) {
            const A* up = static_cast<const A*>(p.decay_up) + (size_t)(head * dim + e) * p.rank;
            if (sizeof(A) == 2 && p.rank % 8 == 0 && ((size_t)p.decay_up & 15) == 0) {
                for (int i = 8 * quarter; i < p.rank; i += 32) {
                    const uint4 raw = __ldg(reinterpret_cast<const uint4*>(up + i));
                    const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float2 w = __bfloat1622float2(pairs[j]);
                        z = fmaf(w.x, low_s[i + 2 * j], fmaf(w.y, low_s[i + 2 * j + 1], z));
                    }
                }
            } else {
                for (int i = quarter; i < p.rank; i += 4) z = fmaf(to_float(up[i]), low_s[i], z);
            }
        }
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        z += __shfl_xor_sync(0xffffffffu, z, 2);
        if (e < dim && quarter == 0) {
            const int column = head * dim + e;
            const float k = row[p.k_off + column], r = row[p.r_off + column];
            const float removal = sigmoid_of(row[p.a_off + column] + p.a_bias[column]);
            k_s[e] = k;
            r_s[e] = r;
            w_s[e] = channel_decay(z + p.w0[column]);
            b_s[e] = removal * k;                  // (times 1 / |k| twice below: once for b, once for u)
            kk = fmaf(k, k, kk);
            rb = fmaf(r, removal * k, rb);
            rk = fmaf(r, k, rk);
        }
    }
    kk = warp_sum(kk);
    rb = warp_sum(rb);
    rk = warp_sum(rk);
    if (lane == 0) {
        scratch[0][warp] = kk;
        scratch[1][warp] = rb;
        scratch[2][warp] = rk;
    }
    __syncthreads();
    kk = rb = rk = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
        kk += scratch[0][w];
        rb += scratch[1][w];
        rk += scratch[2][w];
    }
    const float inv = 1.0f / sqrtf(kk + p.unit_eps);
    rb *= inv;
    float squares = 0.0f;
    for (int first = 0; first < groups; first += at_once) {
        const int g = first + warp / split, j = g * 32 + lane;
        const bool active = g < groups && j < dim;
        float su = 0.0f, sq = 0.0f;
        if (kept) {
#pragma unroll
            for (int i = 0; i < kKeep; ++i) {
                const int e = part + i * split;
                if (active && e < dim) {
                    su = fmaf(cells[i], k_s[e], su);
                    sq = fmaf(cells[i], r_s[e] * w_s[e], sq);
                }
            }
        } else if (active) {
            for (int e = part; e < dim; e += split) {
                const float cell = s_head[(size_t)e * dim + j];
                su = fmaf(cell, k_s[e], su);
                sq = fmaf(cell, r_s[e] * w_s[e], sq);
            }
        }
        __syncthreads();                           // (the partial sums of the pass before have been read)
        part_s[threadIdx.x] = su;
        part_s[kThreads + threadIdx.x] = sq;
        __syncthreads();
        if (active) {
            su = sq = 0.0f;
            const int lead = (warp / split) * split;
            for (int w = lead; w < lead + split; ++w) {
                su += part_s[w * 32 + lane];
                sq += part_s[kThreads + w * 32 + lane];
            }
            su *= inv;                             // u^T S of the old state
            const float vj = row[p.v_off + head * dim + j];
            const float take = -su * inv;          // b_s lacks its own 1 / |k|
            if (kept) {
#pragma unroll
                for (int i = 0; i < kKeep; ++i) {
                    const int e = part + i * split;
                    if (e < dim) s_head[(size_t)e * dim + j] = fmaf(k_s[e], vj, fmaf(b_s[e], take, w_s[e] * cells[i]));
                }
            } else {
                for (int e = part; e < dim; e += split) {
                    float* cell = s_head + (size_t)e * dim + j;
                    *cell = fmaf(k_s[e], vj, fmaf(b_s[e], take, w_s[e] * *cell));
                }
            }
            if (part == 0) {
                const float o = sq - su * rb + vj * rk;
                o_s[j] = o;
                squares += o * o;
            }
        }
    }
    squares = warp_sum(squares);
    if (lane == 0) scratch[3][warp] = squares;
    __syncthreads();
    squares = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) squares += scratch[3][w];
    const float scale = 1.0f / sqrtf(squares / (float)dim + p.eps);
    A* dst = static_cast<A*>(p.out) + ((size_t)t * p.heads + head) * dim;
    for (int j = threadIdx.x; j < dim; j += kThreads) {
        const int column = head * dim + j;
        dst[j] = from_float<A>(o_s[j] * scale * p.norm_w[column] * sigmoid_of(row[p.gate_off + column]));
    }
}

// out[t, c] = act(x[t, c]) of float32 columns that lie in wider rows, rounded once (kind -1: no function)
template <typename A>
__global__ void activation_cast_kernel(const float* x, long long stride, A* out, int tokens, int columns, int kind) {
    chain_release();
    chain_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * columns) return;
    const int t = (int)(i / columns), c = (int)(i % columns);
    out[i] = from_float<A>(kind < 0 ? x[(size_t)t * stride + c] : activate(x[(size_t)t * stride + c], kind));
}

}  // namespace celeg_b200

using namespace celeg_b200;

CELEG_API int celeg_activation_cast(const float* x, long long stride, void* out, int tokens, int columns, int kind,
                                    int act_dtype, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && columns > 0 && stride >= columns && kind >= -1 && kind <= kTanh,
                  "activation_cast: invalid sizes tokens=%d columns=%d stride=%lld kind=%d", tokens, columns, stride, kind);
    CELEG_REQUIRE(act_dtype == kFloat32 || act_dtype == kBFloat16, "activation_cast: unknown dtype code %d", act_dtype);
    if (tokens == 0) return 0;
    const unsigned blocks = (unsigned)(((long long)tokens * columns + 255) / 256);
    if (act_dtype == kFloat32)
        launch_chained(activation_cast_kernel<float>, blocks, 256, 0, stream, x, stride, (float*)out, tokens, columns, kind);
    else
        launch_chained(activation_cast_kernel<__nv_bfloat16>, blocks, 256, 0, stream, x, stride, (__nv_bfloat16*)out, tokens,
                       columns, kind);
    return check_launch("activation_cast");
}

// One token a request (row i of proj is request i's): everything between the two projections. low_off: the columns of
// the decay's first product (rank of them), decay_up [heads * dim, rank] in the matrix type (act_dtype).
CELEG_API int celeg_general_delta_decode(const float* proj, int stride, int r_off, int k_off, int v_off, int gate_off, int a_off,
                                         int low_off, const void* decay_up, int rank, const float* w0, const float* a_bias,
                                         const float* norm_w, float eps, float unit_eps, float* state, long long slot_stride,
                                         const int* span_slot, int tokens, int heads, int dim, void* out, int act_dtype,
                                         cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && tokens <= 65535 && heads > 0 && dim > 0 && dim <= kDeltaMaxDim && rank > 0 && rank <= 4096,
                  "general_delta_decode: invalid sizes tokens=%d heads=%d dim=%d (at most %d) rank=%d (at most 4096)", tokens,
                  heads, dim, kDeltaMaxDim, rank);
    CELEG_REQUIRE(eps > 0.0f && unit_eps > 0.0f, "general_delta_decode: eps %g / %g", eps, unit_eps);
    CELEG_REQUIRE(act_dtype == kFloat32 || act_dtype == kBFloat16, "general_delta_decode: unknown dtype code %d", act_dtype);
    if (tokens == 0) return 0;
    const DeltaDecodeArgs args = {proj, stride, r_off, k_off, v_off, gate_off, a_off, low_off, decay_up, rank, w0, a_bias, norm_w,
                                  state, slot_stride, span_slot, heads, dim, eps, unit_eps, out};
    const size_t smem = (size_t)(((rank + 3) & ~3) + 5 * dim + 2 * kDeltaDecodeThreads) * sizeof(float);
    dim3 grid(heads, tokens);
    // (few rows a thread where that holds the head: half the registers, twice the blocks an SM)
    const int groups = (dim + 31) / 32, split = groups < 8 ? 8 / groups : 1;
    const bool few = dim <= 16 * split;
#define CELEG_DELTA_DECODE(A, KEEP) launch_chained(delta_decode_kernel<A, KEEP>, grid, kDeltaDecodeThreads, smem, stream, args)
    if (act_dtype == kFloat32) {
        if (few) CELEG_DELTA_DECODE(float, 16); else CELEG_DELTA_DECODE(float, 32);
    } else {
        if (few) CELEG_DELTA_DECODE(__nv_bfloat16, 16); else CELEG_DELTA_DECODE(__nv_bfloat16, 32);
    }
#undef CELEG_DELTA_DECODE
    return check_launch("general_delta_decode");
}
