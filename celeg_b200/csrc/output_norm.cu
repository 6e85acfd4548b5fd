// The step between two sublayers of a block that norms what a sublayer puts out (not what it reads):
//
//   y = sum_k weight[t, k] rows[place(t, k)] (+ bias)         the sublayer's output: one row, or a weighted sum of rows
//   x = residual[t] + y / sqrt(mean(y^2) + eps) * norm_w;  residual[t] = x
//   out[t] = x in the activation type, what the next sublayer reads (optional)
//
// in one pass over the row: the experts' weighted sum, the output projection's bias, the norm, the residual sum and the
// copy that the next product reads never meet memory in between. Without rows it is the copy alone. When the next reader
// wants an RMS norm of the stream that can be split (gemv_bf16.cu), out[t] = x * next_w and sumsq[t] = sum(x^2) instead.
// Sums, root and products in float32; one rounding into out.
#include "common.cuh"

namespace celeg_b200 {

struct OutputNormArgs {
    float* residual;
    const void* rows; long long row_stride;           // null: nothing is added
    const int* place;                                 // row of pair t * top + k, or null (the pair itself)
    const float* weights; int top;                    // null: one row a token, weight 1
    const float* bias; const float* norm_w; float eps;
    void* out; const float* next_w; float* sumsq; int sumsq_stride;
    int width;
};

template <typename D> __device__ __forceinline__ float4 load_quad(const D* p);
template <> __device__ __forceinline__ float4 load_quad<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load_quad<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
template <typename A> __device__ __forceinline__ void store_quad(A* p, float4 v);
template <> __device__ __forceinline__ void store_quad<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store_quad<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}

// one block a token; a thread's elements stay in registers between the sums and the result
template <typename D, typename A, int kPerThread>
__global__ void output_norm_vec4_kernel(const OutputNormArgs a) {
    __shared__ float scratch[33];
    chain_release();
    chain_wait();
    const int t = blockIdx.x;
    const int quads = a.width >> 2;
    float4* res = reinterpret_cast<float4*>(a.residual + (size_t)t * a.width);
    const D* rows = static_cast<const D*>(a.rows);
    float4 x[kPerThread], y[kPerThread];
#pragma unroll
    for (int u = 0; u < kPerThread; ++u) {
        const int q = threadIdx.x + u * blockDim.x;
        x[u] = q < quads ? res[q] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        y[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    if (rows) {
        if (a.weights) {
            for (int k = 0; k < a.top; ++k) {
                const int pair = t * a.top + k;
                const float w = a.weights[pair];
                const D* row = rows + (long long)(a.place ? a.place[pair] : pair) * a.row_stride;
#pragma unroll
                for (int u = 0; u < kPerThread; ++u) {
                    const int q = threadIdx.x + u * blockDim.x;
                    if (q >= quads) continue;
                    const float4 v = load_quad<D>(row + 4 * q);
                    y[u].x = fmaf(w, v.x, y[u].x); y[u].y = fmaf(w, v.y, y[u].y);
                    y[u].z = fmaf(w, v.z, y[u].z); y[u].w = fmaf(w, v.w, y[u].w);
                }
            }
        } else {
            const D* row = rows + (long long)t * a.row_stride;
#pragma unroll
            for (int u = 0; u < kPerThread; ++u) {
                const int q = threadIdx.x + u * blockDim.x;
                if (q < quads) y[u] = load_quad<D>(row + 4 * q);
            }
        }
        float sum = 0.0f;
#pragma unroll
        for (int u = 0; u < kPerThread; ++u) {
            const int q = threadIdx.x + u * blockDim.x;
            if (q >= quads) continue;
            if (a.bias) {
                const float4 b = __ldg(reinterpret_cast<const float4*>(a.bias) + q);
                y[u].x += b.x; y[u].y += b.y; y[u].z += b.z; y[u].w += b.w;
            }
            sum += y[u].x * y[u].x + y[u].y * y[u].y + y[u].z * y[u].z + y[u].w * y[u].w;
        }
        const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)a.width + a.eps);
#pragma unroll
        for (int u = 0; u < kPerThread; ++u) {
            const int q = threadIdx.x + u * blockDim.x;
            if (q >= quads) continue;
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.norm_w) + q);
            x[u].x += y[u].x * inv * w.x; x[u].y += y[u].y * inv * w.y;
            x[u].z += y[u].z * inv * w.z; x[u].w += y[u].w * inv * w.w;
            res[q] = x[u];
        }
    }
    if (!a.out) return;
    A* dst = static_cast<A*>(a.out) + (size_t)t * a.width;
    float squares = 0.0f;
#pragma unroll
    for (int u = 0; u < kPerThread; ++u) {
        const int q = threadIdx.x + u * blockDim.x;
        if (q >= quads) continue;
        float4 v = x[u];
        if (a.next_w) {
            squares += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.next_w) + q);
            v.x *= w.x; v.y *= w.y; v.z *= w.z; v.w *= w.w;
        }
        store_quad<A>(dst + 4 * q, v);
    }
    if (a.next_w) {
        squares = block_sum(squares, scratch);
        if (threadIdx.x == 0) a.sumsq[(size_t)t * a.sumsq_stride] = squares;
    }
}

// any width and alignment: the sublayer's output is formed twice (the second reads come from the L1 or L2)
template <typename D, typename A>
__global__ void output_norm_kernel(const OutputNormArgs a) {
    __shared__ float scratch[33];
    chain_release();
    chain_wait();
    const int t = blockIdx.x;
    float* res = a.residual + (size_t)t * a.width;
    const D* rows = static_cast<const D*>(a.rows);
    auto output = [&](int c) {
        float y = 0.0f;
        if (a.weights) {
            for (int k = 0; k < a.top; ++k) {
                const int pair = t * a.top + k;
                y = fmaf(a.weights[pair], to_float(rows[(long long)(a.place ? a.place[pair] : pair) * a.row_stride + c]), y);
            }
        } else {
            y = to_float(rows[(long long)t * a.row_stride + c]);
        }
        return a.bias ? y + a.bias[c] : y;
    };
    float inv = 0.0f;
    if (rows) {
        float sum = 0.0f;
        for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
            const float y = output(c);
            sum += y * y;
        }
        inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)a.width + a.eps);
    }
    A* dst = a.out ? static_cast<A*>(a.out) + (size_t)t * a.width : nullptr;
    float squares = 0.0f;
    for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
        float x = res[c];
        if (rows) {
            x += output(c) * inv * a.norm_w[c];
            res[c] = x;
        }
        squares += x * x;
        if (dst) dst[c] = from_float<A>(a.next_w ? x * a.next_w[c] : x);
    }
    if (dst && a.next_w) {
        squares = block_sum(squares, scratch);
        if (threadIdx.x == 0) a.sumsq[(size_t)t * a.sumsq_stride] = squares;
    }
}

template <typename D, typename A>
static void launch_output_norm(const OutputNormArgs& a, int tokens, cudaStream_t stream) {
    constexpr int kPerThread = 4;
    const bool aligned = (((size_t)a.residual | (size_t)a.rows | (size_t)a.bias | (size_t)a.norm_w | (size_t)a.out |
                           (size_t)a.next_w) & 15) == 0;
    if (a.width % 4 == 0 && a.width <= 1024 * 4 * kPerThread && a.row_stride % 4 == 0 && aligned) {
        const int quads = a.width / 4;
        // (few tokens: a block's time is a chain of latencies, one or two quads a thread; many: fewer, fuller threads)
        const int each = tokens <= 64 && quads <= 1024 ? 1 : kPerThread;
        int threads = ((quads + each - 1) / each + 31) / 32 * 32;
        if (threads < 64) threads = 64;
        launch_chained_class(kChainNorm, output_norm_vec4_kernel<D, A, kPerThread>, tokens, threads, 0, stream, a);
    } else {
        launch_chained_class(kChainNorm, output_norm_kernel<D, A>, tokens, a.width >= 512 ? 256 : 128, 0, stream, a);
    }
}

}  // namespace celeg_b200

using namespace celeg_b200;

// rows_dtype: of `rows`; out_dtype: of `out`. weights null: rows[t] itself is the output.
CELEG_API int celeg_output_norm(float* residual, const void* rows, int rows_dtype, long long row_stride, const int* place,
                                const float* weights, int top, const float* bias, const float* norm_w, float eps, void* out,
                                int out_dtype, const float* next_w, float* sumsq, int sumsq_stride, int tokens, int width,
                                cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && width > 0 && (!rows || (norm_w && eps > 0.0f && row_stride >= width)),
                  "output_norm: invalid sizes tokens=%d width=%d stride=%lld eps=%g", tokens, width, row_stride, eps);
    CELEG_REQUIRE(!weights || top > 0, "output_norm: weights for %d rows a token", top);
    CELEG_REQUIRE(rows || out, "output_norm: nothing to add and nowhere to copy");
    CELEG_REQUIRE(!next_w || (out && sumsq && sumsq_stride >= 1), "output_norm: preparing the norm that follows needs its two outputs");
    CELEG_REQUIRE((rows_dtype == kFloat32 || rows_dtype == kBFloat16) && (out_dtype == kFloat32 || out_dtype == kBFloat16),
                  "output_norm: dtype codes %d / %d", rows_dtype, out_dtype);
    if (tokens == 0) return 0;
    const OutputNormArgs args = {residual, rows, rows ? row_stride : 0, place, weights, top, bias, norm_w, eps, out, next_w,
                                 sumsq, sumsq_stride, width};
    if (rows_dtype == kFloat32 && out_dtype == kFloat32) launch_output_norm<float, float>(args, tokens, stream);
    else if (rows_dtype == kFloat32) launch_output_norm<float, __nv_bfloat16>(args, tokens, stream);
    else if (out_dtype == kFloat32) launch_output_norm<__nv_bfloat16, float>(args, tokens, stream);
    else launch_output_norm<__nv_bfloat16, __nv_bfloat16>(args, tokens, stream);
    return check_launch("output_norm");
}
