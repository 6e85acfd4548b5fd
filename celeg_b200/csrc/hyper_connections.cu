// Several residual streams in place of one (Zhu et al., "Hyper-Connections", 2024, with stored weights): x_1 .. x_n, all
// equal to the embedding row at the start. A sublayer q reads u = sum_s in_q[s] x_s behind a norm, and its output y goes
// back into all streams at once, x_t <- sum_s mix_q[s, t] x_s + out_q[t] y, from the old ones.
//
// What stands between two sublayers is one pass over a token's streams:
//
//   y   the output of the sublayer before: one row, or the weighted sum of two rows that are each RMS-normed first
//   x   the streams with that output mixed in, written back (not where the caller only reads, as before the head)
//   u   the next sublayer's weighted sum, RMS-normed, in the activation type
//
// so the streams are read and written once a sublayer, and nothing in between meets memory. Before the first sublayer
// there is no output to mix in, and the streams are still one row (`single`): the pass reads it and writes u alone; the
// next one still reads that row as every old stream and writes the streams for the first time. Streams, sums, roots and
// weights are float32; one rounding into u's type. Streams lie as [token][stream][width].
#include "common.cuh"

namespace celeg_b200 {

constexpr int kMaxStreams = 16;

struct HyperArgs {
    const float* single;                              // [tokens, width]: every old stream is this row, or null
    float* streams;                                   // [tokens, count, width]
    int count, write;
    const void* y; long long y_stride;                // null: nothing to mix in
    const float* y2; long long y2_stride;             // a second row (then both are normed), or null
    const float* y_w; const float* y2_w; float y_eps, y_scale;      // y_scale (norm(y) y_w + norm(y2) y2_w)
    const float* mix; const float* give;              // [count, count] from, to; [count]
    const float* take;                                // [count], or null: the plain sum
    const float* norm_w; float eps;                   // null: u as it is
    void* out;
    const int* gather;                                // tokens of the rows, or null (row r is token r)
    int width;
};

template <typename D> __device__ __forceinline__ float4 hyper_load(const D* p);
template <> __device__ __forceinline__ float4 hyper_load<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 hyper_load<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void hyper_store(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void hyper_store(__nv_bfloat16* p, const float4& v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ float4 fma4(float w, const float4& a, const float4& b) {
    return make_float4(fmaf(w, a.x, b.x), fmaf(w, a.y, b.y), fmaf(w, a.z, b.z), fmaf(w, a.w, b.w));
}
__device__ __forceinline__ float dot4(const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// The weights of a pass in shared memory: mix [from][to], give, take
struct HyperWeights { float mix[kMaxStreams * kMaxStreams], give[kMaxStreams], take[kMaxStreams]; };

__device__ __forceinline__ void stage_weights(const HyperArgs& a, HyperWeights& w) {
    if (a.y)
        for (int i = threadIdx.x; i < a.count * a.count; i += blockDim.x) w.mix[i] = a.mix[i];
    for (int i = threadIdx.x; i < a.count; i += blockDim.x) {
        w.give[i] = a.y ? a.give[i] : 0.0f;
        w.take[i] = a.take ? a.take[i] : 1.0f;
    }
}

// one block a row, four neighbours a thread and access; S streams at most (exactly S where S <= 4)
constexpr int hyper_threads(int streams) { return streams <= 4 ? 1024 : streams <= 8 ? 512 : 256; }

template <typename D, typename A, int S, int kPerThread>
__global__ void __launch_bounds__(hyper_threads(S)) hyper_vec4_kernel(const HyperArgs a) {
    __shared__ float scratch[33];
    __shared__ HyperWeights w;
    chain_release();
    stage_weights(a, w);                              // (constant data)
    chain_wait();
    const int n = S <= 4 ? S : a.count;
    const int row = blockIdx.x;
    const int t = a.gather ? a.gather[row] : row;
    const int quads = a.width >> 2;
    float4 y[kPerThread], u[kPerThread];
    if (a.y) {
        const D* src = static_cast<const D*>(a.y) + (long long)t * a.y_stride;
#pragma unroll
        for (int i = 0; i < kPerThread; ++i) {
            const int q = threadIdx.x + i * blockDim.x;
            y[i] = q < quads ? hyper_load<D>(src + 4 * q) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        if (a.y2) {
            const float* src2 = a.y2 + (long long)t * a.y2_stride;
            float first = 0.0f, second = 0.0f;
#pragma unroll
            for (int i = 0; i < kPerThread; ++i) {
                const int q = threadIdx.x + i * blockDim.x;
                u[i] = q < quads ? hyper_load<float>(src2 + 4 * q) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                first += dot4(y[i]);
                second += dot4(u[i]);
            }
            const float f = a.y_scale / sqrtf(block_sum(first, scratch) / (float)a.width + a.y_eps);
            const float s = a.y_scale / sqrtf(block_sum(second, scratch) / (float)a.width + a.y_eps);
#pragma unroll
            for (int i = 0; i < kPerThread; ++i) {
                const int q = threadIdx.x + i * blockDim.x;
                if (q >= quads) continue;
                const float4 fw = __ldg(reinterpret_cast<const float4*>(a.y_w) + q);
                const float4 sw = __ldg(reinterpret_cast<const float4*>(a.y2_w) + q);
                y[i] = make_float4(y[i].x * f * fw.x + u[i].x * s * sw.x, y[i].y * f * fw.y + u[i].y * s * sw.y,
                                   y[i].z * f * fw.z + u[i].z * s * sw.z, y[i].w * f * fw.w + u[i].w * s * sw.w);
            }
        }
    }
    __syncthreads();                                  // the weights are staged
    const float4* old_row = reinterpret_cast<const float4*>(a.single ? a.single + (size_t)t * a.width
                                                                     : a.streams + (size_t)t * n * a.width);
    float4* new_row = reinterpret_cast<float4*>(a.streams + (size_t)t * n * a.width);
    const int old_step = a.single ? 0 : quads;        // (one row: the same for every stream)
    float squares = 0.0f;
#pragma unroll
    for (int i = 0; i < kPerThread; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        u[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (q >= quads) continue;
        float4 x[S];
#pragma unroll
        for (int s = 0; s < S; ++s)
            if (s < n) x[s] = old_row[(size_t)s * old_step + q];
        if (a.y) {
#pragma unroll
            for (int to = 0; to < S; ++to) {
                if (to >= n) continue;
                const float g = w.give[to];
                float4 v = make_float4(g * y[i].x, g * y[i].y, g * y[i].z, g * y[i].w);
#pragma unroll
                for (int s = 0; s < S; ++s)
                    if (s < n) v = fma4(w.mix[s * n + to], x[s], v);
                if (a.write) new_row[(size_t)to * quads + q] = v;
                u[i] = fma4(w.take[to], v, u[i]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s)
                if (s < n) u[i] = fma4(w.take[s], x[s], u[i]);
        }
        squares += dot4(u[i]);
    }
    float inv = 1.0f;
    if (a.norm_w) inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)a.width + a.eps);
    A* dst = static_cast<A*>(a.out) + (size_t)row * a.width;
#pragma unroll
    for (int i = 0; i < kPerThread; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        if (q >= quads) continue;
        float4 v = u[i];
        if (a.norm_w) {
            const float4 nw = __ldg(reinterpret_cast<const float4*>(a.norm_w) + q);
            v = make_float4(v.x * inv * nw.x, v.y * inv * nw.y, v.z * inv * nw.z, v.w * inv * nw.w);
        }
        hyper_store(dst + 4 * q, v);
    }
}

// any width and alignment: the sums wait for the norm in shared memory
template <typename D, typename A>
__global__ void hyper_kernel(const HyperArgs a) {
    extern __shared__ float u_s[];                    // [width]
    __shared__ float scratch[33];
    __shared__ HyperWeights w;
    chain_release();
    stage_weights(a, w);
    chain_wait();
    __syncthreads();
    const int n = a.count, row = blockIdx.x;
    const int t = a.gather ? a.gather[row] : row;
    const D* y = a.y ? static_cast<const D*>(a.y) + (long long)t * a.y_stride : nullptr;
    const float* y2 = a.y2 ? a.y2 + (long long)t * a.y2_stride : nullptr;
    float f = 1.0f, s = 0.0f;
    if (y2) {
        float first = 0.0f, second = 0.0f;
        for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
            first += to_float(y[c]) * to_float(y[c]);
            second += y2[c] * y2[c];
        }
        f = a.y_scale / sqrtf(block_sum(first, scratch) / (float)a.width + a.y_eps);
        s = a.y_scale / sqrtf(block_sum(second, scratch) / (float)a.width + a.y_eps);
    }
    const float* old_row = a.single ? a.single + (size_t)t * a.width : a.streams + (size_t)t * n * a.width;
    float* new_row = a.streams + (size_t)t * n * a.width;
    const int old_step = a.single ? 0 : a.width;
    float squares = 0.0f;
    for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
        float x[kMaxStreams];
        float u = 0.0f;
#pragma unroll
        for (int from = 0; from < kMaxStreams; ++from) x[from] = from < n ? old_row[(size_t)from * old_step + c] : 0.0f;
        const float out = y2 ? to_float(y[c]) * f * a.y_w[c] + y2[c] * s * a.y2_w[c] : y ? to_float(y[c]) : 0.0f;
#pragma unroll
        for (int to = 0; to < kMaxStreams; ++to) {
            if (to >= n) continue;
            float v = x[to];
            if (y) {
                v = w.give[to] * out;
#pragma unroll
                for (int from = 0; from < kMaxStreams; ++from)
                    if (from < n) v = fmaf(w.mix[from * n + to], x[from], v);
                if (a.write) new_row[(size_t)to * a.width + c] = v;
            }
            u = fmaf(w.take[to], v, u);
        }
        u_s[c] = u;
        squares += u * u;
    }
    float inv = 1.0f;
    if (a.norm_w) inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)a.width + a.eps);
    A* dst = static_cast<A*>(a.out) + (size_t)row * a.width;
    for (int c = threadIdx.x; c < a.width; c += blockDim.x)       // (a thread reads what it wrote)
        dst[c] = from_float<A>(a.norm_w ? u_s[c] * inv * a.norm_w[c] : u_s[c]);
}

template <typename D, typename A>
static int launch_hyper(const HyperArgs& a, int rows, cudaStream_t stream) {
    constexpr int kPerThread = 4;
    const bool aligned = (((size_t)a.single | (size_t)a.streams | (size_t)a.y | (size_t)a.y2 | (size_t)a.y_w | (size_t)a.y2_w |
                           (size_t)a.norm_w | (size_t)a.out) & 15) == 0;
    if (a.width % 4 == 0 && a.width <= hyper_threads(a.count) * 4 * kPerThread && a.y_stride % 4 == 0 && a.y2_stride % 4 == 0 && aligned) {
        const int quads = a.width / 4;
        // (few rows: a block's time is a chain of latencies, one quad a thread; many: fuller threads)
        const int each = rows <= 148 && quads <= hyper_threads(a.count) ? 1 : quads <= 512 && quads <= 2 * hyper_threads(a.count) ? 2 : kPerThread;
        int threads = ((quads + each - 1) / each + 31) / 32 * 32;
        if (threads < 64) threads = 64;
#define CELEG_HYPER(S)                                                                                             \
        if (each == 1) launch_chained_class(kChainNorm, hyper_vec4_kernel<D, A, S, 1>, rows, threads, 0, stream, a);       \
        else if (each == 2) launch_chained_class(kChainNorm, hyper_vec4_kernel<D, A, S, 2>, rows, threads, 0, stream, a);  \
        else launch_chained_class(kChainNorm, hyper_vec4_kernel<D, A, S, kPerThread>, rows, threads, 0, stream, a)
        switch (a.count) {
            case 1: CELEG_HYPER(1); break;
            case 2: CELEG_HYPER(2); break;
            case 3: CELEG_HYPER(3); break;
            case 4: CELEG_HYPER(4); break;
            default:
                if (a.count <= 8) { CELEG_HYPER(8); }
                else { CELEG_HYPER(kMaxStreams); }
        }
#undef CELEG_HYPER
        return check_launch("hyper_connect");
    }
    const size_t smem = (size_t)a.width * sizeof(float);
    CELEG_REQUIRE(smem <= 200 * 1024, "hyper_connect: a row of %d entries exceeds a block's shared memory", a.width);
    if (smem > 40 * 1024) {
        const cudaError_t status = cudaFuncSetAttribute(hyper_kernel<D, A>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (status != cudaSuccess) {
            set_error("hyper_connect: %s", cudaGetErrorString(status));
            return -2;
        }
    }
    launch_chained_class(kChainNorm, hyper_kernel<D, A>, rows, a.width >= 512 ? 256 : 128, smem, stream, a);
    return check_launch("hyper_connect");
}

// out[t] = scale (a / rms(a) a_w + b / rms(b) b_w), one block a row
template <typename A>
__global__ void normed_pair_kernel(const float* a, const float* b, const float* a_w, const float* b_w, float eps, float scale,
                                   A* out, int width) {
    __shared__ float scratch[33];
    chain_release();
    chain_wait();
    const size_t at = (size_t)blockIdx.x * width;
    float first = 0.0f, second = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        first += a[at + c] * a[at + c];
        second += b[at + c] * b[at + c];
    }
    const float f = scale / sqrtf(block_sum(first, scratch) / (float)width + eps);
    const float s = scale / sqrtf(block_sum(second, scratch) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x)
        out[at + c] = from_float<A>(a[at + c] * f * a_w[c] + b[at + c] * s * b_w[c]);
}

}  // namespace celeg_b200

using namespace celeg_b200;

// y_dtype: of y (with a second row: float32). rows: how many rows are written; gather: their tokens, or null.
CELEG_API int celeg_hyper_connect(const float* single, float* streams, int count, int write, const void* y, int y_dtype,
                                  long long y_stride, const float* y2, long long y2_stride, const float* y_w,
                                  const float* y2_w, float y_eps, float y_scale, const float* mix, const float* give,
                                  const float* take, const float* norm_w, float eps, void* out, int out_dtype,
                                  const int* gather, int rows, int width, cudaStream_t stream) {
    CELEG_REQUIRE(rows >= 0 && width > 0 && count >= 1 && count <= kMaxStreams,
                  "hyper_connect: invalid sizes rows=%d width=%d streams=%d (at most %d)", rows, width, count, kMaxStreams);
    CELEG_REQUIRE(streams && out && (!y || (mix && give && y_stride >= width)) && (!norm_w || eps > 0.0f),
                  "hyper_connect: streams, an output, and the weights of what is mixed in are needed");
    CELEG_REQUIRE(!y2 || (y && y_dtype == kFloat32 && y_w && y2_w && y_eps > 0.0f && y2_stride >= width),
                  "hyper_connect: a second row needs a float32 first one, both norms' weights and an eps");
    CELEG_REQUIRE(!gather || !write, "hyper_connect: gathered rows leave the streams as they are");
    CELEG_REQUIRE((y_dtype == kFloat32 || y_dtype == kBFloat16) && (out_dtype == kFloat32 || out_dtype == kBFloat16),
                  "hyper_connect: dtype codes %d / %d", y_dtype, out_dtype);
    if (rows == 0) return 0;
    const HyperArgs a = {single, streams, count, write, y, y ? y_stride : 0, y2, y2 ? y2_stride : 0, y_w, y2_w, y_eps, y_scale,
                         mix, give, take, norm_w, eps, out, gather, width};
    if (y_dtype == kFloat32)
        return out_dtype == kFloat32 ? launch_hyper<float, float>(a, rows, stream) : launch_hyper<float, __nv_bfloat16>(a, rows, stream);
    return out_dtype == kFloat32 ? launch_hyper<__nv_bfloat16, float>(a, rows, stream)
                                 : launch_hyper<__nv_bfloat16, __nv_bfloat16>(a, rows, stream);
}

CELEG_API int celeg_normed_pair(const float* a, const float* b, const float* a_w, const float* b_w, float eps, float scale,
                                void* out, int out_dtype, int rows, int width, cudaStream_t stream) {
    CELEG_REQUIRE(rows >= 0 && width > 0 && eps > 0.0f && (out_dtype == kFloat32 || out_dtype == kBFloat16),
                  "normed_pair: invalid sizes rows=%d width=%d eps=%g dtype=%d", rows, width, eps, out_dtype);
    if (rows == 0) return 0;
    const int threads = width >= 512 ? 256 : 128;
    if (out_dtype == kFloat32)
        launch_chained_class(kChainNorm, normed_pair_kernel<float>, rows, threads, 0, stream, a, b, a_w, b_w, eps, scale, (float*)out, width);
    else
        launch_chained_class(kChainNorm, normed_pair_kernel<__nv_bfloat16>, rows, threads, 0, stream, a, b, a_w, b_w, eps, scale,
                             (__nv_bfloat16*)out, width);
    return check_launch("normed_pair");
}
