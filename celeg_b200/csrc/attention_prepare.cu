// What stands between an attention mixer's fused [q | k | v] projection (float32 sums) and the paged attention
// kernels, for mixers that need more than a bias: one block a token does, in float32 and in this order,
//
//   1. the biases of q, k and v (optional);
//   2. one RMS norm over the whole q projection and one over the whole k projection, each with a weight as wide as
//      the projection (optional): x / sqrt(mean(x^2) + eps) * w, the mean over all heads' entries together; or the
//      same per head with one weight of a head's size for all heads (`norm_per_head`);
//   3. the rotation of the first `rotary_dim` entries of every q and k head in pairs (i, i + rotary_dim / 2), or of
//      neighbours (2i, 2i + 1) (`interleaved`), by the angle position * frequency_i, cosine and sine times `magnitude`
//      (optional; frequencies come from the host, already scaled as the configuration says);
//   4. a factor on q that grows with the position: 1 + coef * ln(floor((position + 1) / every) + 1) (optional);
//   5. the blend of the values with those an earlier layer made of the same token: v <- (1 - lam) v + lam v_first
//      (`blend` 2), or the note of this layer's values for later layers (`blend` 1: v_first <- v);
//   6. every value head divided by its root mean square, x / sqrt(mean(x^2) + eps), no weight (`unit_values`);
//
// rounds once, and writes q to its buffer and k and v to the token's place in the paged cache. A stored head may be
// wider than the projected one (keys and values brought to one size for kernels that want them alike): the tail is
// zeros, which change no score and no result. Without caches the rows hold queries alone (a layer that reads another
// layer's keys and values).
#include "common.cuh"

namespace celeg_b200 {

struct QkvPrepareArgs {
    const float* proj; int proj_stride;       // rows [q heads | k heads | v heads | ...] as projected, float32
    const float* bias;                        // q, k and v biases one after the other, or null
    const float* q_norm_w; const float* k_norm_w;      // [q width], [k width], or null (both or none)
    float norm_eps;
    int norm_per_head;                        // the norms' weights are [head_dim] and each head has a mean of its own
    int unit_values; float value_eps;
    const float* frequencies; int rotary_dim; // [rotary_dim / 2] or null
    int interleaved; float magnitude;
    float temp_coef; int temp_every;          // every <= 0: no factor
    int blend; float lam; float* first_values; int first_stride;     // [tokens, kv_heads * value_dim] float32
    void* q_out; int q_stride;                // queries in the activation type, head h at h * key_store
    const int* positions; const int* token_span; const int* block_table; int table_stride;
    void* k_cache; void* v_cache; long long page_stride, value_page_stride;
    int q_heads, kv_heads, head_dim, value_dim;    // sizes as projected
    int key_store, value_store;                    // sizes as stored
    int page_tokens;
    int* error_flag;
};

template <typename A>
__global__ void qkv_prepare_kernel(const QkvPrepareArgs p) {
    __shared__ float scratch[33];
    extern __shared__ __align__(16) float row_s[];       // q | k | v as float32, the first values, cos | sin of the angles
    chain_release();
    chain_wait();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int q_width = p.q_heads * p.head_dim, k_width = p.kv_heads * p.head_dim;
    const int qk_width = q_width + k_width;
    // (the token's position and span are asked for first and used last: the row's loads do not wait for them, and
    // the page's number, which hangs on both, is under way while the angles are made)
    const int pos = p.positions[t];
    const int span = p.token_span[t];
    const float* row = p.proj + (size_t)t * p.proj_stride;
    const int v_width = p.kv_heads * p.value_dim;
    const int row_width = qk_width + v_width;
    float* qk = row_s;                                    // q | k | v, biases added
    float* first_s = row_s + ((row_width + 3) & ~3);      // the first values of this token (blend 2)
    float* turn = first_s + (p.blend == 2 ? ((v_width + 3) & ~3) : 0);
    const int half = p.frequencies ? p.rotary_dim >> 1 : 0;
    const float* first_row = p.blend == 2 ? p.first_values + (size_t)t * p.first_stride : nullptr;
    // The row with its biases into shared memory, and the squares of q and of k. Four at a time where the rows allow
    // it, and then every load of a thread is under way before the first is used: a block's time is the time of its
    // chains of dependent loads.
    float q_squares = 0.0f, k_squares = 0.0f;
    const bool by_four = ((row_width | qk_width | q_width | p.proj_stride) & 3) == 0 && ((size_t)p.proj & 15) == 0 &&
                         ((size_t)p.bias & 15) == 0;
    if (by_four) {
        constexpr int kAhead = 4;
        const float4* row4 = reinterpret_cast<const float4*>(row);
        const float4* bias4 = reinterpret_cast<const float4*>(p.bias);
        const int quads = row_width >> 2;
        for (int base = threadIdx.x; base < quads; base += kAhead * blockDim.x) {
            float4 x[kAhead];
#pragma unroll
            for (int u = 0; u < kAhead; ++u) {
                const int i = base + u * blockDim.x;
                x[u] = i < quads ? row4[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
#pragma unroll
            for (int u = 0; u < kAhead; ++u) {
                const int i = base + u * blockDim.x;
                if (i >= quads) continue;
                if (bias4) {
                    const float4 b = __ldg(bias4 + i);
                    x[u].x += b.x; x[u].y += b.y; x[u].z += b.z; x[u].w += b.w;
                }
                reinterpret_cast<float4*>(qk)[i] = x[u];
                const float squares = x[u].x * x[u].x + x[u].y * x[u].y + x[u].z * x[u].z + x[u].w * x[u].w;
                if (4 * i < q_width) q_squares += squares; else if (4 * i < qk_width) k_squares += squares;
            }
        }
    } else {
        for (int i = threadIdx.x; i < row_width; i += blockDim.x) {
            const float x = row[i] + (p.bias ? p.bias[i] : 0.0f);
            qk[i] = x;
            if (i < q_width) q_squares += x * x; else if (i < qk_width) k_squares += x * x;
        }
    }
    if (first_row)
        for (int i = threadIdx.x; i < v_width; i += blockDim.x) first_s[i] = first_row[i];
    const int page = p.kv_heads > 0 ? p.block_table[(size_t)span * p.table_stride + pos / p.page_tokens] : 0;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        sincosf((float)pos * p.frequencies[i], &s, &c);
        turn[i] = c * p.magnitude;
        turn[half + i] = s * p.magnitude;
    }
    float q_factor = 1.0f, k_factor = 1.0f;
    if (p.q_norm_w && !p.norm_per_head) {
        q_factor = 1.0f / sqrtf(block_sum(q_squares, scratch) / (float)q_width + p.norm_eps);
        k_factor = 1.0f / sqrtf(block_sum(k_squares, scratch) / (float)k_width + p.norm_eps);
    }
    __syncthreads();
    const float temperature = p.temp_every > 0
        ? 1.0f + p.temp_coef * logf((float)((pos + 1) / p.temp_every + 1)) : 1.0f;
    A* q_row = static_cast<A*>(p.q_out) + (size_t)t * p.q_stride;
    const long long in_page = pos % p.page_tokens;
    if (page < 0 && threadIdx.x == 0) atomicExch(p.error_flag, 2);
    // a warp a head: norm scale, rotation, the query factor and the store in one pass over shared memory
    for (int unit = warp; unit < p.q_heads + p.kv_heads; unit += warps) {
        const bool is_q = unit < p.q_heads;
        if (!is_q && page < 0) continue;
        const float* head = qk + (size_t)unit * p.head_dim;
        const float* weight = is_q ? p.q_norm_w : p.k_norm_w;
        float factor = is_q ? q_factor : k_factor;
        if (weight && p.norm_per_head) {
            float squares = 0.0f;
            for (int e = lane; e < p.head_dim; e += 32) squares += head[e] * head[e];
            factor = 1.0f / sqrtf(warp_sum(squares) / (float)p.head_dim + p.norm_eps);
        } else if (weight) {
            weight += (size_t)(is_q ? unit : unit - p.q_heads) * p.head_dim;
        }
        const float after = is_q ? temperature : 1.0f;
        A* dst = is_q ? q_row + (size_t)unit * p.key_store
                      : static_cast<A*>(p.k_cache) + (long long)page * p.page_stride +
                            ((long long)(unit - p.q_heads) * p.page_tokens + in_page) * p.key_store;
        for (int i = lane; i < half; i += 32) {
            const int first = p.interleaved ? 2 * i : i, second = p.interleaved ? 2 * i + 1 : i + half;
            float u = head[first] * factor, v = head[second] * factor;
            if (weight) {
                u *= weight[first];
                v *= weight[second];
            }
            dst[first] = from_float<A>((u * turn[i] - v * turn[half + i]) * after);
            dst[second] = from_float<A>((v * turn[i] + u * turn[half + i]) * after);
        }
        for (int e = 2 * half + lane; e < p.head_dim; e += 32)
            dst[e] = from_float<A>(head[e] * factor * (weight ? weight[e] : 1.0f) * after);
        for (int e = p.head_dim + lane; e < p.key_store; e += 32) dst[e] = from_float<A>(0.0f);
    }
    for (int unit = warp; unit < p.kv_heads; unit += warps) {
        A* dst = page < 0 ? nullptr
                          : static_cast<A*>(p.v_cache) + (long long)page * p.value_page_stride +
                                ((long long)unit * p.page_tokens + in_page) * p.value_store;
        auto blended = [&](int column) {
            const float v = qk[qk_width + column];
            return p.blend == 2 ? (1.0f - p.lam) * v + p.lam * first_s[column] : v;
        };
        float unit_factor = 1.0f;
        if (p.unit_values) {
            float squares = 0.0f;
            for (int e = lane; e < p.value_dim; e += 32) {
                const float v = blended(unit * p.value_dim + e);
                squares += v * v;
            }
            unit_factor = 1.0f / sqrtf(warp_sum(squares) / (float)p.value_dim + p.value_eps);
        }
        for (int e = lane; e < p.value_store; e += 32) {
            float v = 0.0f;
            if (e < p.value_dim) {
                const int column = unit * p.value_dim + e;
                v = blended(column);
                if (p.blend == 1) p.first_values[(size_t)t * p.first_stride + column] = v;
                v *= unit_factor;
            }
            if (dst) dst[e] = from_float<A>(v);
        }
    }
}

// The same for rows whose heads need nothing from one another (norms per head or none, pairs of neighbours or no rotation,
// no query factor, no blending, heads stored as wide as they are): a warp a head straight from and to memory, a pair of
// neighbours a lane, angles once a warp, no shared memory and no barrier. E: pairs a lane (heads of up to 64 E entries).
template <typename A> __device__ __forceinline__ void store_pair(A* p, float x, float y);
template <> __device__ __forceinline__ void store_pair<float>(float* p, float x, float y) {
    *reinterpret_cast<float2*>(p) = make_float2(x, y);
}
template <> __device__ __forceinline__ void store_pair<__nv_bfloat16>(__nv_bfloat16* p, float x, float y) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x, y);
}

template <typename A, int E>
__global__ void __launch_bounds__(128) qkv_prepare_heads_kernel(const QkvPrepareArgs p) {
    constexpr int kAhead = 4;                              // heads whose loads are under way together
    chain_release();
    chain_wait();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int pos = p.positions[t];
    const int page = p.kv_heads > 0 ? p.block_table[(size_t)p.token_span[t] * p.table_stride + pos / p.page_tokens] : 0;
    const int in_page = pos % p.page_tokens;
    const int half = p.frequencies ? p.rotary_dim >> 1 : 0;
    const int q_width = p.q_heads * p.head_dim, qk_width = q_width + p.kv_heads * p.head_dim;
    const float* row = p.proj + (size_t)t * p.proj_stride;
    float c[E], s[E];
    const int units = p.q_heads + 2 * p.kv_heads;
    // (few tokens: several blocks share a token's heads)
    const int first = (blockIdx.y * warps + warp), step = gridDim.y * warps;
    for (int base = first; base < units; base += kAhead * step) {
        float2 v[kAhead][E];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int unit = base + a * step;
            const bool value = unit >= p.q_heads + p.kv_heads;
            const int at = value ? qk_width + (unit - p.q_heads - p.kv_heads) * p.value_dim : unit * p.head_dim;
#pragma unroll
            for (int x = 0; x < E; ++x) {
                const int e = 2 * (lane + 32 * x);
                v[a][x] = make_float2(0.0f, 0.0f);
                if (unit < units && e < (value ? p.value_dim : p.head_dim)) {
                    v[a][x] = *reinterpret_cast<const float2*>(row + at + e);
                    if (p.bias) {
                        const float2 b = __ldg(reinterpret_cast<const float2*>(p.bias + at + e));
                        v[a][x].x += b.x;
                        v[a][x].y += b.y;
                    }
                }
            }
        }
        if (base == first) {                               // (the angles, while the first heads are on their way)
#pragma unroll
            for (int x = 0; x < E; ++x) {
                c[x] = 1.0f;
                s[x] = 0.0f;
                const int pair = lane + 32 * x;
                if (pair < half) {
                    sincosf((float)pos * p.frequencies[pair], &s[x], &c[x]);
                    c[x] *= p.magnitude;
                    s[x] *= p.magnitude;
                }
            }
        }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int unit = base + a * step;
            if (unit >= units) continue;                   // (the same for the whole warp)
            const bool is_q = unit < p.q_heads, value = unit >= p.q_heads + p.kv_heads;
            const int size = value ? p.value_dim : p.head_dim;
            const float* weight = value ? nullptr : is_q ? p.q_norm_w : p.k_norm_w;
            float factor = 1.0f;
            if (weight || (value && p.unit_values)) {
                float squares = 0.0f;
#pragma unroll
                for (int x = 0; x < E; ++x) squares += v[a][x].x * v[a][x].x + v[a][x].y * v[a][x].y;
                factor = 1.0f / sqrtf(warp_sum(squares) / (float)size + (value ? p.value_eps : p.norm_eps));
            }
            A* dst;
            if (is_q) {
                dst = static_cast<A*>(p.q_out) + (size_t)t * p.q_stride + (size_t)unit * p.head_dim;
            } else {
                if (page < 0) continue;
                const int head = unit - p.q_heads - (value ? p.kv_heads : 0);
                dst = value ? static_cast<A*>(p.v_cache) + (long long)page * p.value_page_stride
                            : static_cast<A*>(p.k_cache) + (long long)page * p.page_stride;
                dst += ((long long)head * p.page_tokens + in_page) * size;
            }
#pragma unroll
            for (int x = 0; x < E; ++x) {
                const int e = 2 * (lane + 32 * x);
                if (e >= size) continue;
                float u = v[a][x].x * factor, w = v[a][x].y * factor;
                if (weight) {
                    const float2 scale = __ldg(reinterpret_cast<const float2*>(weight + e));
                    u *= scale.x;
                    w *= scale.y;
                }
                if (value || lane + 32 * x >= half) store_pair<A>(dst + e, u, w);
                else store_pair<A>(dst + e, u * c[x] - w * s[x], w * c[x] + u * s[x]);
            }
        }
    }
    if (page < 0 && threadIdx.x == 0) atomicExch(p.error_flag, 2);
}

template <typename A>
static void launch_prepare_heads(const QkvPrepareArgs& args, int tokens, cudaStream_t stream) {
    const int size = args.head_dim > args.value_dim ? args.head_dim : args.value_dim;
    const int units = args.q_heads + 2 * args.kv_heads;
    int share = tokens < 148 ? (148 + tokens - 1) / tokens : 1;      // blocks that share a token, four heads each at least
    if (share > (units + 3) / 4) share = (units + 3) / 4;
    const dim3 grid(tokens, share);
    if (size <= 64) launch_chained(qkv_prepare_heads_kernel<A, 1>, grid, 128, 0, stream, args);
    else launch_chained(qkv_prepare_heads_kernel<A, 2>, grid, 128, 0, stream, args);
}

}  // namespace celeg_b200

using namespace celeg_b200;

CELEG_API int celeg_qkv_prepare(const float* proj, int proj_stride, const float* bias, const float* q_norm_w,
                                const float* k_norm_w, float norm_eps, int norm_per_head, int unit_values, float value_eps,
                                const float* frequencies, int rotary_dim, int interleaved, float magnitude,
                                float temp_coef, int temp_every, int blend, float lam, float* first_values,
                                int first_stride, void* q_out, int q_stride, const int* positions, const int* token_span,
                                const int* block_table, int table_stride, void* k_cache, void* v_cache,
                                long long page_stride, long long value_page_stride, int tokens, int q_heads, int kv_heads,
                                int head_dim, int value_dim, int key_store, int value_store, int page_tokens,
                                int* error_flag, int act_dtype, cudaStream_t stream) {
    // (no caches: the rows hold queries alone, kv_heads is 0)
    CELEG_REQUIRE((kv_heads > 0) == (k_cache != nullptr) && (kv_heads > 0) == (v_cache != nullptr),
                  "qkv_prepare: %d key heads %s caches", kv_heads, k_cache ? "with" : "without");
    CELEG_REQUIRE(tokens >= 0 && q_heads > 0 && kv_heads >= 0 && head_dim > 0 && value_dim > 0 && page_tokens > 0 &&
                  key_store >= head_dim && value_store >= value_dim && q_stride >= q_heads * key_store &&
                  proj_stride >= q_heads * head_dim + kv_heads * (head_dim + value_dim),
                  "qkv_prepare: invalid sizes tokens=%d q_heads=%d kv_heads=%d head_dim=%d value_dim=%d stored %d / %d "
                  "strides %d / %d", tokens, q_heads, kv_heads, head_dim, value_dim, key_store, value_store, proj_stride,
                  q_stride);
    CELEG_REQUIRE(((q_norm_w == nullptr) == (k_norm_w == nullptr) || kv_heads == 0) && (!q_norm_w || norm_eps > 0.0f) &&
                  (!unit_values || value_eps > 0.0f), "qkv_prepare: the norms need both weights and a positive eps");
    CELEG_REQUIRE(!frequencies || (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= head_dim),
                  "qkv_prepare: %d rotated dimensions of a head of %d", rotary_dim, head_dim);
    CELEG_REQUIRE(blend == 0 || ((blend == 1 || blend == 2) && first_values && first_stride >= kv_heads * value_dim),
                  "qkv_prepare: blend %d without a place for the first values (stride %d)", blend, first_stride);
    CELEG_REQUIRE(act_dtype == kFloat32 || act_dtype == kBFloat16, "qkv_prepare: unknown dtype code %d", act_dtype);
    if (tokens == 0) return 0;
    const size_t row_floats = ((size_t)(q_heads + kv_heads) * head_dim + (size_t)kv_heads * value_dim + 3) & ~(size_t)3;
    const size_t first_floats = blend == 2 ? (((size_t)kv_heads * value_dim + 3) & ~(size_t)3) : 0;
    const size_t smem = (row_floats + first_floats + (frequencies ? rotary_dim : 0)) * sizeof(float);
    CELEG_REQUIRE(smem <= 200 * 1024, "qkv_prepare: a row of %zu bytes exceeds a block's shared memory", smem);
    const QkvPrepareArgs args = {proj, proj_stride, bias, q_norm_w, k_norm_w, norm_eps, norm_per_head,
                                 unit_values, value_eps, frequencies, rotary_dim, interleaved, magnitude, temp_coef,
                                 temp_every, blend, lam, first_values, first_stride, q_out, q_stride, positions, token_span, block_table, table_stride, k_cache, v_cache, page_stride,
                                 value_page_stride, q_heads, kv_heads, head_dim, value_dim, key_store, value_store,
                                 page_tokens, error_flag};
    const bool by_heads = (norm_per_head || !q_norm_w) && (interleaved || !frequencies) && temp_every <= 0 && blend == 0 &&
                          key_store == head_dim && value_store == value_dim && head_dim <= 128 && value_dim <= 128 &&
                          ((head_dim | value_dim | proj_stride | q_stride) & 1) == 0 &&
                          (((size_t)proj | (size_t)bias | (size_t)q_norm_w | (size_t)k_norm_w) & 7) == 0 &&
                          (((size_t)q_out | (size_t)k_cache | (size_t)v_cache) & 7) == 0 &&
                          ((page_stride | value_page_stride) & 1) == 0;
    if (by_heads) {
        if (act_dtype == kFloat32) launch_prepare_heads<float>(args, tokens, stream);
        else launch_prepare_heads<__nv_bfloat16>(args, tokens, stream);
        return check_launch("qkv_prepare");
    }
    cudaError_t status = cudaSuccess;
    if (smem > 40 * 1024) {
        status = act_dtype == kFloat32
            ? cudaFuncSetAttribute(qkv_prepare_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
            : cudaFuncSetAttribute(qkv_prepare_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (status != cudaSuccess) {
            set_error("qkv_prepare: %s", cudaGetErrorString(status));
            return -2;
        }
    }
    // A block's time is a chain of dependent loads (position, span, page) and two passes over a short row: more and
    // smaller blocks an SM hide it better than wide ones (2,048 tokens of 16 + 4 heads of 64: 20 us with 256 threads).
    // (few tokens: nothing else hides it, so a block is as wide as its row allows)
    const int threads = tokens <= 148 ? 512 : (q_heads + kv_heads) * head_dim <= 4096 ? 128 : 256;
    if (act_dtype == kFloat32)
        launch_chained(qkv_prepare_kernel<float>, tokens, threads, smem, stream, args);
    else
        launch_chained(qkv_prepare_kernel<__nv_bfloat16>, tokens, threads, smem, stream, args);
    return check_launch("qkv_prepare");
}
