// Matrix states with a decay that depends on the token: per head, with S [dim, vdim], float32 on both precision paths,
//
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t  (+ d x_t)
//
// in two forms. Channel: a_t has one number a key channel, sigmoid(z)^(1 / tau) (Yang et al., "Gated Linear Attention
// Transformers with Hardware-Efficient Training", 2024). Scalar: one number a token and head, exp(-exp(A_log) dt) with a
// step dt = softplus(. + bias) that also scales what is written, and a direct share d of the values in the read-out (Dao
// and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space Duality",
// 2024); there several heads share queries and keys.
//
// Over prompts every span is cut into chunks of 64 tokens, counted from its first token in the step. With P(i..j) the
// product of the decays of tokens i .. j of a chunk (empty: one), S_0 the state before it and n its last token,
//
//   o_i = sum_(j<=i) [ (q_i P(j+1..i))^T k_j ] v_j + (q_i P(1..i))^T S_0        S_n = P(1..n) S_0 + sum_j (k_j P(j+1..n)) v_j^T
//
// so all chunks are worked on side by side but for one element-wise walk over their states:
//
//   prepare   what the chunk's tokens do to one another, and the vectors q P(1..), k P(..n). Scalar: the running sums of
//             the decays' logarithms, each as two floats (a decay of almost nothing makes a sum large beside the differences
//             that later tokens need); products of decays are exponentials of differences of those. Channel: the 64 tokens
//             are eight blocks of eight, and within a block queries and keys are taken to its middle, q_i P(5..i) or
//             q_i / P(i+1..4), k_j P(j+1..4) or k_j / P(5..j): at most four decays are divided by, and as a decay below
//             1e-8 counts as 1e-8 (the old state's share is then below float32's rounding) that stays within range. The
//             sums are one small product; between two blocks it has one more factor a channel, a product of decays.
//   states    sum_j (k_j P(j+1..n)) v_j^T of every chunk, a 64 x 64 tile a block
//   carry     the states at the chunks' starts, one element a thread, and the span's state after its last token
//   outputs   both terms of o, a tile of 64 tokens x 64 columns a block
//
// Decoding is one launch: a block a (token, head) reads, updates and writes the state once.
#include "common.cuh"

namespace celeg_b200 {

constexpr int kChunk = 64;
constexpr int kPitch = kChunk + 4;           // floats of a row of a tile in shared memory: 16-byte rows, banks spread
constexpr int kDecayMaxDim = 256;            // key size of the channel form

__device__ __forceinline__ float softplus_of(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
__device__ __forceinline__ float root_of_sigmoid(float z, float inv_tau) { return expf(-softplus_of(-z) * inv_tau); }

// chunk c holds the step's tokens chunk_begin[c] .. chunk_begin[c + 1] - 1; span s owns the chunks from span_first[s] on
__global__ void chunk_plan_kernel(const int* span_begin, int spans, int chunk, int max_chunks, int* chunk_begin,
                                  int* span_first) {
    chain_release();
    chain_wait();
    if (threadIdx.x != 0 || blockIdx.x != 0) return;
    int n = 0;
    for (int s = 0; s < spans; ++s) {
        span_first[s] = n;
        for (int b = span_begin[s]; b < span_begin[s + 1] && n < max_chunks; b += chunk) chunk_begin[n++] = b;
    }
    span_first[spans] = n;
    for (int i = n; i <= max_chunks; ++i) chunk_begin[i] = span_begin[spans];      // (chunks beyond the last are empty)
}

// ------------------------------------------------------------------------------------------------- prepare, scalar
__device__ __forceinline__ float2 two_floats(double x) {
    const float high = (float)x;
    return make_float2(high, (float)(x - (double)high));
}

// cum[t, h]: the sum of the decays' logarithms from the chunk's first token through t, a float and what it leaves of the double
// that is summed in; dt[t, h]. A block takes 8 heads of a chunk: a warp a head, two neighbouring tokens a lane, the running
// sum by shuffles.
__global__ void __launch_bounds__(256) scalar_decay_kernel(const float* raw, int stride, const float* bias, const float* a_log,
                                                           const int* chunk_begin, float2* cum, float* dt, int heads) {
    __shared__ float raw_s[kChunk][9], dt_s[kChunk][9];
    __shared__ float2 cum_s[kChunk][9];
    chain_release();
    chain_wait();
    const int h0 = blockIdx.x * 8;
    const int begin = chunk_begin[blockIdx.y], count = chunk_begin[blockIdx.y + 1] - begin;
    if (count <= 0) return;
    for (int i = threadIdx.x; i < kChunk * 8; i += 256) {
        const int t = i >> 3, h = i & 7;
        raw_s[t][h] = t < count && h0 + h < heads ? raw[(size_t)(begin + t) * stride + h0 + h] : 0.0f;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (h0 + warp < heads) {
        const float rate = expf(a_log[h0 + warp]), b = bias[h0 + warp];
        const float first = softplus_of(raw_s[2 * lane][warp] + b), second = softplus_of(raw_s[2 * lane + 1][warp] + b);
        const double x = -rate * first, y = -rate * second;      // (products of floats)
        double sum = x + y;
#pragma unroll
        for (int offset = 1; offset < 32; offset <<= 1) {
            const double below = __shfl_up_sync(0xffffffffu, sum, offset);
            if (lane >= offset) sum += below;
        }
        const double up = __shfl_up_sync(0xffffffffu, sum, 1);
        const double before = lane > 0 ? up : 0.0;
        cum_s[2 * lane][warp] = two_floats(before + x);
        cum_s[2 * lane + 1][warp] = two_floats(before + x + y);
        dt_s[2 * lane][warp] = first;
        dt_s[2 * lane + 1][warp] = second;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < count * 8; i += 256) {
        const int t = i >> 3, h = i & 7;
        if (h0 + h >= heads) continue;
        cum[(size_t)(begin + t) * heads + h0 + h] = cum_s[t][h];
        dt[(size_t)(begin + t) * heads + h0 + h] = dt_s[t][h];
    }
}

// exp of the difference of two such sums
__device__ __forceinline__ float decay_between(const float2& later, const float2& earlier) {
    return expf((later.x - earlier.x) + (later.y - earlier.y));
}

// A tile of 64 x 64 floats into shared memory: rows r < rows of `src` (`stride` apart) times scale(r), columns c < columns;
// zeros beyond. 256 threads, four neighbours a load where `four` says the rows allow it.
template <typename Scale>
__device__ __forceinline__ void load_tile(float (*dst)[kPitch], const float* src, long long stride, int rows, int columns,
                                          bool four, Scale scale) {
    if (four) {
        float4 x[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = (threadIdx.x >> 4) + 16 * u, c = (threadIdx.x & 15) * 4;
            x[u] = r < rows && c < columns ? *reinterpret_cast<const float4*>(src + r * stride + c)
                                           : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = (threadIdx.x >> 4) + 16 * u, c = (threadIdx.x & 15) * 4;
            const float f = scale(r);
            *reinterpret_cast<float4*>(&dst[r][c]) = make_float4(x[u].x * f, x[u].y * f, x[u].z * f, x[u].w * f);
        }
        return;
    }
    for (int i = threadIdx.x; i < kChunk * kChunk; i += 256) {
        const int r = i >> 6, c = i & 63;
        dst[r][c] = r < rows && c < columns ? src[r * stride + c] * scale(r) : 0.0f;
    }
}
struct NoScale { __device__ __forceinline__ float operator()(int) const { return 1.0f; } };
// rows that begin at multiples of four floats (every offset in them is one of `sizes`, a sum of multiples where those are)
__device__ __forceinline__ bool by_fours(const float* p, long long stride, int sizes) {
    return ((((unsigned long long)p >> 2) | (unsigned long long)stride | (unsigned)sizes) & 3) == 0;
}

// products[chunk, group, i, j] = q_i . k_j, 64 x 64 a block
__global__ void __launch_bounds__(256) chunk_products_kernel(const float* q, int q_stride, const float* k, int k_stride,
                                                             const int* chunk_begin, float* products, int groups, int dim) {
    __shared__ __align__(16) float q_s[kChunk][kPitch];
    __shared__ __align__(16) float k_s[kChunk][kPitch];
    chain_release();
    chain_wait();
    const int chunk = blockIdx.y, group = blockIdx.x;
    const int begin = chunk_begin[chunk], count = chunk_begin[chunk + 1] - begin;
    if (count <= 0) return;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int e0 = 0; e0 < dim; e0 += kChunk) {
        if (e0 > 0) __syncthreads();
        load_tile(q_s, q + (size_t)begin * q_stride + (size_t)group * dim + e0, q_stride, count, dim - e0,
                  by_fours(q, q_stride, dim), NoScale());
        load_tile(k_s, k + (size_t)begin * k_stride + (size_t)group * dim + e0, k_stride, count, dim - e0,
                  by_fours(k, k_stride, dim), NoScale());
        __syncthreads();
        const int width = min(kChunk, (dim - e0 + 3) & ~3);
#pragma unroll 1
        for (int e = 0; e < width; e += 4) {
            float4 a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(&q_s[ty * 4 + i][e]);
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = *reinterpret_cast<const float4*>(&k_s[tx + 16 * j][e]);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    acc[i][j] = fmaf(a[i].x, b[j].x, fmaf(a[i].y, b[j].y, fmaf(a[i].z, b[j].z, fmaf(a[i].w, b[j].w, acc[i][j]))));
        }
    }
    float* dst = products + ((size_t)chunk * groups + group) * kChunk * kChunk;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) dst[(ty * 4 + i) * kChunk + tx + 16 * j] = acc[i][j];
}

// ------------------------------------------------------------------------------------------------ prepare, channel
struct ChannelPrepareArgs {
    const float* q; int q_stride; const float* k; int k_stride;        // head h at h * dim
    const float* z; int z_stride; const float* bias; float inv_tau, q_scale;
    const int* chunk_begin;
    float* q_out; float* k_out;              // [tokens, heads * dim]: q_scale q P(1..t), k P(t+1..n)
    float* total;                            // [chunks, heads * dim]: P(1..n)
    float* products;                         // [chunks, heads, 64, 64]: (q_scale q_i P(j+1..i)) . k_j, zero for j > i
    int heads, dim;
};

constexpr float kLeastDecay = 1e-8f;
constexpr int kBlock = 8, kBlocks = kChunk / kBlock;

__host__ __device__ constexpr int channel_prepare_floats(int D) { return 2 * kChunk * (D + 4) + (36 + 4 * kBlocks) * D; }

// D: the key size, padded to a multiple of 32
template <int D>
__global__ void __launch_bounds__(256) channel_prepare_kernel(const ChannelPrepareArgs p) {
    constexpr int kPitchD = D + 4;
    extern __shared__ __align__(16) float smem[];
    chain_release();
    chain_wait();
    const int chunk = blockIdx.y, head = blockIdx.x, tid = threadIdx.x;
    const int begin = p.chunk_begin[chunk], count = p.chunk_begin[chunk + 1] - begin;
    if (count <= 0) return;
    const int dim = p.dim;
    float* q_s = smem;                       // [64][kPitchD]: queries, then at their block's middle
    float* k_s = q_s + kChunk * kPitchD;
    float* w_s = k_s + kChunk * kPitchD;     // [36][D]: the factor between the middles of blocks I >= J at I (I + 1) / 2 + J
    float* upper_s = w_s + 36 * D;           // [8][D]: a block's first four decays, its last four
    float* lower_s = upper_s + kBlocks * D;
    float* q_to = lower_s + kBlocks * D;     // [8][D]: from the middle to the chunk's start, to its end
    float* k_to = q_to + kBlocks * D;
    const size_t width = (size_t)p.heads * dim;
    // a thread a (channel, block of eight tokens)
    for (int x = tid; x < D * kBlocks; x += 256) {
        const int e = x % D, block = x / D, i0 = block * kBlock;
        const bool real = e < dim;
        const size_t column = (size_t)head * dim + e;
        const float bias = real ? p.bias[column] : 0.0f;
        float q[kBlock], k[kBlock], a[kBlock];
#pragma unroll
        for (int i = 0; i < kBlock; ++i) {
            const size_t t = (size_t)(begin + i0 + i);
            const bool here = real && i0 + i < count;
            q[i] = here ? p.q[t * p.q_stride + column] : 0.0f;
            k[i] = here ? p.k[t * p.k_stride + column] : 0.0f;
            a[i] = here ? p.z[t * p.z_stride + column] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < kBlock; ++i)
            a[i] = real && i0 + i < count ? fmaxf(root_of_sigmoid(a[i] + bias, p.inv_tau), kLeastDecay) : 1.0f;
        float f = 1.0f;                      // P(i+1..4), tokens 4 .. 1 of the block
#pragma unroll
        for (int i = kBlock / 2 - 1; i >= 0; --i) {
            q_s[(i0 + i) * kPitchD + e] = q[i] * p.q_scale / f;
            k_s[(i0 + i) * kPitchD + e] = k[i] * f;
            f *= a[i];
        }
        upper_s[block * D + e] = f;
        f = 1.0f;                            // P(5..i)
#pragma unroll
        for (int i = kBlock / 2; i < kBlock; ++i) {
            f *= a[i];
            q_s[(i0 + i) * kPitchD + e] = q[i] * p.q_scale * f;
            k_s[(i0 + i) * kPitchD + e] = k[i] / f;
        }
        lower_s[block * D + e] = f;
    }
    __syncthreads();
    for (int x = tid; x < D * kBlocks; x += 256) {
        const int e = x % D, block = x / D;
        float f = lower_s[block * D + e];    // from the middle of `block` to the end of the blocks so far
        w_s[(block * (block + 1) / 2 + block) * D + e] = 1.0f;
        for (int later = block + 1; later < kBlocks; ++later) {
            w_s[(later * (later + 1) / 2 + block) * D + e] = f * upper_s[later * D + e];
            f *= upper_s[later * D + e] * lower_s[later * D + e];
        }
        k_to[block * D + e] = f;
        float g = upper_s[block * D + e];
        for (int earlier = 0; earlier < block; ++earlier) g *= upper_s[earlier * D + e] * lower_s[earlier * D + e];
        q_to[block * D + e] = g;
        if (block == 0 && e < dim) p.total[(size_t)chunk * width + (size_t)head * dim + e] = f * upper_s[e];
    }
    __syncthreads();
    const int tx = tid & 15, ty = tid >> 4;
    float acc[4][4] = {};
    {
        // tokens ty * 4 + i (block I, the warp's number) against tokens tx + 16 j (blocks 2 j and 2 j + 1, none beyond I)
        const int own = ty >> 1;
        const float* w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) w[j] = w_s + (own * (own + 1) / 2 + min((tx >> 3) + 2 * j, own)) * D;
#pragma unroll 1
        for (int e = 0; e < ((dim + 3) & ~3); e += 4) {
            float4 a[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(q_s + (ty * 4 + i) * kPitchD + e);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (2 * j > own) continue;
                const float4 f = *reinterpret_cast<const float4*>(w[j] + e);
                float4 b = *reinterpret_cast<const float4*>(k_s + (tx + 16 * j) * kPitchD + e);
                b.x *= f.x; b.y *= f.y; b.z *= f.z; b.w *= f.w;
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    acc[i][j] = fmaf(a[i].x, b.x, fmaf(a[i].y, b.y, fmaf(a[i].z, b.z, fmaf(a[i].w, b.w, acc[i][j]))));
            }
        }
    }
    float* dst = p.products + ((size_t)chunk * p.heads + head) * kChunk * kChunk;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            dst[(ty * 4 + i) * kChunk + tx + 16 * j] = tx + 16 * j <= ty * 4 + i ? acc[i][j] : 0.0f;
    for (int x = tid; x < count * D; x += 256) {
        const int r = x / D, e = x % D;
        if (e >= dim) continue;
        const size_t at = (size_t)(begin + r) * width + (size_t)head * dim + e;
        p.q_out[at] = q_s[r * kPitchD + e] * q_to[(r >> 3) * D + e];
        p.k_out[at] = k_s[r * kPitchD + e] * k_to[(r >> 3) * D + e];
    }
}

template <int D>
static int launch_channel_prepare(const ChannelPrepareArgs& args, int chunks, cudaStream_t stream) {
    constexpr size_t smem = (size_t)channel_prepare_floats(D) * sizeof(float);
    if (smem > 40 * 1024) {
        const cudaError_t status = cudaFuncSetAttribute(channel_prepare_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (status != cudaSuccess) {
            set_error("channel_decay_scan: %s", cudaGetErrorString(status));
            return -2;
        }
    }
    launch_chained(channel_prepare_kernel<D>, dim3(args.heads, chunks), 256, smem, stream, args);
    return check_launch("channel_prepare");
}

// --------------------------------------------------------------------------------------------- states, carry, outputs
struct ChunkArgs {
    const float* q; int q_stride; const float* k; int k_stride;        // channel: prepared; scalar: as projected, shared
    const float* v; int v_stride;
    const float2* cum; const float* dt;      // scalar: [tokens, heads]
    const float* total;                      // channel: [chunks, heads * dim]
    const float* products;                   // channel: per head; scalar: per group of heads
    const float* direct;                     // scalar: [heads], the values' share of the read-out, or null
    const int* chunk_begin;
    float* states;                           // [chunks, heads, dim, vdim]
    float* out;                              // [tokens, heads * vdim]
    int heads, groups, dim, vdim;
};

// sum_t k_t v_t^T over a chunk's tokens, k taken to the chunk's end
template <bool CHANNEL>
__global__ void __launch_bounds__(256) chunk_states_kernel(const ChunkArgs p) {
    __shared__ __align__(16) float k_s[kChunk][kPitch];
    __shared__ __align__(16) float v_s[kChunk][kPitch];
    __shared__ float w_s[kChunk];
    chain_release();
    chain_wait();
    const int chunk = blockIdx.z, head = blockIdx.y;
    const int begin = p.chunk_begin[chunk], count = p.chunk_begin[chunk + 1] - begin;
    if (count <= 0) return;
    const int v_tiles = (p.vdim + kChunk - 1) / kChunk;
    const int e0 = (blockIdx.x / v_tiles) * kChunk, c0 = (blockIdx.x % v_tiles) * kChunk;
    const int k_at = (CHANNEL ? head : head / (p.heads / p.groups)) * p.dim + e0;
    if (!CHANNEL) {
        if (threadIdx.x < count) {
            const size_t t = (size_t)(begin + threadIdx.x) * p.heads + head;
            w_s[threadIdx.x] = p.dt[t] * decay_between(p.cum[(size_t)(begin + count - 1) * p.heads + head], p.cum[t]);
        }
        __syncthreads();
    }
    const float* k_src = p.k + (size_t)begin * p.k_stride + k_at;
    if (CHANNEL) load_tile(k_s, k_src, p.k_stride, count, p.dim - e0, by_fours(p.k, p.k_stride, p.dim), NoScale());
    else load_tile(k_s, k_src, p.k_stride, count, p.dim - e0, by_fours(p.k, p.k_stride, p.dim),
                   [&](int r) { return r < count ? w_s[r] : 0.0f; });
    load_tile(v_s, p.v + (size_t)begin * p.v_stride + (size_t)head * p.vdim + c0, p.v_stride, count, p.vdim - c0,
              by_fours(p.v, p.v_stride, p.vdim), NoScale());
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
#pragma unroll 8
    for (int t = 0; t < count; ++t) {
        const float4 a = *reinterpret_cast<const float4*>(&k_s[t][ty * 4]);
        const float4 b = *reinterpret_cast<const float4*>(&v_s[t][tx * 4]);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    float* dst = p.states + ((size_t)chunk * p.heads + head) * p.dim * p.vdim;
    const bool four = (p.vdim & 3) == 0;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int e = e0 + ty * 4 + i;
        if (e >= p.dim) continue;
        if (four) {
            if (c0 + tx * 4 < p.vdim)
                *reinterpret_cast<float4*>(dst + (size_t)e * p.vdim + c0 + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            continue;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = c0 + tx * 4 + j;
            if (c < p.vdim) dst[(size_t)e * p.vdim + c] = acc[i][j];
        }
    }
}

// a thread V neighbouring elements of the state: a chunk's own sum is replaced by the state before the chunk
template <bool CHANNEL, int V>
__global__ void __launch_bounds__(128) chunk_carry_kernel(const ChunkArgs p, float* state, long long slot_stride,
                                                          const int* span_slot, const int* span_first) {
    chain_release();
    chain_wait();
    const int elements = p.heads * p.dim * p.vdim;
    const int e = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (e >= elements) return;
    const int span = blockIdx.y;
    const int first = span_first[span], last = span_first[span + 1];
    if (first == last) return;
    const int row = e / p.vdim, head = row / p.dim;                    // row: head * dim + key channel (V divides vdim)
    float* cell = state + (long long)span_slot[span] * slot_stride + e;
    float s[V];
#pragma unroll
    for (int i = 0; i < V; ++i) s[i] = cell[i];
    constexpr int kAhead = 8;
    for (int c0 = first; c0 < last; c0 += kAhead) {
        float own[kAhead][V], keep[kAhead];
        int ends[kAhead];
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int c = c0 + i;
            if (c >= last) continue;
            ends[i] = CHANNEL ? 0 : p.chunk_begin[c + 1] - 1;
            const float* src = p.states + (size_t)c * elements + e;
            if (V == 4) {
                const float4 x = *reinterpret_cast<const float4*>(src);
                own[i][0] = x.x; own[i][1 % V] = x.y; own[i][2 % V] = x.z; own[i][3 % V] = x.w;
            } else {
                own[i][0] = *src;
            }
            if (CHANNEL) keep[i] = p.total[(size_t)c * p.heads * p.dim + row];
        }
        if (!CHANNEL) {
#pragma unroll
            for (int i = 0; i < kAhead; ++i)
                if (c0 + i < last) keep[i] = p.cum[(size_t)ends[i] * p.heads + head].x;
        }
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int c = c0 + i;
            if (c >= last) continue;
            float* dst = p.states + (size_t)c * elements + e;
            if (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(s[0], s[1 % V], s[2 % V], s[3 % V]);
            else *dst = s[0];
            const float f = CHANNEL ? keep[i] : expf(keep[i]);
#pragma unroll
            for (int j = 0; j < V; ++j) s[j] = fmaf(f, s[j], own[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) cell[i] = s[i];
}

__device__ __forceinline__ void tile_product(const float (*a_s)[kPitch], const float (*b_s)[kPitch], int depth, int tx, int ty,
                                             float (&acc)[4][4]) {
#pragma unroll 1
    for (int k = 0; k < depth; k += 4) {
        float4 a[4], b[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const float4*>(&a_s[ty * 4 + i][k]);
#pragma unroll
        for (int u = 0; u < 4; ++u) b[u] = *reinterpret_cast<const float4*>(&b_s[k + u][tx * 4]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float av[4] = {a[i].x, a[i].y, a[i].z, a[i].w};
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                acc[i][0] = fmaf(av[u], b[u].x, acc[i][0]);
                acc[i][1] = fmaf(av[u], b[u].y, acc[i][1]);
                acc[i][2] = fmaf(av[u], b[u].z, acc[i][2]);
                acc[i][3] = fmaf(av[u], b[u].w, acc[i][3]);
            }
        }
    }
}

template <bool CHANNEL>
__global__ void __launch_bounds__(256, 4) chunk_outputs_kernel(const ChunkArgs p) {
    __shared__ __align__(16) float a_s[kChunk][kPitch];
    __shared__ __align__(16) float b_s[kChunk][kPitch];
    __shared__ float2 cum_s[kChunk];
    __shared__ float dt_s[kChunk];
    chain_release();
    chain_wait();
    const int chunk = blockIdx.z, head = blockIdx.y, c0 = blockIdx.x * kChunk;
    const int begin = p.chunk_begin[chunk], count = p.chunk_begin[chunk + 1] - begin;
    if (count <= 0) return;
    const int group = CHANNEL ? head : head / (p.heads / p.groups);
    if (!CHANNEL) {
        if (threadIdx.x < kChunk) {
            const size_t t = (size_t)(begin + threadIdx.x) * p.heads + head;
            cum_s[threadIdx.x] = threadIdx.x < count ? p.cum[t] : make_float2(0.0f, 0.0f);
            dt_s[threadIdx.x] = threadIdx.x < count ? p.dt[t] : 0.0f;
        }
        __syncthreads();
    }
    // the chunk's own tokens
    const float* m = p.products + ((size_t)chunk * (CHANNEL ? p.heads : p.groups) + group) * kChunk * kChunk;
    load_tile(b_s, p.v + (size_t)begin * p.v_stride + (size_t)head * p.vdim + c0, p.v_stride, count, p.vdim - c0,
              by_fours(p.v, p.v_stride, p.vdim), NoScale());
    {
        float4 x[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) x[u] = reinterpret_cast<const float4*>(m)[threadIdx.x + 256 * u];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = (threadIdx.x >> 4) + 16 * u, c = (threadIdx.x & 15) * 4;
            float v[4] = {x[u].x, x[u].y, x[u].z, x[u].w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const bool seen = c + i <= r && r < count;
                if (CHANNEL) v[i] = seen ? v[i] : 0.0f;
                else v[i] = seen ? v[i] * decay_between(cum_s[r], cum_s[c + i]) * dt_s[c + i] : 0.0f;
            }
            *reinterpret_cast<float4*>(&a_s[r][c]) = make_float4(v[0], v[1], v[2], v[3]);
        }
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    tile_product(a_s, b_s, min(kChunk, ty * 4 + 4), tx, ty, acc);      // (zeros beyond the diagonal)
    if (!CHANNEL && p.direct) {
        const float d = p.direct[head];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(d, b_s[ty * 4 + i][tx * 4 + j], acc[i][j]);
    }
    // the state before the chunk
    const float* state = p.states + ((size_t)chunk * p.heads + head) * p.dim * p.vdim;
    for (int e0 = 0; e0 < p.dim; e0 += kChunk) {
        __syncthreads();
        const float* q_src = p.q + (size_t)begin * p.q_stride + (size_t)group * p.dim + e0;
        if (CHANNEL) load_tile(a_s, q_src, p.q_stride, count, p.dim - e0, by_fours(p.q, p.q_stride, p.dim), NoScale());
        else load_tile(a_s, q_src, p.q_stride, count, p.dim - e0, by_fours(p.q, p.q_stride, p.dim),
                       [&](int r) { return expf(cum_s[r].x); });
        load_tile(b_s, state + (size_t)e0 * p.vdim + c0, p.vdim, p.dim - e0, p.vdim - c0, by_fours(p.states, p.vdim, p.dim * p.vdim),
                  NoScale());
        __syncthreads();
        tile_product(a_s, b_s, min(kChunk, (p.dim - e0 + 3) & ~3), tx, ty, acc);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = ty * 4 + i;
        if (r >= count) continue;
        float* dst = p.out + (size_t)(begin + r) * p.heads * p.vdim + (size_t)head * p.vdim + c0;
        if ((p.vdim & 3) == 0) {
            if (c0 + tx * 4 < p.vdim) *reinterpret_cast<float4*>(dst + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            continue;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (c0 + tx * 4 + j < p.vdim) dst[tx * 4 + j] = acc[i][j];
    }
}

// ---------------------------------------------------------------------------------------------------- decoding
struct DecayDecodeArgs {
    const float* q; int q_stride; const float* k; int k_stride; const float* v; int v_stride;
    float q_scale;
    // channel: the decay's low product in float32 rows, its second matrix [heads * dim, rank], bias, 1 / tau; the output's
    // head norm (weight of vdim, shared) and gate
    const float* low; int low_stride; const void* up; int rank; const float* bias; float inv_tau;
    const float* norm_w; float eps; const float* gate; int gate_stride;
    // scalar: the raw steps, their bias, A_log, the direct share
    const float* raw; int raw_stride; const float* dt_bias; const float* a_log; const float* direct;
    float* state; long long slot_stride; const int* span_slot;
    void* out;                               // channel: the gated head in the activation type; scalar: float32 read-outs
    int heads, groups, dim, vdim;
};

// A block a (head, token). A thread owns V neighbouring columns and every n-th row of the state; what it reads it updates,
// adds to its columns' read-out and writes. The row groups' sums meet in shared memory.
template <bool CHANNEL, typename A, int V>
__global__ void __launch_bounds__(256) decay_decode_kernel(const DecayDecodeArgs p) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float scratch[33];
    chain_release();
    chain_wait();
    const int head = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
    const int dim = p.dim, vdim = p.vdim;
    float* q_s = smem;                       // [dim]
    float* k_s = q_s + dim;
    float* a_s = k_s + dim;                  // channel
    float* o_s = a_s + (CHANNEL ? dim : 0);
    o_s = smem + (((o_s - smem) + 3) & ~3);  // [row groups][vdim]
    const int qk_head = CHANNEL ? head : head / (p.heads / p.groups);
    float decay = 1.0f, dt = 1.0f;
    if (!CHANNEL) {
        dt = softplus_of(p.raw[(size_t)t * p.raw_stride + head] + p.dt_bias[head]);
        decay = expf(-expf(p.a_log[head]) * dt);
    }
    for (int e = tid; e < dim; e += 256) {
        q_s[e] = p.q[(size_t)t * p.q_stride + (size_t)qk_head * dim + e] * p.q_scale;
        k_s[e] = p.k[(size_t)t * p.k_stride + (size_t)qk_head * dim + e] * dt;
    }
    if (CHANNEL) {
        // the decay's second product: a quarter warp a channel where the rank is worth it
        const float* low = p.low + (size_t)t * p.low_stride;
        const int part = tid & 7;
        for (int e0 = 0; e0 < dim; e0 += 32) {
            const int e = e0 + (tid >> 3);
            float sum = 0.0f;
            if (e < dim) {
                const A* up = static_cast<const A*>(p.up) + (size_t)(head * dim + e) * p.rank;
                for (int r = part; r < p.rank; r += 8) sum = fmaf(low[r], to_float(up[r]), sum);
            }
#pragma unroll
            for (int offset = 1; offset < 8; offset <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, offset);
            if (part == 0 && e < dim) a_s[e] = root_of_sigmoid(sum + p.bias[(size_t)head * dim + e], p.inv_tau);
        }
    }
    __syncthreads();
    float* s_head = p.state + (long long)p.span_slot[t] * p.slot_stride + (size_t)head * dim * vdim;
    const float* v_row = p.v + (size_t)t * p.v_stride + (size_t)head * vdim;
    const int units = vdim / V;              // column packs
    const int across = min(units, 256), row_groups = 256 / across;
    const int group = tid / across, unit0 = tid % across;
    if (group < row_groups) {
        for (int unit = unit0; unit < units; unit += across) {
            const int c = unit * V;
            float v[V], o[V];
#pragma unroll
            for (int i = 0; i < V; ++i) {
                v[i] = v_row[c + i];
                o[i] = 0.0f;
            }
            constexpr int kAhead = 8;
            for (int e0 = group; e0 < dim; e0 += kAhead * row_groups) {
                float s[kAhead][V];
#pragma unroll
                for (int u = 0; u < kAhead; ++u) {
                    const int e = e0 + u * row_groups;
                    if (e >= dim) continue;
                    const float* cell = s_head + (size_t)e * vdim + c;
                    if (V == 4) {
                        const float4 x = *reinterpret_cast<const float4*>(cell);
                        s[u][0] = x.x; s[u][1 % V] = x.y; s[u][2 % V] = x.z; s[u][3 % V] = x.w;
                    } else {
#pragma unroll
                        for (int i = 0; i < V; ++i) s[u][i] = cell[i];
                    }
                }
#pragma unroll
                for (int u = 0; u < kAhead; ++u) {
                    const int e = e0 + u * row_groups;
                    if (e >= dim) continue;
                    const float keep = CHANNEL ? a_s[e] : decay, ke = k_s[e], qe = q_s[e];
#pragma unroll
                    for (int i = 0; i < V; ++i) {
                        s[u][i] = fmaf(ke, v[i], keep * s[u][i]);
                        o[i] = fmaf(s[u][i], qe, o[i]);
                    }
                    float* cell = s_head + (size_t)e * vdim + c;
                    if (V == 4) *reinterpret_cast<float4*>(cell) = make_float4(s[u][0], s[u][1 % V], s[u][2 % V], s[u][3 % V]);
                    else {
#pragma unroll
                        for (int i = 0; i < V; ++i) cell[i] = s[u][i];
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < V; ++i) o_s[(size_t)group * vdim + c + i] = o[i];
        }
    }
    __syncthreads();
    float squares = 0.0f;
    for (int c = tid; c < vdim; c += 256) {
        float o = 0.0f;
        for (int g = 0; g < row_groups; ++g) o += o_s[(size_t)g * vdim + c];
        if (CHANNEL) {
            o_s[c] = o;                      // (column c is this thread's from here on)
            squares += o * o;
        } else {
            if (p.direct) o = fmaf(p.direct[head], v_row[c], o);
            static_cast<float*>(p.out)[((size_t)t * p.heads + head) * vdim + c] = o;
        }
    }
    if (CHANNEL) {
        const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)vdim + p.eps);
        A* dst = static_cast<A*>(p.out) + ((size_t)t * p.heads + head) * vdim;
        for (int c = tid; c < vdim; c += 256) {
            const float z = p.gate[(size_t)t * p.gate_stride + (size_t)head * vdim + c];
            dst[c] = from_float<A>(o_s[c] * inv * p.norm_w[c] * (z / (1.0f + expf(-z))));
        }
    }
}

template <bool CHANNEL, typename A>
static int launch_decay_decode(const DecayDecodeArgs& p, int tokens, cudaStream_t stream) {
    const bool four = p.vdim % 4 == 0 && p.slot_stride % 4 == 0 && ((size_t)p.state & 15) == 0;
    const int units = four ? p.vdim / 4 : p.vdim;
    const int across = units < 256 ? units : 256, row_groups = 256 / across;
    const size_t smem = ((size_t)3 * p.dim + 4 + (size_t)row_groups * p.vdim) * sizeof(float);
    CELEG_REQUIRE(smem <= 46 * 1024, "decay_decode: head sizes %d and %d exceed a block's shared memory", p.dim, p.vdim);
    dim3 grid(p.heads, tokens);
    if (four) launch_chained(decay_decode_kernel<CHANNEL, A, 4>, grid, 256, smem, stream, p);
    else launch_chained(decay_decode_kernel<CHANNEL, A, 1>, grid, 256, smem, stream, p);
    return check_launch("decay_decode");
}

template <bool CHANNEL>
static int launch_chunks(const ChunkArgs& p, float* state, long long slot_stride, const int* span_slot, const int* span_first,
                         int spans, int chunks, cudaStream_t stream) {
    const int v_tiles = (p.vdim + kChunk - 1) / kChunk, e_tiles = (p.dim + kChunk - 1) / kChunk;
    launch_chained(chunk_states_kernel<CHANNEL>, dim3(v_tiles * e_tiles, p.heads, chunks), 256, 0, stream, p);
    int status = check_launch("chunk_states");
    if (status != 0) return status;
    const long long elements = (long long)p.heads * p.dim * p.vdim;
    if (p.vdim % 4 == 0)                     // (scratch and slots are laid out for 16-byte accesses)
        launch_chained(chunk_carry_kernel<CHANNEL, 4>, dim3((unsigned)((elements / 4 + 127) / 128), spans), 128, 0, stream, p, state,
                       slot_stride, span_slot, span_first);
    else
        launch_chained(chunk_carry_kernel<CHANNEL, 1>, dim3((unsigned)((elements + 127) / 128), spans), 128, 0, stream, p, state,
                       slot_stride, span_slot, span_first);
    status = check_launch("chunk_carry");
    if (status != 0) return status;
    launch_chained(chunk_outputs_kernel<CHANNEL>, dim3(v_tiles, p.heads, chunks), 256, 0, stream, p);
    return check_launch("chunk_outputs");
}

}  // namespace celeg_b200

using namespace celeg_b200;

CELEG_API int celeg_chunk_tokens() { return kChunk; }

// plan: ints [max_chunks + 1 | spans + 1]: the chunks' first tokens (the last chunk's end at the end), the spans' first chunks
CELEG_API int celeg_chunk_plan(const int* span_begin, int spans, int max_chunks, int* plan, cudaStream_t stream) {
    CELEG_REQUIRE(spans >= 0 && max_chunks > 0, "chunk_plan: %d spans, %d chunks", spans, max_chunks);
    launch_chained(chunk_plan_kernel, 1, 32, 0, stream, span_begin, spans, kChunk, max_chunks, plan, plan + max_chunks + 1);
    return check_launch("chunk_plan");
}

// The channel form over the step's spans. q, k: float32 rows, head h at h * dim; z: the decay before its bias; scratch:
// q_out, k_out [tokens, heads * dim], total [chunks, heads * dim], products [chunks, heads, 64, 64], states [chunks, heads,
// dim, vdim]. plan: of celeg_chunk_plan with the same max_chunks (>= what the spans make).
CELEG_API int celeg_channel_decay_scan(const float* q, int q_stride, const float* k, int k_stride, const float* v, int v_stride,
                                       const float* z, int z_stride, const float* bias, float inv_tau, float q_scale,
                                       float* q_out, float* k_out, float* total, float* products, float* states, float* out,
                                       float* state, long long slot_stride, const int* span_slot, const int* plan,
                                       int max_chunks, int spans, int chunks, int heads, int dim, int vdim, cudaStream_t stream) {
    CELEG_REQUIRE(spans >= 0 && chunks >= 0 && heads > 0 && dim > 0 && dim <= kDecayMaxDim && vdim > 0,
                  "channel_decay_scan: invalid sizes spans=%d heads=%d dim=%d (at most %d) vdim=%d", spans, heads, dim,
                  kDecayMaxDim, vdim);
    CELEG_REQUIRE(chunks <= max_chunks && chunks <= 65535 && spans <= 65535 && heads <= 65535,
                  "channel_decay_scan: %d chunks of %d, %d spans or %d heads exceed one launch", chunks, max_chunks, spans, heads);
    if (spans == 0 || chunks == 0) return 0;
    const int* span_first = plan + max_chunks + 1;
    const ChannelPrepareArgs first = {q, q_stride, k, k_stride, z, z_stride, bias, inv_tau, q_scale, plan, q_out, k_out, total,
                                      products, heads, dim};
    const int status = dim <= 32 ? launch_channel_prepare<32>(first, chunks, stream)
                     : dim <= 64 ? launch_channel_prepare<64>(first, chunks, stream)
                     : dim <= 128 ? launch_channel_prepare<128>(first, chunks, stream)
                                  : launch_channel_prepare<256>(first, chunks, stream);
    if (status != 0) return status;
    const ChunkArgs p = {q_out, heads * dim, k_out, heads * dim, v, v_stride, nullptr, nullptr, total, products, nullptr, plan,
                         states, out, heads, heads, dim, vdim};
    return launch_chunks<true>(p, state, slot_stride, span_slot, span_first, spans, chunks, stream);
}

// The scalar form: q and k have `groups` heads of dim that heads / groups heads of v share; raw: the steps before bias and
// softplus, head h in column h. Scratch: cum (two floats each), dt [tokens, heads], products [chunks, groups, 64, 64], states as above.
CELEG_API int celeg_scalar_decay_scan(const float* q, int q_stride, const float* k, int k_stride, const float* v, int v_stride,
                                      const float* raw, int raw_stride, const float* dt_bias, const float* a_log,
                                      const float* direct, float2* cum, float* dt, float* products, float* states, float* out,
                                      float* state, long long slot_stride, const int* span_slot, const int* plan,
                                      int max_chunks, int spans, int chunks, int heads, int groups, int dim, int vdim,
                                      cudaStream_t stream) {
    CELEG_REQUIRE(spans >= 0 && chunks >= 0 && heads > 0 && groups > 0 && heads % groups == 0 && dim > 0 && vdim > 0,
                  "scalar_decay_scan: invalid sizes spans=%d heads=%d groups=%d dim=%d vdim=%d", spans, heads, groups, dim, vdim);
    CELEG_REQUIRE(chunks <= max_chunks && chunks <= 65535 && spans <= 65535 && heads <= 65535,
                  "scalar_decay_scan: %d chunks of %d, %d spans or %d heads exceed one launch", chunks, max_chunks, spans, heads);
    if (spans == 0 || chunks == 0) return 0;
    const int* span_first = plan + max_chunks + 1;
    launch_chained(scalar_decay_kernel, dim3((heads + 7) / 8, chunks), 256, 0, stream, raw, raw_stride, dt_bias, a_log, plan,
                   cum, dt, heads);
    int status = check_launch("scalar_decay");
    if (status != 0) return status;
    launch_chained(chunk_products_kernel, dim3(groups, chunks), 256, 0, stream, q, q_stride, k, k_stride, plan, products, groups, dim);
    status = check_launch("chunk_products");
    if (status != 0) return status;
    const ChunkArgs p = {q, q_stride, k, k_stride, v, v_stride, cum, dt, nullptr, products, direct, plan, states, out, heads,
                         groups, dim, vdim};
    return launch_chunks<false>(p, state, slot_stride, span_slot, span_first, spans, chunks, stream);
}

// A token a request (row i of the inputs is request i's token, its slot span_slot[i]): state update, read-out, and for the
// channel form the decay's second product (up [heads * dim, rank] in the activation type), the head norm, its weight and
// the SiLU gate.
CELEG_API int celeg_channel_decay_decode(const float* q, int q_stride, const float* k, int k_stride, const float* v, int v_stride,
                                         float q_scale, const float* low, int low_stride, const void* up, int rank,
                                         const float* bias, float inv_tau, const float* norm_w, float eps, const float* gate,
                                         int gate_stride, float* state, long long slot_stride, const int* span_slot, int tokens,
                                         int heads, int dim, int vdim, void* out, int act_dtype, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && tokens <= 65535 && heads > 0 && dim > 0 && vdim > 0 && rank > 0 && eps > 0.0f,
                  "channel_decay_decode: invalid sizes tokens=%d heads=%d dim=%d vdim=%d rank=%d", tokens, heads, dim, vdim, rank);
    CELEG_REQUIRE(act_dtype == kFloat32 || act_dtype == kBFloat16, "channel_decay_decode: unknown dtype code %d", act_dtype);
    if (tokens == 0) return 0;
    DecayDecodeArgs p = {};
    p.q = q; p.q_stride = q_stride; p.k = k; p.k_stride = k_stride; p.v = v; p.v_stride = v_stride; p.q_scale = q_scale;
    p.low = low; p.low_stride = low_stride; p.up = up; p.rank = rank; p.bias = bias; p.inv_tau = inv_tau;
    p.norm_w = norm_w; p.eps = eps; p.gate = gate; p.gate_stride = gate_stride;
    p.state = state; p.slot_stride = slot_stride; p.span_slot = span_slot; p.out = out;
    p.heads = heads; p.groups = heads; p.dim = dim; p.vdim = vdim;
    return act_dtype == kFloat32 ? launch_decay_decode<true, float>(p, tokens, stream)
                                 : launch_decay_decode<true, __nv_bfloat16>(p, tokens, stream);
}

CELEG_API int celeg_scalar_decay_decode(const float* q, int q_stride, const float* k, int k_stride, const float* v, int v_stride,
                                        const float* raw, int raw_stride, const float* dt_bias, const float* a_log,
                                        const float* direct, float* state, long long slot_stride, const int* span_slot,
                                        int tokens, int heads, int groups, int dim, int vdim, float* out, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && tokens <= 65535 && heads > 0 && groups > 0 && heads % groups == 0 && dim > 0 && vdim > 0,
                  "scalar_decay_decode: invalid sizes tokens=%d heads=%d groups=%d dim=%d vdim=%d", tokens, heads, groups, dim, vdim);
    if (tokens == 0) return 0;
    DecayDecodeArgs p = {};
    p.q = q; p.q_stride = q_stride; p.k = k; p.k_stride = k_stride; p.v = v; p.v_stride = v_stride; p.q_scale = 1.0f;
    p.raw = raw; p.raw_stride = raw_stride; p.dt_bias = dt_bias; p.a_log = a_log; p.direct = direct;
    p.state = state; p.slot_stride = slot_stride; p.span_slot = span_slot; p.out = out;
    p.heads = heads; p.groups = groups; p.dim = dim; p.vdim = vdim;
    return launch_decay_decode<false, float>(p, tokens, stream);
}
