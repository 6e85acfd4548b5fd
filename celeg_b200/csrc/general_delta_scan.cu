// The generalised delta rule over prompts and portions of prompts: a matrix state per head whose key channels each have a
// decay and a removal rate of their own. Per head with S [dim keys, dim values], float32 on both precision paths:
//
//   u = k / sqrt(sum(k^2) + unit_eps),   w = exp(-e^(-1/2) sigmoid(z + w0)),   b = sigmoid(a + a_bias) u
//   S_t = diag(w_t) S_(t-1) - b_t (u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t
//
// (both terms read the old state; z comes from a product of low rank).
//
// A column of S depends on itself alone, so what runs side by side is (span x head x column), and a token's step hangs on
// the step before it through the sum u^T S. Tokens are therefore taken in chunks of C = 8, counted from the span's first
// token in the step. With P_(i..j) the product of the decays of the chunk's tokens i to j (element by element; empty: one),
// tokens 1 .. C and S_0 the state before the chunk,
//
//   s_i := u_i^T S_(i-1) = (u_i P_(1..i-1))^T S_0 + sum_(j<i) [ (u_i P_(j+1..i-1))^T k_j v_j - (u_i P_(j+1..i-1))^T b_j s_j ]
//   o_i                  = (r_i P_(1..i))^T S_0   + sum_(j<=i) [ (r_i P_(j+1..i))^T k_j v_j - (r_i P_(j+1..i))^T b_j s_j ]
//   S_C                  = diag(P_(1..C)) S_0     + sum_j    [ (k_j P_(j+1..C)) v_j - (b_j P_(j+1..C)) s_j ]
//
// so all 2 C sums over the state are of the SAME state and their latencies overlap, and the eight steps that follow one
// another are over single numbers. What does not depend on the state is made before, for all chunks side by side:
//
//   vectors   the four vectors of every token (u P, r P, k P, b P), the chunk's whole decay, and the numbers of the
//             triangular sums, one record a chunk and head: a warp each. A decay is at least 0.545, a product of eight at
//             least 0.0078, so P_(j+1..i) = P_(1..i) / P_(1..j) loses nothing but rounding, and the triangular sums are
//             8 x 8 products of the vectors u P_(1..i-1) and r P_(1..i) with k / P_(1..j) and b / P_(1..j).
//   scan      a block walks one span's chunks for some columns of one head; a column lives in L lanes of 8 elements each.
//             A record is one bulk copy into a ring of stages, asked for by one thread while earlier chunks are worked on.
//
// A record of a chunk of n tokens, floats, from (head * tokens + first token) * (5 D + 24) on, D = 8 L:
//   [D] the chunk's decay | [n][8] pairs (-r_i.b_j, r_i.k_j) at [j][i], zero for i < j | pairs (-u_i.b_j, u_i.k_j), i = 1 ..
//   n - 1, j < i, filled up to a multiple of four | [n][4][D] the vectors
#include "general_delta.cuh"
#include "tcgen05.cuh"

#include <type_traits>

namespace celeg_b200 {

constexpr int kDeltaChunk = 8;

__host__ __device__ __forceinline__ int delta_record(int padded) { return 5 * padded + 3 * kDeltaChunk; }
__host__ __device__ __forceinline__ int delta_vectors_at(int padded, int n) {
    return padded + 2 * kDeltaChunk * n + ((n * (n - 1) + 3) & ~3);
}

struct DeltaVectorsArgs {
    const float* proj; int stride; int r_off, k_off, a_off;    // columns of a token's row: head h at h * dim
    const float* z; int z_stride;                              // [tokens, heads * dim], before its bias
    const float* w0; const float* a_bias;
    const int* token_span; const int* span_begin;
    float* records;
    int tokens, heads, dim;
    float unit_eps;
};

// One warp a (chunk, head); D: the head's size padded to a power of two (8 .. 256)
template <int D, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) delta_vectors_kernel(const DeltaVectorsArgs a) {
    constexpr int C = kDeltaChunk, kRow = D + 16;              // (rows 16 words apart modulo the banks)
    extern __shared__ __align__(16) float smem[];
    chain_release();
    chain_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * WARPS + warp;
    if (head >= a.heads) return;
    float* us = smem + warp * (4 * C * kRow);                  // u P_(1..i-1) | r P_(1..i) | k / P_(1..j) | b / P_(1..j)
    float* rs = us + C * kRow;
    float* ks = rs + C * kRow;
    float* bs = ks + C * kRow;
    const int t_first = blockIdx.x * C, t_last = min(t_first + C, a.tokens);
    for (int t0 = t_first; t0 < t_last; ++t0) {                // the chunks that begin among these tokens
        const int span = a.token_span[t0];
        const int begin = a.span_begin[span];
        if ((t0 - begin) % C != 0) continue;
        const int count = min(C, a.span_begin[span + 1] - t0);
        const float* row = a.proj + (size_t)t0 * a.stride + (size_t)head * a.dim;
        float inv[C];
#pragma unroll
        for (int i = 0; i < C; ++i) inv[i] = 0.0f;
        for (int e = lane; e < a.dim; e += 32) {
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const float k = i < count ? row[(size_t)i * a.stride + a.k_off + e] : 0.0f;
                inv[i] = fmaf(k, k, inv[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < C; ++i) inv[i] = 1.0f / sqrtf(warp_sum(inv[i]) + a.unit_eps);
        float* record = a.records + ((size_t)head * a.tokens + t0) * delta_record(D);
        float* vectors = record + delta_vectors_at(D, count);
        __syncwarp();                                          // (the chunk before has been read)
        for (int e = lane; e < D; e += 32) {
            const bool real = e < a.dim;
            const int column = head * a.dim + e;
            const float w0 = real ? a.w0[column] : 0.0f, a_bias = real ? a.a_bias[column] : 0.0f;
            float w[C], k[C], b[C];
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const bool here = real && i < count;
                const float* x = row + (size_t)i * a.stride + e;
                k[i] = here ? x[a.k_off] : 0.0f;
                b[i] = here ? x[a.a_off] + a_bias : 0.0f;
                w[i] = here ? a.z[(size_t)(t0 + i) * a.z_stride + column] + w0 : 0.0f;
                rs[i * kRow + e] = here ? x[a.r_off] : 0.0f;
            }
            float before = 1.0f;                               // P_(1..i-1)
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const bool here = real && i < count;
                w[i] = here ? channel_decay(w[i]) : 1.0f;
                const float u = k[i] * inv[i];
                b[i] = sigmoid_of(b[i]) * u;
                const float through = before * w[i];           // P_(1..i)
                const float up = u * before, rp = rs[i * kRow + e] * through, back = 1.0f / through;
                us[i * kRow + e] = up;
                rs[i * kRow + e] = rp;
                ks[i * kRow + e] = k[i] * back;
                bs[i * kRow + e] = b[i] * back;
                if (i < count) {
                    vectors[(4 * i) * D + e] = up;
                    vectors[(4 * i + 1) * D + e] = rp;
                }
                before = through;
            }
            record[e] = before;
            float after = 1.0f;                                // P_(i+1..C)
#pragma unroll
            for (int i = C - 1; i >= 0; --i) {
                if (i < count) {
                    vectors[(4 * i + 2) * D + e] = k[i] * after;
                    vectors[(4 * i + 3) * D + e] = b[i] * after;
                }
                after *= w[i];
            }
        }
        __syncwarp();
        // the triangular sums: lane (i, q) adds up the elements 4 (q + 4 m) .. + 3 of u_i and r_i against every j
        const int i = lane >> 2, q = lane & 3;
        float acc[32];                                         // [u.b | u.k | r.b | r.k][j]
#pragma unroll
        for (int x = 0; x < 32; ++x) acc[x] = 0.0f;
        for (int e = 4 * q; e < D; e += 16) {
            const float4 u = *reinterpret_cast<const float4*>(us + i * kRow + e);
            const float4 r = *reinterpret_cast<const float4*>(rs + i * kRow + e);
#pragma unroll
            for (int j = 0; j < C; ++j) {
                const float4 k = *reinterpret_cast<const float4*>(ks + j * kRow + e);
                const float4 b = *reinterpret_cast<const float4*>(bs + j * kRow + e);
                acc[j] = fmaf(u.x, b.x, fmaf(u.y, b.y, fmaf(u.z, b.z, fmaf(u.w, b.w, acc[j]))));
                acc[8 + j] = fmaf(u.x, k.x, fmaf(u.y, k.y, fmaf(u.z, k.z, fmaf(u.w, k.w, acc[8 + j]))));
                acc[16 + j] = fmaf(r.x, b.x, fmaf(r.y, b.y, fmaf(r.z, b.z, fmaf(r.w, b.w, acc[16 + j]))));
                acc[24 + j] = fmaf(r.x, k.x, fmaf(r.y, k.y, fmaf(r.z, k.z, fmaf(r.w, k.w, acc[24 + j]))));
            }
        }
        // the four lanes of a token: after two exchanges lane q holds the whole sums of kind q
#pragma unroll
        for (int x = 0; x < 16; ++x) {
            const bool upper = (q & 2) != 0;
            const float give = upper ? acc[x] : acc[x + 16];
            acc[x] = (upper ? acc[x + 16] : acc[x]) + __shfl_xor_sync(0xffffffffu, give, 2);
        }
#pragma unroll
        for (int x = 0; x < 8; ++x) {
            const bool upper = (q & 1) != 0;
            const float give = upper ? acc[x] : acc[x + 8];
            acc[x] = (upper ? acc[x + 8] : acc[x]) + __shfl_xor_sync(0xffffffffu, give, 1);
        }
        const float sign = (q & 1) ? 1.0f : -1.0f;
        if (q >= 2) {
#pragma unroll
            for (int j = 0; j < C; ++j)
                if (j < count) record[D + 2 * (j * C + i) + (q & 1)] = i >= j && i < count ? sign * acc[j] : 0.0f;
        } else if (i < count) {
            float* line = record + D + 2 * C * count + i * (i - 1);
#pragma unroll
            for (int j = 0; j < C; ++j)
                if (j < i) line[2 * j + q] = sign * acc[j];
        }
    }
}

struct DeltaScanArgs {
    const float* records;
    const float* v; int v_stride;                              // values: head h at h * dim
    float* out;                                                // [tokens, heads * dim]
    float* state; long long slot_stride;
    const int* span_begin; const int* span_slot;
    int tokens, heads, dim;
    int* error_flag;
};

constexpr int kDeltaWarps = 4;

// What a chunk costs is mostly shared memory's bandwidth (a number that several lanes read costs as much as several
// numbers) in two phases that the sums among lanes keep apart. Measured at 32 heads of 64 and 2,048 tokens: 290 us; four
// elements a lane and twice the lanes a column: 340 us; two multiplications an instruction (fma.rn.f32x2): 290 us.
template <int L>
__global__ void __launch_bounds__(kDeltaWarps * 32, 1) delta_scan_kernel(const DeltaScanArgs p) {
    constexpr int C = kDeltaChunk, D = 8 * L;
    constexpr int kColsWarp = 32 / L, kCols = kDeltaWarps * kColsWarp;
    constexpr int kStages = L >= 16 ? 3 : 4;
    constexpr int kStage = 33 * D + 184;                       // a full chunk's record
    constexpr int kBits = L >= 8 ? 3 : L == 4 ? 2 : L == 2 ? 1 : 0;      // lanes that share out a chunk's tokens: 2^kBits
    constexpr int kMine = C >> kBits;                          // tokens a lane reads out
    extern __shared__ __align__(16) float smem[];
    __shared__ __align__(8) unsigned long long full_bar[kStages];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int sub = lane % L, col_in = warp * kColsWarp + lane / L;
    const int head = blockIdx.y, span = blockIdx.z;
    const int col = blockIdx.x * kCols + col_in;
    const bool col_ok = col < p.dim;
    const int t_begin = p.span_begin[span], t_end = p.span_begin[span + 1];
    if (t_end <= t_begin) return;
    if (tid == 0) {
        for (int s = 0; s < kStages; ++s) mbar_init(smem_u32(&full_bar[s]), 1);
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    __syncthreads();
    const int chunks = (t_end - t_begin + C - 1) / C;
    const float* records = p.records + ((size_t)head * p.tokens + t_begin) * delta_record(D);
    auto issue = [&](int chunk) {                              // (one thread)
        const int n = min(C, t_end - t_begin - chunk * C);
        const unsigned bytes = (unsigned)(delta_vectors_at(D, n) + 4 * n * D) * 4u;
        const unsigned bar = smem_u32(&full_bar[chunk % kStages]);
        mbar_expect_tx(bar, bytes);
        bulk_load(smem_u32(smem + (chunk % kStages) * kStage), records + (size_t)chunk * C * delta_record(D), bytes, bar);
    };
    if (tid == 0)
        for (int c = 0; c < min(chunks, kStages - 1); ++c) issue(c);
    float* s_head = p.state + (long long)p.span_slot[span] * p.slot_stride + (size_t)head * p.dim * p.dim;
    float s[8];
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        const int e = 4 * ((r >> 2) * L + sub) + (r & 3);
        s[r] = (col_ok && e < p.dim) ? s_head[(size_t)e * p.dim + col] : 0.0f;
    }
    int first_token = 0;                                       // of the kMine tokens that this lane reads out
#pragma unroll
    for (int b = 0; b < kBits; ++b) first_token += ((sub >> b) & 1) * (C >> (b + 1));
    const bool writes = col_ok && (sub >> kBits) == 0;
    const float* v_at = p.v + (size_t)head * p.dim + (col_ok ? col : 0);
    float v[C], v_next[C];
#pragma unroll
    for (int i = 0; i < C; ++i) v_next[i] = t_begin + i < t_end ? v_at[(size_t)(t_begin + i) * p.v_stride] : 0.0f;

    bool ok = true;
    int chunk = 0;
    for (; chunk < chunks; ++chunk) {
        const int t0 = t_begin + chunk * C, count = min(C, t_end - t0), stage = chunk % kStages;
        ok = mbar_wait(smem_u32(&full_bar[stage]), (chunk / kStages) & 1);
        ok = __syncthreads_and(ok);                            // (and every thread has left the chunk before)
        if (!ok) break;
        if (tid == 0 && chunk + kStages - 1 < chunks) issue(chunk + kStages - 1);
#pragma unroll
        for (int i = 0; i < C; ++i) v[i] = v_next[i];
#pragma unroll
        for (int i = 0; i < C; ++i) v_next[i] = t0 + C + i < t_end ? v_at[(size_t)(t0 + C + i) * p.v_stride] : 0.0f;
        // (a full chunk's loops have a constant length: no branches between the tokens' loads)
        auto work = [&](auto full, int tokens_here) {
            const int n = decltype(full)::value ? C : tokens_here;
            const float* base = smem + stage * kStage;
            const float* outward = base + D;                       // pairs (-r.b, r.k) at [j][i]
            const float* inward = base + D + 2 * C * n;        // pairs (-u.b, u.k), i(i-1) floats before token i's
            const float* vectors = base + delta_vectors_at(D, n);
            float su[C], sq[C];
#pragma unroll
            for (int i = 0; i < C; ++i) {
                if (i < n) {
                    const float4* up = reinterpret_cast<const float4*>(vectors + (4 * i) * D);
                    const float4* rp = reinterpret_cast<const float4*>(vectors + (4 * i + 1) * D);
                    const float4 u0 = up[sub], u1 = up[L + sub], r0 = rp[sub], r1 = rp[L + sub];
                    su[i] = fmaf(s[0], u0.x, s[1] * u0.y) + fmaf(s[2], u0.z, s[3] * u0.w) +
                            (fmaf(s[4], u1.x, s[5] * u1.y) + fmaf(s[6], u1.z, s[7] * u1.w));
                    sq[i] = fmaf(s[0], r0.x, s[1] * r0.y) + fmaf(s[2], r0.z, s[3] * r0.w) +
                            (fmaf(s[4], r1.x, s[5] * r1.y) + fmaf(s[6], r1.z, s[7] * r1.w));
                } else {
                    su[i] = sq[i] = 0.0f;
                }
            }
            // the lanes of a column exchange halves: afterwards a lane has the whole sums of its own kMine tokens
#pragma unroll
            for (int b = 0; b < kBits; ++b) {
                const int half = C >> (b + 1);
                const bool upper = ((sub >> b) & 1) != 0;
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const float give_u = upper ? su[i] : su[i + half], give_q = upper ? sq[i] : sq[i + half];
                    su[i] = (upper ? su[i + half] : su[i]) + __shfl_xor_sync(0xffffffffu, give_u, 1 << b);
                    sq[i] = (upper ? sq[i + half] : sq[i]) + __shfl_xor_sync(0xffffffffu, give_q, 1 << b);
                }
            }
#pragma unroll
            for (int offset = C; offset < L; offset <<= 1) {
                su[0] += __shfl_xor_sync(0xffffffffu, su[0], offset);
                sq[0] += __shfl_xor_sync(0xffffffffu, sq[0], offset);
            }
            float taken[C];                                        // u_i^T S_(i-1), all tokens in every lane
#pragma unroll
            for (int i = 0; i < C; ++i) {
                int from = 0;                                      // which lane of the column holds token i
#pragma unroll
                for (int b = 0; b < kBits; ++b) from |= ((i >> (2 - b)) & 1) << b;
                taken[i] = __shfl_sync(0xffffffffu, su[i % kMine], (lane & ~((1 << kBits) - 1)) | from);
            }
#pragma unroll
            for (int i = 1; i < C; ++i) {
                if (i < n) {
                    const float2* line = reinterpret_cast<const float2*>(inward + i * (i - 1));
                    // (the values' share first: then one product only hangs on the token before)
#pragma unroll
                    for (int j = 0; j < i; ++j) taken[i] = fmaf(line[j].y, v[j], taken[i]);
#pragma unroll
                    for (int j = 0; j < i; ++j) taken[i] = fmaf(line[j].x, taken[j], taken[i]);
                }
            }
#pragma unroll
            for (int m = 0; m < kMine; ++m) {
                const int i = first_token + m;
                float removed = 0.0f, written = sq[m];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    if (j < n) {
                        const float2 pair = *reinterpret_cast<const float2*>(outward + 2 * (j * C + i));
                        removed = fmaf(pair.x, taken[j], removed);
                        written = fmaf(pair.y, v[j], written);
                    }
                }
                if (writes && i < n)
                    p.out[(size_t)(t0 + i) * p.heads * p.dim + (size_t)head * p.dim + col] = written + removed;
            }
            const float4* dp = reinterpret_cast<const float4*>(base);
            const float4 d0 = dp[sub], d1 = dp[L + sub];
            s[0] *= d0.x; s[1] *= d0.y; s[2] *= d0.z; s[3] *= d0.w;
            s[4] *= d1.x; s[5] *= d1.y; s[6] *= d1.z; s[7] *= d1.w;
#pragma unroll
            for (int i = 0; i < C; ++i) {
                if (i < n) {
                    const float4* kp = reinterpret_cast<const float4*>(vectors + (4 * i + 2) * D);
                    const float4* bp = reinterpret_cast<const float4*>(vectors + (4 * i + 3) * D);
                    const float4 k0 = kp[sub], k1 = kp[L + sub], b0 = bp[sub], b1 = bp[L + sub];
                    const float vi = v[i], ni = -taken[i];
                    s[0] = fmaf(b0.x, ni, fmaf(k0.x, vi, s[0])); s[1] = fmaf(b0.y, ni, fmaf(k0.y, vi, s[1]));
                    s[2] = fmaf(b0.z, ni, fmaf(k0.z, vi, s[2])); s[3] = fmaf(b0.w, ni, fmaf(k0.w, vi, s[3]));
                    s[4] = fmaf(b1.x, ni, fmaf(k1.x, vi, s[4])); s[5] = fmaf(b1.y, ni, fmaf(k1.y, vi, s[5]));
                    s[6] = fmaf(b1.z, ni, fmaf(k1.z, vi, s[6])); s[7] = fmaf(b1.w, ni, fmaf(k1.w, vi, s[7]));
                }
            }
        };
        if (count == C) work(std::true_type{}, C);
        else work(std::false_type{}, count);
    }
    if (!ok) {
        if (tid == 0) {
            atomicExch(p.error_flag, 31);
            // copies that were asked for must land before the shared memory goes away
            for (int c = chunk; c < min(chunks, chunk + kStages - 1); ++c)
                mbar_wait(smem_u32(&full_bar[c % kStages]), (c / kStages) & 1);
        }
        __syncthreads();
        return;
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        const int e = 4 * ((r >> 2) * L + sub) + (r & 3);
        if (col_ok && e < p.dim) s_head[(size_t)e * p.dim + col] = s[r];
    }
}

template <int L>
static int launch_delta_scan(const DeltaVectorsArgs& first, const DeltaScanArgs& p, int spans, cudaStream_t stream) {
    constexpr int D = 8 * L, kCols = kDeltaWarps * (32 / L), kStages = L >= 16 ? 3 : 4;
    constexpr int kVectorsWarps = L >= 32 ? 1 : L >= 16 ? 2 : 4;
    constexpr size_t vectors_smem = (size_t)kVectorsWarps * 4 * kDeltaChunk * (D + 16) * sizeof(float);
    constexpr size_t scan_smem = (size_t)kStages * (33 * D + 184) * sizeof(float);
    auto vectors_kernel = delta_vectors_kernel<D, kVectorsWarps>;
    auto scan_kernel = delta_scan_kernel<L>;
    cudaError_t status = cudaSuccess;
    if (vectors_smem > 40 * 1024)
        status = cudaFuncSetAttribute(vectors_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)vectors_smem);
    if (status == cudaSuccess && scan_smem > 40 * 1024)
        status = cudaFuncSetAttribute(scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan_smem);
    if (status != cudaSuccess) {
        set_error("general_delta_scan: %s", cudaGetErrorString(status));
        return -2;
    }
    dim3 vectors_grid((first.tokens + kDeltaChunk - 1) / kDeltaChunk, (first.heads + kVectorsWarps - 1) / kVectorsWarps);
    launch_chained(vectors_kernel, vectors_grid, kVectorsWarps * 32, vectors_smem, stream, first);
    const int code = check_launch("general_delta_vectors");
    if (code != 0) return code;
    dim3 grid((p.dim + kCols - 1) / kCols, p.heads, spans);
    // (a plain launch: few long blocks, see recurrent_scan.cu)
    scan_kernel<<<grid, kDeltaWarps * 32, scan_smem, stream>>>(p);
    return check_launch("general_delta_scan");
}

static int delta_padded(int dim) {
    int padded = 8;
    while (padded < dim) padded <<= 1;
    return padded;
}

}  // namespace celeg_b200

using namespace celeg_b200;

// Floats of scratch that a step of `tokens` tokens needs (all heads), 0 if the head size is not taken.
CELEG_API int celeg_general_delta_scratch(int heads, int dim) {
    return dim > 0 && dim <= kDeltaMaxDim ? heads * delta_record(delta_padded(dim)) : 0;
}

// The recurrence over the step's spans (two launches). Offsets: columns of r, k, v and the removal rate in a row of
// proj (float32, rows `stride` apart); z: float32 [tokens, heads * dim]. records: scratch of tokens times
// celeg_general_delta_scratch() floats.
CELEG_API int celeg_general_delta_scan(const float* proj, int stride, int r_off, int k_off, int v_off, int a_off,
                                       const float* z, int z_stride, const float* w0, const float* a_bias, float unit_eps,
                                       const int* token_span, const int* span_begin, const int* span_slot, float* records,
                                       float* out, float* state, long long slot_stride, int tokens, int spans, int heads,
                                       int dim, int* error_flag, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && spans >= 0 && heads > 0 && dim > 0 && dim <= kDeltaMaxDim && unit_eps > 0.0f,
                  "general_delta_scan: invalid sizes tokens=%d spans=%d heads=%d dim=%d (at most %d)", tokens, spans, heads, dim,
                  kDeltaMaxDim);
    CELEG_REQUIRE(spans <= 65535 && heads <= 65535, "general_delta_scan: %d spans or %d heads exceed one launch", spans, heads);
    CELEG_REQUIRE(((size_t)records & 15) == 0 && error_flag, "general_delta_scan: the records must be 16-byte aligned, and a flag given");
    if (tokens == 0 || spans == 0) return 0;
    const int padded = delta_padded(dim);
    const DeltaVectorsArgs first = {proj, stride, r_off, k_off, a_off, z, z_stride, w0, a_bias, token_span, span_begin, records,
                                    tokens, heads, dim, unit_eps};
    const DeltaScanArgs p = {records, proj + v_off, stride, out, state, slot_stride, span_begin, span_slot, tokens, heads, dim,
                             error_flag};
    switch (padded) {
        case 8: return launch_delta_scan<1>(first, p, spans, stream);
        case 16: return launch_delta_scan<2>(first, p, spans, stream);
        case 32: return launch_delta_scan<4>(first, p, spans, stream);
        case 64: return launch_delta_scan<8>(first, p, spans, stream);
        case 128: return launch_delta_scan<16>(first, p, spans, stream);
        default: return launch_delta_scan<32>(first, p, spans, stream);
    }
}
