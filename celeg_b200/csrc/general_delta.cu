// The generalised delta rule: a matrix state per head whose key channels each have a decay and a removal rate of their
// own. Per head with S [dim keys, dim values], float32 on both precision paths:
//
//   u = k / sqrt(sum(k^2) + unit_eps),   w = exp(-e^(-1/2) sigmoid(z + w0)),   b = sigmoid(a + a_bias) u
//   S_t = diag(w_t) S_(t-1) - b_t (u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t
//
// (both terms read the old state; z comes from a product of low rank).
//
// Prompts. A column of S depends on itself alone, so what runs side by side is (span x head x column), and a token's
// step hangs on the step before it through the sum u^T S. Tokens are therefore taken in chunks of C = 8, counted from the
// span's first token in the step. With P_(i..j) the product of the decays of the chunk's tokens i to j (element by
// element; empty: one), tokens 1 .. C and S_0 the state before the chunk,
//
//   s_i := u_i^T S_(i-1) = (u_i P_(1..i-1))^T S_0 + sum_(j<i) [ (u_i P_(j+1..i-1))^T k_j v_j - (u_i P_(j+1..i-1))^T b_j s_j ]
//   o_i                  = (r_i P_(1..i))^T S_0   + sum_(j<=i) [ (r_i P_(j+1..i))^T k_j v_j - (r_i P_(j+1..i))^T b_j s_j ]
//   S_C                  = diag(P_(1..C)) S_0     + sum_j    [ (k_j P_(j+1..C)) v_j - (b_j P_(j+1..C)) s_j ]
//
// so all 2 C sums over the state are of the SAME state and their latencies overlap, and the eight steps that follow one
// another are over single numbers. Every P is a product of numbers in (0, 1) formed as such (no quotients), so nothing
// overflows whatever the decays. What does not depend on the state is made before, for all chunks side by side:
//
//   prepare   the four vectors of every token (u P, r P, k P, b P), the chunk's whole decay, and the 128 numbers of a
//             chunk's triangular sums (28 pairs j < i with u, 36 pairs j <= i with r, each against b and k): a warp per
//             (chunk, head)
//   scan      a block walks one span's chunks for some columns of one head; a column lives in L lanes of 8 elements
//             each; the next chunks come in by cp.async while the current one is worked on
//
// Decoding (every request brings one token): one block per (request, head) does everything between the input and the
// output projection, the decay's second product included.
#include "common.cuh"
#include "mma_tiles.cuh"

namespace celeg_b200 {

constexpr int kDeltaChunk = 8;
constexpr int kDeltaSums = 2 * kDeltaChunk * kDeltaChunk;      // a chunk's triangular sums: token i has 4 i + 2, from 2 i^2 on
constexpr int kDeltaMaxDim = 256;
constexpr float kDecaySpan = 0.60653065971263342f;             // e^(-1/2)

__device__ __forceinline__ float sigmoid_of(float x) { return 1.0f / (1.0f + expf(-x)); }
// 1 + expm1: a decay close to one is then its nearest float, without a bias that thousands of steps would add up
__device__ __forceinline__ float channel_decay(float z) { return 1.0f + expm1f(-kDecaySpan * sigmoid_of(z)); }

struct DeltaVectorsArgs {
    const float* proj; int stride; int r_off, k_off, a_off;    // columns of a token's row: head h at h * dim
    const float* z; int z_stride;                              // [tokens, heads * dim], before its bias
    const float* w0; const float* a_bias;
    const int* token_span; const int* span_begin;
    float* vectors;                                            // [tokens][heads][4][dim_pad]: u P, r P, k P, b P
    float* decay;                                              // [tokens][heads][dim_pad], at a chunk's first token
    float* sums;                                               // [heads][tokens][2 C], a chunk's numbers from its first token on
    int tokens, heads, dim, dim_pad;
    float unit_eps;
};

// Lane l of the warp gets the warp's sum of value l: 31 shuffles for 32 sums.
__device__ __forceinline__ float transpose_sum(float (&v)[32], int lane) {
#pragma unroll
    for (int half = 16; half > 0; half >>= 1) {
        const bool upper = (lane & half) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float give = upper ? v[i] : v[i + half];
            const float keep = upper ? v[i + half] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, give, half);
        }
    }
    return v[0];
}

constexpr int kVectorsWarps = 4;

__global__ void __launch_bounds__(kVectorsWarps * 32) delta_vectors_kernel(const DeltaVectorsArgs a) {
    constexpr int C = kDeltaChunk;
    chain_release();
    chain_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * kVectorsWarps + warp;
    if (head >= a.heads) return;
    const int t_first = blockIdx.x * C, t_last = min(t_first + C, a.tokens);
    for (int t0 = t_first; t0 < t_last; ++t0) {                // the chunks that begin among these tokens
        const int span = a.token_span[t0];
        if ((t0 - a.span_begin[span]) % C != 0) continue;
        const int count = min(C, a.span_begin[span + 1] - t0);
        const float* row = a.proj + (size_t)t0 * a.stride + (size_t)head * a.dim;
        float inv[C];
#pragma unroll
        for (int i = 0; i < C; ++i) {
            float squares = 0.0f;
            if (i < count)
                for (int e = lane; e < a.dim; e += 32) {
                    const float k = row[(size_t)i * a.stride + a.k_off + e];
                    squares = fmaf(k, k, squares);
                }
            inv[i] = squares;
        }
#pragma unroll
        for (int i = 0; i < C; ++i) inv[i] = 1.0f / sqrtf(warp_sum(inv[i]) + a.unit_eps);
        float part[4][32];                                     // 128 sums, in the order token i: u.b u.k (j < i), r.b r.k (j <= i)
#pragma unroll
        for (int g = 0; g < 4; ++g)
#pragma unroll
            for (int i = 0; i < 32; ++i) part[g][i] = 0.0f;
        for (int e = lane; e < a.dim_pad; e += 32) {
            const bool real = e < a.dim;
            float w[C], k[C], b[C], r[C];
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const bool here = real && i < count;
                const float* x = row + (size_t)i * a.stride + e;
                const int column = head * a.dim + e;
                k[i] = here ? x[a.k_off] : 0.0f;
                r[i] = here ? x[a.r_off] : 0.0f;
                const float removal = here ? x[a.a_off] + a.a_bias[column] : 0.0f;
                const float z = here ? a.z[(size_t)(t0 + i) * a.z_stride + column] + a.w0[column] : 0.0f;
                w[i] = here ? channel_decay(z) : 1.0f;
                b[i] = sigmoid_of(removal) * (k[i] * inv[i]);
            }
            float before = 1.0f;                               // P_(1..i-1)
            float* vec = a.vectors + (((size_t)t0 * a.heads + head) * 4) * a.dim_pad + e;
            const size_t token_step = (size_t)a.heads * 4 * a.dim_pad;
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const float u = k[i] * inv[i];
                const float through = before * w[i];           // P_(1..i)
                if (i < count) {
                    vec[i * token_step] = u * before;
                    vec[i * token_step + a.dim_pad] = r[i] * through;
                }
                before = through;
                // the triangular sums: u_i P_(j+1..i-1) and r_i P_(j+1..i) against k_j and b_j
                float pu = u, pr = r[i];
                part[(2 * i * i + 4 * i) / 32][(2 * i * i + 4 * i) % 32] =
                    fmaf(pr, b[i], part[(2 * i * i + 4 * i) / 32][(2 * i * i + 4 * i) % 32]);
                part[(2 * i * i + 4 * i + 1) / 32][(2 * i * i + 4 * i + 1) % 32] =
                    fmaf(pr, k[i], part[(2 * i * i + 4 * i + 1) / 32][(2 * i * i + 4 * i + 1) % 32]);
                pr *= w[i];
#pragma unroll
                for (int j = C - 1; j >= 0; --j) {
                    if (j >= i) continue;
                    const int at = 2 * i * i + 4 * j;          // (u.b, u.k, r.b, r.k) of the pair (i, j)
                    part[at / 32][at % 32] = fmaf(pu, b[j], part[at / 32][at % 32]);
                    part[(at + 1) / 32][(at + 1) % 32] = fmaf(pu, k[j], part[(at + 1) / 32][(at + 1) % 32]);
                    part[(at + 2) / 32][(at + 2) % 32] = fmaf(pr, b[j], part[(at + 2) / 32][(at + 2) % 32]);
                    part[(at + 3) / 32][(at + 3) % 32] = fmaf(pr, k[j], part[(at + 3) / 32][(at + 3) % 32]);
                    pu *= w[j];
                    pr *= w[j];
                }
            }
            a.decay[((size_t)t0 * a.heads + head) * a.dim_pad + e] = before;
            float after = 1.0f;                                // P_(i+1..C)
#pragma unroll
            for (int i = C - 1; i >= 0; --i) {
                if (i < count) {
                    vec[i * token_step + 2 * a.dim_pad] = k[i] * after;
                    vec[i * token_step + 3 * a.dim_pad] = b[i] * after;
                }
                after *= w[i];
            }
        }
        float* sums = a.sums + ((size_t)head * a.tokens + t0) * (2 * C);
        const int used = 2 * count * count;                    // (a short last chunk has room for count * 2 C numbers)
#pragma unroll
        for (int g = 0; g < 4; ++g) {
            const float total = transpose_sum(part[g], lane);
            if (32 * g + lane < used) sums[32 * g + lane] = total;
        }
    }
}

struct DeltaScanArgs {
    const float* vectors; const float* decay; const float* sums;
    const float* v; int v_stride;                              // values: head h at h * dim
    float* out;                                                // [tokens, heads * dim]
    float* state; long long slot_stride;
    const int* span_begin; const int* span_slot;
    int tokens, heads, dim, dim_pad;
};

constexpr int kDeltaWarps = 4;

template <int L>
__global__ void __launch_bounds__(kDeltaWarps * 32) delta_scan_kernel(const DeltaScanArgs p) {
    constexpr int C = kDeltaChunk, kRegs = 8, kThreads = kDeltaWarps * 32;
    constexpr int kColsWarp = 32 / L, kCols = kDeltaWarps * kColsWarp;
    constexpr int kDimPad = kRegs * L;
    constexpr int kStages = L >= 16 ? 2 : 3;
    // a stage: [C][4][kDimPad] vectors | [kDimPad] decay | [128] sums | [C][kCols] values
    constexpr int kVectors = C * 4 * kDimPad, kDecayAt = kVectors, kSumsAt = kDecayAt + kDimPad, kValuesAt = kSumsAt + kDeltaSums;
    constexpr int kStage = kValuesAt + C * kCols;
    extern __shared__ __align__(16) float smem[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int sub = lane % L, col_in = warp * kColsWarp + lane / L;
    const int head = blockIdx.y, span = blockIdx.z;
    const int col = blockIdx.x * kCols + col_in;
    const bool col_ok = col < p.dim;
    const int t_begin = p.span_begin[span], t_end = p.span_begin[span + 1];
    if (t_end <= t_begin) return;
    for (int i = tid; i < kStages * kStage; i += kThreads) smem[i] = 0.0f;      // (what copies never write stays zero)
    __syncthreads();
    float* s_head = p.state + (long long)p.span_slot[span] * p.slot_stride + (size_t)head * p.dim * p.dim;
    float s[kRegs];
#pragma unroll
    for (int r = 0; r < kRegs; ++r) {
        const int e = 4 * ((r >> 2) * L + sub) + (r & 3);
        s[r] = (col_ok && e < p.dim) ? s_head[(size_t)e * p.dim + col] : 0.0f;
    }
    const int quads = p.dim_pad >> 2;
    auto issue = [&](int t0, int stage) {
        float* base = smem + stage * kStage;
        const int count = min(C, t_end - t0);
        for (int i = tid; i < count * 4 * quads; i += kThreads) {
            const int piece = i / quads, q = i - piece * quads;          // piece: token * 4 + which vector
            cp_async_16(base + piece * kDimPad + 4 * q,
                        p.vectors + (((size_t)(t0 + (piece >> 2)) * p.heads + head) * 4 + (piece & 3)) * p.dim_pad + 4 * q);
        }
        for (int q = tid; q < quads; q += kThreads)
            cp_async_16(base + kDecayAt + 4 * q, p.decay + ((size_t)t0 * p.heads + head) * p.dim_pad + 4 * q);
        for (int q = tid; q < count * 4; q += kThreads)                   // (2 C numbers a token)
            cp_async_16(base + kSumsAt + 4 * q, p.sums + ((size_t)head * p.tokens + t0) * (2 * C) + 4 * q);
        for (int i = tid; i < count * kCols; i += kThreads) {
            const int tt = i / kCols, c = i % kCols, gc = blockIdx.x * kCols + c;
            if (gc < p.dim) {
                const unsigned to = (unsigned)__cvta_generic_to_shared(base + kValuesAt + i);
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(to),
                             "l"(p.v + (size_t)(t0 + tt) * p.v_stride + (size_t)head * p.dim + gc));
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < kStages - 1; ++i) {
        if (t_begin + i * C < t_end) issue(t_begin + i * C, i);
        else cp_async_commit();
    }
    int stage = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += C) {
        cp_async_wait_group<kStages - 2>();
        __syncthreads();              // this chunk's copies have landed, and every thread has left the chunk before
        {
            const int ahead = t0 + (kStages - 1) * C;
            int to = stage + kStages - 1;
            if (to >= kStages) to -= kStages;
            if (ahead < t_end) issue(ahead, to);
            else cp_async_commit();
        }
        const float* base = smem + stage * kStage;
        const float* sums = base + kSumsAt;
        const int count = min(C, t_end - t0);
        if (count == C) {
            float su[C], sq[C], v[C];
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const float4* up = reinterpret_cast<const float4*>(base + (4 * i) * kDimPad);
                const float4* rp = reinterpret_cast<const float4*>(base + (4 * i + 1) * kDimPad);
                const float4 u0 = up[sub], u1 = up[L + sub], r0 = rp[sub], r1 = rp[L + sub];
                su[i] = fmaf(s[0], u0.x, s[1] * u0.y) + fmaf(s[2], u0.z, s[3] * u0.w) +
                        (fmaf(s[4], u1.x, s[5] * u1.y) + fmaf(s[6], u1.z, s[7] * u1.w));
                sq[i] = fmaf(s[0], r0.x, s[1] * r0.y) + fmaf(s[2], r0.z, s[3] * r0.w) +
                        (fmaf(s[4], r1.x, s[5] * r1.y) + fmaf(s[6], r1.z, s[7] * r1.w));
                v[i] = base[kValuesAt + i * kCols + col_in];
            }
#pragma unroll
            for (int offset = 1; offset < L; offset <<= 1) {
#pragma unroll
                for (int i = 0; i < C; ++i) {
                    su[i] += __shfl_xor_sync(0xffffffffu, su[i], offset);
                    sq[i] += __shfl_xor_sync(0xffffffffu, sq[i], offset);
                }
            }
            // the tokens' sums one from the other; su[i] becomes u_i^T S_(i-1)
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const float2* line = reinterpret_cast<const float2*>(sums + 2 * i * i);
                float with_b = 0.0f, with_k = 0.0f;
#pragma unroll
                for (int j = 0; j < i; ++j) {
                    const float2 ub_uk = line[2 * j], rb_rk = line[2 * j + 1];
                    su[i] = fmaf(ub_uk.y, v[j], fmaf(-ub_uk.x, su[j], su[i]));
                    with_b = fmaf(rb_rk.x, su[j], with_b);
                    with_k = fmaf(rb_rk.y, v[j], with_k);
                }
                const float2 own = line[2 * i];
                sq[i] += fmaf(own.y, v[i], with_k) - fmaf(own.x, su[i], with_b);
            }
            const float4* dp = reinterpret_cast<const float4*>(base + kDecayAt);
            const float4 d0 = dp[sub], d1 = dp[L + sub];
            s[0] *= d0.x; s[1] *= d0.y; s[2] *= d0.z; s[3] *= d0.w;
            s[4] *= d1.x; s[5] *= d1.y; s[6] *= d1.z; s[7] *= d1.w;
#pragma unroll
            for (int i = 0; i < C; ++i) {
                const float4* kp = reinterpret_cast<const float4*>(base + (4 * i + 2) * kDimPad);
                const float4* bp = reinterpret_cast<const float4*>(base + (4 * i + 3) * kDimPad);
                const float4 k0 = kp[sub], k1 = kp[L + sub], b0 = bp[sub], b1 = bp[L + sub];
                const float vi = v[i], ni = -su[i];
                s[0] = fmaf(b0.x, ni, fmaf(k0.x, vi, s[0])); s[1] = fmaf(b0.y, ni, fmaf(k0.y, vi, s[1]));
                s[2] = fmaf(b0.z, ni, fmaf(k0.z, vi, s[2])); s[3] = fmaf(b0.w, ni, fmaf(k0.w, vi, s[3]));
                s[4] = fmaf(b1.x, ni, fmaf(k1.x, vi, s[4])); s[5] = fmaf(b1.y, ni, fmaf(k1.y, vi, s[5]));
                s[6] = fmaf(b1.z, ni, fmaf(k1.z, vi, s[6])); s[7] = fmaf(b1.w, ni, fmaf(k1.w, vi, s[7]));
            }
            float* out = p.out + (size_t)t0 * p.heads * p.dim + (size_t)head * p.dim + col;
            if (sub == 0 && col_ok) {
#pragma unroll
                for (int i = 0; i < C; ++i) out[(size_t)i * p.heads * p.dim] = sq[i];
            }
        } else {
            // the span's last tokens, fewer than a chunk: the same sums, a token at a time in registers by index
            float su[C];
#pragma unroll
            for (int i = 0; i < C; ++i) {
                if (i >= count) continue;
                const float* up = base + (4 * i) * kDimPad;
                const float* rp = up + kDimPad;
                float du = 0.0f, dq = 0.0f;
#pragma unroll
                for (int r = 0; r < kRegs; ++r) {
                    const int e = 4 * ((r >> 2) * L + sub) + (r & 3);
                    du = fmaf(s[r], up[e], du);
                    dq = fmaf(s[r], rp[e], dq);
                }
#pragma unroll
                for (int offset = 1; offset < L; offset <<= 1) {
                    du += __shfl_xor_sync(0xffffffffu, du, offset);
                    dq += __shfl_xor_sync(0xffffffffu, dq, offset);
                }
                const float* line = sums + 2 * i * i;
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    if (j >= i) continue;
                    const float vj = base[kValuesAt + j * kCols + col_in];
                    du = fmaf(line[4 * j + 1], vj, fmaf(-line[4 * j], su[j], du));
                    dq = fmaf(line[4 * j + 3], vj, fmaf(-line[4 * j + 2], su[j], dq));
                }
                su[i] = du;
                const float vi = base[kValuesAt + i * kCols + col_in];
                dq = fmaf(line[4 * i + 1], vi, fmaf(-line[4 * i], du, dq));
                if (sub == 0 && col_ok) p.out[(size_t)(t0 + i) * p.heads * p.dim + (size_t)head * p.dim + col] = dq;
            }
#pragma unroll
            for (int r = 0; r < kRegs; ++r) {
                const int e = 4 * ((r >> 2) * L + sub) + (r & 3);
                s[r] *= base[kDecayAt + e];
#pragma unroll
                for (int i = 0; i < C; ++i) {
                    if (i >= count) continue;
                    const float* kp = base + (4 * i + 2) * kDimPad;
                    s[r] = fmaf(kp[kDimPad + e], -su[i], fmaf(kp[e], base[kValuesAt + i * kCols + col_in], s[r]));
                }
            }
        }
        if (++stage == kStages) stage = 0;
    }
    cp_async_wait_group<0>();
#pragma unroll
    for (int r = 0; r < kRegs; ++r) {
        const int e = 4 * ((r >> 2) * L + sub) + (r & 3);
        if (col_ok && e < p.dim) s_head[(size_t)e * p.dim + col] = s[r];
    }
}

template <int L>
static int launch_delta_scan(const DeltaScanArgs& p, int spans, cudaStream_t stream) {
    constexpr int kCols = kDeltaWarps * (32 / L);
    constexpr int kStages = L >= 16 ? 2 : 3;
    constexpr size_t smem = (size_t)kStages * (kDeltaChunk * 4 * 8 * L + 8 * L + kDeltaSums + kDeltaChunk * kCols) * sizeof(float);
    auto kernel = delta_scan_kernel<L>;
    if (smem > 48 * 1024) {
        const cudaError_t status = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (status != cudaSuccess) {
            set_error("general_delta_scan: %s", cudaGetErrorString(status));
            return -2;
        }
    }
    dim3 grid((p.dim + kCols - 1) / kCols, p.heads, spans);
    // (a plain launch: few long blocks, see recurrent_scan.cu)
    kernel<<<grid, kDeltaWarps * 32, smem, stream>>>(p);
    return check_launch("general_delta_scan");
}

// ---------------------------------------------------------------------------------------------------------
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

template <typename A>
__global__ void __launch_bounds__(kDeltaDecodeThreads) delta_decode_kernel(const DeltaDecodeArgs p) {
    extern __shared__ __align__(16) float smem[];  // tanh [rank] | k r w b [4 dim] | o [dim] | partial sums [2 threads]
    __shared__ float scratch[4][8];
    constexpr int kThreads = kDeltaDecodeThreads, kWarps = kThreads / 32, kKeep = 32;
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
            for (int i = quarter; i < p.rank; i += 4) z = fmaf(to_float(up[i]), low_s[i], z);
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

// out[t, c] = act(x[t, c]) of float32 columns that lie in wider rows, rounded once
template <typename A>
__global__ void activation_cast_kernel(const float* x, long long stride, A* out, int tokens, int columns, int kind) {
    chain_release();
    chain_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * columns) return;
    const int t = (int)(i / columns), c = (int)(i % columns);
    out[i] = from_float<A>(activate(x[(size_t)t * stride + c], kind));
}

}  // namespace celeg_b200

using namespace celeg_b200;

CELEG_API int celeg_activation_cast(const float* x, long long stride, void* out, int tokens, int columns, int kind,
                                    int act_dtype, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && columns > 0 && stride >= columns && kind >= 0 && kind <= kTanh,
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

// The recurrence over the step's spans (two launches). Offsets: columns of r, k, v and the removal rate in a row of
// proj (float32, rows `stride` apart); z: float32 [tokens, heads * dim]. Scratch, with dim_pad = dim rounded up to a
// multiple of 4: vectors [tokens * heads * 4 * dim_pad], decay [tokens * heads * dim_pad], sums [heads * tokens * 16].
CELEG_API int celeg_general_delta_scan(const float* proj, int stride, int r_off, int k_off, int v_off, int a_off,
                                       const float* z, int z_stride, const float* w0, const float* a_bias, float unit_eps,
                                       const int* token_span, const int* span_begin, const int* span_slot, float* vectors,
                                       float* decay, float* sums, float* out, float* state, long long slot_stride, int tokens,
                                       int spans, int heads, int dim, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && spans >= 0 && heads > 0 && dim > 0 && dim <= kDeltaMaxDim && unit_eps > 0.0f,
                  "general_delta_scan: invalid sizes tokens=%d spans=%d heads=%d dim=%d (at most %d)", tokens, spans, heads, dim,
                  kDeltaMaxDim);
    CELEG_REQUIRE(spans <= 65535 && heads <= 65535, "general_delta_scan: %d spans or %d heads exceed one launch", spans, heads);
    CELEG_REQUIRE((((size_t)vectors | (size_t)decay | (size_t)sums) & 15) == 0, "general_delta_scan: scratch must be 16-byte aligned");
    if (tokens == 0 || spans == 0) return 0;
    const int dim_pad = (dim + 3) & ~3;
    const DeltaVectorsArgs first = {proj, stride, r_off, k_off, a_off, z, z_stride, w0, a_bias, token_span, span_begin, vectors,
                                    decay, sums, tokens, heads, dim, dim_pad, unit_eps};
    dim3 grid((tokens + kDeltaChunk - 1) / kDeltaChunk, (heads + kVectorsWarps - 1) / kVectorsWarps);
    launch_chained(delta_vectors_kernel, grid, kVectorsWarps * 32, 0, stream, first);
    const int status = check_launch("general_delta_vectors");
    if (status != 0) return status;
    const DeltaScanArgs p = {vectors, decay, sums, proj + v_off, stride, out, state, slot_stride, span_begin, span_slot, tokens,
                             heads, dim, dim_pad};
    if (dim <= 8) return launch_delta_scan<1>(p, spans, stream);
    if (dim <= 16) return launch_delta_scan<2>(p, spans, stream);
    if (dim <= 32) return launch_delta_scan<4>(p, spans, stream);
    if (dim <= 64) return launch_delta_scan<8>(p, spans, stream);
    if (dim <= 128) return launch_delta_scan<16>(p, spans, stream);
    return launch_delta_scan<32>(p, spans, stream);
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
    if (act_dtype == kFloat32)
        launch_chained(delta_decode_kernel<float>, grid, kDeltaDecodeThreads, smem, stream, args);
    else
        launch_chained(delta_decode_kernel<__nv_bfloat16>, grid, kDeltaDecodeThreads, smem, stream, args);
    return check_launch("general_delta_decode");
}
