// Short causal convolutions over time, one per channel: y[t, c] = act(sum_j w[c, j] u[t - taps + 1 + j, c] + b[c]), the last
// tap for the token itself. Inputs before a span's first token in the step are the request's carried ones (zeros at a
// sequence's start); after the step the last taps - 1 inputs of every request are carried on. Float32 throughout.
//
// A thread takes a few neighbouring channels of a few tokens in a row and keeps the last taps - 1 inputs in registers, so
// an input is read once (plus the overlap at the tile's start). When every span is one token (decoding) the same threads
// move the carried inputs on; otherwise that is a second launch, because other tiles still read them.
#include "common.cuh"

namespace celeg_b200 {

constexpr int kConvTile = 4;          // tokens a thread walks (portions; a decoded token has a thread of its own)

struct ChannelConvArgs {
    const float* in; int in_stride;
    const float* w;                   // [channels, taps]
    const float* bias;                // [channels] or null
    float* carried;                   // this part's carried inputs inside slot 0: [taps - 1, channels], oldest first
    long long slot_stride;
    const int* token_span; const int* span_begin; const int* span_slot;
    float* out; int out_stride;
    int tokens, channels, taps, act, single;          // act: a code of activate() or -1; single: every span is one token
};

template <int V> struct ConvPack { float v[V]; };
template <int V> __device__ __forceinline__ ConvPack<V> conv_load(const float* p) {
    ConvPack<V> r;
    if (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1 % V] = x.y; r.v[2 % V] = x.z; r.v[3 % V] = x.w;
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) r.v[i] = p[i];
    }
    return r;
}
template <int V> __device__ __forceinline__ void conv_store(float* p, const ConvPack<V>& x) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x.v[0], x.v[1 % V], x.v[2 % V], x.v[3 % V]);
    else {
#pragma unroll
        for (int i = 0; i < V; ++i) p[i] = x.v[i];
    }
}

// V neighbouring channels a thread, TAPS taps (a template for up to four; 16: any number up to that)
template <int V, int TAPS, int TILE>
__global__ void __launch_bounds__(128) channel_conv_kernel(const ChannelConvArgs a) {
    const int taps = TAPS <= 4 ? TAPS : a.taps;
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const int t0 = blockIdx.y * (TAPS <= 4 ? TILE : 1);
    const int t1 = min(t0 + (TAPS <= 4 ? TILE : 1), a.tokens);
    chain_release();
    chain_wait();
    if (c >= a.channels) return;
    float w[TAPS <= 4 ? TAPS : 1][V];
    if constexpr (TAPS <= 4) {
#pragma unroll
        for (int i = 0; i < V; ++i)
            if (TAPS == 4) {
                const float4 x = __ldg(reinterpret_cast<const float4*>(a.w) + c + i);
                w[0][i] = x.x; w[1 % TAPS][i] = x.y; w[2 % TAPS][i] = x.z; w[3 % TAPS][i] = x.w;
            } else {
#pragma unroll
                for (int j = 0; j < TAPS; ++j) w[j][i] = __ldg(a.w + (size_t)(c + i) * TAPS + j);
            }
    }
    ConvPack<V> bias;
#pragma unroll
    for (int i = 0; i < V; ++i) bias.v[i] = a.bias ? __ldg(a.bias + c + i) : 0.0f;
    auto finish = [&](int t, ConvPack<V> sum) {
        if (a.act >= 0) {
#pragma unroll
            for (int i = 0; i < V; ++i) sum.v[i] = activate(sum.v[i], a.act);
        }
        conv_store<V>(a.out + (size_t)t * a.out_stride + c, sum);
    };
    if constexpr (TAPS <= 4) {
        constexpr int kKeep = TAPS > 1 ? TAPS - 1 : 1;
        ConvPack<V> history[kKeep];
        ConvPack<V> ahead[TILE];
#pragma unroll
        for (int i = 0; i < TILE; ++i)
            if (t0 + i < t1) ahead[i] = conv_load<V>(a.in + (size_t)(t0 + i) * a.in_stride + c);
        int span = -1;
        const int last_span = TAPS > 1 ? a.token_span[t1 - 1] : 0;
#pragma unroll
        for (int i = 0; i < TILE; ++i) {
            const int t = t0 + i;
            if (t >= t1) continue;
            // the tile's first token, or a span that begins here (only where the tile's last token is of a later span)
            if (TAPS > 1 && (i == 0 || (span != last_span && a.token_span[t] != span))) {
                span = a.token_span[t];
                const int begin = a.span_begin[span];
                const float* carried = a.carried + (long long)a.span_slot[span] * a.slot_stride;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const int s = t - begin - (TAPS - 1) + j;
                    history[j] = conv_load<V>(s >= 0 ? a.in + (size_t)(begin + s) * a.in_stride + c
                                                     : carried + (size_t)(TAPS - 1 + s) * a.channels + c);
                }
            }
            ConvPack<V> sum;
#pragma unroll
            for (int k = 0; k < V; ++k) {
                float v = 0.0f;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) v = fmaf(w[j][k], history[j].v[k], v);
                sum.v[k] = fmaf(w[TAPS - 1][k], ahead[i].v[k], v) + bias.v[k];
            }
#pragma unroll
            for (int j = 0; j + 1 < kKeep; ++j) history[j] = history[j + 1];
            if (TAPS > 1) history[kKeep - 1] = ahead[i];
            if (a.single && TAPS > 1) {
                float* carried = a.carried + (long long)a.span_slot[span] * a.slot_stride;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) conv_store<V>(carried + (size_t)j * a.channels + c, history[j]);
            }
            finish(t, sum);
        }
    } else for (int t = t0; t < t1; ++t) {
        const int span = a.token_span[t], begin = a.span_begin[span];
        float* carried = a.carried + (long long)a.span_slot[span] * a.slot_stride;
        ConvPack<V> sum;
#pragma unroll
        for (int i = 0; i < V; ++i) sum.v[i] = 0.0f;
        for (int j = 0; j < taps; ++j) {
            const int s = t - begin - (taps - 1) + j;
            const ConvPack<V> x = conv_load<V>(s >= 0 ? a.in + (size_t)(begin + s) * a.in_stride + c
                                                      : carried + (size_t)(taps - 1 + s) * a.channels + c);
#pragma unroll
            for (int i = 0; i < V; ++i) sum.v[i] = fmaf(a.w[(size_t)(c + i) * taps + j], x.v[i], sum.v[i]);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) sum.v[i] += bias.v[i];
        if (a.single) {
            for (int j = 0; j + 1 < taps - 1; ++j)
                conv_store<V>(carried + (size_t)j * a.channels + c, conv_load<V>(carried + (size_t)(j + 1) * a.channels + c));
            conv_store<V>(carried + (size_t)(taps - 2) * a.channels + c, conv_load<V>(a.in + (size_t)t * a.in_stride + c));
        }
        finish(t, sum);
    }
}

// The carried inputs after a step with longer spans: one thread per (span, channel) reads all it needs before it writes.
__global__ void channel_conv_carry_kernel(const ChannelConvArgs a, int spans) {
    chain_release();
    chain_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= spans * a.channels) return;
    const int span = i / a.channels, c = i % a.channels;
    const int begin = a.span_begin[span], length = a.span_begin[span + 1] - begin;
    if (length <= 0) return;
    float* mine = a.carried + (long long)a.span_slot[span] * a.slot_stride;
    float keep[15];
#pragma unroll
    for (int r = 0; r < 15; ++r) {
        if (r < a.taps - 1) {
            const int s = length - (a.taps - 1) + r;
            keep[r] = s >= 0 ? a.in[(size_t)(begin + s) * a.in_stride + c] : mine[(size_t)(a.taps - 1 + s) * a.channels + c];
        }
    }
#pragma unroll
    for (int r = 0; r < 15; ++r)
        if (r < a.taps - 1) mine[(size_t)r * a.channels + c] = keep[r];
}

template <int V, int TILE>
static void launch_conv(const ChannelConvArgs& a, cudaStream_t stream) {
    const int tile = a.taps <= 4 ? TILE : 1;
    const int units = a.channels / V;
    dim3 grid((units + 127) / 128, (a.tokens + tile - 1) / tile);
    switch (a.taps) {
        case 1: launch_chained(channel_conv_kernel<V, 1, TILE>, grid, 128, 0, stream, a); break;
        case 2: launch_chained(channel_conv_kernel<V, 2, TILE>, grid, 128, 0, stream, a); break;
        case 3: launch_chained(channel_conv_kernel<V, 3, TILE>, grid, 128, 0, stream, a); break;
        case 4: launch_chained(channel_conv_kernel<V, 4, TILE>, grid, 128, 0, stream, a); break;
        default: launch_chained(channel_conv_kernel<V, 16, TILE>, grid, 128, 0, stream, a);
    }
}

}  // namespace celeg_b200

using namespace celeg_b200;

// in: float32 rows `in_stride` apart, the convolved channels first; out: rows `out_stride` apart. act: a code of activate()
// or -1. single: every span brings exactly one token (then spans = tokens).
CELEG_API int celeg_channel_conv(const float* in, int in_stride, const float* w, const float* bias, float* carried,
                                 long long slot_stride, const int* token_span, const int* span_begin, const int* span_slot,
                                 float* out, int out_stride, int tokens, int spans, int channels, int taps, int act,
                                 int single, cudaStream_t stream) {
    CELEG_REQUIRE(tokens >= 0 && spans >= 0 && channels > 0 && taps >= 1 && taps <= 16 && in_stride >= channels &&
                  out_stride >= channels && act >= -1 && act <= kTanh && (taps == 1 || carried) && ((size_t)w & 15) == 0,
                  "channel_conv: invalid sizes tokens=%d channels=%d taps=%d strides %d / %d act=%d", tokens, channels, taps,
                  in_stride, out_stride, act);
    CELEG_REQUIRE(tokens <= 65535, "channel_conv: %d tokens exceed one launch", tokens);
    if (tokens == 0) return 0;
    const ChannelConvArgs a = {in, in_stride, w, bias, carried, slot_stride, token_span, span_begin, span_slot, out, out_stride,
                               tokens, channels, taps, act, single};
    if (((channels | in_stride | out_stride) & 3) == 0 && (slot_stride & 3) == 0 &&
        (((size_t)in | (size_t)out | (size_t)carried) & 15) == 0) single ? launch_conv<4, 1>(a, stream) : launch_conv<4, kConvTile>(a, stream);
    else single ? launch_conv<1, 1>(a, stream) : launch_conv<1, kConvTile>(a, stream);
    const int status = check_launch("channel_conv");
    if (status != 0 || single || taps == 1) return status;
    const long long units = (long long)spans * channels;
    launch_chained(channel_conv_carry_kernel, (unsigned)((units + 127) / 128), 128, 0, stream, a, spans);
    return check_launch("channel_conv_carry");
}
