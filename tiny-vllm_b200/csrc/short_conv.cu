// A causal convolution over few tokens, one channel at a time, with an activation behind it:
//
//   y[t, c] = act(bias[c] + sum_j taps[j, c] * x[t - (K - 1) + j, c])        act none or SiLU
//
// With `in_bias` the inputs are x + in_bias (the zeros before a request's start stay zeros).
//
// The inputs before a step's first token are the request's last K - 1 ones, kept in a float32 state
// [slots, K - 1, channels] (oldest first, zero when a request starts), which is left as the last K - 1
// inputs of the entry.  K is 2, 4, 8, 16 or 32; fewer taps are padded with zeros in front (the older ones).
// Sums are float32 whatever the storage type of x and y.
//
// A thread walks VEC neighbouring channels through a piece of an entry with the last K - 1 inputs in registers.
// The thread of an entry's first piece is the only one that reads the state and the one that writes it.
#include "common.cuh"

#define CONV_THREADS 128
// tokens a piece, at least K - 1: short ones, whose loads are all in flight together, read the few inputs ahead of
// them once more
template <int K> constexpr int CONV_PIECE = K <= 8 ? 8 : 32;

template <typename T, int K, int VEC>
__global__ void __launch_bounds__(CONV_THREADS) short_conv_kernel(
    const T* __restrict__ x, int64_t x_stride, const float* __restrict__ taps, const float* __restrict__ bias,
    const float* __restrict__ in_bias, int act, float* state, const int* __restrict__ row_starts, const int* __restrict__ state_slots,
    const int* __restrict__ token_row, T* __restrict__ out, int64_t out_stride, int rows, int channels) {
    const int c = (blockIdx.x * CONV_THREADS + threadIdx.x) * VEC;
    constexpr int PIECE = CONV_PIECE<K>;
    int row, before = 0, tokens = 0;
    for (row = 0; row < rows; ++row) {
        tokens = row_starts[row + 1] - row_starts[row];
        const int pieces = (tokens + PIECE - 1) / PIECE;
        if ((int)blockIdx.y < before + pieces) break;
        before += pieces;
    }
    if (row == rows || c >= channels) return;     // the grid is as large as the pieces can be many
    const int piece = blockIdx.y - before;
    const int begin = row_starts[row], i0 = piece * PIECE;
    const int count = min(PIECE, tokens - i0);
    T* dst = out + (int64_t)(begin + i0) * out_stride + c;
    if (token_row[begin] < 0) {                   // a padding row of a recorded batch: no request, no state
        float zero[VEC] = {};
        for (int t = 0; t < count; ++t) store_values<VEC>(dst + (int64_t)t * out_stride, zero);
        return;
    }
    const T* src = x + (int64_t)begin * x_stride + c;
    float* mine = state + (int64_t)state_slots[row] * (K - 1) * channels + c;
    float w[K][VEC], b[VEC] = {}, shift[VEC] = {}, last[K - 1][VEC];
    auto input = [&](const T* p, float* v) {
        load_values<VEC>(p, v);
        if (in_bias) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] = __fadd_rn(v[i], shift[i]);
        }
    };
#pragma unroll
    for (int j = 0; j < K; ++j) load_values<VEC>(taps + (int64_t)j * channels + c, w[j]);
    if (bias) load_values<VEC>(bias + c, b);
    if (in_bias) load_values<VEC>(in_bias + c, shift);
#pragma unroll
    for (int j = 0; j < K - 1; ++j) {
        const int i = i0 - (K - 1) + j;           // before the entry's first token only in its first piece
        if (i < 0) load_values<VEC>(mine + (int64_t)(K - 1 + i) * channels, last[j]);
        else input(src + (int64_t)i * x_stride, last[j]);
    }
    if (piece == 0) {
#pragma unroll
        for (int j = 0; j < K - 1; ++j) {         // in ascending order: an older place takes what a newer one held
            const int i = tokens - (K - 1) + j;
            float v[VEC];
            if (i < 0) load_values<VEC>(mine + (int64_t)(K - 1 + i) * channels, v);
            else input(src + (int64_t)i * x_stride, v);
            store_values<VEC>(mine + (int64_t)j * channels, v);
        }
    }
    src += (int64_t)i0 * x_stride;
    for (int t0 = 0; t0 < count; t0 += 8) {       // eight tokens' loads are in flight together
        float now[8][VEC];
#pragma unroll
        for (int t = 0; t < 8; ++t)
            if (t0 + t < count) input(src + (int64_t)(t0 + t) * x_stride, now[t]);
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            if (t0 + t >= count) break;
            float y[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                float sum = b[v];
#pragma unroll
                for (int j = 0; j < K - 1; ++j) sum = __fmaf_rn(w[j][v], last[j][v], sum);
                sum = __fmaf_rn(w[K - 1][v], now[t][v], sum);
                y[v] = act ? silu_for<T>(sum) : sum;
            }
#pragma unroll
            for (int j = 0; j + 1 < K - 1; ++j)
#pragma unroll
                for (int v = 0; v < VEC; ++v) last[j][v] = last[j + 1][v];
#pragma unroll
            for (int v = 0; v < VEC; ++v) last[K - 2][v] = now[t][v];
            store_values<VEC>(dst + (int64_t)(t0 + t) * out_stride, y);
        }
    }
}

// x: the first channel of the first token, rows `x_stride` elements apart; taps float32 [taps_count, channels];
// bias and in_bias float32 [channels] or null; act 0 none, 1 SiLU; `tokens`: of all entries.
extern "C" int tvb_short_conv(const void* x, long long x_stride, const float* taps, int taps_count, const float* bias,
                              const float* in_bias, int act, float* state, const int* row_starts, const int* state_slots,
                              const int* token_row, void* out, long long out_stride, int rows, int tokens, int channels,
                              int dtype, void* stream) {
    if (rows <= 0 || tokens <= 0) return 0;
    if (channels <= 0 || act < 0 || act > 1 || !state || !taps) return TVB_BAD_ARGUMENT;
    const size_t element = dtype == TVB_BF16 ? 2 : 4;
    const bool by_four = taps_count <= 8 && channels % 4 == 0 && x_stride % 4 == 0 && out_stride % 4 == 0 &&
                         (uintptr_t)x % (4 * element) == 0 && (uintptr_t)out % (4 * element) == 0 &&
                         (uintptr_t)taps % 16 == 0 && (uintptr_t)bias % 16 == 0 && (uintptr_t)in_bias % 16 == 0 &&
                         (uintptr_t)state % 16 == 0;
    const int per = CONV_THREADS * (by_four ? 4 : 1);
    const long long pieces = tokens / (taps_count <= 8 ? 8 : 32) + (long long)rows;        // at least those of all entries
    if (pieces > 65535) return TVB_BAD_ARGUMENT;
    const dim3 grid((channels + per - 1) / per, (unsigned)pieces);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, K, VEC) short_conv_kernel<T, K, VEC><<<grid, CONV_THREADS, 0, s>>>(                                     \
        (const T*)x, x_stride, taps, bias, in_bias, act, state, row_starts, state_slots, token_row, (T*)out, out_stride, rows, channels)
#define BY_TAPS(T)                                                                                                     \
    switch (taps_count) {                                                                                              \
        case 2: if (by_four) GO(T, 2, 4); else GO(T, 2, 1); break;                                                     \
        case 4: if (by_four) GO(T, 4, 4); else GO(T, 4, 1); break;                                                     \
        case 8: if (by_four) GO(T, 8, 4); else GO(T, 8, 1); break;                                                     \
        case 16: GO(T, 16, 1); break;                                                                                  \
        case 32: GO(T, 32, 1); break;                                                                                  \
        default: return TVB_BAD_ARGUMENT;                                                                              \
    }
    if (dtype == TVB_F32) { BY_TAPS(float) }
    else if (dtype == TVB_BF16) { BY_TAPS(bf16) }
    else return TVB_BAD_ARGUMENT;
#undef BY_TAPS
#undef GO
    return tvb_last_error();
}
