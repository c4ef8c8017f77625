// A residual of several float32 streams, and the kernels around it.
//
//   hyper_norm       x'_t = sum_s mix[s, t] x_s + out[t] y      all streams at once from the old ones
//                    u    = sum_t in[t] x'_t                    (in null: the sum of the streams)
//                    v    = round_T((u - mean(u)) / sqrt(mean((u - mean(u))^2) + eps) * w + b)
//                    The write behind a sublayer and the norm in front of the next in one pass over a row, one
//                    block a row.  Without y nothing is written and u is read from the streams as they are.
//                    The streams may still all equal one row [width] (the embedding): `spread`.  With `gather`
//                    only the named rows of v are produced and the streams are not written.
//   normed_pair_sum  y = factor * (l / rms(l) * w_l + r / rms(r) * w_r), l and r with optional biases, float32
//
// hyper_norm takes y either as one row or as such a pair (two sublayers side by side, each normed by itself).
// Everything is float32 with one rounding, when v is stored; the order of additions inside a row depends on the
// sizes alone, so a row's result does not depend on the batch it is in.
#include "common.cuh"

#define HYPER_MAX_STREAMS 32
#define HYPER_MAX_THREADS 512

// A pair of rows that is still to be normed and added up, or one row (right null, weights null).
struct HyperUpdate {
    const void* left;
    const void* right;
    const float* left_weight;
    const float* right_weight;
    const float* left_bias;
    const float* right_bias;
    float eps, factor;
};

// Sums of two values over the block at once (as block_sum).
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int warps = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    const float2 mine = lane < warps ? scratch[lane] : make_float2(0.0f, 0.0f);
    return make_float2(warp_sum(mine.x), warp_sum(mine.y));
}

__device__ __forceinline__ float inverse_rms(float squares, int width, float eps) {
    return __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(squares, (float)width), eps)));
}

// The pair's two rows, biases added, into shared memory (a thread reads back only what it wrote), and the two
// inverse root mean squares.
template <typename Y, int VEC>
__device__ __forceinline__ float2 load_pair_rows(const HyperUpdate& u, int64_t row, int width, float* left_s,
                                                 float* right_s, float2* scratch) {
    const Y* lr = (const Y*)u.left + row * width;
    const Y* rr = (const Y*)u.right + row * width;
    float pl = 0.0f, pr = 0.0f;
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float l[VEC], r[VEC], b[VEC];
        load_values<VEC>(lr + i, l);
        load_values<VEC>(rr + i, r);
        if (u.left_bias) {
            load_values<VEC>(u.left_bias + i, b);
#pragma unroll
            for (int j = 0; j < VEC; ++j) l[j] = __fadd_rn(l[j], b[j]);
        }
        if (u.right_bias) {
            load_values<VEC>(u.right_bias + i, b);
#pragma unroll
            for (int j = 0; j < VEC; ++j) r[j] = __fadd_rn(r[j], b[j]);
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            pl = __fmaf_rn(l[j], l[j], pl);
            pr = __fmaf_rn(r[j], r[j], pr);
        }
        store_values<VEC>(left_s + i, l);
        store_values<VEC>(right_s + i, r);
    }
    const float2 squares = block_sum2(pl, pr, scratch);
    return make_float2(inverse_rms(squares.x, width, u.eps), inverse_rms(squares.y, width, u.eps));
}

template <int VEC>
__device__ __forceinline__ void pair_values(const HyperUpdate& u, int i, const float* left_s, const float* right_s,
                                            float2 inverse, float* y) {
    float l[VEC], r[VEC], wl[VEC], wr[VEC];
    load_values<VEC>(left_s + i, l);
    load_values<VEC>(right_s + i, r);
    load_values<VEC>(u.left_weight + i, wl);
    load_values<VEC>(u.right_weight + i, wr);
#pragma unroll
    for (int j = 0; j < VEC; ++j)
        y[j] = __fmul_rn(u.factor, __fadd_rn(__fmul_rn(__fmul_rn(l[j], inverse.x), wl[j]),
                                             __fmul_rn(__fmul_rn(r[j], inverse.y), wr[j])));
}

// STREAMS: the number of streams (compiled for the usual ones), or 0: `streams` of them, up to HYPER_MAX_STREAMS
template <typename Y, typename T, int VEC, int STREAMS>
__global__ void __launch_bounds__(HYPER_MAX_THREADS) hyper_norm_kernel(const float* stream_in, int spread, HyperUpdate update, const float* __restrict__ mix,
                                  const float* __restrict__ w_out, const float* __restrict__ w_in,
                                  const float* __restrict__ weight, const float* __restrict__ bias,
                                  T* __restrict__ out, float* stream_out, const int* __restrict__ gather, int streams,
                                  int width, float eps) {
    constexpr int MOST = STREAMS > 0 ? STREAMS : HYPER_MAX_STREAMS, UNROLL = STREAMS > 0 ? STREAMS : 1;
    extern __shared__ __align__(16) float row_values[];     // [width] u, then for a pair [width] left, [width] right
    __shared__ float scratch[32];
    __shared__ float2 scratch2[32];
    __shared__ float mix_s[MOST * MOST], out_s[MOST], in_s[MOST];
    const int count = STREAMS > 0 ? STREAMS : streams;
    for (int i = threadIdx.x; i < count * count; i += blockDim.x) mix_s[i] = mix ? mix[i] : 0.0f;
    for (int i = threadIdx.x; i < count; i += blockDim.x) {
        out_s[i] = w_out ? w_out[i] : 0.0f;
        in_s[i] = w_in ? w_in[i] : 1.0f;
    }
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    const int out_row = blockIdx.x;
    const int64_t row = gather ? gather[out_row] : out_row;
    const float* sr = stream_in + row * width * (spread ? 1 : count);
    float* dst = stream_out + (int64_t)out_row * width * count;
    const bool writes = update.left != nullptr;
    const bool pair = update.right != nullptr;
    float* left_s = row_values + width;
    float* right_s = left_s + width;
    float2 inverse = make_float2(1.0f, 1.0f);
    if (pair) inverse = load_pair_rows<Y, VEC>(update, row, width, left_s, right_s, scratch2);
    float part = 0.0f;
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float x[MOST][VEC], y[VEC], u[VEC];
#pragma unroll(UNROLL)
        for (int s = 0; s < (STREAMS > 0 ? STREAMS : count); ++s) {
            if (spread && s > 0) {
#pragma unroll
                for (int j = 0; j < VEC; ++j) x[s][j] = x[0][j];
            } else load_values<VEC>(sr + (int64_t)s * width + i, x[s]);
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = 0.0f;
        if (writes) {
            if (pair) pair_values<VEC>(update, i, left_s, right_s, inverse, y);
            else load_values<VEC>((const Y*)update.left + row * width + i, y);
#pragma unroll(UNROLL)
            for (int t = 0; t < (STREAMS > 0 ? STREAMS : count); ++t) {
                float next[VEC];
#pragma unroll
                for (int j = 0; j < VEC; ++j) next[j] = __fmul_rn(mix_s[t], x[0][j]);
#pragma unroll(UNROLL)
                for (int s = 1; s < (STREAMS > 0 ? STREAMS : count); ++s) {
                    const float m = mix_s[s * count + t];
#pragma unroll
                    for (int j = 0; j < VEC; ++j) next[j] = __fmaf_rn(m, x[s][j], next[j]);
                }
                const float share = out_s[t], read = in_s[t];
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    next[j] = __fmaf_rn(share, y[j], next[j]);
                    u[j] = __fmaf_rn(read, next[j], u[j]);
                }
                if (!gather) store_values<VEC>(dst + (int64_t)t * width + i, next);
            }
        } else {
#pragma unroll(UNROLL)
            for (int s = 0; s < (STREAMS > 0 ? STREAMS : count); ++s) {
#pragma unroll
                for (int j = 0; j < VEC; ++j) u[j] = __fmaf_rn(in_s[s], x[s][j], u[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) part = __fadd_rn(part, u[j]);
        store_values<VEC>(row_values + i, u);
    }
    const float mean = __fdiv_rn(block_sum(part, scratch), (float)width);
    part = 0.0f;
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float u[VEC];
        load_values<VEC>(row_values + i, u);
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            u[j] = __fsub_rn(u[j], mean);
            part = __fmaf_rn(u[j], u[j], part);
        }
        store_values<VEC>(row_values + i, u);
    }
    const float factor = inverse_rms(block_sum(part, scratch), width, eps);
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float u[VEC], w[VEC], b[VEC];
        load_values<VEC>(row_values + i, u);
        load_values<VEC>(weight + i, w);
        load_values<VEC>(bias + i, b);
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = __fmaf_rn(__fmul_rn(u[j], factor), w[j], b[j]);
        store_values<VEC>(out + (int64_t)out_row * width + i, u);
    }
}

static inline bool aligned_to(const void* p, size_t bytes) { return (uintptr_t)p % bytes == 0; }

// stream_in: float32 [rows, streams, width], or [rows, width] with `spread`; y (left) and, for a pair, right of
// y_dtype [rows, width]; mix [streams, streams] (from, to), w_out and w_in [streams], weight, bias and the pair's
// weights and biases [width], all float32; out [rows, width] of `dtype`; stream_out float32 [rows, streams, width]
// (may be stream_in unless `spread`).  left null: nothing is written (mix, w_out unused).
extern "C" int tvb_hyper_norm(const float* stream_in, int spread, const void* left, const void* right, int y_dtype,
                              const float* left_weight, const float* right_weight, const float* left_bias,
                              const float* right_bias, float pair_eps, float pair_factor, const float* mix,
                              const float* w_out, const float* w_in, const float* weight, const float* bias, void* out,
                              int dtype, float* stream_out, const int* gather, int rows, int streams, int width,
                              float eps, int pdl, void* stream) {
    if (rows <= 0) return 0;
    if (width <= 0 || streams <= 0 || streams > HYPER_MAX_STREAMS || !stream_in || !weight || !bias || !out ||
        (left && (!mix || !w_out || (!gather && !stream_out))) || (right && (!left || !left_weight || !right_weight)) ||
        (left && !gather && spread && stream_out == stream_in))
        return TVB_BAD_ARGUMENT;
    const size_t smem = (size_t)width * sizeof(float) * (right ? 3 : 1);
    if (smem > 200 * 1024) return TVB_BAD_ARGUMENT;
    const size_t y_size = y_dtype == TVB_BF16 ? 2 : 4, t_size = dtype == TVB_BF16 ? 2 : 4;
    const bool by_four = width % 4 == 0 && aligned_to(stream_in, 16) && aligned_to(stream_out, 16) &&
                         aligned_to(left, 4 * y_size) && aligned_to(right, 4 * y_size) && aligned_to(left_weight, 16) &&
                         aligned_to(right_weight, 16) && aligned_to(left_bias, 16) && aligned_to(right_bias, 16) &&
                         aligned_to(weight, 16) && aligned_to(bias, 16) && aligned_to(out, 4 * t_size);
    const int per = by_four ? width / 4 : width;
    const int threads = per >= 1024 ? HYPER_MAX_THREADS : (per >= 256 ? 256 : (per >= 128 ? 128 : (per >= 64 ? 64 : 32)));
    cudaStream_t s = (cudaStream_t)stream;
    HyperUpdate update{left, right, left_weight, right_weight, left_bias, right_bias, pair_eps, pair_factor};
    auto go = [&](auto kernel, auto* typed_out) -> int {
        if (smem > 40 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        TvbLaunch launch(dim3(rows), dim3(threads), smem, s, pdl);
        cudaError_t e = cudaLaunchKernelEx(&launch.config, kernel, stream_in, spread, update, mix, w_out, w_in, weight,
                                           bias, typed_out, stream_out, gather, streams, width, eps);
        return e == cudaSuccess ? tvb_last_error() : (int)e;
    };
#define BY_STREAMS(Y, T, VEC)                                                             \
    switch (streams) {                                                                    \
        case 1: return go(hyper_norm_kernel<Y, T, VEC, 1>, (T*)out);                      \
        case 2: return go(hyper_norm_kernel<Y, T, VEC, 2>, (T*)out);                      \
        case 3: return go(hyper_norm_kernel<Y, T, VEC, 3>, (T*)out);                      \
        case 4: return go(hyper_norm_kernel<Y, T, VEC, 4>, (T*)out);                      \
        case 8: return go(hyper_norm_kernel<Y, T, VEC, 8>, (T*)out);                      \
        default: return go(hyper_norm_kernel<Y, T, 1, 0>, (T*)out);                       \
    }
    if (dtype == TVB_F32 && y_dtype == TVB_F32) { if (by_four) { BY_STREAMS(float, float, 4) } else { BY_STREAMS(float, float, 1) } }
    if (dtype == TVB_BF16 && y_dtype == TVB_F32) { if (by_four) { BY_STREAMS(float, bf16, 4) } else { BY_STREAMS(float, bf16, 1) } }
    if (dtype == TVB_BF16 && y_dtype == TVB_BF16) { if (by_four) { BY_STREAMS(bf16, bf16, 4) } else { BY_STREAMS(bf16, bf16, 1) } }
#undef BY_STREAMS
    return TVB_BAD_ARGUMENT;
}

template <typename Y, int VEC>
__global__ void normed_pair_sum_kernel(HyperUpdate update, float* __restrict__ out, int width) {
    extern __shared__ __align__(16) float row_values[];
    __shared__ float2 scratch2[32];
    const int64_t row = blockIdx.x;
    const float2 inverse = load_pair_rows<Y, VEC>(update, row, width, row_values, row_values + width, scratch2);
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float y[VEC];
        pair_values<VEC>(update, i, row_values, row_values + width, inverse, y);
        store_values<VEC>(out + row * width + i, y);
    }
}

extern "C" int tvb_normed_pair_sum(const void* left, const void* right, int y_dtype, const float* left_weight,
                                   const float* right_weight, const float* left_bias, const float* right_bias,
                                   float eps, float factor, float* out, int rows, int width, void* stream) {
    if (rows <= 0) return 0;
    if (width <= 0 || !left || !right || !left_weight || !right_weight || !out) return TVB_BAD_ARGUMENT;
    const size_t smem = (size_t)width * sizeof(float) * 2;
    if (smem > 200 * 1024) return TVB_BAD_ARGUMENT;
    const size_t y_size = y_dtype == TVB_BF16 ? 2 : 4;
    const bool by_four = width % 4 == 0 && aligned_to(left, 4 * y_size) && aligned_to(right, 4 * y_size) &&
                         aligned_to(left_weight, 16) && aligned_to(right_weight, 16) && aligned_to(left_bias, 16) &&
                         aligned_to(right_bias, 16) && aligned_to(out, 16);
    const int per = by_four ? width / 4 : width;
    const int threads = per >= 256 ? 256 : (per >= 128 ? 128 : (per >= 64 ? 64 : 32));
    HyperUpdate update{left, right, left_weight, right_weight, left_bias, right_bias, eps, factor};
    auto go = [&](auto kernel) -> int {
        if (smem > 40 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        kernel<<<rows, threads, smem, (cudaStream_t)stream>>>(update, out, width);
        return tvb_last_error();
    };
    if (y_dtype == TVB_F32) return by_four ? go(normed_pair_sum_kernel<float, 4>) : go(normed_pair_sum_kernel<float, 1>);
    if (y_dtype == TVB_BF16) return by_four ? go(normed_pair_sum_kernel<bf16, 4>) : go(normed_pair_sum_kernel<bf16, 1>);
    return TVB_BAD_ARGUMENT;
}

// y[row] += bias, in place: y of `dtype` [rows, width], bias float32 [width]
template <typename T>
__global__ void add_row_bias_kernel(T* y, const float* __restrict__ bias, int width, int64_t count) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < count) y[i] = from_float<T>(__fadd_rn(to_float<T>(y[i]), bias[i % width]));
}

extern "C" int tvb_add_row_bias(void* y, const float* bias, int rows, int width, int dtype, void* stream) {
    if (rows <= 0) return 0;
    if (width <= 0 || !y || !bias) return TVB_BAD_ARGUMENT;
    const int64_t count = (int64_t)rows * width, blocks = (count + 255) / 256;
    if (blocks > 2147483647LL) return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == TVB_F32) add_row_bias_kernel<float><<<(unsigned)blocks, 256, 0, s>>>((float*)y, bias, width, count);
    else if (dtype == TVB_BF16) add_row_bias_kernel<bf16><<<(unsigned)blocks, 256, 0, s>>>((bf16*)y, bias, width, count);
    else return TVB_BAD_ARGUMENT;
    return tvb_last_error();
}
