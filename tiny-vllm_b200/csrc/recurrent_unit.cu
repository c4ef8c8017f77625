// A linear recurrent unit with gates: a float32 state of one number a channel and request.
//
//   r = sigmoid(pre_r + b_r), i = sigmoid(pre_i + b_i)        pre: products of square matrices with parts of u
//   log a = c * r                                             c <= 0, one number a channel
//   S <- a S + sqrt(1 - a^2) i u,    out = S act(y + b_y)     act: the tanh form of GELU, SiLU or none
//
//   recurrent_unit_scan   prompts: a cluster of CTAs walks one entry for 32 channels, a block of UNIT_BLOCK tokens a CTA
//                         at a time: the CTAs' warps take UNIT_RUN tokens each, side by side, leave what their tokens
//                         make of a state of zero and the product of their decays, and walk their tokens again from the
//                         state these give them (the CTAs read one another's sums from shared memory)
//   recurrent_unit_step   one token a request: with `w` the gates' products are done here too (a CTA a block of gate
//                         channels, whose weights are read once for all its requests), else the gates come as `pre`
//
// Gates, decays, state and sums are float32 whatever the storage type of u, y and out.
#include "common.cuh"

#define UNIT_WARPS 8
#define UNIT_RUN 8
#define UNIT_BLOCK (UNIT_WARPS * UNIT_RUN)
#define UNIT_MOST_CTAS 8          // of a cluster
#define UNIT_ACT_NONE 0
#define UNIT_ACT_SILU 1
#define UNIT_ACT_GELU_TANH 2
#define UNIT_LOG2E 1.4426950408889634f

// The unit's float32 functions.  With 16-bit storage they take the special-function unit's 2^x, 1 / x and root (a few
// units in the last place, far below the rounding of what goes in).  Both the decay a = 1 + e and what is written,
// sqrt(1 - a^2) = sqrt(-e (2 + e)), come from e = exp(x) - 1, x <= 0: a channel that keeps hundreds of tokens multiplies
// a hundreds of times, and an exponential that is one unit off to one side there would show.
template <typename T> struct Unit;
template <> struct Unit<float> {
    static __device__ __forceinline__ float sigmoid(float z) { return __fdiv_rn(1.0f, __fadd_rn(1.0f, expf(-z))); }
    static __device__ __forceinline__ float lost(float x) { return expm1f(x); }
    static __device__ __forceinline__ float root(float x) { return __fsqrt_rn(x); }
};
template <> struct Unit<bf16> {
    static __device__ __forceinline__ float sigmoid(float z) {
        return reciprocal_unit(1.0f + exp2_unit(__fmul_rn(-z, UNIT_LOG2E)));
    }
    static __device__ __forceinline__ float lost(float x) {       // by its series where the difference would cancel
        const float series = x * __fmaf_rn(x, __fmaf_rn(x, __fmaf_rn(x, 0.041666668f, 0.16666667f), 0.5f), 1.0f);
        return x > -0.0625f ? series : exp2_unit(__fmul_rn(x, UNIT_LOG2E)) - 1.0f;
    }
    static __device__ __forceinline__ float root(float x) {
        float y;
        asm("sqrt.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
        return y;
    }
};

template <typename T> __device__ __forceinline__ float branch_act(float z, int act) {
    if (act == UNIT_ACT_NONE) return z;
    if (act == UNIT_ACT_SILU) return silu_for<T>(z);
    // 0.5 z (1 + tanh(t)) = z sigmoid(2 t), t = sqrt(2 / pi) (z + 0.044715 z^3)
    const float inner = __fmul_rn(0.7978845608028654f, __fmaf_rn(__fmul_rn(0.044715f, z), __fmul_rn(z, z), z));
    return __fmul_rn(z, Unit<T>::sigmoid(__fmul_rn(2.0f, inner)));
}

struct UnitArgs {
    int64_t u_stride, y_stride, out_stride;
    const float* pre;                             // element (token, block, j): r's at j, i's at size + j
    int64_t pre_token, pre_block;
    const float *bias_r, *bias_i, *decay, *bias_y;            // [channels] each, bias_y may be null
    float* state;                                 // [slots, channels]
    const int *row_starts, *state_slots, *token_row;
    int channels, size, act;                      // size: channels of a block of gates
};

// Decay and new input of one channel at one token.
template <typename T> __device__ __forceinline__ void unit_terms(float pre_r, float pre_i, float u, float br, float bi,
                                                                 float c, float& a, float& b) {
    const float e = Unit<T>::lost(__fmul_rn(c, Unit<T>::sigmoid(__fadd_rn(pre_r, br))));
    a = __fadd_rn(1.0f, e);
    const float written = Unit<T>::root(fmaxf(__fmul_rn(-e, __fadd_rn(2.0f, e)), 0.0f));
    b = __fmul_rn(__fmul_rn(written, Unit<T>::sigmoid(__fadd_rn(pre_i, bi))), u);
}

// The address in the shared memory of the cluster's CTA `rank` of what `p` is in this CTA's.
__device__ __forceinline__ float load_of_cta(const float* p, int rank) {
    uint32_t address;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(address) : "r"(smem_address(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];\n" : "=f"(v) : "r"(address) : "memory");
    return v;
}

template <typename T>
__global__ void __launch_bounds__(UNIT_WARPS * 32, 3) recurrent_unit_scan_kernel(
    const T* __restrict__ u, const T* __restrict__ y, T* __restrict__ out, UnitArgs args, int ctas) {
    __shared__ float products[2][UNIT_WARPS][32], ends[2][UNIT_WARPS][32], block_product[2][32], block_end[2][32];
    const int row = blockIdx.z, rank = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int begin = args.row_starts[row], count = args.row_starts[row + 1] - begin;
    const int channel = blockIdx.y * 32 + lane;
    const bool live = channel < args.channels;
    const int at = live ? channel : 0;
    const bool owned = count > 0 && args.token_row[begin] >= 0;
    if (!owned) {                                 // the whole cluster leaves: a padding row of a recorded batch
        if (live)
            for (int t = rank * UNIT_WARPS + warp; t < count; t += ctas * UNIT_WARPS)
                out[(int64_t)(begin + t) * args.out_stride + at] = from_float<T>(0.0f);
        return;
    }
    float* mine = args.state + (int64_t)args.state_slots[row] * args.channels + at;
    const float br = args.bias_r[at], bi = args.bias_i[at], c = args.decay[at];
    const float by = args.bias_y ? args.bias_y[at] : 0.0f;
    float carry = live ? mine[0] : 0.0f;          // the state before the cluster's tokens, in every warp
    // this warp's first token and the pointers to it
    int t0 = (rank * UNIT_WARPS + warp) * UNIT_RUN;
    const T* u_in = u + (int64_t)(begin + t0) * args.u_stride + at;
    const T* y_in = y + (int64_t)(begin + t0) * args.y_stride + at;
    T* dst = out + (int64_t)(begin + t0) * args.out_stride + at;
    const float* pre_in = args.pre + (int64_t)(begin + t0) * args.pre_token + (int64_t)(at / args.size) * args.pre_block + at % args.size;
    const int step = ctas * UNIT_BLOCK;
    for (int first = 0, turn = 0; first < count; first += step, turn ^= 1) {
        float a[UNIT_RUN], b[UNIT_RUN], pre_r[UNIT_RUN], pre_i[UNIT_RUN];
        T u_now[UNIT_RUN], y_now[UNIT_RUN];
        const int here = live ? count - t0 : 0;   // tokens of the entry from this warp's first on
#pragma unroll
        for (int t = 0; t < UNIT_RUN; ++t)        // all loads of a block are in flight together
            if (t < here) {
                pre_r[t] = pre_in[t * args.pre_token];
                pre_i[t] = pre_in[t * args.pre_token + args.size];
                u_now[t] = u_in[t * args.u_stride];
                y_now[t] = y_in[t * args.y_stride];
            }
        float product = 1.0f, end = 0.0f;
#pragma unroll
        for (int t = 0; t < UNIT_RUN; ++t) {
            a[t] = 1.0f;                          // tokens past the end keep the state as it is
            b[t] = 0.0f;
            if (t < here) unit_terms<T>(pre_r[t], pre_i[t], to_float<T>(u_now[t]), br, bi, c, a[t], b[t]);
            product = __fmul_rn(product, a[t]);
            end = __fmaf_rn(a[t], end, b[t]);
        }
        products[turn][warp][lane] = product;
        ends[turn][warp][lane] = end;
        __syncthreads();
        if (ctas > 1) {
            if (warp == 0) {                      // the CTA's tokens as one, for the other CTAs
                float all = 1.0f, s = 0.0f;
#pragma unroll
                for (int w = 0; w < UNIT_WARPS; ++w) {
                    s = __fmaf_rn(products[turn][w][lane], s, ends[turn][w][lane]);
                    all = __fmul_rn(all, products[turn][w][lane]);
                }
                block_product[turn][lane] = all;
                block_end[turn][lane] = s;
            }
            cluster_arrive();
            cluster_wait();
        }
        float s = carry;
        if (ctas > 1) {
            for (int r = 0; r < ctas; ++r) {      // to this CTA's tokens, and on to the next round's
                if (r == rank) s = carry;
                carry = __fmaf_rn(load_of_cta(&block_product[turn][lane], r), carry, load_of_cta(&block_end[turn][lane], r));
            }
        } else {
#pragma unroll
            for (int w = 0; w < UNIT_WARPS; ++w) carry = __fmaf_rn(products[turn][w][lane], carry, ends[turn][w][lane]);
        }
        for (int w = 0; w < warp; ++w) s = __fmaf_rn(products[turn][w][lane], s, ends[turn][w][lane]);
#pragma unroll
        for (int t = 0; t < UNIT_RUN; ++t) {
            s = __fmaf_rn(a[t], s, b[t]);
            if (t < here)
                dst[t * args.out_stride] =
                    from_float<T>(__fmul_rn(s, branch_act<T>(__fadd_rn(to_float<T>(y_now[t]), by), args.act)));
        }
        t0 += step;
        u_in += (int64_t)step * args.u_stride;
        y_in += (int64_t)step * args.y_stride;
        dst += (int64_t)step * args.out_stride;
        pre_in += (int64_t)step * args.pre_token;
    }
    if (rank == 0 && warp == 0 && live) mine[0] = carry;
    if (ctas > 1) {                               // no CTA leaves while another reads its shared memory
        cluster_arrive();
        cluster_wait();
    }
}

// One token a request, gates given: a thread a (request, channel).
template <typename T>
__global__ void __launch_bounds__(128) recurrent_unit_step_kernel(const T* __restrict__ u, const T* __restrict__ y,
                                                                  T* __restrict__ out, UnitArgs args) {
    const int row = blockIdx.y, channel = blockIdx.x * 128 + threadIdx.x;
    if (channel >= args.channels) return;
    const int64_t token = args.row_starts[row];
    float result = 0.0f;
    if (args.token_row[token] >= 0) {
        const float* pre = args.pre + token * args.pre_token + (int64_t)(channel / args.size) * args.pre_block + channel % args.size;
        float a, b;
        unit_terms<T>(pre[0], pre[args.size], to_float<T>(u[token * args.u_stride + channel]), args.bias_r[channel],
                      args.bias_i[channel], args.decay[channel], a, b);
        float* mine = args.state + (int64_t)args.state_slots[row] * args.channels + channel;
        const float s = __fmaf_rn(a, mine[0], b);
        mine[0] = s;
        result = __fmul_rn(s, branch_act<T>(__fadd_rn(to_float<T>(y[token * args.y_stride + channel]),
                                                      args.bias_y ? args.bias_y[channel] : 0.0f), args.act));
    }
    out[token * args.out_stride + channel] = from_float<T>(result);
}

// One token a request, the gates' products inside.  A CTA takes GATE_CHANNELS channels of one block of gates for up to
// ROWS requests: u of the block waits in shared memory (float32), a warp takes a channel at a time, its lanes eight (or
// one) neighbouring weights of the channel's two rows, and the 2 ROWS sums are added by halving over the lanes.
#define GATE_CHANNELS 8
#define GATE_WARPS 4
// VEC neighbouring weights as they were loaded
template <typename T, int VEC> struct Weights;
template <typename T> struct Weights<T, 1> {
    T v;
    __device__ __forceinline__ void load(const T* p) { v = *p; }
    __device__ __forceinline__ void spread(float* x) const { x[0] = to_float<T>(v); }
};
template <> struct Weights<float, 8> {
    float v[8];
    __device__ __forceinline__ void load(const float* p) { load_values<4>(p, v); load_values<4>(p + 4, v + 4); }
    __device__ __forceinline__ void spread(float* x) const {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = v[i];
    }
};
template <> struct Weights<bf16, 8> {
    uint4 v;
    __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void spread(float* x) const { unpack_bf16x8(v, x); }
};

template <typename T, int ROWS, int VEC>
__global__ void __launch_bounds__(GATE_WARPS * 32) recurrent_unit_gated_step_kernel(
    const T* __restrict__ u, const T* __restrict__ y, const T* __restrict__ w, T* __restrict__ out, UnitArgs args, int rows) {
    extern __shared__ __align__(16) float u_s[];              // [ROWS][size rounded up to 8]
    __shared__ float gates[2 * ROWS][GATE_CHANNELS];
    constexpr int SUMS = 2 * ROWS;
    const int size = args.size, padded = (size + 7) / 8 * 8;
    const int parts = (size + GATE_CHANNELS - 1) / GATE_CHANNELS;
    const int block = blockIdx.x / parts, j0 = blockIdx.x % parts * GATE_CHANNELS;
    const int row0 = blockIdx.y * ROWS, here = min(ROWS, rows - row0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    constexpr int MINE = GATE_CHANNELS / GATE_WARPS;                  // a warp's channels: their first weights are on
    Weights<T, VEC> ahead_r[MINE], ahead_i[MINE];                    // their way before u is there
#pragma unroll
    for (int i = 0; i < MINE; ++i) {
        const int j = j0 + warp + i * GATE_WARPS;
        if (j < size && lane * VEC < size) {
            const T* w_r = w + ((int64_t)block * 2 * size + j) * size + lane * VEC;
            ahead_r[i].load(w_r);
            ahead_i[i].load(w_r + (int64_t)size * size);
        }
    }
    for (int e = threadIdx.x; e < ROWS * padded; e += GATE_WARPS * 32) {
        const int q = e / padded, k = e % padded;
        u_s[e] = q < here && k < size ? to_float<T>(u[(int64_t)args.row_starts[row0 + q] * args.u_stride + block * size + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MINE; ++i) {
        const int c = warp + i * GATE_WARPS;
        if (j0 + c >= size) break;
        const T* w_r = w + ((int64_t)block * 2 * size + j0 + c) * size;
        const T* w_i = w_r + (int64_t)size * size;
        float sums[SUMS];
#pragma unroll
        for (int e = 0; e < SUMS; ++e) sums[e] = 0.0f;
        for (int k = lane * VEC; k < size; k += 32 * VEC) {
            float r[VEC], in[VEC];
            if (k == lane * VEC) { ahead_r[i].spread(r); ahead_i[i].spread(in); }
            else { Weights<T, VEC> x; x.load(w_r + k); x.spread(r); x.load(w_i + k); x.spread(in); }
#pragma unroll
            for (int q = 0; q < ROWS; ++q) {
                float x[VEC];
                if constexpr (VEC == 8) { load_values<4>(&u_s[q * padded + k], x); load_values<4>(&u_s[q * padded + k + 4], x + 4); }
                else x[0] = u_s[q * padded + k];
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    sums[2 * q] = __fmaf_rn(r[v], x[v], sums[2 * q]);
                    sums[2 * q + 1] = __fmaf_rn(in[v], x[v], sums[2 * q + 1]);
                }
            }
        }
        // halving over the lanes: the lane whose bit is set keeps the upper half; lanes left over add plainly
        int owner = 0;
#pragma unroll
        for (int bit = 16, n = SUMS; bit >= 1; bit >>= 1) {
            if (n > 1) {
                const bool upper = (lane & bit) != 0;
#pragma unroll
                for (int e = 0; e < n / 2; ++e) {
                    const float hand = upper ? sums[e] : sums[e + n / 2], keep = upper ? sums[e + n / 2] : sums[e];
                    sums[e] = keep + __shfl_xor_sync(0xffffffffu, hand, bit);
                }
                if (upper) owner += n / 2;
                n >>= 1;
            } else sums[0] += __shfl_xor_sync(0xffffffffu, sums[0], bit);
        }
        gates[owner][c] = sums[0];                // lanes with the same owner hold the same sum
    }
    __syncthreads();
    for (int e = threadIdx.x; e < here * GATE_CHANNELS; e += GATE_WARPS * 32) {
        const int q = e / GATE_CHANNELS, c = e % GATE_CHANNELS;
        if (j0 + c >= size) continue;
        const int channel = block * size + j0 + c;
        const int64_t token = args.row_starts[row0 + q];
        float result = 0.0f;
        if (args.token_row[token] >= 0) {         // a padding row of a recorded batch has no request and no state
            float a, b;
            unit_terms<T>(gates[2 * q][c], gates[2 * q + 1][c], u_s[q * padded + j0 + c], args.bias_r[channel],
                          args.bias_i[channel], args.decay[channel], a, b);
            float* mine = args.state + (int64_t)args.state_slots[row0 + q] * args.channels + channel;
            const float s = __fmaf_rn(a, mine[0], b);
            mine[0] = s;
            result = __fmul_rn(s, branch_act<T>(__fadd_rn(to_float<T>(y[token * args.y_stride + channel]),
                                                          args.bias_y ? args.bias_y[channel] : 0.0f), args.act));
        }
        out[token * args.out_stride + channel] = from_float<T>(result);
    }
}

// u, y, out: [tokens, >= channels] of the storage type with row strides; pre float32 with strides for the token and for
// the block of gates (`size` channels each; r's pre-activations, then i's), or, with `single`, null and w [blocks, 2
// size, size] of the storage type (u's products are done here); bias_r, bias_i, decay float32 [channels], bias_y too
// or null; state float32 [slots, channels].  `single`: every entry is one token; `tokens`: of all
// entries.
extern "C" int tvb_recurrent_unit(const void* u, long long u_stride, const void* y, long long y_stride, const float* pre,
                                  long long pre_token, long long pre_block, const void* w, const float* bias_r,
                                  const float* bias_i, const float* decay, const float* bias_y, float* state,
                                  const int* row_starts, const int* state_slots, const int* token_row, void* out,
                                  long long out_stride, int rows, int tokens, int channels, int size, int act, int single,
                                  int dtype, void* stream) {
    if (rows <= 0) return 0;
    if (channels <= 0 || size <= 0 || channels % size || rows > 65535 || act < 0 || act > 2 || !state || !bias_r || !bias_i ||
        !decay || (!pre == !w) || (w && !single))
        return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const UnitArgs args{u_stride, y_stride, out_stride, pre, pre_token, pre_block, bias_r, bias_i, decay, bias_y, state,
                        row_starts, state_slots, token_row, channels, size, act};
    if (w) {
        const int parts = (size + GATE_CHANNELS - 1) / GATE_CHANNELS;
        const int together = rows == 1 ? 1 : rows == 2 ? 2 : rows <= 4 ? 4 : 8;
        const size_t smem = (size_t)together * ((size + 7) / 8 * 8) * sizeof(float);
        if (smem > 40 * 1024) return TVB_BAD_ARGUMENT;
        const dim3 grid(channels / size * parts, (rows + together - 1) / together);
        const bool wide = size % 8 == 0 && (uintptr_t)w % 16 == 0;
#define GO(T, R, V) recurrent_unit_gated_step_kernel<T, R, V><<<grid, GATE_WARPS * 32, smem, s>>>(                      \
        (const T*)u, (const T*)y, (const T*)w, (T*)out, args, rows)
#define BY_VEC(T, R) if (wide) GO(T, R, 8); else GO(T, R, 1)
#define BY_ROWS(T)                                   \
    if (together == 1) { BY_VEC(T, 1); }             \
    else if (together == 2) { BY_VEC(T, 2); }        \
    else if (together == 4) { BY_VEC(T, 4); }        \
    else { BY_VEC(T, 8); }
        if (dtype == TVB_F32) { BY_ROWS(float) }
        else if (dtype == TVB_BF16) { BY_ROWS(bf16) }
        else return TVB_BAD_ARGUMENT;
#undef BY_ROWS
#undef BY_VEC
#undef GO
        return tvb_last_error();
    }
    if (single) {
        const dim3 grid((channels + 127) / 128, rows);
        if (dtype == TVB_F32)
            recurrent_unit_step_kernel<float><<<grid, 128, 0, s>>>((const float*)u, (const float*)y, (float*)out, args);
        else if (dtype == TVB_BF16)
            recurrent_unit_step_kernel<bf16><<<grid, 128, 0, s>>>((const bf16*)u, (const bf16*)y, (bf16*)out, args);
        else return TVB_BAD_ARGUMENT;
        return tvb_last_error();
    }
    // as many CTAs a cluster as the step's longest entry could use, while SMs would idle otherwise
    const int groups = (channels + 31) / 32;
    int ctas = 1;
    while (ctas < UNIT_MOST_CTAS && 2 * ctas * UNIT_BLOCK <= tokens && (long long)groups * rows * ctas < 4 * 148) ctas *= 2;
    if (groups > 65535) return TVB_BAD_ARGUMENT;
    TvbLaunch launch(dim3(ctas, groups, rows), dim3(UNIT_WARPS * 32), 0, s, 0, ctas);
    cudaError_t e;
    if (dtype == TVB_F32)
        e = cudaLaunchKernelEx(&launch.config, recurrent_unit_scan_kernel<float>, (const float*)u, (const float*)y, (float*)out, args, ctas);
    else if (dtype == TVB_BF16)
        e = cudaLaunchKernelEx(&launch.config, recurrent_unit_scan_kernel<bf16>, (const bf16*)u, (const bf16*)y, (bf16*)out, args, ctas);
    else return TVB_BAD_ARGUMENT;
    return e == cudaSuccess ? tvb_last_error() : (int)e;
}
