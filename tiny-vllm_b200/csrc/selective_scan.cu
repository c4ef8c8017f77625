// The selective scan: a float32 state [channels, SCAN_STATE] a request whose decay, input and output directions
// come from the token (compiled per size of the state).
//
//   dt = softplus(pre + bias)                                  pre: a product's output, one number a channel
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n        B, C: SCAN_STATE numbers a token, shared by the channels
//   y_c = sum_n S[c, n] C_n + D_c x_c,    out = y silu(z)
//
//   selective_scan   prompts: a CTA walks one entry for a block of channels, token by token in blocks of SCAN_BLOCK
//                    that wait in shared memory while the next block's loads are in flight
//   selective_step   one token a request: the state is read and written once
//
// Step sizes, exponentials, state and sums are float32 whatever the storage type of x, z, B, C and out.
#include "common.cuh"

#ifndef SCAN_STATE
#define SCAN_STATE 16
#endif

#define SCAN_THREADS 128
#define SCAN_BLOCK (SCAN_STATE <= 64 ? 32 : 16)      // tokens that wait in shared memory
#define SCAN_PAD 4
#define SCAN_FILL 256                                // CTAs from which the GPU counts as full
// lanes that share a channel: eight (fewer where the state is smaller), sixteen while SMs would idle otherwise or where
// the state is larger than eight lanes hold
constexpr int SCAN_FEWEST = SCAN_STATE <= 2 ? 2 : SCAN_STATE <= 4 ? 4 : SCAN_STATE <= 128 ? 8 : 16;
constexpr int SCAN_MOST = SCAN_STATE > 8 ? 16 : SCAN_FEWEST;
#define SCAN_LOG2E 1.4426950408889634f

static_assert(SCAN_STATE >= 1 && SCAN_STATE <= 256, "selective_scan: state size");

// The scan's float32 functions.  With 16-bit storage they take the special-function unit's 2^x and log2 (a few units
// in the last place, far below the rounding of what goes in); decays are then prepared as a log2 e.
//   decay     exp(dt * a)
//   softplus  max(z, 0) + ln(1 + exp(-|z|))
template <typename T> struct Scan;
template <> struct Scan<float> {
    static __device__ __forceinline__ float prepare(float a) { return a; }
    static __device__ __forceinline__ float decay(float dt, float a) { return expf(__fmul_rn(dt, a)); }
    static __device__ __forceinline__ float softplus(float z) { return __fadd_rn(fmaxf(z, 0.0f), log1pf(expf(-fabsf(z)))); }
};
template <> struct Scan<bf16> {
    static __device__ __forceinline__ float prepare(float a) { return __fmul_rn(a, SCAN_LOG2E); }
    static __device__ __forceinline__ float decay(float dt, float a) { return exp2_unit(__fmul_rn(dt, a)); }
    static __device__ __forceinline__ float softplus(float z) {
        const float u = exp2_unit(__fmul_rn(-fabsf(z), SCAN_LOG2E));
        float log2;
        asm("lg2.approx.ftz.f32 %0, %1;\n" : "=f"(log2) : "f"(1.0f + u));
        // the series of ln(1 + u) where 1 + u would round u away
        const float series = u * __fmaf_rn(u, __fmaf_rn(u, __fmaf_rn(u, -0.25f, 0.33333333f), -0.5f), 1.0f);
        return fmaxf(z, 0.0f) + (u < 0.015625f ? series : __fmul_rn(log2, 0.69314718f));
    }
};

// LANES lanes share a channel, lane l holds the numbers l, l + LANES, ... of its state, and does so for TILE channels
// (B and C are read from shared memory once for all of them).  Shared memory holds dt and dt * x by channel and B and
// C by state number, four tokens to a 16-byte access.  A lane's partial sums of y are
// added by halving: at every step a lane hands half of its sums to the lane one bit away and keeps the other half,
// so that lane g ends with complete sums of SUB / LANES tokens.
// A thread moves BOTH neighbouring channels (or numbers of B and C) at a time: 2 where sizes and addresses allow it.
template <typename T, int BOTH> struct Raw;
template <typename T> struct Raw<T, 1> {
    T v;
    __device__ __forceinline__ void load(const T* p) { v = *p; }
    __device__ __forceinline__ float at(int) const { return to_float<T>(v); }
};
template <> struct Raw<float, 2> {
    float2 v;
    __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float2*>(p); }
    __device__ __forceinline__ float at(int i) const { return i ? v.y : v.x; }
};
template <> struct Raw<bf16, 2> {
    uint32_t v;
    __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint32_t*>(p); }
    __device__ __forceinline__ float at(int i) const { return __uint_as_float(i ? v & 0xffff0000u : v << 16); }
};
template <int BOTH> __device__ __forceinline__ void store_both(float* p, const float* y) {
    if constexpr (BOTH == 2) *reinterpret_cast<float2*>(p) = make_float2(y[0], y[1]);
    else *p = y[0];
}
template <int BOTH> __device__ __forceinline__ void store_both(bf16* p, const float* y) {
    if constexpr (BOTH == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(y[0], y[1]);
    else *p = __float2bfloat16_rn(y[0]);
}

template <typename T, int LANES, int TILE, int BOTH>
__global__ void __launch_bounds__(SCAN_THREADS) selective_scan_kernel(
    const T* __restrict__ x, int64_t x_stride, const float* __restrict__ pre, const T* __restrict__ z, int64_t z_stride,
    const T* __restrict__ b, const T* __restrict__ c, int64_t bc_stride, const float* __restrict__ a,
    const float* __restrict__ d, const float* __restrict__ dt_bias, float* __restrict__ state,
    const int* __restrict__ row_starts, const int* __restrict__ state_slots, const int* __restrict__ token_row,
    T* __restrict__ out, int64_t out_stride, int channels) {
    constexpr int N = SCAN_STATE, ROWS = (N + LANES - 1) / LANES;
    constexpr int APART = SCAN_THREADS / LANES, CH = APART * TILE;     // a thread's channels are APART apart
    constexpr int SUB = LANES > 8 ? LANES : 8, LEFT = SUB / LANES, WIDTH = SCAN_BLOCK + SCAN_PAD;
    constexpr int MOVERS = CH / BOTH, STEP = SCAN_THREADS / MOVERS;   // threads a token when values move, tokens at once
    constexpr int PER = SCAN_BLOCK / STEP;                            // places a thread moves
    constexpr int PLACES = SCAN_BLOCK * (N / BOTH), BC = (PLACES + SCAN_THREADS - 1) / SCAN_THREADS;
    constexpr bool AHEAD = BC <= 16;                                  // B and C of the next block wait in registers
    static_assert(SCAN_BLOCK % SUB == 0 && STEP <= SCAN_BLOCK && SCAN_THREADS % MOVERS == 0 && CH % BOTH == 0, "selective_scan: tile");
    __shared__ __align__(16) float dt_s[CH][WIDTH];
    __shared__ __align__(16) float u_s[CH][WIDTH];                    // dt * x, then y
    __shared__ __align__(16) float b_s[LANES * ROWS][WIDTH];
    __shared__ __align__(16) float c_s[LANES * ROWS][WIDTH];
    const int row = blockIdx.y, tid = threadIdx.x, lane = tid % LANES, mine = tid / LANES;
    const int begin = row_starts[row], count = row_starts[row + 1] - begin;
    if (count <= 0) return;
    const int c0 = blockIdx.x * CH;
    const int move_ch = tid % MOVERS * BOTH, move_t = tid / MOVERS;   // this thread's channels and first token when it moves values
    const bool live = c0 + move_ch < channels;
    T* dst = out + (int64_t)begin * out_stride + c0 + move_ch;
    if (token_row[begin] < 0) {                   // a padding row of a recorded batch: no request, no state
        const float zero[BOTH] = {};
        if (live)
            for (int t = move_t; t < count; t += STEP) store_both<BOTH>(dst + (int64_t)t * out_stride, zero);
        return;
    }
    float* state_of = state + ((int64_t)state_slots[row] * channels + c0 + mine) * N + lane;
    const float* a_of = a + (int64_t)(c0 + mine) * N + lane;
    float s[TILE][ROWS], decay[TILE][ROWS];
#pragma unroll
    for (int k = 0; k < TILE; ++k)
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const bool has = c0 + mine + k * APART < channels && lane + r * LANES < N;
            s[k][r] = has ? state_of[k * APART * N + r * LANES] : 0.0f;
            decay[k][r] = has ? Scan<T>::prepare(a_of[k * APART * N + r * LANES]) : 0.0f;
        }
    if (LANES * ROWS > N)
        for (int e = tid; e < (LANES * ROWS - N) * SCAN_BLOCK; e += SCAN_THREADS) {
            b_s[N + e / SCAN_BLOCK][e % SCAN_BLOCK] = 0.0f;
            c_s[N + e / SCAN_BLOCK][e % SCAN_BLOCK] = 0.0f;
        }
    float skip[BOTH], shift[BOTH];
#pragma unroll
    for (int i = 0; i < BOTH; ++i) {
        skip[i] = live ? d[c0 + move_ch + i] : 0.0f;
        shift[i] = live && dt_bias ? dt_bias[c0 + move_ch + i] : 0.0f;
    }
    const T* x_in = x + (int64_t)(begin + move_t) * x_stride + c0 + move_ch;
    const T* z_in = z + (int64_t)(begin + move_t) * z_stride + c0 + move_ch;
    const float* pre_in = pre + (int64_t)(begin + move_t) * channels + c0 + move_ch;
    const T* b_in = b + (int64_t)begin * bc_stride;
    const T* c_in = c + (int64_t)begin * bc_stride;
    dst += (int64_t)move_t * out_stride;
    const int64_t x_step = (int64_t)STEP * x_stride, z_step = (int64_t)STEP * z_stride, pre_step = (int64_t)STEP * channels,
                  out_step = (int64_t)STEP * out_stride;

    // the next block as it was loaded: nothing waits for it before it is put into shared memory
    Raw<T, BOTH> x_next[PER], z_next[PER], b_next[AHEAD ? BC : 1], c_next[AHEAD ? BC : 1];
    Raw<float, BOTH> p_next[PER];
    auto fetch = [&](int first) {                 // the pointers stand at the block's first token
#pragma unroll
        for (int j = 0; j < PER; ++j)
            if (live && first + move_t + j * STEP < count) {
                x_next[j].load(x_in + j * x_step);
                z_next[j].load(z_in + j * z_step);
                p_next[j].load(pre_in + j * pre_step);
            }
        if constexpr (AHEAD) {
#pragma unroll
            for (int j = 0; j < BC; ++j) {
                const int e = tid + j * SCAN_THREADS, t = e / (N / BOTH), n = e % (N / BOTH) * BOTH;
                if ((PLACES % SCAN_THREADS == 0 || e < PLACES) && first + t < count) {
                    b_next[j].load(b_in + (int64_t)t * bc_stride + n);
                    c_next[j].load(c_in + (int64_t)t * bc_stride + n);
                }
            }
        }
        x_in += PER * x_step;
        z_in += PER * z_step;
        pre_in += PER * pre_step;
        b_in += SCAN_BLOCK * bc_stride;
        c_in += SCAN_BLOCK * bc_stride;
    };

    fetch(0);
    for (int first = 0; first < count; first += SCAN_BLOCK) {
        __syncthreads();                          // the block before is read
        Raw<T, BOTH> x_now[PER], z_now[PER];
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = move_t + j * STEP;
            // tokens past the end move nothing: dt = 0 keeps the state as it is
            const bool ok = live && first + t < count;
#pragma unroll
            for (int i = 0; i < BOTH; ++i) {
                const float dt = ok ? Scan<T>::softplus(__fadd_rn(p_next[j].at(i), shift[i])) : 0.0f;
                dt_s[move_ch + i][t] = dt;
                u_s[move_ch + i][t] = ok ? __fmul_rn(dt, x_next[j].at(i)) : 0.0f;
            }
            x_now[j] = x_next[j];
            z_now[j] = z_next[j];
        }
#pragma unroll
        for (int j = 0; j < BC; ++j) {
            const int e = tid + j * SCAN_THREADS, t = e / (N / BOTH), n = e % (N / BOTH) * BOTH;
            if (PLACES % SCAN_THREADS == 0 || e < PLACES) {
                const bool ok = first + t < count;
                Raw<T, BOTH> b_now, c_now;
                if constexpr (AHEAD) { b_now = b_next[j]; c_now = c_next[j]; }
                else if (ok) {                    // the pointers stand one block ahead
                    b_now.load(b_in + (int64_t)(t - SCAN_BLOCK) * bc_stride + n);
                    c_now.load(c_in + (int64_t)(t - SCAN_BLOCK) * bc_stride + n);
                }
#pragma unroll
                for (int i = 0; i < BOTH; ++i) {
                    b_s[n + i][t] = ok ? b_now.at(i) : 0.0f;
                    c_s[n + i][t] = ok ? c_now.at(i) : 0.0f;
                }
            }
        }
        __syncthreads();
        if (first + SCAN_BLOCK < count) fetch(first + SCAN_BLOCK);
#pragma unroll 1
        for (int sub = 0; sub < SCAN_BLOCK && first + sub < count; sub += SUB) {
            float sums[TILE][SUB];
#pragma unroll
            for (int k = 0; k < TILE; ++k)
#pragma unroll
                for (int i = 0; i < SUB; ++i) sums[k][i] = 0.0f;
#pragma unroll
            for (int t = 0; t < SUB; t += 4) {
                float dt[TILE][4], u[TILE][4];
#pragma unroll
                for (int k = 0; k < TILE; ++k) {
                    load_values<4>(&dt_s[mine + k * APART][sub + t], dt[k]);
                    load_values<4>(&u_s[mine + k * APART][sub + t], u[k]);
                }
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    float bb[4], cc[4];
                    load_values<4>(&b_s[lane + r * LANES][sub + t], bb);
                    load_values<4>(&c_s[lane + r * LANES][sub + t], cc);
#pragma unroll
                    for (int k = 0; k < TILE; ++k)
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            s[k][r] = __fmaf_rn(Scan<T>::decay(dt[k][i], decay[k][r]), s[k][r], __fmul_rn(u[k][i], bb[i]));
                            sums[k][t + i] = __fmaf_rn(s[k][r], cc[i], sums[k][t + i]);
                        }
                }
            }
#pragma unroll
            for (int bit = LANES / 2, n = SUB; bit >= 1; bit >>= 1, n >>= 1) {
                const bool upper = (lane & bit) != 0;
#pragma unroll
                for (int k = 0; k < TILE; ++k)
#pragma unroll
                    for (int i = 0; i < n / 2; ++i) {
                        const float hand = upper ? sums[k][i] : sums[k][i + n / 2];
                        const float keep = upper ? sums[k][i + n / 2] : sums[k][i];
                        sums[k][i] = keep + __shfl_xor_sync(0xffffffffu, hand, bit);
                    }
            }
            __syncwarp();                         // the channels' lanes have read dt * x of these tokens
#pragma unroll
            for (int k = 0; k < TILE; ++k)
#pragma unroll
                for (int i = 0; i < LEFT; ++i) u_s[mine + k * APART][sub + lane * LEFT + i] = sums[k][i];
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = move_t + j * STEP;
            if (live && first + t < count) {
                float y[BOTH];
#pragma unroll
                for (int i = 0; i < BOTH; ++i)
                    y[i] = __fmul_rn(__fmaf_rn(skip[i], x_now[j].at(i), u_s[move_ch + i][t]), silu_for<T>(z_now[j].at(i)));
                store_both<BOTH>(dst + j * out_step, y);
            }
        }
        dst += PER * out_step;
    }
#pragma unroll
    for (int k = 0; k < TILE; ++k)
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            if (c0 + mine + k * APART < channels && lane + r * LANES < N) state_of[k * APART * N + r * LANES] = s[k][r];
}

// x: [tokens, >= channels]; pre float32 [tokens, channels]; z, b, c as x, each with a row stride; a float32
// [channels, SCAN_STATE]; d, dt_bias float32 [channels]; state float32 [slots, channels, SCAN_STATE]; out
// [tokens, >= channels].  `lanes` (0: chosen): SCAN_FEWEST or SCAN_MOST lanes a channel; `tile` (0: chosen): one or two channels a
// thread; a thread holds at most 16 numbers of state.
extern "C" int tvb_selective_scan(const void* x, long long x_stride, const float* pre, const void* z, long long z_stride,
                                  const void* b, const void* c, long long bc_stride, const float* a, const float* d,
                                  const float* dt_bias, float* state, const int* row_starts, const int* state_slots,
                                  const int* token_row, void* out, long long out_stride, int rows, int channels,
                                  int lanes, int tile, int dtype, void* stream) {
    if (rows <= 0) return 0;
    if (channels <= 0 || rows > 65535 || !state || !a || !d || !pre) return TVB_BAD_ARGUMENT;
    auto ctas = [&](int l, int t) { return (long long)rows * ((channels + SCAN_THREADS / l * t - 1) / (SCAN_THREADS / l * t)); };
    if (lanes == 0) lanes = SCAN_MOST > SCAN_FEWEST && ctas(SCAN_FEWEST, 1) < SCAN_FILL ? SCAN_MOST : SCAN_FEWEST;
    const bool pairs = lanes >= 8 && 16 * lanes >= 2 * SCAN_STATE;        // two channels a thread where CTAs are plenty
    if (tile == 0) tile = pairs && ctas(lanes, 2) >= 4 * SCAN_FILL ? 2 : 1;
    if ((lanes != SCAN_FEWEST && lanes != SCAN_MOST) || tile < 1 || tile > 2 || (tile == 2 && !pairs)) return TVB_BAD_ARGUMENT;
    const int ch = SCAN_THREADS / lanes * tile;
    const dim3 grid((channels + ch - 1) / ch, rows);
    cudaStream_t s = (cudaStream_t)stream;
    const size_t element = dtype == TVB_BF16 ? 2 : 4;
    auto even = [&](const void* p, long long stride) { return (uintptr_t)p % (2 * element) == 0 && stride % 2 == 0; };
    const bool both = SCAN_STATE % 2 == 0 && channels % 2 == 0 && even(x, x_stride) && even(z, z_stride) && even(b, bc_stride) &&
                      even(c, bc_stride) && even(out, out_stride) && (uintptr_t)pre % 8 == 0;
#define GO(T, L, K) if (both) GO_BY(T, L, K, 1 + (SCAN_STATE % 2 == 0 && SCAN_STATE <= 64)); else GO_BY(T, L, K, 1)
#define GO_BY(T, L, K, B) selective_scan_kernel<T, L, K, B><<<grid, SCAN_THREADS, 0, s>>>(                            \
        (const T*)x, x_stride, pre, (const T*)z, z_stride, (const T*)b, (const T*)c, bc_stride, a, d, dt_bias, state, \
        row_starts, state_slots, token_row, (T*)out, out_stride, channels)
#define BY_TILE(T, L)                                                                 \
    if constexpr (SCAN_STATE * 2 <= 16 * L && L >= 8) {                               \
        if (tile == 2) { GO(T, L, 2); } else { GO(T, L, 1); }                         \
    } else { GO(T, L, 1); }
#define BY_LANES(T)                                                                   \
    if constexpr (SCAN_MOST > SCAN_FEWEST) {                                          \
        if (lanes == SCAN_MOST) { BY_TILE(T, SCAN_MOST) } else { BY_TILE(T, SCAN_FEWEST) } \
    } else { BY_TILE(T, SCAN_FEWEST) }
    if (dtype == TVB_F32) { BY_LANES(float) }
    else if (dtype == TVB_BF16) { BY_LANES(bf16) }
    else return TVB_BAD_ARGUMENT;
#undef BY_LANES
#undef BY_TILE
#undef GO_BY
#undef GO
    return tvb_last_error();
}

// One token a request; a CTA takes TOGETHER requests for a block of channels (the weights below are read once for all
// of them).  The lanes of a channel take its state VEC numbers at a time.  With `dt_weight` the step
// size's product is done here too: pre_c = sum_k low_k W[c, k], low being `rank` numbers a token (rank a multiple
// of 8, rows of W 16-byte aligned in 16-bit storage).
__device__ __forceinline__ void load_eight(const float* p, float* v) {
    load_values<4>(p, v);
    load_values<4>(p + 4, v + 4);
}
__device__ __forceinline__ void load_eight(const bf16* p, float* v) { unpack_bf16x8(*reinterpret_cast<const uint4*>(p), v); }

template <int N> struct Pow2 { static constexpr int value = 2 * Pow2<(N + 1) / 2>::value; };      // the power of two at least N
template <> struct Pow2<1> { static constexpr int value = 1; };

#define STEP_VEC (SCAN_STATE % 4 == 0 ? 4 : 1)
constexpr int STEP_ALL = Pow2<(SCAN_STATE + STEP_VEC - 1) / STEP_VEC>::value;
constexpr int STEP_LANES = STEP_ALL > 32 ? 32 : STEP_ALL;
#define STEP_MAX_RANK 1024

template <typename T, bool FUSED, int TOGETHER>
__global__ void __launch_bounds__(SCAN_THREADS) selective_step_kernel(
    const T* x, int64_t x_stride, const float* pre, const T* low, const T* __restrict__ dt_weight, int rank, const T* z,
    int64_t z_stride, const T* b, const T* c, int64_t bc_stride, const float* __restrict__ a,
    const float* __restrict__ d, const float* __restrict__ dt_bias, float* __restrict__ state,
    const int* __restrict__ row_starts, const int* __restrict__ state_slots, const int* __restrict__ token_row,
    T* __restrict__ out, int64_t out_stride, int rows, int channels) {
    constexpr int N = SCAN_STATE, VEC = STEP_VEC, LANES = STEP_LANES, CH = SCAN_THREADS / LANES;
    constexpr int CHUNKS = (N + VEC - 1) / VEC, TURNS = (CHUNKS + LANES - 1) / LANES;
    extern __shared__ __align__(16) float low_s[];                    // [TOGETHER][rank]
    const int lane = threadIdx.x % LANES, channel = blockIdx.x * CH + threadIdx.x / LANES;
    const int row0 = blockIdx.y * TOGETHER, here = min(TOGETHER, rows - row0);
    const bool live = channel < channels;
    int token[TOGETHER];
    bool owned[TOGETHER];                         // a padding row of a recorded batch has no request and no state
    float* mine[TOGETHER];
    float s[TOGETHER][TURNS][VEC], dt[TOGETHER];
#pragma unroll
    for (int q = 0; q < TOGETHER; ++q) {
        token[q] = q < here ? row_starts[row0 + q] : -1;
        owned[q] = q < here && token_row[token[q]] >= 0;
        mine[q] = state + ((int64_t)(owned[q] ? state_slots[row0 + q] : 0) * channels + (live ? channel : 0)) * N;
        dt[q] = 0.0f;
#pragma unroll
        for (int i = 0; i < TURNS; ++i)
            if (owned[q] && live && lane + i * LANES < CHUNKS) load_values<VEC>(mine[q] + (lane + i * LANES) * VEC, s[q][i]);
    }
    if constexpr (FUSED) {
        for (int k = threadIdx.x; k < here * rank; k += SCAN_THREADS)
            low_s[k] = to_float<T>(low[(int64_t)row_starts[row0 + k / rank] * bc_stride + k % rank]);
        __syncthreads();
        if (live)
            for (int k0 = lane * 8; k0 < rank; k0 += 4 * LANES * 8) {
                float w[4][8];                    // four accesses to the weights are in flight together
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (k0 + j * LANES * 8 < rank) load_eight(dt_weight + (int64_t)channel * rank + k0 + j * LANES * 8, w[j]);
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (k0 + j * LANES * 8 < rank) {
#pragma unroll
                        for (int q = 0; q < TOGETHER; ++q)
                            if (q < here) {
                                const float* from = low_s + q * rank + k0 + j * LANES * 8;
                                float l[8];
                                load_values<4>(from, l);
                                load_values<4>(from + 4, l + 4);
#pragma unroll
                                for (int i = 0; i < 8; ++i) dt[q] = __fmaf_rn(w[j][i], l[i], dt[q]);
                            }
                    }
            }
#pragma unroll
        for (int bit = LANES / 2; bit >= 1; bit >>= 1)
#pragma unroll
            for (int q = 0; q < TOGETHER; ++q) dt[q] += __shfl_xor_sync(0xffffffffu, dt[q], bit);
    }
    float decay[TURNS][VEC];
#pragma unroll
    for (int i = 0; i < TURNS; ++i)
        if (live && lane + i * LANES < CHUNKS) {
            load_values<VEC>(a + (int64_t)channel * N + (lane + i * LANES) * VEC, decay[i]);
#pragma unroll
            for (int j = 0; j < VEC; ++j) decay[i][j] = Scan<T>::prepare(decay[i][j]);
        }
    const float shift = live && dt_bias ? dt_bias[channel] : 0.0f, skip = live ? d[channel] : 0.0f;
#pragma unroll
    for (int q = 0; q < TOGETHER; ++q) {
        float y = 0.0f, xv = 0.0f;
        if (owned[q] && live) {
            const float step = Scan<T>::softplus(__fadd_rn(FUSED ? dt[q] : pre[(int64_t)token[q] * channels + channel], shift));
            xv = to_float<T>(x[(int64_t)token[q] * x_stride + channel]);
            const float u = __fmul_rn(step, xv);
            const T* b_row = b + (int64_t)token[q] * bc_stride;
            const T* c_row = c + (int64_t)token[q] * bc_stride;
#pragma unroll
            for (int i = 0; i < TURNS; ++i) {
                const int n = (lane + i * LANES) * VEC;
                if (lane + i * LANES < CHUNKS) {
#pragma unroll
                    for (int j = 0; j < VEC; ++j) {
                        s[q][i][j] = __fmaf_rn(Scan<T>::decay(step, decay[i][j]), s[q][i][j], __fmul_rn(u, to_float<T>(b_row[n + j])));
                        y = __fmaf_rn(s[q][i][j], to_float<T>(c_row[n + j]), y);
                    }
                    store_values<VEC>(mine[q] + n, s[q][i]);
                }
            }
        }
#pragma unroll
        for (int bit = LANES / 2; bit >= 1; bit >>= 1) y += __shfl_xor_sync(0xffffffffu, y, bit);
        if (q < here && live && lane == 0) {
            float result = 0.0f;
            if (owned[q])
                result = __fmul_rn(__fmaf_rn(skip, xv, y), silu_for<T>(to_float<T>(z[(int64_t)token[q] * z_stride + channel])));
            out[(int64_t)token[q] * out_stride + channel] = from_float<T>(result);
        }
    }
}

// As tvb_selective_scan, every entry one token.  Either pre (float32 [tokens, channels]) or low (rows `bc_stride`
// apart, as b and c) and dt_weight [channels, rank].
extern "C" int tvb_selective_step(const void* x, long long x_stride, const float* pre, const void* low,
                                  const void* dt_weight, int rank, const void* z, long long z_stride, const void* b,
                                  const void* c, long long bc_stride, const float* a, const float* d,
                                  const float* dt_bias, float* state, const int* row_starts, const int* state_slots,
                                  const int* token_row, void* out, long long out_stride, int rows, int channels,
                                  int dtype, void* stream) {
    if (rows <= 0) return 0;
    if (channels <= 0 || rows > 65535 || !state || !a || !d || (!pre == !dt_weight)) return TVB_BAD_ARGUMENT;
    if (dt_weight && (rank <= 0 || rank % 8 || rank > STEP_MAX_RANK || !low || (uintptr_t)dt_weight % 16)) return TVB_BAD_ARGUMENT;
    if (STEP_VEC == 4 && (((uintptr_t)state | (uintptr_t)a) & 15)) return TVB_BAD_ARGUMENT;
    constexpr int ch = SCAN_THREADS / STEP_LANES;
    const int blocks = (channels + ch - 1) / ch;
    // with the product inside, as many requests a CTA as still give every SM two CTAs
    int together = 1;
    if (dt_weight)
        while (together < 4 && together < rows && (long long)blocks * ((rows + 2 * together - 1) / (2 * together)) >= 2 * 148)
            together *= 2;
    const dim3 grid(blocks, (rows + together - 1) / together);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, F, R) selective_step_kernel<T, F, R><<<grid, SCAN_THREADS, F ? R * rank * sizeof(float) : 0, s>>>(      \
        (const T*)x, x_stride, pre, (const T*)low, (const T*)dt_weight, rank, (const T*)z, z_stride, (const T*)b,    \
        (const T*)c, bc_stride, a, d, dt_bias, state, row_starts, state_slots, token_row, (T*)out, out_stride, rows, channels)
#define BY_ROWS(T)                                                                                                   \
    if (!dt_weight) GO(T, false, 1);                                                                                 \
    else if (together == 1) GO(T, true, 1);                                                                          \
    else if (together == 2) GO(T, true, 2);                                                                          \
    else GO(T, true, 4)
    if (dtype == TVB_F32) { BY_ROWS(float); }
    else if (dtype == TVB_BF16) { BY_ROWS(bf16); }
    else return TVB_BAD_ARGUMENT;
#undef BY_ROWS
#undef GO
    return tvb_last_error();
}

extern "C" int tvb_selective_scan_state() { return SCAN_STATE; }
