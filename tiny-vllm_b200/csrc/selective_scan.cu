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
#define SCAN_LOG2E 1.4426950408889634f

static_assert(SCAN_STATE >= 1 && SCAN_STATE <= 256, "selective_scan: state size");

__device__ __forceinline__ float softplus(float z) { return __fadd_rn(fmaxf(z, 0.0f), log1pf(expf(-fabsf(z)))); }
__device__ __forceinline__ float silu_of(float z) { return __fdiv_rn(z, __fadd_rn(1.0f, expf(-z))); }

// exp(dt * a): with 16-bit storage the exponential unit's 2^x on dt * (a log2 e), `a` being stored so
template <typename T> struct Decay;
template <> struct Decay<float> {
    static __device__ __forceinline__ float prepare(float a) { return a; }
    static __device__ __forceinline__ float of(float dt, float a) { return expf(__fmul_rn(dt, a)); }
};
template <> struct Decay<bf16> {
    static __device__ __forceinline__ float prepare(float a) { return __fmul_rn(a, SCAN_LOG2E); }
    static __device__ __forceinline__ float of(float dt, float a) {
        float y;
        asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(__fmul_rn(dt, a)));
        return y;
    }
};

// LANES lanes share a channel, a lane holds ROWS neighbouring numbers of its state.  Shared memory holds dt and
// dt * x by channel and B and C by state number, four tokens to a 16-byte access.  A lane's partial sums of y are
// added by halving: at every step a lane hands half of its sums to the lane one bit away and keeps the other half,
// so that lane g ends with complete sums of SUB / LANES tokens.
template <typename T, int LANES>
__global__ void __launch_bounds__(SCAN_THREADS) selective_scan_kernel(
    const T* __restrict__ x, int64_t x_stride, const float* __restrict__ pre, const T* __restrict__ z, int64_t z_stride,
    const T* __restrict__ b, const T* __restrict__ c, int64_t bc_stride, const float* __restrict__ a,
    const float* __restrict__ d, const float* __restrict__ dt_bias, float* __restrict__ state,
    const int* __restrict__ row_starts, const int* __restrict__ state_slots, const int* __restrict__ token_row,
    T* __restrict__ out, int64_t out_stride, int channels) {
    constexpr int N = SCAN_STATE, ROWS = (N + LANES - 1) / LANES, CH = SCAN_THREADS / LANES;
    constexpr int SUB = LANES > 8 ? LANES : 8, LEFT = SUB / LANES, WIDTH = SCAN_BLOCK + SCAN_PAD;
    constexpr int PER = SCAN_BLOCK * CH / SCAN_THREADS;               // (token, channel) pairs a thread moves
    constexpr int BC = (SCAN_BLOCK * N + SCAN_THREADS - 1) / SCAN_THREADS;
    constexpr bool AHEAD = BC <= 16;                                  // B and C of the next block wait in registers
    static_assert(SCAN_BLOCK % SUB == 0 && PER * LANES == SCAN_BLOCK, "selective_scan: tile");
    __shared__ __align__(16) float dt_s[CH][WIDTH];
    __shared__ __align__(16) float u_s[CH][WIDTH];                    // dt * x, then y
    __shared__ __align__(16) float b_s[LANES * ROWS][WIDTH];
    __shared__ __align__(16) float c_s[LANES * ROWS][WIDTH];
    const int row = blockIdx.y, tid = threadIdx.x, lane = tid % LANES, mine = tid / LANES;
    const int begin = row_starts[row], count = row_starts[row + 1] - begin;
    if (count <= 0) return;
    const int c0 = blockIdx.x * CH;
    const int move_ch = tid % CH, move_t = tid / CH;                  // this thread's channel when it moves values
    const bool live = c0 + move_ch < channels;
    T* dst = out + (int64_t)begin * out_stride + c0 + move_ch;
    if (token_row[begin] < 0) {                   // a padding row of a recorded batch: no request, no state
        if (live)
            for (int t = move_t; t < count; t += SCAN_THREADS / CH) dst[(int64_t)t * out_stride] = from_float<T>(0.0f);
        return;
    }
    const int channel = c0 + mine;
    float* state_row = state + ((int64_t)state_slots[row] * channels + channel) * N + lane * ROWS;
    float s[ROWS], decay[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const bool has = channel < channels && lane * ROWS + r < N;
        s[r] = has ? state_row[r] : 0.0f;
        decay[r] = has ? Decay<T>::prepare(a[(int64_t)channel * N + lane * ROWS + r]) : 0.0f;
    }
    if (LANES * ROWS > N)
        for (int e = tid; e < (LANES * ROWS - N) * SCAN_BLOCK; e += SCAN_THREADS) {
            b_s[N + e / SCAN_BLOCK][e % SCAN_BLOCK] = 0.0f;
            c_s[N + e / SCAN_BLOCK][e % SCAN_BLOCK] = 0.0f;
        }
    const float skip = live ? d[c0 + move_ch] : 0.0f, shift = live && dt_bias ? dt_bias[c0 + move_ch] : 0.0f;
    const T* x_in = x + (int64_t)begin * x_stride + c0 + move_ch;
    const T* z_in = z + (int64_t)begin * z_stride + c0 + move_ch;
    const float* pre_in = pre + (int64_t)begin * channels + c0 + move_ch;
    const T* b_in = b + (int64_t)begin * bc_stride;
    const T* c_in = c + (int64_t)begin * bc_stride;

    float x_next[PER], z_next[PER], p_next[PER], b_next[AHEAD ? BC : 1], c_next[AHEAD ? BC : 1];
    auto fetch = [&](int first) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = first + move_t + j * (SCAN_THREADS / CH);
            const bool ok = live && t < count;
            x_next[j] = ok ? to_float<T>(x_in[(int64_t)t * x_stride]) : 0.0f;
            z_next[j] = ok ? to_float<T>(z_in[(int64_t)t * z_stride]) : 0.0f;
            p_next[j] = ok ? pre_in[(int64_t)t * channels] : 0.0f;
        }
        if constexpr (AHEAD) {
#pragma unroll
            for (int j = 0; j < BC; ++j) {
                const int e = tid + j * SCAN_THREADS, t = first + e / N;
                const bool ok = e < SCAN_BLOCK * N && t < count;
                b_next[j] = ok ? to_float<T>(b_in[(int64_t)t * bc_stride + e % N]) : 0.0f;
                c_next[j] = ok ? to_float<T>(c_in[(int64_t)t * bc_stride + e % N]) : 0.0f;
            }
        }
    };

    fetch(0);
    for (int first = 0; first < count; first += SCAN_BLOCK) {
        __syncthreads();                          // the block before is read
        float x_now[PER], z_now[PER];
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = move_t + j * (SCAN_THREADS / CH);
            // tokens past the end move nothing: dt = 0 keeps the state as it is
            const float dt = live && first + t < count ? softplus(__fadd_rn(p_next[j], shift)) : 0.0f;
            dt_s[move_ch][t] = dt;
            u_s[move_ch][t] = __fmul_rn(dt, x_next[j]);
            x_now[j] = x_next[j];
            z_now[j] = z_next[j];
        }
        if constexpr (AHEAD) {
#pragma unroll
            for (int j = 0; j < BC; ++j) {
                const int e = tid + j * SCAN_THREADS;
                if (e < SCAN_BLOCK * N) { b_s[e % N][e / N] = b_next[j]; c_s[e % N][e / N] = c_next[j]; }
            }
        } else {
            for (int e = tid; e < SCAN_BLOCK * N; e += SCAN_THREADS) {
                const int t = first + e / N;
                b_s[e % N][e / N] = t < count ? to_float<T>(b_in[(int64_t)t * bc_stride + e % N]) : 0.0f;
                c_s[e % N][e / N] = t < count ? to_float<T>(c_in[(int64_t)t * bc_stride + e % N]) : 0.0f;
            }
        }
        __syncthreads();
        if (first + SCAN_BLOCK < count) fetch(first + SCAN_BLOCK);
#pragma unroll 1
        for (int sub = 0; sub < SCAN_BLOCK && first + sub < count; sub += SUB) {
            float sums[SUB];
#pragma unroll
            for (int i = 0; i < SUB; ++i) sums[i] = 0.0f;
#pragma unroll
            for (int t = 0; t < SUB; t += 4) {
                const float4 dt4 = *reinterpret_cast<const float4*>(&dt_s[mine][sub + t]);
                const float4 u4 = *reinterpret_cast<const float4*>(&u_s[mine][sub + t]);
                const float dt[4] = {dt4.x, dt4.y, dt4.z, dt4.w}, u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    const float4 b4 = *reinterpret_cast<const float4*>(&b_s[lane * ROWS + r][sub + t]);
                    const float4 c4 = *reinterpret_cast<const float4*>(&c_s[lane * ROWS + r][sub + t]);
                    const float bb[4] = {b4.x, b4.y, b4.z, b4.w}, cc[4] = {c4.x, c4.y, c4.z, c4.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        s[r] = __fmaf_rn(Decay<T>::of(dt[i], decay[r]), s[r], __fmul_rn(u[i], bb[i]));
                        sums[t + i] = __fmaf_rn(s[r], cc[i], sums[t + i]);
                    }
                }
            }
#pragma unroll
            for (int bit = LANES / 2, n = SUB; bit >= 1; bit >>= 1, n >>= 1) {
                const bool upper = (lane & bit) != 0;
#pragma unroll
                for (int i = 0; i < n / 2; ++i) {
                    const float hand = upper ? sums[i] : sums[i + n / 2];
                    const float keep = upper ? sums[i + n / 2] : sums[i];
                    sums[i] = keep + __shfl_xor_sync(0xffffffffu, hand, bit);
                }
            }
            __syncwarp();                         // the channel's lanes have read dt * x of these tokens
#pragma unroll
            for (int i = 0; i < LEFT; ++i) u_s[mine][sub + lane * LEFT + i] = sums[i];
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = move_t + j * (SCAN_THREADS / CH);
            if (live && first + t < count)
                dst[(int64_t)(first + t) * out_stride] =
                    from_float<T>(__fmul_rn(__fmaf_rn(skip, x_now[j], u_s[move_ch][t]), silu_of(z_now[j])));
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
        if (channel < channels && lane * ROWS + r < N) state_row[r] = s[r];
}

// x: [tokens, >= channels]; pre float32 [tokens, channels]; z, b, c as x, each with a row stride; a float32
// [channels, SCAN_STATE]; d, dt_bias float32 [channels]; state float32 [slots, channels, SCAN_STATE]; out
// [tokens, >= channels].  `lanes` (0: chosen): 2, 4, 8 or 16 lanes a channel, at most 16 state numbers a lane.
extern "C" int tvb_selective_scan(const void* x, long long x_stride, const float* pre, const void* z, long long z_stride,
                                  const void* b, const void* c, long long bc_stride, const float* a, const float* d,
                                  const float* dt_bias, float* state, const int* row_starts, const int* state_slots,
                                  const int* token_row, void* out, long long out_stride, int rows, int channels,
                                  int lanes, int dtype, void* stream) {
    if (rows <= 0) return 0;
    if (channels <= 0 || rows > 65535 || !state || !a || !d || !pre) return TVB_BAD_ARGUMENT;
    if (lanes == 0) {                             // the fewest with at most 16 numbers a lane, more while SMs would idle
        for (lanes = 2; lanes < 16 && lanes * 16 < SCAN_STATE; lanes *= 2) {}
        while (lanes < 16 && lanes < SCAN_STATE &&
               (long long)rows * ((channels + SCAN_THREADS / lanes - 1) / (SCAN_THREADS / lanes)) < 2 * 148)
            lanes *= 2;
    }
    if ((lanes != 2 && lanes != 4 && lanes != 8 && lanes != 16) || lanes * 16 < SCAN_STATE) return TVB_BAD_ARGUMENT;
    const int ch = SCAN_THREADS / lanes;
    const dim3 grid((channels + ch - 1) / ch, rows);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, L) selective_scan_kernel<T, L><<<grid, SCAN_THREADS, 0, s>>>(                                          \
        (const T*)x, x_stride, pre, (const T*)z, z_stride, (const T*)b, (const T*)c, bc_stride, a, d, dt_bias, state, \
        row_starts, state_slots, token_row, (T*)out, out_stride, channels)
#define BY_LANES(T)                                                                   \
    if (lanes == 16) GO(T, 16);                                                       \
    else if constexpr (SCAN_STATE <= 128) {                                           \
        if (lanes == 8) GO(T, 8);                                                     \
        else if constexpr (SCAN_STATE <= 64) {                                        \
            if (lanes == 4) GO(T, 4);                                                 \
            else if constexpr (SCAN_STATE <= 32) GO(T, 2);                            \
        }                                                                             \
    }
    if (dtype == TVB_F32) { BY_LANES(float) }
    else if (dtype == TVB_BF16) { BY_LANES(bf16) }
    else return TVB_BAD_ARGUMENT;
#undef BY_LANES
#undef GO
    return tvb_last_error();
}

// One token a request.  The lanes of a channel take its state VEC numbers at a time.  With `dt_weight` the step
// size's product is done here too: pre_c = sum_k low_k W[c, k], low being `rank` numbers a token (rank a multiple
// of 8, rows of W 16-byte aligned in 16-bit storage).
template <typename T> __device__ __forceinline__ float dot8(const T* w, const float* low);
template <> __device__ __forceinline__ float dot8<float>(const float* w, const float* low) {
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) sum = __fmaf_rn(w[i], low[i], sum);
    return sum;
}
template <> __device__ __forceinline__ float dot8<bf16>(const bf16* w, const float* low) {
    float v[8], sum = 0.0f;
    unpack_bf16x8(*reinterpret_cast<const uint4*>(w), v);
#pragma unroll
    for (int i = 0; i < 8; ++i) sum = __fmaf_rn(v[i], low[i], sum);
    return sum;
}

template <int N> struct Pow2 { static constexpr int value = 2 * Pow2<(N + 1) / 2>::value; };      // the power of two at least N
template <> struct Pow2<1> { static constexpr int value = 1; };

#define STEP_VEC (SCAN_STATE % 4 == 0 ? 4 : 1)
constexpr int STEP_ALL = Pow2<(SCAN_STATE + STEP_VEC - 1) / STEP_VEC>::value;
constexpr int STEP_LANES = STEP_ALL > 32 ? 32 : STEP_ALL;
#define STEP_MAX_RANK 1024

template <typename T, bool FUSED>
__global__ void __launch_bounds__(SCAN_THREADS) selective_step_kernel(
    const T* x, int64_t x_stride, const float* pre, const T* low, const T* __restrict__ dt_weight, int rank, const T* z,
    int64_t z_stride, const T* b, const T* c, int64_t bc_stride, const float* __restrict__ a,
    const float* __restrict__ d, const float* __restrict__ dt_bias, float* __restrict__ state,
    const int* __restrict__ row_starts, const int* __restrict__ state_slots, const int* __restrict__ token_row,
    T* __restrict__ out, int64_t out_stride, int channels) {
    constexpr int N = SCAN_STATE, VEC = STEP_VEC, LANES = STEP_LANES, CH = SCAN_THREADS / LANES;
    constexpr int CHUNKS = (N + VEC - 1) / VEC, TURNS = (CHUNKS + LANES - 1) / LANES;
    extern __shared__ __align__(16) float low_s[];
    const int row = blockIdx.y, lane = threadIdx.x % LANES;
    const int channel = blockIdx.x * CH + threadIdx.x / LANES;
    const int token = row_starts[row];
    const bool live = channel < channels;
    if (token_row[token] < 0) {                   // a padding row of a recorded batch: no request, no state
        if (live && lane == 0) out[(int64_t)token * out_stride + channel] = from_float<T>(0.0f);
        return;
    }
    float* mine = state + ((int64_t)state_slots[row] * channels + (live ? channel : 0)) * N;
    float s[TURNS][VEC];
#pragma unroll
    for (int i = 0; i < TURNS; ++i)
        if (live && lane + i * LANES < CHUNKS) load_values<VEC>(mine + (lane + i * LANES) * VEC, s[i]);
    float dt = 0.0f;
    if constexpr (FUSED) {
        for (int k = threadIdx.x; k < rank; k += SCAN_THREADS) low_s[k] = to_float<T>(low[(int64_t)token * bc_stride + k]);
        __syncthreads();
        if (live)
            for (int k = lane * 8; k < rank; k += LANES * 8) dt += dot8<T>(dt_weight + (int64_t)channel * rank + k, low_s + k);
#pragma unroll
        for (int bit = LANES / 2; bit >= 1; bit >>= 1) dt += __shfl_xor_sync(0xffffffffu, dt, bit);
    } else if (live) dt = pre[(int64_t)token * channels + channel];
    float y = 0.0f, xv = 0.0f;
    if (live) {
        dt = softplus(dt_bias ? __fadd_rn(dt, dt_bias[channel]) : dt);
        xv = to_float<T>(x[(int64_t)token * x_stride + channel]);
        const float u = __fmul_rn(dt, xv);
#pragma unroll
        for (int i = 0; i < TURNS; ++i) {
            const int n = (lane + i * LANES) * VEC;
            if (lane + i * LANES < CHUNKS) {
                float av[VEC];
                load_values<VEC>(a + (int64_t)channel * N + n, av);
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    const float bn = to_float<T>(b[(int64_t)token * bc_stride + n + j]);
                    const float cn = to_float<T>(c[(int64_t)token * bc_stride + n + j]);
                    s[i][j] = __fmaf_rn(Decay<T>::of(dt, Decay<T>::prepare(av[j])), s[i][j], __fmul_rn(u, bn));
                    y = __fmaf_rn(s[i][j], cn, y);
                }
                store_values<VEC>(mine + n, s[i]);
            }
        }
    }
#pragma unroll
    for (int bit = LANES / 2; bit >= 1; bit >>= 1) y += __shfl_xor_sync(0xffffffffu, y, bit);
    if (live && lane == 0)
        out[(int64_t)token * out_stride + channel] = from_float<T>(
            __fmul_rn(__fmaf_rn(d[channel], xv, y), silu_of(to_float<T>(z[(int64_t)token * z_stride + channel]))));
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
    const dim3 grid((channels + ch - 1) / ch, rows);
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, F) selective_step_kernel<T, F><<<grid, SCAN_THREADS, F ? rank * sizeof(float) : 0, s>>>(               \
        (const T*)x, x_stride, pre, (const T*)low, (const T*)dt_weight, rank, (const T*)z, z_stride, (const T*)b,    \
        (const T*)c, bc_stride, a, d, dt_bias, state, row_starts, state_slots, token_row, (T*)out, out_stride, channels)
    if (dtype == TVB_F32) { if (dt_weight) GO(float, true); else GO(float, false); }
    else if (dtype == TVB_BF16) { if (dt_weight) GO(bf16, true); else GO(bf16, false); }
    else return TVB_BAD_ARGUMENT;
#undef GO
    return tvb_last_error();
}

extern "C" int tvb_selective_scan_state() { return SCAN_STATE; }
