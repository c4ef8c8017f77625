// The gated delta rule: a float32 state [dim, vdim] a head and request that corrects what it holds under a key.
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          g, beta: one number a token and head
//
// q and k are unit vectors over a head (q also scaled), shared by the value heads of a group.  With p = S^T k and w =
// S^T q of the state before the token, u = beta (v - g p) and o = g w + (k . q) u: one pass over the state for both
// sums, one for the update.
//
//   delta_prepare   q and k heads of the convolved projection -> float32 unit vectors (rows padded with zeros to a
//                   multiple of four), and per head g, beta and k . q
//   delta_scan      prompts: a CTA walks one entry for a block of value columns of one head; LANES lanes share a column,
//                   a thread holds ROWS rows of it in registers, in pairs for two-wide float32 arithmetic; tokens come
//                   in blocks of DELTA_BLOCK through shared memory, the next block's copies in flight meanwhile.  p is
//                   added over the lanes token by token (the next state waits for it), w a block of tokens at a time
//   delta_step      one token a request: the whole mixer between convolution and output projection in one launch
//
// Unit vectors, decays, step sizes, state and sums are float32 whatever the storage type.
#include "common.cuh"

#define DELTA_THREADS 128
#define DELTA_BLOCK 8

__device__ __forceinline__ float delta_softplus(float z) { return __fadd_rn(fmaxf(z, 0.0f), log1pf(expf(-fabsf(z)))); }
__device__ __forceinline__ float delta_sigmoid(float z) { return __fdiv_rn(1.0f, __fadd_rn(1.0f, expf(-z))); }
// exp(rate softplus(a + bias)), rate = -exp(A_log); taken as 1 + (exp(x) - 1): a head that keeps hundreds of tokens
// multiplies it hundreds of times, and an exponential that is one unit off to one side there would show
__device__ __forceinline__ float delta_decay(float a, float bias, float rate) {
    return __fadd_rn(1.0f, expm1f(__fmul_rn(rate, delta_softplus(__fadd_rn(a, bias)))));
}

// two float32 numbers in one 64-bit register: the arithmetic unit's two-wide forms
__device__ __forceinline__ uint64_t pair_of(float a, float b) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(a), "f"(b));
    return d;
}
__device__ __forceinline__ float pair_sum(uint64_t p) {
    float a, b;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(p));
    return __fadd_rn(a, b);
}
__device__ __forceinline__ uint64_t pair_fma(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t pair_mul(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t pair_add(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// ------------------------------------------------------------------------------------------- prepare
// A warp a (token, key head).
template <typename T>
__global__ void __launch_bounds__(128) delta_prepare_kernel(
    const T* __restrict__ mixed, int64_t mixed_stride, int q_at, int k_at, const T* __restrict__ proj, int64_t proj_stride,
    int beta_at, int decay_at, const float* __restrict__ rate, const float* __restrict__ dt_bias, float q_scale,
    float unit_eps, float* __restrict__ q_out, float* __restrict__ k_out, float4* __restrict__ scalars, int tokens,
    int key_heads, int group, int dim, int padded) {
    const int lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= (int64_t)tokens * key_heads) return;
    const int64_t token = item / key_heads;
    const int kh = (int)(item % key_heads);
    const T* q = mixed + token * mixed_stride + q_at + (int64_t)kh * dim;
    const T* k = mixed + token * mixed_stride + k_at + (int64_t)kh * dim;
    float qq = 0.0f, kk = 0.0f, qk = 0.0f;
    for (int d = lane; d < dim; d += 32) {
        const float a = to_float<T>(q[d]), b = to_float<T>(k[d]);
        qq = __fmaf_rn(a, a, qq);
        kk = __fmaf_rn(b, b, kk);
        qk = __fmaf_rn(a, b, qk);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    const float iq = __fmul_rn(__fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(qq, unit_eps))), q_scale);
    const float ik = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(kk, unit_eps)));
    const int64_t to = item * padded;
    for (int d = lane; d < padded; d += 32) {
        q_out[to + d] = d < dim ? __fmul_rn(to_float<T>(q[d]), iq) : 0.0f;
        k_out[to + d] = d < dim ? __fmul_rn(to_float<T>(k[d]), ik) : 0.0f;
    }
    const T* row = proj + token * proj_stride;
    for (int j = lane; j < group; j += 32) {
        const int head = kh * group + j;
        const float g = delta_decay(to_float<T>(row[decay_at + head]), dt_bias[head], rate[head]);
        const float beta = delta_sigmoid(to_float<T>(row[beta_at + head]));
        scalars[token * key_heads * group + head] = make_float4(g, beta, __fmul_rn(__fmul_rn(qk, iq), ik), 0.0f);
    }
}

// ---------------------------------------------------------------------------------------------- scan
template <typename T, int LANES, int ROWS>
__global__ void __launch_bounds__(DELTA_THREADS) delta_scan_kernel(
    const float* __restrict__ q, const float* __restrict__ k, const float4* __restrict__ scalars, const T* __restrict__ v,
    int64_t v_stride, float* __restrict__ state, const int* __restrict__ row_starts, const int* __restrict__ state_slots,
    const int* __restrict__ token_row, float* __restrict__ out, int heads, int group, int dim, int padded, int vdim) {
    constexpr int COLS = DELTA_THREADS / LANES, WIDTH = LANES * ROWS, QUADS = ROWS / 4, PAIRS = ROWS / 2;
    constexpr int WORDS = DELTA_BLOCK * WIDTH / 4;           // 16-byte words of q (and of k) a block
    constexpr int V_LOADS = (DELTA_BLOCK * COLS + DELTA_THREADS - 1) / DELTA_THREADS;
    __shared__ __align__(16) float q_s[2][DELTA_BLOCK][WIDTH], k_s[2][DELTA_BLOCK][WIDTH];
    __shared__ __align__(16) float4 s_s[2][DELTA_BLOCK];
    __shared__ float v_s[2][DELTA_BLOCK][COLS];
    const int row = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, lane = tid % LANES, mine = tid / LANES;
    const int begin = row_starts[row], count = row_starts[row + 1] - begin;
    if (count <= 0) return;
    const int c = col0 + mine;
    const bool live = c < vdim;
    const int64_t out_stride = (int64_t)heads * vdim;
    float* o = out + (int64_t)begin * out_stride + (int64_t)head * vdim + c;
    if (token_row[begin] < 0) {                   // a padding row of a recorded batch: no request, no state
        if (live)
            for (int t = lane; t < count; t += LANES) o[(int64_t)t * out_stride] = 0.0f;
        return;
    }
    const int key_heads = heads / group;
    const float* q_in = q + ((int64_t)begin * key_heads + head / group) * padded;
    const float* k_in = k + ((int64_t)begin * key_heads + head / group) * padded;
    const float4* s_in = scalars + (int64_t)begin * heads + head;
    const T* v_in = v + (int64_t)begin * v_stride + (int64_t)head * vdim + col0;
    const int64_t key_stride = (int64_t)key_heads * padded;
    float* state_of = state + (((int64_t)state_slots[row] * heads + head) * dim) * vdim + c;

    // rows 4 (lane + LANES j) .. + 3: the lanes of a column read neighbouring 16-byte words of q and k
    uint64_t s[PAIRS];
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
        const int d = 4 * (lane + LANES * (i >> 1)) + 2 * (i & 1);
        s[i] = pair_of(live && d < dim ? state_of[(int64_t)d * vdim] : 0.0f,
                       live && d + 1 < dim ? state_of[(int64_t)(d + 1) * vdim] : 0.0f);
    }
    T v_next[V_LOADS];
    auto copy = [&](int first, int to) {          // tokens first .. first + DELTA_BLOCK - 1; zeros past the end
        for (int e = tid; e < WORDS; e += DELTA_THREADS) {
            const int t = e / (WIDTH / 4), d = e % (WIDTH / 4) * 4;
            const bool ok = first + t < count && d < padded;
            const int64_t at = ok ? (int64_t)(first + t) * key_stride + d : 0;
            cp_async_16(&q_s[to][t][d], q_in + at, ok);
            cp_async_16(&k_s[to][t][d], k_in + at, ok);
        }
        if (tid < DELTA_BLOCK) cp_async_16(&s_s[to][tid], s_in + (first + tid < count ? (int64_t)(first + tid) * heads : 0), first + tid < count);
        cp_async_commit();
    };
    auto fetch = [&](int first) {
#pragma unroll
        for (int j = 0; j < V_LOADS; ++j) {
            const int e = tid + j * DELTA_THREADS, t = e / COLS, cc = e % COLS;
            const bool ok = e < DELTA_BLOCK * COLS && first + t < count && col0 + cc < vdim;
            v_next[j] = ok ? v_in[(int64_t)(first + t) * v_stride + cc] : from_float<T>(0.0f);
        }
    };
    auto stage = [&](int to) {
#pragma unroll
        for (int j = 0; j < V_LOADS; ++j) {
            const int e = tid + j * DELTA_THREADS;
            if (e < DELTA_BLOCK * COLS) v_s[to][e / COLS][e % COLS] = to_float<T>(v_next[j]);
        }
    };
    copy(0, 0);
    fetch(0);
    for (int first = 0, turn = 0; first < count; first += DELTA_BLOCK, turn ^= 1) {
        stage(turn);
        cp_async_wait<0>();
        __syncthreads();                          // this block is there, the one before is read
        if (first + DELTA_BLOCK < count) {
            copy(first + DELTA_BLOCK, turn ^ 1);
            fetch(first + DELTA_BLOCK);
        }
        const int here = min(DELTA_BLOCK, count - first);
        float sums[DELTA_BLOCK], writes[DELTA_BLOCK];
#pragma unroll
        for (int t = 0; t < DELTA_BLOCK; ++t) {
            sums[t] = writes[t] = 0.0f;
            if (t >= here) continue;
            const float4 scalar = s_s[turn][t];
            uint64_t kk[PAIRS], p0 = 0, p1 = 0, w0 = 0, w1 = 0;
#pragma unroll
            for (int j = 0; j < QUADS; ++j) {
                const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(&k_s[turn][t][4 * (lane + LANES * j)]);
                kk[2 * j] = k2.x;
                kk[2 * j + 1] = k2.y;
                p0 = pair_fma(s[2 * j], k2.x, p0);
                p1 = pair_fma(s[2 * j + 1], k2.y, p1);
            }
            float p = pair_sum(pair_add(p0, p1));
#pragma unroll
            for (int j = 0; j < QUADS; ++j) {
                const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(&q_s[turn][t][4 * (lane + LANES * j)]);
                w0 = pair_fma(s[2 * j], q2.x, w0);
                w1 = pair_fma(s[2 * j + 1], q2.y, w1);
            }
#pragma unroll
            for (int bit = LANES / 2; bit >= 1; bit >>= 1) p += __shfl_xor_sync(0xffffffffu, p, bit);
            const float u = __fmul_rn(scalar.y, __fmaf_rn(-scalar.x, p, v_s[turn][t][mine]));
            const uint64_t u2 = pair_of(u, u), g2 = pair_of(scalar.x, scalar.x);
#pragma unroll
            for (int i = 0; i < PAIRS; ++i) s[i] = pair_fma(kk[i], u2, pair_mul(g2, s[i]));
            sums[t] = pair_sum(pair_add(w0, w1));
            writes[t] = u;
        }
        // w of the block's tokens: lanes beyond one a token add plainly, then halving leaves lane l token l % DELTA_BLOCK
        int token = 0;
#pragma unroll
        for (int bit = LANES / 2, n = DELTA_BLOCK; bit >= 1; bit >>= 1) {
            if (bit >= DELTA_BLOCK) {
#pragma unroll
                for (int i = 0; i < DELTA_BLOCK; ++i) sums[i] += __shfl_xor_sync(0xffffffffu, sums[i], bit);
            } else {
                const bool upper = (lane & bit) != 0;
#pragma unroll
                for (int i = 0; i < n / 2; ++i) {
                    const float hand = upper ? sums[i] : sums[i + n / 2], keep = upper ? sums[i + n / 2] : sums[i];
                    sums[i] = keep + __shfl_xor_sync(0xffffffffu, hand, bit);
                }
                if (upper) token += n / 2;
                n >>= 1;
            }
        }
        static_assert(LANES >= DELTA_BLOCK, "delta_scan: a lane a token");
        float u = writes[0];
#pragma unroll
        for (int t = 1; t < DELTA_BLOCK; ++t) u = token == t ? writes[t] : u;
        if (live && token < here && lane < DELTA_BLOCK) {
            const float4 scalar = s_s[turn][token];
            o[(int64_t)(first + token) * out_stride] = __fmaf_rn(scalar.z, u, __fmul_rn(scalar.x, sums[0]));
        }
    }
    if (!live) return;
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
        const int d = 4 * (lane + LANES * (i >> 1)) + 2 * (i & 1);
        float a, b;
        asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(s[i]));
        if (d < dim) state_of[(int64_t)d * vdim] = a;
        if (d + 1 < dim) state_of[(int64_t)(d + 1) * vdim] = b;
    }
}

// ---------------------------------------------------------------------------------------------- step
// A CTA a (request, head).  A thread owns VEC neighbouring columns of the state and one of the slices of its rows, which
// it keeps in registers between the two passes where a slice has at most DELTA_HELD rows.
#define DELTA_STEP_THREADS 256
#define DELTA_HELD 16

struct DeltaStepArgs {
    int64_t mixed_stride, proj_stride, out_stride;
    int q_at, k_at, v_at, beta_at, decay_at, gate_at, gate_act, unit_norm;
    const float *rate, *dt_bias, *norm_weight;
    float q_scale, unit_eps, eps;
    float* state;
    const int *row_starts, *state_slots, *token_row;
    int heads, group, dim, vdim;
};

template <typename T, int VEC, bool HELD>
__global__ void __launch_bounds__(DELTA_STEP_THREADS) delta_step_kernel(const T* __restrict__ mixed, const T* __restrict__ proj,
                                                                        T* __restrict__ out, DeltaStepArgs args) {
    extern __shared__ __align__(16) float step_shared[];
    __shared__ float scratch[32];
    const int dim = args.dim, vdim = args.vdim, row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
    float* q_s = step_shared;                     // [dim]
    float* k_s = q_s + dim;                       // [dim]
    float* u_s = k_s + dim;                       // [vdim]
    float* o_s = u_s + vdim;                      // [vdim]
    float* p_s = o_s + vdim;                      // [slices][columns rounded up to VEC], then the same for w
    const int64_t token = args.row_starts[row];
    T* dst = out + token * args.out_stride + (int64_t)head * vdim;
    if (args.token_row[token] < 0) {              // a padding row of a recorded batch: no request, no state
        for (int c = tid; c < vdim; c += DELTA_STEP_THREADS) dst[c] = from_float<T>(0.0f);
        return;
    }
    const int groups = (vdim + VEC - 1) / VEC, slices = max(1, DELTA_STEP_THREADS / groups);
    const int lead = tid % groups, slice = tid / groups, width = groups * VEC;
    const int per = (dim + slices - 1) / slices, first = slice * per, last = min(dim, first + per);
    const bool works = tid < groups * slices;
    float* mine = args.state + (((int64_t)args.state_slots[row] * args.heads + head) * dim) * vdim + lead * VEC;
    float s[HELD ? DELTA_HELD : 1][VEC];
    if constexpr (HELD) {                         // the whole state is on its way before anything else is looked at
#pragma unroll
        for (int i = 0; i < DELTA_HELD; ++i)
            if (works && first + i < last) load_values<VEC>(mine + (int64_t)(first + i) * vdim, s[i]);
    }
    const T* src = mixed + token * args.mixed_stride;
    const T* other = proj + token * args.proj_stride;
    const int key_at = head / args.group * dim;
    float qq = 0.0f, kk = 0.0f, qk = 0.0f;
    for (int d = tid; d < dim; d += DELTA_STEP_THREADS) {
        const float a = to_float<T>(src[args.q_at + key_at + d]), b = to_float<T>(src[args.k_at + key_at + d]);
        q_s[d] = a;
        k_s[d] = b;
        qq = __fmaf_rn(a, a, qq);
        kk = __fmaf_rn(b, b, kk);
        qk = __fmaf_rn(a, b, qk);
    }
    qq = block_sum(qq, scratch);
    kk = block_sum(kk, scratch);
    qk = block_sum(qk, scratch);                  // q_s and k_s are there for everyone
    const float iq = __fmul_rn(__fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(qq, args.unit_eps))), args.q_scale);
    const float ik = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(kk, args.unit_eps)));
    const float kq = __fmul_rn(__fmul_rn(qk, iq), ik);
    const float g = delta_decay(to_float<T>(other[args.decay_at + head]), args.dt_bias[head], args.rate[head]);
    const float beta = delta_sigmoid(to_float<T>(other[args.beta_at + head]));
    if (works) {
        float p[VEC], w[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) p[j] = w[j] = 0.0f;
        auto add = [&](const float* x, int d) {
            const float kd = __fmul_rn(k_s[d], ik), qd = __fmul_rn(q_s[d], iq);
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                p[j] = __fmaf_rn(x[j], kd, p[j]);
                w[j] = __fmaf_rn(x[j], qd, w[j]);
            }
        };
        if constexpr (HELD) {
#pragma unroll
            for (int i = 0; i < DELTA_HELD; ++i)
                if (first + i < last) add(s[i], first + i);
        } else {
            for (int d = first; d < last; ++d) {
                float x[VEC];
                load_values<VEC>(mine + (int64_t)d * vdim, x);
                add(x, d);
            }
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            p_s[slice * width + lead * VEC + j] = p[j];
            p_s[(slices + slice) * width + lead * VEC + j] = w[j];
        }
    }
    __syncthreads();
    float part = 0.0f;
    for (int c = tid; c < vdim; c += DELTA_STEP_THREADS) {
        float p = 0.0f, w = 0.0f;
        for (int sl = 0; sl < slices; ++sl) {
            p = __fadd_rn(p, p_s[sl * width + c]);
            w = __fadd_rn(w, p_s[(slices + sl) * width + c]);
        }
        const float u = __fmul_rn(beta, __fmaf_rn(-g, p, to_float<T>(src[args.v_at + (int64_t)head * vdim + c])));
        const float o = __fmaf_rn(kq, u, __fmul_rn(g, w));
        u_s[c] = u;
        o_s[c] = o;
        part = __fmaf_rn(o, o, part);
    }
    const float squares = block_sum(part, scratch);           // u_s and o_s are there for everyone
    if (works) {
        float u[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = lead * VEC + j < vdim ? u_s[lead * VEC + j] : 0.0f;
        auto move = [&](float* x, int d) {
            const float kd = __fmul_rn(k_s[d], ik);
#pragma unroll
            for (int j = 0; j < VEC; ++j) x[j] = __fmaf_rn(kd, u[j], __fmul_rn(g, x[j]));
            store_values<VEC>(mine + (int64_t)d * vdim, x);
        };
        if constexpr (HELD) {
#pragma unroll
            for (int i = 0; i < DELTA_HELD; ++i)
                if (first + i < last) move(s[i], first + i);
        } else {
            for (int d = first; d < last; ++d) {
                float x[VEC];
                load_values<VEC>(mine + (int64_t)d * vdim, x);
                move(x, d);
            }
        }
    }
    const float factor = args.unit_norm ? __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(squares, (float)vdim), args.eps))) : 1.0f;
    for (int c = tid; c < vdim; c += DELTA_STEP_THREADS) {
        float x = __fmul_rn(o_s[c], factor);
        if (args.norm_weight) x = __fmul_rn(x, args.norm_weight[c]);
        if (args.gate_at >= 0) {
            const float z = to_float<T>(other[args.gate_at + (int64_t)head * vdim + c]);
            x = __fmul_rn(x, args.gate_act == 1 ? __fmul_rn(z, delta_sigmoid(z)) : args.gate_act == 2 ? delta_sigmoid(z) : z);
        }
        dst[c] = from_float<T>(x);
    }
}

// mixed: [tokens, >= columns] of the storage type, q heads from q_at, k heads from k_at (key_heads of `dim` each); proj:
// the same rows with one number a head from beta_at and decay_at on; rate, dt_bias float32 [heads]; q_out, k_out float32
// [tokens, key_heads, padded], padded a multiple of four at least dim; scalars float32 [tokens, heads, 4].
extern "C" int tvb_delta_prepare(const void* mixed, long long mixed_stride, int q_at, int k_at, const void* proj,
                                 long long proj_stride, int beta_at, int decay_at, const float* rate, const float* dt_bias,
                                 float q_scale, float unit_eps, float* q_out, float* k_out, float* scalars, int tokens,
                                 int key_heads, int group, int dim, int padded, int dtype, void* stream) {
    if (tokens <= 0) return 0;
    if (key_heads <= 0 || group <= 0 || dim <= 0 || padded < dim || padded % 4 || (uintptr_t)scalars % 16) return TVB_BAD_ARGUMENT;
    const long long blocks = ((long long)tokens * key_heads + 3) / 4;
    if (blocks > 2147483647LL) return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T) delta_prepare_kernel<T><<<(unsigned)blocks, 128, 0, s>>>(                                                 \
        (const T*)mixed, mixed_stride, q_at, k_at, (const T*)proj, proj_stride, beta_at, decay_at, rate, dt_bias, q_scale, \
        unit_eps, q_out, k_out, (float4*)scalars, tokens, key_heads, group, dim, padded)
    if (dtype == TVB_F32) GO(float);
    else if (dtype == TVB_BF16) GO(bf16);
    else return TVB_BAD_ARGUMENT;
#undef GO
    return tvb_last_error();
}

// q, k, scalars as delta_prepare leaves them; v: [tokens, heads * vdim] of the storage type, rows `v_stride` apart; state
// float32 [slots, heads, dim, vdim]; out float32 [tokens, heads * vdim].
extern "C" int tvb_delta_scan(const float* q, const float* k, const float* scalars, const void* v, long long v_stride,
                              float* state, const int* row_starts, const int* state_slots, const int* token_row, float* out,
                              int rows, int heads, int group, int dim, int padded, int vdim, int dtype, void* stream) {
    if (rows <= 0) return 0;
    if (heads <= 0 || heads > 65535 || group <= 0 || heads % group || dim <= 0 || dim > 256 || padded < dim || padded % 4 ||
        vdim <= 0 || !state || ((uintptr_t)q | (uintptr_t)k | (uintptr_t)scalars) % 16)
        return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T, LANES, ROWS) {                                                                                            \
        const dim3 grid(rows, heads, (vdim + DELTA_THREADS / LANES - 1) / (DELTA_THREADS / LANES));                     \
        if (grid.z > 65535) return TVB_BAD_ARGUMENT;                                                                    \
        delta_scan_kernel<T, LANES, ROWS><<<grid, DELTA_THREADS, 0, s>>>(q, k, (const float4*)scalars, (const T*)v,     \
            v_stride, state, row_starts, state_slots, token_row, out, heads, group, dim, padded, vdim); }
#define BY_DIM(T)                          \
    if (dim <= 32) GO(T, 8, 4)             \
    else if (dim <= 64) GO(T, 8, 8)        \
    else if (dim <= 128) GO(T, 8, 16)      \
    else GO(T, 16, 16)
    if (dtype == TVB_F32) { BY_DIM(float) }
    else if (dtype == TVB_BF16) { BY_DIM(bf16) }
    else return TVB_BAD_ARGUMENT;
#undef BY_DIM
#undef GO
    return tvb_last_error();
}

// As the two above together with the norm over a head and the gate, every entry of row_starts one token; out [tokens,
// heads * vdim] of the storage type.  gate_at < 0: no gate; gate_act 0 none, 1 SiLU, 2 sigmoid.
extern "C" int tvb_delta_step(const void* mixed, long long mixed_stride, int q_at, int k_at, int v_at, const void* proj,
                              long long proj_stride, int beta_at, int decay_at, int gate_at, int gate_act, const float* rate,
                              const float* dt_bias, float q_scale, float unit_eps, const float* norm_weight, int unit_norm,
                              float eps, float* state, const int* row_starts, const int* state_slots, const int* token_row,
                              void* out, long long out_stride, int rows, int heads, int group, int dim, int vdim, int dtype,
                              void* stream) {
    if (rows <= 0) return 0;
    if (heads <= 0 || heads > 65535 || group <= 0 || heads % group || dim <= 0 || dim > 256 || vdim <= 0 || !state)
        return TVB_BAD_ARGUMENT;
    const bool by_four = vdim % 4 == 0 && ((uintptr_t)state & 15) == 0;
    const int vec = by_four ? 4 : 1, groups = (vdim + vec - 1) / vec;
    if (groups > DELTA_STEP_THREADS) return TVB_BAD_ARGUMENT;
    const int slices = DELTA_STEP_THREADS / groups;
    const bool held = (dim + slices - 1) / slices <= DELTA_HELD;
    const size_t smem = (size_t)(2 * dim + 2 * vdim + 2 * slices * groups * vec) * sizeof(float);
    if (smem > 48 * 1024) return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const DeltaStepArgs args{mixed_stride, proj_stride, out_stride, q_at, k_at, v_at, beta_at, decay_at, gate_at, gate_act,
                             unit_norm, rate, dt_bias, norm_weight, q_scale, unit_eps, eps, state, row_starts, state_slots,
                             token_row, heads, group, dim, vdim};
    const dim3 grid(rows, heads);
#define GO(T, V, H) delta_step_kernel<T, V, H><<<grid, DELTA_STEP_THREADS, smem, s>>>((const T*)mixed, (const T*)proj, (T*)out, args)
#define BY_FORM(T)                                                                        \
    if (by_four) { if (held) GO(T, 4, true); else GO(T, 4, false); }                      \
    else { if (held) GO(T, 1, true); else GO(T, 1, false); }
    if (dtype == TVB_F32) { BY_FORM(float) }
    else if (dtype == TVB_BF16) { BY_FORM(bf16) }
    else return TVB_BAD_ARGUMENT;
#undef BY_FORM
#undef GO
    return tvb_last_error();
}
