// The gated delta rule: a float32 state [dim, vdim] a head and request that corrects what it holds under a key.
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          g, beta: one number a token and head
//
// q and k are unit vectors over a head (q also scaled), shared by the value heads of a group.
//
//   delta_prepare   q and k heads of the convolved projection -> float32 unit vectors (rows padded with zeros to a
//                   multiple of four); and per piece of DELTA_BLOCK tokens of an entry and head, how its tokens act on
//                   one another.  With S the state before the piece, G_t the product of its decays up to and with token
//                   t, D_ts that of the decays behind token s up to and with t, the writes of a piece solve
//                     u_t + sum_{s < t} beta_t D_ts (k_s . k_t) u_s = r_t,     r_t = beta_t v_t - beta_t G_t S^T k_t
//                   With T the inverse of that lower triangle (its entries are at most 1 in size: they are products of
//                   k_t, of contractions and of k_s),
//                     o_t = G_t S^T q_t + sum_s M_ts r_s,        M = (D_ts (k_s . q_t))_{s <= t} T
//                     S  <- G_last S + sum_t k_t u'_t^T,         u'_t = D_last,t sum_s T_ts r_s
//   delta_scan      prompts: a CTA walks one entry for a block of value columns of one head, piece by piece; LANES lanes
//                   share COLS columns, a thread holds ROWS rows of them in registers, in pairs for two-wide float32
//                   arithmetic.  All of a piece's sums over the state are taken at once and added by halving over the
//                   lanes, which leaves a lane one token's sums of one or two columns; from them the lanes make the
//                   piece's outputs and writes; the state is read and written once a piece.  The next piece's copies are
//                   in flight meanwhile
//   delta_step      one token a request: the whole mixer between convolution and output projection in one launch.  With
//                   p = S^T k and w = S^T q of the state before the token, u = beta (v - g p) and o = g w + (k . q) u
//
// Unit vectors, decays, step sizes, products between tokens, state and sums are float32 whatever the storage type.
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
// coefficients of a piece and head: beta [8], beta_t G_t [8], G_t [8], then (D_last,t T_ts) [8][8] and M [8][8]
#define DELTA_COEFFICIENTS (3 * DELTA_BLOCK + 2 * DELTA_BLOCK * DELTA_BLOCK)
#define DELTA_MAX_DIM 256

// The piece of an entry that block `index` takes: pieces are counted through the entries in order.
__device__ __forceinline__ bool piece_of(const int* row_starts, int rows, int index, int& row, int& begin, int& count) {
    int before = 0, tokens = 0;
    for (row = 0; row < rows; ++row) {
        tokens = row_starts[row + 1] - row_starts[row];
        const int pieces = (tokens + DELTA_BLOCK - 1) / DELTA_BLOCK;
        if (index < before + pieces) break;
        before += pieces;
    }
    if (row == rows) return false;                // the grid is as large as the pieces can be many
    const int first = (index - before) * DELTA_BLOCK;
    begin = row_starts[row] + first;
    count = min(DELTA_BLOCK, tokens - first);
    return true;
}

// A CTA a (piece, key head).
template <typename T>
__global__ void __launch_bounds__(128) delta_prepare_kernel(
    const T* __restrict__ mixed, int64_t mixed_stride, int q_at, int k_at, const T* __restrict__ proj, int64_t proj_stride,
    int beta_at, int decay_at, const float* __restrict__ rate, const float* __restrict__ dt_bias, float q_scale,
    float unit_eps, float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ coefficients,
    const int* __restrict__ row_starts, const int* __restrict__ token_row, int rows, int key_heads, int group, int dim,
    int padded) {
    constexpr int N = DELTA_BLOCK, STRIDE = DELTA_MAX_DIM + 4;
    __shared__ __align__(16) float vectors[2 * N][STRIDE];           // k of the piece's tokens, then q
    __shared__ float kk[N][N], qk[N][N];
    __shared__ float below[4][N][N], through[4][N][N], inverse_s[4][N][N], last_s[4][N];     // a warp's head
    const int kh = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int row, begin, count;
    if (!piece_of(row_starts, rows, blockIdx.x, row, begin, count) || token_row[begin] < 0) return;
    for (int v = warp; v < 2 * N; v += 4) {
        const int t = v % N;
        const bool is_key = v < N;
        if (t >= count) {
            for (int d = lane; d < padded; d += 32) vectors[v][d] = 0.0f;
            continue;
        }
        const T* src = mixed + (int64_t)(begin + t) * mixed_stride + (is_key ? k_at : q_at) + (int64_t)kh * dim;
        float squares = 0.0f;
        for (int d = lane; d < dim; d += 32) {
            const float x = to_float<T>(src[d]);
            vectors[v][d] = x;
            squares = __fmaf_rn(x, x, squares);
        }
        squares = warp_sum(squares);
        float inverse = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(squares, unit_eps)));
        if (!is_key) inverse = __fmul_rn(inverse, q_scale);
        float* dst = (is_key ? k_out : q_out) + ((int64_t)(begin + t) * key_heads + kh) * padded;
        for (int d = lane; d < padded; d += 32) {                    // a thread reads back only what it wrote
            const float x = d < dim ? __fmul_rn(vectors[v][d], inverse) : 0.0f;
            vectors[v][d] = x;
            dst[d] = x;
        }
    }
    __syncthreads();
    {                                             // one of the 2 * 64 products between the piece's vectors a thread
        const bool is_key = threadIdx.x < N * N;
        const int t = threadIdx.x / N % N, s = threadIdx.x % N;
        float sum = 0.0f;
        if (s <= t)
            for (int d = 0; d < padded; d += 4) {
                const float4 a = *reinterpret_cast<const float4*>(&vectors[s][d]);
                const float4 b = *reinterpret_cast<const float4*>(&vectors[is_key ? t : N + t][d]);
                sum = __fmaf_rn(a.x, b.x, __fmaf_rn(a.y, b.y, __fmaf_rn(a.z, b.z, __fmaf_rn(a.w, b.w, sum))));
            }
        (is_key ? kk : qk)[t][s] = sum;
    }
    __syncthreads();
    for (int j = warp; j < group; j += 4) {       // a warp a head
        const int head = kh * group + j;
        // lane t holds token t's numbers; tokens past the end write nothing and decay nothing
        const bool ok = lane < count;
        const T* src = proj + (int64_t)(begin + (ok ? lane : 0)) * proj_stride;
        const float g = ok ? delta_decay(to_float<T>(src[decay_at + head]), dt_bias[head], rate[head]) : 1.0f;
        const float beta = ok ? delta_sigmoid(to_float<T>(src[beta_at + head])) : 0.0f;
        float all = g;                            // the product up to and with token `lane`
#pragma unroll
        for (int delta = 1; delta < N; delta <<= 1) {
            const float other = __shfl_up_sync(0xffffffffu, all, delta);
            if (lane >= delta) all = __fmul_rn(all, other);
        }
        float* to = coefficients + ((int64_t)blockIdx.x * key_heads * group + head) * DELTA_COEFFICIENTS;
        if (lane < N) {
            to[lane] = beta;
            to[N + lane] = __fmul_rn(beta, all);
            to[2 * N + lane] = all;
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {    // two entries of the triangles a lane
            const int t = 4 * half + lane / N, s = lane % N;
            float decay = 1.0f;
#pragma unroll
            for (int r = 1; r < N; ++r) {
                const float gr = __shfl_sync(0xffffffffu, g, r);
                if (r > s && r <= t) decay = __fmul_rn(decay, gr);
            }
            const float bt = __shfl_sync(0xffffffffu, beta, t);
            below[warp][t][s] = s < t ? __fmul_rn(__fmul_rn(bt, decay), kk[t][s]) : 0.0f;
            through[warp][t][s] = s <= t ? __fmul_rn(decay, qk[t][s]) : 0.0f;
            if (t == N - 1) last_s[warp][s] = decay;
        }
        __syncwarp();
        if (lane < N) {                           // column `lane` of the inverse, row by row
            float x[N];
#pragma unroll
            for (int t = 0; t < N; ++t) {
                float sum = t == lane ? 1.0f : 0.0f;
#pragma unroll
                for (int r = 0; r < t; ++r) sum = __fmaf_rn(-below[warp][t][r], x[r], sum);
                x[t] = sum;
                inverse_s[warp][t][lane] = sum;
            }
        }
        __syncwarp();
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = 4 * half + lane / N, s = lane % N;
            float sum = 0.0f;
#pragma unroll
            for (int r = 0; r < N; ++r) sum = __fmaf_rn(through[warp][t][r], inverse_s[warp][r][s], sum);
            to[3 * N + t * N + s] = __fmul_rn(last_s[warp][t], inverse_s[warp][t][s]);
            to[3 * N + N * N + t * N + s] = sum;
        }
        __syncwarp();
    }
}

// ---------------------------------------------------------------------------------------------- scan
template <typename T, int LANES, int ROWS, int COLS>
__global__ void __launch_bounds__(DELTA_THREADS, ROWS * COLS <= 16 ? 4 : 2) delta_scan_kernel(
    const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ coefficients, const T* __restrict__ v,
    int64_t v_stride, float* __restrict__ state, const int* __restrict__ row_starts, const int* __restrict__ state_slots,
    const int* __restrict__ token_row, float* __restrict__ out, int heads, int group, int dim, int padded, int vdim) {
    constexpr int N = DELTA_BLOCK, GROUPS = DELTA_THREADS / LANES, ALL = GROUPS * COLS;   // columns a CTA
    constexpr int WIDTH = LANES * ROWS, QUADS = ROWS / 4, PAIRS = ROWS / 2;
    constexpr int VALUES = N * COLS, HOLDERS = VALUES < LANES ? VALUES : LANES, OWN = VALUES / HOLDERS;
    constexpr int WORDS = N * WIDTH / 4;                     // 16-byte words of q (and of k) a piece
    constexpr int V_LOADS = (N * ALL + DELTA_THREADS - 1) / DELTA_THREADS;
    static_assert(N == 8 && (COLS == 2 || COLS == 4) && COLS % OWN == 0 && ROWS % 4 == 0, "delta_scan: a lane has one token's columns");
    static_assert(DELTA_COEFFICIENTS % 4 == 0 && DELTA_COEFFICIENTS / 4 <= DELTA_THREADS, "delta_scan: coefficients");
    __shared__ __align__(16) float q_s[2][N][WIDTH], k_s[2][N][WIDTH];
    __shared__ __align__(16) float c_s[2][DELTA_COEFFICIENTS];
    __shared__ __align__(16) float v_s[2][N][ALL], u_s[GROUPS][N][COLS];
    const int row = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * ALL;
    const int tid = threadIdx.x, lane = tid % LANES, mine = tid / LANES;
    const int begin = row_starts[row], count = row_starts[row + 1] - begin;
    if (count <= 0) return;
    const int c0 = col0 + mine * COLS;            // the thread's first column
    const int64_t out_stride = (int64_t)heads * vdim;
    // after the sums a lane has token `token` and columns `own` .. of the group's
    const int token = lane % HOLDERS * OWN / COLS, own = lane % HOLDERS * OWN % COLS;
    float* o = out + (int64_t)begin * out_stride + (int64_t)head * vdim + c0 + own;
    if (token_row[begin] < 0) {                   // a padding row of a recorded batch: no request, no state
        for (int t = token; t < count; t += N)
            for (int i = 0; i < OWN; ++i)
                if (lane < HOLDERS && c0 + own + i < vdim) o[(int64_t)t * out_stride + i] = 0.0f;
        return;
    }
    int before = 0;                               // pieces of the entries before this one
    for (int r = 0; r < row; ++r) before += (row_starts[r + 1] - row_starts[r] + N - 1) / N;
    const int key_heads = heads / group;
    const float* q_in = q + ((int64_t)begin * key_heads + head / group) * padded;
    const float* k_in = k + ((int64_t)begin * key_heads + head / group) * padded;
    const float* c_in = coefficients + ((int64_t)before * heads + head) * DELTA_COEFFICIENTS;
    const T* v_in = v + (int64_t)begin * v_stride + (int64_t)head * vdim + col0;
    const int64_t key_stride = (int64_t)key_heads * padded;
    float* state_of = state + (((int64_t)state_slots[row] * heads + head) * dim) * vdim + c0;

    // rows 4 (lane + LANES j) .. + 3: the lanes read neighbouring 16-byte words of q and k
    uint64_t s[COLS][PAIRS];
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            const int d = 4 * (lane + LANES * (i >> 1)) + 2 * (i & 1);
            const bool live = c0 + c < vdim;
            s[c][i] = pair_of(live && d < dim ? state_of[(int64_t)d * vdim + c] : 0.0f,
                              live && d + 1 < dim ? state_of[(int64_t)(d + 1) * vdim + c] : 0.0f);
        }
    T v_next[V_LOADS];
    auto copy = [&](int first, int to) {          // the piece that starts at token `first`; zeros past the end
#pragma unroll
        for (int e0 = 0; e0 < WORDS; e0 += DELTA_THREADS) {
            const int e = e0 + tid, t = e / (WIDTH / 4), d = e % (WIDTH / 4) * 4;
            if (WORDS % DELTA_THREADS == 0 || e < WORDS) {
                const bool ok = first + t < count && d < padded;
                const int64_t at = ok ? (int64_t)(first + t) * key_stride + d : 0;
                cp_async_16(&q_s[to][t][d], q_in + at, ok);
                cp_async_16(&k_s[to][t][d], k_in + at, ok);
            }
        }
        if (tid < DELTA_COEFFICIENTS / 4)
            cp_async_16(&c_s[to][4 * tid], c_in + (int64_t)(first / N) * heads * DELTA_COEFFICIENTS + 4 * tid, true);
        cp_async_commit();
    };
    auto fetch = [&](int first) {
#pragma unroll
        for (int j = 0; j < V_LOADS; ++j) {
            const int e = tid + j * DELTA_THREADS, t = e / ALL, cc = e % ALL;
            const bool ok = e < N * ALL && first + t < count && col0 + cc < vdim;
            v_next[j] = ok ? v_in[(int64_t)(first + t) * v_stride + cc] : from_float<T>(0.0f);
        }
    };
    auto stage = [&](int to) {
#pragma unroll
        for (int j = 0; j < V_LOADS; ++j) {
            const int e = tid + j * DELTA_THREADS;
            if (N * ALL % DELTA_THREADS == 0 || e < N * ALL) v_s[to][e / ALL][e % ALL] = to_float<T>(v_next[j]);
        }
    };
    // the lanes' parts of S^T x_t of a piece's tokens, then halving: a lane keeps the sums of its token and columns
    auto over_lanes = [&](float* part, float* sums) {
#pragma unroll
        for (int bit = LANES / 2; bit >= 1; bit >>= 1) {
            const int n = VALUES / HOLDERS * 2 * bit;     // values left before this step
            if (bit >= HOLDERS) {                 // more lanes than values: the upper lanes' parts are added first
#pragma unroll
                for (int i = 0; i < VALUES; ++i) part[i] += __shfl_xor_sync(0xffffffffu, part[i], bit);
            } else {
                const bool upper = (lane & bit) != 0;
#pragma unroll
                for (int i = 0; i < n / 2; ++i) {
                    const float hand = upper ? part[i] : part[i + n / 2], keep = upper ? part[i + n / 2] : part[i];
                    part[i] = keep + __shfl_xor_sync(0xffffffffu, hand, bit);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < OWN; ++i) sums[i] = part[i];
    };
    auto over_rows = [&](const ulonglong2* x, float* part) {
        uint64_t sum[COLS];
#pragma unroll
        for (int c = 0; c < COLS; ++c) sum[c] = 0;
#pragma unroll
        for (int j = 0; j < QUADS; ++j)
#pragma unroll
            for (int c = 0; c < COLS; ++c) sum[c] = pair_fma(s[c][2 * j + 1], x[j].y, pair_fma(s[c][2 * j], x[j].x, sum[c]));
#pragma unroll
        for (int c = 0; c < COLS; ++c) part[c] = pair_sum(sum[c]);
    };
    copy(0, 0);
    fetch(0);
    for (int first = 0, turn = 0; first < count; first += N, turn ^= 1) {
        stage(turn);
        cp_async_wait<0>();
        __syncthreads();                          // this piece is there, the one before is read
        if (first + N < count) {
            copy(first + N, turn ^ 1);
            fetch(first + N);
        }
        const float* coefficient = c_s[turn];
        float p[OWN], w[OWN], r[OWN], write[OWN], result[OWN], row_t[N], row_m[N];
        ulonglong2 keys[N][QUADS];                // wait in registers for the update
        float part[VALUES];
#pragma unroll
        for (int t = 0; t < N; ++t)
#pragma unroll
            for (int j = 0; j < QUADS; ++j) keys[t][j] = *reinterpret_cast<const ulonglong2*>(&k_s[turn][t][4 * (lane + LANES * j)]);
#pragma unroll
        for (int t = 0; t < N; ++t) over_rows(keys[t], part + t * COLS);
        over_lanes(part, p);
#pragma unroll
        for (int t = 0; t < N; ++t) {
            ulonglong2 query[QUADS];
#pragma unroll
            for (int j = 0; j < QUADS; ++j) query[j] = *reinterpret_cast<const ulonglong2*>(&q_s[turn][t][4 * (lane + LANES * j)]);
            over_rows(query, part + t * COLS);
        }
        over_lanes(part, w);
        const float beta = coefficient[token], along = coefficient[N + token], so_far = coefficient[2 * N + token];
        load_values<4>(coefficient + 3 * N + token * N, row_t);
        load_values<4>(coefficient + 3 * N + token * N + 4, row_t + 4);
        load_values<4>(coefficient + 3 * N + N * N + token * N, row_m);
        load_values<4>(coefficient + 3 * N + N * N + token * N + 4, row_m + 4);
#pragma unroll
        for (int i = 0; i < OWN; ++i) {
            r[i] = __fmaf_rn(-along, p[i], __fmul_rn(beta, v_s[turn][token][mine * COLS + own + i]));
            write[i] = 0.0f;
            result[i] = __fmul_rn(so_far, w[i]);
        }
#pragma unroll
        for (int e = 0; e < N; ++e)
#pragma unroll
            for (int i = 0; i < OWN; ++i) {       // of the lane that has token e and the same columns
                const float x = __shfl_sync(0xffffffffu, r[i], (e * COLS + own) / OWN, LANES);
                write[i] = __fmaf_rn(row_t[e], x, write[i]);
                result[i] = __fmaf_rn(row_m[e], x, result[i]);
            }
#pragma unroll
        for (int i = 0; i < OWN; ++i)
            if (lane < HOLDERS) u_s[mine][token][own + i] = write[i];
        __syncwarp();
        const float whole = coefficient[3 * N - 1];
        const uint64_t whole2 = pair_of(whole, whole);
#pragma unroll
        for (int c = 0; c < COLS; ++c)
#pragma unroll
            for (int i = 0; i < PAIRS; ++i) s[c][i] = pair_mul(whole2, s[c][i]);
#pragma unroll
        for (int t = 0; t < N; ++t) {
            float x[COLS];
            if constexpr (COLS == 4) load_values<4>(u_s[mine][t], x);
            else { const float2 y = *reinterpret_cast<const float2*>(u_s[mine][t]); x[0] = y.x; x[1] = y.y; }
#pragma unroll
            for (int j = 0; j < QUADS; ++j) {
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    const uint64_t x2 = pair_of(x[c], x[c]);
                    s[c][2 * j] = pair_fma(keys[t][j].x, x2, s[c][2 * j]);
                    s[c][2 * j + 1] = pair_fma(keys[t][j].y, x2, s[c][2 * j + 1]);
                }
            }
        }
        if (lane < HOLDERS && first + token < count) {
#pragma unroll
            for (int i = 0; i < OWN; ++i)
                if (c0 + own + i < vdim) o[(int64_t)(first + token) * out_stride + i] = result[i];
        }
    }
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
            const int d = 4 * (lane + LANES * (i >> 1)) + 2 * (i & 1);
            float a, b;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(s[c][i]));
            if (c0 + c < vdim && d < dim) state_of[(int64_t)d * vdim + c] = a;
            if (c0 + c < vdim && d + 1 < dim) state_of[(int64_t)(d + 1) * vdim + c] = b;
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
// [tokens, key_heads, padded], padded a multiple of four at least dim; coefficients float32 [pieces, heads,
// tvb_delta_coefficients()], `pieces` at least those of all entries (tokens / tvb_delta_block() + rows always is).
extern "C" int tvb_delta_prepare(const void* mixed, long long mixed_stride, int q_at, int k_at, const void* proj,
                                 long long proj_stride, int beta_at, int decay_at, const float* rate, const float* dt_bias,
                                 float q_scale, float unit_eps, float* q_out, float* k_out, float* coefficients,
                                 const int* row_starts, const int* token_row, int rows, int pieces, int key_heads, int group,
                                 int dim, int padded, int dtype, void* stream) {
    if (rows <= 0 || pieces <= 0) return 0;
    if (key_heads <= 0 || key_heads > 65535 || group <= 0 || dim <= 0 || dim > DELTA_MAX_DIM || padded < dim || padded % 4 ||
        padded > DELTA_MAX_DIM)
        return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
#define GO(T) delta_prepare_kernel<T><<<dim3(pieces, key_heads), 128, 0, s>>>(                                          \
        (const T*)mixed, mixed_stride, q_at, k_at, (const T*)proj, proj_stride, beta_at, decay_at, rate, dt_bias, q_scale, \
        unit_eps, q_out, k_out, coefficients, row_starts, token_row, rows, key_heads, group, dim, padded)
    if (dtype == TVB_F32) GO(float);
    else if (dtype == TVB_BF16) GO(bf16);
    else return TVB_BAD_ARGUMENT;
#undef GO
    return tvb_last_error();
}

extern "C" int tvb_delta_block() { return DELTA_BLOCK; }
extern "C" int tvb_delta_coefficients() { return DELTA_COEFFICIENTS; }

// q, k, coefficients as delta_prepare leaves them; v: [tokens, heads * vdim] of the storage type, rows `v_stride` apart;
// state float32 [slots, heads, dim, vdim]; out float32 [tokens, heads * vdim].  `cols` (0: chosen): two or four columns a
// thread.
extern "C" int tvb_delta_scan(const float* q, const float* k, const float* coefficients, const void* v, long long v_stride,
                              float* state, const int* row_starts, const int* state_slots, const int* token_row, float* out,
                              int rows, int heads, int group, int dim, int padded, int vdim, int cols, int dtype,
                              void* stream) {
    if (rows <= 0) return 0;
    if (heads <= 0 || heads > 65535 || group <= 0 || heads % group || dim <= 0 || dim > DELTA_MAX_DIM || padded < dim ||
        padded % 4 || vdim <= 0 || !state || ((uintptr_t)q | (uintptr_t)k | (uintptr_t)coefficients) % 16)
        return TVB_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    // two columns a thread where four would leave many SMs without a CTA
    const int groups = DELTA_THREADS / (dim <= 64 ? 16 : 32);
    const bool few = cols == 0 ? (long long)rows * heads * ((vdim + 4 * groups - 1) / (4 * groups)) < 100 : cols == 2;
    if (cols != 0 && cols != 2 && cols != 4) return TVB_BAD_ARGUMENT;
#define GO(T, LANES, ROWS, COLS) {                                                                                      \
        const dim3 grid(rows, heads, (vdim + groups * COLS - 1) / (groups * COLS));                                     \
        if (grid.z > 65535) return TVB_BAD_ARGUMENT;                                                                    \
        delta_scan_kernel<T, LANES, ROWS, COLS><<<grid, DELTA_THREADS, 0, s>>>(q, k, coefficients, (const T*)v,         \
            v_stride, state, row_starts, state_slots, token_row, out, heads, group, dim, padded, vdim); }
#define BY_COLS(T, LANES, ROWS) if (few) GO(T, LANES, ROWS, 2) else GO(T, LANES, ROWS, 4)
#define BY_DIM(T)                              \
    if (dim <= 64) { BY_COLS(T, 16, 4) }       \
    else if (dim <= 128) { BY_COLS(T, 32, 4) } \
    else { BY_COLS(T, 32, 8) }
    if (dtype == TVB_F32) { BY_DIM(float) }
    else if (dtype == TVB_BF16) { BY_DIM(bf16) }
    else return TVB_BAD_ARGUMENT;
#undef BY_DIM
#undef BY_COLS
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
