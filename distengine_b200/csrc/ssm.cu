// The state-space mixer (Mamba-2): per head h a state S [N, P] (float32, in the slot of its
// request) that decays by one number a token, takes an outer product in and is read out,
//
//   S_t = exp(a_t) S_(t-1) + dt_t b_t x_t^T;   y_t = S_t^T c_t + D x_t,    a_t = -exp(A_log) dt_t
//
// x_t [P] of the head, b_t and c_t [N] of the head's group.  x, b and c are what a short causal
// convolution over time (one filter a channel, with bias) and silu leave of the projection; its last
// K - 1 inputs are part of the slot's state.  dt_t = softplus(projection + dt_bias).  Everything
// here is float32 arithmetic; T (float32 or bfloat16) is the type of the projection that comes in
// and of the rows that go out.
//
//   prep         convolution, silu, dt and a of every token (steps with portions)
//   walk         token after token through the state: a block holds 4 CQ columns of a head's state
//                in registers.  Single tokens (`fused`: the convolution too) and short portions
//   chunk_*      portions of some length, 64 tokens a chunk, three kernels: what every chunk adds
//                to the state by itself (a matrix product over its tokens), the states at the
//                chunks' starts one after the other, and every chunk's read-outs:
//                  y_t = exp(l_t) c_t^T S_start + sum over s <= t of exp(l_t - l_s) dt_s (c_t . b_s) x_s
//                the products c . b once for all heads of a group;
//                with l the running sum of a inside the chunk.  The sums l are kept in double
//                precision: what enters is the difference of two of them, which may be small
//                between large ones.
//   gated_group_norm   y silu(z) in parts, each over its own root mean square, times the weight;
//                and the slots' kept convolution inputs move on
//
// Every exponent is of a number <= 0, so nothing grows; a state does not depend on how its tokens
// were cut into steps beyond rounding.

#include "common.cuh"

DE_DEFINE_PDL_SWITCH

namespace {

__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

template <typename T> struct Quad;
template <> struct Quad<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <> struct Quad<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        v[0] = __uint_as_float(t.x << 16);
        v[1] = __uint_as_float(t.x & 0xffff0000u);
        v[2] = __uint_as_float(t.y << 16);
        v[3] = __uint_as_float(t.y & 0xffff0000u);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]);
        const __nv_bfloat162 b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 t;
        t.x = *reinterpret_cast<const unsigned*>(&a);
        t.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = t;
    }
};

// The mixer's sizes; C = H P + 2 G N channels pass the convolution, [x | b | c].
struct Shape {
    int H, G, N, P, K, C;
};

struct Conv {                  // the convolution and where its kept inputs lie in a slot's row
    const float* taps;         // [K][C]
    const float* bias;         // [C]
    const float* state;
    long long slot_stride;
    int offset;
};

// One channel of one token: row `n` of xbc, `off` its place in its sequence's portion; inputs
// before the portion come from the slot (zeros at a sequence's start).
template <typename T>
__device__ __forceinline__ float conv_one(const T* __restrict__ xbc, int ld, const Conv& cv,
                                          const float* kept, int n, int off, int K, int C, int c) {
    float acc = cv.bias[c];
    for (int j = 0; j < K; ++j) {
        const int rel = off - (K - 1) + j;
        const float x = rel >= 0 ? to_float(xbc[(size_t)(n - (K - 1) + j) * ld + c])
                                 : kept[(size_t)(off + j) * C + c];
        acc = fmaf(cv.taps[(size_t)j * C + c], x, acc);
    }
    return silu_f(acc);
}

// The rates of token n, by the block's threads.
template <typename T>
__device__ __forceinline__ void rates_of(int n, const T* __restrict__ dt, int ld_dt,
                                         const float* __restrict__ dt_bias,
                                         const float* __restrict__ a_log, float* __restrict__ rates,
                                         int H) {
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
        const float d = softplus_f(to_float(dt[(size_t)n * ld_dt + h]) + dt_bias[h]);
        rates[(size_t)n * 2 * H + h] = d;
        rates[(size_t)n * 2 * H + H + h] = -expf(a_log[h]) * d;
    }
}

// out [n][C], rates [n][2 H]: dt, then a.  grid (runs of RUN tokens, blocks of 512 channels): a
// thread has four neighbouring channels and keeps their last KK - 1 inputs in registers while it
// goes through its tokens.  KK = K.
constexpr int RUN = 8;
template <typename T, int KK>
__global__ void __launch_bounds__(128)
prep_run_kernel(const T* __restrict__ xbc, int ld, const T* __restrict__ dt, int ld_dt, Conv cv,
                const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                const int* __restrict__ token_seq, const int* __restrict__ token_slot,
                const int* __restrict__ positions, const int* __restrict__ seq_pos0,
                float* __restrict__ out, float* __restrict__ rates, Shape sh, int n_tokens) {
    const int n0 = blockIdx.x * RUN, n1 = min(n_tokens, n0 + RUN), C = sh.C;
    const int c = (blockIdx.y * 128 + threadIdx.x) * 4;
    float w[KK][4], bias[4], x[KK][4];
    if (c < C) {
        Quad<float>::load(cv.bias + c, bias);
#pragma unroll
        for (int j = 0; j < KK; ++j) Quad<float>::load(cv.taps + (size_t)j * C + c, w[j]);
    }
    pdl_wait();
    if (c < C) {
        float own[RUN][4];                           // the run's inputs, asked for at once
#pragma unroll
        for (int i = 0; i < RUN; ++i)
            if (n0 + i < n1) Quad<T>::load(xbc + (size_t)(n0 + i) * ld + c, own[i]);
#pragma unroll
        for (int i = 0; i < RUN; ++i) {
            const int n = n0 + i;
            if (n >= n1) break;
            const int off = positions[n] - seq_pos0[token_seq[n]];
            if (i == 0 || off == 0) {                // the inputs before this token
                const float* kept =
                    cv.state + (size_t)token_slot[n] * cv.slot_stride + cv.offset;
#pragma unroll
                for (int j = 0; j < KK - 1; ++j) {
                    if (off - (KK - 1) + j >= 0)
                        Quad<T>::load(xbc + (size_t)(n - (KK - 1) + j) * ld + c, x[j]);
                    else Quad<float>::load(kept + (size_t)(off + j) * C + c, x[j]);
                }
            }
            float acc[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                x[KK - 1][e] = own[i][e];
                acc[e] = bias[e];
#pragma unroll
                for (int j = 0; j < KK; ++j) acc[e] = fmaf(w[j][e], x[j][e], acc[e]);
                acc[e] = silu_f(acc[e]);
#pragma unroll
                for (int j = 0; j + 1 < KK; ++j) x[j][e] = x[j + 1][e];
            }
            Quad<float>::store(out + (size_t)n * C + c, acc);
        }
    }
    if (blockIdx.y == 0)
        for (int n = n0; n < n1; ++n) rates_of(n, dt, ld_dt, dt_bias, a_log, rates, sh.H);
    pdl_trigger();
}

// The same for any K, sizes and alignment: a thread a channel.  grid (tokens, blocks of channels).
template <typename T>
__global__ void __launch_bounds__(128)
prep_kernel(const T* __restrict__ xbc, int ld, const T* __restrict__ dt, int ld_dt, Conv cv,
            const float* __restrict__ dt_bias, const float* __restrict__ a_log,
            const int* __restrict__ token_seq, const int* __restrict__ token_slot,
            const int* __restrict__ positions, const int* __restrict__ seq_pos0,
            float* __restrict__ out, float* __restrict__ rates, Shape sh) {
    const int n = blockIdx.x, C = sh.C;
    const int off = positions[n] - seq_pos0[token_seq[n]];
    const float* kept = cv.state + (size_t)token_slot[n] * cv.slot_stride + cv.offset;
    pdl_wait();
    const int c = blockIdx.y * 128 + threadIdx.x;
    if (c < C) out[(size_t)n * C + c] = conv_one(xbc, ld, cv, kept, n, off, sh.K, C, c);
    if (blockIdx.y == 0) rates_of(n, dt, ld_dt, dt_bias, a_log, rates, sh.H);
    pdl_trigger();
}

// ------------------------------------------------------------------------------------------
// Token after token.  grid (sequences, heads, tiles of 4 CQ columns), 256 threads: thread = CQ *
// row group + column quad; register r of row group g is row g + RG r of the state.
// FUSED: every sequence brings one token, whose convolution and rates are formed here (xbc and dt
// are columns of the projection); otherwise both come from `prep` and only sequences of at most
// `longest` tokens are walked.
// ------------------------------------------------------------------------------------------
template <typename T, bool FUSED, int CQ, int R>
__global__ void __launch_bounds__(256, R <= 8 ? 4 : 2)
walk_kernel(const T* __restrict__ xbc, int ld, const T* __restrict__ dt_in, int ld_dt, Conv cv,
            const float* __restrict__ dt_bias, const float* __restrict__ a_log,
            const float* __restrict__ ready, const float* __restrict__ rates,
            const float* __restrict__ skip, float* state, long long slot_stride,
            const int* __restrict__ seq_slot, const int* __restrict__ seq_qstart,
            const int* __restrict__ seq_qlen, int longest, float* __restrict__ y, Shape sh,
            int vec) {
    constexpr int RG = 256 / CQ, PT = 4 * CQ;
    extern __shared__ __align__(16) float vecs[];    // [PT] x, [N] b, [N] c
    __shared__ float red[8][PT];
    const int s = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PT;
    const int N = sh.N, P = sh.P, H = sh.H, C = sh.C;
    const int qlen = seq_qlen[s], tok0 = seq_qstart[s];
    pdl_wait();
    if (!FUSED && qlen > longest) return;
    const int tid = threadIdx.x, cq = tid % CQ, rg = tid / CQ, lane = tid & 31, warp = tid >> 5;
    const int col = p0 + 4 * cq, g = h / (H / sh.G);
    float* S_g = state + (size_t)seq_slot[s] * slot_stride + (size_t)h * N * P;
    float S[R][4];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = rg + RG * r;
#pragma unroll
        for (int e = 0; e < 4; ++e) S[r][e] = 0.0f;
        if (i < N) {
            if (vec) {
                if (col < P) Quad<float>::load(S_g + (size_t)i * P + col, S[r]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (col + e < P) S[r][e] = S_g[(size_t)i * P + col + e];
            }
        }
    }
    float *xs = vecs, *bs = vecs + PT, *cs = bs + N;
    const float d_skip = skip[h], rate = expf(a_log[h]);
    const float* kept = cv.state + (size_t)seq_slot[s] * cv.slot_stride + cv.offset;
    for (int t = 0; t < qlen; ++t) {
        const int n = tok0 + t;
        for (int i = tid; i < PT + 2 * N; i += 256) {
            int c;
            if (i < PT) c = p0 + i < P ? h * P + p0 + i : -1;
            else if (i < PT + N) c = H * P + g * N + (i - PT);
            else c = H * P + (sh.G + g) * N + (i - PT - N);
            float v = 0.0f;
            if (c >= 0)
                v = FUSED ? conv_one(xbc, ld, cv, kept, n, 0, sh.K, C, c)
                          : ready[(size_t)n * C + c];
            vecs[i] = v;
        }
        float dt, a;
        if (FUSED) {
            dt = softplus_f(to_float(dt_in[(size_t)n * ld_dt + h]) + dt_bias[h]);
            a = -rate * dt;
        } else {
            dt = rates[(size_t)n * 2 * H + h];
            a = rates[(size_t)n * 2 * H + H + h];
        }
        const float decay = expf(a);
        __syncthreads();
        float x[4], o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        Quad<float>::load(xs + 4 * cq, x);
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int i = rg + RG * r;
            if (i < N) {
                const float b = dt * bs[i], c = cs[i];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    S[r][e] = fmaf(b, x[e], decay * S[r][e]);
                    o[e] = fmaf(S[r][e], c, o[e]);
                }
            }
        }
#pragma unroll
        for (int step = CQ; step < 32; step <<= 1)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[e] += __shfl_xor_sync(0xffffffffu, o[e], step);
        if (lane < CQ) Quad<float>::store(&red[warp][4 * lane], o);
        __syncthreads();
        if (tid < PT && p0 + tid < P) {
            float sum = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; ++w) sum += red[w][tid];
            y[(size_t)n * (H * P) + h * P + p0 + tid] = fmaf(d_skip, xs[tid], sum);
        }
        if (!FUSED) __syncthreads();                 // the vectors may be filled again
    }
    pdl_trigger();
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = rg + RG * r;
        if (i < N) {
            if (vec) {
                if (col < P) Quad<float>::store(S_g + (size_t)i * P + col, S[r]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (col + e < P) S_g[(size_t)i * P + col + e] = S[r][e];
            }
        }
    }
}

// ------------------------------------------------------------------------------------------
// Chunks.  An item is (sequence, first token, tokens, 0); 128 threads work on tiles of 64 x 64.
// ------------------------------------------------------------------------------------------
constexpr int L = 64;          // tokens of a chunk
constexpr int WIDE = L + 4;    // row pitch of a tile of 64 columns
constexpr int SLICE = 32;      // of N, a stage of the read-out
constexpr int NARROW = SLICE + 4;

// Running sums of a over the chunk's tokens, in double precision, and dt; tokens beyond the
// chunk's add nothing.  Warp 0 works; the caller synchronises.
__device__ __forceinline__ void chunk_sums(const float* __restrict__ rates, int tok0, int count,
                                           int H, int h, double* cum, float* dts) {
    if (threadIdx.x >= 32) return;
    const int lane = threadIdx.x;
    double v[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int t = 2 * lane + u;
        const float* r = rates + (size_t)(tok0 + t) * 2 * H;
        dts[t] = t < count ? r[h] : 0.0f;
        v[u] = t < count ? (double)r[H + h] : 0.0;
    }
    v[1] += v[0];
    double run = v[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
    }
    const double before = run - v[1];
    cum[2 * lane] = before + v[0];
    cum[2 * lane + 1] = run;
}

__device__ __forceinline__ void tiles_arrived() {
    asm volatile("cp.async.wait_all;\n" ::: "memory");
    __syncthreads();
}

// The first `count` rows and `cols` columns of src into tile [ROWS][pitch] of WIDTH columns, zeros
// elsewhere.  The copies are asynchronous: `tiles_arrived` waits for all of them.
template <int ROWS, int WIDTH>
__device__ __forceinline__ void fill_tile(float* tile, int pitch, const float* __restrict__ src,
                                          size_t ld, int count, int cols, int vec) {
    if (vec) {
        constexpr int QUADS = WIDTH / 4;
        const unsigned base = (unsigned)__cvta_generic_to_shared(tile);
#pragma unroll
        for (int u = 0; u < ROWS * QUADS / 128; ++u) {
            const int i = threadIdx.x + 128 * u, t = i / QUADS, c = 4 * (i % QUADS);
            const bool in = t < count && c < cols;   // (outside: no bytes, the rest is zeroed)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(
                             base + (unsigned)((t * pitch + c) * sizeof(float))),
                         "l"(in ? src + t * ld + c : src), "r"(in ? 16 : 0)
                         : "memory");
        }
    } else {
        for (int i = threadIdx.x; i < ROWS * WIDTH; i += 128) {
            const int t = i / WIDTH, c = i - t * WIDTH;
            tile[t * pitch + c] = (t < count && c < cols) ? src[t * ld + c] : 0.0f;
        }
    }
}

// The products c_t . b_s of a chunk's tokens, the same for all heads of a group:
// products[item][g][t][s] (s <= t is used).  128 threads.
__device__ __forceinline__ void chunk_products(const float* __restrict__ c_src,
                                               const float* __restrict__ b_src, const Shape& sh,
                                               int count, float* Cs, float* Bs,
                                               float* __restrict__ dst, int vec) {
    const int tr = threadIdx.x >> 4, tc = threadIdx.x & 15;    // rows tr + 8 i, columns tc + 16 j
    float G[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) G[i][j] = 0.0f;
    for (int n0 = 0; n0 < sh.N; n0 += SLICE) {
        __syncthreads();
        fill_tile<L, SLICE>(Cs, NARROW, c_src + n0, sh.C, count, min(SLICE, sh.N - n0), vec);
        fill_tile<L, SLICE>(Bs, NARROW, b_src + n0, sh.C, count, min(SLICE, sh.N - n0), vec);
        tiles_arrived();
#pragma unroll 2
        for (int k = 0; k < SLICE; k += 4) {
            float b[4][4];
#pragma unroll
            for (int j = 0; j < 4; ++j) Quad<float>::load(Bs + (tc + 16 * j) * NARROW + k, b[j]);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                float c[4];
                Quad<float>::load(Cs + (tr + 8 * i) * NARROW + k, c);
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int j = 0; j < 4; ++j) G[i][j] = fmaf(c[u], b[j][u], G[i][j]);
            }
        }
    }
    pdl_trigger();
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) dst[(tr + 8 * i) * L + tc + 16 * j] = G[i][j];
}

// What the chunk adds to the state by itself: out[item][h][n][p] = sum_t exp(l_last - l_t) dt_t
// b_t[n] x_t[p]; decays[item][h] = exp(l_last).  grid (items, H, 1 + tiles of n times tiles of p):
// of the first layer of blocks one a group forms the products c . b.
__global__ void __launch_bounds__(128, 6)
chunk_state_kernel(const float* __restrict__ xbc, const float* __restrict__ rates,
                   const int4* __restrict__ items, float* __restrict__ out,
                   float* __restrict__ decays, float* __restrict__ products, Shape sh, int vec) {
    __shared__ __align__(16) float Bs[L * WIDE], Xs[L * WIDE];
    __shared__ double cum[L];
    __shared__ float dts[L], ws[L];
    const int4 item = items[blockIdx.x];
    const int per = sh.H / sh.G, h = blockIdx.y, g = h / per, N = sh.N, P = sh.P;
    const int p_tiles = (P + 63) >> 6;
    const int tok0 = item.y, count = item.z;
    pdl_wait();
    const float* row = xbc + (size_t)tok0 * sh.C;
    if (blockIdx.z == 0) {                           // the longest blocks come first
        if (h % per == 0)
            chunk_products(row + sh.H * P + (sh.G + g) * N, row + sh.H * P + g * N, sh, count, Bs,
                           Xs, products + ((size_t)blockIdx.x * sh.G + g) * L * L, vec);
        return;
    }
    const int tile = blockIdx.z - 1, n0 = tile / p_tiles * 64, p0 = tile % p_tiles * 64;
    fill_tile<L, 64>(Xs, WIDE, row + h * P + p0, sh.C, count, min(64, P - p0), vec);
    fill_tile<L, 64>(Bs, WIDE, row + sh.H * P + g * N + n0, sh.C, count, min(64, N - n0), vec);
    chunk_sums(rates, tok0, count, sh.H, h, cum, dts);
    tiles_arrived();
    if (threadIdx.x < L)
        ws[threadIdx.x] = expf((float)(cum[L - 1] - cum[threadIdx.x])) * dts[threadIdx.x];
    if (tile == 0 && threadIdx.x == 0)
        decays[(size_t)blockIdx.x * sh.H + h] = expf((float)cum[L - 1]);
    __syncthreads();
    const int tr = threadIdx.x >> 4, tc = threadIdx.x & 15;     // rows 4 tr, 4 tr + 32; columns 4 tc
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
#pragma unroll 4
    for (int t = 0; t < count; ++t) {
        float b0[4], b1[4], x[4];
        Quad<float>::load(Bs + t * WIDE + 4 * tr, b0);
        Quad<float>::load(Bs + t * WIDE + 32 + 4 * tr, b1);
        Quad<float>::load(Xs + t * WIDE + 4 * tc, x);
        const float w = ws[t];
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] *= w;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                acc[i][j] = fmaf(b0[i], x[j], acc[i][j]);
                acc[4 + i][j] = fmaf(b1[i], x[j], acc[4 + i][j]);
            }
    }
    pdl_trigger();
    float* dst = out + ((size_t)blockIdx.x * sh.H + h) * N * P;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int n = n0 + 4 * tr + (i & 3) + (i >> 2) * 32, p = p0 + 4 * tc;
        if (n >= N) continue;
        if (vec) {
            if (p < P) Quad<float>::store(dst + (size_t)n * P + p, acc[i]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (p + j < P) dst[(size_t)n * P + p + j] = acc[i][j];
        }
    }
}

// The states at the chunks' starts: out[item] becomes the state before the chunk, the slot keeps
// the state after the last one.  long_seqs: (sequence, first item, items, 0).  A thread has VEC
// elements of the state.
template <int VEC>
__global__ void __launch_bounds__(256)
chunk_pass_kernel(float* __restrict__ out, const float* __restrict__ decays,
                  const int4* __restrict__ long_seqs, const int* __restrict__ seq_slot,
                  float* __restrict__ state, long long slot_stride, int H, int NP) {
    const int4 seq = long_seqs[blockIdx.x];
    const size_t at = ((size_t)blockIdx.y * 256 + threadIdx.x) * VEC;
    const size_t total = (size_t)H * NP;
    pdl_wait();
    if (at >= total) return;
    const int h = (int)(at / NP);
    float* S_g = state + (size_t)seq_slot[seq.x] * slot_stride + at;
    float S[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) S[e] = S_g[e];
    float* chunk = out + (size_t)seq.y * total + at;
    constexpr int AHEAD = 8;                         // chunks in flight
    for (int i0 = 0; i0 < seq.z; i0 += AHEAD) {
        float add[AHEAD][VEC], dec[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int i = i0 + u;
            dec[u] = i < seq.z ? decays[(size_t)(seq.y + i) * H + h] : 1.0f;
            if constexpr (VEC == 4) {
                if (i < seq.z) Quad<float>::load(chunk + (size_t)i * total, add[u]);
            } else {
                add[u][0] = i < seq.z ? chunk[(size_t)i * total] : 0.0f;
            }
        }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int i = i0 + u;
            if (i >= seq.z) break;
            if constexpr (VEC == 4) Quad<float>::store(chunk + (size_t)i * total, S);
            else chunk[(size_t)i * total] = S[0];
#pragma unroll
            for (int e = 0; e < VEC; ++e) S[e] = fmaf(dec[u], S[e], add[u][e]);
        }
    }
    pdl_trigger();
#pragma unroll
    for (int e = 0; e < VEC; ++e) S_g[e] = S[e];
}

// The chunk's read-outs.  grid (items, H, tiles of p).  Thread (tr, tc) has the rows t = tr + 8 i
// and the columns p = 4 tc + j of y.
__global__ void __launch_bounds__(128, 5)
chunk_out_kernel(const float* __restrict__ xbc, const float* __restrict__ rates,
                 const int4* __restrict__ items, const float* __restrict__ starts,
                 const float* __restrict__ products, const float* __restrict__ skip,
                 float* __restrict__ y, Shape sh, int vec) {
    // first the stages of c [64][NARROW] and of the state [SLICE][WIDE], then x [64][WIDE]; the
    // weights of the chunk's tokens beside them
    __shared__ __align__(16) float stage[L * NARROW + SLICE * WIDE], Gs[L * WIDE];
    __shared__ double cum[L];
    __shared__ float dts[L];
    static_assert(L * NARROW + SLICE * WIDE >= L * WIDE, "x takes the stages' place");
    const int4 item = items[blockIdx.x];
    const int h = blockIdx.y, g = h / (sh.H / sh.G), N = sh.N, P = sh.P, p0 = blockIdx.z * 64;
    const int tok0 = item.y, count = item.z;
    float *Cs = stage, *Ss = stage + L * NARROW, *Xs = stage;
    const int tr = threadIdx.x >> 4, tc = threadIdx.x & 15;
    pdl_wait();
    const float* row = xbc + (size_t)tok0 * sh.C;
    const float* c_src = row + sh.H * P + (sh.G + g) * N;
    const float* s_src = starts + ((size_t)blockIdx.x * sh.H + h) * N * P + p0;
    const int p_cols = min(64, P - p0);
    // c . b of the group's chunk, made weights once the running sums are there
    const float* p_src = products + ((size_t)blockIdx.x * sh.G + g) * L * L;
    fill_tile<L, 64>(Gs, WIDE, p_src, L, L, L, 1);
    float Y[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) Y[i][j] = 0.0f;
    for (int n0 = 0; n0 < N; n0 += SLICE) {
        const int cols = min(SLICE, N - n0);
        if (n0 > 0) __syncthreads();
        fill_tile<L, SLICE>(Cs, NARROW, c_src + n0, sh.C, count, cols, vec);
        fill_tile<SLICE, 64>(Ss, WIDE, s_src + (size_t)n0 * P, P, cols, p_cols, vec);
        if (n0 == 0) chunk_sums(rates, tok0, count, sh.H, h, cum, dts);
        tiles_arrived();
#pragma unroll 2
        for (int k = 0; k < SLICE; k += 4) {
            float st[4][4];
#pragma unroll
            for (int u = 0; u < 4; ++u) Quad<float>::load(Ss + (k + u) * WIDE + 4 * tc, st[u]);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                float c[4];
                Quad<float>::load(Cs + (tr + 8 * i) * NARROW + k, c);
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int j = 0; j < 4; ++j) Y[i][j] = fmaf(c[u], st[u][j], Y[i][j]);
            }
        }
    }
    __syncthreads();
    fill_tile<L, 64>(Xs, WIDE, row + h * P + p0, sh.C, count, p_cols, vec);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = tr + 8 * i;
        const double lt = cum[t];
        const float from_start = expf((float)lt);
        float m[4];
        Quad<float>::load(Gs + t * WIDE + 4 * tc, m);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int s = 4 * tc + j;
            m[j] = s <= t ? m[j] * expf((float)(lt - cum[s])) * dts[s] : 0.0f;
            Y[i][j] *= from_start;
        }
        Quad<float>::store(Gs + t * WIDE + 4 * tc, m);
    }
    tiles_arrived();
#pragma unroll 2
    for (int s = 0; s < L; s += 4) {
        float x[4][4];
#pragma unroll
        for (int u = 0; u < 4; ++u) Quad<float>::load(Xs + (s + u) * WIDE + 4 * tc, x[u]);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float m[4];
            Quad<float>::load(Gs + (tr + 8 * i) * WIDE + s, m);
#pragma unroll
            for (int u = 0; u < 4; ++u)
#pragma unroll
                for (int j = 0; j < 4; ++j) Y[i][j] = fmaf(m[u], x[u][j], Y[i][j]);
        }
    }
    pdl_trigger();
    const float d = skip[h];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = tr + 8 * i, p = 4 * tc;
        if (t >= count) continue;
        float x[4];
        Quad<float>::load(Xs + t * WIDE + p, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] = fmaf(d, x[j], Y[i][j]);
        float* dst = y + (size_t)(tok0 + t) * (sh.H * P) + h * P + p0 + p;
        if (vec) {
            if (p < p_cols) Quad<float>::store(dst, x);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (p + j < p_cols) dst[j] = x[j];
        }
    }
}

// ------------------------------------------------------------------------------------------
// After the state: g = y silu(z), every one of `parts` equal pieces of the row over its own root
// mean square, times the weight.  grid (tokens, parts).  K > 1: the blocks of a sequence's last
// token also move the slot's kept convolution inputs (rows of xbc) on, a share of the channels
// each; whatever reads the old ones has run before.
// ------------------------------------------------------------------------------------------
struct Keep {
    const void* xbc;
    int ld, C, K, offset, vec;
    float* state;
    long long slot_stride;
    const int *token_seq, *positions, *seq_pos0, *seq_qlen, *seq_slot;
};

// Whether token n is its sequence's last; then the kept inputs move on.  `who` of `of` workers.
template <typename T>
__device__ __forceinline__ void keep_inputs(const Keep& kp, int n, int who, int of) {
    if (kp.K <= 1) return;
    const int s = kp.token_seq[n], qlen = kp.seq_qlen[s];
    if (kp.positions[n] - kp.seq_pos0[s] != qlen - 1) return;
    float* kept = kp.state + (size_t)kp.seq_slot[s] * kp.slot_stride + kp.offset;
    const T* xbc = (const T*)kp.xbc + (size_t)(n - (qlen - 1)) * kp.ld;
    constexpr int AT_ONCE = 3;
    if (kp.K - 1 <= AT_ONCE && kp.vec) {             // all of a quad's new rows, then the stores
        for (int c = 4 * who; c < kp.C; c += 4 * of) {
            float v[AT_ONCE][4];
#pragma unroll
            for (int i = 0; i < AT_ONCE; ++i) {
                if (i >= kp.K - 1) break;
                const int rel = qlen - (kp.K - 1) + i;
                if (rel >= 0) Quad<T>::load(xbc + (size_t)rel * kp.ld + c, v[i]);
                else Quad<float>::load(kept + (size_t)(i + qlen) * kp.C + c, v[i]);
            }
#pragma unroll
            for (int i = 0; i < AT_ONCE; ++i) {
                if (i >= kp.K - 1) break;
                Quad<float>::store(kept + (size_t)i * kp.C + c, v[i]);
            }
        }
        return;
    }
    for (int c = who; c < kp.C; c += of)
        for (int i = 0; i < kp.K - 1; ++i) {         // ascending: what is read lies ahead
            const int rel = qlen - (kp.K - 1) + i;
            kept[(size_t)i * kp.C + c] = rel >= 0 ? to_float(xbc[(size_t)rel * kp.ld + c])
                                                  : kept[(size_t)(i + qlen) * kp.C + c];
        }
}

// A block a (token, part).
template <typename T>
__global__ void gated_group_norm_kernel(const float* __restrict__ y, const T* __restrict__ z,
                                        int ldz, const float* __restrict__ weight,
                                        T* __restrict__ out, int cols, int parts, float eps,
                                        Keep kp) {
    __shared__ float scratch[33];
    const int n = blockIdx.x, part = cols / parts, base = blockIdx.y * part;
    const float* yr = y + (size_t)n * cols + base;
    const T* zr = z + (size_t)n * ldz + base;
    pdl_wait();
    keep_inputs<T>(kp, n, blockIdx.y * blockDim.x + threadIdx.x, gridDim.y * blockDim.x);
    float ss = 0.0f;
    for (int i = threadIdx.x; i < part; i += blockDim.x) {
        const float v = yr[i] * silu_f(to_float(zr[i]));
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    for (int i = threadIdx.x; i < part; i += blockDim.x)
        out[(size_t)n * cols + base + i] =
            from_float<T>(yr[i] * silu_f(to_float(zr[i])) * inv * weight[base + i]);
    pdl_trigger();
}

// Rows of whole quads, parts of at most 128 QUADS elements: `warps` warps a part, each thread
// holding QUADS groups of four elements in registers.  A block takes parts of several warps of one
// token.
template <typename T, int QUADS>
__global__ void gated_group_norm_quads_kernel(const float* __restrict__ y, const T* __restrict__ z,
                                              int ldz, const float* __restrict__ weight,
                                              T* __restrict__ out, int cols, int parts, int warps,
                                              float eps, Keep kp) {
    __shared__ float scratch[32];
    const int n = blockIdx.x, part = cols / parts, width = 32 * warps;
    const int mine = blockIdx.y * (blockDim.x / width) + threadIdx.x / width;
    const int lane = threadIdx.x % width, warp = threadIdx.x >> 5;
    const size_t base = (size_t)mine * part;
    const bool live = mine < parts;
    pdl_wait();
    keep_inputs<T>(kp, n, blockIdx.y * blockDim.x + threadIdx.x, gridDim.y * blockDim.x);
    float v[QUADS][4], ss = 0.0f;
#pragma unroll
    for (int u = 0; u < QUADS; ++u) {
        const int i = 4 * (lane + u * width);
        if (live && i < part) {
            float b[4];
            Quad<float>::load(y + (size_t)n * cols + base + i, v[u]);
            Quad<T>::load(z + (size_t)n * ldz + base + i, b);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                v[u][e] *= silu_f(b[e]);
                ss = fmaf(v[u][e], v[u][e], ss);
            }
        }
    }
    ss = warp_sum(ss);
    if (warps > 1) {
        if ((threadIdx.x & 31) == 0) scratch[warp] = ss;
        __syncthreads();
        ss = 0.0f;
        for (int u = 0; u < warps; ++u) ss += scratch[warp / warps * warps + u];
    }
    const float inv = 1.0f / sqrtf(ss / (float)part + eps);
#pragma unroll
    for (int u = 0; u < QUADS; ++u) {
        const int i = 4 * (lane + u * width);
        if (live && i < part) {
            float w[4];
            Quad<float>::load(weight + base + i, w);
#pragma unroll
            for (int e = 0; e < 4; ++e) w[e] *= v[u][e] * inv;
            Quad<T>::store(out + (size_t)n * cols + base + i, w);
        }
    }
    pdl_trigger();
}

bool shape_ok(const Shape& s) {
    return s.H > 0 && s.G > 0 && s.H % s.G == 0 && s.N > 0 && s.N <= 256 && s.P > 0 && s.K > 0 &&
           s.H <= 65535;
}
bool aligned16(const void* p) { return (uintptr_t)p % 16 == 0; }

}  // namespace

DE_EXPORT int de_ssm_max_state() { return 256; }
DE_EXPORT int de_ssm_chunk() { return L; }

DE_EXPORT int de_ssm_prep(int dtype, const void* xbc, int ld, const void* dt, int ld_dt,
                          const float* taps, const float* bias, const float* dt_bias,
                          const float* a_log, const float* state, long long slot_stride,
                          int conv_offset, const int* token_seq, const int* token_slot,
                          const int* positions, const int* seq_pos0, float* out, float* rates,
                          int n, int H, int G, int N, int P, int K, void* stream) {
    if (n <= 0) return 0;
    const Shape sh = {H, G, N, P, K, H * P + 2 * G * N};
    if (!shape_ok(sh)) return -2;
    const Conv cv = {taps, bias, state, slot_stride, conv_offset};
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = sh.C % 4 == 0 && ld % 4 == 0 && aligned16(xbc) && aligned16(taps) &&
                     aligned16(bias) && aligned16(state) && slot_stride % 4 == 0 &&
                     conv_offset % 4 == 0 && aligned16(out);
#define PREP_ARGS(T)                                                                            \
    (const T*)xbc, ld, (const T*)dt, ld_dt, cv, dt_bias, a_log, token_seq, token_slot, positions, \
        seq_pos0, out, rates, sh
    if (vec && K <= 4) {
        const dim3 runs((n + RUN - 1) / RUN, (sh.C + 511) / 512);
        if (runs.y > 65535) return -2;
#define RUNS(T, KK)                                                                             \
    return de_launch(prep_run_kernel<T, KK>, runs, dim3(128), 0, s, PREP_ARGS(T), n)
#define BY_TAPS(T)                                                                              \
    do {                                                                                        \
        if (K == 1) RUNS(T, 1);                                                                 \
        if (K == 2) RUNS(T, 2);                                                                 \
        if (K == 3) RUNS(T, 3);                                                                 \
        RUNS(T, 4);                                                                             \
    } while (0)
        if (dtype == DE_BF16) BY_TAPS(__nv_bfloat16);
        BY_TAPS(float);
#undef BY_TAPS
#undef RUNS
    }
    const dim3 grid(n, (sh.C + 127) / 128);
    if (grid.y > 65535) return -2;
    if (dtype == DE_BF16)
        return de_launch(prep_kernel<__nv_bfloat16>, grid, dim3(128), 0, s,
                         PREP_ARGS(__nv_bfloat16));
    return de_launch(prep_kernel<float>, grid, dim3(128), 0, s, PREP_ARGS(float));
#undef PREP_ARGS
}

// fused 1: every sequence brings one token; xbc and dt are columns of the projection (type dtype).
// fused 0: `ready` and `rates` are prep's outputs, sequences beyond `longest` tokens are left out.
DE_EXPORT int de_ssm_walk(int dtype, int fused, const void* xbc, int ld, const void* dt, int ld_dt,
                          const float* taps, const float* bias, const float* dt_bias,
                          const float* a_log, const float* ready, const float* rates,
                          const float* skip, float* state, long long slot_stride, int conv_offset,
                          const int* seq_slot, const int* seq_qstart, const int* seq_qlen,
                          int n_seqs, int longest, float* y, int H, int G, int N, int P, int K,
                          void* stream) {
    if (n_seqs <= 0) return 0;
    const Shape sh = {H, G, N, P, K, H * P + 2 * G * N};
    if (!shape_ok(sh)) return -2;
    const Conv cv = {taps, bias, state, slot_stride, conv_offset};
    cudaStream_t s = (cudaStream_t)stream;
    const int vec = P % 4 == 0 && aligned16(state) && slot_stride % 4 == 0;
    const int cq = P <= 32 ? 8 : 16, pt = 4 * cq;
    const dim3 grid(n_seqs, H, (P + pt - 1) / pt);
    const size_t smem = (size_t)(pt + 2 * N) * sizeof(float);
    const int rg = 256 / cq, r = (N + rg - 1) / rg;
#define WALK(T, F, CQ, R)                                                                       \
    return de_launch(walk_kernel<T, F, CQ, R>, grid, dim3(256), smem, s, (const T*)xbc, ld,     \
                     (const T*)dt, ld_dt, cv, dt_bias, a_log, ready, rates, skip, state,        \
                     slot_stride, seq_slot, seq_qstart, seq_qlen, longest, y, sh, vec)
#define ROWS(T, F)                                                                              \
    do {                                                                                        \
        if (cq == 8) {                                                                          \
            if (r <= 2) WALK(T, F, 8, 2);                                                       \
            if (r <= 4) WALK(T, F, 8, 4);                                                       \
            WALK(T, F, 8, 8);                                                                   \
        }                                                                                       \
        if (r <= 4) WALK(T, F, 16, 4);                                                          \
        if (r <= 8) WALK(T, F, 16, 8);                                                          \
        WALK(T, F, 16, 16);                                                                     \
    } while (0)
    if (!fused) ROWS(float, false);
    if (dtype == DE_BF16) ROWS(__nv_bfloat16, true);
    ROWS(float, true);
#undef ROWS
#undef WALK
}

static int chunk_vec(const Shape& sh, const void* a, const void* b) {
    return sh.P % 4 == 0 && sh.N % 4 == 0 && aligned16(a) && aligned16(b);
}

DE_EXPORT int de_ssm_chunk_state(const float* xbc, const float* rates, const void* items,
                                 int n_items, float* out, float* decays, float* products, int H,
                                 int G, int N, int P, int K, void* stream) {
    if (n_items <= 0) return 0;
    const Shape sh = {H, G, N, P, K, H * P + 2 * G * N};
    if (!shape_ok(sh)) return -2;
    const dim3 grid(n_items, H, ((N + 63) / 64) * ((P + 63) / 64) + 1);
    if (grid.z > 65535) return -2;
    return de_launch(chunk_state_kernel, grid, dim3(128), 0, (cudaStream_t)stream, xbc, rates,
                     (const int4*)items, out, decays, products, sh, chunk_vec(sh, xbc, out));
}

DE_EXPORT int de_ssm_chunk_pass(float* out, const float* decays, const void* long_seqs, int n_long,
                                const int* seq_slot, float* state, long long slot_stride, int H,
                                int N, int P, void* stream) {
    if (n_long <= 0) return 0;
    const long long total = (long long)H * N * P;
    const bool vec = ((long long)N * P) % 4 == 0 && aligned16(out) && aligned16(state) &&
                     slot_stride % 4 == 0;
    const long long blocks = (total + (vec ? 1024 : 256) - 1) / (vec ? 1024 : 256);
    if (blocks > 65535) return -2;
    const dim3 grid(n_long, (unsigned)blocks);
    if (vec)
        return de_launch(chunk_pass_kernel<4>, grid, dim3(256), 0, (cudaStream_t)stream, out, decays,
                         (const int4*)long_seqs, seq_slot, state, slot_stride, H, N * P);
    return de_launch(chunk_pass_kernel<1>, grid, dim3(256), 0, (cudaStream_t)stream, out, decays,
                     (const int4*)long_seqs, seq_slot, state, slot_stride, H, N * P);
}

DE_EXPORT int de_ssm_chunk_out(const float* xbc, const float* rates, const void* items,
                               int n_items, const float* starts, const float* products,
                               const float* skip, float* y, int H, int G, int N, int P, int K, void* stream) {
    if (n_items <= 0) return 0;
    const Shape sh = {H, G, N, P, K, H * P + 2 * G * N};
    if (!shape_ok(sh)) return -2;
    const dim3 grid(n_items, H, (P + 63) / 64);
    return de_launch(chunk_out_kernel, grid, dim3(128), 0, (cudaStream_t)stream, xbc, rates,
                     (const int4*)items, starts, products, skip, y, sh,
                     chunk_vec(sh, xbc, starts) && aligned16(y));
}

// keep_K > 1: the slots' kept convolution inputs (keep_C columns of xbc) move on as well.
DE_EXPORT int de_gated_group_norm(int dtype, const float* y, const void* z, int ldz,
                                  const float* weight, void* out, int n, int cols, int parts,
                                  float eps, const void* xbc, int ld_xbc, int keep_C, int keep_K,
                                  int keep_offset, float* state, long long slot_stride,
                                  const int* token_seq, const int* positions, const int* seq_pos0,
                                  const int* seq_qlen, const int* seq_slot, void* stream) {
    if (n <= 0) return 0;
    if (parts <= 0 || cols <= 0 || cols % parts || parts > 65535) return -2;
    const bool keep_vec = keep_C % 4 == 0 && ld_xbc % 4 == 0 && keep_offset % 4 == 0 &&
                          slot_stride % 4 == 0 && aligned16(xbc) && aligned16(state);
    const Keep kp = {xbc, ld_xbc, keep_C, keep_K, keep_offset, keep_vec, state, slot_stride,
                     token_seq, positions, seq_pos0, seq_qlen, seq_slot};
    cudaStream_t s = (cudaStream_t)stream;
    const int part = cols / parts;
    const bool vec = part % 4 == 0 && ldz % 4 == 0 && aligned16(y) && aligned16(z) &&
                     aligned16(weight) && aligned16(out);
    if (vec && part <= 32 * 32 * 16) {
        // four quads a thread if the part has them; a power of two of warps, in blocks of at
        // least 256 threads where there are so many parts
        int warps = 1;
        while (warps < 32 && part > 128 * 4 * warps) warps <<= 1;
        int per = 1;
        while (per * warps < 8 && per < parts) per <<= 1;
        const dim3 grid(n, (parts + per - 1) / per), block(32 * warps * per);
#define NORM(T, Q)                                                                              \
    return de_launch(gated_group_norm_quads_kernel<T, Q>, grid, block, 0, s, y, (const T*)z,    \
                     ldz, weight, (T*)out, cols, parts, warps, eps, kp)
        if (dtype == DE_BF16) {
            if (part <= 128 * warps) NORM(__nv_bfloat16, 1);
            NORM(__nv_bfloat16, 4);
        }
        if (part <= 128 * warps) NORM(float, 1);
        NORM(float, 4);
#undef NORM
    }
    const int threads = part > 256 ? 512 : (part > 128 ? 256 : 128);
#define NORM(T)                                                                                 \
    return de_launch(gated_group_norm_kernel<T>, dim3(n, parts), dim3(threads), 0, s, y,        \
                     (const T*)z, ldz, weight, (T*)out, cols, parts, eps, kp)
    if (dtype == DE_BF16) NORM(__nv_bfloat16);
    NORM(float);
#undef NORM
}
