// The gated linear recurrence: a short causal convolution over time on every channel, two gates from
// a block-diagonal product, and a state per channel that decays by an input-dependent number.
//
//   u_t   = cb + sum_j taps[j] * (x_(t - K + 1 + j) + xb)      zeros before the sequence's start
//   r, i  = sigmoid(R_b u_b + rb), sigmoid(I_b u_b + ib)        per block b of n channels
//   a     = exp(-rate * r)                                      rate = 8 softplus(lambda)
//   S_t   = a S_(t-1) + sqrt(1 - a^2) i u
//   out_t = S_t * gelu(y_t + yb) * scale
//
// x and y are columns of the layer's stacked projection.  A slot holds the channels' S (float32)
// and, K > 1, a ring of K rows: row p mod K is the projection x (without bias) of position p.  One
// row more than the convolution looks back, so a step of single tokens may write position p's row
// while other blocks still read the rows of p - 1 ... p - K + 1.
//
// A recurrence that multiplies and adds composes: over tokens s+1 ... t, S_t = P S_s + L.  Steps are
// cut into chunks of CHUNK consecutive tokens of the *flat* batch, wherever sequences begin and end:
// a sequence's first token of the step takes its S from the slot and has P = 0, so nothing of what
// precedes it in the chunk gets through.
//
//   conv    u of every token as the sum of two bfloat16 terms (16 bits of mantissa), in memory
//   gates   one block a chunk and 64 channels: both gate products, a and the input's factor, then P
//           and L of every token from the chunk's start on (in segments that are joined), to memory
//   carry   S at every chunk's start, channel by channel along the chunks
//   out     S_t = L + P S_start, the output branch, the slots' new S and kept rows
//   step    single tokens (bfloat16): all of it in one kernel, 16 sequences and 32 channels a block
//
// Everything is float32 except x, y, the gates' matrices and out, which have the activation type.
// For float32, and for blocks that are not whole 16-byte pieces, there is a gates kernel that forms
// u itself and works in plain float32.  With bfloat16 operands the exponentials, quotients and roots are the hardware's
// float32 approximations (a few units in the last place); with float32 ones the library's.

#include "common.cuh"

DE_DEFINE_PDL_SWITCH

namespace {

constexpr int CHUNK = 64;        // tokens of a chunk, rows of a block of the gates kernel
constexpr int OT = 64;           // channels of a block of the gates kernel
constexpr int KS = 64;           // channels of u that are staged at a time
constexpr int LDW = KS + 8;      // row stride of staged operands of the tensor cores
constexpr int THREADS = 256;
constexpr int SEGMENTS = THREADS / OT;
constexpr int MAX_TAPS = 16;
constexpr int STEP_ROWS = 16;    // sequences of a block of the step kernel
constexpr int STEP_OT = 32;      // and its channels

struct Lru {
    const void* x;
    int ldx;
    const void* y;
    int ldy;
    const float *xb, *yb;        // [W]
    const float *taps, *cb;      // [K][W], [W]
    const void *ra, *ri;         // [W][n], row b n + o: output o of block b
    const float *rb, *ib;        // [W]
    const float* rate;           // [W]
    float* state;
    long long slot_stride;
    int ring;                    // where a slot's kept rows begin
    int K, W, n, N;
    const int *token_seq, *token_slot, *positions, *seq_pos0, *seq_qlen;
    void* out;
    int ldo;
    float scale;
};

template <bool FAST> __device__ __forceinline__ float sigmoid_f(float x) {
    if constexpr (FAST) return __fdividef(1.0f, 1.0f + __expf(-x));   // (x far below 0: 1 / inf = 0)
    return 1.0f / (1.0f + expf(-x));
}
// z (1 + tanh(t)) / 2 is z sigmoid(2 t)
template <bool FAST> __device__ __forceinline__ float gelu(float z) {
    if constexpr (FAST)
        return z * sigmoid_f<true>(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));
    return de_activate(z, 3);
}

__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int bytes = ok ? 16 : 0;                     // 0: sixteen zero bytes, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src), "r"(bytes)
                 : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int LEFT> __device__ __forceinline__ void cp_wait() {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(LEFT) : "memory");
}
__device__ __forceinline__ void ldmatrix4(unsigned (&f)[4], const void* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(f[0]), "=r"(f[1]), "=r"(f[2]), "=r"(f[3]) : "r"(a));
}
__device__ __forceinline__ void mma16816(float (&c)[4], unsigned a0, unsigned a1, unsigned a2,
                                         unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, "
                 "{%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// two floats as two terms each: hi rounds the float, low rounds what hi leaves
__device__ __forceinline__ void two_terms(float a, float b, unsigned& hi, unsigned& low) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - __bfloat162float(h.x),
                                                   b - __bfloat162float(h.y));
    hi = *reinterpret_cast<const unsigned*>(&h);
    low = *reinterpret_cast<const unsigned*>(&l);
}

// What a token's gates make of it: the decay and what joins the state; zr and zi with their biases.
// 1 - a^2 = 1 - e^x with x = 2 log a: by the exponential's series where x is small and the
// difference would lose its digits.
template <bool FAST>
__device__ __forceinline__ void gated(float rate, float zr, float zi, float u, float& a, float& b) {
    const float la = -rate * sigmoid_f<FAST>(zr);
    if constexpr (FAST) {
        const float x = 2.0f * la;
        a = __expf(la);
        float s = fmaf(x, 1.0f / 8.0f, 1.0f);
        s = fmaf(x * (1.0f / 7.0f), s, 1.0f);
        s = fmaf(x * (1.0f / 6.0f), s, 1.0f);
        s = fmaf(x * (1.0f / 5.0f), s, 1.0f);
        s = fmaf(x * (1.0f / 4.0f), s, 1.0f);
        s = fmaf(x * (1.0f / 3.0f), s, 1.0f);
        s = fmaf(x * 0.5f, s, 1.0f);
        const float keep = x > -0.5f ? -x * s : fmaf(-a, a, 1.0f);
        float root;
        asm("sqrt.approx.f32 %0, %1;\n" : "=f"(root) : "f"(keep));
        b = root * sigmoid_f<true>(zi) * u;
    } else {
        a = expf(la);
        b = sqrtf(-expm1f(2.0f * la)) * sigmoid_f<false>(zi) * u;
    }
}
template <typename T>
__device__ __forceinline__ float branch(const Lru& p, int token, int c) {
    return gelu<sizeof(T) == 2>(to_float(((const T*)p.y)[(size_t)token * p.ldy + c]) + p.yb[c]);
}
__device__ __forceinline__ void load_pair(const float* p, float& a, float& b) {
    a = p[0];
    b = p[1];
}
__device__ __forceinline__ void load_pair(const __nv_bfloat16* p, float& a, float& b) {
    const unsigned u = *reinterpret_cast<const unsigned*>(p);          // (an even place)
    a = __uint_as_float(u << 16);
    b = __uint_as_float(u & 0xffff0000u);
}

// ------------------------------------------------------------------------------------- gates
// P and L along the chunk of one block, from a and b in shared memory: a thread takes a channel of a
// segment of LEN tokens, then what the segments before it bring.  ch: the thread's channel (mine:
// it exists).
constexpr int LEN = CHUNK / SEGMENTS;
__device__ __forceinline__ void scan_chunk(const Lru& p, const float* As, const float* Bs, float* seg,
                                           const int* off_s, const int* slot_s, int n0, int count,
                                           int ch, bool mine, float* __restrict__ prod,
                                           float* __restrict__ local) {
    const int oc = threadIdx.x % OT, sg = threadIdx.x / OT, m0 = sg * LEN;
    float P[LEN], L[LEN], p1 = 1.0f, l1 = 0.0f;
#pragma unroll
    for (int i = 0; i < LEN; ++i) {
        const int m = m0 + i;
        const float a = As[m * (OT + 1) + oc], b = Bs[m * (OT + 1) + oc];
        if (off_s[m] == 0) {                           // a sequence begins: the same for the warp
            l1 = mine ? p.state[(size_t)slot_s[m] * p.slot_stride + ch] : 0.0f;
            p1 = 0.0f;
        }
        l1 = fmaf(a, l1, b);
        p1 *= a;
        P[i] = p1;
        L[i] = l1;
    }
    // (behind the last token of the step nothing reads the segment's end)
    seg[(sg * OT + oc) * 2] = p1;
    seg[(sg * OT + oc) * 2 + 1] = l1;
    __syncthreads();
    float Pb = 1.0f, Lb = 0.0f;
    for (int q = 0; q < sg; ++q) {
        const float pq = seg[(q * OT + oc) * 2], lq = seg[(q * OT + oc) * 2 + 1];
        Lb = fmaf(pq, Lb, lq);
        Pb *= pq;
    }
    if (!mine) return;
    float* pr = prod + (size_t)(n0 + m0) * p.W + ch;
    float* lo = local + (size_t)(n0 + m0) * p.W + ch;
#pragma unroll
    for (int i = 0; i < LEN; ++i) {
        if (m0 + i < count) {
            pr[(size_t)i * p.W] = P[i] * Pb;
            lo[(size_t)i * p.W] = fmaf(P[i], Lb, L[i]);
        }
    }
}

// u of four tokens and eight channels a thread (the channels of a part are whole pieces of eight).
constexpr int CONV_ROWS = 4;
__global__ void __launch_bounds__(128) lru_conv_kernel(Lru p, __nv_bfloat16* __restrict__ uh,
                                                       __nv_bfloat16* __restrict__ ul) {
    const int c = 8 * (blockIdx.y * 128 + threadIdx.x), t0 = blockIdx.x * CONV_ROWS, back = p.K - 1;
    int pos[CONV_ROWS], off[CONV_ROWS], slot[CONV_ROWS];
#pragma unroll
    for (int i = 0; i < CONV_ROWS; ++i) {
        const int t = min(t0 + i, p.N - 1);
        pos[i] = p.positions[t];
        off[i] = pos[i] - p.seq_pos0[p.token_seq[t]];
        slot[i] = p.token_slot[t];
    }
    const bool in = c < p.W;
    float u[CONV_ROWS][8], b[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        b[e] = in ? p.xb[c + e] : 0.0f;
        u[0][e] = in ? p.cb[c + e] : 0.0f;
#pragma unroll
        for (int i = 1; i < CONV_ROWS; ++i) u[i][e] = u[0][e];
    }
    pdl_wait();
    if (in) {
        const __nv_bfloat16* x = (const __nv_bfloat16*)p.x + c;
        for (int j = 0; j < p.K; ++j) {
            float t[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) t[e] = p.taps[(size_t)j * p.W + c + e];
#pragma unroll
            for (int i = 0; i < CONV_ROWS; ++i) {
                if (t0 + i >= p.N) continue;
                float v[8];
                if (off[i] + j >= back) {              // a token of this step
                    const uint4 q = *reinterpret_cast<const uint4*>(x + (size_t)(t0 + i - back + j) *
                                                                            p.ldx);
                    const unsigned w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        v[2 * e] = __uint_as_float(w[e] << 16);
                        v[2 * e + 1] = __uint_as_float(w[e] & 0xffff0000u);
                    }
                } else {
                    const int ps = pos[i] - back + j;
                    if (ps < 0) continue;              // before the sequence's start
                    const float* kept = p.state + (size_t)slot[i] * p.slot_stride + p.ring +
                                        (size_t)(ps % p.K) * p.W + c;
#pragma unroll
                    for (int e = 0; e < 8; ++e) v[e] = kept[e];
                }
#pragma unroll
                for (int e = 0; e < 8; ++e) u[i][e] = fmaf(t[e], v[e] + b[e], u[i][e]);
            }
        }
    }
    pdl_trigger();
    if (!in) return;
#pragma unroll
    for (int i = 0; i < CONV_ROWS; ++i) {
        if (t0 + i >= p.N) break;
        unsigned hi[4], low[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) two_terms(u[i][2 * e], u[i][2 * e + 1], hi[e], low[e]);
        const size_t at = (size_t)(t0 + i) * p.W + c;
        *reinterpret_cast<uint4*>(uh + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(ul + at) = make_uint4(low[0], low[1], low[2], low[3]);
    }
}

// On the tensor cores: a slab of 64 channels of the part at a time (rows of both matrices and of
// both terms of u, two slabs in flight), a warp 16 tokens and 32 channels of both gates.  The slab
// that holds the block's own channels comes last, so that their u is still there for the input.
__global__ void __launch_bounds__(THREADS, 3)
lru_gates_mma_kernel(Lru p, const __nv_bfloat16* __restrict__ uh, const __nv_bfloat16* __restrict__ ul,
                     float* __restrict__ prod, float* __restrict__ local) {
    using T = __nv_bfloat16;
    constexpr int STAGE = (2 * OT + 2 * CHUNK) * LDW;  // rows of r, of i, of u's terms
    extern __shared__ __align__(16) unsigned char raw[];
    T* stages = reinterpret_cast<T*>(raw);             // [2][STAGE]
    int* off_s = reinterpret_cast<int*>(stages + 2 * STAGE);       // [CHUNK] each
    int* slot_s = off_s + CHUNK;
    static_assert((2 * CHUNK * (OT + 1) + 2 * THREADS) * 4 <= STAGE * 2, "a stage holds a and b");

    const int tiles = (p.n + OT - 1) / OT;
    const int own = blockIdx.y % tiles, o0 = own * OT, c0 = blockIdx.y / tiles * p.n;
    const int n0 = blockIdx.x * CHUNK, count = min(CHUNK, p.N - n0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slabs = tiles;                           // (KS = OT)

    const int r0 = threadIdx.x >> 3, piece = 8 * (threadIdx.x & 7);
    const T* ra = (const T*)p.ra + (size_t)(c0 + o0 + r0) * p.n + piece;
    const T* ri = (const T*)p.ri + (size_t)(c0 + o0 + r0) * p.n + piece;
    const T* u1 = uh + (size_t)(n0 + r0) * p.W + c0 + piece;
    const T* u2 = ul + (size_t)(n0 + r0) * p.W + c0 + piece;
    auto load_w = [&](int k0, T* st) {
        T* d = st + r0 * LDW + piece;
#pragma unroll
        for (int i = 0; i < OT / 32; ++i) {
            const bool ok = o0 + r0 + 32 * i < p.n && k0 + piece < p.n;
            const size_t at = (size_t)(32 * i) * p.n + k0;
            cp16(d + 32 * i * LDW, ok ? ra + at : (const T*)p.ra, ok);
            cp16(d + (OT + 32 * i) * LDW, ok ? ri + at : (const T*)p.ri, ok);
        }
    };
    auto load_u = [&](int k0, T* st) {
        T* d = st + (2 * OT + r0) * LDW + piece;
#pragma unroll
        for (int i = 0; i < CHUNK / 32; ++i) {
            const bool ok = r0 + 32 * i < count && k0 + piece < p.n;
            const size_t at = (size_t)(32 * i) * p.W + k0;
            cp16(d + 32 * i * LDW, ok ? u1 + at : uh, ok);
            cp16(d + (CHUNK + 32 * i) * LDW, ok ? u2 + at : ul, ok);
        }
    };
    const auto slab_of = [&](int s) { return (own + 1 + s) % slabs * KS; };
    if (threadIdx.x < CHUNK) {
        const int m = threadIdx.x;
        off_s[m] = m < count ? p.positions[n0 + m] - p.seq_pos0[p.token_seq[n0 + m]] : 1;
        slot_s[m] = m < count ? p.token_slot[n0 + m] : 0;
    }
    load_w(slab_of(0), stages);
    pdl_wait();
    load_u(slab_of(0), stages);
    cp_commit();

    const int wm = warp >> 1, wn = warp & 1;
    float zr[4][4], zi[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) zr[j][e] = zi[j][e] = 0.0f;
    for (int s = 0; s < slabs; ++s) {
        T* st = stages + (s & 1) * STAGE;
        if (s + 1 < slabs) {
            T* next = stages + (~s & 1) * STAGE;
            load_w(slab_of(s + 1), next);
            load_u(slab_of(s + 1), next);
        }
        cp_commit();
        cp_wait<1>();
        __syncthreads();
        const int mat = lane >> 3, r8 = lane & 7;
        const T* ua = st + (2 * OT + wm * 16 + (mat & 1) * 8 + r8) * LDW + (mat >> 1) * 8;
        const T* wa = st + (wn * 32 + (mat >> 1) * 8 + r8) * LDW + (mat & 1) * 8;
#pragma unroll
        for (int kk = 0; kk < KS / 16; ++kk) {
            unsigned ah[4], al[4];
            ldmatrix4(ah, ua + kk * 16);
            ldmatrix4(al, ua + CHUNK * LDW + kk * 16);
#pragma unroll
            for (int g = 0; g < 2; ++g) {
                float(&z)[4][4] = g ? zi : zr;
#pragma unroll
                for (int j = 0; j < 4; j += 2) {
                    unsigned b[4];
                    ldmatrix4(b, wa + (g * OT + j * 8) * LDW + kk * 16);
                    mma16816(z[j], al[0], al[1], al[2], al[3], b[0], b[1]);
                    mma16816(z[j + 1], al[0], al[1], al[2], al[3], b[2], b[3]);
                    mma16816(z[j], ah[0], ah[1], ah[2], ah[3], b[0], b[1]);
                    mma16816(z[j + 1], ah[0], ah[1], ah[2], ah[3], b[2], b[3]);
                }
            }
        }
        if (s + 1 < slabs) __syncthreads();            // the stage may be loaded again
    }
    pdl_trigger();
    // gates, decays and inputs, into the stage that the last slab does not lie in
    const T* last = stages + ((slabs - 1) & 1) * STAGE + 2 * OT * LDW;
    float* As = reinterpret_cast<float*>(stages + (slabs & 1) * STAGE);
    float* Bs = As + CHUNK * (OT + 1);
    float* seg = Bs + CHUNK * (OT + 1);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int c = wn * 32 + j * 8 + 2 * (lane & 3), g = c0 + o0 + c;
        const bool in = o0 + c < p.n;                  // (n is even: both channels or none)
        float rb[2], ib[2], rate[2];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            rb[q] = in ? p.rb[g + q] : 0.0f;
            ib[q] = in ? p.ib[g + q] : 0.0f;
            rate[q] = in ? p.rate[g + q] : 0.0f;
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int m = wm * 16 + (lane >> 2) + 8 * e;
            float h[2], l[2];
            load_pair(last + m * LDW + c, h[0], h[1]);
            load_pair(last + (CHUNK + m) * LDW + c, l[0], l[1]);
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                float a, b;
                gated<true>(rate[q], zr[j][2 * e + q] + rb[q], zi[j][2 * e + q] + ib[q],
                            h[q] + l[q], a, b);
                As[m * (OT + 1) + c + q] = a;          // (rows and columns beyond the end: unused)
                Bs[m * (OT + 1) + c + q] = b;
            }
        }
    }
    __syncthreads();
    const int oc = threadIdx.x % OT;
    scan_chunk(p, As, Bs, seg, off_s, slot_s, n0, count, c0 + o0 + oc, o0 + oc < p.n, prod, local);
}

// In plain float32 arithmetic, any sizes; also single tokens (`single`).
template <typename T>
__global__ void __launch_bounds__(THREADS)
lru_gates_kernel(Lru p, float* __restrict__ prod, float* __restrict__ local, int single) {
    constexpr int WS = 2 * OT * LDW;                   // staged matrix rows: r, then i
    extern __shared__ __align__(16) unsigned char raw[];
    const int back = p.K - 1;                          // rows before the chunk that are staged too
    const int xs = (CHUNK + back) * KS;
    T* Ws = reinterpret_cast<T*>(raw);                 // [2][2 OT][LDW]
    T* Xs = Ws + 2 * WS;                               // [2][CHUNK + back][KS]
    unsigned char* after = reinterpret_cast<unsigned char*>(Xs + 2 * xs);
    float* Uf = reinterpret_cast<float*>(after);       // [CHUNK][KS + 1]
    float* Us = Uf + CHUNK * (KS + 1);                 // [CHUNK][OT + 1]
    int* pos_s = reinterpret_cast<int*>(Us + CHUNK * (OT + 1));    // [CHUNK] each
    int* off_s = pos_s + CHUNK;
    int* slot_s = off_s + CHUNK;
    float* As = reinterpret_cast<float*>(raw);         // [CHUNK][OT + 1] each, when the products are done
    float* Bs = As + CHUNK * (OT + 1);
    float* seg = Bs + CHUNK * (OT + 1);                // [SEGMENTS][OT][2]

    const int tiles = (p.n + OT - 1) / OT;
    const int blk = blockIdx.y / tiles, o0 = (blockIdx.y % tiles) * OT, c0 = blk * p.n;
    const int n0 = blockIdx.x * CHUNK, count = min(CHUNK, p.N - n0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* x = (const T*)p.x;

    auto load_w = [&](int k0, int st) {
        T* w = Ws + st * WS;
        for (int e = threadIdx.x; e < 2 * OT * KS; e += THREADS) {
            const int r = e / KS, k = k0 + e % KS, o = o0 + r % OT;
            const T* src = (const T*)(r < OT ? p.ra : p.ri);
            w[r * LDW + (k - k0)] = o < p.n && k < p.n ? src[(size_t)(c0 + o) * p.n + k]
                                                       : from_float<T>(0.0f);
        }
    };
    auto load_x = [&](int k0, int st) {
        T* d = Xs + st * xs;
        for (int e = threadIdx.x; e < (count + back) * KS; e += THREADS) {
            const int r = e / KS, k = k0 + e % KS, t = n0 - back + r;
            d[e] = t >= 0 && k < p.n ? x[(size_t)t * p.ldx + c0 + k] : from_float<T>(0.0f);
        }
    };

    if (threadIdx.x < CHUNK) {
        const int m = threadIdx.x;
        int ps = 0, of = 1, sl = 0;
        if (m < count) {
            ps = p.positions[n0 + m];
            of = ps - p.seq_pos0[p.token_seq[n0 + m]];
            sl = p.token_slot[n0 + m];
        }
        pos_s[m] = ps;
        off_s[m] = of;
        slot_s[m] = sl;
    }
    load_w(0, 0);
    pdl_wait();
    load_x(0, 0);

    // the products: a thread four tokens and four channels of both gates
    const int tm = threadIdx.x >> 4, tn = threadIdx.x & 15;
    float zr[4][4], zi[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) zr[j][e] = zi[j][e] = 0.0f;

    const int slabs = (p.n + KS - 1) / KS;
    bool plain = true;               // the warp's eight tokens look back at tokens of this step only
    for (int s = 0; s < slabs; ++s) {
        const int st = s & 1, k0 = s * KS;
        if (s + 1 < slabs) {
            load_w(k0 + KS, st ^ 1);
            load_x(k0 + KS, st ^ 1);
        }
        __syncthreads();
        {   // u of the slab: a thread two channels of eight tokens
            const int ch = 2 * lane, m0 = warp * (CHUNK / 8), c = c0 + k0 + ch;
            if (s == 0)
                for (int i = 0; i < CHUNK / 8; ++i) plain &= m0 + i >= count || off_s[m0 + i] >= back;
            const bool in0 = k0 + ch < p.n, in1 = k0 + ch + 1 < p.n;
            float u[CHUNK / 8][2];
            const float b0 = in0 ? p.xb[c] : 0.0f, b1 = in1 ? p.xb[c + 1] : 0.0f;
            const float d0 = in0 ? p.cb[c] : 0.0f, d1 = in1 ? p.cb[c + 1] : 0.0f;
#pragma unroll
            for (int i = 0; i < CHUNK / 8; ++i) {
                u[i][0] = d0;
                u[i][1] = d1;
            }
            const T* xr = Xs + st * xs + ch;
            for (int j = 0; j < p.K; ++j) {
                const float t0 = in0 ? p.taps[(size_t)j * p.W + c] : 0.0f;
                const float t1 = in1 ? p.taps[(size_t)j * p.W + c + 1] : 0.0f;
                if (plain) {
#pragma unroll
                    for (int i = 0; i < CHUNK / 8; ++i) {
                        float v0, v1;
                        load_pair(xr + (m0 + i + j) * KS, v0, v1);
                        u[i][0] = fmaf(t0, v0 + b0, u[i][0]);
                        u[i][1] = fmaf(t1, v1 + b1, u[i][1]);
                    }
                    continue;
                }
#pragma unroll
                for (int i = 0; i < CHUNK / 8; ++i) {
                    const int m = m0 + i;
                    if (m >= count) continue;
                    float v0, v1;
                    if (off_s[m] + j >= back) {        // a token of this step
                        v0 = to_float(xr[(m + j) * KS]);
                        v1 = to_float(xr[(m + j) * KS + 1]);
                    } else {
                        const int ps = pos_s[m] - back + j;
                        if (ps < 0) continue;          // before the sequence's start
                        const float* kept = p.state + (size_t)slot_s[m] * p.slot_stride + p.ring +
                                            (size_t)(ps % p.K) * p.W;
                        v0 = in0 ? kept[c] : 0.0f;
                        v1 = in1 ? kept[c + 1] : 0.0f;
                    }
                    u[i][0] = fmaf(t0, v0 + b0, u[i][0]);
                    u[i][1] = fmaf(t1, v1 + b1, u[i][1]);
                }
            }
            const int oc = k0 + ch - o0;               // the place among the block's own channels
#pragma unroll
            for (int i = 0; i < CHUNK / 8; ++i) {
                const int m = m0 + i;
                if (m >= count || !in0) u[i][0] = 0.0f;
                if (m >= count || !in1) u[i][1] = 0.0f;
                Uf[m * (KS + 1) + ch] = u[i][0];
                Uf[m * (KS + 1) + ch + 1] = u[i][1];
                if (oc >= 0 && oc < OT) {              // (KS = OT: a slab is all inside or all outside)
                    Us[m * (OT + 1) + oc] = u[i][0];
                    Us[m * (OT + 1) + oc + 1] = u[i][1];
                }
            }
        }
        __syncthreads();
        const T* w = Ws + st * WS;
        for (int k = 0; k < KS; ++k) {
            float uv[4], rv[4], iv[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                uv[e] = Uf[(tm * 4 + e) * (KS + 1) + k];
                rv[e] = to_float(w[(tn + 16 * e) * LDW + k]);
                iv[e] = to_float(w[(OT + tn + 16 * e) * LDW + k]);
            }
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) {
                    zr[a][b] = fmaf(uv[a], rv[b], zr[a][b]);
                    zi[a][b] = fmaf(uv[a], iv[b], zi[a][b]);
                }
        }
        __syncthreads();
    }
    pdl_trigger();
    // gates, decays and inputs
    constexpr bool FAST = sizeof(T) == 2;
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int c = tn + 16 * j, m = tm * 4 + 2 * q;     // and row m + 1
            const int g = c0 + o0 + c;
            const bool in = o0 + c < p.n;
            const float rb = in ? p.rb[g] : 0.0f, ib = in ? p.ib[g] : 0.0f;
            const float rate = in ? p.rate[g] : 0.0f;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float a, b;
                gated<FAST>(rate, zr[2 * q + e][j] + rb, zi[2 * q + e][j] + ib,
                            Us[(m + e) * (OT + 1) + c], a, b);
                As[(m + e) * (OT + 1) + c] = a;        // (rows and columns beyond the end: unused)
                Bs[(m + e) * (OT + 1) + c] = b;
            }
        }
    __syncthreads();
    const int oc = threadIdx.x % OT, sg = threadIdx.x / OT;
    const bool mine = o0 + oc < p.n;
    const int ch = c0 + o0 + oc;
    const int m0 = sg * LEN;
    if (single) {
        // every token is its sequence's only one of the step: no product reaches past it
        for (int m = m0; m < min(count, m0 + LEN); ++m) {
            if (!mine) break;
            float* row = p.state + (size_t)slot_s[m] * p.slot_stride;
            const float S = fmaf(As[m * (OT + 1) + oc], row[ch], Bs[m * (OT + 1) + oc]);
            row[ch] = S;
            if (p.K > 1)
                row[p.ring + (size_t)(pos_s[m] % p.K) * p.W + ch] =
                    to_float(x[(size_t)(n0 + m) * p.ldx + ch]);
            ((T*)p.out)[(size_t)(n0 + m) * p.ldo + ch] =
                from_float<T>(S * branch<T>(p, n0 + m, ch) * p.scale);
        }
        return;
    }
    scan_chunk(p, As, Bs, seg, off_s, slot_s, n0, count, ch, mine, prod, local);
}

// ------------------------------------------------------------------------------------- carry
// carry[k] = S before the first token of chunk k (0 for the first, whose tokens have P = 0).  A block
// takes 32 channels; its warps share the chunks out in consecutive runs, each forms what its run
// multiplies and adds, and then walks the run again from what the runs before it bring.
constexpr int RUNS = 8;
__global__ void __launch_bounds__(32 * RUNS)
lru_carry_kernel(const float* __restrict__ prod, const float* __restrict__ local,
                 float* __restrict__ carry, int W, int chunks) {
    __shared__ float Ps[RUNS][32], Ls[RUNS][32];
    const int lane = threadIdx.x & 31, run = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    const int len = (chunks + RUNS - 1) / RUNS, k0 = run * len, k1 = min(chunks, k0 + len);
    pdl_wait();
    float P = 1.0f, L = 0.0f;
    if (c < W) {
#pragma unroll 8
        for (int k = k0; k < k1; ++k) {
            if (k + 1 == chunks) break;                // the last chunk brings nothing to another
            const size_t at = (size_t)(k * CHUNK + CHUNK - 1) * W + c;
            const float pk = prod[at];
            L = fmaf(pk, L, local[at]);
            P *= pk;
        }
    }
    Ps[run][lane] = P;
    Ls[run][lane] = L;
    __syncthreads();
    pdl_trigger();
    if (c >= W) return;
    float S = 0.0f;
    for (int q = 0; q < run; ++q) S = fmaf(Ps[q][lane], S, Ls[q][lane]);
#pragma unroll 8
    for (int k = k0; k < k1; ++k) {
        carry[(size_t)k * W + c] = S;
        if (k + 1 == chunks) break;
        const size_t at = (size_t)(k * CHUNK + CHUNK - 1) * W + c;
        S = fmaf(prod[at], S, local[at]);
    }
}

// --------------------------------------------------------------------------------------- out
template <typename T> struct Four;                     // four neighbouring elements
template <> struct Four<float> {
    static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&f)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    }
};
template <> struct Four<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[4]) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        f[0] = __uint_as_float(u.x << 16);
        f[1] = __uint_as_float(u.x & 0xffff0000u);
        f[2] = __uint_as_float(u.y << 16);
        f[3] = __uint_as_float(u.y & 0xffff0000u);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[4]) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]);
        const __nv_bfloat162 b = __floats2bfloat162_rn(f[2], f[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a),
                                                  *reinterpret_cast<const unsigned*>(&b));
    }
};

// carry null: a single chunk.  VEC: four channels a thread.
template <typename T, bool VEC>
__global__ void lru_out_kernel(Lru p, const float* __restrict__ prod,
                               const float* __restrict__ local, const float* __restrict__ carry) {
    constexpr int E = VEC ? 4 : 1;
    const int t = blockIdx.x, seq = p.token_seq[t], pos = p.positions[t];
    const int left = p.seq_qlen[seq] - 1 - (pos - p.seq_pos0[seq]);   // tokens behind this one
    float* row = p.state + (size_t)p.token_slot[t] * p.slot_stride;
    const float* cr = carry ? carry + (size_t)(t / CHUNK) * p.W : nullptr;
    const T* x = (const T*)p.x + (size_t)t * p.ldx;
    const T* y = (const T*)p.y + (size_t)t * p.ldy;
    T* out = (T*)p.out + (size_t)t * p.ldo;
    pdl_wait();
    pdl_trigger();
    for (int c = threadIdx.x * E; c < p.W; c += blockDim.x * E) {
        float S[E], g[E];
        if constexpr (VEC) {
            float P[4], yb[4];
            Four<float>::load(local + (size_t)t * p.W + c, S);
            if (cr) {
                float s0[4];
                Four<float>::load(prod + (size_t)t * p.W + c, P);
                Four<float>::load(cr + c, s0);
#pragma unroll
                for (int e = 0; e < 4; ++e) S[e] = fmaf(P[e], s0[e], S[e]);
            }
            Four<T>::load(y + c, g);
            Four<float>::load(p.yb + c, yb);
#pragma unroll
            for (int e = 0; e < 4; ++e) g[e] = S[e] * gelu<sizeof(T) == 2>(g[e] + yb[e]) * p.scale;
            Four<T>::store(out + c, g);
            if (left == 0) Four<float>::store(row + c, S);
            if (p.K > 1 && left < p.K) {
                Four<T>::load(x + c, g);
                Four<float>::store(row + p.ring + (size_t)(pos % p.K) * p.W + c, g);
            }
        } else {
            S[0] = local[(size_t)t * p.W + c];
            if (cr) S[0] = fmaf(prod[(size_t)t * p.W + c], cr[c], S[0]);
            g[0] = S[0] * gelu<sizeof(T) == 2>(to_float(y[c]) + p.yb[c]) * p.scale;
            out[c] = from_float<T>(g[0]);
            if (left == 0) row[c] = S[0];
            if (p.K > 1 && left < p.K) row[p.ring + (size_t)(pos % p.K) * p.W + c] = to_float(x[c]);
        }
    }
}

// -------------------------------------------------------------------------------------- step
// Single tokens, bfloat16.  A block takes 16 sequences and 32 channels: u of the whole part that
// the channels' gates read, as two bfloat16 terms, in shared memory; the warps share the part out
// in pieces of 32 channels (their matrix rows are asked for before the wait for the kernel before
// this one) and their sums are added up in ascending order.
// TAPS: the convolution's, or 0 for any number of them.
template <int TAPS>
__global__ void __launch_bounds__(THREADS) lru_step_kernel(Lru p) {
    using T = __nv_bfloat16;
    extern __shared__ __align__(16) unsigned char raw[];
    const int np = (p.n + 31) / 32 * 32, ldu = np + 8;
    T* Uh = reinterpret_cast<T*>(raw);                 // [16][ldu]
    T* Ul = Uh + STEP_ROWS * ldu;
    float* Us = reinterpret_cast<float*>(Ul + STEP_ROWS * ldu);   // [16][32 + 1]
    constexpr int LDR = 2 * STEP_OT + 2;
    float* Red = Us + STEP_ROWS * (STEP_OT + 1);       // [8 warps][16][LDR]: r, then i
    __shared__ int pos_s[STEP_ROWS], slot_s[STEP_ROWS];
    __shared__ long long kept_s[STEP_ROWS][MAX_TAPS];  // where a row's kept inputs lie, or -1
    const int K = TAPS > 0 ? TAPS : p.K;

    const int tiles = (p.n + STEP_OT - 1) / STEP_OT;
    const int blk = blockIdx.y / tiles, o0 = (blockIdx.y % tiles) * STEP_OT, c0 = blk * p.n;
    const int n0 = blockIdx.x * STEP_ROWS, count = min(STEP_ROWS, p.N - n0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int pieces = np / 32;
    const T* x = (const T*)p.x;

    uint4 w[8];                                        // rows of r, then of i, 8 channels of each
    auto load_w = [&](int piece) {
        const int k = piece * 32 + 8 * tig;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int o = o0 + (j & 3) * 8 + gid;
            const T* src = (const T*)(j < 4 ? p.ra : p.ri);
            w[j] = o < p.n && k < p.n
                       ? __ldg(reinterpret_cast<const uint4*>(src + (size_t)(c0 + o) * p.n + k))
                       : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    if (warp < pieces) load_w(warp);
    // a thread's two results, and the two channels (of every `groups`-th row) whose u it forms
    const int rm = threadIdx.x >> 4, rc = 2 * (threadIdx.x & 15);
    const int ch = c0 + o0 + rc;
    const bool have = rm < count && o0 + rc < p.n;     // (n is even: both channels or none)
    float rb[2], ib[2], rate[2], yb[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        rb[e] = have ? p.rb[ch + e] : 0.0f;
        ib[e] = have ? p.ib[ch + e] : 0.0f;
        rate[e] = have ? p.rate[ch + e] : 0.0f;
        yb[e] = have ? p.yb[ch + e] : 0.0f;
    }
    {
        const int r = threadIdx.x / MAX_TAPS, j = threadIdx.x % MAX_TAPS, m = n0 + min(r, count - 1);
        const int pos = p.positions[m], slot = p.token_slot[m], ps = pos - (K - 1) + j;
        if (j == 0) {
            pos_s[r] = pos;
            slot_s[r] = slot;
        }
        // (nothing before the sequence's start; j = K - 1 is the token itself)
        kept_s[r][j] = r < count && j < K - 1 && ps >= 0
                           ? (long long)slot * p.slot_stride + p.ring + (long long)(ps % K) * p.W
                           : -1;
    }
    static_assert(THREADS == STEP_ROWS * MAX_TAPS, "a thread a row and tap");
    __syncthreads();
    pdl_wait();

    // what the last part needs of this thread's two results, asked for now
    float S0[2] = {0.0f, 0.0f}, yv[2] = {0.0f, 0.0f}, xv[2] = {0.0f, 0.0f};
    float* row = p.state + (size_t)slot_s[rm] * p.slot_stride;
    if (have) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            S0[e] = row[ch + e];
            yv[e] = to_float(((const T*)p.y)[(size_t)(n0 + rm) * p.ldy + ch + e]) + yb[e];
            xv[e] = to_float(x[(size_t)(n0 + rm) * p.ldx + ch + e]);
        }
    }
    const int half = np / 2, groups = max(1, THREADS / half);
    for (int pair = threadIdx.x % (THREADS / groups); pair < half; pair += THREADS / groups) {
        const int k = 2 * pair, c = c0 + k, oc = k - o0, r0 = threadIdx.x / (THREADS / groups);
        if (r0 >= groups) break;
        const bool in = k < p.n;
        const float2 none = make_float2(0.0f, 0.0f);
        auto pair_of = [&](const float* v) { return in ? *reinterpret_cast<const float2*>(v) : none; };
        const float2 b = pair_of(p.xb + c), d = pair_of(p.cb + c);
        for (int m0 = r0; m0 < STEP_ROWS; m0 += 4 * groups) {          // four rows at a time
            float u[4][2];
            auto add = [&](int i, const float2& t, const float2& v) {
                u[i][0] = fmaf(t.x, v.x + b.x, u[i][0]);
                u[i][1] = fmaf(t.y, v.y + b.y, u[i][1]);
            };
            auto kept = [&](long long at) {
                return at >= 0 && in ? *reinterpret_cast<const float2*>(p.state + at + c) : none;
            };
            float2 now[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int m = m0 + i * groups;
                now[i] = none;
                if (m < count && in) load_pair(x + (size_t)(n0 + m) * p.ldx + c, now[i].x, now[i].y);
                u[i][0] = d.x;
                u[i][1] = d.y;
            }
            if constexpr (TAPS > 1) {                  // everything is asked for at once
                float2 v[TAPS - 1][4];
                long long at[TAPS - 1][4];
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int m = min(m0 + i * groups, STEP_ROWS - 1);
                        at[j][i] = kept_s[m][j];
                        v[j][i] = kept(at[j][i]);
                    }
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const float2 t = pair_of(p.taps + (size_t)j * p.W + c);
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (at[j][i] >= 0) add(i, t, v[j][i]);
                }
            } else {
                for (int j = 0; j + 1 < K; ++j) {
                    const float2 t = pair_of(p.taps + (size_t)j * p.W + c);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const long long at = kept_s[min(m0 + i * groups, STEP_ROWS - 1)][j];
                        if (at >= 0) add(i, t, kept(at));
                    }
                }
            }
            const float2 t = pair_of(p.taps + (size_t)(K - 1) * p.W + c);
#pragma unroll
            for (int i = 0; i < 4; ++i) add(i, t, now[i]);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int m = m0 + i * groups;
                if (m >= STEP_ROWS) continue;
                if (m >= count || !in) u[i][0] = u[i][1] = 0.0f;
                unsigned hi, low;
                two_terms(u[i][0], u[i][1], hi, low);
                *reinterpret_cast<unsigned*>(Uh + m * ldu + k) = hi;
                *reinterpret_cast<unsigned*>(Ul + m * ldu + k) = low;
                if (oc >= 0 && oc < STEP_OT) {
                    Us[m * (STEP_OT + 1) + oc] = u[i][0];
                    Us[m * (STEP_OT + 1) + oc + 1] = u[i][1];
                }
            }
        }
    }
    __syncthreads();
    float z[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) z[j][e] = 0.0f;
    for (int piece = warp; piece < pieces; piece += THREADS / 32) {
        // a lane's eight channels of a row serve two products of 16: which channel stands in which
        // place of the product is free, as long as both operands agree
        const int k = piece * 32 + 8 * tig;
        const uint4 h0 = *reinterpret_cast<const uint4*>(Uh + gid * ldu + k);
        const uint4 h1 = *reinterpret_cast<const uint4*>(Uh + (gid + 8) * ldu + k);
        const uint4 l0 = *reinterpret_cast<const uint4*>(Ul + gid * ldu + k);
        const uint4 l1 = *reinterpret_cast<const uint4*>(Ul + (gid + 8) * ldu + k);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            mma16816(z[j], l0.x, l1.x, l0.y, l1.y, w[j].x, w[j].y);
            mma16816(z[j], l0.z, l1.z, l0.w, l1.w, w[j].z, w[j].w);
            mma16816(z[j], h0.x, h1.x, h0.y, h1.y, w[j].x, w[j].y);
            mma16816(z[j], h0.z, h1.z, h0.w, h1.w, w[j].z, w[j].w);
        }
        if (piece + THREADS / 32 < pieces) load_w(piece + THREADS / 32);
    }
    const int used = min(pieces, THREADS / 32);
    if (warp < used) {
        float* red = Red + (size_t)warp * STEP_ROWS * LDR;
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                red[(gid + 8 * (e >> 1)) * LDR + j * 8 + 2 * tig + (e & 1)] = z[j][e];
    }
    __syncthreads();
    pdl_trigger();
    if (!have) return;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        float zr = 0.0f, zi = 0.0f;
        for (int q = 0; q < used; ++q) {
            zr += Red[((size_t)q * STEP_ROWS + rm) * LDR + rc + e];
            zi += Red[((size_t)q * STEP_ROWS + rm) * LDR + STEP_OT + rc + e];
        }
        float a, b;
        gated<true>(rate[e], zr + rb[e], zi + ib[e], Us[rm * (STEP_OT + 1) + rc + e], a, b);
        const float S = fmaf(a, S0[e], b);
        row[ch + e] = S;
        if (K > 1) row[p.ring + (size_t)(pos_s[rm] % K) * p.W + ch + e] = xv[e];
        ((T*)p.out)[(size_t)(n0 + rm) * p.ldo + ch + e] =
            from_float<T>(S * gelu<true>(yv[e]) * p.scale);
    }
}

size_t gates_smem(int elem, int K) {
    return (size_t)elem * (2 * 2 * OT * LDW + 2 * (CHUNK + K - 1) * KS) + CHUNK * (KS + 1) * 4 +
           CHUNK * (OT + 1) * 4 + 3 * CHUNK * 4;
}
constexpr size_t MMA_SMEM = (size_t)2 * 2 * (2 * OT + 2 * CHUNK) * LDW + 2 * CHUNK * 4;
size_t step_smem(int n) {
    const int np = (n + 31) / 32 * 32;
    return (size_t)2 * 2 * STEP_ROWS * (np + 8) + STEP_ROWS * (STEP_OT + 1) * 4 +
           (size_t)(THREADS / 32) * STEP_ROWS * (2 * STEP_OT + 2) * 4;
}

template <typename F> int allow_smem(F kernel, size_t smem) {
    if (smem <= 48 * 1024) return 0;
    return de_check(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem));
}

template <typename T>
int launch_gates(const Lru& p, float* prod, float* local, int single, cudaStream_t s) {
    const size_t smem = gates_smem(sizeof(T), p.K);
    const int e = allow_smem(lru_gates_kernel<T>, smem);
    if (e) return e;
    const int tiles = (p.n + OT - 1) / OT;
    return de_launch(lru_gates_kernel<T>, dim3((p.N + CHUNK - 1) / CHUNK, p.W / p.n * tiles),
                     dim3(THREADS), smem, s, p, prod, local, single);
}

}  // namespace

DE_EXPORT int de_lru_chunk() { return CHUNK; }
DE_EXPORT int de_lru_max_taps() { return MAX_TAPS; }

// stage 0: gates (prod, local [N][W]; terms: room for u's two terms, 2 [N][W], or null); 1: carry
// ([chunks][W]); 2: out; 3: a step of single tokens.  dtype: of x, y, the matrices and out.
DE_EXPORT int de_lru(int stage, int dtype, const void* x, int ldx, const void* y, int ldy,
                     const float* xb, const float* yb, const float* taps, const float* cb,
                     const void* ra, const void* ri, const float* rb, const float* ib,
                     const float* rate, float* state, long long slot_stride, int ring, int K, int W,
                     int n, int N, const int* token_seq, const int* token_slot,
                     const int* positions, const int* seq_pos0, const int* seq_qlen, void* out,
                     int ldo, float scale, void* terms, float* prod, float* local, float* carry,
                     void* stream) {
    if (N <= 0) return 0;
    if (K < 1 || K > MAX_TAPS || n < 1 || W < 1 || W % n != 0) return -2;
    const Lru p = {x, ldx, y, ldy, xb, yb, taps, cb, ra, ri, rb, ib, rate, state, slot_stride,
                   ring, K, W, n, N, token_seq, token_slot, positions, seq_pos0, seq_qlen, out, ldo,
                   scale};
    cudaStream_t s = (cudaStream_t)stream;
    const bool bf16 = dtype == DE_BF16;
    const int chunks = (N + CHUNK - 1) / CHUNK;
    if (W / n * ((n + STEP_OT - 1) / STEP_OT) > 65535) return -2;
    // whole 16-byte pieces of the projection and of the matrices' rows
    const bool pieces = bf16 && n % 8 == 0 && ldx % 8 == 0 && (uintptr_t)x % 16 == 0 &&
                        (uintptr_t)ra % 16 == 0 && (uintptr_t)ri % 16 == 0;
    if (stage == 0 || stage == 3) {
        if (stage == 0 && (prod == nullptr || local == nullptr)) return -2;
        // (pairs of channels are read as one from the slots and from the vectors)
        const bool pairs = slot_stride % 2 == 0 && ring % 2 == 0 && (uintptr_t)state % 8 == 0 &&
                           (uintptr_t)xb % 8 == 0 && (uintptr_t)cb % 8 == 0 && (uintptr_t)taps % 8 == 0;
        if (stage == 3 && pieces && pairs && step_smem(n) <= 200 * 1024) {
            const size_t smem = step_smem(n);
            auto kernel = K == 2 ? lru_step_kernel<2> : K == 3 ? lru_step_kernel<3>
                          : K == 4 ? lru_step_kernel<4> : lru_step_kernel<0>;
            const int e = allow_smem(kernel, smem);
            if (e) return e;
            const int tiles = (n + STEP_OT - 1) / STEP_OT;
            return de_launch(kernel, dim3((N + STEP_ROWS - 1) / STEP_ROWS, W / n * tiles),
                             dim3(THREADS), smem, s, p);
        }
        const int single = stage == 3;
        if (pieces && !single && terms != nullptr && (uintptr_t)terms % 16 == 0) {
            __nv_bfloat16 *uh = (__nv_bfloat16*)terms, *ul = uh + (size_t)N * W;
            int e = de_launch(lru_conv_kernel, dim3((N + CONV_ROWS - 1) / CONV_ROWS, (W + 1023) / 1024),
                              dim3(128), 0, s, p, uh, ul);
            if (e) return e;
            e = allow_smem(lru_gates_mma_kernel, MMA_SMEM);
            if (e) return e;
            return de_launch(lru_gates_mma_kernel, dim3(chunks, W / n * ((n + OT - 1) / OT)),
                             dim3(THREADS), MMA_SMEM, s, p, (const __nv_bfloat16*)uh,
                             (const __nv_bfloat16*)ul, prod, local);
        }
        if (bf16) return launch_gates<__nv_bfloat16>(p, prod, local, single, s);
        return launch_gates<float>(p, prod, local, single, s);
    }
    if (stage == 1) {
        if (carry == nullptr) return -2;
        return de_launch(lru_carry_kernel, dim3((W + 31) / 32), dim3(32 * RUNS), 0, s, (const float*)prod,
                         (const float*)local, carry, W, chunks);
    }
    if (stage != 2 || (chunks > 1 && carry == nullptr)) return -2;
    const float* from = chunks > 1 ? carry : nullptr;
    const int threads = W >= 1024 ? 256 : 128;
    const int four = bf16 ? 8 : 16;                     // bytes of four elements
    const bool vec = W % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && ldo % 4 == 0 &&
                     slot_stride % 4 == 0 && ring % 4 == 0 && (uintptr_t)state % 16 == 0 &&
                     (uintptr_t)x % four == 0 && (uintptr_t)y % four == 0 &&
                     (uintptr_t)out % four == 0 && (uintptr_t)yb % 16 == 0 &&
                     (uintptr_t)prod % 16 == 0 && (uintptr_t)local % 16 == 0 &&
                     (uintptr_t)carry % 16 == 0;
#define OUT(T, V)                                                                             \
    return de_launch(lru_out_kernel<T, V>, dim3(N), dim3(threads), 0, s, p, (const float*)prod, \
                     (const float*)local, from)
    if (bf16) {
        if (vec) OUT(__nv_bfloat16, true);
        OUT(__nv_bfloat16, false);
    }
    if (vec) OUT(float, true);
    OUT(float, false);
#undef OUT
}
