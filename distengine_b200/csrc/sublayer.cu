// Row kernels for blocks whose norm stands on a sublayer's output instead of its input, with a
// gate on that output, and for a stream that is a weighted average over the depth:
//
//   norm_stream        x <- x / sqrt(mean(x^2) + eps) * w in place on the float32 stream (the norm
//                      of the embedding rows), with a copy in the activation type
//   gated_normed_add   g = y * sigmoid(z + b);  out = x + g / sqrt(mean(g^2) + eps) * w
//                      y a sublayer's result, z the gate's product on the sublayer's input
//   depth_mix          x = sum over j < count of c[j] * X_j    (X_j the embedding rows and every
//                      layer's result so far, c a learned vector of the layer)
//   poly_norm          out = a N(z) + b N(z^2) + c N(z^3) + e, N dividing a row by its root mean
//                      square (eps inside the root), powers element by element
//   join_rmsnorm       x <- x + y / sqrt(mean(y^2) + eps) * w (+ v) and out = the RMS norm of the
//                      new x: the norm on a branch's result, the sum (with a vector v that every
//                      row receives) and the norm before the next branch in one pass; or out =
//                      the new x rounded, where the next branch reads the stream itself
//
// All sums, statistics and the stream are float32 whatever the activation type; every kernel that
// writes the stream can also write its rounding to the activation type, which the next matrix
// products read.  One block a row (depth_mix: a thread four elements); a row's sums have an order
// that depends on the block's size only.

#include "common.cuh"

DE_DEFINE_PDL_SWITCH

namespace {

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

template <typename T, typename W>
__global__ void norm_stream_kernel(float* __restrict__ x, const W* __restrict__ weight,
                                   T* __restrict__ rows, int width, float eps) {
    __shared__ float scratch[33];
    const size_t row = blockIdx.x;
    float* xr = x + row * width;
    pdl_wait();
    float ss = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) ss = fmaf(xr[i], xr[i], ss);
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
    pdl_trigger();
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = xr[i] * inv * to_float(weight[i]);
        xr[i] = v;
        if (rows != nullptr) rows[row * width + i] = from_float<T>(v);
    }
}

// Y: the sublayer's result (activation type or float32); T: the activation type of the gate's
// product and of the rounded copy.  `in` and `out` may be the same rows or different ones.
template <typename T, typename Y, typename W>
__global__ void gated_normed_add_kernel(const Y* __restrict__ y, const T* __restrict__ gate,
                                        int ld_gate, const float* __restrict__ bias,
                                        const W* __restrict__ weight, const float* in,
                                        float* out, T* __restrict__ rows, int width, float eps) {
    extern __shared__ float g[];                     // [width]
    __shared__ float scratch[33];
    const size_t row = blockIdx.x;
    pdl_wait();
    float ss = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = to_float(y[row * width + i]) *
                        sigmoid_f(to_float(gate[row * ld_gate + i]) + bias[i]);
        g[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
    pdl_trigger();
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = in[row * width + i] + g[i] * inv * to_float(weight[i]);
        out[row * width + i] = v;
        if (rows != nullptr) rows[row * width + i] = from_float<T>(v);
    }
}

// history [count][total] float32 with `stride` elements between two members.
template <typename T>
__global__ void depth_mix_kernel(const float* __restrict__ history, size_t stride,
                                 const float* __restrict__ coef, int count, size_t total,
                                 float* __restrict__ x, T* __restrict__ rows) {
    pdl_wait();
    pdl_trigger();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total;
         i += (size_t)gridDim.x * blockDim.x) {
        float s = 0.0f;
        for (int j = 0; j < count; ++j) s = fmaf(coef[j], history[j * stride + i], s);
        x[i] = s;
        if (rows != nullptr) rows[i] = from_float<T>(s);
    }
}

// 16 bytes of T as floats and back
template <typename T> struct Chunk;
template <> struct Chunk<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float* p, float* f) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* f) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    }
};
template <> struct Chunk<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* f) {
        const uint4 u = *reinterpret_cast<const uint4*>(p);
        const unsigned w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* f) {
        unsigned w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
            w[i] = *reinterpret_cast<const unsigned*>(&h);
        }
        *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
    }
};

// four neighbouring elements, 8 or 16 bytes
__device__ __forceinline__ void load4(const float* p, float (&f)[4]) { Chunk<float>::load(p, f); }
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(u.x << 16);
    f[1] = __uint_as_float(u.x & 0xffff0000u);
    f[2] = __uint_as_float(u.y << 16);
    f[3] = __uint_as_float(u.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) { Chunk<float>::store(p, f); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&f)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]);
    const __nv_bfloat162 b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a),
                                              *reinterpret_cast<const unsigned*>(&b));
}

// Three sums over a block at once; every thread gets the results.  The order of the additions
// depends on the block's size only.
__device__ __forceinline__ void block_sum3(float& a, float& b, float& c, float* scratch /* 99 */) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int warps = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    c = warp_sum(c);
    if (lane == 0) {
        scratch[warp] = a;
        scratch[32 + warp] = b;
        scratch[64 + warp] = c;
    }
    __syncthreads();
    if (warp < 3) {
        float t = lane < warps ? scratch[32 * warp + lane] : 0.0f;
        t = warp_sum(t);
        if (lane == 0) scratch[96 + warp] = t;
    }
    __syncthreads();
    a = scratch[96];
    b = scratch[97];
    c = scratch[98];
}

// VEC: rows are whole 16-byte pieces at 16-byte addresses; a thread then takes pieces, and the
// second pass finds the row in the caches.
template <typename T, bool VEC>
__global__ void poly_norm_kernel(const T* __restrict__ z, int ldz, const float* __restrict__ coef,
                                 T* __restrict__ out, int ldo, int cols, float eps) {
    __shared__ float scratch[99];
    constexpr int PN = Chunk<T>::N;
    const size_t row = blockIdx.x;
    const T* zr = z + row * ldz;
    pdl_wait();
    float s1 = 0.0f, s2 = 0.0f, s3 = 0.0f;
    if (VEC) {
        for (int i = threadIdx.x * PN; i < cols; i += blockDim.x * PN) {
            float f[PN];
            Chunk<T>::load(zr + i, f);
#pragma unroll
            for (int e = 0; e < PN; ++e) {
                const float v = f[e], v2 = v * v, v3 = v2 * v;
                s1 = fmaf(v, v, s1);
                s2 = fmaf(v2, v2, s2);
                s3 = fmaf(v3, v3, s3);
            }
        }
    } else {
        for (int i = threadIdx.x; i < cols; i += blockDim.x) {
            const float v = to_float(zr[i]), v2 = v * v, v3 = v2 * v;
            s1 = fmaf(v, v, s1);
            s2 = fmaf(v2, v2, s2);
            s3 = fmaf(v3, v3, s3);
        }
    }
    block_sum3(s1, s2, s3, scratch);
    const float n = (float)cols;
    const float i1 = coef[0] / sqrtf(s1 / n + eps);
    const float i2 = coef[1] / sqrtf(s2 / n + eps);
    const float i3 = coef[2] / sqrtf(s3 / n + eps);
    const float e0 = coef[3];
    pdl_trigger();
    if (VEC) {
        for (int i = threadIdx.x * PN; i < cols; i += blockDim.x * PN) {
            float f[PN];
            Chunk<T>::load(zr + i, f);
#pragma unroll
            for (int e = 0; e < PN; ++e) {
                const float v = f[e], v2 = v * v;
                f[e] = v * i1 + v2 * i2 + v2 * v * i3 + e0;
            }
            Chunk<T>::store(out + row * ldo + i, f);
        }
    } else {
        for (int i = threadIdx.x; i < cols; i += blockDim.x) {
            const float v = to_float(zr[i]), v2 = v * v;
            out[row * ldo + i] = from_float<T>(v * i1 + v2 * i2 + v2 * v * i3 + e0);
        }
    }
}

// Y: the branch's type; T: the output's; W: of both norm weights.  y null: no branch.  wy null: the
// branch joins as it is.  vec null: no vector.  out null: the sum only.  w null: out is the sum,
// rounded.  rows: out[i] is the norm
// of row rows[i], and x stays as it is.  A thread holds CHUNKS groups of four neighbouring elements
// of the row in registers (CHUNKS 0: the row lies in shared memory, any width).
// The branch may also come as the terms of a weighted sum (`mixed`): y holds `top` rows for each row
// of x, summed with weight[row][top], and, unless null, shared[row] times side[row] joins them.
struct Join {
    const void *wy, *w;
    const float* weight;       // null: y is the branch's rows
    const void* shared;        // of y's type
    const float* side;
    int top;
    const float* vec;
    const int* rows;
    int width;
    float eps_y, eps;
};

template <typename Y>
__device__ __forceinline__ float branch_at(const Y* __restrict__ y, const Join& j, size_t row, int i) {
    if (j.weight == nullptr) return to_float(y[row * j.width + i]);
    float s = 0.0f;
    for (int k = 0; k < j.top; ++k)
        s = fmaf(j.weight[row * j.top + k], to_float(y[(row * j.top + k) * j.width + i]), s);
    if (j.shared != nullptr)
        s = fmaf(j.side[row], to_float(((const Y*)j.shared)[row * j.width + i]), s);
    return s;
}
template <typename Y>
__device__ __forceinline__ void branch_at4(const Y* __restrict__ y, const Join& j, size_t row, int i,
                                           float (&b)[4]) {
    if (j.weight == nullptr) {
        load4(y + row * j.width + i, b);
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) b[e] = 0.0f;
#pragma unroll 4
    for (int k = 0; k < j.top; ++k) {
        const float w = j.weight[row * j.top + k];
        float t[4];
        load4(y + (row * j.top + k) * j.width + i, t);
#pragma unroll
        for (int e = 0; e < 4; ++e) b[e] = fmaf(w, t[e], b[e]);
    }
    if (j.shared != nullptr) {
        const float w = j.side[row];
        float t[4];
        load4((const Y*)j.shared + row * j.width + i, t);
#pragma unroll
        for (int e = 0; e < 4; ++e) b[e] = fmaf(w, t[e], b[e]);
    }
}

template <typename T, typename Y, typename W, int CHUNKS>
__global__ void join_rmsnorm_kernel(float* __restrict__ x, const Y* __restrict__ y,
                                    T* __restrict__ out, Join j) {
    __shared__ float scratch[33];
    const int row = j.rows ? j.rows[blockIdx.x] : (int)blockIdx.x;
    float* xr = x + (size_t)row * j.width;
    const W *wy = (const W*)j.wy, *w = (const W*)j.w;
    T* o = out ? out + (size_t)blockIdx.x * j.width : nullptr;
    pdl_wait();
    if constexpr (CHUNKS > 0) {
        const int quads = j.width >> 2;
        float v[CHUNKS][4], b[CHUNKS][4];
        float ss = 0.0f;
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int q = threadIdx.x + c * blockDim.x;
            if (q < quads) {
                load4(xr + 4 * q, v[c]);
                if (y) branch_at4(y, j, row, 4 * q, b[c]);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    if (!y) b[c][e] = 0.0f;
                    ss = fmaf(b[c][e], b[c][e], ss);
                }
            }
        }
        float inv = 1.0f;
        if (wy) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)j.width + j.eps_y);
        ss = 0.0f;
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int q = threadIdx.x + c * blockDim.x;
            if (q < quads) {
                float g[4] = {1.0f, 1.0f, 1.0f, 1.0f}, a[4] = {0.0f, 0.0f, 0.0f, 0.0f};
                if (wy) load4(wy + 4 * q, g);
                if (j.vec) load4(j.vec + 4 * q, a);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    v[c][e] = v[c][e] + b[c][e] * inv * g[e] + a[e];
                    ss = fmaf(v[c][e], v[c][e], ss);
                }
                if (!j.rows) store4(xr + 4 * q, v[c]);
            }
        }
        if (!o) return;
        if (!w) {
            pdl_trigger();
#pragma unroll
            for (int c = 0; c < CHUNKS; ++c) {
                const int q = threadIdx.x + c * blockDim.x;
                if (q < quads) store4(o + 4 * q, v[c]);
            }
            return;
        }
        inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)j.width + j.eps);
        pdl_trigger();
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int q = threadIdx.x + c * blockDim.x;
            if (q < quads) {
                float g[4];
                load4(w + 4 * q, g);
#pragma unroll
                for (int e = 0; e < 4; ++e) g[e] = v[c][e] * inv * g[e];
                store4(o + 4 * q, g);
            }
        }
    } else {
        extern __shared__ float held[];              // [width]
        float inv = 1.0f, ss = 0.0f;
        for (int i = threadIdx.x; i < j.width; i += blockDim.x) {
            const float b = y ? branch_at(y, j, row, i) : 0.0f;
            held[i] = b;                             // (its own elements only, so no barrier)
            ss = fmaf(b, b, ss);
        }
        if (wy) {
            inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)j.width + j.eps_y);
        }
        ss = 0.0f;
        for (int i = threadIdx.x; i < j.width; i += blockDim.x) {
            const float v = xr[i] + held[i] * inv * (wy ? to_float(wy[i]) : 1.0f) +
                            (j.vec ? j.vec[i] : 0.0f);
            held[i] = v;
            ss = fmaf(v, v, ss);
            if (!j.rows) xr[i] = v;
        }
        if (!o) return;
        if (!w) {
            pdl_trigger();
            for (int i = threadIdx.x; i < j.width; i += blockDim.x) o[i] = from_float<T>(held[i]);
            return;
        }
        inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)j.width + j.eps);
        pdl_trigger();
        for (int i = threadIdx.x; i < j.width; i += blockDim.x)
            o[i] = from_float<T>(held[i] * inv * to_float(w[i]));
    }
}

int row_threads(int width) { return width >= 2048 ? 512 : (width >= 512 ? 256 : 128); }

}  // namespace

DE_EXPORT int de_norm_stream(int dtype, int weight_dtype, float* x, const void* weight, void* rows,
                             int n, int width, float eps, void* stream) {
    if (n <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = row_threads(width);
#define NS(T, W)                                                                                 \
    return de_launch(norm_stream_kernel<T, W>, dim3(n), dim3(threads), 0, s, x, (const W*)weight, \
                     (T*)rows, width, eps)
    if (dtype == DE_BF16) {
        if (weight_dtype == DE_BF16) NS(__nv_bfloat16, __nv_bfloat16);
        NS(__nv_bfloat16, float);
    }
    if (weight_dtype == DE_BF16) NS(float, __nv_bfloat16);
    NS(float, float);
#undef NS
}

// dtype: of gate and rows; y_dtype: of y.
DE_EXPORT int de_gated_normed_add(int dtype, int y_dtype, int weight_dtype, const void* y,
                                  const void* gate, int ld_gate, const float* bias,
                                  const void* weight, const float* in, float* out, void* rows,
                                  int n, int width, float eps, void* stream) {
    if (n <= 0) return 0;
    if (dtype == DE_F32 && y_dtype != DE_F32) return -2;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = row_threads(width);
    const size_t smem = (size_t)width * sizeof(float);
#define GNA(T, Y, W)                                                                             \
    do {                                                                                         \
        if (smem > 48 * 1024) {                                                                  \
            cudaError_t e = cudaFuncSetAttribute(gated_normed_add_kernel<T, Y, W>,               \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                                 (int)smem);                                     \
            if (e != cudaSuccess) return (int)e;                                                 \
        }                                                                                        \
        return de_launch(gated_normed_add_kernel<T, Y, W>, dim3(n), dim3(threads), smem, s,      \
                         (const Y*)y, (const T*)gate, ld_gate, bias, (const W*)weight, in, out,  \
                         (T*)rows, width, eps);                                                  \
    } while (0)
    if (dtype == DE_BF16) {
        if (y_dtype == DE_BF16) {
            if (weight_dtype == DE_BF16) GNA(__nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
            GNA(__nv_bfloat16, __nv_bfloat16, float);
        }
        if (weight_dtype == DE_BF16) GNA(__nv_bfloat16, float, __nv_bfloat16);
        GNA(__nv_bfloat16, float, float);
    }
    if (weight_dtype == DE_BF16) GNA(float, float, __nv_bfloat16);
    GNA(float, float, float);
#undef GNA
}

DE_EXPORT int de_depth_mix(int dtype, const float* history, long long stride, const float* coef,
                           int count, long long total, float* x, void* rows, void* stream) {
    if (total <= 0 || count <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    size_t blocks = ((size_t)total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == DE_BF16)
        return de_launch(depth_mix_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, s,
                         history, (size_t)stride, coef, count, (size_t)total, x,
                         (__nv_bfloat16*)rows);
    return de_launch(depth_mix_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, s, history,
                     (size_t)stride, coef, count, (size_t)total, x, (float*)rows);
}

DE_EXPORT int de_poly_norm(int dtype, const void* z, int ldz, const float* coef, void* out,
                           int ldo, int n, int cols, float eps, void* stream) {
    if (n <= 0 || cols <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = row_threads(cols);
    const int pn = dtype == DE_BF16 ? 8 : 4;
    const bool vec = cols % pn == 0 && ldz % pn == 0 && ldo % pn == 0 &&
                     (uintptr_t)z % 16 == 0 && (uintptr_t)out % 16 == 0;
#define POLY(T, V)                                                                             \
    return de_launch(poly_norm_kernel<T, V>, dim3(n), dim3(threads), 0, s, (const T*)z, ldz,   \
                     coef, (T*)out, ldo, cols, eps)
    if (dtype == DE_BF16) {
        if (vec) POLY(__nv_bfloat16, true);
        POLY(__nv_bfloat16, false);
    }
    if (vec) POLY(float, true);
    POLY(float, false);
#undef POLY
}

// dtype: of out; y_dtype: of y; weight_dtype: of both weights.  mix (with top, shared, side): see
// Join.  n_out: rows of x, or of `rows`.
DE_EXPORT int de_join_rmsnorm(int dtype, int y_dtype, int weight_dtype, float* x, const void* y,
                              const float* mix, int top, const void* shared, const float* side,
                              const void* wy, float eps_y, const float* vec, const void* w,
                              float eps, void* out, const int* rows, int n_out, int width,
                              void* stream) {
    if (n_out <= 0) return 0;
    if (dtype == DE_F32 && y_dtype != DE_F32) return -2;
    cudaStream_t s = (cudaStream_t)stream;
    if (mix != nullptr && (y == nullptr || top <= 0 || (shared != nullptr && side == nullptr)))
        return -2;
    const Join j = {wy, w, mix, shared, side, top, vec, rows, width, eps_y, eps};
    const bool aligned = width % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)y % 16 == 0 &&
                         (uintptr_t)wy % 16 == 0 && (uintptr_t)vec % 16 == 0 &&
                         (uintptr_t)w % 16 == 0 && (uintptr_t)out % 16 == 0 &&
                         (uintptr_t)shared % 16 == 0;
    const int quads = width / 4;
    const size_t smem = (size_t)width * sizeof(float);
    if (smem > 200 * 1024) return -2;
#define JOIN_AS(T, Y, W, CH, TH, SM)                                                             \
    return de_launch(join_rmsnorm_kernel<T, Y, W, CH>, dim3(n_out), dim3(TH), SM, s, x,          \
                     (const Y*)y, (T*)out, j)
#define JOIN(T, Y, W)                                                                            \
    do {                                                                                         \
        if (aligned && quads <= 128) JOIN_AS(T, Y, W, 1, 128, 0);                                \
        if (aligned && quads <= 256) JOIN_AS(T, Y, W, 1, 256, 0);                                \
        if (aligned && quads <= 512) JOIN_AS(T, Y, W, 1, 512, 0);                                \
        if (aligned && quads <= 1024) JOIN_AS(T, Y, W, 2, 512, 0);                               \
        if (aligned && quads <= 2048) JOIN_AS(T, Y, W, 4, 512, 0);                               \
        if (smem > 48 * 1024) {                                                                  \
            cudaError_t e = cudaFuncSetAttribute(join_rmsnorm_kernel<T, Y, W, 0>,                \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                                 (int)smem);                                     \
            if (e != cudaSuccess) return (int)e;                                                 \
        }                                                                                        \
        JOIN_AS(T, Y, W, 0, row_threads(width), smem);                                           \
    } while (0)
    if (dtype == DE_BF16) {
        if (y_dtype == DE_BF16) {
            if (weight_dtype == DE_BF16) JOIN(__nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
            JOIN(__nv_bfloat16, __nv_bfloat16, float);
        }
        if (weight_dtype == DE_BF16) JOIN(__nv_bfloat16, float, __nv_bfloat16);
        JOIN(__nv_bfloat16, float, float);
    }
    if (weight_dtype == DE_BF16) JOIN(float, float, __nv_bfloat16);
    JOIN(float, float, float);
#undef JOIN
#undef JOIN_AS
}
