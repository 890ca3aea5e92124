// The residual stream of layers that norm what a sublayer returns (and read the stream as it is):
//
//   embed   x = E[tok] / rms(E[tok]) * w
//   join    x += y / rms(y) * w,  y a branch, or the sum of two branches that are normed first:
//           y = m1 (y1 + b1) / rms(y1 + b1) * w1 + m2 (y2 + b2) / rms(y2 + b2) * w2
//
// with rms(v) = sqrt(mean(v^2) + eps), and, for layers that norm a branch on both sides with norms of any kind,
//
//   join_branch   x += m norm_1(y) (+ e);  h = norm_2(x),   norm(v) = (v - c mean(v)) / sqrt(mean((v - c mean(v))^2) + eps) * w + b
//
// with c 1 for a layer norm and 0 for an RMS norm.  Every kernel also leaves what the next sublayer reads: the new stream in the
// activations' dtype, or normed once more where the next layer has a norm of its own.  A block per row, the row held in
// registers, everything in float32, sums in an order that the row's length alone fixes.
#include "common.cuh"

namespace {

constexpr int MAX_THREADS = 1024;

// Sums of N numbers over the block (every thread gets them).  red: [2][N][32] floats, used in turn by successive calls.
template <int N>
__device__ __forceinline__ void block_sums(float (&v)[N], float* red, int& turn) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    float* r = red + turn * N * 32;
    turn ^= 1;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        v[i] = warp_sum(v[i]);
        if (lane == 0) r[i * 32 + warp] = v[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) {
        float t = 0.f;
        for (int w = 0; w < warps; ++w) t += r[i * 32 + w];
        v[i] = t;
    }
}

// VW neighbouring numbers of a row.
template <int VW> struct Piece { float v[VW]; };
template <int VW> __device__ __forceinline__ Piece<VW> load_piece(const float* p) {
    Piece<VW> r;
    if constexpr (VW == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VW> __device__ __forceinline__ Piece<VW> load_piece(const __nv_bfloat16* p) {
    Piece<VW> r;
    if constexpr (VW == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
    } else {
        r.v[0] = __bfloat162float(*p);
    }
    return r;
}
template <int VW> __device__ __forceinline__ void store_piece(float* p, const Piece<VW>& r) {
    if constexpr (VW == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VW> __device__ __forceinline__ void store_piece(__nv_bfloat16* p, const Piece<VW>& r) {
    if constexpr (VW == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

template <typename TW, typename TO, int NV, int VW>
__global__ void __launch_bounds__(MAX_THREADS) embedding_norm_kernel(const TW* __restrict__ table, const int* __restrict__ tokens,
                                                                     const float* __restrict__ gain, float* __restrict__ x,
                                                                     TO* __restrict__ h, int D, int V, float eps) {
    __shared__ float red[2 * 32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int tok = tokens[t], turn = 0;
    if (tok < 0 || tok >= V) tok = 0;            // range is checked on the host before launch
    const TW* row = table + (size_t)tok * D;
    Piece<VW> v[NV];
    float s[1] = {0.f};
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            v[i] = load_piece<VW>(row + d);
#pragma unroll
            for (int c = 0; c < VW; ++c) s[0] = fmaf(v[i].v[c], v[i].v[c], s[0]);
        }
    }
    block_sums(s, red, turn);
    const float scale = 1.f / sqrtf(s[0] / (float)D + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            const Piece<VW> g = load_piece<VW>(gain + d);
#pragma unroll
            for (int c = 0; c < VW; ++c) v[i].v[c] *= scale * g.v[c];
            store_piece(x + (size_t)t * D + d, v[i]);
            if (h) store_piece(h + (size_t)t * D + d, v[i]);
        }
    }
}

struct JoinArgs {
    const float *y1, *b1, *w1;       // first branch, its bias (or null), its own norm's weight (two branches)
    const float *y2, *b2, *w2;       // second branch (or null)
    float m1, m2, eps_in;
    const float* gain;
    float eps;
    float* x;
    void* h;                         // what the next sublayer reads, or null
    const float* next_gain;          // null: the stream itself
    float next_eps;
    int D;
};

template <typename TO, int NV, int VW, bool TWO>
__global__ void __launch_bounds__(MAX_THREADS) join_kernel(JoinArgs a) {
    __shared__ float red[2 * 2 * 32];
    pdl_launch_dependents();
    pdl_wait();
    const int D = a.D;
    const size_t at = (size_t)blockIdx.x * D;
    int turn = 0;
    Piece<VW> y[NV], z[TWO ? NV : 1];
    float s[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            y[i] = load_piece<VW>(a.y1 + at + d);
            if (a.b1) {
                const Piece<VW> b = load_piece<VW>(a.b1 + d);
#pragma unroll
                for (int c = 0; c < VW; ++c) y[i].v[c] += b.v[c];
            }
#pragma unroll
            for (int c = 0; c < VW; ++c) s[0] = fmaf(y[i].v[c], y[i].v[c], s[0]);
            if constexpr (TWO) {
                z[i] = load_piece<VW>(a.y2 + at + d);
                if (a.b2) {
                    const Piece<VW> b = load_piece<VW>(a.b2 + d);
#pragma unroll
                    for (int c = 0; c < VW; ++c) z[i].v[c] += b.v[c];
                }
#pragma unroll
                for (int c = 0; c < VW; ++c) s[1] = fmaf(z[i].v[c], z[i].v[c], s[1]);
            }
        }
    }
    block_sums(s, red, turn);
    if constexpr (TWO) {
        const float k1 = a.m1 / sqrtf(s[0] / (float)D + a.eps_in), k2 = a.m2 / sqrtf(s[1] / (float)D + a.eps_in);
        s[0] = s[1] = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int d = (threadIdx.x + i * blockDim.x) * VW;
            if (d < D) {
                const Piece<VW> w1 = load_piece<VW>(a.w1 + d), w2 = load_piece<VW>(a.w2 + d);
#pragma unroll
                for (int c = 0; c < VW; ++c) {
                    y[i].v[c] = y[i].v[c] * k1 * w1.v[c] + z[i].v[c] * k2 * w2.v[c];
                    s[0] = fmaf(y[i].v[c], y[i].v[c], s[0]);
                }
            }
        }
        block_sums(s, red, turn);
    }
    const float k = 1.f / sqrtf(s[0] / (float)D + a.eps);
    s[0] = s[1] = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            const Piece<VW> g = load_piece<VW>(a.gain + d);
            Piece<VW> x = load_piece<VW>(a.x + at + d);
#pragma unroll
            for (int c = 0; c < VW; ++c) {
                x.v[c] = x.v[c] + y[i].v[c] * k * g.v[c];
                s[0] = fmaf(x.v[c], x.v[c], s[0]);
            }
            store_piece(a.x + at + d, x);
            if (a.h && !a.next_gain) store_piece((TO*)a.h + at + d, x);
            y[i] = x;
        }
    }
    if (!a.h || !a.next_gain) return;
    block_sums(s, red, turn);
    const float kn = 1.f / sqrtf(s[0] / (float)D + a.next_eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            const Piece<VW> g = load_piece<VW>(a.next_gain + d);
#pragma unroll
            for (int c = 0; c < VW; ++c) y[i].v[c] *= kn * g.v[c];
            store_piece((TO*)a.h + at + d, y[i]);
        }
    }
}

struct AnyNorm {
    const float *w, *b;              // b or null
    float eps;
    int center;
};
struct JoinBranchArgs {
    const float* y;
    AnyNorm n1;
    float m;
    const float* extra;              // joins the stream as well (or null)
    float* x;
    void* h;                         // the rows of the norm that reads the stream next, or null
    AnyNorm n2;
    int D;
};

// v <- norm(v) without weight and bias; returns the factor, the mean is taken off in place.
template <int NV, int VW>
__device__ __forceinline__ float norm_factor(Piece<VW> (&v)[NV], int D, const AnyNorm& n, float* red, int& turn) {
    float s[1] = {0.f};
    if (n.center) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if ((threadIdx.x + i * blockDim.x) * VW < D)
#pragma unroll
                for (int c = 0; c < VW; ++c) s[0] += v[i].v[c];
        block_sums(s, red, turn);
        const float mean = s[0] / (float)D;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int c = 0; c < VW; ++c) v[i].v[c] -= mean;
    }
    s[0] = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
        if ((threadIdx.x + i * blockDim.x) * VW < D)
#pragma unroll
            for (int c = 0; c < VW; ++c) s[0] = fmaf(v[i].v[c], v[i].v[c], s[0]);
    block_sums(s, red, turn);
    return 1.f / sqrtf(s[0] / (float)D + n.eps);
}

template <typename TO, int NV, int VW>
__global__ void __launch_bounds__(MAX_THREADS) join_branch_kernel(const __grid_constant__ JoinBranchArgs a) {
    __shared__ float red[2 * 32];
    pdl_launch_dependents();
    pdl_wait();
    const int D = a.D;
    const size_t at = (size_t)blockIdx.x * D;
    int turn = 0;
    Piece<VW> y[NV], x[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            y[i] = load_piece<VW>(a.y + at + d);
            x[i] = load_piece<VW>(a.x + at + d);
        }
    }
    const float k = norm_factor<NV, VW>(y, D, a.n1, red, turn);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            const Piece<VW> w = load_piece<VW>(a.n1.w + d);
            Piece<VW> b{};
            if (a.n1.b) b = load_piece<VW>(a.n1.b + d);
#pragma unroll
            for (int c = 0; c < VW; ++c) x[i].v[c] = fmaf(a.m, fmaf(y[i].v[c] * k, w.v[c], b.v[c]), x[i].v[c]);
            if (a.extra) {
                const Piece<VW> e = load_piece<VW>(a.extra + at + d);
#pragma unroll
                for (int c = 0; c < VW; ++c) x[i].v[c] += e.v[c];
            }
            store_piece(a.x + at + d, x[i]);
        }
    }
    if (!a.h) return;
    const float kn = norm_factor<NV, VW>(x, D, a.n2, red, turn);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = (threadIdx.x + i * blockDim.x) * VW;
        if (d < D) {
            const Piece<VW> w = load_piece<VW>(a.n2.w + d);
            Piece<VW> b{};
            if (a.n2.b) b = load_piece<VW>(a.n2.b + d);
#pragma unroll
            for (int c = 0; c < VW; ++c) x[i].v[c] = fmaf(x[i].v[c] * kn, w.v[c], b.v[c]);
            store_piece((TO*)a.h + at + d, x[i]);
        }
    }
}

// Pieces a thread holds and threads of a block for rows of n pieces; 0 where the row is too long.
int shape_of(int n, int& threads) {
    threads = n < 256 ? (n + 31) / 32 * 32 : (n <= 1024 ? 256 : (n <= 2048 ? 512 : MAX_THREADS));
    const int nv = (n + threads - 1) / threads;
    return nv <= 1 ? 1 : nv <= 2 ? 2 : nv <= 4 ? 4 : nv <= 8 ? 8 : 0;
}

template <typename TO, int VW>
int join_launch(const JoinArgs& a, int T, cudaStream_t stream) {
    int threads = 0;
    const int nv = shape_of(a.D / VW, threads);
#define LQ_GO(NV) (a.y2 ? launch_pdl(join_kernel<TO, NV, VW, true>, dim3(T), dim3(threads), 0, stream, a) \
                        : launch_pdl(join_kernel<TO, NV, VW, false>, dim3(T), dim3(threads), 0, stream, a))
    switch (nv) {
        case 1: return LQ_GO(1);
        case 2: return LQ_GO(2);
        case 4: return LQ_GO(4);
        case 8: return LQ_GO(8);
    }
#undef LQ_GO
    return LQ_BAD_SIZE;
}

template <typename TO, int VW>
int join_branch_launch(const JoinBranchArgs& a, int T, cudaStream_t stream) {
    int threads = 0;
    const int nv = shape_of(a.D / VW, threads);
#define LQ_GO(NV) launch_pdl(join_branch_kernel<TO, NV, VW>, dim3(T), dim3(threads), 0, stream, a)
    switch (nv) {
        case 1: return LQ_GO(1);
        case 2: return LQ_GO(2);
        case 4: return LQ_GO(4);
        case 8: return LQ_GO(8);
    }
#undef LQ_GO
    return LQ_BAD_SIZE;
}

template <typename TW, typename TO, int VW>
int embed_launch(const void* table, const int* tokens, const float* gain, float* x, void* h, int T, int D, int V, float eps,
                 cudaStream_t stream) {
    int threads = 0;
    const int nv = shape_of(D / VW, threads);
#define LQ_GO(NV) launch_pdl(embedding_norm_kernel<TW, TO, NV, VW>, dim3(T), dim3(threads), 0, stream, (const TW*)table, tokens, gain, x, (TO*)h, D, V, eps)
    switch (nv) {
        case 1: return LQ_GO(1);
        case 2: return LQ_GO(2);
        case 4: return LQ_GO(4);
        case 8: return LQ_GO(8);
    }
#undef LQ_GO
    return LQ_BAD_SIZE;
}

}  // namespace

// x [T, D] float32 = the tokens' rows of the table [V, D], normed; h (or null): the same rows in h_dtype.
LQ_EXPORT int lq_embedding_norm(const void* table, int table_dtype, const int* tokens, const float* gain, float eps, float* x, void* h,
                                int h_dtype, int T, int D, int V, cudaStream_t stream) {
    if (T <= 0) return LQ_OK;
    typedef __nv_bfloat16 bf;
    if ((table_dtype != LQ_F32 && table_dtype != LQ_BF16) || (h_dtype != LQ_F32 && h_dtype != LQ_BF16)) return LQ_BAD_DTYPE;
    const bool vec = D % 4 == 0 && (((uintptr_t)table | (uintptr_t)gain | (uintptr_t)x | (uintptr_t)h) & 15) == 0;
#define LQ_GO(TW, TO) (vec ? embed_launch<TW, TO, 4>(table, tokens, gain, x, h, T, D, V, eps, stream) \
                           : embed_launch<TW, TO, 1>(table, tokens, gain, x, h, T, D, V, eps, stream))
    if (table_dtype == LQ_F32) return h_dtype == LQ_F32 ? LQ_GO(float, float) : LQ_GO(float, bf);
    return h_dtype == LQ_F32 ? LQ_GO(bf, float) : LQ_GO(bf, bf);
#undef LQ_GO
}

// One branch (y2 null; w1, m1, m2 and eps_in are not read) or two.  Biases may be null.  h (or null): see JoinArgs.
LQ_EXPORT int lq_join_normed(const float* y1, const float* b1, const float* w1, float m1, const float* y2, const float* b2,
                             const float* w2, float m2, float eps_in, const float* gain, float eps, float* x, void* h, int h_dtype,
                             const float* next_gain, float next_eps, int T, int D, cudaStream_t stream) {
    if (T <= 0) return LQ_OK;
    if (h_dtype != LQ_F32 && h_dtype != LQ_BF16) return LQ_BAD_DTYPE;
    if (y2 && (!w1 || !w2)) return LQ_BAD_SIZE;
    JoinArgs a{y1, b1, w1, y2, b2, w2, m1, m2, eps_in, gain, eps, x, h, next_gain, next_eps, D};
    const uintptr_t all = (uintptr_t)y1 | (uintptr_t)b1 | (uintptr_t)w1 | (uintptr_t)y2 | (uintptr_t)b2 | (uintptr_t)w2 | (uintptr_t)gain |
                          (uintptr_t)x | (uintptr_t)h | (uintptr_t)next_gain;
    const bool vec = D % 4 == 0 && (all & 15) == 0;
    typedef __nv_bfloat16 bf;
    if (h_dtype == LQ_F32) return vec ? join_launch<float, 4>(a, T, stream) : join_launch<float, 1>(a, T, stream);
    return vec ? join_launch<bf, 4>(a, T, stream) : join_launch<bf, 1>(a, T, stream);
}

// x += m norm(y; w1, b1, eps1) (+ extra), in place (float32 [T, D]); with h the rows of the norm (w2, b2, eps2) of the new
// stream in h_dtype.  center1, center2: the mean is taken off first (layer norms).  Biases and extra may be null.
LQ_EXPORT int lq_join_branch(const float* y, const float* w1, const float* b1, float eps1, int center1, float m, const float* extra, float* x,
                             void* h, int h_dtype, const float* w2, const float* b2, float eps2, int center2, int T, int D,
                             cudaStream_t stream) {
    if (T <= 0) return LQ_OK;
    if (h_dtype != LQ_F32 && h_dtype != LQ_BF16) return LQ_BAD_DTYPE;
    if (!w1 || (h && !w2)) return LQ_BAD_SIZE;
    JoinBranchArgs a{y, {w1, b1, eps1, center1}, m, extra, x, h, {w2, b2, eps2, center2}, D};
    const uintptr_t all = (uintptr_t)y | (uintptr_t)w1 | (uintptr_t)b1 | (uintptr_t)extra | (uintptr_t)x | (uintptr_t)h | (uintptr_t)w2 | (uintptr_t)b2;
    const bool vec = D % 4 == 0 && (all & 15) == 0;
    typedef __nv_bfloat16 bf;
    if (h_dtype == LQ_F32) return vec ? join_branch_launch<float, 4>(a, T, stream) : join_branch_launch<float, 1>(a, T, stream);
    return vec ? join_branch_launch<bf, 4>(a, T, stream) : join_branch_launch<bf, 1>(a, T, stream);
}

// ------------------------------------------------------------------ columns of a product's rows as another product's input
// The n columns at `off` of float32 rows, in the output's dtype, padded with zeros to `ld`.  split (bfloat16 only): out
// is [T, 2 ld], each number as the bfloat16 nearest to it and, ld columns on, the bfloat16 nearest to what is left, so that
// a product with the weight laid out twice sees the number to sixteen bits.
template <typename TO>
__global__ void __launch_bounds__(256) take_columns_kernel(const float* __restrict__ rows, int stride, int off, int n,
                                                           TO* __restrict__ out, int ld, int split, size_t total) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= total) return;
    const size_t t = i / ld;
    const int c = (int)(i % ld);
    const float v = c < n ? rows[t * stride + off + c] : 0.f;
    const TO hi = from_f32<TO>(v);
    out[t * ld * (split ? 2 : 1) + c] = hi;
    if (split) out[t * ld * 2 + ld + c] = from_f32<TO>(v - to_f32(hi));
}

LQ_EXPORT int lq_take_columns(const float* rows, int stride, int off, int n, void* out, int dtype, int ld, int split, int T,
                              cudaStream_t stream) {
    const size_t total = (size_t)T * ld;
    if (total == 0) return LQ_OK;
    if (n > ld || (split && dtype != LQ_BF16)) return LQ_BAD_SIZE;
    const dim3 grid((unsigned)((total + 255) / 256));
    if (dtype == LQ_F32) return launch_pdl(take_columns_kernel<float>, grid, dim3(256), 0, stream, rows, stride, off, n, (float*)out, ld, 0, total);
    if (dtype == LQ_BF16)
        return launch_pdl(take_columns_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, rows, stride, off, n, (__nv_bfloat16*)out, ld, split, total);
    return LQ_BAD_DTYPE;
}
