// The gated delta rule with one decay per head, for prompts and portions.  Per head, with S [dk, dv] in float32:
//
//   S' = a_t S_(t-1)      u_t = b_t (v_t - S'^T k_t)      S_t = S' + k_t u_t^T      o_t = S_t^T q_t
//
// q, k (G key heads), v (H value heads; value head h reads key head h / (H / G)) come from projections whose channels each
// pass a causal convolution over time and silu; q and k are then unit vectors per head, x / sqrt(sum(x^2) + unit_eps), q also
// times q_scale; b = sigmoid(x_b); a = exp(-rate_h softplus(x_a + bias_h)).  A head's output leaves over its root mean square,
// times a weight that the heads share, times silu of a gate.  Everything is float32 (the logarithms of the decays are added
// up in float64, so that their differences keep their digits after a token that forgets nearly everything).
//
// A sequence's rows are cut into chunks of 64 tokens.  With l_t the sum of log a over a chunk's tokens up to t and S_0 the
// state ahead of the chunk,
//   u_t = b_t (v_t - e^(l_t) S_0^T k_t - sum_(s<t) e^(l_t - l_s) (k_t . k_s) u_s)
//   o_t = e^(l_t) S_0^T q_t + sum_(s<=t) e^(l_t - l_s) (q_t . k_s) u_s
//   S_64 = e^(l_64) S_0 + sum_s e^(l_64 - l_s) k_s u_s^T
// The sums over s < t are a unit lower triangle, so u = V' - W S_0 with V' and W the triangle's solutions for b v and
// b e^l k.  Three kernels:
//   prepare  (a block per chunk and head, all chunks at once): convolution, unit vectors, the triangle and its solutions
//   scan     (a block per sequence, head and some value columns; chunks one after the other): u, the state, S_0 of every chunk
//   output   (a block per chunk and head, all chunks at once): o, its norm, weight and gate
// Only the scan is a chain, one step per 64 tokens, and its steps are two small products.  The state takes a chunk's decay as
// S + (e^l - 1) S with e^l - 1 from expm1.
//
// Decays enter as e^(l_t - l_s) with s <= t only: never above one, and a decay of zero (a logarithm of -200 at least) is harmless.
#include "delta.cuh"

namespace {

constexpr int HC = 64;                // tokens of a chunk
constexpr int LT = HC + 4;            // row length of vectors laid out by channels, [channel][token]
constexpr int SC = 132;               // scalars of a (chunk, head): e^(l_t) [64], e^(l_64 - l_s) [64], e^(l_64) - 1, three unused
constexpr float LOG_FLOOR = -200.f;   // e^-200 is zero in float32: a decay of zero keeps a logarithm that can be added up

struct HeadDeltaArgs {
    const float* rows;                // [T, stride]: q at column 0, k, v, then b (H) at b_off, decays (H) at a_off, gate (H dv) at g_off
    int stride, b_off, a_off, g_off;
    const float* taps_w;              // [taps, C], C = 2 G dk + H dv
    int taps, C;
    float* ring;                      // [slots][taps][C]: the convolution's last inputs, position p in row p % taps
    const float* dt_bias;             // [H]
    const float* rate;                // [H]
    float* state;                     // [slots][H][dk][dv]
    const int* cu_rows;               // [B + 1]
    const int* slots;                 // [B]
    const int* tok_pos;               // [T]
    float *K, *Q;                     // [chunk][G][64][ld]
    float* W;                         // [chunk][H][64][ld]
    float* V;                         // [chunk][H][tiles][64][n]: V', then u
    float* N;                         // [chunk][H][64][64]
    float* S0;                        // [chunk][H][dk][tiles * n]
    float* sc;                        // [chunk][H][SC]
    const float* norm_w;              // [dv]
    float norm_eps;
    void* out;                        // [T, H dv]
    int out_bf16;
    int H, G, dk, dv, ld, n, tiles;
    float q_scale, unit_eps;
};

__host__ __device__ __forceinline__ int pad4(int n) { return (n + 3) / 4 * 4; }
// Rows of key channels: whole fours, an odd number of them, so that eight neighbouring rows start in different banks.
__host__ __device__ __forceinline__ int row_length(int dk) { const int p = pad4(dk) / 4; return 4 * (p % 2 ? p + 2 : p + 1); }
// Where the chunks of sequence b start: unique and never overlapping, whatever the sequences' lengths are.
__device__ __forceinline__ int first_chunk(const int* cu_rows, int b) { return cu_rows[b] / HC + b; }

// ------------------------------------------------------------------ prepare
// NT threads; TM: rows of a thread's tile of the triangle (4 columns wide).
template <int NT, int TM>
__global__ void __launch_bounds__(NT, NT == 128 ? 4 : 2) prepare_kernel(const __grid_constant__ HeadDeltaArgs a) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    __shared__ double sl[HC];
    __shared__ float sb[HC], se[HC], s_inv[2][HC];
    const int dk = a.dk, dv = a.dv, dk4 = pad4(dk), tid = threadIdx.x, h = blockIdx.z, b = blockIdx.y, rep = a.H / a.G, g = h / rep;
    pdl_wait();
    const int t0 = blockIdx.x * HC, row0 = a.cu_rows[b] + t0, n = min(HC, a.cu_rows[b + 1] - row0);
    if (n <= 0) return;
    const int taps = a.taps, keep = taps - 1, pos0 = a.tok_pos[a.cu_rows[b]];
    const float* ring = a.ring + (size_t)a.slots[b] * taps * a.C;
    const size_t chunk = first_chunk(a.cu_rows, b) + blockIdx.x;
    float* kT = sm;                              // [dk4][LT]
    float* qT = kT + (size_t)dk4 * LT;           // [max(dk4, dv)][LT]; the values' columns once the triangle is there
    float* M = qT + (size_t)max(dk4, dv) * LT;   // [HC][LT]

    // The raw input of channel c at the chunk's row i (in front of the step: a row of an earlier one, zero ahead of the sequence).
    auto input = [&](int i, int c) -> float {
        if (t0 + i >= 0) return a.rows[(ptrdiff_t)(row0 + i) * a.stride + c];
        const int p = pos0 + t0 + i;
        return p >= 0 ? ring[(size_t)(p % taps) * a.C + c] : 0.f;
    };
    // Convolution and silu of channel c for the tokens t .. t + 15 (zero behind the chunk's last one), to dst[0 .. 15].
    auto conv16 = [&](int c, int t, float* dst) {
        float y[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) y[i] = 0.f;
        if (taps <= 4) {
            float x[19], w[4];                   // rows t - 3 .. t + 15; fewer taps leave the first weights at zero
#pragma unroll
            for (int j = 0; j < 4; ++j) w[j] = j >= 4 - taps ? a.taps_w[(size_t)(j - (4 - taps)) * a.C + c] : 0.f;
            if (t0 + t >= 3 && t + 16 <= n) {
                const float* p = a.rows + (ptrdiff_t)(row0 + t - 3) * a.stride + c;
#pragma unroll
                for (int i = 0; i < 19; ++i) x[i] = p[(ptrdiff_t)i * a.stride];
            } else {
#pragma unroll
                for (int i = 0; i < 19; ++i) x[i] = i >= 4 - taps && t - 3 + i < n ? input(t - 3 + i, c) : 0.f;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < 16; ++i) y[i] = fmaf(w[j], x[i + j], y[i]);
        } else {
            for (int j = 0; j < taps; ++j) {
                const float w = a.taps_w[(size_t)j * a.C + c];
#pragma unroll
                for (int i = 0; i < 16; ++i)
                    if (t + i < n) y[i] = fmaf(w, input(t + i - keep + j, c), y[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < 16; i += 4) {
#pragma unroll
            for (int k = 0; k < 4; ++k) y[i + k] = t + i + k < n ? __fdividef(y[i + k], 1.f + __expf(-y[i + k])) : 0.f;
            *reinterpret_cast<float4*>(dst + i) = make_float4(y[i], y[i + 1], y[i + 2], y[i + 3]);
        }
    };

    for (int j = tid; j < 2 * dk4 * (HC / 16); j += NT) {
        const int c = j % (2 * dk4), t = j / (2 * dk4) * 16, r = c % dk4;
        float* dst = (c < dk4 ? qT : kT) + (size_t)r * LT + t;
        if (r < dk) {
            conv16((c < dk4 ? 0 : a.G * dk) + g * dk + r, t, dst);
        } else {
#pragma unroll
            for (int i = 0; i < 16; i += 4) *reinterpret_cast<float4*>(dst + i) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    if (tid < HC) {
        const bool in = tid < n;
        const float* x = a.rows + (size_t)(row0 + (in ? tid : 0)) * a.stride;
        sb[tid] = in ? sigmoid_f(x[a.b_off + h]) : 0.f;
        const float l = in ? -a.rate[h] * softplus_f(x[a.a_off + h] + a.dt_bias[h]) : 0.f;
        sl[tid] = (double)fmaxf(l, LOG_FLOOR);
    }
    __syncthreads();
    // Unit vectors' factors, and the running sum of the decays' logarithms.
    for (int j = tid; j < 2 * HC; j += NT) {
        const float* p = (j < HC ? qT : kT) + (j & (HC - 1));
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        for (int r = 0; r < dk4; r += 4)
#pragma unroll
            for (int i = 0; i < 4; ++i) { const float v = p[(r + i) * LT]; s[i] = fmaf(v, v, s[i]); }
        s_inv[j >> 6][j & (HC - 1)] = (j < HC ? a.q_scale : 1.f) / sqrtf((s[0] + s[1]) + (s[2] + s[3]) + a.unit_eps);
    }
    if (tid < 32) {
        double l0 = sl[2 * tid], l1 = l0 + sl[2 * tid + 1], run = l1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, run, o);
            if (tid >= o) run += up;
        }
        double before = __shfl_up_sync(0xffffffffu, run, 1);
        if (tid == 0) before = 0.0;
        const double last = __shfl_sync(0xffffffffu, run, 31);
        l0 += before;
        l1 += before;
        sl[2 * tid] = l0;
        sl[2 * tid + 1] = l1;
        float* sc = a.sc + (chunk * a.H + h) * SC;
        se[2 * tid] = expf((float)l0);
        se[2 * tid + 1] = expf((float)l1);
        sc[2 * tid] = se[2 * tid];
        sc[2 * tid + 1] = se[2 * tid + 1];
        sc[HC + 2 * tid] = expf((float)(last - l0));
        sc[HC + 2 * tid + 1] = expf((float)(last - l1));
        if (tid == 0) sc[2 * HC] = expm1f((float)last);
    }
    __syncthreads();
    {
        // Scale the vectors where they lie; the first value head of a group also leaves them, by tokens, for the kernels behind.
        const bool first = h % rep == 0;
        float* gq = a.Q + (chunk * a.G + g) * HC * a.ld;
        float* gk = a.K + (chunk * a.G + g) * HC * a.ld;
        for (int j = tid; j < 2 * dk4 * (HC / 4); j += NT) {
            const int c = j % (2 * dk4), t = j / (2 * dk4) * 4, r = c % dk4, key = c >= dk4;
            float4* p = reinterpret_cast<float4*>((key ? kT : qT) + (size_t)r * LT + t);
            const float4 f = *reinterpret_cast<const float4*>(&s_inv[key][t]);
            float4 v = *p;
            v.x *= f.x; v.y *= f.y; v.z *= f.z; v.w *= f.w;
            *p = v;
            if (first) {
                float* dst = (key ? gk : gq) + (size_t)t * a.ld + r;
                dst[0] = v.x; dst[a.ld] = v.y; dst[2 * a.ld] = v.z; dst[3 * a.ld] = v.w;
            }
        }
    }
    __syncthreads();
    // The triangles: tiles of TM rows and 4 columns that hold an entry on or below the diagonal.
    float* gN = a.N + (chunk * a.H + h) * HC * HC;
    {
        constexpr int PER = TM / 4;              // tile row i has PER (i + 1) tiles
        constexpr int TILES = PER * (HC / TM) * (HC / TM + 1) / 2;
        for (int j = tid; j < TILES; j += NT) {
            int ti = 0;
            while (PER * (ti + 1) * (ti + 2) / 2 <= j) ++ti;
            const int si = j - PER * ti * (ti + 1) / 2, t = ti * TM, s = si * 4;
            float kk[TM][4] = {}, qk[TM][4] = {};
#pragma unroll 2
            for (int r = 0; r < dk4; ++r) {
                const float* kr = kT + r * LT;
                const float4 x = *reinterpret_cast<const float4*>(kr + s);
#pragma unroll
                for (int i4 = 0; i4 < TM / 4; ++i4) {
                    const float4 y = *reinterpret_cast<const float4*>(kr + t + 4 * i4), z = *reinterpret_cast<const float4*>(qT + r * LT + t + 4 * i4);
                    const float yv[4] = {y.x, y.y, y.z, y.w}, zv[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        float (&m)[4] = kk[4 * i4 + i];
                        float (&q)[4] = qk[4 * i4 + i];
                        m[0] = fmaf(yv[i], x.x, m[0]); m[1] = fmaf(yv[i], x.y, m[1]); m[2] = fmaf(yv[i], x.z, m[2]); m[3] = fmaf(yv[i], x.w, m[3]);
                        q[0] = fmaf(zv[i], x.x, q[0]); q[1] = fmaf(zv[i], x.y, q[1]); q[2] = fmaf(zv[i], x.z, q[2]); q[3] = fmaf(zv[i], x.w, q[3]);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < TM; ++i) {
                const int tt = t + i;
                const double l = sl[tt];
                const float bt = sb[tt];
                float m[4], q[4];
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const float d = s + c <= tt ? expf((float)(l - sl[s + c])) : 0.f;
                    m[c] = s + c < tt ? bt * d * kk[i][c] : 0.f;
                    q[c] = d * qk[i][c];
                    if (s + c > tt) q[c] = 0.f;
                }
                *reinterpret_cast<float4*>(M + tt * LT + s) = make_float4(m[0], m[1], m[2], m[3]);
                *reinterpret_cast<float4*>(gN + tt * HC + s) = make_float4(q[0], q[1], q[2], q[3]);
            }
        }
        for (int j = tid; j < HC * (HC / 4); j += NT) {           // what lies wholly above the diagonal
            const int t = j / (HC / 4), s = j % (HC / 4) * 4;
            if (s > t / TM * TM + TM - 1) *reinterpret_cast<float4*>(gN + t * HC + s) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    __syncthreads();
    for (int j = tid; j < dv * (HC / 16); j += NT) {
        const int e = j % dv, t = j / dv * 16;
        conv16(2 * a.G * dk + h * dv + e, t, qT + (size_t)e * LT + t);
    }
    __syncthreads();
    // The triangle's solutions, where the columns lie: W's from b e^l k, V' from b v.  Two columns a thread (an entry of the
    // triangle read from shared memory serves both; four leave too few warps), sixteen rows at a time: what the rows above them
    // leave, then the rows themselves one after the other.  (What lies between dk4 and ld, and behind dv, is never read into anything that counts.)
    constexpr int CT = 2;
    const int cols = dk4 + dv, per = (cols + CT - 1) / CT;
    for (int c = tid; c < per; c += NT) {
        float* src[CT];
        float* dst[CT];
        int step[CT];
        bool key[CT];
#pragma unroll
        for (int j = 0; j < CT; ++j) {
            const int col = min(c + j * per, cols - 1);
            key[j] = col < dk4;
            const int e = key[j] ? col : col - dk4;
            src[j] = (key[j] ? kT : qT) + (size_t)e * LT;
            dst[j] = key[j] ? a.W + (chunk * a.H + h) * HC * a.ld + e : a.V + ((chunk * a.H + h) * a.tiles + e / a.n) * HC * a.n + e % a.n;
            step[j] = key[j] ? a.ld : a.n;
        }
#pragma unroll 1
        for (int r0 = 0; r0 < HC; r0 += 16) {
            float x[CT][16];
#pragma unroll
            for (int t = 0; t < 16; t += 4) {
                const float4 bt = *reinterpret_cast<const float4*>(sb + r0 + t), et = *reinterpret_cast<const float4*>(se + r0 + t);
#pragma unroll
                for (int j = 0; j < CT; ++j) {
                    const float4 v = *reinterpret_cast<const float4*>(src[j] + r0 + t);
                    x[j][t] = v.x * bt.x * (key[j] ? et.x : 1.f);
                    x[j][t + 1] = v.y * bt.y * (key[j] ? et.y : 1.f);
                    x[j][t + 2] = v.z * bt.z * (key[j] ? et.z : 1.f);
                    x[j][t + 3] = v.w * bt.w * (key[j] ? et.w : 1.f);
                }
            }
#pragma unroll 1
            for (int s0 = 0; s0 < r0; s0 += 4) {
                float4 y[CT];
#pragma unroll
                for (int j = 0; j < CT; ++j) y[j] = *reinterpret_cast<const float4*>(src[j] + s0);
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float4 m = *reinterpret_cast<const float4*>(M + (r0 + i) * LT + s0);
#pragma unroll
                    for (int j = 0; j < CT; ++j)
                        x[j][i] = fmaf(-m.w, y[j].w, fmaf(-m.z, y[j].z, fmaf(-m.y, y[j].y, fmaf(-m.x, y[j].x, x[j][i]))));
                }
            }
#pragma unroll
            for (int i = 1; i < 16; ++i)
#pragma unroll
                for (int q = 0; q < i; q += 4) {
                    const float4 m = *reinterpret_cast<const float4*>(M + (r0 + i) * LT + r0 + q);       // zero on and above the diagonal
                    const float mv[4] = {m.x, m.y, m.z, m.w};
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        if (q + k < i)
#pragma unroll
                            for (int j = 0; j < CT; ++j) x[j][i] = fmaf(-mv[k], x[j][q + k], x[j][i]);
                }
#pragma unroll
            for (int j = 0; j < CT; ++j) {
                if (c + j * per >= cols) break;
#pragma unroll
                for (int t = 0; t < 16; ++t) dst[j][(size_t)(r0 + t) * step[j]] = x[j][t];
#pragma unroll
                for (int t = 0; t < 16; t += 4) *reinterpret_cast<float4*>(src[j] + r0 + t) = make_float4(x[j][t], x[j][t + 1], x[j][t + 2], x[j][t + 3]);
            }
        }
    }
}

// ------------------------------------------------------------------ scan
// 4 WC J value columns of a head; 2 WC warps work, one more brings the chunks' vectors into shared memory by bulk copies.  RI:
// key channels in groups of 64.  A thread holds 4 RI rows and J columns of the state.  (What the lanes read from shared memory
// bounds the two products: wide tiles of few threads read less.)
template <int RI, int WC, int J>
__global__ void __launch_bounds__((2 * WC + 1) * 32, 1) scan_kernel(const __grid_constant__ HeadDeltaArgs a, int stages) {
    using namespace tc;
    constexpr int N = 4 * WC * J, WORKERS = 2 * WC * 32;
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(8) uint64_t full[4], empty[4];
    const int dk = a.dk, dv = a.dv, dk4 = pad4(dk), ld = a.ld, H = a.H, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int b = blockIdx.x, h = blockIdx.y, tile = blockIdx.z, col0 = tile * N, g = h / (H / a.G);
    const int stage_floats = 2 * HC * ld + HC * N + SC;
    float* sT = sm + (size_t)stages * stage_floats;       // [N][ld]: the state by columns
    float* us = sT + N * ld;                              // [HC][N]: u_s e^(l_64 - l_s)
    if (tid == 0) {
        for (int i = 0; i < stages; ++i) {
            mbar_init(smem_u32(&full[i]), 1);
            mbar_init(smem_u32(&empty[i]), 2 * WC);
        }
        mbar_fence_init();
    }
    __syncthreads();
    pdl_wait();
    const int row0 = a.cu_rows[b], row1 = a.cu_rows[b + 1], n_chunks = (row1 - row0 + HC - 1) / HC;
    const size_t chunk0 = first_chunk(a.cu_rows, b);
    if (warp == 2 * WC) {
        if (lane == 0) {
            int i = 0;
            for (; i < n_chunks; ++i) {
                const int s = i % stages;
                if (!mbar_wait(smem_u32(&empty[s]), ((i / stages) & 1) ^ 1)) { give_up(1); break; }
                const uint32_t bar = smem_u32(&full[s]), dst = smem_u32(sm + (size_t)s * stage_floats);
                const size_t ch = chunk0 + i;
                mbar_expect_tx(bar, stage_floats * 4);
                bulk_load(dst, a.W + (ch * H + h) * HC * ld, HC * ld * 4, bar);
                bulk_load(dst + HC * ld * 4, a.K + (ch * a.G + g) * HC * ld, HC * ld * 4, bar);
                bulk_load(dst + 2 * HC * ld * 4, a.V + ((ch * H + h) * a.tiles + tile) * HC * N, HC * N * 4, bar);
                bulk_load(dst + (2 * HC * ld + HC * N) * 4, a.sc + (ch * H + h) * SC, SC * 4, bar);
            }
            // After a wait that gave up, the copies that were started must land before the shared memory goes away.
            if (i < n_chunks)
                for (int back = 1; back <= stages && back <= i; ++back) mbar_wait(smem_u32(&full[(i - back) % stages]), ((i - back) / stages) & 1);
        }
        return;
    }
    {
        // The convolution's last inputs go to the ring; the blocks of a sequence share its channels.
        const int share = gridDim.y * gridDim.z, mine = blockIdx.y * gridDim.z + blockIdx.z, taps = a.taps;
        const int per = (a.C + share - 1) / share, lo = mine * per, hi = min(a.C, lo + per), n = row1 - row0;
        float* ring = a.ring + (size_t)a.slots[b] * taps * a.C;
        for (int i = max(0, n - taps); i < n; ++i) {
            const int p = a.tok_pos[row0 + i];
            for (int c = lo + tid; c < hi; c += WORKERS) ring[(size_t)(p % taps) * a.C + c] = a.rows[(size_t)(row0 + i) * a.stride + c];
        }
    }
    const int wr = warp & 1, wc = warp >> 1, l8 = lane & 7, l4 = lane >> 3;
    // This thread's part of the state: rows 4 (l8 + 8 wr + 16 i) .. + 3, columns c0 .. c0 + J - 1.
    const int c0 = J * (l4 + 4 * wc);
    float S[RI][4][J];
    float* st = a.state + ((size_t)a.slots[b] * H + h) * dk * dv;
    auto row_of = [&](int i) { return 4 * (l8 + 8 * wr + 16 * i); };
#pragma unroll
    for (int i = 0; i < RI; ++i)
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int c = 0; c < J; ++c) {
                const int row = row_of(i) + r, col = col0 + c0 + c;
                S[i][r][c] = row < dk && col < dv ? st[(size_t)row * dv + col] : 0.f;
            }
    auto share_state = [&]() {
#pragma unroll
        for (int i = 0; i < RI; ++i)
            if (row_of(i) < dk4)
#pragma unroll
                for (int c = 0; c < J; ++c)
                    *reinterpret_cast<float4*>(sT + (c0 + c) * ld + row_of(i)) = make_float4(S[i][0][c], S[i][1][c], S[i][2][c], S[i][3][c]);
    };
    share_state();
    asm volatile("bar.sync 1, %0;" ::"n"(WORKERS) : "memory");
    for (int ch = 0; ch < n_chunks; ++ch) {
        const int s = ch % stages;
        const float* w = sm + (size_t)s * stage_floats;
        const float *k = w + HC * ld, *v = k + HC * ld, *sc = v + HC * N;
        {
            // The state ahead of the chunk, for the output kernel.
            float* S0 = a.S0 + ((chunk0 + ch) * H + h) * (size_t)dk * a.tiles * N + col0 + c0;
#pragma unroll
            for (int i = 0; i < RI; ++i)
#pragma unroll
                for (int r = 0; r < 4; ++r)
                    if (row_of(i) + r < dk) {
                        float* at = S0 + (size_t)(row_of(i) + r) * a.tiles * N;
                        if constexpr (J == 4) *reinterpret_cast<float4*>(at) = make_float4(S[i][r][0], S[i][r][1], S[i][r][2], S[i][r][3]);
                        else *reinterpret_cast<float2*>(at) = make_float2(S[i][r][0], S[i][r][1]);
                    }
        }
        const unsigned bad = mbar_wait(smem_u32(&full[s]), (ch / stages) & 1) ? 0u : 1u;
        if (bad) give_up(2);
        // u = V' - W S_0: rows l8 + 8 wr + 16 i, columns l4 + 4 wc + 4 WC j.
        f2 acc[4][J];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < J; ++j) acc[i][j] = 0ull;
        const float* wp = w + (size_t)(l8 + 8 * wr) * ld;
        const float* sp = sT + (size_t)(l4 + 4 * wc) * ld;
#pragma unroll 4
        for (int r = 0; r < dk4; r += 4) {
            ulonglong2 x[4], y[J];
#pragma unroll
            for (int i = 0; i < 4; ++i) x[i] = *reinterpret_cast<const ulonglong2*>(wp + 16 * i * ld + r);
#pragma unroll
            for (int j = 0; j < J; ++j) y[j] = *reinterpret_cast<const ulonglong2*>(sp + 4 * WC * j * ld + r);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    acc[i][j] = fma2(x[i].x, y[j].x, acc[i][j]);
                    acc[i][j] = fma2(x[i].y, y[j].y, acc[i][j]);
                }
        }
        float* gu = a.V + (((chunk0 + ch) * H + h) * a.tiles + tile) * HC * N;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const int t = l8 + 8 * wr + 16 * i, c = l4 + 4 * wc + 4 * WC * j;
                const float2 f = unpack2(acc[i][j]);
                const float u = v[t * N + c] - (f.x + f.y);
                gu[t * N + c] = u;
                us[t * N + c] = u * sc[HC + t];
            }
        unsigned any;
        asm volatile("{ .reg .pred p, q; setp.ne.u32 q, %1, 0; barrier.cta.red.or.pred p, 1, %2, q; selp.u32 %0, 1, 0, p; }"
                     : "=r"(any) : "r"(bad), "n"(WORKERS) : "memory");
        if (any) break;                          // every worker leaves together
        // S_64 = S_0 + (e^l - 1) S_0 + sum_s k_s (u_s e^(l_64 - l_s))^T
        const float E = sc[2 * HC];
        f2 A[RI][2][J];                          // rows in pairs
#pragma unroll
        for (int i = 0; i < RI; ++i)
#pragma unroll
            for (int p = 0; p < 2; ++p)
#pragma unroll
                for (int c = 0; c < J; ++c)
                    A[i][p][c] = pack2(fmaf(S[i][2 * p][c], E, S[i][2 * p][c]), fmaf(S[i][2 * p + 1][c], E, S[i][2 * p + 1][c]));
        const float* kp[RI];                     // rows behind the last key channel repeat the last ones and are not used
#pragma unroll
        for (int i = 0; i < RI; ++i) kp[i] = k + min(row_of(i), dk4 - 4);
#pragma unroll 8
        for (int t = 0; t < HC; ++t) {
            f2 u[J];
            if constexpr (J == 4) {
                const float4 f = *reinterpret_cast<const float4*>(us + t * N + c0);
                u[0] = pack2(f.x, f.x); u[1] = pack2(f.y, f.y); u[2] = pack2(f.z, f.z); u[3] = pack2(f.w, f.w);
            } else {
                const float2 f = *reinterpret_cast<const float2*>(us + t * N + c0);
                u[0] = pack2(f.x, f.x); u[1] = pack2(f.y, f.y);
            }
#pragma unroll
            for (int i = 0; i < RI; ++i) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(kp[i] + t * ld);
#pragma unroll
                for (int c = 0; c < J; ++c) {
                    A[i][0][c] = fma2(x.x, u[c], A[i][0][c]);
                    A[i][1][c] = fma2(x.y, u[c], A[i][1][c]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < RI; ++i)
#pragma unroll
            for (int p = 0; p < 2; ++p)
#pragma unroll
                for (int c = 0; c < J; ++c) {
                    const float2 f = unpack2(A[i][p][c]);
                    S[i][2 * p][c] = f.x;
                    S[i][2 * p + 1][c] = f.y;
                }
        share_state();
        asm volatile("bar.sync 1, %0;" ::"n"(WORKERS) : "memory");
        if (lane == 0) mbar_arrive(smem_u32(&empty[s]));
    }
#pragma unroll
    for (int i = 0; i < RI; ++i)
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int c = 0; c < J; ++c) {
                const int row = row_of(i) + r, col = col0 + c0 + c;
                if (row < dk && col < dv) st[(size_t)row * dv + col] = S[i][r][c];
            }
}

// ------------------------------------------------------------------ output
// o = [e^l q | N] [S_0; u] as one product of 64 rows, its right side in tiles of 32 rows; a thread makes rows tg + 16 i and
// columns 4 cg + 64 j .. + 3.  CJ: value columns in groups of 64.
__device__ __forceinline__ void copy16(uint32_t dst, const float* src, bool valid) {
    const int bytes = valid ? 16 : 0;            // 0 source bytes: the 16 destination bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__host__ __device__ __forceinline__ int output_lda(int dk) { return (dk + 31) / 32 * 32 + HC + 4; }

template <typename TO, int CJ>
__global__ void __launch_bounds__(256, CJ <= 2 ? 2 : 1) output_kernel(const __grid_constant__ HeadDeltaArgs a) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    constexpr int BW = 64 * CJ;                  // columns of a tile
    const int dk = a.dk, dv = a.dv, H = a.H, tid = threadIdx.x, h = blockIdx.z, b = blockIdx.y, g = h / (H / a.G);
    pdl_wait();
    const int t0 = blockIdx.x * HC, row0 = a.cu_rows[b] + t0, n = min(HC, a.cu_rows[b + 1] - row0);
    if (n <= 0) return;
    const size_t chunk = first_chunk(a.cu_rows, b) + blockIdx.x;
    const int dkp = (dk + 31) / 32 * 32, lda = output_lda(dk), dvp = a.tiles * a.n;
    float* A = sm;                               // [HC][lda]
    float* B = A + HC * lda;                     // [2][32][BW]
    const float* S0 = a.S0 + (chunk * H + h) * (size_t)dk * dvp;
    const float* U = a.V + (chunk * H + h) * a.tiles * (size_t)HC * a.n;
    const int n_tiles = dkp / 32 + HC / 32;
    auto load = [&](int tile, int stage) {
        float* dst = B + stage * 32 * BW;
        for (int j = tid; j < 32 * (BW / 4); j += 256) {
            const int r = j / (BW / 4), c = j % (BW / 4) * 4, row = tile * 32 + r;
            const float* src;
            bool ok = c < dvp;
            if (row < dkp) {
                ok = ok && row < dk;
                src = S0 + (size_t)row * dvp + c;
            } else {
                src = U + ((size_t)(c / a.n) * HC + row - dkp) * a.n + c % a.n;
            }
            copy16((uint32_t)__cvta_generic_to_shared(dst + r * BW + c), ok ? src : a.sc, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, 0);
    const float* sc = a.sc + (chunk * H + h) * SC;
    const float* gq = a.Q + (chunk * a.G + g) * HC * a.ld;
    for (int j = tid; j < HC * (dkp / 4); j += 256) {
        const int t = j / (dkp / 4), r = j % (dkp / 4) * 4;
        float4 v = r < a.ld ? *reinterpret_cast<const float4*>(gq + (size_t)t * a.ld + r) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float e = sc[t];
        v.x = r < dk ? v.x * e : 0.f; v.y = r + 1 < dk ? v.y * e : 0.f; v.z = r + 2 < dk ? v.z * e : 0.f; v.w = r + 3 < dk ? v.w * e : 0.f;
        *reinterpret_cast<float4*>(A + t * lda + r) = v;
    }
    const float* gN = a.N + (chunk * H + h) * HC * HC;
    for (int j = tid; j < HC * (HC / 4); j += 256) {
        const int t = j / (HC / 4), s = j % (HC / 4) * 4;
        *reinterpret_cast<float4*>(A + t * lda + dkp + s) = *reinterpret_cast<const float4*>(gN + t * HC + s);
    }
    const int tg = tid >> 4, cg = tid & 15;
    float acc[4][CJ][4] = {};
    for (int tile = 0; tile < n_tiles; ++tile) {
        if (tile + 1 < n_tiles) {
            load(tile + 1, (tile + 1) & 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* Bt = B + (tile & 1) * 32 * BW + 4 * cg;
        const float* At = A + tg * lda + tile * 32;
#pragma unroll
        for (int r = 0; r < 32; r += 4) {
            float4 x[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) x[i] = *reinterpret_cast<const float4*>(At + 16 * i * lda + r);
#pragma unroll
            for (int q = 0; q < 4; ++q)
#pragma unroll
                for (int j = 0; j < CJ; ++j) {
                    const float4 y = *reinterpret_cast<const float4*>(Bt + (r + q) * BW + 64 * j);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float f = q == 0 ? x[i].x : q == 1 ? x[i].y : q == 2 ? x[i].z : x[i].w;
                        acc[i][j][0] = fmaf(f, y.x, acc[i][j][0]);
                        acc[i][j][1] = fmaf(f, y.y, acc[i][j][1]);
                        acc[i][j][2] = fmaf(f, y.z, acc[i][j][2]);
                        acc[i][j][3] = fmaf(f, y.w, acc[i][j][3]);
                    }
                }
        }
        __syncthreads();
    }
    // Each head over its root mean square, times the shared weight and the gate; the sixteen lanes of a row add its squares.
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = tg + 16 * i;
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < CJ; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c)
                if (4 * cg + 64 * j + c < dv) ss = fmaf(acc[i][j][c], acc[i][j][c], ss);
#pragma unroll
        for (int o = 8; o >= 1; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / (float)dv + a.norm_eps);
        if (t >= n) continue;
        const float* gate = a.rows + (size_t)(row0 + t) * a.stride + a.g_off + h * dv;
        TO* out = (TO*)a.out + ((size_t)(row0 + t) * H + h) * dv;
#pragma unroll
        for (int j = 0; j < CJ; ++j) {
            const int c = 4 * cg + 64 * j;
            if (c >= dv) continue;
            float y[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) y[q] = c + q < dv ? acc[i][j][q] * inv * a.norm_w[c + q] * silu_f(gate[c + q]) : 0.f;
            if (dv % 4 == 0) {
                if constexpr (sizeof(TO) == 4) {
                    *reinterpret_cast<float4*>(out + c) = make_float4(y[0], y[1], y[2], y[3]);
                } else {
                    __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[1]), hi = __floats2bfloat162_rn(y[2], y[3]);
                    *reinterpret_cast<uint2*>(out + c) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
                }
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (c + q < dv) out[c + q] = from_f32<TO>(y[q]);
            }
        }
    }
}

// ------------------------------------------------------------------ launches
constexpr size_t MOST_SMEM = 224 * 1024;

template <typename F> bool allow_smem(F kernel, size_t smem) {
    return smem <= 48 * 1024 || cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) == cudaSuccess;
}

// Value columns of a scan block: 32, or 16 where 32 would leave multiprocessors without a block.
int scan_columns(int B, int H, int dv) { return (long)B * H * ((dv + 31) / 32) >= 100 ? 32 : 16; }

template <int NT, int TM> int go_prepare(const HeadDeltaArgs& a, dim3 grid, cudaStream_t stream) {
    const size_t smem = (size_t)(pad4(a.dk) + (pad4(a.dk) > a.dv ? pad4(a.dk) : a.dv) + HC) * LT * sizeof(float);
    if (smem > MOST_SMEM) return LQ_BAD_SIZE;
    if (!allow_smem(prepare_kernel<NT, TM>, smem)) return lq_launch_status();
    return launch_pdl(prepare_kernel<NT, TM>, grid, dim3(NT), smem, stream, a);
}

template <int RI, int WC, int J> int go_scan(const HeadDeltaArgs& a, int B, cudaStream_t stream) {
    constexpr int N = 4 * WC * J;
    const size_t stage = (size_t)(2 * HC * a.ld + HC * N + SC) * sizeof(float), rest = (size_t)(N * a.ld + HC * N) * sizeof(float);
    int stages = 3;
    while (stages > 1 && stages * stage + rest > MOST_SMEM) --stages;
    const size_t smem = stages * stage + rest;
    if (smem > MOST_SMEM) return LQ_BAD_SIZE;
    if (!allow_smem(scan_kernel<RI, WC, J>, smem)) return lq_launch_status();
    return launch_after(scan_kernel<RI, WC, J>, dim3(B, a.H, a.tiles), dim3((2 * WC + 1) * 32), smem, stream, a, stages);
}

template <typename TO, int CJ> int go_output(const HeadDeltaArgs& a, dim3 grid, cudaStream_t stream) {
    const size_t smem = (size_t)(HC * output_lda(a.dk) + 2 * 32 * 64 * CJ) * sizeof(float);
    if (smem > MOST_SMEM) return LQ_BAD_SIZE;
    if (!allow_smem(output_kernel<TO, CJ>, smem)) return lq_launch_status();
    return launch_pdl(output_kernel<TO, CJ>, grid, dim3(256), smem, stream, a);
}

struct Scratch { long long K, Q, W, V, N, S0, sc, total; };
Scratch scratch_of(int T, int B, int H, int G, int dk, int dv) {
    const long long chunks = T / HC + B, ld = row_length(dk), n = scan_columns(B, H, dv), dvp = (dv + n - 1) / n * n;
    Scratch s;
    s.K = 0;
    s.Q = s.K + chunks * G * HC * ld;
    s.W = s.Q + chunks * G * HC * ld;
    s.V = s.W + chunks * H * HC * ld;
    s.N = s.V + chunks * H * HC * dvp;
    s.S0 = s.N + chunks * H * HC * HC;
    s.sc = s.S0 + chunks * H * dk * dvp;
    s.total = s.sc + chunks * H * SC;
    return s;
}

}  // namespace

// Floats of scratch that a step with prompts needs.
LQ_EXPORT long long lq_head_delta_scratch_floats(int T, int B, int H, int G, int dk, int dv) { return scratch_of(T, B, H, G, dk, dv).total; }

// rows [T, stride] float32 -> out [T, H dv] (out_dtype); state and ring are moved on.  dk and dv at most 256.
LQ_EXPORT int lq_head_delta_prompt(const float* rows, int stride, int b_off, int a_off, int g_off, const float* taps_w, int taps, float* ring,
                                   const float* dt_bias, const float* rate, float* state, const int* cu_rows, const int* slots,
                                   const int* tok_pos, float* scratch, const float* norm_w, float norm_eps, void* out, int out_dtype, int T,
                                   int B, int max_new, int H, int G, int dk, int dv, float q_scale, float unit_eps, cudaStream_t stream) {
    if (B <= 0 || max_new <= 0) return LQ_OK;
    if (dk < 1 || dk > 256 || dv < 1 || dv > 256 || G < 1 || H % G || taps < 1) return LQ_BAD_SIZE;
    if (out_dtype != LQ_F32 && out_dtype != LQ_BF16) return LQ_BAD_DTYPE;
    const Scratch s = scratch_of(T, B, H, G, dk, dv);
    const int n = scan_columns(B, H, dv);
    HeadDeltaArgs a{rows, stride, b_off, a_off, g_off, taps_w, taps, 2 * G * dk + H * dv, ring, dt_bias, rate, state, cu_rows, slots, tok_pos,
                    scratch + s.K, scratch + s.Q, scratch + s.W, scratch + s.V, scratch + s.N, scratch + s.S0, scratch + s.sc,
                    norm_w, norm_eps, out, out_dtype == LQ_BF16, H, G, dk, dv, row_length(dk), n, (dv + n - 1) / n, q_scale, unit_eps};
    const dim3 grid((max_new + HC - 1) / HC, B, H);
    int rc = dk + dv <= 160 ? go_prepare<128, 8>(a, grid, stream) : go_prepare<256, 4>(a, grid, stream);
    if (rc != LQ_OK) return rc;
    const int ri = (pad4(dk) + 63) / 64, cj = (a.tiles * n + 63) / 64;
#define LQ_GO(RI) case RI: rc = n == 32 ? go_scan<RI, RI <= 2 ? 2 : 4, RI <= 2 ? 4 : 2>(a, B, stream) : go_scan<RI, 2, 2>(a, B, stream); break;
    switch (ri) { LQ_GO(1) LQ_GO(2) LQ_GO(3) LQ_GO(4) default: rc = LQ_BAD_SIZE; }
#undef LQ_GO
    if (rc != LQ_OK) return rc;
#define LQ_GO(CJ) case CJ: return out_dtype == LQ_F32 ? go_output<float, CJ>(a, grid, stream) : go_output<__nv_bfloat16, CJ>(a, grid, stream);
    switch (cj) { LQ_GO(1) LQ_GO(2) LQ_GO(3) LQ_GO(4) }
#undef LQ_GO
    return LQ_BAD_SIZE;
}

LQ_EXPORT int lq_head_delta_status() { return tc::status_read(); }
LQ_EXPORT int* lq_head_delta_status_word() { return tc::status_word(); }
