// Gated delta rule with a decay per key channel.  Per head, with S [dk, dv] in float32:
//
//   S' = diag(a_t) S_(t-1)      u_t = b_t (v_t - S'^T k_t)      S_t = S' + k_t u_t^T      o_t = S_t^T q_t
//
// q, k (G key heads) and v (H value heads; value head h reads key head h / (H / G)) come from projections whose
// channels each pass a causal convolution over time and silu; q and k are then made unit vectors per head,
// x / sqrt(sum(x^2) + unit_eps), q also times q_scale; b = sigmoid(x_b); a = exp(-rate_h softplus(z + bias)).
// Everything here is float32 whatever the activations' storage is.
//
// Prompts and portions (two kernels).  delta_prepare_kernel turns the projections' rows into records of DC tokens:
// with A_t the product of the record's decays up to token t,
//   S_0^T (A_t k_t) and S_0^T (A_t q_t) are what tokens t would read from the state ahead of the record,
//   M_ts = sum_r k_t[r] k_s[r] a_(s+1)[r] ... a_t[r]   and   N_ts (q_t in place of k_t)   what a token of the record adds to that,
//   u_t = b_t (v_t - S_0^T (A_t k_t) - sum_(s<t) M_ts u_s)          o_t = S_0^T (A_t q_t) + sum_(s<=t) N_ts u_s
//   S_DC = diag(A_DC) S_0 + sum_s (a_(s+1) ... a_DC k_s) u_s^T
// Products of decays only, never a quotient, so a decay of zero is harmless.  delta_scan_kernel walks a sequence's
// records with the state in registers: one round of sums over the key rows per record instead of one per token.
//
// Single tokens (one kernel, delta_single_kernel): convolution, unit vectors, the decays' and the output gate's second
// products (over their small inner sizes), the recurrence, the head's norm and the gate; the state is read and written once.
//
// The convolution's last inputs are kept per slot as a ring of `taps` rows, the row of position p at p % taps: a step
// of one token writes a row that it does not read.
#include "common.cuh"

constexpr int DC = 4;                 // tokens of a record
constexpr int LPC = 8;                // lanes that share a value column: lane l holds key rows 4 l .. 4 l + 3 of every 32
constexpr int DSCAL = 4 + 16 + 16;    // scalars of a record: b [4], M [4][4] (t, s), N [4][4]

typedef unsigned long long f2;        // two float32 side by side
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
    f2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
    f2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f2 pack2(float lo, float hi) {
    f2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 unpack2(f2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

struct DeltaArgs {
    const float* rows;           // [T, stride]: q at column 0, then k (G * dk each), v (H * dv), b (H), ...
    int stride, b_off;
    const float* taps_w;         // [taps, C] the convolution's weights by taps, C = 2 G dk + H dv
    int taps, C;
    float* ring;                 // [slots][taps][C]
    const float* z;              // prompts: [T, H * dk] the decays' pre-activations
    const float* z_bias;         // [H * dk]
    const float* rate;           // [H]
    float* state;                // [slots][H][dk][dv]
    const int* cu_rows;          // [B + 1]
    const int* slots;            // [B]
    const int* tok_pos;          // [T]
    float* records;              // prompts: see delta_record_floats
    float* raw;                  // prompts: [T, H, dv] the heads' outputs, neither normed nor gated
    int H, G, dk, dv;
    float q_scale, unit_eps;
};

// A record's rows of key channels are padded with zeros to whole 32s.
__host__ __device__ __forceinline__ int pad_rows(int dk) { return (dk + 31) / 32 * 32; }
__host__ __device__ __forceinline__ int pad4(int n) { return (n + 3) / 4 * 4; }
// Per (record, head): A_t k_t [DC][DKP], A_t q_t [DC][DKP], decayed k_s [DC][DKP], A_DC [DKP], v [DC][pad4(dv)], scalars.
__host__ __device__ __forceinline__ int record_floats(int dk, int dv) { return (3 * DC + 1) * pad_rows(dk) + DC * pad4(dv) + DSCAL; }
// Where the records of sequence b start: unique and never overlapping, whatever the sequences' lengths are.
__device__ __forceinline__ int first_record(const int* cu_rows, int b) { return cu_rows[b] / DC + b; }

// One block per (record, sequence, value head).
constexpr int DP_THREADS = 128;
__global__ void __launch_bounds__(DP_THREADS) delta_prepare_kernel(DeltaArgs a) {
    pdl_launch_dependents();
    extern __shared__ float sm[];
    const int dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float* sq = sm;                              // [DC][dk]
    float* sk = sq + DC * dk;                    // [DC][dk]
    __shared__ float inv_q[DC], inv_k[DC], red[DP_THREADS / 32][32];
    pdl_wait();
    const int b = blockIdx.y, h = blockIdx.z, g = h / (a.H / a.G);
    const int row0 = a.cu_rows[b], n_rows = a.cu_rows[b + 1] - row0, t0 = blockIdx.x * DC;
    if (t0 >= n_rows) return;
    const int n = min(DC, n_rows - t0), taps = a.taps, keep = taps - 1;
    const int pos0 = a.tok_pos[row0];            // the step's first position of this sequence
    const float* ring = a.ring + (size_t)a.slots[b] * taps * a.C;
    const int dkp = pad_rows(dk), dvp = pad4(dv);
    float* rec = a.records + ((size_t)(first_record(a.cu_rows, b) + blockIdx.x) * a.H + h) * record_floats(dk, dv);
    float* rec_v = rec + (3 * DC + 1) * dkp;
    float* rec_s = rec_v + DC * dvp;
    // The raw input of channel c at the step's row i (below 0: a row of an earlier step, zero ahead of the sequence).
    auto input = [&](int i, int c) -> float {
        if (i >= 0) return a.rows[(size_t)(row0 + i) * a.stride + c];
        const int p = pos0 + i;
        return p >= 0 ? ring[(size_t)(p % taps) * a.C + c] : 0.f;
    };
    // Convolution and silu: q and k of the head to shared memory, v straight into the record.
    for (int e = tid; e < 2 * dk + dvp; e += DP_THREADS) {
        const int c = e < dk ? g * dk + e : (e < 2 * dk ? a.G * dk + g * dk + (e - dk) : 2 * a.G * dk + h * dv + (e - 2 * dk));
        float acc[DC] = {};
        if (e < 2 * dk + dv) {
            if (taps <= 5) {
                float w[5], x[DC + 4];
#pragma unroll
                for (int j = 0; j < 5; ++j) w[j] = j < taps ? a.taps_w[(size_t)j * a.C + c] : 0.f;
#pragma unroll
                for (int i = 0; i < DC + 4; ++i) x[i] = (i < n + keep) ? input(t0 + i - keep, c) : 0.f;
#pragma unroll
                for (int t = 0; t < DC; ++t)
#pragma unroll
                    for (int j = 0; j < 5; ++j)
                        if (j < taps) acc[t] = fmaf(w[j], x[t + j], acc[t]);
            } else {
                for (int t = 0; t < n; ++t)
                    for (int j = 0; j < taps; ++j) acc[t] = fmaf(a.taps_w[(size_t)j * a.C + c], input(t0 + t - keep + j, c), acc[t]);
            }
        }
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            const float y = (t < n && e < 2 * dk + dv) ? silu_f(acc[t]) : 0.f;
            if (e < dk) sq[t * dk + e] = y;
            else if (e < 2 * dk) sk[t * dk + e - dk] = y;
            else rec_v[t * dvp + e - 2 * dk] = y;
        }
    }
    __syncthreads();
    // Unit vectors: a warp per token.
    for (int t = warp; t < DC; t += DP_THREADS / 32) {
        float s0 = 0.f, s1 = 0.f;
        for (int r = lane; r < dk; r += 32) {
            s0 = fmaf(sq[t * dk + r], sq[t * dk + r], s0);
            s1 = fmaf(sk[t * dk + r], sk[t * dk + r], s1);
        }
        s0 = warp_sum(s0);
        s1 = warp_sum(s1);
        if (lane == 0) {
            inv_q[t] = a.q_scale / sqrtf(s0 + a.unit_eps);
            inv_k[t] = 1.f / sqrtf(s1 + a.unit_eps);
        }
    }
    __syncthreads();
    // Decays, the decayed vectors, and every thread's share of the sixteen sums over the key channels:
    // M_10, M_20, M_21, M_30, M_31, M_32, then N_00, N_10, N_11, N_20, ... N_33.
    float part[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) part[i] = 0.f;
    const float rate = a.rate[h];
    for (int r = tid; r < dkp; r += DP_THREADS) {
        float d[DC], k[DC], q[DC];
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            const bool in = r < dk && t < n;
            d[t] = 1.f;
            k[t] = q[t] = 0.f;
            if (in) {
                const float z = a.z[(size_t)(row0 + t0 + t) * a.H * dk + h * dk + r] + a.z_bias[h * dk + r];
                d[t] = expf(-rate * softplus_f(z));
                k[t] = sk[t * dk + r] * inv_k[t];
                q[t] = sq[t * dk + r] * inv_q[t];
            }
        }
        float A = 1.f;
        float kd[DC];                            // k_s times the decays after s, up to the token being walked
        int m = 0, nn = 6;
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            A *= d[t];
#pragma unroll
            for (int s = 0; s < t; ++s) {
                kd[s] *= d[t];
                part[m] = fmaf(kd[s], k[t], part[m]);
                ++m;
            }
            kd[t] = k[t];
#pragma unroll
            for (int s = 0; s <= t; ++s) {
                part[nn] = fmaf(kd[s], q[t], part[nn]);
                ++nn;
            }
            rec[t * dkp + r] = A * k[t];
            rec[(DC + t) * dkp + r] = A * q[t];
        }
#pragma unroll
        for (int s = 0; s < DC; ++s) rec[(2 * DC + s) * dkp + r] = kd[s];
        rec[3 * DC * dkp + r] = r < dk ? A : 0.f;
    }
    // Sixteen sums over a warp at once (a lane hands half of its values across and keeps the other half), then the warps.
#pragma unroll
    for (int w = 8; w >= 1; w >>= 1) {
        const bool upper = lane & w;
#pragma unroll
        for (int t = 0; t < w; ++t) {
            const float give = upper ? part[t] : part[t + w];
            const float mine = upper ? part[t + w] : part[t];
            part[t] = mine + __shfl_xor_sync(0xffffffffu, give, w);
        }
    }
    red[warp][lane] = part[0] + __shfl_xor_sync(0xffffffffu, part[0], 16);
    __syncthreads();
    if (tid < DSCAL) {
        float v = 0.f;
        if (tid < 4) {
            v = tid < n ? sigmoid_f(a.rows[(size_t)(row0 + t0 + tid) * a.stride + a.b_off + h]) : 0.f;
        } else {
            const bool is_n = tid >= 20;
            const int t = (tid - (is_n ? 20 : 4)) >> 2, s = tid & 3;
            const int at = is_n ? (s <= t ? 6 + t * (t + 1) / 2 + s : -1) : (s < t ? t * (t - 1) / 2 + s : -1);
            if (at >= 0)
#pragma unroll
                for (int w = 0; w < DP_THREADS / 32; ++w) v += red[w][at];
        }
        rec_s[tid] = v;
    }
}

// One block per (sequence, value head, some value columns): a warp takes 4 * NC neighbouring columns, eight lanes each
// with KR of the key rows and NC columns.  A record is brought into shared memory while the ones before it are worked on.
constexpr int DS_STAGES = 4;
template <int KR, int NC>
__global__ void __launch_bounds__(256, 1) delta_scan_kernel(DeltaArgs a, int cols) {
    pdl_launch_dependents();
    constexpr int DKP = KR * LPC, PIECES = KR / 4;
    extern __shared__ __align__(16) float sm[];
    const int dv = a.dv, dvp = pad4(dv), H = a.H, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & 7;
    const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols;
    const int vec_floats = (3 * DC + 1) * DKP, stage_floats = vec_floats + DC * cols + DSCAL;
    const int rf = record_floats(a.dk, dv);
    const int c0 = warp * 4 * NC + (lane >> 3) * NC;         // this thread's first column inside the block's
    pdl_wait();
    const int row0 = a.cu_rows[b], row1 = a.cu_rows[b + 1], n_rec = (row1 - row0 + DC - 1) / DC;
    const float* rec0 = a.records + ((size_t)first_record(a.cu_rows, b) * H + h) * rf;
    const int vcols = min(cols, dvp - col0);                 // columns (whole fours) that the record has
    auto fetch = [&](int i) {
        if (i < n_rec) {
            const float* src = rec0 + (size_t)i * H * rf;
            const uint32_t dst = (uint32_t)__cvta_generic_to_shared(sm + (i % DS_STAGES) * stage_floats);
            for (int e = tid; e < vec_floats / 4; e += blockDim.x) cp_async16(dst + e * 16, src + e * 4);
            const int v4 = vcols / 4;
            for (int e = tid; e < DC * v4; e += blockDim.x)
                cp_async16(dst + (vec_floats + (e / v4) * cols + (e % v4) * 4) * 4, src + vec_floats + (e / v4) * dvp + col0 + (e % v4) * 4);
            for (int e = tid; e < DSCAL / 4; e += blockDim.x)
                cp_async16(dst + (vec_floats + DC * cols + e * 4) * 4, src + vec_floats + DC * dvp + e * 4);
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < DS_STAGES - 1; ++i) fetch(i);
    // The convolution's last inputs go to the ring; the blocks of a sequence share its channels.  (The records ahead
    // of this kernel were made from the ring as it was.)
    {
        const int share = gridDim.y * gridDim.z, mine = blockIdx.y * gridDim.z + blockIdx.z, taps = a.taps;
        const int per = (a.C + share - 1) / share, lo = mine * per, hi = min(a.C, lo + per), n = row1 - row0;
        float* ring = a.ring + (size_t)a.slots[b] * taps * a.C;
        for (int i = max(0, n - taps); i < n; ++i) {
            const int p = a.tok_pos[row0 + i];
            for (int c = lo + tid; c < hi; c += blockDim.x)
                ring[(size_t)(p % taps) * a.C + c] = a.rows[(size_t)(row0 + i) * a.stride + c];
        }
    }
    float* st = a.state + ((size_t)a.slots[b] * H + h) * a.dk * dv;
    f2 S[KR / 2][NC];                            // rows 32 i + 4 l + {0, 1}, {2, 3} as pairs 2 i, 2 i + 1
#pragma unroll
    for (int i = 0; i < PIECES; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int r = i * 32 + l * 4 + 2 * p, col = col0 + c0 + c;
                const bool in = c0 + c < cols && col < dv;
                S[2 * i + p][c] = pack2(in && r < a.dk ? st[(size_t)r * dv + col] : 0.f, in && r + 1 < a.dk ? st[(size_t)(r + 1) * dv + col] : 0.f);
            }
    for (int i = 0; i < n_rec; ++i) {
        cp_async_wait<DS_STAGES - 2>();
        __syncthreads();                         // record i is there, and everyone is done with the one before it
        fetch(i + DS_STAGES - 1);
        const float* rec = sm + (i % DS_STAGES) * stage_floats;
        const float* vs = rec + vec_floats + c0;
        const float4* sc = reinterpret_cast<const float4*>(rec + vec_floats + DC * cols);
        f2 acc2[2 * DC][NC];
#pragma unroll
        for (int t = 0; t < 2 * DC; ++t)
#pragma unroll
            for (int c = 0; c < NC; ++c) acc2[t][c] = 0ull;
#pragma unroll
        for (int j = 0; j < PIECES; ++j)
#pragma unroll
            for (int t = 0; t < 2 * DC; ++t) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(rec + t * DKP + j * 32 + l * 4);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    acc2[t][c] = fma2(S[2 * j][c], x.x, acc2[t][c]);
                    acc2[t][c] = fma2(S[2 * j + 1][c], x.y, acc2[t][c]);
                }
            }
        float mine[NC], u[DC][NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            float acc[2 * DC];
#pragma unroll
            for (int t = 0; t < 2 * DC; ++t) {
                const float2 f = unpack2(acc2[t][c]);
                acc[t] = f.x + f.y;
            }
            // Eight sums over the column's eight lanes: lane l is left with sum number l.
#pragma unroll
            for (int w = 4; w >= 1; w >>= 1) {
                const bool upper = l & w;
#pragma unroll
                for (int t = 0; t < w; ++t) {
                    const float give = upper ? acc[t] : acc[t + w];
                    const float keep = upper ? acc[t + w] : acc[t];
                    acc[t] = keep + __shfl_xor_sync(0xffffffffu, give, w);
                }
            }
            mine[c] = acc[0];
        }
        const float4 beta = sc[0], m1 = sc[2], m2 = sc[3], m3 = sc[4];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            float r[DC];
#pragma unroll
            for (int t = 0; t < DC; ++t) r[t] = vs[t * cols + c] - __shfl_sync(0xffffffffu, mine[c], (lane & 24) + t);
            u[0][c] = beta.x * r[0];
            u[1][c] = beta.y * (r[1] - m1.x * u[0][c]);
            u[2][c] = beta.z * (r[2] - m2.x * u[0][c] - m2.y * u[1][c]);
            u[3][c] = beta.w * (r[3] - m3.x * u[0][c] - m3.y * u[1][c] - m3.z * u[2][c]);
        }
        if (l >= DC) {
            const int t = l - DC, row = row0 + i * DC + t;
            const float4 nt = sc[5 + t];
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (row < row1 && c0 + c < cols && col0 + c0 + c < dv)
                    a.raw[((size_t)row * H + h) * dv + col0 + c0 + c] = mine[c] + nt.x * u[0][c] + nt.y * u[1][c] + nt.z * u[2][c] + nt.w * u[3][c];
        }
#pragma unroll
        for (int j = 0; j < PIECES; ++j) {
            const ulonglong2 A = *reinterpret_cast<const ulonglong2*>(rec + 3 * DC * DKP + j * 32 + l * 4);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                S[2 * j][c] = mul2(S[2 * j][c], A.x);
                S[2 * j + 1][c] = mul2(S[2 * j + 1][c], A.y);
            }
        }
#pragma unroll
        for (int s = 0; s < DC; ++s) {
            f2 uu[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) uu[c] = pack2(u[s][c], u[s][c]);
#pragma unroll
            for (int j = 0; j < PIECES; ++j) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(rec + (2 * DC + s) * DKP + j * 32 + l * 4);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    S[2 * j][c] = fma2(x.x, uu[c], S[2 * j][c]);
                    S[2 * j + 1][c] = fma2(x.y, uu[c], S[2 * j + 1][c]);
                }
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 0; i < PIECES; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int r = i * 32 + l * 4 + 2 * p, col = col0 + c0 + c;
                if (c0 + c < cols && col < dv) {
                    const float2 f = unpack2(S[2 * i + p][c]);
                    if (r < a.dk) st[(size_t)r * dv + col] = f.x;
                    if (r + 1 < a.dk) st[(size_t)(r + 1) * dv + col] = f.y;
                }
            }
}

static int scan_columns(int B, int H, int dv) {
    // Columns of a block: 32, or fewer where that leaves multiprocessors without a block.
    int cols = 32;
    while (cols > 8 && (long)B * H * ((dv + cols - 1) / cols) < 100) cols >>= 1;
    return cols;
}

template <int KR, int NC>
static int scan_launch(const DeltaArgs& a, int B, cudaStream_t stream) {
    const int cols = scan_columns(B, a.H, a.dv), threads = cols / (4 * NC) * 32;
    const size_t smem = (size_t)DS_STAGES * ((3 * DC + 1) * KR * LPC + DC * cols + DSCAL) * sizeof(float);
    if (smem > 48 * 1024 &&
        cudaFuncSetAttribute(delta_scan_kernel<KR, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return lq_launch_status();
    return launch_pdl(delta_scan_kernel<KR, NC>, dim3(B, a.H, (a.dv + cols - 1) / cols), dim3(threads), smem, stream, a, cols);
}

// Floats of scratch that a step with prompts needs for its records.
LQ_EXPORT long long lq_delta_record_floats(int T, int B, int H, int dk, int dv) {
    return (long long)(T / DC + B) * H * record_floats(dk, dv);
}

// Prompts and portions: rows [T, stride] float32 (q, k, v, b side by side), z [T, H dk] float32 -> raw [T, H, dv].
LQ_EXPORT int lq_delta_prompt(const float* rows, int stride, int b_off, const float* taps_w, int taps, float* ring, const float* z,
                              const float* z_bias, const float* rate, float* state, const int* cu_rows, const int* slots,
                              const int* tok_pos, float* records, float* raw, int B, int max_new, int H, int G, int dk, int dv,
                              float q_scale, float unit_eps, cudaStream_t stream) {
    if (B <= 0 || max_new <= 0) return LQ_OK;
    if (dk < 1 || dk > 256 || dv < 1 || G < 1 || H % G || taps < 1) return LQ_BAD_SIZE;
    DeltaArgs a{rows, stride, b_off, taps_w, taps, 2 * G * dk + H * dv, ring, z, z_bias, rate, state, cu_rows, slots, tok_pos,
                records, raw, H, G, dk, dv, q_scale, unit_eps};
    const int rc = launch_pdl(delta_prepare_kernel, dim3((max_new + DC - 1) / DC, B, H), dim3(DP_THREADS), (size_t)2 * DC * dk * sizeof(float),
                              stream, a);
    if (rc != LQ_OK) return rc;
    const int kr = pad_rows(dk) / LPC;
    if (kr <= 4) return scan_launch<4, 2>(a, B, stream);
    if (kr <= 8) return scan_launch<8, 2>(a, B, stream);
    if (kr <= 12) return scan_launch<12, 2>(a, B, stream);
    if (kr <= 16) return scan_launch<16, 2>(a, B, stream);
    if (kr <= 20) return scan_launch<20, 1>(a, B, stream);
    if (kr <= 24) return scan_launch<24, 1>(a, B, stream);
    if (kr <= 28) return scan_launch<28, 1>(a, B, stream);
    return scan_launch<32, 1>(a, B, stream);
}

// ------------------------------------------------------------------ one token per sequence
struct DeltaSingleArgs {
    DeltaArgs d;
    int a_off, ra, g_off, rg;    // columns of rows that hold W_a1 x (ra of them) and W_g1 x (rg)
    const void* a2;              // [H * dk, ra_ld]
    const void* g2;              // [H * dv, rg_ld]
    int ra_ld, rg_ld;            // row lengths (whole eights; what lies beyond ra, rg is zero)
    const float* norm_w;         // [dv]
    float norm_eps;
    void* out;                   // [B, H * dv]
    int cg;                      // threads side by side along a row of the state
};

template <typename TW> __device__ __forceinline__ float dot_row(const TW* w, const float* x, int n);
template <> __device__ __forceinline__ float dot_row<float>(const float* w, const float* x, int n) {
    float s0 = 0.f, s1 = 0.f;
    for (int i = 0; i < n; i += 4) {
        const float4 f = *reinterpret_cast<const float4*>(w + i);
        s0 = fmaf(f.x, x[i], s0); s1 = fmaf(f.y, x[i + 1], s1);
        s0 = fmaf(f.z, x[i + 2], s0); s1 = fmaf(f.w, x[i + 3], s1);
    }
    return s0 + s1;
}
template <> __device__ __forceinline__ float dot_row<__nv_bfloat16>(const __nv_bfloat16* w, const float* x, int n) {
    float s0 = 0.f, s1 = 0.f;
    for (int i = 0; i < n; i += 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(w + i);
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 f = __bfloat1622float2(p[j]);
            s0 = fmaf(f.x, x[i + 2 * j], s0);
            s1 = fmaf(f.y, x[i + 2 * j + 1], s1);
        }
    }
    return s0 + s1;
}

// One block per (sequence, value head).  The state's rows are dealt to groups of `cg` threads; a thread holds VW
// neighbouring columns of up to KR rows in registers between the read and the write.  Columns beyond cg * VW take
// another turn.
constexpr int DT_THREADS = 256;
template <typename T, typename TW, int KR, int VW>
__global__ void __launch_bounds__(DT_THREADS) delta_single_kernel(DeltaSingleArgs s) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    const DeltaArgs& a = s.d;
    const int dk = a.dk, dv = a.dv, H = a.H, G = a.G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int b = blockIdx.x, h = blockIdx.y, g = h / (H / G), taps = a.taps, keep = taps - 1;
    const int cg = s.cg, rg = DT_THREADS / cg, group = tid / cg, cl = tid % cg;
    float* sq = sm;                              // [dk]
    float* sk = sq + dk;                         // [dk]
    float* sa = sk + dk;                         // [dk] decays
    float* sv = sa + dk;                         // [dv]
    float* so = sv + dv;                         // [dv]
    float* sgate = so + dv;                      // [dv]
    float* xa = sgate + dv;                      // [ra_ld]
    float* xg = xa + s.ra_ld;                    // [rg_ld]
    float* red = xg + s.rg_ld;                   // [rg][2][cg * VW]
    __shared__ float sums[3], part[DT_THREADS / 32];
    pdl_wait();
    const int row = a.cu_rows[b], pos = a.tok_pos[row], slot = a.slots[b];
    const float* x = a.rows + (size_t)row * a.stride;
    float* ring = a.ring + (size_t)slot * taps * a.C;
    float* st = a.state + ((size_t)slot * H + h) * dk * dv;
    const bool live = group < rg;
    // The first columns of the state are on their way while the token's vectors are made.
    float S[KR][VW];
    auto load_state = [&](int col) {
#pragma unroll
        for (int i = 0; i < KR; ++i) {
            const int r = group + i * rg;
            const bool in = live && r < dk && col < dv;
            if constexpr (VW == 4) {
                const float4 f = in ? *reinterpret_cast<const float4*>(st + (size_t)r * dv + col) : make_float4(0.f, 0.f, 0.f, 0.f);
                S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
            } else {
                S[i][0] = in ? st[(size_t)r * dv + col] : 0.f;
            }
        }
    };
    load_state(cl * VW);
    for (int i = tid; i < s.ra_ld + s.rg_ld; i += DT_THREADS)
        xa[i] = i < s.ra_ld ? (i < s.ra ? x[s.a_off + i] : 0.f) : (i - s.ra_ld < s.rg ? x[s.g_off + i - s.ra_ld] : 0.f);
    for (int e = tid; e < 2 * dk + dv; e += DT_THREADS) {
        const int c = e < dk ? g * dk + e : (e < 2 * dk ? G * dk + g * dk + (e - dk) : 2 * G * dk + h * dv + (e - 2 * dk));
        const float own = x[c];
        float acc = 0.f;
        for (int j = 0; j < taps; ++j) {
            const int p = pos - keep + j;
            const float v = j == keep ? own : (p >= 0 ? ring[(size_t)(p % taps) * a.C + c] : 0.f);
            acc = fmaf(a.taps_w[(size_t)j * a.C + c], v, acc);
        }
        sq[e < 2 * dk ? e : dk + e] = silu_f(acc);                   // sq, sk, (sa), sv lie one after another
        // Of the value heads that share a key head, the first one's block moves its channels' ring on.
        if (e >= 2 * dk || h % (H / G) == 0) ring[(size_t)(pos % taps) * a.C + c] = own;
    }
    __syncthreads();
    if (warp == 0) {
        float qq = 0.f, kk = 0.f, qk = 0.f;
        for (int r = lane; r < dk; r += 32) {
            qq = fmaf(sq[r], sq[r], qq);
            kk = fmaf(sk[r], sk[r], kk);
            qk = fmaf(sq[r], sk[r], qk);
        }
        qq = warp_sum(qq);
        kk = warp_sum(kk);
        qk = warp_sum(qk);
        if (lane == 0) {
            sums[0] = a.q_scale / sqrtf(qq + a.unit_eps);
            sums[1] = 1.f / sqrtf(kk + a.unit_eps);
            sums[2] = qk * sums[0] * sums[1];
        }
    }
    for (int e = tid; e < dk + dv; e += DT_THREADS) {
        if (e < dk) {
            const float z = dot_row<TW>((const TW*)s.a2 + (size_t)(h * dk + e) * s.ra_ld, xa, s.ra_ld) + a.z_bias[h * dk + e];
            sa[e] = expf(-a.rate[h] * softplus_f(z));
        } else {
            sgate[e - dk] = sigmoid_f(dot_row<TW>((const TW*)s.g2 + (size_t)(h * dv + e - dk) * s.rg_ld, xg, s.rg_ld));
        }
    }
    const float beta = sigmoid_f(x[a.b_off + h]);
    __syncthreads();
    const float iq = sums[0], ik = sums[1], qk = sums[2];
    const int tile = cg * VW;
    for (int c0 = 0; c0 < dv; c0 += tile) {
        const int col = c0 + cl * VW;
        if (c0 > 0) {
            load_state(col);
            __syncthreads();                     // the sums of the columns before have been read
        }
        float rk[VW], rq[VW];
#pragma unroll
        for (int v = 0; v < VW; ++v) rk[v] = rq[v] = 0.f;
#pragma unroll
        for (int i = 0; i < KR; ++i) {
            const int r = group + i * rg;
            if (live && r < dk) {
                const float d = sa[r], k = sk[r], q = sq[r];
#pragma unroll
                for (int v = 0; v < VW; ++v) {
                    S[i][v] *= d;
                    rk[v] = fmaf(S[i][v], k, rk[v]);
                    rq[v] = fmaf(S[i][v], q, rq[v]);
                }
            }
        }
        if (live) {
#pragma unroll
            for (int v = 0; v < VW; ++v) {
                red[(group * 2) * tile + cl * VW + v] = rk[v];
                red[(group * 2 + 1) * tile + cl * VW + v] = rq[v];
            }
        }
        __syncthreads();
        float u[VW];
        if (live && col < dv) {
#pragma unroll
            for (int v = 0; v < VW; ++v) {
                float sum_k = 0.f;
                for (int w = 0; w < rg; ++w) sum_k += red[(w * 2) * tile + cl * VW + v];
                u[v] = beta * (sv[col + v] - ik * sum_k);
            }
            if (group == 0) {
#pragma unroll
                for (int v = 0; v < VW; ++v) {
                    float sum_q = 0.f;
                    for (int w = 0; w < rg; ++w) sum_q += red[(w * 2 + 1) * tile + cl * VW + v];
                    so[col + v] = fmaf(qk, u[v], iq * sum_q);
                }
            }
#pragma unroll
            for (int i = 0; i < KR; ++i) {
                const int r = group + i * rg;
                if (r < dk) {
                    const float k = sk[r] * ik;
                    if constexpr (VW == 4) {
                        *reinterpret_cast<float4*>(st + (size_t)r * dv + col) =
                            make_float4(fmaf(k, u[0], S[i][0]), fmaf(k, u[1], S[i][1]), fmaf(k, u[2], S[i][2]), fmaf(k, u[3], S[i][3]));
                    } else {
                        st[(size_t)r * dv + col] = fmaf(k, u[0], S[i][0]);
                    }
                }
            }
        }
    }
    __syncthreads();
    // The head over its root mean square, times the shared weight and the gate.
    float ss = 0.f;
    for (int d = tid; d < dv; d += DT_THREADS) ss = fmaf(so[d], so[d], ss);
    ss = warp_sum(ss);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < DT_THREADS / 32; ++w) total += part[w];
    const float inv = 1.f / sqrtf(total / (float)dv + s.norm_eps);
    T* out = (T*)s.out + ((size_t)row * H + h) * dv;
    for (int d = tid; d < dv; d += DT_THREADS) out[d] = from_f32<T>(so[d] * inv * s.norm_w[d] * sgate[d]);
}

template <typename T, typename TW>
static int single_launch(DeltaSingleArgs& s, int B, cudaStream_t stream) {
    const int dk = s.d.dk, dv = s.d.dv, vw = dv % 4 == 0 ? 4 : 1;
    // As many threads along a row as there are columns, unless that leaves a thread too many rows.
    int cg = min((dv + vw - 1) / vw, DT_THREADS);
    while (cg > 1 && (dk + DT_THREADS / cg - 1) / (DT_THREADS / cg) > 16) cg = (cg + 1) / 2;
    s.cg = cg;
    const int rg = DT_THREADS / cg, kr = (dk + rg - 1) / rg;
    if (kr > 16) return LQ_BAD_SIZE;
    const size_t smem = (size_t)(3 * dk + 3 * dv + s.ra_ld + s.rg_ld + rg * 2 * cg * vw) * sizeof(float);
    auto go = [&](auto kernel) {
        if (smem > 48 * 1024 &&
            cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return lq_launch_status();
        return launch_pdl(kernel, dim3(B, s.d.H), dim3(DT_THREADS), smem, stream, s);
    };
    if (vw == 4) {
        if (kr <= 4) return go(delta_single_kernel<T, TW, 4, 4>);
        if (kr <= 8) return go(delta_single_kernel<T, TW, 8, 4>);
        return go(delta_single_kernel<T, TW, 16, 4>);
    }
    return go(delta_single_kernel<T, TW, 16, 1>);
}

// One token per sequence (row cu_rows[b] of rows): out [B, H dv], normed and gated.
LQ_EXPORT int lq_delta_single(const float* rows, int stride, int b_off, const float* taps_w, int taps, float* ring,
                              const float* z_bias, const float* rate, float* state, const int* cu_rows, const int* slots,
                              const int* tok_pos, int a_off, int ra, const void* a2, int ra_ld, int g_off, int rg, const void* g2,
                              int rg_ld, int w_dtype, const float* norm_w, float norm_eps, void* out, int out_dtype, int B, int H,
                              int G, int dk, int dv, float q_scale, float unit_eps, cudaStream_t stream) {
    if (B <= 0) return LQ_OK;
    if (dk < 1 || dk > 256 || dv < 1 || dv > 4096 || G < 1 || H % G || taps < 1 || ra_ld % 8 || rg_ld % 8 || ra > ra_ld || rg > rg_ld)
        return LQ_BAD_SIZE;
    DeltaSingleArgs s{{rows, stride, b_off, taps_w, taps, 2 * G * dk + H * dv, ring, nullptr, z_bias, rate, state, cu_rows, slots, tok_pos,
                       nullptr, nullptr, H, G, dk, dv, q_scale, unit_eps},
                      a_off, ra, g_off, rg, a2, g2, ra_ld, rg_ld, norm_w, norm_eps, out, 1};
    typedef __nv_bfloat16 bf;
    if (out_dtype == LQ_F32 && w_dtype == LQ_F32) return single_launch<float, float>(s, B, stream);
    if (out_dtype == LQ_F32 && w_dtype == LQ_BF16) return single_launch<float, bf>(s, B, stream);
    if (out_dtype == LQ_BF16 && w_dtype == LQ_F32) return single_launch<bf, float>(s, B, stream);
    if (out_dtype == LQ_BF16 && w_dtype == LQ_BF16) return single_launch<bf, bf>(s, B, stream);
    return LQ_BAD_DTYPE;
}
