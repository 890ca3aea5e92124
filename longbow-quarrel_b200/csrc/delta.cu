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
// Products of decays only, never a quotient, so a decay of zero is harmless.  The state itself takes a decay as
// S + (a - 1) S with a - 1 from expm1: a decay close to one, rounded and then applied for a thousand tokens, would leave a
// trace of its rounding in what the first of them wrote.  delta_scan_kernel walks a sequence's
// records with the state in registers: one round of sums over the key rows per record instead of one per token.
//
// Linear attention with a fixed decay per head, S_t = d S_(t-1) + k_t v_t^T, o_t = S_t^T q_t (q, k and v through silu), takes
// the same road for prompts: it is the rule with u_t = v_t, so its records hold A_t q_t, the decayed k_s, A_DC - 1, N and v
// alone (linear_prepare_kernel), and the scan reads nothing out ahead of the write.
//
// Single tokens (one kernel, delta_single_kernel): convolution, unit vectors, the decays' and the output gate's second
// products (over their small inner sizes), the recurrence, the head's norm and the gate; the state is read and written once.
// The same kernel without the second products serves the rule with one decay per head (head_delta.cu has its prompts).
//
// The convolution's last inputs are kept per slot as a ring of `taps` rows, the row of position p at p % taps: a step
// of one token writes a row that it does not read.
#include "delta.cuh"

constexpr int DC = 4;                 // tokens of a record
// Scalars of a record: b [4], M [4][4] (t, s), N [4][4]; or N alone.
template <bool RULE> constexpr int scalars() { return RULE ? 4 + 16 + 16 : 16; }
// Vectors of a record over the key channels: A_t k_t [DC], A_t q_t [DC], decayed k_s [DC], A_DC - 1; without the first DC.
template <bool RULE> constexpr int vectors() { return RULE ? 3 * DC + 1 : 2 * DC + 1; }

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
    // Fixed decays: rows of either dtype, q, k and v where they lie, a decay per head.
    const void* lin_rows;
    int lin_stride, q_off, k_off, v_off;
    const float* decay;
};

// A record's rows of key channels are padded with zeros to whole 32s.
__host__ __device__ __forceinline__ int pad_rows(int dk) { return (dk + 31) / 32 * 32; }
__host__ __device__ __forceinline__ int pad4(int n) { return (n + 3) / 4 * 4; }
// Per (record, head): scalars, vectors [DKP] each, v [DC][pad4(dv)].
template <bool RULE> __host__ __device__ __forceinline__ int record_floats(int dk, int dv) {
    return scalars<RULE>() + vectors<RULE>() * pad_rows(dk) + DC * pad4(dv);
}
// Where the records of sequence b start: unique and never overlapping, whatever the sequences' lengths are.
__device__ __forceinline__ int first_record(const int* cu_rows, int b) { return cu_rows[b] / DC + b; }

// A warp per (record, value head), four heads a block; lane l holds the key channels l, l + 32, ... of its head (CPL of them),
// so every sum over them stays inside the warp.
constexpr int DP_WARPS = 4;
template <int CPL>
__global__ void __launch_bounds__(DP_WARPS * 32, CPL <= 2 ? 6 : CPL <= 4 ? 5 : 1) delta_prepare_kernel(DeltaArgs a) {
    pdl_launch_dependents();
    const int dk = a.dk, dv = a.dv, lane = threadIdx.x & 31, h = blockIdx.z * DP_WARPS + (threadIdx.x >> 5), b = blockIdx.y;
    pdl_wait();
    if (h >= a.H) return;
    const int g = h / (a.H / a.G), t0 = blockIdx.x * DC, row0 = a.cu_rows[b], n_rows = a.cu_rows[b + 1] - row0;
    if (t0 >= n_rows) return;
    const int n = min(DC, n_rows - t0), taps = a.taps, keep = taps - 1;
    const int pos0 = a.tok_pos[row0];            // the step's first position of this sequence
    const float* ring = a.ring + (size_t)a.slots[b] * taps * a.C;
    const int dkp = pad_rows(dk), dvp = pad4(dv);
    float* rec = a.records + ((size_t)(first_record(a.cu_rows, b) + blockIdx.x) * a.H + h) * record_floats<true>(dk, dv);
    float* vec = rec + scalars<true>();
    float* rec_v = vec + vectors<true>() * dkp;
    // The raw input of channel c at the step's row i (below 0: a row of an earlier step, zero ahead of the sequence).
    auto input = [&](int i, int c) -> float {
        if (i >= 0) return a.rows[(size_t)(row0 + i) * a.stride + c];
        const int p = pos0 + i;
        return p >= 0 ? ring[(size_t)(p % taps) * a.C + c] : 0.f;
    };
    // Convolution and silu of channel c for the record's tokens; zero behind the last one.
    auto conv = [&](int c, float (&y)[DC]) {
#pragma unroll
        for (int t = 0; t < DC; ++t) y[t] = 0.f;
        if (taps == 4 && t0 >= 3 && n == DC) {   // the usual case: four taps, every row the step's own
            const float* p = a.rows + (size_t)(row0 + t0 - 3) * a.stride + c;
            float x[DC + 3];
#pragma unroll
            for (int i = 0; i < DC + 3; ++i, p += a.stride) x[i] = *p;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float w = a.taps_w[(size_t)j * a.C + c];
#pragma unroll
                for (int t = 0; t < DC; ++t) y[t] = fmaf(w, x[t + j], y[t]);
            }
#pragma unroll
            for (int t = 0; t < DC; ++t) y[t] = silu_f(y[t]);
            return;
        }
        if (taps <= 5) {
            float x[DC + 4];
#pragma unroll
            for (int i = 0; i < DC + 4; ++i) x[i] = (i < n + keep) ? input(t0 + i - keep, c) : 0.f;
#pragma unroll
            for (int j = 0; j < 5; ++j)
                if (j < taps) {
                    const float w = a.taps_w[(size_t)j * a.C + c];
#pragma unroll
                    for (int t = 0; t < DC; ++t) y[t] = fmaf(w, x[t + j], y[t]);
                }
        } else {
            for (int j = 0; j < taps; ++j) {
                const float w = a.taps_w[(size_t)j * a.C + c];
#pragma unroll
                for (int t = 0; t < DC; ++t)
                    if (t < n) y[t] = fmaf(w, input(t0 + t - keep + j, c), y[t]);
            }
        }
#pragma unroll
        for (int t = 0; t < DC; ++t) y[t] = t < n ? silu_f(y[t]) : 0.f;
    };
    float q[CPL][DC], k[CPL][DC], z[CPL][DC];
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int r = i * 32 + lane;
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            q[i][t] = k[i][t] = 0.f;
            z[i][t] = (r < dk && t < n) ? a.z[(size_t)(row0 + t0 + t) * a.H * dk + h * dk + r] + a.z_bias[h * dk + r] : 0.f;
        }
        if (r < dk) {
            conv(g * dk + r, q[i]);
            conv(a.G * dk + g * dk + r, k[i]);
        }
    }
    // Unit vectors.
#pragma unroll
    for (int t = 0; t < DC; ++t) {
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            s0 = fmaf(q[i][t], q[i][t], s0);
            s1 = fmaf(k[i][t], k[i][t], s1);
        }
        s0 = a.q_scale / sqrtf(warp_sum(s0) + a.unit_eps);
        s1 = 1.f / sqrtf(warp_sum(s1) + a.unit_eps);
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            q[i][t] *= s0;
            k[i][t] *= s1;
        }
    }
    // Decays, the decayed vectors, and the lane's share of the sixteen sums over the key channels:
    // M_10, M_20, M_21, M_30, M_31, M_32, then N_00, N_10, N_11, N_20, ... N_33.
    float part[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) part[i] = 0.f;
    const float rate = a.rate[h];
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int r = i * 32 + lane;
        float A = 1.f, log_a = 0.f;
        float kd[DC];                            // k_s times the decays after s, up to the token being walked
        int m = 0, nn = 6;
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            float d = 1.f;
            if (r < dk && t < n) {
                const float log_d = -rate * softplus_f(z[i][t]);
                d = expf(log_d);
                log_a += log_d;
            }
            A *= d;
#pragma unroll
            for (int s = 0; s < t; ++s) {
                kd[s] *= d;
                part[m] = fmaf(kd[s], k[i][t], part[m]);
                ++m;
            }
            kd[t] = k[i][t];
#pragma unroll
            for (int s = 0; s <= t; ++s) {
                part[nn] = fmaf(kd[s], q[i][t], part[nn]);
                ++nn;
            }
            vec[t * dkp + r] = A * k[i][t];
            vec[(DC + t) * dkp + r] = A * q[i][t];
        }
#pragma unroll
        for (int s = 0; s < DC; ++s) vec[(2 * DC + s) * dkp + r] = kd[s];
        vec[3 * DC * dkp + r] = expm1f(log_a);
    }
    for (int e = lane; e < dvp; e += 32) {
        float y[DC] = {};
        if (e < dv) conv(2 * a.G * dk + h * dv + e, y);
#pragma unroll
        for (int t = 0; t < DC; ++t) rec_v[t * dvp + e] = y[t];
    }
    // Sixteen sums over a warp at once (a lane hands half of its values across and keeps the other half): lane l gets sum l & 15.
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
    const float sum = part[0] + __shfl_xor_sync(0xffffffffu, part[0], 16);
    // Lane l writes entry l & 15 of M (l < 16) or N: row t, column s.
    const int t = (lane >> 2) & 3, s = lane & 3;
    const int at = lane >= 16 ? (s <= t ? 6 + t * (t + 1) / 2 + s : -1) : (s < t ? t * (t - 1) / 2 + s : -1);
    const float entry = __shfl_sync(0xffffffffu, sum, at < 0 ? 0 : at);
    rec[4 + lane] = at < 0 ? 0.f : entry;
    if (lane < DC) rec[lane] = lane < n ? sigmoid_f(a.rows[(size_t)(row0 + t0 + lane) * a.stride + a.b_off + h]) : 0.f;
}

// The records of linear attention with a fixed decay per head: a warp per (record, head) as above.
template <typename T, int CPL>
__global__ void __launch_bounds__(DP_WARPS * 32) linear_prepare_kernel(DeltaArgs a) {
    pdl_launch_dependents();
    const int dk = a.dk, dv = a.dv, lane = threadIdx.x & 31, h = blockIdx.z * DP_WARPS + (threadIdx.x >> 5), b = blockIdx.y;
    pdl_wait();
    if (h >= a.H) return;
    const int t0 = blockIdx.x * DC, row0 = a.cu_rows[b], n_rows = a.cu_rows[b + 1] - row0;
    if (t0 >= n_rows) return;
    const int n = min(DC, n_rows - t0), dkp = pad_rows(dk), dvp = pad4(dv);
    float* rec = a.records + ((size_t)(first_record(a.cu_rows, b) + blockIdx.x) * a.H + h) * record_floats<false>(dk, dv);
    float* vec = rec + scalars<false>();
    float* rec_v = vec + vectors<false>() * dkp;
    const T* x = (const T*)a.lin_rows + (size_t)(row0 + t0) * a.lin_stride;
    const float d = a.decay[h];
    float part[16];                              // N_00, N_10, N_11, N_20, ... N_33, less the powers of d; six unused
#pragma unroll
    for (int i = 0; i < 16; ++i) part[i] = 0.f;
    // What is left of the state's size behind each token, and behind the record (nothing decays where there is no token).
    float A[DC], last = 1.f;
#pragma unroll
    for (int t = 0; t < DC; ++t) A[t] = last = t < n ? last * d : last;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int r = i * 32 + lane;
        float q[DC], k[DC];
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            const bool in = r < dk && t < n;
            q[t] = in ? silu_f(to_f32(x[(size_t)t * a.lin_stride + a.q_off + h * dk + r])) : 0.f;
            k[t] = in ? silu_f(to_f32(x[(size_t)t * a.lin_stride + a.k_off + h * dk + r])) : 0.f;
        }
        int nn = 0;
#pragma unroll
        for (int t = 0; t < DC; ++t)
#pragma unroll
            for (int s = 0; s <= t; ++s) {
                part[nn] = fmaf(k[s], q[t], part[nn]);
                ++nn;
            }
#pragma unroll
        for (int t = 0; t < DC; ++t) {
            float left = k[t];                   // k_t behind the record's later tokens
#pragma unroll
            for (int s = t + 1; s < DC; ++s)
                if (s < n) left *= d;
            vec[t * dkp + r] = A[t] * q[t];
            vec[(DC + t) * dkp + r] = left;
        }
        // d^n - 1 by the binomial of d - 1, so that a decay close to one keeps its digits.
        const float e = d - 1.f;
        float E = 0.f;
#pragma unroll
        for (int t = 0; t < DC; ++t)
            if (t < n) E = fmaf(E, d, e);
        vec[2 * DC * dkp + r] = E;
    }
    for (int c = lane; c < dvp; c += 32)
#pragma unroll
        for (int t = 0; t < DC; ++t)
            rec_v[t * dvp + c] = (c < dv && t < n) ? silu_f(to_f32(x[(size_t)t * a.lin_stride + a.v_off + h * dv + c])) : 0.f;
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
    const float sum = part[0] + __shfl_xor_sync(0xffffffffu, part[0], 16);
    const int t = (lane >> 2) & 3, s = lane & 3;
    const float entry = __shfl_sync(0xffffffffu, sum, s <= t ? t * (t + 1) / 2 + s : 0);
    if (lane < 16) {
        float p = 1.f;
        for (int j = s; j < t; ++j) p *= d;
        rec[lane] = s <= t ? p * entry : 0.f;
    }
}

// One block per (sequence, value head, some value columns): a warp takes 32 / LPC groups of NC neighbouring columns, LPC lanes
// share a group, each with KR of the key rows.  The last warp brings the records into a ring in shared memory by bulk
// copies; the others take them from there at their own pace.
constexpr int DS_STAGES = 6;
template <int KR, int LPC, int NC, bool RULE>
__device__ __forceinline__ void scan_records(const DeltaArgs& a, int cols) {
    using namespace tc;
    pdl_launch_dependents();
    constexpr int DKP = KR * LPC, PIECES = KR / 4, SPAN = 4 * LPC;
    // Vectors that the state is read out with: with the rule first those of k, then (QV on) those of q.
    constexpr int READ = RULE ? 2 * DC : DC, QV = RULE ? DC : 0, PER = READ * NC / LPC, KD = READ;
    static_assert(PER >= 1 && PER <= NC && NC % PER == 0, "every lane is left with sums of one token");
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(8) uint64_t full[DS_STAGES], empty[DS_STAGES];
    const int dv = a.dv, dvp = pad4(dv), H = a.H, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & (LPC - 1);
    const int consumers = (blockDim.x >> 5) - 1;
    const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols;
    constexpr int HEAD = scalars<RULE>() + vectors<RULE>() * DKP;        // a record ahead of its values
    const int stage_floats = HEAD + DC * cols;
    const int rf = record_floats<RULE>(a.dk, dv);
    if (tid == 0) {
        for (int i = 0; i < DS_STAGES; ++i) {
            mbar_init(smem_u32(&full[i]), 1);
            mbar_init(smem_u32(&empty[i]), consumers);
        }
        mbar_fence_init();
    }
    __syncthreads();
    pdl_wait();
    const int row0 = a.cu_rows[b], row1 = a.cu_rows[b + 1], n_rec = (row1 - row0 + DC - 1) / DC;
    if (warp == consumers) {
        if (lane == 0) {
            const float* src = a.records + ((size_t)first_record(a.cu_rows, b) * H + h) * rf;
            const uint32_t v_bytes = (uint32_t)min(cols, dvp - col0) * 4;            // whole fours
            int i = 0;
            for (; i < n_rec; ++i, src += (size_t)H * rf) {
                const int s = i % DS_STAGES;
                if (!mbar_wait(smem_u32(&empty[s]), ((i / DS_STAGES) & 1) ^ 1)) { give_up(1); break; }
                const uint32_t bar = smem_u32(&full[s]), dst = smem_u32(sm + s * stage_floats);
                mbar_expect_tx(bar, HEAD * 4 + DC * v_bytes);
                bulk_load(dst, src, HEAD * 4, bar);
#pragma unroll
                for (int t = 0; t < DC; ++t) bulk_load(dst + (HEAD + t * cols) * 4, src + HEAD + t * dvp + col0, v_bytes, bar);
            }
            // After a wait that gave up, the copies that were started must land before the shared memory goes away.
            if (i < n_rec)
                for (int back = 1; back <= DS_STAGES && back <= i; ++back) mbar_wait(smem_u32(&full[(i - back) % DS_STAGES]), ((i - back) / DS_STAGES) & 1);
        }
        return;
    }
    // The convolution's last inputs go to the ring; the blocks of a sequence share its channels.  (The records ahead
    // of this kernel were made from the ring as it was.)
    if constexpr (RULE) {
        const int share = gridDim.y * gridDim.z, mine = blockIdx.y * gridDim.z + blockIdx.z, taps = a.taps;
        const int per = (a.C + share - 1) / share, lo = mine * per, hi = min(a.C, lo + per), n = row1 - row0;
        float* ring = a.ring + (size_t)a.slots[b] * taps * a.C;
        for (int i = max(0, n - taps); i < n; ++i) {
            const int p = a.tok_pos[row0 + i];
            for (int c = lo + tid; c < hi; c += consumers * 32)
                ring[(size_t)(p % taps) * a.C + c] = a.rows[(size_t)(row0 + i) * a.stride + c];
        }
    }
    const int c0 = warp * (32 / LPC) * NC + (lane / LPC) * NC;       // this thread's first column inside the block's
    float* st = a.state + ((size_t)a.slots[b] * H + h) * a.dk * dv;
    f2 S[KR / 2][NC];                            // rows SPAN i + 4 l + {0, 1}, {2, 3} as pairs 2 i, 2 i + 1
#pragma unroll
    for (int i = 0; i < PIECES; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int r = i * SPAN + l * 4 + 2 * p, col = col0 + c0 + c;
                const bool in = c0 + c < cols && col < dv;
                S[2 * i + p][c] = pack2(in && r < a.dk ? st[(size_t)r * dv + col] : 0.f, in && r + 1 < a.dk ? st[(size_t)(r + 1) * dv + col] : 0.f);
            }
    for (int i = 0; i < n_rec; ++i) {
        const int stage = i % DS_STAGES;
        if (!mbar_wait(smem_u32(&full[stage]), (i / DS_STAGES) & 1)) { give_up(2); break; }
        const float* rec = sm + stage * stage_floats;
        const float* vec = rec + scalars<RULE>() + l * 4;
        const float* vs = rec + HEAD + c0;
        const float4* sc = reinterpret_cast<const float4*>(rec);
        f2 acc2[READ][NC];
#pragma unroll
        for (int t = 0; t < READ; ++t)
#pragma unroll
            for (int c = 0; c < NC; ++c) acc2[t][c] = 0ull;
#pragma unroll
        for (int j = 0; j < PIECES; ++j)
#pragma unroll
            for (int t = 0; t < READ; ++t) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(vec + t * DKP + j * SPAN);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    acc2[t][c] = fma2(S[2 * j][c], x.x, acc2[t][c]);
                    acc2[t][c] = fma2(S[2 * j + 1][c], x.y, acc2[t][c]);
                }
            }
        // What token t reads from the state with k (sum t * NC + c of column c) and with q (sum (QV + t) * NC + c) is added up
        // over the LPC lanes of the columns: in each step a lane hands half of its sums across and keeps the other half, so
        // lane l is left with the sums PER l .. PER l + PER - 1.
        float acc[READ * NC];
#pragma unroll
        for (int t = 0; t < READ; ++t)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float2 f = unpack2(acc2[t][c]);
                acc[t * NC + c] = f.x + f.y;
            }
#pragma unroll
        for (int w = LPC / 2; w >= 1; w >>= 1) {
            const bool upper = l & w;
            const int half = PER * w;
#pragma unroll
            for (int v = 0; v < half; ++v) {
                const float give = upper ? acc[v] : acc[v + half];
                const float keep = upper ? acc[v + half] : acc[v];
                acc[v] = keep + __shfl_xor_sync(0xffffffffu, give, w);
            }
        }
        float u[DC][NC];
        if constexpr (RULE) {
            const float4 beta = sc[0], m1 = sc[2], m2 = sc[3], m3 = sc[4];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float r[DC];
#pragma unroll
                for (int t = 0; t < DC; ++t)
                    r[t] = vs[t * cols + c] - __shfl_sync(0xffffffffu, acc[(t * NC + c) % PER], (lane & ~(LPC - 1)) + (t * NC + c) / PER);
                u[0][c] = beta.x * r[0];
                u[1][c] = beta.y * (r[1] - m1.x * u[0][c]);
                u[2][c] = beta.z * (r[2] - m2.x * u[0][c] - m2.y * u[1][c]);
                u[3][c] = beta.w * (r[3] - m3.x * u[0][c] - m3.y * u[1][c] - m3.z * u[2][c]);
            }
        } else {
#pragma unroll
            for (int t = 0; t < DC; ++t)
#pragma unroll
                for (int c = 0; c < NC; ++c) u[t][c] = vs[t * cols + c];
        }
        if (l * PER >= QV * NC) {                // the lanes that hold sums with q
            const int t = (l * PER) / NC - QV, cc = (l * PER) % NC, row = row0 + i * DC + t;
            const float4 nt = sc[(RULE ? 5 : 0) + t];
#pragma unroll
            for (int v = 0; v < PER; ++v) {
                const int col = c0 + cc + v;
                // u of column cc + v: picked without indexing registers by a number that is not known when compiling
                float u0 = u[0][v], u1 = u[1][v], u2 = u[2][v], u3 = u[3][v];
#pragma unroll
                for (int c = v + PER; c < NC; c += PER)
                    if (cc + v == c) { u0 = u[0][c]; u1 = u[1][c]; u2 = u[2][c]; u3 = u[3][c]; }
                if (row < row1 && col < cols && col0 + col < dv)
                    a.raw[((size_t)row * H + h) * dv + col0 + col] = acc[v] + nt.x * u0 + nt.y * u1 + nt.z * u2 + nt.w * u3;
            }
        }
        f2 uu[DC][NC];
#pragma unroll
        for (int s = 0; s < DC; ++s)
#pragma unroll
            for (int c = 0; c < NC; ++c) uu[s][c] = pack2(u[s][c], u[s][c]);
#pragma unroll
        for (int j = 0; j < PIECES; ++j) {
            const ulonglong2 E = *reinterpret_cast<const ulonglong2*>(vec + (KD + DC) * DKP + j * SPAN);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                S[2 * j][c] = fma2(S[2 * j][c], E.x, S[2 * j][c]);
                S[2 * j + 1][c] = fma2(S[2 * j + 1][c], E.y, S[2 * j + 1][c]);
            }
#pragma unroll
            for (int s = 0; s < DC; ++s) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(vec + (KD + s) * DKP + j * SPAN);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    S[2 * j][c] = fma2(x.x, uu[s][c], S[2 * j][c]);
                    S[2 * j + 1][c] = fma2(x.y, uu[s][c], S[2 * j + 1][c]);
                }
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&empty[stage]));
    }
#pragma unroll
    for (int i = 0; i < PIECES; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const int r = i * SPAN + l * 4 + 2 * p, col = col0 + c0 + c;
                if (c0 + c < cols && col < dv) {
                    const float2 f = unpack2(S[2 * i + p][c]);
                    if (r < a.dk) st[(size_t)r * dv + col] = f.x;
                    if (r + 1 < a.dk) st[(size_t)(r + 1) * dv + col] = f.y;
                }
            }
}

template <int KR, int LPC, int NC>
__global__ void __launch_bounds__(288, 1) delta_scan_kernel(const __grid_constant__ DeltaArgs a, int cols) { scan_records<KR, LPC, NC, true>(a, cols); }
template <int KR, int LPC, int NC>
__global__ void __launch_bounds__(288, 1) linear_records_kernel(const __grid_constant__ DeltaArgs a, int cols) { scan_records<KR, LPC, NC, false>(a, cols); }

static int scan_columns(int B, int H, int dv, int least, int most) {
    // Columns of a block: as many as it has warps for, or fewer where that leaves multiprocessors without a block.
    int cols = most;
    while (cols / 2 >= least && cols % 8 == 0 && (long)B * H * ((dv + cols - 1) / cols) < 100) cols >>= 1;
    return cols;
}

template <bool RULE, int KR, int LPC, int NC>
static int scan_launch(const DeltaArgs& a, int B, cudaStream_t stream) {
    constexpr int PER_WARP = 32 / LPC * NC;
    const int cols = scan_columns(B, a.H, a.dv, PER_WARP, 32 < 8 * PER_WARP ? 32 : 8 * PER_WARP), threads = (cols / PER_WARP + 1) * 32;
    const size_t smem = (size_t)DS_STAGES * (scalars<RULE>() + vectors<RULE>() * KR * LPC + DC * cols) * sizeof(float);
    auto go = [&](auto kernel) {
        if (smem > 48 * 1024 &&
            cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return lq_launch_status();
        // Not ahead of its time: blocks that start while the records are still being made take what room they find, several
        // on one multiprocessor, and stay there; started afterwards they spread out (measured: half the time).
        return launch_after(kernel, dim3(B, a.H, (a.dv + cols - 1) / cols), dim3(threads), smem, stream, a, cols);
    };
    if constexpr (RULE) return go(delta_scan_kernel<KR, LPC, NC>);
    else return go(linear_records_kernel<KR, LPC, NC>);
}

template <int CPL>
static int prepare_launch(const DeltaArgs& a, int B, int max_new, cudaStream_t stream) {
    return launch_pdl(delta_prepare_kernel<CPL>, dim3((max_new + DC - 1) / DC, B, (a.H + DP_WARPS - 1) / DP_WARPS), dim3(DP_WARPS * 32), 0,
                      stream, a);
}

// Floats of scratch that a step with prompts needs for its records.
LQ_EXPORT long long lq_delta_record_floats(int T, int B, int H, int dk, int dv) {
    return (long long)(T / DC + B) * H * record_floats<true>(dk, dv);
}
LQ_EXPORT long long lq_linear_record_floats(int T, int B, int H, int dk, int dv) {
    return (long long)(T / DC + B) * H * record_floats<false>(dk, dv);
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
    switch (pad_rows(dk) / 32) {
#define LQ_GO(CPL) case CPL: { \
        const int rc = prepare_launch<CPL>(a, B, max_new, stream); \
        return rc != LQ_OK ? rc : scan_launch<true, 4 * CPL, 8, 2>(a, B, stream); }
        LQ_GO(1) LQ_GO(2) LQ_GO(3) LQ_GO(4) LQ_GO(5) LQ_GO(6) LQ_GO(7) LQ_GO(8)
#undef LQ_GO
    }
    return LQ_BAD_SIZE;
}

// The same for linear attention with a fixed decay per head: rows [T, stride] of either dtype, H heads of q at q_off, of k at
// k_off (dk each) and of v at v_off (dv each), all through silu -> raw [T, H, dv].
LQ_EXPORT int lq_linear_prompt(const void* rows, int dtype, int stride, int q_off, int k_off, int v_off, const float* decay, float* state,
                               const int* cu_rows, const int* slots, float* records, float* raw, int B, int max_new, int H, int dk, int dv,
                               cudaStream_t stream) {
    if (B <= 0 || max_new <= 0) return LQ_OK;
    if (dk < 1 || dk > 256 || dv < 1) return LQ_BAD_SIZE;
    if (dtype != LQ_F32 && dtype != LQ_BF16) return LQ_BAD_DTYPE;
    DeltaArgs a{};
    a.state = state; a.cu_rows = cu_rows; a.slots = slots; a.records = records; a.raw = raw;
    a.H = a.G = H; a.dk = dk; a.dv = dv;
    a.lin_rows = rows; a.lin_stride = stride; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.decay = decay;
    const dim3 grid((max_new + DC - 1) / DC, B, (H + DP_WARPS - 1) / DP_WARPS), block(DP_WARPS * 32);
    switch (pad_rows(dk) / 32) {
#define LQ_GO(CPL) case CPL: { \
        const int rc = dtype == LQ_F32 ? launch_pdl(linear_prepare_kernel<float, CPL>, grid, block, 0, stream, a) \
                                       : launch_pdl(linear_prepare_kernel<__nv_bfloat16, CPL>, grid, block, 0, stream, a); \
        return rc != LQ_OK ? rc : scan_launch<false, 4 * CPL, 8, 2>(a, B, stream); }
        LQ_GO(1) LQ_GO(2) LQ_GO(3) LQ_GO(4) LQ_GO(5) LQ_GO(6) LQ_GO(7) LQ_GO(8)
#undef LQ_GO
    }
    return LQ_BAD_SIZE;
}

LQ_EXPORT int lq_delta_status() { return tc::status_read(); }
LQ_EXPORT int* lq_delta_status_word() { return tc::status_word(); }

// ------------------------------------------------------------------ one token per sequence
struct DeltaSingleArgs {
    DeltaArgs d;
    int a_off, ra, g_off, rg;    // columns of rows that hold W_a1 x (ra of them) and W_g1 x (rg)
    const void* a2;              // [H * dk, ra_ld]
    const void* g2;              // [H * dv, rg_ld]
    int ra_ld, rg_ld;            // row lengths (whole eights; what lies beyond ra, rg is zero)
    const float* norm_w;         // [dv]
    float norm_eps;
    void* out;                   // [B, H * dv], float32 or bfloat16
    int out_bf16;
    int cg;                      // threads side by side along a row of the state
};
// With one decay per head a_off and g_off are the columns of the decays' pre-activations [H] and of the output gate [H, dv]
// themselves, z_bias and rate are [H], and the gate is silu; there are no second products.

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
template <typename TW, int KR, int VW, bool HEAD>
__global__ void __launch_bounds__(DT_THREADS) delta_single_kernel(DeltaSingleArgs s) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];
    const DeltaArgs& a = s.d;
    const int dk = a.dk, dv = a.dv, H = a.H, G = a.G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int b = blockIdx.x, h = blockIdx.y, g = h / (H / G), taps = a.taps, keep = taps - 1;
    const int cg = s.cg, rg = DT_THREADS / cg, group = tid / cg, cl = tid % cg;
    float* sq = sm;                              // [dk]
    float* sk = sq + dk;                         // [dk]
    float* sa = sk + dk;                         // [dk] decays, less one
    float* sv = sa + dk;                         // [dv]
    float* so = sv + dv;                         // [dv]
    float* sgate = so + dv;                      // [dv]
    float* xa = sgate + dv;                      // [ra_ld]
    float* xg = xa + s.ra_ld;                    // [rg_ld]
    float* red = xg + s.rg_ld;                   // [rg][2][cg * VW]
    __shared__ float sums[3], part[DT_THREADS / 32];
    // Row, position and slot are written before the step starts, the state and the ring by the step before: they are read,
    // and the second products' weights asked for, before the kernel ahead is known to have finished.
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
    if constexpr (!HEAD)
    for (int e = tid; e < dk + dv; e += DT_THREADS) {
        const TW* w = e < dk ? (const TW*)s.a2 + (size_t)(h * dk + e) * s.ra_ld : (const TW*)s.g2 + (size_t)(h * dv + e - dk) * s.rg_ld;
        asm volatile("prefetch.global.L2 [%0];" ::"l"(w));
    }
    // Channel e of q, k (key head g) and v (head h), side by side as below; its sum over the taps on earlier inputs.
    auto channel = [&](int e) { return e < dk ? g * dk + e : (e < 2 * dk ? G * dk + g * dk + (e - dk) : 2 * G * dk + h * dv + (e - 2 * dk)); };
    for (int e = tid; e < 2 * dk + dv; e += DT_THREADS) {
        const int c = channel(e);
        float acc = 0.f;
#pragma unroll 4
        for (int j = 0; j < keep; ++j) {
            const int p = pos - keep + j;
            if (p >= 0) acc = fmaf(a.taps_w[(size_t)j * a.C + c], ring[(size_t)(p % taps) * a.C + c], acc);
        }
        sq[e < 2 * dk ? e : dk + e] = acc;                           // sq, sk, (sa), sv lie one after another
    }
    pdl_wait();
    if constexpr (!HEAD)
    for (int i = tid; i < s.ra_ld + s.rg_ld; i += DT_THREADS)
        xa[i] = i < s.ra_ld ? (i < s.ra ? x[s.a_off + i] : 0.f) : (i - s.ra_ld < s.rg ? x[s.g_off + i - s.ra_ld] : 0.f);
    for (int e = tid; e < 2 * dk + dv; e += DT_THREADS) {
        const int c = channel(e);
        const float own = x[c];
        float& y = sq[e < 2 * dk ? e : dk + e];                      // (the thread's own sum)
        y = silu_f(fmaf(a.taps_w[(size_t)keep * a.C + c], own, y));
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
    float head_decay = 0.f;                      // less one
    if constexpr (HEAD) {
        head_decay = expm1f(-a.rate[h] * softplus_f(x[s.a_off + h] + a.z_bias[h]));
        for (int e = tid; e < dv; e += DT_THREADS) sgate[e] = silu_f(x[s.g_off + h * dv + e]);
    } else
    for (int e = tid; e < dk + dv; e += DT_THREADS) {
        if (e < dk) {
            const float z = dot_row<TW>((const TW*)s.a2 + (size_t)(h * dk + e) * s.ra_ld, xa, s.ra_ld) + a.z_bias[h * dk + e];
            sa[e] = expm1f(-a.rate[h] * softplus_f(z));
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
                const float d = HEAD ? head_decay : sa[r], k = sk[r], q = sq[r];
#pragma unroll
                for (int v = 0; v < VW; ++v) {
                    S[i][v] = fmaf(S[i][v], d, S[i][v]);
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
    const size_t at = ((size_t)row * H + h) * dv;
    for (int d = tid; d < dv; d += DT_THREADS) {
        const float y = so[d] * inv * s.norm_w[d] * sgate[d];
        if (s.out_bf16) ((__nv_bfloat16*)s.out)[at + d] = __float2bfloat16_rn(y);
        else ((float*)s.out)[at + d] = y;
    }
}

template <typename TW, bool HEAD = false>
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
        if (kr <= 4) return go(delta_single_kernel<TW, 4, 4, HEAD>);
        if (kr <= 8) return go(delta_single_kernel<TW, 8, 4, HEAD>);
        return go(delta_single_kernel<TW, 16, 4, HEAD>);
    }
    return go(delta_single_kernel<TW, 16, 1, HEAD>);
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
                      a_off, ra, g_off, rg, a2, g2, ra_ld, rg_ld, norm_w, norm_eps, out, out_dtype == LQ_BF16, 1};
    if (out_dtype != LQ_F32 && out_dtype != LQ_BF16) return LQ_BAD_DTYPE;
    if (w_dtype == LQ_F32) return single_launch<float>(s, B, stream);
    if (w_dtype == LQ_BF16) return single_launch<__nv_bfloat16>(s, B, stream);
    return LQ_BAD_DTYPE;
}

// The same with one decay per head (z_bias and rate [H]): rows hold the decays' pre-activations at column a_off [H] and the
// output gate's at g_off [H, dv]; out [B, H dv] = the head over its root mean square times norm_w times silu(gate).
LQ_EXPORT int lq_head_delta_single(const float* rows, int stride, int b_off, const float* taps_w, int taps, float* ring,
                                   const float* z_bias, const float* rate, float* state, const int* cu_rows, const int* slots,
                                   const int* tok_pos, int a_off, int g_off, const float* norm_w, float norm_eps, void* out, int out_dtype,
                                   int B, int H, int G, int dk, int dv, float q_scale, float unit_eps, cudaStream_t stream) {
    if (B <= 0) return LQ_OK;
    if (dk < 1 || dk > 256 || dv < 1 || dv > 4096 || G < 1 || H % G || taps < 1) return LQ_BAD_SIZE;
    if (out_dtype != LQ_F32 && out_dtype != LQ_BF16) return LQ_BAD_DTYPE;
    DeltaSingleArgs s{{rows, stride, b_off, taps_w, taps, 2 * G * dk + H * dv, ring, nullptr, z_bias, rate, state, cu_rows, slots, tok_pos,
                       nullptr, nullptr, H, G, dk, dv, q_scale, unit_eps},
                      a_off, 0, g_off, 0, nullptr, nullptr, 0, 0, norm_w, norm_eps, out, out_dtype == LQ_BF16, 1};
    return single_launch<float, true>(s, B, stream);
}
