// Recurrences over a matrix state per head whose decays depend on the token, with the state in a slot of the cache
// manager (fp32, zero when a request begins).  Two kinds:
//
//   kind 0, a decay per key channel (gated linear attention), a_t = sigmoid(z_t + bias)^(1 / tau) per channel of the head:
//       S_t = diag(a_t) S_(t-1) + k_t v_t^T                       o_t = S_t^T q_t
//   kind 1, a matrix memory with exponential gates: log input gate i, log forget gate f per head and token, and a running
//   maximum m (0 when a request begins) that keeps every exponential at most 1:
//       i = cap tanh(zi / cap),  f = logsigmoid(cap tanh(zf / cap)),  m_t = max(f + m_(t-1), i)
//       S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k_t v_t^T,   n_t likewise with k_t alone
//       o_t = S_t^T q_t,   den_t = max(|n_t . q_t|, exp(-m_t)) + 1e-6     (the consumer divides, see heads_finish)
//
// q, k [heads x dk] and v [heads x dv] are columns of the token's projection row; q is multiplied by qscale.  Everything
// from the projections on is fp32.  A state slot holds S [heads][dk][dv] and, for kind 1, n [heads][dk] and
// m [heads][ceil(dv / 16) + 1]: a copy of the head's m for every 16 value columns and one for n, so that no CTA reads what
// another one writes.
//
// The scan walks the tokens of an entry one after the other and serves single tokens, short entries and float32; its
// result is bit-identical however a request was cut.  Longer bfloat16 entries run in blocks of 16 tokens on the tensor
// cores (state_prepare_kernel, state_blocks_kernel); the two differ by rounding only.
#include "common.cuh"

namespace {

struct StateArgs {
    const void* proj;            // [tokens, row_stride] activations
    long long row_stride;
    int q_col, k_col, v_col;
    float qscale;
    const float* z;              // kind 0: [tokens, H * dk] raw decays, their bias [H * dk] and 1 / tau
    const float* z_bias;
    float inv_tau;
    const float* gates;          // kind 1: raw gates [n_parts][tokens][2 H] (input gates, then forget gates), parts to be added
    int n_parts;
    long long part_stride;
    const float* gate_bias;      // [2 H]
    float cap;
    float* state;
    long long slot_stride;
    const int* slots;
    const int* cu;               // [n_seqs + 1]
    float* o;                    // [tokens, H * dv] fp32
    float* den;                  // kind 1: [tokens, H]
    int n_seqs, H, dk, dv;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// log decay of a head's channel
__device__ __forceinline__ float log_decay(const StateArgs& a, float z, int channel) { return log_sigmoid(__fadd_rn(z, a.z_bias[channel])) * a.inv_tau; }
__device__ __forceinline__ int m_copies(int dv) { return (dv + 15) / 16 + 1; }

// a token's raw gate logits of one head: column h the input gate's, column H + h the forget gate's
__device__ __forceinline__ float raw_gate(const StateArgs& a, size_t t, int col) {
    const float* p = a.gates + t * 2 * a.H + col;
    float z = p[0];
    for (int s = 1; s < a.n_parts; ++s) z += p[(size_t)s * a.part_stride];
    return __fadd_rn(z, a.gate_bias[col]);
}
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// ---------------------------------------------------------------------------
// Token by token.  Grid (tiles of 32 value columns, heads, entries); a CTA of four warps (two for dk <= 16) holds a
// [dk, 32] tile of the state in registers.  A warp owns eight columns, its lanes split the rows four ways in groups of
// four (row = 16 g + 4 r + e), so q, k and the decays come from shared memory as conflict-free 16-byte loads and the four
// row groups of a column meet in two shuffles.  Tokens are staged CH at a time (FEW: a step of single tokens, where
// staging more would only cost registers and instructions), the next ones on their way into registers meanwhile.  n and
// den belong to the first warp of tile 0.
// ---------------------------------------------------------------------------
template <int G, bool FEW> struct ScanShape {
    static constexpr int DP = 16 * G;
    static constexpr int WARPS = G >= 2 ? 4 : 2;
    static constexpr int THREADS = WARPS * 32;
    static constexpr int CT = WARPS * 8;                // columns of a tile
    static constexpr int CH = FEW ? (G == 3 ? 8 : 4) : G <= 8 ? 16 : 8;   // tokens staged at a time
    static constexpr int PER = CH * DP / THREADS;       // staged (token, row) pairs per thread
    static constexpr int PERV = CH * CT / THREADS;      // staged (token, column) pairs per thread
    static_assert(CH * DP % THREADS == 0 && CH * CT % THREADS == 0, "the threads stage whole chunks");
};

template <int G, int KIND, int U>
__device__ __forceinline__ void scan_tokens(float (&S)[4 * G], const float (*sq)[16 * G], const float (*sk)[16 * G],
                                            const float (*sd)[16 * G], const float (*sv)[ScanShape<G, false>::CT], const float* keep,
                                            const float* put, int tt, int r, int cw, bool store, float* o_at, size_t o_stride) {
    float acc[U];
#pragma unroll
    for (int x = 0; x < U; ++x) {
        float vj = sv[tt + x][cw];
        float kp = 1.f;
        if (KIND == 1) { vj *= put[tt + x]; kp = keep[tt + x]; }
        float s = 0.f;
#pragma unroll
        for (int g = 0; g < G; ++g) {
            const float4 k4 = *reinterpret_cast<const float4*>(&sk[tt + x][16 * g + 4 * r]);
            const float4 q4 = *reinterpret_cast<const float4*>(&sq[tt + x][16 * g + 4 * r]);
            float dd[4] = {kp, kp, kp, kp};
            if (KIND == 0) *reinterpret_cast<float4*>(dd) = *reinterpret_cast<const float4*>(&sd[tt + x][16 * g + 4 * r]);
            const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                S[4 * g + e] = fmaf(dd[e], S[4 * g + e], __fmul_rn(kk[e], vj));
                s = fmaf(S[4 * g + e], qq[e], s);
            }
        }
        acc[x] = s;
    }
#pragma unroll
    for (int x = 0; x < U; ++x) acc[x] += __shfl_xor_sync(0xffffffffu, acc[x], 8);
#pragma unroll
    for (int x = 0; x < U; ++x) acc[x] += __shfl_xor_sync(0xffffffffu, acc[x], 16);
    if (store) {
#pragma unroll
        for (int x = 0; x < U; ++x) o_at[(size_t)(tt + x) * o_stride] = acc[x];
    }
}

template <typename T, int G, int KIND, bool FEW>
__global__ void __launch_bounds__(ScanShape<G, FEW>::THREADS) state_scan_kernel(StateArgs a, int max_len) {
    using Sh = ScanShape<G, FEW>;
    constexpr int DP = Sh::DP, THREADS = Sh::THREADS, CT = Sh::CT, CH = Sh::CH, PER = Sh::PER, PERV = Sh::PERV;
    __shared__ __align__(16) float sq[CH][DP];
    __shared__ __align__(16) float sk[CH][DP];
    __shared__ __align__(16) float sd[KIND == 0 ? CH : 1][DP];
    __shared__ float sv[CH][CT];
    __shared__ float keep[CH], put[CH], least[CH];
    pdl_trigger();
    pdl_wait();
    const int tile = blockIdx.x, head = blockIdx.y, b = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int jj = lane & 7, r = lane >> 3;
    const int cw = warp * 8 + jj, col = tile * CT + cw;
    const int dk = a.dk, dv = a.dv, H = a.H;
    const bool col_ok = col < dv;
    const int t0 = a.cu[b], t1 = a.cu[b + 1];
    if (t1 <= t0 || (max_len > 0 && t1 - t0 > max_len)) return;
    float* slot = a.state + (size_t)a.slots[b] * a.slot_stride;
    float* Sg = slot + (size_t)head * dk * dv;
    float* ng = slot + (size_t)H * dk * dv + (size_t)head * dk;
    const int MB = m_copies(dv);
    float* mg = slot + (size_t)H * dk * dv + (size_t)H * dk + (size_t)head * MB;
    const bool owns_n = KIND == 1 && tile == 0 && warp == 0;
    constexpr int NR = (DP + 31) / 32;      // rows of n per lane: lane, lane + 32, ...

    float S[4 * G];
#pragma unroll
    for (int g = 0; g < G; ++g)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 16 * g + 4 * r + e;
            S[4 * g + e] = (col_ok && i < dk) ? Sg[(size_t)i * dv + col] : 0.f;
        }
    float nn[NR];
    float m = 0.f;
    if (KIND == 1) {
#pragma unroll
        for (int x = 0; x < NR; ++x) nn[x] = (owns_n && lane + 32 * x < dk) ? ng[lane + 32 * x] : 0.f;
        if (warp == 0) m = mg[tile * (CT / 16)];
    }

    const T* proj = (const T*)a.proj;
    const T* qs = proj + a.q_col + (size_t)head * dk;
    const T* ks = proj + a.k_col + (size_t)head * dk;
    const T* vs = proj + a.v_col + (size_t)head * dv + (size_t)tile * CT;
    T pq[PER], pk[PER], pv[PERV];
    float pd[KIND == 0 ? PER : 1], pi = 0.f, pf = 0.f;
    auto fetch = [&](int c0) {
        const int n = min(CH, t1 - c0);
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int e = p * THREADS + tid, tt = e / DP, i = e - tt * DP;
            const bool real = tt < n && i < dk;
            const size_t row = (size_t)(c0 + tt) * a.row_stride + i;
            pq[p] = real ? qs[row] : from_f32<T>(0.f);
            pk[p] = real ? ks[row] : from_f32<T>(0.f);
            if (KIND == 0) pd[p] = real ? a.z[((size_t)(c0 + tt) * H + head) * dk + i] : 0.f;
        }
#pragma unroll
        for (int p = 0; p < PERV; ++p) {
            const int e = p * THREADS + tid, tt = e / CT, c = e - tt * CT;
            pv[p] = (tt < n && tile * CT + c < dv) ? vs[(size_t)(c0 + tt) * a.row_stride + c] : from_f32<T>(0.f);
        }
        if (KIND == 1 && warp == 0 && lane < n) {
            pi = raw_gate(a, c0 + lane, head);
            pf = raw_gate(a, c0 + lane, H + head);
        }
    };
    fetch(t0);

    for (int c0 = t0; c0 < t1; c0 += CH) {
        const int n = min(CH, t1 - c0);
        __syncthreads();      // the tokens before are done with the staged rows
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int e = p * THREADS + tid, tt = e / DP, i = e - tt * DP;
            sq[tt][i] = to_f32<T>(pq[p]) * a.qscale;
            sk[tt][i] = to_f32<T>(pk[p]);
            if (KIND == 0) sd[tt][i] = i < dk ? expf(log_decay(a, pd[p], head * dk + i)) : 0.f;
        }
#pragma unroll
        for (int p = 0; p < PERV; ++p) {
            const int e = p * THREADS + tid, tt = e / CT, c = e - tt * CT;
            sv[tt][c] = to_f32<T>(pv[p]);
        }
        if (KIND == 1 && warp == 0) {
            const float gi = lane < n ? soft_cap(pi, a.cap) : 0.f;
            const float gf = lane < n ? log_sigmoid(soft_cap(pf, a.cap)) : 0.f;
            float before = 0.f, after = 0.f;
            for (int tt = 0; tt < n; ++tt) {
                const float next = fmaxf(__shfl_sync(0xffffffffu, gf, tt) + m, __shfl_sync(0xffffffffu, gi, tt));
                if (lane == tt) { before = m; after = next; }
                m = next;
            }
            if (lane < n) {
                keep[lane] = expf((gf + before) - after);
                put[lane] = expf(gi - after);
                least[lane] = expf(-after);
            }
        }
        __syncthreads();
        if (c0 + CH < t1) fetch(c0 + CH);
        float* o_at = a.o + ((size_t)c0 * H + head) * dv + col;
        const bool store = col_ok && r == 0;
        const float (*dd)[DP] = KIND == 0 ? sd : sk;
        int tt = 0;
        if (!FEW)
            for (; tt + 4 <= n; tt += 4) scan_tokens<G, KIND, 4>(S, sq, sk, dd, sv, keep, put, tt, r, cw, store, o_at, (size_t)H * dv);
        for (; tt < n; ++tt) scan_tokens<G, KIND, 1>(S, sq, sk, dd, sv, keep, put, tt, r, cw, store, o_at, (size_t)H * dv);
        if (owns_n) {
            for (tt = 0; tt < n; ++tt) {
                float dot = 0.f;
#pragma unroll
                for (int x = 0; x < NR; ++x) {
                    const int i = lane + 32 * x;
                    if (i < DP) {
                        nn[x] = fmaf(keep[tt], nn[x], put[tt] * sk[tt][i]);
                        dot = fmaf(nn[x], sq[tt][i], dot);
                    }
                }
                dot = warp_sum(dot);
                if (lane == 0) a.den[(size_t)(c0 + tt) * H + head] = fmaxf(fabsf(dot), least[tt]) + 1e-6f;
            }
        }
    }
    if (col_ok) {
#pragma unroll
        for (int g = 0; g < G; ++g)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = 16 * g + 4 * r + e;
                if (i < dk) Sg[(size_t)i * dv + col] = S[4 * g + e];
            }
    }
    if (KIND == 1 && warp == 0) {
        if (lane < CT / 16 && tile * (CT / 16) + lane < MB - 1) mg[tile * (CT / 16) + lane] = m;
        if (owns_n) {
            if (lane == 0) mg[MB - 1] = m;
#pragma unroll
            for (int x = 0; x < NR; ++x)
                if (lane + 32 * x < dk) ng[lane + 32 * x] = nn[x];
        }
    }
}

// ---------------------------------------------------------------------------
// Blocks of 16 tokens on the tensor cores (bfloat16 activations, fp32 accumulators).  With B_i the sum of the block's log
// decays up to token i (kind 0; per channel) and the state S before the block:
//     o_i = S^T (exp(B_i) q_i) + sum_(j <= i) A_ij v_j,     A_ij = sum_d q_i k_j exp(B_i - B_j)
//     S'  = diag(exp(B_n)) S + sum_j (exp(B_n - B_j) k_j) v_j^T
// Kind 1: with b_i the sum of the log forget gates, g_j = i_j - b_j and G_i = max_(j <= i) g_j, the same with
// A_ij = (q_i . k_j) exp(g_j - G_i) and keys exp(g_j - G_n) k_j, all relative to the block's own maxima; with the m before
// the block and M_i = max(m, G_i) the first term gets exp(m - M_i), the second exp(G_i - M_i), and m_i = b_i + M_i.
//
// state_prepare_kernel, parallel over (block, head), leaves a record of MMA operands in the order in which a warp's lanes
// take them (one 16-byte vector per lane, "fragment"); operands that are not bf16 numbers enter as a rounded value and a
// rounded remainder (16 bits of mantissa).  state_blocks_kernel walks an entry's blocks: a warp holds S^T for 16 value
// columns as accumulators, which are in the layout of the next product's left operand, so the state never leaves its
// registers.  Several warps share a tile, each with some of the channels; they hand their shares of a block's outputs over
// through shared memory, and the first one writes the sum while the next block runs.  For kind 1 one more tile carries n
// as the row of a value column of ones.
// ---------------------------------------------------------------------------
constexpr int SB = 16;      // tokens of a block

__device__ __forceinline__ void sb_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t sb_pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// (x0, x1) = hi + lo, each a pair of bf16 numbers
__device__ __forceinline__ void sb_split(float x0, float x1, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x0, x1);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = sb_pack(x0 - __low2float(h), x1 - __high2float(h));
}

// A record's fragments (of 32 16-byte vectors): scaled queries [KS][2], scaled keys [2 KS], scores [2], scalars [1], values [DT]
__host__ __device__ constexpr int rec_keys(int KS) { return 2 * KS; }
__host__ __device__ constexpr int rec_scores(int KS) { return 4 * KS; }
__host__ __device__ constexpr int rec_scalars(int KS) { return 4 * KS + 2; }
__host__ __device__ constexpr int rec_values(int KS) { return 4 * KS + 3; }

// blocks of an entry that runs in blocks
__device__ __forceinline__ int entry_blocks(const int* cu, int s, int n_seqs, int min_len) {
    if (s >= n_seqs) return 0;
    const int len = cu[s + 1] - cu[s];
    return len >= min_len ? (len + SB - 1) / SB : 0;
}

template <int KS, int KIND>
__global__ void __launch_bounds__(128) state_prepare_kernel(StateArgs a, uint4* rec, int min_len, int vec) {
    constexpr int KD = 16 * KS, QP = KD + 8;
    extern __shared__ __align__(16) unsigned char sp_smem[];
    float* sB = reinterpret_cast<float*>(sp_smem);                                              // kind 0: [16][QP] sums of log decays
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sB + (KIND == 0 ? SB * QP : 64));       // [16][QP]
    __nv_bfloat16* sK = sQ + SB * QP;                                                           // [16][QP]
    __nv_bfloat16* sV = sK + SB * QP;                                                           // [16][VP]
    __shared__ int where[2];
    __shared__ float4 half[64];      // the other warp's share of the scores
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int head = blockIdx.y, blk = blockIdx.x, H = a.H, dk = a.dk, dv = a.dv;
    const int DT = (dv + 15) / 16, VP = DT * 16 + 8;
    if (warp == 0) {      // which entry this block belongs to
        if (lane == 0) where[0] = -1;
        __syncwarp();
        int base = 0;
        for (int s0 = 0; s0 < a.n_seqs; s0 += 32) {
            const int nb = entry_blocks(a.cu, s0 + lane, a.n_seqs, min_len);
            int incl = nb;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += up;
            }
            if (blk >= base + incl - nb && blk < base + incl) { where[0] = s0 + lane; where[1] = blk - (base + incl - nb); }
            base += __shfl_sync(0xffffffffu, incl, 31);
            if (blk < base) break;
        }
    }
    __syncthreads();
    if (where[0] < 0) return;
    const int t0 = a.cu[where[0]] + where[1] * SB;
    const int n = min(SB, a.cu[where[0] + 1] - t0);

    const __nv_bfloat16* proj = (const __nv_bfloat16*)a.proj + (size_t)t0 * a.row_stride;
    auto load_rows = [&](__nv_bfloat16* dst, int pitch, int cols, int padded, int col) {      // [16][padded], zero beyond the tokens and columns
        if (vec) {
            const int per = padded / 8;
            for (int e = tid; e < SB * per; e += 128) {
                const int j = e / per, c = (e - j * per) * 8;
                uint4 v = make_uint4(0, 0, 0, 0);
                if (j < n && c < cols) v = *reinterpret_cast<const uint4*>(proj + (size_t)j * a.row_stride + col + c);
                *reinterpret_cast<uint4*>(dst + j * pitch + c) = v;
            }
        } else {
            for (int e = tid; e < SB * padded; e += 128) {
                const int j = e / padded, c = e - j * padded;
                dst[j * pitch + c] = (j < n && c < cols) ? proj[(size_t)j * a.row_stride + col + c] : __float2bfloat16_rn(0.f);
            }
        }
    };
    load_rows(sQ, QP, dk, KD, a.q_col + head * dk);
    load_rows(sK, QP, dk, KD, a.k_col + head * dk);
    load_rows(sV, VP, dv, DT * 16, a.v_col + head * dv);
    float* gb = sB;           // kind 1: b [16], g [16], G [16]
    if (KIND == 0) {
        for (int d = tid; d < KD; d += 128) {
            float x[SB];
#pragma unroll
            for (int j = 0; j < SB; ++j) x[j] = (j < n && d < dk) ? a.z[((size_t)(t0 + j) * H + head) * dk + d] : 0.f;
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < SB; ++j) {
                if (j < n && d < dk) sum += log_decay(a, x[j], head * dk + d);
                sB[j * QP + d] = sum;
            }
        }
    } else if (warp == 0) {
        float f = 0.f, in = 0.f;
        if (lane < n) {
            in = soft_cap(raw_gate(a, t0 + lane, head), a.cap);
            f = log_sigmoid(soft_cap(raw_gate(a, t0 + lane, H + head), a.cap));
        }
#pragma unroll
        for (int o = 1; o < SB; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, f, o);
            if (lane >= o) f += up;
        }
        const float gj = lane < n ? in - f : -INFINITY;
        float top = gj;
#pragma unroll
        for (int o = 1; o < SB; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, top, o);
            if (lane >= o) top = fmaxf(top, up);
        }
        if (lane < SB) { gb[lane] = f; gb[16 + lane] = gj; gb[32 + lane] = top; }
    }
    __syncthreads();

    uint4* out = rec + ((size_t)blk * H + head) * (size_t)(rec_values(KS) + DT) * 32;
    auto q_at = [&](int i, int d) { return __bfloat162float(sQ[i * QP + d]); };
    auto k_at = [&](int j, int d) { return __bfloat162float(sK[j * QP + d]); };
    if (warp == 1) {          // queries: token 8 nt + g, channels 16 ks + 2 t (+ 1) (+ 8)
#pragma unroll
        for (int ks = 0; ks < KS; ++ks)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                const int i = 8 * nt + g, d = 16 * ks + 2 * t;
                uint4 w = make_uint4(0, 0, 0, 0);
                if (KIND == 1) {
                    w.x = *reinterpret_cast<const uint32_t*>(sQ + i * QP + d);
                    w.y = *reinterpret_cast<const uint32_t*>(sQ + i * QP + d + 8);
                } else {
                    float x[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int c = d + (e & 1) + (e >> 1) * 8;
                        x[e] = q_at(i, c) * a.qscale * __expf(sB[i * QP + c]);
                    }
                    sb_split(x[0], x[1], w.x, w.z);
                    sb_split(x[2], x[3], w.y, w.w);
                }
                out[(ks * 2 + nt) * 32 + lane] = w;
            }
    } else if (warp == 2) {   // keys: channel 8 nt + g, tokens 2 t (+ 1) (+ 8)
#pragma unroll
        for (int nt = 0; nt < 2 * KS; ++nt) {
            const int d = 8 * nt + g;
            float x[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = 2 * t + (e & 1) + (e >> 1) * 8;
                const float w = KIND == 0 ? __expf(sB[(SB - 1) * QP + d] - sB[j * QP + d]) : __expf(gb[16 + j] - gb[32 + SB - 1]);
                x[e] = k_at(j, d) * w;
            }
            uint4 w;
            sb_split(x[0], x[1], w.x, w.z);
            sb_split(x[2], x[3], w.y, w.w);
            out[(rec_keys(KS) + nt) * 32 + lane] = w;
        }
    } else if (warp == 3) {   // scalars; values: column 16 vt + g (+ 8), tokens 2 t (+ 1) (+ 8)
        float* sc = reinterpret_cast<float*>(out + rec_scalars(KS) * 32);
        if (KIND == 0) {
            for (int d = lane; d < KD; d += 32) sc[d] = __expf(sB[(SB - 1) * QP + d]);
        } else if (lane < SB) {
            sc[lane] = gb[lane];
            sc[16 + lane] = gb[32 + lane];
        }
        for (int vt = 0; vt < DT; ++vt) {
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int c = 16 * vt + g + (e & 1) * 8, j = 2 * t + (e >> 1) * 8;
                __nv_bfloat162 p;
                p.x = sV[j * VP + c];
                p.y = sV[(j + 1) * VP + c];
                w[e] = *reinterpret_cast<uint32_t*>(&p);
            }
            out[(rec_values(KS) + vt) * 32 + lane] = make_uint4(w[0], w[1], w[2], w[3]);
        }
    }
    // scores A_ij, i the rows: the first and the last warp, each every other 16 channels
    float acc[2][4];
    if (warp == 0 || warp == 3) {
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] = 0.f;
        // Both exponents are taken about half of the block's whole decay in a channel, so neither factor leaves fp32's range
        // unless a channel decays by more than exp(-100) within the block: then every pair is formed by itself.
        bool far = false;
        if (KIND == 0) {
            for (int d = lane; d < KD; d += 32) far = far || sB[(SB - 1) * QP + d] < -100.f;
            far = __any_sync(0xffffffffu, far);
        }
        if (!far) {
#pragma unroll 1
            for (int ks = warp == 0 ? 0 : 1; ks < KS; ks += 2) {
                const int d = 16 * ks + 2 * t;
                uint32_t ah[4], al[4];
                float mid[4];
                if (KIND == 0) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) mid[e] = 0.5f * sB[(SB - 1) * QP + d + (e & 1) + (e >> 1) * 8];
                }
#pragma unroll
                for (int q = 0; q < 4; ++q) {      // rows g, g + 8; channels d, d + 8
                    const int i = g + (q & 1) * 8, c = d + (q >> 1) * 8;
                    if (KIND == 1) {
                        ah[q] = *reinterpret_cast<const uint32_t*>(sQ + i * QP + c);
                        al[q] = 0;
                    } else {
                        const float m0 = mid[(q >> 1) * 2], m1 = mid[(q >> 1) * 2 + 1];
                        sb_split(q_at(i, c) * a.qscale * __expf(sB[i * QP + c] - m0), q_at(i, c + 1) * a.qscale * __expf(sB[i * QP + c + 1] - m1), ah[q], al[q]);
                    }
                }
#pragma unroll
                for (int nt = 0; nt < 2; ++nt) {   // tokens j = 8 nt + g
                    const int j = 8 * nt + g;
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        const int c = d + q * 8;
                        if (KIND == 1) {
                            bh[q] = *reinterpret_cast<const uint32_t*>(sK + j * QP + c);
                            bl[q] = 0;
                        } else {
                            sb_split(k_at(j, c) * __expf(mid[2 * q] - sB[j * QP + c]), k_at(j, c + 1) * __expf(mid[2 * q + 1] - sB[j * QP + c + 1]), bh[q], bl[q]);
                        }
                    }
                    sb_mma(acc[nt], ah[0], ah[1], ah[2], ah[3], bh[0], bh[1]);
                    if (KIND == 0) {
                        sb_mma(acc[nt], ah[0], ah[1], ah[2], ah[3], bl[0], bl[1]);
                        sb_mma(acc[nt], al[0], al[1], al[2], al[3], bh[0], bh[1]);
                    }
                }
            }
        } else if (warp == 0) {
#pragma unroll 1
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll 1
                for (int e = 0; e < 4; ++e) {
                    const int i = g + (e >> 1) * 8, j = 8 * nt + 2 * t + (e & 1);
                    float sum = 0.f;
                    if (j <= i)
                        for (int d = 0; d < dk; ++d) sum = fmaf(q_at(i, d) * a.qscale * k_at(j, d), __expf(sB[i * QP + d] - sB[j * QP + d]), sum);
                    if (nt == 0) { if (e == 0) acc[0][0] = sum; else if (e == 1) acc[0][1] = sum; else if (e == 2) acc[0][2] = sum; else acc[0][3] = sum; }
                    else { if (e == 0) acc[1][0] = sum; else if (e == 1) acc[1][1] = sum; else if (e == 2) acc[1][2] = sum; else acc[1][3] = sum; }
                }
        }
        if (warp == 3) {
            half[lane] = make_float4(acc[0][0], acc[0][1], acc[0][2], acc[0][3]);
            half[32 + lane] = make_float4(acc[1][0], acc[1][1], acc[1][2], acc[1][3]);
        }
    }
    __syncthreads();
    if (warp == 0) {
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            const float4 h = half[32 * nt + lane];
            acc[nt][0] += h.x; acc[nt][1] += h.y; acc[nt][2] += h.z; acc[nt][3] += h.w;
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = g + (e >> 1) * 8, j = 8 * nt + 2 * t + (e & 1);
                float x = j <= i ? acc[nt][e] : 0.f;
                if (KIND == 1) x = j <= i ? x * a.qscale * __expf(gb[16 + j] - gb[32 + i]) : 0.f;
                acc[nt][e] = x;
            }
        // as the right operand of (values^T A^T): tokens j in pairs, column i = 8 nt + g
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            uint4 w;
            sb_split(acc[0][2 * nt], acc[0][2 * nt + 1], w.x, w.z);
            sb_split(acc[1][2 * nt], acc[1][2 * nt + 1], w.y, w.w);
            out[(rec_scores(KS) + nt) * 32 + lane] = w;
        }
    }
}

constexpr int SB_STAGES = 4;      // blocks on their way from memory
// warps that share a tile of 16 value columns, each with 32 of its channels
__host__ __device__ constexpr int tile_warps(int KS) { return KS / 2; }
__host__ __device__ constexpr int stage_vecs(int KS) { return (rec_values(KS) + 1) * 32; }

// grid (tiles of 16 value columns and, for kind 1, one for n; heads; entries)
template <int KS, int KIND>
__global__ void __launch_bounds__(32 * tile_warps(KS)) state_blocks_kernel(StateArgs a, const uint4* rec, int min_len) {
    constexpr int NW = tile_warps(KS), KH = KS / NW, THREADS = 32 * NW, COMMON = rec_values(KS) * 32, STAGE = stage_vecs(KS);
    static_assert(KS % 2 == 0 && KS % NW == 0, "a tile's warps share its channels evenly");
    extern __shared__ __align__(16) uint4 sb_smem[];               // [stages][STAGE], then [2][NW - 1][2][32] float4
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int tile = blockIdx.x, head = blockIdx.y, b = blockIdx.z, H = a.H, dk = a.dk, dv = a.dv, DT = (dv + 15) / 16;
    const int nb = entry_blocks(a.cu, b, a.n_seqs, min_len);
    if (nb == 0) return;
    int base = 0;             // the entry's first block among all
    for (int s = lane; s < b; s += 32) base += entry_blocks(a.cu, s, a.n_seqs, min_len);
    base = __reduce_add_sync(0xffffffffu, base);
    const int t0 = a.cu[b], t1 = a.cu[b + 1];
    const bool is_n = KIND == 1 && tile == DT;
    float4* other = reinterpret_cast<float4*>(sb_smem + SB_STAGES * STAGE);      // the other warps' shares of a block's outputs

    // a thread copies the vectors tid, tid + THREADS, ... of a record; the next block's record lies rec_step further on
    const size_t rec_step = (size_t)(rec_values(KS) + DT) * 32 * H;
    const uint4* src = rec + (size_t)base * rec_step + (size_t)head * ((rec_values(KS) + DT) * 32) + tid;
    const uint32_t dst0 = (uint32_t)__cvta_generic_to_shared(sb_smem + tid);
    int to_load = 0;
    auto load = [&]() {
        if (to_load < nb) {
            const uint32_t dst = dst0 + (uint32_t)(to_load % SB_STAGES) * (STAGE * 16);
#pragma unroll
            for (int x = 0; x < (COMMON + THREADS - 1) / THREADS; ++x)
                if ((x + 1) * THREADS <= COMMON || tid < COMMON - x * THREADS)
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst + x * THREADS * 16), "l"(src + x * THREADS) : "memory");
            if (warp == NW - 1 && !is_n)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst + (COMMON - 32 * (NW - 1)) * 16), "l"(src + COMMON - 32 * (NW - 1) + 32 * tile) : "memory");
            src += rec_step;
            ++to_load;
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
#pragma unroll
    for (int s = 0; s < SB_STAGES - 1; ++s) load();

    float* slot = a.state + (size_t)a.slots[b] * a.slot_stride;
    float* Sg = slot + (size_t)head * dk * dv;
    float* ng = slot + (size_t)H * dk * dv + (size_t)head * dk;
    const int MB = m_copies(dv);
    float* mg = slot + (size_t)H * dk * dv + (size_t)H * dk + (size_t)head * MB + (is_n ? MB - 1 : tile);
    float S[2 * KH][4];       // S^T: row 16 tile + g (+ 8), channel 16 KH warp + 8 nt + 2 t (+ 1)
    auto state_at = [&](int nt, int e) -> float* {
        const int d = 16 * KH * warp + 8 * nt + 2 * t + (e & 1), c = 16 * tile + g + (e >> 1) * 8;
        if (d >= dk) return nullptr;
        if (is_n) return (g == 0 && e < 2) ? ng + d : nullptr;
        return c < dv ? Sg + (size_t)d * dv + c : nullptr;
    };
#pragma unroll
    for (int nt = 0; nt < 2 * KH; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float* p = state_at(nt, e);
            S[nt][e] = p ? *p : 0.f;
        }
    float m = KIND == 1 ? *mg : 0.f;
    uint4 v = make_uint4(g == 0 ? 0x3f803f80u : 0u, 0u, g == 0 ? 0x3f803f80u : 0u, 0u);      // a value column of ones (n)

    float mine[2][4], m_at[2][2];      // the first warp's share of the block before and that block's maxima
    const bool col0 = 16 * tile + g < dv, col1 = 16 * tile + g + 8 < dv;
    const size_t row = (size_t)H * dv;
    float* o_at = a.o + ((size_t)(t0 + 2 * t) * H + head) * dv + 16 * tile + g;      // this lane's first token of the next block to write
    auto put_out = [&](int blk) {      // row (value column) 16 tile + g (+ 8), tokens 8 nt + 2 t (+ 1)
        const float4* from = other + (blk & 1) * (NW - 1) * 64 + lane;
        const int left = t1 - (t0 + blk * SB + 2 * t);      // the lane's tokens that are there: 8 nt + e < left
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            float o[4] = {mine[nt][0], mine[nt][1], mine[nt][2], mine[nt][3]};
#pragma unroll
            for (int p = 0; p < NW - 1; ++p) {
                const float4 x = from[64 * p + 32 * nt];
                o[0] += x.x; o[1] += x.y; o[2] += x.z; o[3] += x.w;
            }
            if (KIND == 1 && is_n) {
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    if (g == 0 && 8 * nt + e < left)
                        a.den[(size_t)(t0 + blk * SB + 2 * t + 8 * nt + e) * H + head] = fmaxf(fabsf(o[e]), expf(-m_at[nt][e])) + 1e-6f;
            } else {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float* at = o_at + (8 * nt + e) * row;
                    if (col0 && 8 * nt + e < left) at[0] = o[e];
                    if (col1 && 8 * nt + e < left) at[8] = o[2 + e];
                }
            }
        }
        o_at += SB * row;
    };

    for (int blk = 0; blk <= nb; ++blk) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(SB_STAGES - 2) : "memory");
        __syncthreads();      // this block's record and the other warps' shares of the one before are here
        load();
        if (warp == 0 && blk > 0) put_out(blk - 1);
        if (blk == nb) break;
        const uint4* st = sb_smem + (blk % SB_STAGES) * STAGE + lane;
        const float* sc = reinterpret_cast<const float*>(sb_smem + (blk % SB_STAGES) * STAGE + rec_scalars(KS) * 32);
        if (!is_n) v = st[COMMON];
        // an MMA's result takes tens of cycles and few warps share a scheduler: the rounded values' products and the remainders'
        // have accumulators of their own
        float oi[3][2][4], oa[2][4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) oi[0][nt][e] = oi[1][nt][e] = oi[2][nt][e] = oa[nt][e] = 0.f;
        if (warp == NW - 1) {      // the last warp has the block's own tokens
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                const uint4 w = st[(rec_scores(KS) + nt) * 32];
                sb_mma(oa[nt], v.x, v.y, v.z, v.w, w.x, w.y);
                sb_mma(oa[nt], v.x, v.y, v.z, v.w, w.z, w.w);
            }
        }
        const uint4* qs = st + warp * (KH * 2 * 32);
#pragma unroll
        for (int ks = 0; ks < KH; ++ks) {
            uint32_t h[4], l[4];
            sb_split(S[2 * ks][0], S[2 * ks][1], h[0], l[0]);
            sb_split(S[2 * ks][2], S[2 * ks][3], h[1], l[1]);
            sb_split(S[2 * ks + 1][0], S[2 * ks + 1][1], h[2], l[2]);
            sb_split(S[2 * ks + 1][2], S[2 * ks + 1][3], h[3], l[3]);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                const uint4 w = qs[(ks * 2 + nt) * 32];
                sb_mma(oi[0][nt], h[0], h[1], h[2], h[3], w.x, w.y);
                sb_mma(oi[1][nt], l[0], l[1], l[2], l[3], w.x, w.y);
                if (KIND == 0) sb_mma(oi[2][nt], h[0], h[1], h[2], h[3], w.z, w.w);
            }
        }
        // the state after the block
        float c1 = 1.f, c2 = 1.f;
        const float m_before = m;
        if (KIND == 1) {
            const float G = sc[16 + SB - 1], M = fmaxf(m, G);
            c1 = __expf(m - M);
            c2 = __expf(G - M);
            m = sc[SB - 1] + M;
        }
        const uint4* kts = st + (rec_keys(KS) + warp * 2 * KH) * 32;
        const float* dec = sc + 16 * KH * warp + 2 * t;
#pragma unroll
        for (int nt = 0; nt < 2 * KH; ++nt) {
            const uint4 w = kts[nt * 32];
            float u[4] = {0.f, 0.f, 0.f, 0.f};
            sb_mma(u, v.x, v.y, v.z, v.w, w.x, w.y);
            sb_mma(u, v.x, v.y, v.z, v.w, w.z, w.w);
            float d0 = c1, d1 = c1;
            if (KIND == 0) {
                const float2 d = *reinterpret_cast<const float2*>(dec + 8 * nt);
                d0 = d.x;
                d1 = d.y;
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) S[nt][e] = fmaf(e & 1 ? d1 : d0, S[nt][e], KIND == 1 ? c2 * u[e] : u[e]);
        }
        // this warp's share of the block's outputs
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            float fi[2] = {1.f, 1.f}, fa[2] = {1.f, 1.f};
            if (KIND == 1) {
                const float2 G = *reinterpret_cast<const float2*>(sc + 16 + 8 * nt + 2 * t), B = *reinterpret_cast<const float2*>(sc + 8 * nt + 2 * t);
                const float M0 = fmaxf(m_before, G.x), M1 = fmaxf(m_before, G.y);
                fi[0] = __expf(m_before - M0) * a.qscale;
                fi[1] = __expf(m_before - M1) * a.qscale;
                fa[0] = __expf(G.x - M0);
                fa[1] = __expf(G.y - M1);
                m_at[nt][0] = B.x + M0;
                m_at[nt][1] = B.y + M1;
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float x = oi[0][nt][e] + oi[1][nt][e];
                if (KIND == 0) x += oi[2][nt][e];
                if (KIND == 1) x *= fi[e & 1];
                if (warp == NW - 1) x = KIND == 1 ? fmaf(fa[e & 1], oa[nt][e], x) : x + oa[nt][e];
                mine[nt][e] = x;
            }
            if (NW > 1 && warp > 0) other[((blk & 1) * (NW - 1) + warp - 1) * 64 + 32 * nt + lane] = make_float4(mine[nt][0], mine[nt][1], mine[nt][2], mine[nt][3]);
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
#pragma unroll
    for (int nt = 0; nt < 2 * KH; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            float* p = state_at(nt, e);
            if (p) *p = S[nt][e];
        }
    if (KIND == 1 && tid == 0) *mg = m;
}

// ---------------------------------------------------------------------------
// out[t, h dv + j] = T( post * (u_j / sqrt(mean_j(u^2) + eps)) * w * act(gate) ) with u = o[t, h] / den[t, h] (den null: u = o):
// a unit norm over each head's fp32 values, a gain (one per value column of all heads, or shared by the heads: w_period
// = H dv or dv), a gate from the token's projection row (act 0 none, 1 silu, 2 sigmoid).  GS lanes per (token, head).
// ---------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(128) heads_finish_kernel(const float* o, const float* den, const float* w, int w_period, const T* proj,
                                                           long long row_stride, int g_col, int act, float post, T* out, long long out_stride,
                                                           long long n_rows, int H, int dv, int GS, float eps) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & (GS - 1);
    const long long row = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / GS;
    const bool real = row < n_rows;
    const long long rr = real ? row : 0;
    const size_t t = (size_t)(rr / H);
    const int head = (int)(rr - (long long)t * H);
    const float* src = o + (size_t)rr * dv;
    const float d = den ? den[rr] : 1.f;
    float ss = 0.f;
    for (int j = lane * VEC; j < dv; j += GS * VEC) {
        const Vec<float, VEC> x = load_vec<float, VEC>(src + j);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float u = den ? x.v[k] / d : x.v[k];
            ss = fmaf(u, u, ss);
        }
    }
    for (int m = GS >> 1; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    if (!real) return;
    const float rstd = 1.0f / sqrtf(ss / (float)dv + eps);
    const float* wr = w + ((long long)head * dv) % w_period;
    const T* gr = act ? proj + t * row_stride + g_col + (size_t)head * dv : nullptr;
    T* dst = out + t * out_stride + (size_t)head * dv;
    for (int j = lane * VEC; j < dv; j += GS * VEC) {
        const Vec<float, VEC> x = load_vec<float, VEC>(src + j), g = load_vec<float, VEC>(wr + j);
        Vec<T, VEC> z, y;
        if (act) z = load_vec<T, VEC>(gr + j);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            float v = __fmul_rn(__fmul_rn(den ? x.v[k] / d : x.v[k], rstd), g.v[k]);
            if (act) {
                const float s = to_f32<T>(z.v[k]), sig = 1.0f / (1.0f + expf(-s));
                v = __fmul_rn(v, act == 1 ? s * sig : sig);
            }
            y.v[k] = from_f32<T>(v * post);
        }
        store_vec<T, VEC>(dst + j, y);
    }
}

StateArgs state_args(const void* proj, long long row_stride, int q_col, int k_col, int v_col, float qscale, const float* z,
                     const float* z_bias, float tau, const float* gates, int n_parts, long long part_stride, const float* gate_bias, float cap, float* state,
                     long long slot_stride, const int* slots, const int* cu, float* o, float* den, int n_seqs, int H, int dk, int dv) {
    StateArgs a;
    a.proj = proj; a.row_stride = row_stride; a.q_col = q_col; a.k_col = k_col; a.v_col = v_col; a.qscale = qscale; a.z = z; a.z_bias = z_bias; a.inv_tau = 1.0f / tau;
    a.gates = gates; a.n_parts = n_parts; a.part_stride = part_stride; a.gate_bias = gate_bias; a.cap = cap; a.state = state;
    a.slot_stride = slot_stride; a.slots = slots; a.cu = cu; a.o = o; a.den = den; a.n_seqs = n_seqs; a.H = H; a.dk = dk; a.dv = dv;
    return a;
}

int check_state(const StateArgs& a, int kind) {
    if (a.H <= 0 || a.dk <= 0 || a.dv <= 0 || !a.proj || !a.state || !a.slots || !a.cu || !a.o || a.q_col < 0 || a.k_col < 0 || a.v_col < 0) return PYRE_ERR_BAD_ARG;
    if (kind == 0 && (!a.z || !a.z_bias || !(a.inv_tau > 0.f))) return PYRE_ERR_BAD_ARG;
    if (kind == 1 && (!a.gates || a.n_parts < 1 || !a.gate_bias || !(a.cap > 0.f) || !a.den)) return PYRE_ERR_BAD_ARG;
    if (kind != 0 && kind != 1) return PYRE_ERR_BAD_ARG;
    const long long need = (long long)a.H * a.dk * a.dv + (kind == 1 ? (long long)a.H * (a.dk + (a.dv + 15) / 16 + 1) : 0);
    if (need > a.slot_stride) return PYRE_ERR_BAD_ARG;
    if (a.H > 65535 || a.n_seqs > 65535) return PYRE_ERR_UNSUPPORTED;
    return 0;
}

template <typename T, int G>
void launch_scan(const StateArgs& a, int kind, int max_len, bool few, cudaStream_t stream) {
    const dim3 grid(ceil_div(a.dv, ScanShape<G, false>::CT), a.H, a.n_seqs), block(ScanShape<G, false>::THREADS);
    if (kind == 0 && few) pyre_launch(state_scan_kernel<T, G, 0, true>, grid, block, 0, stream, a, max_len);
    else if (kind == 0) pyre_launch(state_scan_kernel<T, G, 0, false>, grid, block, 0, stream, a, max_len);
    else if (few) pyre_launch(state_scan_kernel<T, G, 1, true>, grid, block, 0, stream, a, max_len);
    else pyre_launch(state_scan_kernel<T, G, 1, false>, grid, block, 0, stream, a, max_len);
}

template <int KS, int KIND>
int launch_chunked(const StateArgs& a, uint4* rec, int min_len, int n_blocks, int vec, cudaStream_t stream) {
    constexpr int KD = 16 * KS, QP = KD + 8;
    const int DT = ceil_div(a.dv, 16), tiles = DT + (KIND == 1 ? 1 : 0);
    const size_t smem_p = (size_t)(KIND == 0 ? SB * QP : 64) * 4 + (size_t)SB * (2 * QP + DT * 16 + 8) * 2;
    const size_t smem_b = ((size_t)SB_STAGES * stage_vecs(KS) + (size_t)2 * (tile_warps(KS) - 1) * 64) * 16;
    if (smem_p > 227 * 1024 || smem_b > 227 * 1024) return PYRE_ERR_UNSUPPORTED;
    static size_t have_p[PYRE_MAX_DEVICES] = {}, have_b[PYRE_MAX_DEVICES] = {};
    const int dev = pyre_current_device();
    if (have_p[dev] < smem_p) {
        const cudaError_t e = cudaFuncSetAttribute(state_prepare_kernel<KS, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
        if (e != cudaSuccess) return (int)e;
        have_p[dev] = smem_p;
    }
    if (have_b[dev] < smem_b) {
        const cudaError_t e = cudaFuncSetAttribute(state_blocks_kernel<KS, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_b);
        if (e != cudaSuccess) return (int)e;
        have_b[dev] = smem_b;
    }
    pyre_launch(state_prepare_kernel<KS, KIND>, dim3(n_blocks, a.H), dim3(128), smem_p, stream, a, rec, min_len, vec);
    PYRE_LAUNCH_CHECK();
    pyre_launch(state_blocks_kernel<KS, KIND>, dim3(tiles, a.H, a.n_seqs), dim3(32 * tile_warps(KS)), smem_b, stream, a, (const uint4*)rec, min_len);
    PYRE_LAUNCH_CHECK();
    return 0;
}

}  // namespace

// The entries of at most max_len tokens (0: all of them), token by token.
PYRE_API int pyre_state_scan(const void* proj, long long row_stride, int q_col, int k_col, int v_col, float qscale, const float* z,
                             const float* z_bias, float tau, const float* gates, int n_parts, long long part_stride, const float* gate_bias, float cap, float* state,
                             long long slot_stride, const int* slots, const int* cu_seqlens, float* o, float* den, int n_tokens,
                             int n_seqs, int H, int dk, int dv, int max_len, int kind, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    const StateArgs a = state_args(proj, row_stride, q_col, k_col, v_col, qscale, z, z_bias, tau, gates, n_parts, part_stride, gate_bias, cap,
                                   state, slot_stride, slots, cu_seqlens, o, den, n_seqs, H, dk, dv);
    const int rc = check_state(a, kind);
    if (rc) return rc;
    if (dk > 256) return PYRE_ERR_UNSUPPORTED;
    const bool few = n_tokens <= 2 * n_seqs;      // (nearly) all entries bring one token
#define PICK(TT) do { if (dk <= 16) launch_scan<TT, 1>(a, kind, max_len, few, stream); else if (dk <= 32) launch_scan<TT, 2>(a, kind, max_len, few, stream); \
                      else if (dk <= 48) launch_scan<TT, 3>(a, kind, max_len, few, stream); else if (dk <= 64) launch_scan<TT, 4>(a, kind, max_len, few, stream); \
                      else if (dk <= 96) launch_scan<TT, 6>(a, kind, max_len, few, stream); else if (dk <= 128) launch_scan<TT, 8>(a, kind, max_len, few, stream); \
                      else launch_scan<TT, 16>(a, kind, max_len, few, stream); } while (0)
    if (dtype == PYRE_BF16) PICK(__nv_bfloat16);
    else if (dtype == PYRE_F32) PICK(float);
    else return PYRE_ERR_BAD_ARG;
#undef PICK
    PYRE_LAUNCH_CHECK();
    return 0;
}

// Floats of scratch per (block of 16 tokens, head) of pyre_state_chunked; 0: sizes it does not take.
PYRE_API int pyre_state_record_floats(int dk, int dv, int kind) {
    (void)kind;
    if (dk <= 0 || dk > 128 || dv <= 0 || dv > 512) return 0;
    const int KS = dk <= 32 ? 2 : dk <= 64 ? 4 : dk <= 96 ? 6 : 8;
    return (rec_values(KS) + ceil_div(dv, 16)) * 128;
}

// The entries of at least min_len tokens, in blocks of 16 on the tensor cores (bfloat16 activations).  n_blocks: the sum of
// ceil(tokens / 16) over those entries; scratch: n_blocks * H * pyre_state_record_floats floats, 16-byte aligned.
PYRE_API int pyre_state_chunked(const void* proj, long long row_stride, int q_col, int k_col, int v_col, float qscale, const float* z,
                                const float* z_bias, float tau, const float* gates, int n_parts, long long part_stride, const float* gate_bias, float cap, float* state,
                                long long slot_stride, const int* slots, const int* cu_seqlens, float* o, float* den, void* scratch,
                                int n_tokens, int n_seqs, int H, int dk, int dv, int min_len, int n_blocks, int kind, cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0 || n_blocks <= 0) return 0;
    const StateArgs a = state_args(proj, row_stride, q_col, k_col, v_col, qscale, z, z_bias, tau, gates, n_parts, part_stride, gate_bias, cap,
                                   state, slot_stride, slots, cu_seqlens, o, den, n_seqs, H, dk, dv);
    const int rc = check_state(a, kind);
    if (rc) return rc;
    if (min_len < 1 || !scratch || ((uintptr_t)scratch & 15)) return PYRE_ERR_BAD_ARG;
    if (pyre_state_record_floats(dk, dv, kind) == 0) return PYRE_ERR_UNSUPPORTED;
    // rows of 8 elements at a time where everything starts on 16-byte boundaries
    const int vec = row_stride % 8 == 0 && q_col % 8 == 0 && k_col % 8 == 0 && v_col % 8 == 0 && dk % 8 == 0 && dv % 8 == 0 && ((uintptr_t)proj & 15) == 0;
    uint4* rec = (uint4*)scratch;
#define GO(KSV) (kind == 0 ? launch_chunked<KSV, 0>(a, rec, min_len, n_blocks, vec, stream) : launch_chunked<KSV, 1>(a, rec, min_len, n_blocks, vec, stream))
    if (dk <= 32) return GO(2);
    if (dk <= 64) return GO(4);
    if (dk <= 96) return GO(6);
    return GO(8);
#undef GO
}

PYRE_API int pyre_heads_finish(const float* o, const float* den, const float* w, int w_period, const void* proj, long long row_stride,
                               int g_col, int act, float post, void* out, long long out_stride, int n_tokens, int H, int dv, float eps,
                               int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (H <= 0 || dv <= 0 || !o || !w || (w_period != dv && w_period != H * dv) || act < 0 || act > 2 || (act && (!proj || g_col < 0)) ||
        out_stride < (long long)H * dv)
        return PYRE_ERR_BAD_ARG;
    const bool vec = dv % 4 == 0 && out_stride % 4 == 0 && (!act || (row_stride % 4 == 0 && g_col % 4 == 0)) &&
                     (((uintptr_t)o | (uintptr_t)w) & 15) == 0 && (((uintptr_t)proj | (uintptr_t)out) & (dtype == PYRE_BF16 ? 7 : 15)) == 0;
    int GS = 4;
    while (GS < 32 && GS * (vec ? 4 : 1) < dv) GS *= 2;
    const long long n_rows = (long long)n_tokens * H;
    const dim3 grid((unsigned)ceil_div_ll(n_rows * GS, 128));
#define GO(TT, V) pyre_launch(heads_finish_kernel<TT, V>, grid, dim3(128), 0, stream, o, den, w, w_period, (const TT*)proj, row_stride, g_col, act, post, (TT*)out, out_stride, n_rows, H, dv, GS, eps)
    if (dtype == PYRE_BF16) { if (vec) GO(__nv_bfloat16, 4); else GO(__nv_bfloat16, 1); }
    else if (dtype == PYRE_F32) { if (vec) GO(float, 4); else GO(float, 1); }
    else return PYRE_ERR_BAD_ARG;
#undef GO
    PYRE_LAUNCH_CHECK();
    return 0;
}
