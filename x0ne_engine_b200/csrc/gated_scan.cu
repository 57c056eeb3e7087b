// Linear attention whose matrix state is decayed and written through gates, in four kernels and a fallback.  Per sequence
// and head, token by token over the rows the sequence brings, from the state S [D key channels][V value columns]:
//   S[d][c] = w[d] S[d][c] + k[d] v[c];     o[c] = sum_d q[d] S[d][c]
// Two ways of gating share the kernels:
//   channel gates (HGRN2):  f = l + (1 - l) sigmoid(z + b) per channel, w = f, k = 1 - f, q = silu(q_raw)
//   head gates (the matrix memory of xLSTM):  with i = cap tanh((i_raw + b_i) / cap), f = logsigmoid(cap tanh((f_raw + b_f) / cap))
//           and a running maximum m (0 at a sequence's start):  m' = max(f + m, i), w = exp(f + m - m'), k = exp(i - m') k_raw;
//           one more column, written with v = 1, sums the keys (its o is n . q), and exp(-m') is left for the normaliser
//
// The state of a sequence is one float32 array: S transposed, [heads][C columns][D] (C = V, or V + 1 with the key sum as the
// last column), then for head gates [heads][2] running maxima: the maximum after the token at position p lies at p % 2, so
// that the blocks of a one-token step can read the old one while one of them writes the new.  The projections come as
// float32 (one packed product).  Everything here is float32; every sum runs in one order that depends on D alone (a lane's
// channels: even ones and odd ones as two fused multiply-add chains, then the lanes as a shuffle tree), so a token's result
// is the same bits however its sequence is cut into passes, whatever else is in a pass and whichever kernel runs.
#include "common.cuh"

#define GS_CW 4                         // state columns of a warp
#define GS_COLS 16                      // of a block
#define GS_U 8                          // tokens worked on side by side
#define GS_STAGES 3
#define GS_THREADS (GS_COLS / GS_CW * 32)       // working threads of a block

__device__ __forceinline__ float gs_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gs_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float gs_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gs_capped(float z, float cap) { return cap * tanhf(z / cap); }

// two float32 operations per instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 gs_dup(float a) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(a));
    return r;
}
__device__ __forceinline__ f32x2 gs_pack(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void gs_unpack(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 gs_mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 gs_fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

// Channels of a lane: 2 lane, 2 lane + 1 for KI = 2; else groups of four, 128 channels apart (16-byte reads without conflicts).
template <int KI> __device__ __forceinline__ int gs_channel(int lane, int pair) {      // the even channel of the lane's pair
    if (KI == 2) return 2 * lane;
    return (pair >> 1) * 128 + 4 * lane + 2 * (pair & 1);
}
template <int KI> __device__ __forceinline__ void gs_load_pairs(f32x2 (&r)[KI / 2], const float* row, int lane) {
    if (KI == 2) {
        r[0] = *reinterpret_cast<const f32x2*>(row + 2 * lane);
    } else {
#pragma unroll
        for (int g = 0; g < KI / 4; ++g) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + g * 128 + 4 * lane);
            r[2 * g] = x.x;
            r[2 * g + 1] = x.y;
        }
    }
}

// One token: the state's step and this lane's share of the results.
template <int KI, int CW>
__device__ __forceinline__ void gs_step(f32x2 (&S)[KI / 2][CW], const f32x2 (&q)[KI / 2], const f32x2 (&k)[KI / 2], const f32x2 (&w)[KI / 2],
                                        const f32x2 (&v)[CW], float* acc) {
#pragma unroll
    for (int c = 0; c < CW; ++c) {
        f32x2 a = 0ull;
#pragma unroll
        for (int p = 0; p < KI / 2; ++p) {
            S[p][c] = gs_fma2(w[p], S[p][c], gs_mul2(k[p], v[c]));
            a = p == 0 ? gs_mul2(q[p], S[p][c]) : gs_fma2(q[p], S[p][c], a);
        }
        float lo, hi;
        gs_unpack(a, lo, hi);
        acc[c] = lo + hi;
    }
}

// Sums N values (a power of two) over the lanes of the warp: at every level the lanes of a pair share the values out.  The
// tree of every value is the same (lanes 16 apart, then 8, 4, 2, 1).  Value x ends up in the lanes whose top log2(N) bits
// are x.
template <int N>
__device__ __forceinline__ float gs_reduce(float (&v)[N], int lane) {
    int left = N;
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) {
        if (left > 1) {
            left >>= 1;
            const bool up = (lane & off) != 0;
#pragma unroll
            for (int i = 0; i < N / 2; ++i)
                if (i < left) {
                    const float mine = up ? v[i + left] : v[i], other = up ? v[i] : v[i + left];
                    v[i] = mine + __shfl_xor_sync(0xffffffffu, other, off);
                }
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
        }
    }
    return v[0];
}

__device__ __forceinline__ void gs_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void gs_cp4(float* dst, const float* src, bool ok) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 4 : 0)
                 : "memory");
}

template <int KI, int CW>
__device__ __forceinline__ void gs_load_state(f32x2 (&S)[KI / 2][CW], const float* st, int col0, int C, int D, int lane) {
#pragma unroll
    for (int c = 0; c < CW; ++c)
#pragma unroll
        for (int p = 0; p < KI / 2; p += (KI == 2 ? 1 : 2)) {
            const int d = gs_channel<KI>(lane, p);
            const float* row = st + (int64_t)(col0 + c) * D + d;
            const bool in = col0 + c < C;
            if (KI > 2 && (D & 3) == 0) {
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if (in && d < D) x = *reinterpret_cast<const float4*>(row);
                S[p][c] = gs_pack(x.x, x.y);
                S[p + (KI > 2)][c] = gs_pack(x.z, x.w);
            } else {
                S[p][c] = gs_pack(in && d < D ? row[0] : 0.f, in && d + 1 < D ? row[1] : 0.f);
                if (KI > 2) S[p + (KI > 2)][c] = gs_pack(in && d + 2 < D ? row[2] : 0.f, in && d + 3 < D ? row[3] : 0.f);
            }
        }
}
template <int KI, int CW>
__device__ __forceinline__ void gs_store_state(const f32x2 (&S)[KI / 2][CW], float* st, int col0, int C, int D, int lane) {
#pragma unroll
    for (int c = 0; c < CW; ++c)
#pragma unroll
        for (int p = 0; p < KI / 2; p += (KI == 2 ? 1 : 2)) {
            const int d = gs_channel<KI>(lane, p);
            float* row = st + (int64_t)(col0 + c) * D + d;
            if (col0 + c >= C) continue;
            float x0, x1, x2 = 0.f, x3 = 0.f;
            gs_unpack(S[p][c], x0, x1);
            if (KI > 2) gs_unpack(S[p + (KI > 2)][c], x2, x3);
            if (KI > 2 && (D & 3) == 0) {
                if (d < D) *reinterpret_cast<float4*>(row) = make_float4(x0, x1, x2, x3);
            } else {
                if (d < D) row[0] = x0;
                if (d + 1 < D) row[1] = x1;
                if (KI > 2 && d + 2 < D) row[2] = x2;
                if (KI > 2 && d + 3 < D) row[3] = x3;
            }
        }
}

// Where a token's inputs lie.  Every pointer is that of row 0, head 0; rows are *_ld values apart, a head's values follow
// the head's before it.
struct GatedScanArgs {
    const float* q;
    const float* k;
    const float* w;         // channel gates: the decays [rows][w_ld]; head gates: null
    const float* v;
    int64_t q_ld, k_ld, w_ld, v_ld;
    const float* gates;     // head gates: [rows][heads][2], decay and write strength; else null
    float* o;               // [rows][heads * V]
    float* nq;              // head gates: [rows][heads], the key sum's result
    float* state;
    int64_t state_stride;
    const int32_t* seq_first_row;
    const int32_t* seq_slot;
    int32_t heads, D, V, C;
};

// ----------------------------------------------------------------------------------------
// Scan over many tokens.  A block takes one sequence, one head and GS_COLS columns of S (columns do not depend on one
// another); a warp keeps CW columns with all their channels spread over its lanes in registers (two columns per warp
// and twice the warps read shared memory twice as often and were slower at every size).  A warp of its own copies the inputs,
// TB tokens at a time, into a ring of GS_STAGES stages of shared memory by cp.async.  GS_U tokens are worked on side by side: only S is carried from one to the next (one fused multiply-add per value), and their results are summed over the
// lanes together, each lane ending up with one (token, column).
// ----------------------------------------------------------------------------------------
template <int KI, bool HEAD_GATES>
__global__ void __launch_bounds__(GS_THREADS + 32) gated_scan_kernel(GatedScanArgs a, int vec) {
    constexpr int CW = GS_CW, WARPS = GS_COLS / CW, THREADS = GS_THREADS + 32;       // the working warps, and the one that copies
    constexpr int NB = 32 * KI;
    constexpr int TB = KI >= 8 ? 8 : 16;
    constexpr int ARR = HEAD_GATES ? 2 : 3;
    constexpr int STAGE = TB * (ARR * NB + GS_COLS + (HEAD_GATES ? 2 : 0));
    extern __shared__ __align__(16) float gs_smem[];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int seq = blockIdx.x, head = blockIdx.y, j0 = blockIdx.z * GS_COLS, col0 = j0 + warp * CW;
    const int D = a.D;
    // channels past the head's last stay zero in every stage: the copies never touch them
    for (int i = tid; i < GS_STAGES * STAGE; i += THREADS) gs_smem[i] = 0.f;
    pdl_wait();
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0) return;
    float* st = a.state + (int64_t)slot * a.state_stride + (int64_t)head * a.C * D;
    const int n_stages = (n_tok + TB - 1) / TB;
    __syncthreads();

    if (warp == WARPS) {
        const int64_t hd0 = (int64_t)head * D, hv0 = (int64_t)head * a.V + j0;
        const float* src[3] = {a.q + row0 * a.q_ld + hd0, a.k + row0 * a.k_ld + hd0, HEAD_GATES ? nullptr : a.w + row0 * a.w_ld + hd0};
        const int64_t ld[3] = {a.q_ld, a.k_ld, a.w_ld};
        auto fetch = [&](int stage) {
            if (stage < n_stages) {
                float* base = gs_smem + (stage % GS_STAGES) * STAGE;
                const int t0 = stage * TB, nt = min(TB, n_tok - t0);
#pragma unroll
                for (int r = 0; r < ARR; ++r) {
                    const float* p = src[r] + t0 * ld[r];
                    float* dst = base + r * TB * NB;
                    if (vec) {
#pragma unroll 4
                        for (int t = 0; t < nt; ++t, p += ld[r], dst += NB)
#pragma unroll
                            for (int c = 4 * lane; c < NB; c += 128)
                                if (c < D) gs_cp16(dst + c, p + c);
                    } else {
                        for (int t = 0; t < nt; ++t, p += ld[r], dst += NB)
                            for (int c = lane; c < D; c += 32) gs_cp4(dst + c, p + c, true);
                    }
                }
                float* vb = base + ARR * TB * NB;
                const float* pv = a.v + (row0 + t0) * a.v_ld + hv0;
#pragma unroll
                for (int x = 0; x < TB * GS_COLS / 32; ++x) {
                    const int e = lane + x * 32, t = e / GS_COLS, c = e % GS_COLS;
                    const bool ok = t < nt && j0 + c < a.V;
                    gs_cp4(vb + e, ok ? pv + t * a.v_ld + c : a.v, ok);
                }
                if (HEAD_GATES && lane < 2 * TB) {
                    const int t = lane >> 1;
                    const bool ok = t < nt;
                    gs_cp4(vb + TB * GS_COLS + lane, ok ? a.gates + ((int64_t)(row0 + t0 + t) * a.heads + head) * 2 + (lane & 1) : a.gates, ok);
                }
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
#pragma unroll
        for (int s = 0; s < GS_STAGES - 1; ++s) fetch(s);
        for (int s = 0; s < n_stages; ++s) {
            asm volatile("cp.async.wait_group %0;" ::"n"(GS_STAGES - 2) : "memory");
            __syncthreads();                // stage s has arrived, and the working warps are done with stage s - 1
            fetch(s + GS_STAGES - 1);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        return;
    }

    f32x2 S[KI / 2][CW];
    gs_load_state<KI, CW>(S, st, col0, a.C, D, lane);
    auto token = [&](const float* base, int t, float* acc) {
        f32x2 q[KI / 2], k[KI / 2], w[KI / 2], v[CW];
        gs_load_pairs<KI>(q, base + t * NB, lane);
        gs_load_pairs<KI>(k, base + (TB + t) * NB, lane);
        const float* vb = base + ARR * TB * NB;
        float vv[CW];
#pragma unroll
        for (int c = 0; c < CW; c += 2) {
            const float2 x = *reinterpret_cast<const float2*>(vb + t * GS_COLS + warp * CW + c);
            vv[c] = x.x;
            vv[c + 1] = x.y;
        }
        if (HEAD_GATES) {
            const float2 g = *reinterpret_cast<const float2*>(vb + TB * GS_COLS + 2 * t);
#pragma unroll
            for (int c = 0; c < CW; ++c) {
                if (col0 + c == a.V) vv[c] = 1.0f;          // the key sum's column
                vv[c] *= g.y;
            }
            w[0] = gs_dup(g.x);
#pragma unroll
            for (int p = 1; p < KI / 2; ++p) w[p] = w[0];
        } else {
            gs_load_pairs<KI>(w, base + (2 * TB + t) * NB, lane);
        }
#pragma unroll
        for (int c = 0; c < CW; ++c) v[c] = gs_dup(vv[c]);
        gs_step<KI, CW>(S, q, k, w, v, acc);
    };
    auto put = [&](int t, int c, float x) {
        const int64_t row = row0 + t;
        if (col0 + c < a.V) a.o[row * ((int64_t)a.heads * a.V) + (int64_t)head * a.V + col0 + c] = x;
        else if (HEAD_GATES && col0 + c == a.V) a.nq[row * a.heads + head] = x;
    };

    // after a group of tokens this lane holds the result of token grp_t of the group in column grp_col
    constexpr int SHARE = 32 / (GS_U * CW);
    const int grp_t = lane / SHARE / CW, grp_col = col0 + lane / SHARE % CW;
    const bool grp_sum = HEAD_GATES && grp_col == a.V, grp_live = lane % SHARE == 0 && grp_col < a.C;
    const int64_t grp_ld = grp_sum ? a.heads : (int64_t)a.heads * a.V;
    float* grp_dst = (grp_sum ? a.nq + head : a.o + (int64_t)head * a.V + grp_col) + (row0 + grp_t) * grp_ld;

    for (int s = 0; s < n_stages; ++s) {
        __syncthreads();
        const float* base = gs_smem + (s % GS_STAGES) * STAGE;
        const int t0 = s * TB, nt = min(TB, n_tok - t0);
        if (col0 >= a.C) continue;
        int t = 0;
#pragma unroll 1
        for (; t + GS_U <= nt; t += GS_U) {
            float acc[GS_U * CW];
#pragma unroll
            for (int u = 0; u < GS_U; ++u) token(base, t + u, acc + u * CW);
            const float x = gs_reduce<GS_U * CW>(acc, lane);
            if (grp_live) grp_dst[(t0 + t) * grp_ld] = x;
        }
#pragma unroll 1
        for (; t < nt; ++t) {
            float acc[CW];
            token(base, t, acc);
            const float x = gs_reduce<CW>(acc, lane);
            if (lane % (32 / CW) == 0) put(t0 + t, lane / (32 / CW), x);
        }
    }
    gs_store_state<KI, CW>(S, st, col0, a.C, D, lane);
}

// Any D: S stays in global memory; a thread owns a column.
__global__ void gated_scan_any_kernel(GatedScanArgs a) {
    pdl_prologue();
    const int seq = blockIdx.x, head = blockIdx.y, c = blockIdx.z * blockDim.x + threadIdx.x;
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0 || c >= a.C) return;
    float* S = a.state + (int64_t)slot * a.state_stride + ((int64_t)head * a.C + c) * a.D;
    for (int64_t row = row0; row < row0 + n_tok; ++row) {
        float g = 1.f, b = 1.f;
        if (a.gates != nullptr) {
            g = a.gates[(row * a.heads + head) * 2];
            b = a.gates[(row * a.heads + head) * 2 + 1];
        }
        const float vc = (c < a.V ? a.v[row * a.v_ld + (int64_t)head * a.V + c] : 1.0f) * b;
        float acc = 0.f;
        for (int d = 0; d < a.D; ++d) {
            const int64_t at = (int64_t)head * a.D + d;
            const float w = a.w != nullptr ? a.w[row * a.w_ld + at] : g;
            const float s = fmaf(w, S[d], a.k[row * a.k_ld + at] * vc);
            S[d] = s;
            acc = fmaf(a.q[row * a.q_ld + at], s, acc);
        }
        if (c < a.V) a.o[row * ((int64_t)a.heads * a.V) + (int64_t)head * a.V + c] = acc;
        else a.nq[row * a.heads + head] = acc;
    }
}

// ----------------------------------------------------------------------------------------
// One token per sequence: gates and step in one launch, the state read and written straight from and to memory.
// ----------------------------------------------------------------------------------------
struct GatedRaw {
    const float* src;       // the packed projection, float32 [rows][ld]
    int64_t ld;
    int32_t q_col, k_col, v_col;        // k_col: the keys, or with channel gates the forget gates' projection
    int32_t i_col, f_col;               // head gates
    const float* f_bias;                // [heads * D] (channel gates) or [heads]
    const float* i_bias;                // [heads] (head gates)
    const float* lower;                 // [heads * D] (channel gates)
    float cap;                          // head gates
    int64_t m_off;                      // head gates: place of the running maxima in a state row
    float* em;                          // head gates: [rows][heads], exp(-m) after the token
    const int32_t* seq_pos0;
};

__device__ __forceinline__ void gs_channel_gate(float z, float lower, float& k, float& f) {
    const float e = expf(-fabsf(z)), r = 1.0f / (1.0f + e);
    const float hi = r, lo = e * r;                     // sigmoid(|z|), sigmoid(-|z|): neither loses its small digits
    const float s = z >= 0.f ? hi : lo, c = z >= 0.f ? lo : hi;
    f = fmaf(1.0f - lower, s, lower);
    k = (1.0f - lower) * c;                             // 1 - f
}
// the gates of one head at one token: m is the running maximum before it, and after it on return
__device__ __forceinline__ void gs_head_gate(float i, float f, float& m, float& decay, float& write) {
    const float keep = f + m, mn = fmaxf(keep, i);
    decay = expf(keep - mn);
    write = expf(i - mn);
    m = mn;
}

template <int KI, bool HEAD_GATES>
__global__ void __launch_bounds__(GS_THREADS) gated_step_kernel(GatedScanArgs a, GatedRaw x) {
    pdl_launch_dependents();
    // the block's threads work the gates out once, a channel each, and leave them where every column's lanes read them
    constexpr int CW = GS_CW, NB = 32 * KI, PER = (NB + GS_THREADS - 1) / GS_THREADS;
    __shared__ __align__(16) float qs[NB], ks[NB], ws[HEAD_GATES ? 4 : NB];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * GS_COLS + warp * CW;
    const int D = a.D;
    float low[PER], fb[PER];
    if (!HEAD_GATES) {
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            const int d = tid + e * GS_THREADS;
            low[e] = d < D ? x.lower[(int64_t)head * D + d] : 0.f;
            fb[e] = d < D ? x.f_bias[(int64_t)head * D + d] : 0.f;
        }
    }
    const float hfb = HEAD_GATES ? x.f_bias[head] : 0.f, hib = HEAD_GATES ? x.i_bias[head] : 0.f;
    pdl_wait();
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok != 1) return;
    float* st = a.state + (int64_t)slot * a.state_stride + (int64_t)head * a.C * D;
    f32x2 S[KI / 2][CW];
    gs_load_state<KI, CW>(S, st, col0, a.C, D, lane);
    const float* row = x.src + (int64_t)row0 * x.ld;
    float vv[CW];
#pragma unroll
    for (int c = 0; c < CW; ++c) vv[c] = col0 + c < a.V ? row[x.v_col + (int64_t)head * a.V + col0 + c] : 0.f;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        const int d = tid + e * GS_THREADS;
        if (d >= NB) break;
        float q = 0.f, k = 0.f, f = 0.f;
        if (d < D) {
            q = row[x.q_col + (int64_t)head * D + d];
            k = row[x.k_col + (int64_t)head * D + d];
            if (!HEAD_GATES) {
                q = gs_silu(q);
                gs_channel_gate(k + fb[e], low[e], k, f);
            }
        }
        qs[d] = q;
        ks[d] = k;
        if (!HEAD_GATES) ws[d] = f;
    }
    f32x2 q[KI / 2], k[KI / 2], w[KI / 2], v[CW];
    if (HEAD_GATES) {
        float* mm = a.state + (int64_t)slot * a.state_stride + x.m_off + 2 * head;
        const int pos = x.seq_pos0[seq];
        float m = mm[(pos + 1) & 1], decay, write;
        gs_head_gate(gs_capped(row[x.i_col + head] + hib, x.cap), gs_log_sigmoid(gs_capped(row[x.f_col + head] + hfb, x.cap)), m, decay, write);
        if (blockIdx.z == 0 && tid == 0) {
            mm[pos & 1] = m;
            x.em[(int64_t)row0 * a.heads + head] = expf(-m);
        }
#pragma unroll
        for (int c = 0; c < CW; ++c) vv[c] = (col0 + c == a.V ? 1.0f : vv[c]) * write;
#pragma unroll
        for (int p = 0; p < KI / 2; ++p) w[p] = gs_dup(decay);
    }
    __syncthreads();
    gs_load_pairs<KI>(q, qs, lane);
    gs_load_pairs<KI>(k, ks, lane);
    if (!HEAD_GATES) gs_load_pairs<KI>(w, ws, lane);
#pragma unroll
    for (int c = 0; c < CW; ++c) v[c] = gs_dup(vv[c]);
    float acc[CW];
    gs_step<KI, CW>(S, q, k, w, v, acc);
    gs_store_state<KI, CW>(S, st, col0, a.C, D, lane);
    const float r = gs_reduce<CW>(acc, lane);
    const int c = lane / (32 / CW);
    if (lane % (32 / CW) == 0) {
        if (col0 + c < a.V) a.o[(int64_t)row0 * a.heads * a.V + (int64_t)head * a.V + col0 + c] = r;
        else if (HEAD_GATES && col0 + c == a.V) a.nq[(int64_t)row0 * a.heads + head] = r;
    }
}

// ----------------------------------------------------------------------------------------
// Gates of many tokens, ahead of the scan
// ----------------------------------------------------------------------------------------
// Channel gates: the queries' activation, the write strengths and the decays of every row, [rows][3][heads * D].
__global__ void channel_gates_kernel(GatedRaw x, float* __restrict__ out, int64_t total, int hd) {
    pdl_prologue();
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t row = i / hd;
        const int c = (int)(i - row * hd);
        const float* src = x.src + row * x.ld;
        float k, f;
        gs_channel_gate(src[x.k_col + c] + x.f_bias[c], x.lower[c], k, f);
        float* dst = out + row * 3 * hd + c;
        dst[0] = gs_silu(src[x.q_col + c]);
        dst[hd] = k;
        dst[2 * (int64_t)hd] = f;
    }
}
// the same with 4 channels per thread (hd, ld and columns multiples of 4, 16-byte aligned bases)
__global__ void channel_gates_vec_kernel(GatedRaw x, float* __restrict__ out, int64_t total4, int hd) {
    pdl_prologue();
    const int h4 = hd / 4;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total4; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t row = i / h4;
        const int c = (int)(i - row * h4) * 4;
        const float* src = x.src + row * x.ld;
        const float4 z = *reinterpret_cast<const float4*>(src + x.k_col + c), q = *reinterpret_cast<const float4*>(src + x.q_col + c);
        const float4 b = *reinterpret_cast<const float4*>(x.f_bias + c), l = *reinterpret_cast<const float4*>(x.lower + c);
        float4 k, f;
        gs_channel_gate(z.x + b.x, l.x, k.x, f.x);
        gs_channel_gate(z.y + b.y, l.y, k.y, f.y);
        gs_channel_gate(z.z + b.z, l.z, k.z, f.z);
        gs_channel_gate(z.w + b.w, l.w, k.w, f.w);
        float* dst = out + row * 3 * hd + c;
        *reinterpret_cast<float4*>(dst) = make_float4(gs_silu(q.x), gs_silu(q.y), gs_silu(q.z), gs_silu(q.w));
        *reinterpret_cast<float4*>(dst + hd) = k;
        *reinterpret_cast<float4*>(dst + 2 * (int64_t)hd) = f;
    }
}

// Head gates: a block per (sequence, head).  All threads work out the gates of GS_GATE_TOKENS tokens, one thread walks the
// running maximum through them (an addition and a maximum per token), all threads turn that into decays and write strengths.
#define GS_GATE_TOKENS 1024
__global__ void __launch_bounds__(256) head_gates_kernel(GatedRaw x, float* __restrict__ gates, float* __restrict__ state, int64_t state_stride,
                                                         const int32_t* __restrict__ seq_first_row, const int32_t* __restrict__ seq_slot, int heads) {
    __shared__ __align__(16) float is[GS_GATE_TOKENS + 8], fs[GS_GATE_TOKENS + 8], ms[GS_GATE_TOKENS];     // ms: the maximum before a token
    pdl_launch_dependents();
    const int tid = threadIdx.x, seq = blockIdx.x, head = blockIdx.y;
    const float fb = x.f_bias[head], ib = x.i_bias[head];
    pdl_wait();
    const int slot = seq_slot[seq];
    const int row0 = seq_first_row[seq], n_tok = seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0) return;
    const int pos0 = x.seq_pos0[seq];
    float* mm = state + (int64_t)slot * state_stride + x.m_off + 2 * head;
    float m = tid == 0 ? mm[(pos0 + 1) & 1] : 0.f;
    for (int t0 = 0; t0 < n_tok; t0 += GS_GATE_TOKENS) {
        const int nt = min(GS_GATE_TOKENS, n_tok - t0);
        const int padded = (nt + 7) / 8 * 8;
        float ri[GS_GATE_TOKENS / 256], rf[GS_GATE_TOKENS / 256];
#pragma unroll
        for (int e = 0; e < GS_GATE_TOKENS / 256; ++e) {
            const float* src = x.src + (int64_t)(row0 + t0 + min(tid + 256 * e, nt - 1)) * x.ld;
            ri[e] = src[x.i_col + head];
            rf[e] = src[x.f_col + head];
        }
#pragma unroll
        for (int e = 0; e < GS_GATE_TOKENS / 256; ++e) {
            const int t = tid + 256 * e;
            if (t < padded) {           // (places past the last token leave the maximum as it is)
                is[t] = t < nt ? gs_capped(ri[e] + ib, x.cap) : -INFINITY;
                fs[t] = t < nt ? gs_log_sigmoid(gs_capped(rf[e] + fb, x.cap)) : 0.f;
            }
        }
        __syncthreads();
        if (tid == 0) {
            // eight tokens at a time, the next eight on their way: a token costs an addition and a maximum, no read to wait for
            float4 f0 = *reinterpret_cast<float4*>(fs), f1 = *reinterpret_cast<float4*>(fs + 4);
            float4 i0 = *reinterpret_cast<float4*>(is), i1 = *reinterpret_cast<float4*>(is + 4);
#pragma unroll 2
            for (int t = 0; t < padded; t += 8) {
                const float4 nf0 = *reinterpret_cast<float4*>(fs + t + 8), nf1 = *reinterpret_cast<float4*>(fs + t + 12);
                const float4 ni0 = *reinterpret_cast<float4*>(is + t + 8), ni1 = *reinterpret_cast<float4*>(is + t + 12);
                float4 b0, b1;
                b0.x = m; m = fmaxf(f0.x + m, i0.x);
                b0.y = m; m = fmaxf(f0.y + m, i0.y);
                b0.z = m; m = fmaxf(f0.z + m, i0.z);
                b0.w = m; m = fmaxf(f0.w + m, i0.w);
                b1.x = m; m = fmaxf(f1.x + m, i1.x);
                b1.y = m; m = fmaxf(f1.y + m, i1.y);
                b1.z = m; m = fmaxf(f1.z + m, i1.z);
                b1.w = m; m = fmaxf(f1.w + m, i1.w);
                *reinterpret_cast<float4*>(ms + t) = b0;
                *reinterpret_cast<float4*>(ms + t + 4) = b1;
                f0 = nf0; f1 = nf1; i0 = ni0; i1 = ni1;
            }
        }
        __syncthreads();
        for (int t = tid; t < nt; t += 256) {
            float before = ms[t], decay, write;
            gs_head_gate(is[t], fs[t], before, decay, write);
            const int64_t at = (int64_t)(row0 + t0 + t) * heads + head;
            *reinterpret_cast<float2*>(gates + 2 * at) = make_float2(decay, write);
            x.em[at] = expf(-before);
        }
        __syncthreads();
    }
    if (tid == 0) mm[(pos0 + n_tok - 1) & 1] = m;
}

// ----------------------------------------------------------------------------------------
// Per-head norm of a scan's results on their way to the output product:
//   y = o                                     or, with head gates (nq, em): y = s o / (max(|s nq|, em) + tiny)
//   out = y / sqrt(mean(y^2) + eps) * weight [* sigmoid(gate)] * post
// weight: V values for all heads (shared), or one per (head, value).  gate: float32 at row * gate_ld + head * V + value.
// out rows are out_ld values apart.  One warp per (row, head).
// ----------------------------------------------------------------------------------------
struct HeadNormArgs {
    const float* o;
    const float* nq;
    const float* em;
    float q_scale, tiny;
    const float* weight;
    int32_t shared;
    const float* gate;
    int64_t gate_ld;
    float eps, post;
    int64_t out_ld;
    int32_t heads, V;
};

template <typename T>
__global__ void scan_head_norm_kernel(HeadNormArgs a, T* __restrict__ out, uint32_t items) {
    pdl_prologue();
    const int lane = threadIdx.x & 31;
    const uint32_t item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const uint32_t row = item / (uint32_t)a.heads, head = item - row * (uint32_t)a.heads;
    const float* src = a.o + (int64_t)item * a.V;
    float f = 1.f;
    if (a.nq != nullptr) f = a.q_scale / (fmaxf(fabsf(a.nq[item] * a.q_scale), a.em[item]) + a.tiny);
    const float* w = a.weight + (a.shared ? 0 : (int64_t)head * a.V);
    const float* g = a.gate != nullptr ? a.gate + (int64_t)row * a.gate_ld + (int64_t)head * a.V : nullptr;
    T* dst = out + (int64_t)row * a.out_ld + (int64_t)head * a.V;
    float ss = 0.f;
    for (int i = lane; i < a.V; i += 32) {
        const float v = src[i] * f;
        ss = fmaf(v, v, ss);
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)a.V + a.eps) * a.post;
    for (int i = lane; i < a.V; i += 32) {
        float y = src[i] * f * r * w[i];
        if (g != nullptr) y *= gs_sigmoid(g[i]);
        dst[i] = from_f32<T>(y);
    }
}

// The same for V a multiple of 8 up to 256 and 16-byte aligned rows: LANES lanes (a power of two, the fewest that hold V) have 8
// values of a head each.
__device__ __forceinline__ void gs_load8(const float* p, float* v) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void gs_store8(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void gs_store8(bf16* p, const float* v) {
    uint4 r;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = r;
}

template <typename T, int LANES>
__global__ void __launch_bounds__(128) scan_head_norm_vec_kernel(HeadNormArgs a, T* __restrict__ out, uint32_t items) {
    pdl_prologue();
    const uint32_t item = (blockIdx.x * 128 + threadIdx.x) / LANES;
    const int i = (threadIdx.x % LANES) * 8;
    const bool live = item < items && i < a.V;
    const uint32_t at = live ? item : 0, row = at / (uint32_t)a.heads, head = at - row * (uint32_t)a.heads;
    const int c = live ? i : 0;
    float v[8], g[8], w[8];
    gs_load8(a.o + (int64_t)at * a.V + c, v);
    gs_load8(a.weight + (a.shared ? 0 : (int64_t)head * a.V) + c, w);
    if (a.gate != nullptr) gs_load8(a.gate + (int64_t)row * a.gate_ld + (int64_t)head * a.V + c, g);
    const float f = a.nq != nullptr ? a.q_scale / (fmaxf(fabsf(a.nq[at] * a.q_scale), a.em[at]) + a.tiny) : 1.f;
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        v[e] = live ? v[e] * f : 0.f;
        ss = fmaf(v[e], v[e], ss);
    }
#pragma unroll
    for (int off = LANES / 2; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    const float r = 1.0f / sqrtf(ss / (float)a.V + a.eps) * a.post;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        v[e] = v[e] * r * w[e];
        if (a.gate != nullptr) v[e] *= gs_sigmoid(g[e]);
    }
    if (live) gs_store8(out + (int64_t)row * a.out_ld + (int64_t)head * a.V + i, v);
}

// ----------------------------------------------------------------------------------------
// host side
// ----------------------------------------------------------------------------------------
static bool gs_aligned16(const void* p) { return (((uintptr_t)p) & 15) == 0; }

template <int KI, bool HEAD_GATES>
static int gated_scan_launch(const GatedScanArgs& a, int n_seqs, int vec, cudaStream_t stream) {
    constexpr int NB = 32 * KI, TB = KI >= 8 ? 8 : 16;
    constexpr size_t SMEM = sizeof(float) * GS_STAGES * TB * ((HEAD_GATES ? 2 : 3) * NB + GS_COLS + (HEAD_GATES ? 2 : 0));
    static OncePerDevice configured;
    if (SMEM > 48 * 1024 && configured.need()) {
        const cudaError_t e = cudaFuncSetAttribute(gated_scan_kernel<KI, HEAD_GATES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        X0NE_REQUIRE(e == cudaSuccess, "gated_scan: %zu bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        configured.done();
    }
    // Launched without the early-start attribute: blocks that start while the kernel before still fills the GPU gather on the
    // first multiprocessors that have room, two on one while others stay empty, and stay there for the whole scan.
    gated_scan_kernel<KI, HEAD_GATES><<<dim3(n_seqs, a.heads, (a.C + GS_COLS - 1) / GS_COLS), dim3(GS_THREADS + 32), SMEM, stream>>>(a, vec);
    X0NE_LAUNCH_CHECK();
}

static int gated_check(const GatedScanArgs& a, int n_seqs, const char* what) {
    const bool hg = a.C == a.V + 1;
    X0NE_REQUIRE(n_seqs >= 0 && n_seqs <= 0x7fffffff && a.heads > 0 && a.heads <= 65535 && a.D > 0 && a.D <= 65536 && a.V > 0 && a.V <= 65536 && (a.C == a.V || hg),
                 "%s: %d sequences, %d heads, %d x %d state of %d columns", what, n_seqs, a.heads, a.D, a.V, a.C);
    X0NE_REQUIRE(a.state_stride >= (int64_t)a.heads * a.C * a.D && a.o != nullptr && (!hg || a.nq != nullptr), "%s: the state row is too short, or an output is missing", what);
    return 0;
}

// Scan over the rows of every sequence.  gates given: head gates (C = V + 1, w null); else channel gates (C = V).
X0NE_API int x0ne_gated_scan(GatedScanArgs a, int n_seqs, cudaStream_t stream) {
    if (int e = gated_check(a, n_seqs, "gated_scan")) return e;
    const bool hg = a.gates != nullptr;
    X0NE_REQUIRE(hg == (a.C == a.V + 1) && hg == (a.w == nullptr), "gated_scan: decays per channel or gates per head, not both or neither");
    if (n_seqs == 0) return 0;
    const bool al = a.D % 4 == 0 && gs_aligned16(a.state) && a.state_stride % 4 == 0;
    X0NE_REQUIRE(a.D % 4 != 0 || al, "gated_scan: the state is not 16-byte aligned");
    const int vec = al && gs_aligned16(a.q) && gs_aligned16(a.k) && gs_aligned16(a.w) && a.q_ld % 4 == 0 && a.k_ld % 4 == 0 && (hg || a.w_ld % 4 == 0);
    if (a.D > 256) {
        const int threads = a.C >= 128 ? 128 : (a.C + 31) / 32 * 32;
        x0ne_launch(gated_scan_any_kernel, dim3(n_seqs, a.heads, (a.C + threads - 1) / threads), dim3(threads), 0, stream, a);
        X0NE_LAUNCH_CHECK();
    }
#define GS_SCAN(KI) return hg ? gated_scan_launch<KI, true>(a, n_seqs, vec, stream) : gated_scan_launch<KI, false>(a, n_seqs, vec, stream)
    if (a.D <= 64) GS_SCAN(2);
    if (a.D <= 128) GS_SCAN(4);
    GS_SCAN(8);
#undef GS_SCAN
}

// The widest head whose one-token steps x0ne_gated_step takes (wider ones go through the gates' kernels and the scan).
X0NE_API int x0ne_gated_step_max_dim() { return 256; }

// Gates and step of a pass in which every sequence brings exactly one row.
X0NE_API int x0ne_gated_step(GatedScanArgs a, GatedRaw x, int n_seqs, cudaStream_t stream) {
    if (int e = gated_check(a, n_seqs, "gated_step")) return e;
    const bool hg = a.C == a.V + 1;
    X0NE_REQUIRE(a.D <= 256 && (a.D % 4 != 0 || (gs_aligned16(a.state) && a.state_stride % 4 == 0)), "gated_step: heads of %d, or a misaligned state", a.D);
    X0NE_REQUIRE(x.src != nullptr && x.f_bias != nullptr && (hg ? x.i_bias != nullptr && x.em != nullptr && x.cap > 0.f && x.seq_pos0 != nullptr &&
                 x.m_off >= (int64_t)a.heads * a.C * a.D && a.state_stride >= x.m_off + 2 * a.heads : x.lower != nullptr), "gated_step: a gate's tensor is missing");
    if (n_seqs == 0) return 0;
    const dim3 grid(n_seqs, a.heads, (a.C + GS_COLS - 1) / GS_COLS), block(GS_THREADS);
#define GS_STEP(KI)                                                                                      \
    do {                                                                                                 \
        if (hg) x0ne_launch(gated_step_kernel<KI, true>, grid, block, 0, stream, a, x);                  \
        else x0ne_launch(gated_step_kernel<KI, false>, grid, block, 0, stream, a, x);                    \
    } while (0)
    if (a.D <= 64) GS_STEP(2);
    else if (a.D <= 128) GS_STEP(4);
    else GS_STEP(8);
#undef GS_STEP
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_channel_gates(GatedRaw x, float* out, int n_rows, int hd, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && hd > 0 && x.src != nullptr && x.f_bias != nullptr && x.lower != nullptr && x.ld >= hd, "channel_gates: rows %d of %d channels", n_rows, hd);
    if (n_rows == 0) return 0;
    const bool vec = hd % 4 == 0 && x.ld % 4 == 0 && x.q_col % 4 == 0 && x.k_col % 4 == 0 && gs_aligned16(x.src) && gs_aligned16(x.f_bias) &&
                     gs_aligned16(x.lower) && gs_aligned16(out);
    const int64_t total = (int64_t)n_rows * hd / (vec ? 4 : 1);
    const int64_t blocks = (total + 255) / 256;
    const dim3 grid((unsigned)(blocks < 148 * 64 ? blocks : 148 * 64));
    if (vec) x0ne_launch(channel_gates_vec_kernel, grid, dim3(256), 0, stream, x, out, total, hd);
    else x0ne_launch(channel_gates_kernel, grid, dim3(256), 0, stream, x, out, total, hd);
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_head_gates(GatedRaw x, float* gates, float* state, int64_t state_stride, const int32_t* seq_first_row, const int32_t* seq_slot,
                             int n_seqs, int heads, cudaStream_t stream) {
    X0NE_REQUIRE(n_seqs >= 0 && heads > 0 && heads <= 65535 && x.src != nullptr && x.f_bias != nullptr && x.i_bias != nullptr && x.em != nullptr && x.cap > 0.f &&
                     x.seq_pos0 != nullptr && state_stride >= x.m_off + 2 * heads, "head_gates: %d sequences, %d heads", n_seqs, heads);
    if (n_seqs == 0) return 0;
    x0ne_launch(head_gates_kernel, dim3(n_seqs, heads), dim3(256), 0, stream, x, gates, state, state_stride, seq_first_row, seq_slot, heads);
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_scan_head_norm(HeadNormArgs a, void* out, int dt, int n_rows, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && a.heads > 0 && a.V > 0 && a.o != nullptr && a.weight != nullptr && a.out_ld >= (int64_t)a.heads * a.V &&
                     (a.nq == nullptr || a.em != nullptr), "scan_head_norm: rows %d heads %d of %d", n_rows, a.heads, a.V);
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "scan_head_norm: unknown dtype tag %d", dt);
    if (n_rows == 0) return 0;
    const int64_t items = (int64_t)n_rows * a.heads;
    X0NE_REQUIRE(items < (1ll << 31), "scan_head_norm: %lld heads in all", (long long)items);
    const bool vec = a.V % 8 == 0 && a.V <= 256 && a.out_ld % 8 == 0 && a.gate_ld % 4 == 0 && gs_aligned16(a.o) && gs_aligned16(a.weight) &&
                     gs_aligned16(a.gate) && gs_aligned16(out);
    const dim3 block(128);
#define GS_HEAD_NORM_VEC(T, L) x0ne_launch(scan_head_norm_vec_kernel<T, L>, dim3((unsigned)((items * L + 127) / 128)), block, 0, stream, a, (T*)out, (uint32_t)items)
#define GS_HEAD_NORM(T)                                                                                                                             \
    do {                                                                                                                                            \
        if (!vec) x0ne_launch(scan_head_norm_kernel<T>, dim3((unsigned)((items + 3) / 4)), block, 0, stream, a, (T*)out, (uint32_t)items);          \
        else if (a.V <= 32) GS_HEAD_NORM_VEC(T, 4);                                                                                                 \
        else if (a.V <= 64) GS_HEAD_NORM_VEC(T, 8);                                                                                                 \
        else if (a.V <= 128) GS_HEAD_NORM_VEC(T, 16);                                                                                               \
        else GS_HEAD_NORM_VEC(T, 32);                                                                                                               \
    } while (0)
    if (dt == X0NE_F32) GS_HEAD_NORM(float);
    else GS_HEAD_NORM(bf16);
#undef GS_HEAD_NORM
#undef GS_HEAD_NORM_VEC
    X0NE_LAUNCH_CHECK();
}
