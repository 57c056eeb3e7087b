// The gated delta rule: a linear recurrence with a matrix state per head whose every write corrects what the state already
// answers for its key.  Per sequence and value head, token by token, with q and k of the key head it shares:
//   S = g S;   u = beta (v - S^T k);   S = S + k u^T;   o = S^T q
// q, k and v are projections that pass a causal convolution of K taps per channel and silu; q and k are then unit vectors,
//   x / sqrt(sum(x^2) + 1e-6), q times q_scale besides;  beta = sigmoid(b);  g = exp(-A softplus(a + dt_bias)) per head, A > 0.
// A head's o goes on as  o / sqrt(mean(o^2) + eps) * weight * silu(gate).
//
// Kernels: `delta_prepare` (convolution, activation, unit vectors, gates of many tokens), `delta_scan`, `delta_head_norm`;
// `delta_step` does all of it for passes in which every sequence brings one token; `delta_scan_any` for wider heads.
//
// The state of a sequence is one float32 row: S transposed, [heads][V columns][D], then at `ring_off` the convolution's last
// inputs as a ring of K rows of `channels` values (q, k, v side by side), the input of position p in row p % K.  A token at
// p reads the rows of p - 1 .. p - K + 1 and its own goes into the one row it does not read, so the blocks of a one-token
// step may read the ring while one of them writes it.  In passes of many tokens the scan, which runs after the convolution,
// brings the ring up to date.
//
// Everything is float32.  Every sum runs in an order that depends on the sizes alone and the kernels share their device
// functions, so a token's result is the same bits however its sequence is cut into passes and whatever else a pass holds.
#include "common.cuh"

#define DR_TINY 1e-6f
#define DR_WINDOW 3             // inputs before the current one that `delta_prepare` keeps in registers
#define DR_MAX_TAPS 64
#define DR_TB 16                // tokens the scan stages at a time
#define DR_STAGES 3
#define DR_SCAN_WARPS 4         // working warps of a scan block
#define DR_STEP_MAX_WARPS 16

struct DeltaArgs {
    const float* src;           // the packed projection [rows][ld]
    int64_t ld;
    int32_t q_col, k_col, v_col, a_col, b_col, g_col;
    const float* conv;          // [channels][taps]: q's channels, then k's, then v's
    const float* A;             // [heads]
    const float* dt_bias;       // [heads]
    const float* norm_w;        // [V]
    float q_scale, eps;
    float* state;
    int64_t state_stride, ring_off;
    const int32_t* row_slot;
    const int32_t* row_pos;
    const int32_t* seq_first_row;
    const int32_t* seq_slot;
    const int32_t* seq_pos0;
    float* qkv;                 // prepared rows [rows][channels]
    float* gates;               // [rows][heads][2]: g, beta
    float* o;                   // [rows][heads * V]
    int32_t heads, kv_heads, D, V, taps, n_rows;
};

__device__ __forceinline__ int dr_channels(const DeltaArgs& a) { return 2 * a.kv_heads * a.D + a.heads * a.V; }
__device__ __forceinline__ float dr_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_beta(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// g close to one multiplies the state once per token: rounded once, from a double exponential
__device__ __forceinline__ float dr_decay(float z, float A) { return (float)exp(-(double)A * (double)dr_softplus(z)); }

// where channel c of the convolution stands in a projection row
__device__ __forceinline__ int dr_src_col(const DeltaArgs& a, int c) {
    const int hd = a.kv_heads * a.D;
    return c < hd ? a.q_col + c : c < 2 * hd ? a.k_col + (c - hd) : a.v_col + (c - 2 * hd);
}

// ----------------------------------------------------------------------------------------
// two float32 operations per instruction
// ----------------------------------------------------------------------------------------
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 dr_dup(float a) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(a));
    return r;
}
__device__ __forceinline__ f32x2 dr_pack(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void dr_unpack(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 dr_mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 dr_fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 dr_add2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// ----------------------------------------------------------------------------------------
// A column of S is shared by L neighbouring lanes; lane l of them holds the channels 4 (l + L i) .. + 3, i < KI / 4, as
// packed pairs.  Dot products: two chains of pairs (first and second half of every four), summed, then a butterfly over the
// L lanes.
// ----------------------------------------------------------------------------------------
template <int L, int KI> struct DrLane {
    f32x2 v[KI / 2];
    __device__ __forceinline__ void load(const float* row, int l) {           // a row of L * KI values in shared memory
#pragma unroll
        for (int i = 0; i < KI / 4; ++i) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + 4 * (l + L * i));
            v[2 * i] = x.x;
            v[2 * i + 1] = x.y;
        }
    }
    __device__ __forceinline__ void load_state(const float* col, int l, int D, bool in) {
#pragma unroll
        for (int i = 0; i < KI / 4; ++i) {
            const int d = 4 * (l + L * i);
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if ((D & 3) == 0) {
                if (in && d < D) x = *reinterpret_cast<const float4*>(col + d);
            } else if (in) {
                if (d < D) x.x = col[d];
                if (d + 1 < D) x.y = col[d + 1];
                if (d + 2 < D) x.z = col[d + 2];
                if (d + 3 < D) x.w = col[d + 3];
            }
            v[2 * i] = dr_pack(x.x, x.y);
            v[2 * i + 1] = dr_pack(x.z, x.w);
        }
    }
    __device__ __forceinline__ void store_state(float* col, int l, int D, bool in) const {
        if (!in) return;
#pragma unroll
        for (int i = 0; i < KI / 4; ++i) {
            const int d = 4 * (l + L * i);
            float4 x;
            dr_unpack(v[2 * i], x.x, x.y);
            dr_unpack(v[2 * i + 1], x.z, x.w);
            if ((D & 3) == 0) {
                if (d < D) *reinterpret_cast<float4*>(col + d) = x;
            } else {
                if (d < D) col[d] = x.x;
                if (d + 1 < D) col[d + 1] = x.y;
                if (d + 2 < D) col[d + 2] = x.z;
                if (d + 3 < D) col[d + 3] = x.w;
            }
        }
    }
    __device__ __forceinline__ float dot(const DrLane& b) const {
        f32x2 x = dr_mul2(v[0], b.v[0]), y = dr_mul2(v[1], b.v[1]);
#pragma unroll
        for (int i = 1; i < KI / 4; ++i) {
            x = dr_fma2(v[2 * i], b.v[2 * i], x);
            y = dr_fma2(v[2 * i + 1], b.v[2 * i + 1], y);
        }
        float lo, hi;
        dr_unpack(dr_add2(x, y), lo, hi);
        return lo + hi;
    }
    // S = g S + k u
    __device__ __forceinline__ void decay(float g) {
        const f32x2 gg = dr_dup(g);
#pragma unroll
        for (int i = 0; i < KI / 2; ++i) v[i] = dr_mul2(v[i], gg);
    }
    __device__ __forceinline__ void write(const DrLane& k, float u) {
        const f32x2 uu = dr_dup(u);
#pragma unroll
        for (int i = 0; i < KI / 2; ++i) v[i] = dr_fma2(k.v[i], uu, v[i]);
    }
};

template <int L>
__device__ __forceinline__ float dr_lanes_sum(float x) {
#pragma unroll
    for (int off = L / 2; off >= 1; off >>= 1) x += __shfl_xor_sync(0xffffffffu, x, off);
    return x;
}

// One token of a column: returns this lane's share of o.  (The decayed state answers g times what the state before answered.)
template <int L, int KI>
__device__ __forceinline__ float dr_token(DrLane<L, KI>& S, const DrLane<L, KI>& q, const DrLane<L, KI>& k, float v, float g, float beta) {
    const float known = dr_lanes_sum<L>(S.dot(k));
    S.decay(g);
    const float u = beta * fmaf(-g, known, v);
    S.write(k, u);
    return S.dot(q);
}

// L values per lane, summed over the L lanes that share a column: lane l ends up with the sum of value l (same tree as dr_lanes_sum)
template <int L>
__device__ __forceinline__ float dr_lanes_share(float (&x)[L], int l) {
#pragma unroll
    for (int off = L / 2; off >= 1; off >>= 1) {
        const bool up = (l & off) != 0;
#pragma unroll
        for (int i = 0; i < off; ++i) {
            const float mine = up ? x[i + off] : x[i], other = up ? x[i] : x[i + off];
            x[i] = mine + __shfl_xor_sync(0xffffffffu, other, off);
        }
    }
    return x[0];
}

// A warp brings the row of D values it holds (value lane + 32 j in x[j]) to unit length, times `scale`.
template <int NJ>
__device__ __forceinline__ void dr_unit(float (&x)[NJ], float scale) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) ss = fmaf(x[j], x[j], ss);
    const float r = scale / sqrtf(warp_sum(ss) + DR_TINY);
#pragma unroll
    for (int j = 0; j < NJ; ++j) x[j] *= r;
}

// A warp norms and gates one head's o (in shared or global memory).
template <typename T>
__device__ __forceinline__ void dr_head_norm(const float* o, const float* gate, const float* w, T* out, int V, float eps, int lane) {
    float ss = 0.f;
    for (int i = lane; i < V; i += 32) ss = fmaf(o[i], o[i], ss);
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps);
    for (int i = lane; i < V; i += 32) out[i] = from_f32<T>(o[i] * r * w[i] * dr_silu(gate[i]));
}

// ----------------------------------------------------------------------------------------
// Convolution, activation, unit vectors and gates of many tokens.  A warp takes one head of q, k or v (or, the last unit, all
// heads' gates) and walks `stretch` rows with the inputs it still needs in registers.
// ----------------------------------------------------------------------------------------
template <int NJ>
__global__ void __launch_bounds__(128) delta_prepare_kernel(DeltaArgs a, int stretch) {
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int G = a.kv_heads, units = 2 * G + a.heads + 1;
    const int64_t item = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int64_t part = item / units;
    const int unit = (int)(item - part * units);
    const int64_t first = part * stretch;
    if (first >= a.n_rows) return;
    const int last = (int)min((int64_t)a.n_rows, first + stretch);
    if (unit == units - 1) {
        for (int h = lane; h < a.heads; h += 32) {
            const float A = a.A[h], db = a.dt_bias[h];
            pdl_wait();
            for (int64_t row = first; row < last; ++row) {
                const float* s = a.src + row * a.ld;
                *reinterpret_cast<float2*>(a.gates + (row * a.heads + h) * 2) = make_float2(dr_decay(s[a.a_col + h] + db, A), dr_beta(s[a.b_col + h]));
            }
        }
        return;
    }
    const bool is_v = unit >= 2 * G;
    const int n = is_v ? a.V : a.D;
    const int c0 = is_v ? 2 * G * a.D + (unit - 2 * G) * a.V : unit * a.D;           // the head's first channel
    const int col0 = is_v ? a.v_col + (unit - 2 * G) * a.V : unit < G ? a.q_col + unit * a.D : a.k_col + (unit - G) * a.D;
    const int channels = dr_channels(a), K = a.taps;
    for (int j0 = 0; j0 < n; j0 += 32 * NJ) {             // (one round for heads whose norm needs all of them; values may take more)
        float w[NJ][DR_WINDOW + 1], before[NJ][DR_WINDOW];       // tap i of w meets the input DR_WINDOW - i tokens ago
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int c = j0 + lane + 32 * j;
#pragma unroll
            for (int i = 0; i <= DR_WINDOW; ++i) {
                const int tap = K - 1 - (DR_WINDOW - i);
                w[j][i] = c < n && tap >= 0 ? a.conv[(int64_t)(c0 + c) * K + tap] : 0.f;
            }
        }
        pdl_wait();
        bool fresh = true;
        for (int64_t row = first; row < last; ++row) {
            const int slot = a.row_slot[row], pos = a.row_pos[row];
            const bool goes_on = row > 0 && slot >= 0 && a.row_slot[row - 1] == slot && a.row_pos[row - 1] == pos - 1;
            if (fresh || !goes_on) {            // the inputs ahead of this row: rows above it in its sequence, then the kept ones
                bool above = true;
#pragma unroll
                for (int back = 1; back <= DR_WINDOW; ++back) {
                    above = above && row - back >= 0 && slot >= 0 && a.row_slot[row - back] == slot && a.row_pos[row - back] == pos - back;
#pragma unroll
                    for (int j = 0; j < NJ; ++j) {
                        const int c = j0 + lane + 32 * j;
                        float x = 0.f;
                        if (c < n && back < K && slot >= 0 && pos - back >= 0)
                            x = above ? a.src[(row - back) * a.ld + col0 + c]
                                      : a.state[(int64_t)slot * a.state_stride + a.ring_off + (int64_t)((pos - back) % K) * channels + c0 + c];
                        before[j][DR_WINDOW - back] = x;
                    }
                }
                fresh = false;
            }
            const float* s = a.src + row * a.ld + col0;
            float y[NJ];
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const int c = j0 + lane + 32 * j;
                const float x = c < n ? s[c] : 0.f;
                float acc = 0.f;
#pragma unroll
                for (int i = 0; i < DR_WINDOW; ++i) acc = fmaf(w[j][i], before[j][i], acc);
                acc = fmaf(w[j][DR_WINDOW], x, acc);
#pragma unroll
                for (int i = 0; i + 1 < DR_WINDOW; ++i) before[j][i] = before[j][i + 1];
                before[j][DR_WINDOW - 1] = x;
                y[j] = c < n ? dr_silu(acc) : 0.f;
            }
            if (!is_v) dr_unit<NJ>(y, unit < G ? a.q_scale : 1.0f);
            float* dst = a.qkv + row * channels + c0 + j0;
#pragma unroll
            for (int j = 0; j < NJ; ++j)
                if (j0 + lane + 32 * j < n) dst[lane + 32 * j] = y[j];
        }
    }
}

// One channel at one row, any number of taps.
__device__ __forceinline__ float dr_conv_at(const DeltaArgs& a, int64_t row, int slot, int pos, int above, int c) {
    const int K = a.taps, channels = dr_channels(a), col = dr_src_col(a, c);
    float acc = 0.f;
    for (int back = K - 1; back >= 0; --back) {
        float x = 0.f;
        if (back <= above) x = a.src[(row - back) * a.ld + col];
        else if (slot >= 0 && pos - back >= 0) x = a.state[(int64_t)slot * a.state_stride + a.ring_off + (int64_t)((pos - back) % K) * channels + c];
        acc = fmaf(a.conv[(int64_t)c * K + K - 1 - back], x, acc);
    }
    return dr_silu(acc);
}

// Any head width and number of taps: a block per (row, unit), the sum of squares in the same order (lane + 32 j of one warp).
__global__ void __launch_bounds__(32) delta_prepare_any_kernel(DeltaArgs a) {
    pdl_prologue();
    const int lane = threadIdx.x, G = a.kv_heads, unit = blockIdx.y;
    const int64_t row = blockIdx.x;
    if (unit == 2 * G + a.heads) {
        const float* s = a.src + row * a.ld;
        for (int h = lane; h < a.heads; h += 32)
            *reinterpret_cast<float2*>(a.gates + (row * a.heads + h) * 2) =
                make_float2(dr_decay(s[a.a_col + h] + a.dt_bias[h], a.A[h]), dr_beta(s[a.b_col + h]));
        return;
    }
    const bool is_v = unit >= 2 * G;
    const int n = is_v ? a.V : a.D, c0 = is_v ? 2 * G * a.D + (unit - 2 * G) * a.V : unit * a.D;
    const int slot = a.row_slot[row], pos = a.row_pos[row];
    int above = 0;
    while (above < a.taps - 1 && row - above - 1 >= 0 && slot >= 0 && a.row_slot[row - above - 1] == slot && a.row_pos[row - above - 1] == pos - above - 1) ++above;
    float* dst = a.qkv + row * dr_channels(a) + c0;
    float ss = 0.f;
    for (int c = lane; c < n; c += 32) {
        const float y = dr_conv_at(a, row, slot, pos, above, c0 + c);
        dst[c] = y;
        ss = fmaf(y, y, ss);
    }
    if (is_v) return;
    const float r = (unit < G ? a.q_scale : 1.0f) / sqrtf(warp_sum(ss) + DR_TINY);
    for (int c = lane; c < n; c += 32) dst[c] *= r;
}

// The inputs of a sequence's last rows of the pass go into its ring: the channels of one value head, and of the key head it
// shares if it is the first that shares it.  Called by all threads of the blocks that answer for these channels.
__device__ __forceinline__ void dr_keep_inputs(const DeltaArgs& a, int seq, int slot, int row0, int n_tok, int head, int tid, int threads) {
    const int rep = a.heads / a.kv_heads, G = a.kv_heads, K = a.taps, channels = dr_channels(a);
    const int n_keep = min(K, n_tok), own = a.V + (head % rep == 0 ? 2 * a.D : 0);
    if (K == 1) return;
    float* ring = a.state + (int64_t)slot * a.state_stride + a.ring_off;
    const int pos0 = a.seq_pos0[seq];
    for (int i = tid; i < n_keep * own; i += threads) {
        const int t = n_tok - n_keep + i / own, e = i % own;
        const int c = e < a.V ? 2 * G * a.D + head * a.V + e : e < a.V + a.D ? (head / rep) * a.D + e - a.V : (G + head / rep) * a.D + e - a.V - a.D;
        ring[(int64_t)((pos0 + t) % K) * channels + c] = a.src[(int64_t)(row0 + t) * a.ld + dr_src_col(a, c)];
    }
}

// ----------------------------------------------------------------------------------------
// Scan over many tokens.  A block takes one sequence, one value head and a few columns of S (columns do not depend on one
// another), a column per L lanes.  A warp of its own copies the inputs, DR_TB tokens at a time, into a ring of DR_STAGES
// stages of shared memory by cp.async.  What a token costs in time is one dot product, its sum over L lanes and one update.
// ----------------------------------------------------------------------------------------
__device__ __forceinline__ void dr_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void dr_cp4(float* dst, const float* src, bool ok) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 4 : 0) : "memory");
}

template <int L, int KI, int WARPS> constexpr int dr_scan_cols() { return WARPS * (32 / L); }
template <int L, int KI, int WARPS> constexpr int dr_scan_stage() { return DR_TB * (2 * L * KI + dr_scan_cols<L, KI, WARPS>() + 2); }

template <int L, int KI, int WARPS>
__global__ void __launch_bounds__(WARPS * 32 + 32) delta_scan_kernel(DeltaArgs a, int vec) {
    constexpr int NB = L * KI, COLS = dr_scan_cols<L, KI, WARPS>(), STAGE = dr_scan_stage<L, KI, WARPS>(), THREADS = WARPS * 32 + 32;
    extern __shared__ __align__(16) float dr_smem[];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int seq = blockIdx.x, head = blockIdx.y, j0 = blockIdx.z * COLS;
    const int D = a.D, V = a.V, channels = dr_channels(a);
    // channels past the head's last stay zero in every stage: the copies never touch them
    for (int i = tid; i < DR_STAGES * STAGE; i += THREADS) dr_smem[i] = 0.f;
    pdl_wait();
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0) return;
    const int n_stages = (n_tok + DR_TB - 1) / DR_TB;
    __syncthreads();

    if (warp == WARPS) {
        const int kh = head / (a.heads / a.kv_heads);
        const float* base_row = a.qkv + (int64_t)row0 * channels;
        const int qc = kh * D, kc = (a.kv_heads + kh) * D, vc = 2 * a.kv_heads * D + head * V + j0;
        auto fetch = [&](int stage) {
            if (stage < n_stages) {
                float* base = dr_smem + (stage % DR_STAGES) * STAGE;
                const int t0 = stage * DR_TB, nt = min(DR_TB, n_tok - t0);
                const float* row = base_row + (int64_t)t0 * channels;
                for (int t = 0; t < nt; ++t, row += channels) {
                    float* kd = base + t * 2 * NB;
                    if (vec) {
#pragma unroll
                        for (int c = 4 * lane; c < NB; c += 128)
                            if (c < D) {
                                dr_cp16(kd + c, row + kc + c);
                                dr_cp16(kd + NB + c, row + qc + c);
                            }
                    } else {
                        for (int c = lane; c < D; c += 32) {
                            dr_cp4(kd + c, row + kc + c, true);
                            dr_cp4(kd + NB + c, row + qc + c, true);
                        }
                    }
                }
                float* vb = base + DR_TB * 2 * NB;
                row = base_row + (int64_t)t0 * channels;
                for (int e = lane; e < DR_TB * COLS; e += 32) {
                    const int t = e / COLS, c = e % COLS;
                    const bool ok = t < nt && j0 + c < V;
                    dr_cp4(vb + e, ok ? row + (int64_t)t * channels + vc + c : a.qkv, ok);
                }
                const int t = lane >> 1;
                const bool ok = t < nt;
                dr_cp4(vb + DR_TB * COLS + lane, ok ? a.gates + ((int64_t)(row0 + t0 + t) * a.heads + head) * 2 + (lane & 1) : a.gates, ok);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
#pragma unroll
        for (int s = 0; s < DR_STAGES - 1; ++s) fetch(s);
        for (int s = 0; s < n_stages; ++s) {
            asm volatile("cp.async.wait_group %0;" ::"n"(DR_STAGES - 2) : "memory");
            __syncthreads();                // stage s has arrived, and the working warps are done with stage s - 1
            fetch(s + DR_STAGES - 1);
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (blockIdx.z == 0) dr_keep_inputs(a, seq, slot, row0, n_tok, head, lane, 32);
        return;
    }

    const int l = lane % L, mycol = warp * (32 / L) + lane / L, col = j0 + mycol;
    const bool in = col < V;
    float* st = a.state + (int64_t)slot * a.state_stride + ((int64_t)head * V + (in ? col : 0)) * D;
    DrLane<L, KI> S;
    S.load_state(st, l, D, in);
    const int64_t o_ld = (int64_t)a.heads * V;
    float* od = a.o + (int64_t)row0 * o_ld + (int64_t)head * V + col;
    for (int s = 0; s < n_stages; ++s) {
        __syncthreads();
        const float* base = dr_smem + (s % DR_STAGES) * STAGE;
        const float* vb = base + DR_TB * 2 * NB + mycol;
        const float* gb = base + DR_TB * (2 * NB + COLS);
        const int t0 = s * DR_TB, nt = min(DR_TB, n_tok - t0);
        int t = 0;
#pragma unroll 1
        for (; t + L <= nt; t += L) {
            float acc[L];
#pragma unroll
            for (int x = 0; x < L; ++x) {
                DrLane<L, KI> k, q;
                k.load(base + (t + x) * 2 * NB, l);
                q.load(base + (t + x) * 2 * NB + NB, l);
                const float2 g = *reinterpret_cast<const float2*>(gb + 2 * (t + x));
                acc[x] = dr_token(S, q, k, vb[(t + x) * COLS], g.x, g.y);
            }
            const float x = dr_lanes_share<L>(acc, l);
            if (in) od[(int64_t)(t0 + t + l) * o_ld] = x;
        }
#pragma unroll 1
        for (; t < nt; ++t) {
            DrLane<L, KI> k, q;
            k.load(base + t * 2 * NB, l);
            q.load(base + t * 2 * NB + NB, l);
            const float2 g = *reinterpret_cast<const float2*>(gb + 2 * t);
            const float x = dr_lanes_sum<L>(dr_token(S, q, k, vb[t * COLS], g.x, g.y));
            if (in && l == 0) od[(int64_t)(t0 + t) * o_ld] = x;
        }
    }
    S.store_state(st, l, D, in);
}

// Any D: S stays in global memory; a thread owns a column.
__global__ void delta_scan_any_kernel(DeltaArgs a) {
    pdl_prologue();
    const int seq = blockIdx.x, head = blockIdx.y, col = blockIdx.z * blockDim.x + threadIdx.x;
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0) return;
    if (blockIdx.z == 0) dr_keep_inputs(a, seq, slot, row0, n_tok, head, threadIdx.x, blockDim.x);
    if (col >= a.V) return;
    const int channels = dr_channels(a), kh = head / (a.heads / a.kv_heads);
    float* S = a.state + (int64_t)slot * a.state_stride + ((int64_t)head * a.V + col) * a.D;
    for (int64_t row = row0; row < row0 + n_tok; ++row) {
        const float* q = a.qkv + row * channels + kh * a.D;
        const float* k = q + a.kv_heads * a.D;
        const float v = a.qkv[row * channels + 2 * a.kv_heads * a.D + head * a.V + col];
        const float g = a.gates[(row * a.heads + head) * 2], beta = a.gates[(row * a.heads + head) * 2 + 1];
        float known = 0.f, o = 0.f;
        for (int d = 0; d < a.D; ++d) known = fmaf(S[d], k[d], known);
        const float u = beta * fmaf(-g, known, v);
        for (int d = 0; d < a.D; ++d) {
            const float s = fmaf(k[d], u, g * S[d]);
            S[d] = s;
            o = fmaf(s, q[d], o);
        }
        a.o[row * ((int64_t)a.heads * a.V) + (int64_t)head * a.V + col] = o;
    }
}

template <typename T>
__global__ void __launch_bounds__(128) delta_head_norm_kernel(DeltaArgs a, T* __restrict__ out, int64_t out_ld) {
    pdl_prologue();
    const int lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= (int64_t)a.n_rows * a.heads) return;
    const int64_t row = item / a.heads;
    const int head = (int)(item - row * a.heads);
    dr_head_norm<T>(a.o + item * a.V, a.src + row * a.ld + a.g_col + (int64_t)head * a.V, a.norm_w, out + row * out_ld + (int64_t)head * a.V, a.V, a.eps, lane);
}

// ----------------------------------------------------------------------------------------
// One token per sequence: convolution, unit vectors, gates, the step and the head's norm and gate in one launch.  A block takes
// one (sequence, value head); its columns of S are read and written straight from and to memory, the first of them while
// the token's q, k and v are worked out.
// ----------------------------------------------------------------------------------------
template <typename T, int L, int KI, int NJ>
__global__ void __launch_bounds__(DR_STEP_MAX_WARPS * 32) delta_step_kernel(DeltaArgs a, T* __restrict__ out, int64_t out_ld) {
    constexpr int NB = L * KI, CPW = 32 / L;
    extern __shared__ __align__(16) float dr_smem[];
    float* ks = dr_smem;                        // [NB]
    float* qs = ks + NB;                        // [NB]
    float* vs = qs + NB;                        // [V]
    float* os = vs + a.V;                       // [V]
    __shared__ float gate2[2];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
    const int seq = blockIdx.x, head = blockIdx.y;
    const int D = a.D, V = a.V, G = a.kv_heads, rep = a.heads / G, kh = head / rep, K = a.taps, channels = dr_channels(a);
    const int slot = a.seq_slot[seq];                                        // (tables are older than any running kernel)
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    const int pos = a.seq_pos0[seq];
    if (slot < 0 || n_tok != 1) return;
    float* st_row = a.state + (int64_t)slot * a.state_stride;
    float* st = st_row + (int64_t)head * V * D;
    const int l = lane % L, sub = lane / L;
    DrLane<L, KI> S;
    // (S was last written by the step before, which is complete: kernels of a step wait for one another in turn)
    const float A = a.A[head], db = a.dt_bias[head];
    pdl_wait();
    {
        const int col = warp * CPW + sub;
        S.load_state(st + (int64_t)(col < V ? col : 0) * D, l, D, col < V);
    }
    const float* src = a.src + (int64_t)row0 * a.ld;
    float* ring = st_row + a.ring_off;
    auto conv = [&](int c, bool keep) -> float {
        const float x = src[dr_src_col(a, c)];
        float acc = 0.f;
        for (int back = K - 1; back >= 1; --back) {
            const float y = pos - back >= 0 ? ring[(int64_t)((pos - back) % K) * channels + c] : 0.f;
            acc = fmaf(a.conv[(int64_t)c * K + K - 1 - back], y, acc);
        }
        acc = fmaf(a.conv[(int64_t)c * K + K - 1], x, acc);
        if (keep && K > 1) ring[(int64_t)(pos % K) * channels + c] = x;
        return dr_silu(acc);
    };
    // warps 0 and 1: q and k; the rest (or, with two warps, both of them again): v; the last thread: gates
    for (int role = warp; role < 2; role += warps) {
        const int c0 = (role == 0 ? 0 : G * D) + kh * D;
        float x[NJ];
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int c = lane + 32 * j;
            x[j] = c < D ? conv(c0 + c, head % rep == 0) : 0.f;
        }
        dr_unit<NJ>(x, role == 0 ? a.q_scale : 1.0f);
        float* dst = role == 0 ? qs : ks;
#pragma unroll
        for (int j = 0; j < NJ; ++j) dst[lane + 32 * j] = x[j];
        if (32 * NJ < NB)
            for (int c = 32 * NJ + lane; c < NB; c += 32) dst[c] = 0.f;
    }
    const int v0 = warps > 2 ? 64 : 0;
    if (tid >= v0)
        for (int c = tid - v0; c < V; c += blockDim.x - v0) vs[c] = conv(2 * G * D + head * V + c, true);
    if (tid == blockDim.x - 1) {
        gate2[0] = dr_decay(src[a.a_col + head] + db, A);
        gate2[1] = dr_beta(src[a.b_col + head]);
    }
    __syncthreads();
    DrLane<L, KI> k, q;
    k.load(ks, l);
    q.load(qs, l);
    const float g = gate2[0], beta = gate2[1];
    for (int col = warp * CPW + sub; col - sub < V; col += warps * CPW) {
        const bool in = col < V;
        if (col != warp * CPW + sub) S.load_state(st + (int64_t)(in ? col : 0) * D, l, D, in);
        const float o = dr_lanes_sum<L>(dr_token(S, q, k, in ? vs[col] : 0.f, g, beta));
        S.store_state(st + (int64_t)(in ? col : 0) * D, l, D, in);
        if (in && l == 0) os[col] = o;
    }
    __syncthreads();
    if (warp == 0) dr_head_norm<T>(os, src + a.g_col + (int64_t)head * V, a.norm_w, out + (int64_t)row0 * out_ld + (int64_t)head * V, V, a.eps, lane);
}

// ----------------------------------------------------------------------------------------
// host side
// ----------------------------------------------------------------------------------------
static bool dr_aligned16(const void* p) { return (((uintptr_t)p) & 15) == 0; }

static int dr_check(const DeltaArgs& a, int n_seqs, const char* what) {
    X0NE_REQUIRE(n_seqs >= 0 && a.n_rows >= 0 && a.heads > 0 && a.heads <= 65535 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.D > 0 && a.D <= 65536 &&
                     a.V > 0 && a.V <= 65536 && a.taps >= 1 && a.taps <= DR_MAX_TAPS,
                 "%s: %d sequences, %d heads over %d, %d x %d, %d taps (at most %d)", what, n_seqs, a.heads, a.kv_heads, a.D, a.V, a.taps, DR_MAX_TAPS);
    const int64_t channels = 2ll * a.kv_heads * a.D + (int64_t)a.heads * a.V;
    X0NE_REQUIRE(channels < (1ll << 30) && a.ring_off >= (int64_t)a.heads * a.V * a.D && a.state_stride >= a.ring_off + (a.taps > 1 ? a.taps * channels : 0),
                 "%s: the state row is too short", what);
    X0NE_REQUIRE(a.src != nullptr && a.state != nullptr && (a.D % 4 != 0 || (dr_aligned16(a.state) && a.state_stride % 4 == 0)), "%s: a pointer is missing or misaligned", what);
    return 0;
}

X0NE_API int x0ne_delta_prepare(DeltaArgs a, cudaStream_t stream) {
    if (int e = dr_check(a, 0, "delta_prepare")) return e;
    X0NE_REQUIRE(a.qkv != nullptr && a.gates != nullptr && a.conv != nullptr && a.A != nullptr && a.dt_bias != nullptr, "delta_prepare: a tensor is missing");
    if (a.n_rows == 0) return 0;
    const int units = 2 * a.kv_heads + a.heads + 1;
    if (a.D > 256 || a.taps > DR_WINDOW + 1) {
        X0NE_REQUIRE(units <= 65535, "delta_prepare: %d heads", units);
        x0ne_launch(delta_prepare_any_kernel, dim3(a.n_rows, units), dim3(32), 0, stream, a);
        X0NE_LAUNCH_CHECK();
    }
    const int stretch = a.n_rows >= 1024 ? 16 : a.n_rows >= 128 ? 4 : 1;
    const int64_t items = (int64_t)((a.n_rows + stretch - 1) / stretch) * units;
    X0NE_REQUIRE((items + 3) / 4 <= 0x7fffffff, "delta_prepare: too many rows");
    const dim3 grid((unsigned)((items + 3) / 4)), block(128);
    if (a.D <= 32) x0ne_launch(delta_prepare_kernel<1>, grid, block, 0, stream, a, stretch);
    else if (a.D <= 64) x0ne_launch(delta_prepare_kernel<2>, grid, block, 0, stream, a, stretch);
    else if (a.D <= 128) x0ne_launch(delta_prepare_kernel<4>, grid, block, 0, stream, a, stretch);
    else x0ne_launch(delta_prepare_kernel<8>, grid, block, 0, stream, a, stretch);
    X0NE_LAUNCH_CHECK();
}

template <int L, int KI, int WARPS>
static int delta_scan_launch(const DeltaArgs& a, int n_seqs, int vec, cudaStream_t stream) {
    constexpr size_t SMEM = sizeof(float) * DR_STAGES * dr_scan_stage<L, KI, WARPS>();
    constexpr int COLS = dr_scan_cols<L, KI, WARPS>();
    static OncePerDevice configured;
    if (SMEM > 48 * 1024 && configured.need()) {
        const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<L, KI, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        X0NE_REQUIRE(e == cudaSuccess, "delta_scan: %zu bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        configured.done();
    }
    // without the early start: blocks that start while the kernel before still fills the GPU gather on the first multiprocessors
    // that have room and stay there for the whole scan
    delta_scan_kernel<L, KI, WARPS><<<dim3(n_seqs, a.heads, (a.V + COLS - 1) / COLS), dim3(WARPS * 32 + 32), SMEM, stream>>>(a, vec);
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_delta_scan(DeltaArgs a, int n_seqs, cudaStream_t stream) {
    if (int e = dr_check(a, n_seqs, "delta_scan")) return e;
    X0NE_REQUIRE(a.qkv != nullptr && a.gates != nullptr && a.o != nullptr && a.seq_pos0 != nullptr && a.seq_first_row != nullptr && a.seq_slot != nullptr, "delta_scan: a tensor is missing");
    if (n_seqs == 0) return 0;
    if (a.D > 256) {
        const int threads = a.V >= 128 ? 128 : (a.V + 31) / 32 * 32;
        x0ne_launch(delta_scan_any_kernel, dim3(n_seqs, a.heads, (a.V + threads - 1) / threads), dim3(threads), 0, stream, a);
        X0NE_LAUNCH_CHECK();
    }
    const int64_t channels = 2ll * a.kv_heads * a.D + (int64_t)a.heads * a.V;
    const int vec = a.D % 4 == 0 && channels % 4 == 0 && dr_aligned16(a.qkv);
    if (a.D <= 32) return delta_scan_launch<4, 8, 2>(a, n_seqs, vec, stream);
    if (a.D <= 64) return delta_scan_launch<4, 16, 2>(a, n_seqs, vec, stream);
    if (a.D <= 128) return delta_scan_launch<4, 32, 2>(a, n_seqs, vec, stream);
    return delta_scan_launch<8, 32, 4>(a, n_seqs, vec, stream);
}

X0NE_API int x0ne_delta_head_norm(DeltaArgs a, void* out, int dt, int64_t out_ld, cudaStream_t stream) {
    if (int e = dr_check(a, 0, "delta_head_norm")) return e;
    X0NE_REQUIRE(a.o != nullptr && a.norm_w != nullptr && out_ld >= (int64_t)a.heads * a.V && (dt == X0NE_F32 || dt == X0NE_BF16), "delta_head_norm: a tensor is missing");
    if (a.n_rows == 0) return 0;
    const int64_t items = (int64_t)a.n_rows * a.heads;
    const dim3 grid((unsigned)((items + 3) / 4)), block(128);
    if (dt == X0NE_F32) x0ne_launch(delta_head_norm_kernel<float>, grid, block, 0, stream, a, (float*)out, out_ld);
    else x0ne_launch(delta_head_norm_kernel<bf16>, grid, block, 0, stream, a, (bf16*)out, out_ld);
    X0NE_LAUNCH_CHECK();
}

// The widest heads whose one-token passes x0ne_delta_step takes (others go through the kernels for many tokens).
X0NE_API int x0ne_delta_step_max_dim() { return 256; }
X0NE_API int x0ne_delta_step_max_values() { return 2048; }

X0NE_API int x0ne_delta_step(DeltaArgs a, void* out, int dt, int64_t out_ld, int n_seqs, cudaStream_t stream) {
    if (int e = dr_check(a, n_seqs, "delta_step")) return e;
    X0NE_REQUIRE(a.D <= 256 && a.V <= 2048, "delta_step: heads of %d x %d", a.D, a.V);
    X0NE_REQUIRE(a.conv != nullptr && a.A != nullptr && a.dt_bias != nullptr && a.norm_w != nullptr && a.seq_pos0 != nullptr && a.seq_first_row != nullptr &&
                     a.seq_slot != nullptr && out_ld >= (int64_t)a.heads * a.V && (dt == X0NE_F32 || dt == X0NE_BF16), "delta_step: a tensor is missing");
    if (n_seqs == 0) return 0;
    const dim3 grid(n_seqs, a.heads);
#define DR_STEP_AS(T, L, KI, NJ)                                                                                              \
    do {                                                                                                                      \
        int warps = (a.V + 32 / L - 1) / (32 / L);                                                                            \
        if (warps < 4) warps = 4;                                                                                             \
        if (warps > DR_STEP_MAX_WARPS) warps = DR_STEP_MAX_WARPS;                                                             \
        x0ne_launch(delta_step_kernel<T, L, KI, NJ>, grid, dim3(32 * warps), (size_t)(2 * L * KI + 2 * a.V) * sizeof(float), stream, a, (T*)out, out_ld); \
    } while (0)
#define DR_STEP(L, KI, NJ)                                   \
    do {                                                     \
        if (dt == X0NE_F32) DR_STEP_AS(float, L, KI, NJ);    \
        else DR_STEP_AS(bf16, L, KI, NJ);                    \
    } while (0)
    if (a.D <= 32) DR_STEP(4, 8, 1);
    else if (a.D <= 64) DR_STEP(4, 16, 2);
    else if (a.D <= 128) DR_STEP(4, 32, 4);
    else DR_STEP(8, 32, 8);
#undef DR_STEP
#undef DR_STEP_AS
    X0NE_LAUNCH_CHECK();
}
