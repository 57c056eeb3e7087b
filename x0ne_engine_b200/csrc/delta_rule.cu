// The gated delta rule: a linear recurrence with a matrix state per head whose every write corrects what the state already
// answers for its key.  Per sequence and value head, token by token, with q and k of the key head it shares:
//   S = g S;   u = beta (v - S^T k);   S = S + k u^T;   o = S^T q
// q, k and v are projections that pass a causal convolution of K taps per channel and silu; q and k are then unit vectors,
//   x / sqrt(sum(x^2) + 1e-6), q times q_scale besides;  beta = sigmoid(b);  g = exp(-A softplus(a + dt_bias)) per head, A > 0.
// A head's o goes on as  o / sqrt(mean(o^2) + eps) * weight * silu(gate).
//
// Kernels: `delta_prepare` (convolution, activation, unit vectors, gates of many tokens), `delta_scan` or (bfloat16 runs)
// `delta_coef` and `delta_chunk_scan`, `delta_head_norm`; `delta_step` does all of it for passes in which every sequence brings one token; `delta_scan_any` for wider heads.
//
// The state of a sequence is one float32 row: S transposed, [heads][V columns][D], then at `ring_off` the convolution's last
// inputs as a ring of K rows of `channels` values (q, k, v side by side), the input of position p in row p % K.  A token at
// p reads the rows of p - 1 .. p - K + 1 and its own goes into the one row it does not read, so the blocks of a one-token
// step may read the ring while one of them writes it.  In passes of many tokens the scan, which runs after the convolution,
// brings the ring up to date.
//
// Everything is float32.  Every sum runs in an order that depends on the sizes alone and the kernels share their device
// functions, so (the scan by chunks apart, whose chunks start with a pass) a token's result is the same bits however its
// sequence is cut into passes and whatever else a pass holds.
#include "common.cuh"

#define DR_TINY 1e-6f
#define DR_WINDOW 3             // inputs before the current one that `delta_prepare` keeps in registers
#define DR_MAX_TAPS 64
#define DR_TB 16                // tokens the scan stages at a time
#define DR_STAGES 3
#define DR_COLS 16              // columns of S a scan's block takes
#define DR_STEP_MAX_WARPS 8
#define DR_STEP_CW 4            // columns per lane of the one-token kernel
#define DR_CHUNK 8              // tokens the scan by chunks takes together (one tile of the tensor cores)
#define DR_CHUNK_STAGES 4
#define DR_COEF 20              // numbers per (token, head) it reads besides q, k and v

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
    // what `delta_prepare` leaves, a plane per head (n_rows rows each), so that a scan copies the rows of several tokens as one piece:
    // q of every key head, then k ([rows][row_len], zeros past the head's channels), then v of every value head by blocks of
    // DR_COLS columns ([rows][DR_COLS], zeros past the last)
    float* planes;
    float* gates;               // [heads][rows][4]: g, beta, two places that are not used
    float* o;                   // [rows][heads * V]
    int32_t heads, kv_heads, D, V, taps, n_rows, row_len;
};

__host__ __device__ __forceinline__ int dr_row_len(int D) { return (D <= 32 ? 32 : D <= 64 ? 64 : D <= 128 ? 128 : D <= 256 ? 256 : (D + 3) / 4 * 4) + 8; }
__host__ __device__ __forceinline__ int dr_blocks(int V) { return (V + DR_COLS - 1) / DR_COLS; }
// the plane of key head kh (which 0: q, 1: k), and of columns block * DR_COLS .. of value head `head`
__device__ __forceinline__ float* dr_plane_qk(const DeltaArgs& a, int which, int kh) { return a.planes + (int64_t)(which * a.kv_heads + kh) * a.n_rows * a.row_len; }
__device__ __forceinline__ float* dr_plane_v(const DeltaArgs& a, int head, int block) {
    return a.planes + (int64_t)2 * a.kv_heads * a.n_rows * a.row_len + (int64_t)(head * dr_blocks(a.V) + block) * a.n_rows * DR_COLS;
}

__device__ __forceinline__ int dr_channels(const DeltaArgs& a) { return 2 * a.kv_heads * a.D + a.heads * a.V; }
__device__ __forceinline__ float dr_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_beta(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// g multiplies the state once per token: close to one it is one plus the small difference, which loses nothing but one rounding
__device__ __forceinline__ float dr_decay(float z, float A) {
    const float x = -A * dr_softplus(z);
    return x > -0.5f ? 1.0f + expm1f(x) : expf(x);
}

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
// packed pairs, of CW neighbouring columns.  Dot products: two chains of pairs (first and second half of every four), summed,
// then a butterfly over the L lanes.
// ----------------------------------------------------------------------------------------
template <int L, int KI> struct DrRow {          // a lane's channels of q or k
    f32x2 v[KI / 2];
    __device__ __forceinline__ void load(const float* row, int l) {           // a row of L * KI values in shared memory
#pragma unroll
        for (int i = 0; i < KI / 4; ++i) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + 4 * (l + L * i));
            v[2 * i] = x.x;
            v[2 * i + 1] = x.y;
        }
    }
};
template <int L, int KI, int CW> struct DrState {
    f32x2 v[CW][KI / 2];
    // column c of the lane's columns lies D * c values behind `col`; the first `n_in` of them exist
    __device__ __forceinline__ void load(const float* col, int l, int D, int n_in) {
#pragma unroll
        for (int c = 0; c < CW; ++c)
#pragma unroll
            for (int i = 0; i < KI / 4; ++i) {
                const int d = 4 * (l + L * i);
                const float* p = col + (int64_t)c * D + d;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if ((D & 3) == 0) {
                    if (c < n_in && d < D) x = *reinterpret_cast<const float4*>(p);
                } else if (c < n_in) {
                    if (d < D) x.x = p[0];
                    if (d + 1 < D) x.y = p[1];
                    if (d + 2 < D) x.z = p[2];
                    if (d + 3 < D) x.w = p[3];
                }
                v[c][2 * i] = dr_pack(x.x, x.y);
                v[c][2 * i + 1] = dr_pack(x.z, x.w);
            }
    }
    __device__ __forceinline__ void store(float* col, int l, int D, int n_in) const {
#pragma unroll
        for (int c = 0; c < CW; ++c) {
            if (c >= n_in) continue;
#pragma unroll
            for (int i = 0; i < KI / 4; ++i) {
                const int d = 4 * (l + L * i);
                float* p = col + (int64_t)c * D + d;
                float4 x;
                dr_unpack(v[c][2 * i], x.x, x.y);
                dr_unpack(v[c][2 * i + 1], x.z, x.w);
                if ((D & 3) == 0) {
                    if (d < D) *reinterpret_cast<float4*>(p) = x;
                } else {
                    if (d < D) p[0] = x.x;
                    if (d + 1 < D) p[1] = x.y;
                    if (d + 2 < D) p[2] = x.z;
                    if (d + 3 < D) p[3] = x.w;
                }
            }
        }
    }
    __device__ __forceinline__ float dot(int c, const DrRow<L, KI>& b) const {
        f32x2 x = dr_mul2(v[c][0], b.v[0]), y = dr_mul2(v[c][1], b.v[1]);
#pragma unroll
        for (int i = 1; i < KI / 4; ++i) {
            x = dr_fma2(v[c][2 * i], b.v[2 * i], x);
            y = dr_fma2(v[c][2 * i + 1], b.v[2 * i + 1], y);
        }
        float lo, hi;
        dr_unpack(dr_add2(x, y), lo, hi);
        return lo + hi;
    }
};

template <int L>
__device__ __forceinline__ float dr_lanes_sum(float x) {
#pragma unroll
    for (int off = L / 2; off >= 1; off >>= 1) x += __shfl_xor_sync(0xffffffffu, x, off);
    return x;
}

// One token: S = g S + k u with u = beta (v - g S^T k) (the decayed state answers g times what the state before answers), and this
// lane's share of o in acc.
template <int L, int KI, int CW>
__device__ __forceinline__ void dr_token(DrState<L, KI, CW>& S, const DrRow<L, KI>& q, const DrRow<L, KI>& k, const float (&v)[CW], float g, float beta, float* acc) {
    float u[CW];
#pragma unroll
    for (int c = 0; c < CW; ++c) u[c] = S.dot(c, k);
#pragma unroll
    for (int off = L / 2; off >= 1; off >>= 1)
#pragma unroll
        for (int c = 0; c < CW; ++c) u[c] += __shfl_xor_sync(0xffffffffu, u[c], off);
    const f32x2 gg = dr_dup(g);
#pragma unroll
    for (int c = 0; c < CW; ++c) {
        const f32x2 uu = dr_dup(beta * fmaf(-g, u[c], v[c]));
#pragma unroll
        for (int i = 0; i < KI / 2; ++i) S.v[c][i] = dr_fma2(k.v[i], uu, dr_mul2(S.v[c][i], gg));
        acc[c] = S.dot(c, q);
    }
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
__device__ __forceinline__ float dr_unit_factor(const float (&x)[NJ], float scale) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) ss = fmaf(x[j], x[j], ss);
    return scale / sqrtf(warp_sum(ss) + DR_TINY);
}
template <int NJ>
__device__ __forceinline__ void dr_unit(float (&x)[NJ], float scale) {
    const float r = dr_unit_factor<NJ>(x, scale);
#pragma unroll
    for (int j = 0; j < NJ; ++j) x[j] *= r;
}

// A warp norms and gates one head's o (in shared or global memory); `vec`: V a multiple of 4 and everything 16-byte aligned.
__device__ __forceinline__ void dr_store4(float* p, const float4& y) { *reinterpret_cast<float4*>(p) = y; }
__device__ __forceinline__ void dr_store4(bf16* p, const float4& y) {
    __nv_bfloat162 h[2] = {__floats2bfloat162_rn(y.x, y.y), __floats2bfloat162_rn(y.z, y.w)};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(h);
}
template <typename T>
__device__ __forceinline__ void dr_head_norm(const float* o, const float* gate, const float* w, T* out, int V, float eps, int vec, int lane) {
    float ss = 0.f;
    if (vec && V <= 128) {              // a lane has four values at most: everything is asked for at once
        const bool in = 4 * lane < V;
        const int i = in ? 4 * lane : 0;
        const float4 g = *reinterpret_cast<const float4*>(gate + i), ww = *reinterpret_cast<const float4*>(w + i);
        const float4 x = *reinterpret_cast<const float4*>(o + i);
        if (in) {
            ss = fmaf(x.x, x.x, ss); ss = fmaf(x.y, x.y, ss); ss = fmaf(x.z, x.z, ss); ss = fmaf(x.w, x.w, ss);
        }
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps);
        if (in) dr_store4(out + i, make_float4(x.x * r * ww.x * dr_silu(g.x), x.y * r * ww.y * dr_silu(g.y), x.z * r * ww.z * dr_silu(g.z), x.w * r * ww.w * dr_silu(g.w)));
        return;
    }
    if (vec) {
        for (int i = 4 * lane; i < V; i += 128) {
            const float4 x = *reinterpret_cast<const float4*>(o + i);
            ss = fmaf(x.x, x.x, ss); ss = fmaf(x.y, x.y, ss); ss = fmaf(x.z, x.z, ss); ss = fmaf(x.w, x.w, ss);
        }
    } else {
        for (int i = lane; i < V; i += 32) ss = fmaf(o[i], o[i], ss);
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps);
    if (vec) {
        for (int i = 4 * lane; i < V; i += 128) {
            const float4 x = *reinterpret_cast<const float4*>(o + i), g = *reinterpret_cast<const float4*>(gate + i), ww = *reinterpret_cast<const float4*>(w + i);
            dr_store4(out + i, make_float4(x.x * r * ww.x * dr_silu(g.x), x.y * r * ww.y * dr_silu(g.y), x.z * r * ww.z * dr_silu(g.z), x.w * r * ww.w * dr_silu(g.w)));
        }
    } else {
        for (int i = lane; i < V; i += 32) out[i] = from_f32<T>(o[i] * r * w[i] * dr_silu(gate[i]));
    }
}

// ----------------------------------------------------------------------------------------
// Convolution, activation, unit vectors and gates of many tokens.  A warp takes one head of q, k or v (or, the last unit, all
// heads' gates) and walks `stretch` rows (at most 31) with the inputs it still needs in registers.
// ----------------------------------------------------------------------------------------
template <int NJ>
__global__ void __launch_bounds__(128, NJ <= 4 ? 6 : 4) delta_prepare_kernel(DeltaArgs a, int stretch) {
    pdl_launch_dependents();
    constexpr int GROUP = NJ >= 4 ? 2 : 4;          // rows whose inputs are fetched together
    const int lane = threadIdx.x & 31;
    const int G = a.kv_heads, units = 2 * G + a.heads + 1;
    const int64_t item = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int64_t part = item / units;
    const int unit = (int)(item - part * units);
    const int64_t first = part * stretch;
    if (first >= a.n_rows) return;
    const int n_rows = (int)min((int64_t)a.n_rows - first, (int64_t)stretch);
    if (unit == units - 1) {
        pdl_wait();
        for (int e = lane; e < n_rows * a.heads; e += 32) {
            const int64_t row = first + e / a.heads;
            const int h = e % a.heads;
            const float* s = a.src + row * a.ld;
            *reinterpret_cast<float4*>(a.gates + ((int64_t)h * a.n_rows + row) * 4) = make_float4(dr_decay(s[a.a_col + h] + a.dt_bias[h], a.A[h]), dr_beta(s[a.b_col + h]), 0.f, 0.f);
        }
        return;
    }
    const bool is_v = unit >= 2 * G;
    const int n = is_v ? a.V : a.D;
    const int c0 = is_v ? 2 * G * a.D + (unit - 2 * G) * a.V : unit * a.D;           // the head's first channel
    const int col0 = is_v ? a.v_col + (unit - 2 * G) * a.V : unit < G ? a.q_col + unit * a.D : a.k_col + (unit - G) * a.D;
    const int channels = dr_channels(a), K = a.taps;
    // bit i: row i of the stretch (at most 31 rows) goes on where the row above it stands
    int slot_l = -1, pos_l = 0;
    bool on_l = false;
    if (lane < n_rows) {
        const int64_t row = first + lane;
        slot_l = a.row_slot[row];
        pos_l = a.row_pos[row];
        on_l = row > 0 && slot_l >= 0 && a.row_slot[row - 1] == slot_l && a.row_pos[row - 1] == pos_l - 1;
    }
    const unsigned on = __ballot_sync(0xffffffffu, on_l);
    // value lane + 32 j of row r goes to out[j * out_j + r * out_row] (zeros past the head's last)
    float* const out = is_v ? dr_plane_v(a, unit - 2 * G, lane / DR_COLS) + lane % DR_COLS : dr_plane_qk(a, unit < G ? 0 : 1, unit % G) + lane;
    const int64_t out_j = is_v ? (int64_t)(32 / DR_COLS) * a.n_rows * DR_COLS : 32;
    const int out_row = is_v ? DR_COLS : a.row_len, out_n = is_v ? dr_blocks(n) * DR_COLS : 32 * NJ;
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
        for (int r0 = 0; r0 < n_rows; r0 += GROUP) {
            float x[GROUP][NJ];
#pragma unroll
            for (int e = 0; e < GROUP; ++e) {
                const float* s = a.src + (first + min(r0 + e, n_rows - 1)) * a.ld + col0;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int c = j0 + lane + 32 * j;
                    x[e][j] = c < n ? s[c] : 0.f;
                }
            }
#pragma unroll
            for (int e = 0; e < GROUP; ++e) {
                const int r = r0 + e;
                if (r >= n_rows) break;
                const int64_t row = first + r;
                if (r == 0 || !((on >> r) & 1u)) {            // the inputs ahead of this row: rows above it in its sequence, then the kept ones
                    const int slot = __shfl_sync(0xffffffffu, slot_l, r), pos = __shfl_sync(0xffffffffu, pos_l, r);
                    bool above = true;
#pragma unroll
                    for (int back = 1; back <= DR_WINDOW; ++back) {
                        above = above && row - back >= 0 && slot >= 0 && a.row_slot[row - back] == slot && a.row_pos[row - back] == pos - back;
#pragma unroll
                        for (int j = 0; j < NJ; ++j) {
                            const int c = j0 + lane + 32 * j;
                            float y = 0.f;
                            if (c < n && back < K && slot >= 0 && pos - back >= 0)
                                y = above ? a.src[(row - back) * a.ld + col0 + c]
                                          : a.state[(int64_t)slot * a.state_stride + a.ring_off + (int64_t)((pos - back) % K) * channels + c0 + c];
                            before[j][DR_WINDOW - back] = y;
                        }
                    }
                }
                float y[NJ];
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    float acc = 0.f;
#pragma unroll
                    for (int i = 0; i < DR_WINDOW; ++i) acc = fmaf(w[j][i], before[j][i], acc);
                    acc = fmaf(w[j][DR_WINDOW], x[e][j], acc);
#pragma unroll
                    for (int i = 0; i + 1 < DR_WINDOW; ++i) before[j][i] = before[j][i + 1];
                    before[j][DR_WINDOW - 1] = x[e][j];
                    y[j] = j0 + lane + 32 * j < n ? dr_silu(acc) : 0.f;
                }
                if (!is_v) dr_unit<NJ>(y, unit < G ? a.q_scale : 1.0f);
                float* to = out + (j0 / 32) * out_j + row * out_row;
#pragma unroll
                for (int j = 0; j < NJ; ++j)
                    if (j0 + lane + 32 * j < out_n) to[j * out_j] = y[j];
            }
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
            *reinterpret_cast<float4*>(a.gates + ((int64_t)h * a.n_rows + row) * 4) =
                make_float4(dr_decay(s[a.a_col + h] + a.dt_bias[h], a.A[h]), dr_beta(s[a.b_col + h]), 0.f, 0.f);
        return;
    }
    const bool is_v = unit >= 2 * G;
    const int n = is_v ? a.V : a.D, c0 = is_v ? 2 * G * a.D + (unit - 2 * G) * a.V : unit * a.D;
    const int slot = a.row_slot[row], pos = a.row_pos[row];
    int above = 0;
    while (above < a.taps - 1 && row - above - 1 >= 0 && slot >= 0 && a.row_slot[row - above - 1] == slot && a.row_pos[row - above - 1] == pos - above - 1) ++above;
    if (is_v) {
        for (int c = lane; c < dr_blocks(n) * DR_COLS; c += 32)
            dr_plane_v(a, unit - 2 * G, c / DR_COLS)[row * DR_COLS + c % DR_COLS] = c < n ? dr_conv_at(a, row, slot, pos, above, c0 + c) : 0.f;
        return;
    }
    float* dst = dr_plane_qk(a, unit < G ? 0 : 1, unit % G) + row * a.row_len;
    float ss = 0.f;
    for (int c = lane; c < n; c += 32) {
        const float y = dr_conv_at(a, row, slot, pos, above, c0 + c);
        dst[c] = y;
        ss = fmaf(y, y, ss);
    }
    for (int c = n + lane; c < a.row_len; c += 32) dst[c] = 0.f;
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
// What feeds both scans: a warp of its own that copies the inputs of TB tokens at a time into a ring of NS stages of shared
// memory: four bulk copies, [TB][ROW] of k and of q, [TB][DR_COLS] of v and [TB][COEF] of the token's other numbers, counted by the
// stage's "full" barrier; the working warps hand a stage back by its "empty" barrier.  Rows past a sequence's last are zeros.
// (A bulk copy per row kept the copy engine busy for 70 cycles each, 2,300 per 8 tokens: several times what the working warps take.)
// ----------------------------------------------------------------------------------------
#define DR_WAIT_CYCLES 2000000000ll
#define DR_STATUS_BIT (1 << 19)

__device__ __forceinline__ uint32_t dr_smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void dr_bar_init(uint64_t* bar, int count) { asm volatile("mbarrier.init.shared.b64 [%0], %1;" ::"r"(dr_smem_addr(bar)), "r"(count) : "memory"); }
__device__ __forceinline__ void dr_bar_arrive(uint64_t* bar) { asm volatile("mbarrier.arrive.shared.b64 _, [%0];" ::"r"(dr_smem_addr(bar)) : "memory"); }
__device__ __forceinline__ void dr_bar_expect(uint64_t* bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared.b64 _, [%0], %1;" ::"r"(dr_smem_addr(bar)), "r"(bytes) : "memory");
}
// false if the wait ran out (then the status word says so)
__device__ __forceinline__ bool dr_bar_wait(uint64_t* bar, int parity, int* status) {
    uint32_t done = 0;
    long long start = 0;
    for (;;) {
        asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                     : "=r"(done) : "r"(dr_smem_addr(bar)), "r"(parity) : "memory");
        if (done) return true;
        const long long now = clock64();
        if (start == 0) start = now;
        if (now - start > DR_WAIT_CYCLES) {
            atomicOr(status, DR_STATUS_BIT);
            return false;
        }
    }
}
__device__ __forceinline__ void dr_bulk(float* dst, const float* src, int bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(dr_smem_addr(dst)), "l"(src), "r"(bytes), "r"(dr_smem_addr(bar)) : "memory");
}

template <int TB, int ROW, int COEF, int NS>
struct DrFeed {
    static constexpr int STAGE = TB * (2 * ROW + DR_COLS + COEF), K = 0, Q = TB * ROW, V = 2 * TB * ROW, X = V + TB * DR_COLS;      // where k, q, v, the rest lie
    static_assert(ROW % 4 == 0 && DR_COLS % 4 == 0 && COEF % 4 == 0, "rows of whole 16-byte pieces");
    float* smem;                // [NS][STAGE]
    uint64_t* full;             // [NS]
    uint64_t* empty;            // [NS]
    int* status;

    // all threads of the block, before its first __syncthreads
    __device__ __forceinline__ void init(int tid, int warps) {
        if (tid == 0) {
            for (int i = 0; i < NS; ++i) {
                dr_bar_init(full + i, 1);
                dr_bar_init(empty + i, warps);
            }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __device__ __forceinline__ const float* stage(int s) const { return smem + (s % NS) * STAGE; }
    __device__ __forceinline__ bool wait_full(int s) const {
        const bool ok = dr_bar_wait(full + s % NS, (s / NS) & 1, status);
        return __all_sync(0xffffffffu, ok);             // (the lanes come together again)
    }
    __device__ __forceinline__ void hand_back(int s, int lane) const {
        __syncwarp();
        if (lane == 0) dr_bar_arrive(empty + s % NS);
    }

    // the feeding warp's whole life; rest: this head's [rows][COEF]
    __device__ __forceinline__ void run(const DeltaArgs& a, const float* rest, int row0, int n_tok, int head, int block, int lane) const {
        const int kh = head / (a.heads / a.kv_heads), n_stages = (n_tok + TB - 1) / TB;
        // lanes 0 .. 3 copy k, q, v and the rest
        const int len = lane < 2 ? ROW : lane == 2 ? DR_COLS : COEF, place = lane == 0 ? K : lane == 1 ? Q : lane == 2 ? V : X;
        const float* src = (lane == 0 ? dr_plane_qk(a, 1, kh) : lane == 1 ? dr_plane_qk(a, 0, kh) : lane == 2 ? dr_plane_v(a, head, block) : rest) + (int64_t)row0 * len;
        for (int s = 0; s < n_stages; ++s) {
            float* base = smem + (s % NS) * STAGE;
            uint64_t* bar = full + s % NS;
            const int t0 = s * TB, nt = min(TB, n_tok - t0);
            if (s >= NS && !dr_bar_wait(empty + s % NS, ((s / NS) - 1) & 1, status)) break;
            __syncwarp();
            if (nt < TB) {
                for (int i = nt * ROW + lane; i < TB * ROW; i += 32) base[K + i] = base[Q + i] = 0.f;
                for (int i = nt * DR_COLS + lane; i < TB * DR_COLS; i += 32) base[V + i] = 0.f;
                for (int i = nt * COEF + lane; i < TB * COEF; i += 32) base[X + i] = 0.f;
                __syncwarp();
            }
            if (lane == 0) dr_bar_expect(bar, (uint32_t)(nt * (2 * ROW + DR_COLS + COEF)) * 4);
            __syncwarp();
            if (lane < 4) dr_bulk(base + place, src + (int64_t)t0 * len, nt * len * 4, bar);
        }
        __syncwarp();
        // nothing of its own may be in flight when the block ends
        for (int s = max(0, n_stages - NS); s < n_stages; ++s)
            if (!wait_full(s)) break;
    }
};

// ----------------------------------------------------------------------------------------
// Scan over many tokens, one after the other.  A block takes one sequence, one value head and a few columns of S (columns do not
// depend on one another), CW columns per L lanes.  What a token costs in time is one dot product, its sum over L lanes and one
// update.
// ----------------------------------------------------------------------------------------
template <int L, int KI> using DrScanFeed = DrFeed<DR_TB, L * KI + 8, 4, DR_STAGES>;

template <int L, int KI, int CW>
__global__ void __launch_bounds__(DR_COLS / CW * L + 32) delta_scan_kernel(DeltaArgs a, int* status) {
    using Feed = DrScanFeed<L, KI>;
    constexpr int ROW = L * KI + 8, WARPS = DR_COLS / CW * L / 32;
    extern __shared__ __align__(16) float dr_smem[];
    __shared__ uint64_t bars[2 * DR_STAGES];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int seq = blockIdx.x, head = blockIdx.y, j0 = blockIdx.z * DR_COLS;
    const int D = a.D, V = a.V;
    Feed feed{dr_smem, bars, bars + DR_STAGES, status};
    feed.init(tid, WARPS);
    pdl_wait();
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0) return;
    const int n_stages = (n_tok + DR_TB - 1) / DR_TB;
    __syncthreads();
    if (warp == WARPS) {
        feed.run(a, a.gates + (int64_t)head * a.n_rows * 4, row0, n_tok, head, blockIdx.z, lane);
        if (blockIdx.z == 0) dr_keep_inputs(a, seq, slot, row0, n_tok, head, lane, 32);
        return;
    }

    const int l = lane % L, mycol = (warp * (32 / L) + lane / L) * CW, col = j0 + mycol, n_in = V - col;       // (n_in may be zero or less)
    float* st = a.state + (int64_t)slot * a.state_stride + ((int64_t)head * V + (n_in > 0 ? col : 0)) * D;
    DrState<L, KI, CW> S;
    S.load(st, l, D, n_in);
    const int64_t o_ld = (int64_t)a.heads * V;
    // after a group of U tokens lane l of a column's lanes holds the result of token l / CW in column l % CW
    constexpr int U = L / CW;
    float* od = a.o + (int64_t)row0 * o_ld + (int64_t)head * V + col;
    const int my_t = l / CW, my_c = l % CW;
    auto token = [&](const float* base, int t, float* acc) {
        DrRow<L, KI> k, q;
        k.load(base + Feed::K + t * ROW, l);
        q.load(base + Feed::Q + t * ROW, l);
        const float* vb = base + Feed::V + t * DR_COLS + mycol;
        const float2 g = *reinterpret_cast<const float2*>(base + Feed::X + 4 * t);
        float v[CW];
#pragma unroll
        for (int c = 0; c < CW; ++c) v[c] = vb[c];
        dr_token<L, KI, CW>(S, q, k, v, g.x, g.y, acc);
    };
    for (int s = 0; s < n_stages; ++s) {
        if (!feed.wait_full(s)) return;
        const float* base = feed.stage(s);
        const int t0 = s * DR_TB, nt = min(DR_TB, n_tok - t0);
        int t = 0;
#pragma unroll 1
        for (; t + U <= nt; t += U) {
            float acc[L];
#pragma unroll
            for (int x = 0; x < U; ++x) token(base, t + x, acc + x * CW);
            const float x = dr_lanes_share<L>(acc, l);
            if (my_c < n_in) od[(int64_t)(t0 + t + my_t) * o_ld + my_c] = x;
        }
#pragma unroll 1
        for (; t < nt; ++t) {
            float acc[CW];
            token(base, t, acc);
#pragma unroll
            for (int c = 0; c < CW; ++c) {
                const float x = dr_lanes_sum<L>(acc[c]);
                if (c < n_in && l == 0) od[(int64_t)(t0 + t) * o_ld + c] = x;
            }
        }
        feed.hand_back(s, lane);
    }
    S.store(st, l, D, n_in);
}

// ----------------------------------------------------------------------------------------
// Scan by chunks of C = DR_CHUNK tokens (passes of many tokens in bfloat16 runs).  Within a chunk, with S the state before it,
// p_t = S^T k_t, r_t = S^T q_t, and c(t, s) the product of the decays of the tokens s + 1 .. t (s = -1: from the chunk's first):
//   u_t = z_t - sum_{s < t} M[t][s] u_s,   z_t = beta_t v_t - beta_t c(t, -1) p_t,   M[t][s] = beta_t c(t, s) k_t . k_s
//   o_t = c(t, -1) r_t + sum_{s <= t} N[t][s] u_s,   N[t][s] = c(t, s) q_t . k_s
//   S   = c(C-1, -1) S + sum_s c(C-1, s) k_s u_s^T
// which is the rule itself, written so that every product with S of a chunk is taken from one S.  With T = (I + M)^-1 (a
// triangular solve by numbers of the token and head alone), u = T z and o = c r + (N T) z.  `delta_coef`, one block per (chunk, key
// head), leaves the rows of T and N T, beta_t, beta_t c(t, -1), c(t, -1) and c(C-1, t) at [head][row][DR_COEF].  Chunks count
// from the first row a sequence brings to the pass.
//
// The products run on the tensor cores (mma.sync m16n8k8) with every float32 operand x as the two tf32 numbers hi = tf32(x) and
// lo = tf32(x - hi): hi hi + hi lo + lo hi, float32 sums.  hi and lo hold 22 bits of x and a sign each, what is dropped is below
// 2^-22 of the product.  The state, decays and all sums stay float32.  The order of sums differs from the token-by-token kernels'.
// ----------------------------------------------------------------------------------------
__global__ void __launch_bounds__(64) delta_coef_kernel(DeltaArgs a, float* __restrict__ coef) {
    constexpr int C = DR_CHUNK;
    extern __shared__ __align__(16) float dr_smem[];
    __shared__ float M[C][C + 1], N[C][C + 1], T[C][C + 1];
    pdl_prologue();
    const int seq = blockIdx.y, kh = blockIdx.z, tid = threadIdx.x;
    const int slot = a.seq_slot[seq], first = a.seq_first_row[seq] + (int)blockIdx.x * C, nt = min(C, a.seq_first_row[seq + 1] - first);
    if (slot < 0 || nt <= 0) return;
    const int D = a.D, Dp = (D + 3) / 4 * 4 + 4, rep = a.heads / a.kv_heads;
    float* ks = dr_smem;                    // [C][Dp]
    float* qs = ks + C * Dp;                // [C][Dp]
    for (int i = tid; i < 2 * C * (Dp / 4); i += 64) {
        const int r = i / (Dp / 4), d = (i - r * (Dp / 4)) * 4, t = r % C;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t < nt && d < a.row_len) x = *reinterpret_cast<const float4*>(dr_plane_qk(a, r < C ? 1 : 0, kh) + (int64_t)(first + t) * a.row_len + d);
        *reinterpret_cast<float4*>(dr_smem + r * Dp + d) = x;
    }
    __syncthreads();
    const int t = tid / C, s = tid % C;
    float kk = 0.f, qk = 0.f;
    for (int d = 0; d < D; d += 4) {
        const float4 x = *reinterpret_cast<const float4*>(ks + s * Dp + d), k = *reinterpret_cast<const float4*>(ks + t * Dp + d), q = *reinterpret_cast<const float4*>(qs + t * Dp + d);
        kk = fmaf(k.x, x.x, kk); kk = fmaf(k.y, x.y, kk); kk = fmaf(k.z, x.z, kk); kk = fmaf(k.w, x.w, kk);
        qk = fmaf(q.x, x.x, qk); qk = fmaf(q.y, x.y, qk); qk = fmaf(q.z, x.z, qk); qk = fmaf(q.w, x.w, qk);
    }
    for (int h = kh * rep; h < (kh + 1) * rep; ++h) {
        const float* g = a.gates + ((int64_t)h * a.n_rows + first) * 4;
        float gr[C];
#pragma unroll
        for (int r = 0; r < C; ++r) gr[r] = r < nt ? g[r * 4] : 1.f;
        const float beta = t < nt ? g[t * 4 + 1] : 0.f;
        float between = 1.f, since = 1.f, after = 1.f;       // c(t, s), c(t, -1), c(C-1, t)
#pragma unroll
        for (int r = 0; r < C; ++r) {
            if (r > s && r <= t) between *= gr[r];
            if (r <= t) since *= gr[r];
            else after *= gr[r];
        }
        M[t][s] = s < t ? beta * (between * kk) : 0.f;
        N[t][s] = s <= t ? between * qk : 0.f;
        __syncthreads();
        if (tid < C) {                  // column tid of T by forward substitution
            float x[C];
#pragma unroll
            for (int r = 0; r < C; ++r) {
                float acc = r == tid ? 1.f : 0.f;
#pragma unroll
                for (int e = 0; e < r; ++e) acc = fmaf(-M[r][e], x[e], acc);
                x[r] = acc;
                T[r][tid] = acc;
            }
        }
        __syncthreads();
        if (t < nt) {
            float nt_ts = 0.f;
#pragma unroll
            for (int e = 0; e < C; ++e) nt_ts = fmaf(N[t][e], T[e][s], nt_ts);
            float* dst = coef + ((int64_t)h * a.n_rows + first + t) * DR_COEF;
            dst[s] = T[t][s];
            dst[C + s] = nt_ts;
            if (s == 0) *reinterpret_cast<float4*>(dst + 2 * C) = make_float4(beta, beta * since, since, after);
        }
    }
}

// The nearest number with 10 fraction bits (halves away from zero), by adding half of the last of them to the magnitude's bits and
// cutting the rest off; the tensor cores ignore what lo has beyond them.
__device__ __forceinline__ void dr_split(float x, uint32_t& hi, uint32_t& lo) {
    hi = (__float_as_uint(x) + 0x1000u) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi)) + 0x1000u;
}
__device__ __forceinline__ void dr_mma(float (&c)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// An accumulator tile as the A operand of the next product: its columns 2t and 2t + 1 take the places t and t + 4 of the inner
// index, so the B operand holds inner index 2t in b[0] and 2t + 1 in b[1].
struct DrA {
    uint32_t hi[4], lo[4];
    __device__ __forceinline__ explicit DrA(const float (&c)[4]) {
        dr_split(c[0], hi[0], lo[0]);
        dr_split(c[2], hi[1], lo[1]);
        dr_split(c[1], hi[2], lo[2]);
        dr_split(c[3], hi[3], lo[3]);
    }
};
struct DrB {
    uint32_t hi[2], lo[2];
    __device__ __forceinline__ DrB(float x, float y) {
        dr_split(x, hi[0], lo[0]);
        dr_split(y, hi[1], lo[1]);
    }
};

#define DR_CHUNK_WARPS 4        // working warps of a block: each takes a share of the channels
template <int NT> constexpr int dr_chunk_row() { return DR_CHUNK_WARPS * NT * 8 + 8; }         // a row of k or q in shared memory
template <int NT> using DrChunkFeed = DrFeed<DR_CHUNK, dr_chunk_row<NT>(), DR_COEF, DR_CHUNK_STAGES>;
constexpr int dr_chunk_parts() { return 2 * DR_CHUNK_WARPS * 4 * 32 * 2; }

// A block takes one sequence, one value head and 16 columns of S; a warp keeps NT tiles of 16 columns x 8 channels as
// accumulators.  A chunk: the warps' shares of p and r meet in shared memory, every warp goes on with the sums, and adds the chunk's
// writes to its own channels.  A warp without channels makes the results from the sums, another copies the inputs ahead.
template <int NT>
__global__ void __launch_bounds__(DR_CHUNK_WARPS * 32 + 64) delta_chunk_scan_kernel(DeltaArgs a, const float* __restrict__ coef, int* status) {
    using Feed = DrChunkFeed<NT>;
    constexpr int C = DR_CHUNK, WARPS = DR_CHUNK_WARPS, ROW = dr_chunk_row<NT>(), COLS = DR_COLS, NS = DR_CHUNK_STAGES;
    static_assert(C == 8 && COLS == 16 && WARPS == 4, "a chunk is one tile of 8 tokens; four warps exchange their parts");
    extern __shared__ __align__(16) float dr_smem[];
    __shared__ uint64_t bars[2 * NS];
    float2* parts = reinterpret_cast<float2*>(dr_smem + NS * Feed::STAGE);          // [2][WARPS][4][32]
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int seq = blockIdx.x, head = blockIdx.y, j0 = blockIdx.z * COLS;
    const int D = a.D, V = a.V;
    Feed feed{dr_smem, bars, bars + NS, status};
    feed.init(tid, WARPS + 1);
    pdl_wait();
    const int slot = a.seq_slot[seq];
    const int row0 = a.seq_first_row[seq], n_tok = a.seq_first_row[seq + 1] - row0;
    if (slot < 0 || n_tok <= 0) return;
    const int n_stages = (n_tok + C - 1) / C;
    __syncthreads();
    if (warp == WARPS + 1) {
        feed.run(a, coef + (int64_t)head * a.n_rows * DR_COEF, row0, n_tok, head, blockIdx.z, lane);
        if (blockIdx.z == 0) dr_keep_inputs(a, seq, slot, row0, n_tok, head, lane, 32);
        return;
    }

    const int g = lane >> 2, t2 = 2 * (lane & 3);           // this lane's columns g, g + 8 and tokens / channels t2, t2 + 1 of a tile
    // the sums of the warps' parts of tile x (0: p, 1: r) of chunk s, once all of them are there
    auto gather = [&](int s, int x, float (&sum)[4]) {
        const float2* from = parts + (s & 1) * WARPS * 4 * 32 + lane;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float2 y[WARPS];
#pragma unroll
            for (int w = 0; w < WARPS; ++w) y[w] = from[(w * 4 + 2 * x + e) * 32];
            sum[2 * e] = (y[0].x + y[1].x) + (y[2].x + y[3].x);
            sum[2 * e + 1] = (y[0].y + y[1].y) + (y[2].y + y[3].y);
        }
    };
    auto exchange = [&]() { asm volatile("bar.sync 1, %0;" ::"n"(DR_CHUNK_WARPS * 32 + 32) : "memory"); };
    // a warp whose wait ran out goes on with what is there, and waits no more, so that the others' exchanges end; the status word
    // says so
    bool alive = true;
    if (warp == WARPS) {                // the results
        const int64_t o_ld = (int64_t)a.heads * V;
        float* od = a.o + (int64_t)row0 * o_ld + (int64_t)head * V + j0;
        for (int s = 0; s < n_stages; ++s, od += (int64_t)C * o_ld) {
            if (alive) alive = feed.wait_full(s);
            const float* base = feed.stage(s);
            const float* vb = base + Feed::V;
            const float* cb = base + Feed::X;
            const int nt = min(C, n_tok - s * C);
            const float4 m0 = *reinterpret_cast<const float4*>(cb + t2 * DR_COEF + 2 * C), m1 = *reinterpret_cast<const float4*>(cb + (t2 + 1) * DR_COEF + 2 * C);
            const float v00 = vb[t2 * COLS + g], v01 = vb[(t2 + 1) * COLS + g], v10 = vb[t2 * COLS + g + 8], v11 = vb[(t2 + 1) * COLS + g + 8];
            const float2 rn = *reinterpret_cast<const float2*>(cb + g * DR_COEF + C + t2);
            const DrB BN(rn.x, rn.y);
            exchange();
            float p[4], r[4];
            gather(s, 0, p);
            gather(s, 1, r);
            const float z[4] = {fmaf(-m0.y, p[0], m0.x * v00), fmaf(-m1.y, p[1], m1.x * v01), fmaf(-m0.y, p[2], m0.x * v10), fmaf(-m1.y, p[3], m1.x * v11)};
            const DrA Z(z);
            float o[4] = {m0.z * r[0], m1.z * r[1], m0.z * r[2], m1.z * r[3]}, ol[4] = {};
            dr_mma(o, Z.hi, BN.hi);
            dr_mma(ol, Z.hi, BN.lo);
            dr_mma(ol, Z.lo, BN.hi);
            feed.hand_back(s, lane);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int c = g + (e >= 2 ? 8 : 0), t = t2 + (e & 1);
                if (t < nt && j0 + c < V) od[(int64_t)t * o_ld + c] = o[e] + ol[e];
            }
        }
        return;
    }

    const int ch0 = warp * NT * 8;
    float* st = a.state + (int64_t)slot * a.state_stride + ((int64_t)head * V + j0) * D;
    float S[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = g + (e >= 2 ? 8 : 0), d = ch0 + 8 * j + t2 + (e & 1);
            S[j][e] = j0 + c < V && d < D ? st[(int64_t)c * D + d] : 0.f;
        }
    for (int s = 0; s < n_stages; ++s) {
        if (alive) alive = feed.wait_full(s);
        const float* base = feed.stage(s);
        const float* vb = base + Feed::V;
        const float* cb = base + Feed::X;
        const int nt = min(C, n_tok - s * C);
        // this warp's share of p (tile 0: columns x tokens) and r (tile 1)
        float hh[2][4] = {}, hl[2][4] = {}, lh[2][4] = {};
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const DrA A(S[j]);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const float2 b = *reinterpret_cast<const float2*>(base + (x == 0 ? Feed::K : Feed::Q) + g * ROW + ch0 + 8 * j + t2);
                const DrB B(b.x, b.y);
                dr_mma(hh[x], A.hi, B.hi);
                dr_mma(hl[x], A.hi, B.lo);
                dr_mma(lh[x], A.lo, B.hi);
            }
        }
        float2* mine = parts + ((s & 1) * WARPS + warp) * 4 * 32 + lane;
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 4; e += 2)
                mine[(2 * x + e / 2) * 32] = make_float2(hh[x][e] + (hl[x][e] + lh[x][e]), hh[x][e + 1] + (hl[x][e + 1] + lh[x][e + 1]));
        // what the chunk's other numbers need, asked for before the exchange; the decayed state and the operands of its update too
        const float4 m0 = *reinterpret_cast<const float4*>(cb + t2 * DR_COEF + 2 * C), m1 = *reinterpret_cast<const float4*>(cb + (t2 + 1) * DR_COEF + 2 * C);
        const float v00 = vb[t2 * COLS + g], v01 = vb[(t2 + 1) * COLS + g], v10 = vb[t2 * COLS + g + 8], v11 = vb[(t2 + 1) * COLS + g + 8];
        const float2 rt = *reinterpret_cast<const float2*>(cb + g * DR_COEF + t2);
        const float all = cb[(nt - 1) * DR_COEF + 2 * C + 2];
        const DrB BT(rt.x, rt.y);
        float kx[NT][2];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const float* kd = base + Feed::K + t2 * ROW + ch0 + 8 * j + g;
            kx[j][0] = kd[0];
            kx[j][1] = kd[ROW];
#pragma unroll
            for (int e = 0; e < 4; ++e) S[j][e] *= all;
        }
        exchange();
        float p[4];
        gather(s, 0, p);
        const float z[4] = {fmaf(-m0.y, p[0], m0.x * v00), fmaf(-m1.y, p[1], m1.x * v01), fmaf(-m0.y, p[2], m0.x * v10), fmaf(-m1.y, p[3], m1.x * v11)};
        const DrA Z(z);
        float u[4] = {}, ul[4] = {}, uh[4] = {};
        dr_mma(u, Z.hi, BT.hi);
        dr_mma(ul, Z.hi, BT.lo);
        dr_mma(uh, Z.lo, BT.hi);
        const float w[4] = {m0.w * (u[0] + (ul[0] + uh[0])), m1.w * (u[1] + (ul[1] + uh[1])), m0.w * (u[2] + (ul[2] + uh[2])), m1.w * (u[3] + (ul[3] + uh[3]))};
        const DrA W(w);
        float low[NT][4] = {};
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const DrB B(kx[j][0], kx[j][1]);
            dr_mma(S[j], W.hi, B.hi);
            dr_mma(low[j], W.hi, B.lo);
            dr_mma(low[j], W.lo, B.hi);
        }
        feed.hand_back(s, lane);
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[j][e] += low[j][e];
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = g + (e >= 2 ? 8 : 0), d = ch0 + 8 * j + t2 + (e & 1);
            if (j0 + c < V && d < D) st[(int64_t)c * D + d] = S[j][e];
        }
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
    const int kh = head / (a.heads / a.kv_heads);
    float* S = a.state + (int64_t)slot * a.state_stride + ((int64_t)head * a.V + col) * a.D;
    for (int64_t row = row0; row < row0 + n_tok; ++row) {
        const float* q = dr_plane_qk(a, 0, kh) + row * a.row_len;
        const float* k = dr_plane_qk(a, 1, kh) + row * a.row_len;
        const float v = dr_plane_v(a, head, col / DR_COLS)[row * DR_COLS + col % DR_COLS];
        const float g = a.gates[((int64_t)head * a.n_rows + row) * 4], beta = a.gates[((int64_t)head * a.n_rows + row) * 4 + 1];
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
__global__ void __launch_bounds__(128) delta_head_norm_kernel(DeltaArgs a, T* __restrict__ out, int64_t out_ld, int vec) {
    pdl_prologue();
    const int lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= (int64_t)a.n_rows * a.heads) return;
    const int64_t row = item / a.heads;
    const int head = (int)(item - row * a.heads);
    dr_head_norm<T>(a.o + item * a.V, a.src + row * a.ld + a.g_col + (int64_t)head * a.V, a.norm_w, out + row * out_ld + (int64_t)head * a.V, a.V, a.eps, vec, lane);
}

// ----------------------------------------------------------------------------------------
// One token per sequence: convolution, unit vectors, gates, the step and the head's norm and gate in one launch.  A block takes
// one (sequence, value head); its columns of S are read and written straight from and to memory, the first of them while
// the token's q, k and v are worked out.
// ----------------------------------------------------------------------------------------
template <typename T, int L, int KI, int NJ>
__global__ void __launch_bounds__(DR_STEP_MAX_WARPS * 32, 3) delta_step_kernel(DeltaArgs a, T* __restrict__ out, int64_t out_ld, int vec) {
    constexpr int NB = L * KI, CW = DR_STEP_CW, CPW = 32 / L * CW, WIN = DR_WINDOW;
    extern __shared__ __align__(16) float dr_smem[];
    float* ks = dr_smem;                        // [NB], not yet of unit length
    float* qs = ks + NB;                        // [NB]
    float* os = qs + NB;                        // [V rounded up to 4]
    float* vs = os + (a.V + 3) / 4 * 4;         // [V]
    __shared__ float numbers[4];                // what q and k are multiplied by, g, beta
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
    float* ring = st_row + a.ring_off;
    const float* src = a.src + (int64_t)row0 * a.ld;
    const int l = lane % L, sub = lane / L * CW;
    for (int i = tid; i < 2 * NB; i += blockDim.x)
        if (i % NB >= D) dr_smem[i] = 0.f;
    pdl_wait();
    DrState<L, KI, CW> S;
    S.load(st + (int64_t)min(warp * CPW + sub, V - 1) * D, l, D, V - warp * CPW - sub);
    // the channels of this head's q, k and v, one after the other; the first head that shares q and k keeps their inputs
    for (int e = tid; e < 2 * D + V; e += blockDim.x) {
        const int c = e < D ? kh * D + e : e < 2 * D ? G * D + kh * D + e - D : 2 * G * D + head * V + e - 2 * D;
        const float* w = a.conv + (int64_t)c * K;
        const float x = src[dr_src_col(a, c)];
        float y[WIN], wy[WIN];
#pragma unroll
        for (int i = 0; i < WIN; ++i) {
            const int back = WIN - i;
            y[i] = back < K && pos - back >= 0 ? ring[(int64_t)((pos - back) % K) * channels + c] : 0.f;
            wy[i] = back < K ? w[K - 1 - back] : 0.f;
        }
        const float wx = w[K - 1];
        float acc = 0.f;
        for (int back = K - 1; back > WIN; --back) acc = fmaf(w[K - 1 - back], pos - back >= 0 ? ring[(int64_t)((pos - back) % K) * channels + c] : 0.f, acc);
#pragma unroll
        for (int i = 0; i < WIN; ++i) acc = fmaf(wy[i], y[i], acc);
        acc = dr_silu(fmaf(wx, x, acc));
        (e < D ? qs + e : e < 2 * D ? ks + e - D : vs + e - 2 * D)[0] = acc;
        if (K > 1 && (e >= 2 * D || head % rep == 0)) ring[(int64_t)(pos % K) * channels + c] = x;
    }
    if (tid == blockDim.x - 1) {
        numbers[2] = dr_decay(src[a.a_col + head] + a.dt_bias[head], a.A[head]);
        numbers[3] = dr_beta(src[a.b_col + head]);
    }
    __syncthreads();
    if (warp < 2) {
        const float* from = warp == 0 ? qs : ks;
        float x[NJ];
#pragma unroll
        for (int j = 0; j < NJ; ++j) x[j] = lane + 32 * j < D ? from[lane + 32 * j] : 0.f;
        const float r = dr_unit_factor<NJ>(x, warp == 0 ? a.q_scale : 1.0f);
        if (lane == 0) numbers[warp] = r;
    }
    __syncthreads();
    DrRow<L, KI> k, q;
    k.load(ks, l);
    q.load(qs, l);
    const f32x2 rq = dr_dup(numbers[0]), rk = dr_dup(numbers[1]);
#pragma unroll
    for (int i = 0; i < KI / 2; ++i) {
        q.v[i] = dr_mul2(q.v[i], rq);
        k.v[i] = dr_mul2(k.v[i], rk);
    }
    const float g = numbers[2], beta = numbers[3];
    for (int base = warp * CPW; base < V; base += warps * CPW) {
        const int col = base + sub, n_in = V - col;
        float* at = st + (int64_t)min(col, V - 1) * D;
        if (base != warp * CPW) S.load(at, l, D, n_in);
        float v[CW], acc[CW];
#pragma unroll
        for (int c = 0; c < CW; ++c) v[c] = c < n_in ? vs[col + c] : 0.f;
        dr_token<L, KI, CW>(S, q, k, v, g, beta, acc);
        S.store(at, l, D, n_in);
#pragma unroll
        for (int c = 0; c < CW; ++c) {
            const float o = dr_lanes_sum<L>(acc[c]);
            if (c < n_in && l == 0) os[col + c] = o;
        }
    }
    __syncthreads();
    if (warp == 0) dr_head_norm<T>(os, src + a.g_col + (int64_t)head * V, a.norm_w, out + (int64_t)row0 * out_ld + (int64_t)head * V, V, a.eps, vec, lane);
}

// ----------------------------------------------------------------------------------------
// host side
// ----------------------------------------------------------------------------------------
static bool dr_aligned16(const void* p) { return (((uintptr_t)p) & 15) == 0; }

// whether the heads' norm moves four values at a time (the same answer for a layer's passes of many tokens and of one)
static int dr_norm_vec(const DeltaArgs& a, const void* out, int64_t out_ld) {
    return a.V % 4 == 0 && a.ld % 4 == 0 && a.g_col % 4 == 0 && out_ld % 4 == 0 && dr_aligned16(a.src) && dr_aligned16(a.norm_w) && dr_aligned16(out);
}

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
    X0NE_REQUIRE(a.planes != nullptr && dr_aligned16(a.planes) && a.row_len == dr_row_len(a.D) && a.gates != nullptr && dr_aligned16(a.gates) && a.conv != nullptr && a.A != nullptr && a.dt_bias != nullptr, "delta_prepare: a tensor is missing");
    if (a.n_rows == 0) return 0;
    const int units = 2 * a.kv_heads + a.heads + 1;
    if (a.D > 256 || a.taps > DR_WINDOW + 1) {
        X0NE_REQUIRE(units <= 65535, "delta_prepare: %d heads", units);
        x0ne_launch(delta_prepare_any_kernel, dim3(a.n_rows, units), dim3(32), 0, stream, a);
        X0NE_LAUNCH_CHECK();
    }
    const int stretch = a.n_rows >= 1024 ? 16 : a.n_rows >= 128 ? 4 : 1;          // (at most 31)
    const int64_t items = (int64_t)((a.n_rows + stretch - 1) / stretch) * units;
    X0NE_REQUIRE((items + 3) / 4 <= 0x7fffffff, "delta_prepare: too many rows");
    const dim3 grid((unsigned)((items + 3) / 4)), block(128);
    if (a.D <= 32) x0ne_launch(delta_prepare_kernel<1>, grid, block, 0, stream, a, stretch);
    else if (a.D <= 64) x0ne_launch(delta_prepare_kernel<2>, grid, block, 0, stream, a, stretch);
    else if (a.D <= 128) x0ne_launch(delta_prepare_kernel<4>, grid, block, 0, stream, a, stretch);
    else x0ne_launch(delta_prepare_kernel<8>, grid, block, 0, stream, a, stretch);
    X0NE_LAUNCH_CHECK();
}

template <int L, int KI, int CW>
static int delta_scan_launch(const DeltaArgs& a, int n_seqs, int* status, cudaStream_t stream) {
    constexpr size_t SMEM = sizeof(float) * DR_STAGES * DrScanFeed<L, KI>::STAGE;
    static OncePerDevice configured;
    if (SMEM > 48 * 1024 && configured.need()) {
        const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<L, KI, CW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        X0NE_REQUIRE(e == cudaSuccess, "delta_scan: %zu bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        configured.done();
    }
    // without the early start: blocks that start while the kernel before still fills the GPU gather on the first multiprocessors
    // that have room and stay there for the whole scan
    delta_scan_kernel<L, KI, CW><<<dim3(n_seqs, a.heads, dr_blocks(a.V)), dim3(DR_COLS / CW * L + 32), SMEM, stream>>>(a, status);
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_delta_scan(DeltaArgs a, int n_seqs, int* status, cudaStream_t stream) {
    if (int e = dr_check(a, n_seqs, "delta_scan")) return e;
    X0NE_REQUIRE(a.planes != nullptr && dr_aligned16(a.planes) && a.row_len == dr_row_len(a.D) && a.gates != nullptr && dr_aligned16(a.gates) && a.o != nullptr && a.seq_pos0 != nullptr && a.seq_first_row != nullptr && a.seq_slot != nullptr && status != nullptr, "delta_scan: a tensor is missing");
    if (n_seqs == 0) return 0;
    if (a.D > 256) {
        const int threads = a.V >= 128 ? 128 : (a.V + 31) / 32 * 32;
        x0ne_launch(delta_scan_any_kernel, dim3(n_seqs, a.heads, (a.V + threads - 1) / threads), dim3(threads), 0, stream, a);
        X0NE_LAUNCH_CHECK();
    }
    if (a.D <= 32) return delta_scan_launch<8, 4, 1>(a, n_seqs, status, stream);
    if (a.D <= 64) return delta_scan_launch<16, 4, 1>(a, n_seqs, status, stream);
    if (a.D <= 128) return delta_scan_launch<16, 8, 1>(a, n_seqs, status, stream);
    return delta_scan_launch<32, 8, 2>(a, n_seqs, status, stream);
}

template <int NT>
static int delta_chunk_launch(const DeltaArgs& a, const float* coef, int n_seqs, int* status, cudaStream_t stream) {
    constexpr size_t SMEM = sizeof(float) * (DR_CHUNK_STAGES * DrChunkFeed<NT>::STAGE + dr_chunk_parts());
    static OncePerDevice configured;
    if (SMEM > 48 * 1024 && configured.need()) {
        const cudaError_t e = cudaFuncSetAttribute(delta_chunk_scan_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        X0NE_REQUIRE(e == cudaSuccess, "delta_chunk_scan: %zu bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        configured.done();
    }
    delta_chunk_scan_kernel<NT><<<dim3(n_seqs, a.heads, dr_blocks(a.V)), dim3(DR_CHUNK_WARPS * 32 + 64), SMEM, stream>>>(a, coef, status);
    X0NE_LAUNCH_CHECK();
}

// The scan by chunks: heads of up to 256 channels; coef: [rows][heads][DR_COEF]; at most max_seq_rows rows per sequence.
X0NE_API int x0ne_delta_chunk_scan(DeltaArgs a, float* coef, int n_seqs, int max_seq_rows, int* status, cudaStream_t stream) {
    if (int e = dr_check(a, n_seqs, "delta_chunk_scan")) return e;
    X0NE_REQUIRE(a.planes != nullptr && dr_aligned16(a.planes) && a.row_len == dr_row_len(a.D) && a.gates != nullptr && dr_aligned16(a.gates) && a.o != nullptr && coef != nullptr && dr_aligned16(coef) && a.seq_pos0 != nullptr && a.seq_first_row != nullptr &&
                     a.seq_slot != nullptr && status != nullptr, "delta_chunk_scan: a tensor is missing");
    X0NE_REQUIRE(a.D <= 256 && max_seq_rows >= 0 && n_seqs <= 65535 && a.kv_heads <= 65535, "delta_chunk_scan: heads of %d, %d sequences", a.D, n_seqs);
    if (n_seqs == 0 || max_seq_rows == 0) return 0;
    const size_t smem = (size_t)2 * DR_CHUNK * ((a.D + 3) / 4 * 4 + 4) * sizeof(float);
    x0ne_launch(delta_coef_kernel, dim3((max_seq_rows + DR_CHUNK - 1) / DR_CHUNK, n_seqs, a.kv_heads), dim3(64), smem, stream, a, coef);
    const cudaError_t e = cudaGetLastError();
    X0NE_REQUIRE(e == cudaSuccess, "delta_coef: %s", cudaGetErrorString(e));
    if (a.D <= 32) return delta_chunk_launch<1>(a, coef, n_seqs, status, stream);
    if (a.D <= 64) return delta_chunk_launch<2>(a, coef, n_seqs, status, stream);
    if (a.D <= 128) return delta_chunk_launch<4>(a, coef, n_seqs, status, stream);
    return delta_chunk_launch<8>(a, coef, n_seqs, status, stream);
}

X0NE_API int x0ne_delta_head_norm(DeltaArgs a, void* out, int dt, int64_t out_ld, cudaStream_t stream) {
    if (int e = dr_check(a, 0, "delta_head_norm")) return e;
    X0NE_REQUIRE(a.o != nullptr && a.norm_w != nullptr && out_ld >= (int64_t)a.heads * a.V && (dt == X0NE_F32 || dt == X0NE_BF16), "delta_head_norm: a tensor is missing");
    if (a.n_rows == 0) return 0;
    const int64_t items = (int64_t)a.n_rows * a.heads;
    const dim3 grid((unsigned)((items + 3) / 4)), block(128);
    const int vec = dr_norm_vec(a, out, out_ld);
    if (dt == X0NE_F32) x0ne_launch(delta_head_norm_kernel<float>, grid, block, 0, stream, a, (float*)out, out_ld, vec);
    else x0ne_launch(delta_head_norm_kernel<bf16>, grid, block, 0, stream, a, (bf16*)out, out_ld, vec);
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
    const int vec = dr_norm_vec(a, out, out_ld);
#define DR_STEP_AS(T, L, KI, NJ)                                                                                              \
    do {                                                                                                                      \
        constexpr int CPW = 32 / L * DR_STEP_CW;                                                                              \
        int warps = (a.V + CPW - 1) / CPW;                                                                                    \
        if (warps < 4) warps = 4;                                                                                             \
        if (warps > DR_STEP_MAX_WARPS) warps = DR_STEP_MAX_WARPS;                                                             \
        x0ne_launch(delta_step_kernel<T, L, KI, NJ>, grid, dim3(32 * warps), (size_t)(2 * L * KI + 2 * a.V + 4) * sizeof(float), stream, a, (T*)out, out_ld, vec); \
    } while (0)
#define DR_STEP(L, KI, NJ)                                   \
    do {                                                     \
        if (dt == X0NE_F32) DR_STEP_AS(float, L, KI, NJ);    \
        else DR_STEP_AS(bf16, L, KI, NJ);                    \
    } while (0)
    if (a.D <= 32) DR_STEP(8, 4, 1);
    else if (a.D <= 64) DR_STEP(16, 4, 2);
    else if (a.D <= 128) DR_STEP(16, 8, 4);
    else DR_STEP(32, 8, 8);
#undef DR_STEP
#undef DR_STEP_AS
    X0NE_LAUNCH_CHECK();
}
