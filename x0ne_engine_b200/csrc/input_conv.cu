// A short causal convolution on the rows a mixer reads, per channel, added to them:
//   y[t][c] = h[t][c] + sum_j w[j][c] h[t - (K - 1) + j][c]        (the last tap meets the row itself)
// Inputs ahead of a sequence's first token are zeros.  A sequence keeps its last K - 1 inputs, float32 [K - 1][width] at
// `off` of its state row, oldest first (zeros when the slot is taken).  Sums are float32, one order for a (row, channel)
// whatever the cut; the result is rounded once to the activation type.
//
//   input_conv        rows of many tokens: a thread walks a stretch of one sequence's rows of its channels; the thread of
//                     the sequence's first stretch alone reads the kept inputs and, after it, leaves the new ones
//   norm_conv_step    one row per sequence: residual add (of a result that is normed first, or of none), norm and
//                     convolution in one launch
#include "common.cuh"

#define IC_ROWS 16          // rows of a stretch (at least the taps - 1 whose first rows read the kept inputs)
#define IC_VEC_ROWS 8       // the same for the vectorised kernel, which takes up to 5 taps
#define IC_MAX_TAPS 17

__device__ __forceinline__ void ic_load8(const float* p, float* v) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ic_load8(const bf16* p, float* v) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void ic_store8(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void ic_store8(bf16* p, const float* v) {
    uint4 r;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = r;
}

// 8 values as they were read: an instruction that unpacked them would wait for the read
template <typename T> struct IcRaw;
template <> struct IcRaw<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) {
        a = reinterpret_cast<const float4*>(p)[0];
        b = reinterpret_cast<const float4*>(p)[1];
    }
    __device__ __forceinline__ void unpack(float* v) const { v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w; }
};
template <> struct IcRaw<bf16> {
    uint4 a;
    __device__ __forceinline__ void load(const bf16* p) { a = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void unpack(float* v) const {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x;
            v[2 * i + 1] = f.y;
        }
    }
};

// Any width and number of taps: a thread per channel; every input is read where it lies.
template <typename T>
__global__ void input_conv_any_kernel(const T* __restrict__ h, const float* __restrict__ w, float* __restrict__ state, int64_t state_stride,
                                      int64_t off, T* __restrict__ out, const int32_t* __restrict__ seq_first_row,
                                      const int32_t* __restrict__ seq_slot, int width, int taps) {
    pdl_prologue();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.y;
    const int row0 = seq_first_row[seq], n_tok = seq_first_row[seq + 1] - row0, slot = seq_slot[seq];
    const int t0 = blockIdx.z * IC_ROWS, t1 = min(n_tok, t0 + IC_ROWS), kept = taps - 1;
    if (c >= width || t0 >= n_tok || slot < 0) return;
    float* st = state + (int64_t)slot * state_stride + off + c;
    const T* src = h + (int64_t)row0 * width + c;
    for (int t = t0; t < t1; ++t) {
        float acc = 0.f, last = 0.f;
        for (int j = 0; j < taps; ++j) {
            const int at = t - kept + j;
            last = at >= 0 ? to_f32(src[(int64_t)at * width]) : st[(int64_t)(at + kept) * width];
            acc = fmaf(w[(int64_t)j * width + c], last, acc);
        }
        out[(int64_t)(row0 + t) * width + c] = from_f32<T>(last + acc);
    }
    if (t0 == 0)
        for (int i = 0; i < kept; ++i) {        // (ascending: a kept input moves down, never over one still needed)
            const int at = n_tok - kept + i;
            st[(int64_t)i * width] = at >= 0 ? to_f32(src[(int64_t)at * width]) : st[(int64_t)(at + kept) * width];
        }
}

// TAPS at compile time, 8 channels per thread; a stretch's rows are all asked for before the first is used.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) input_conv_vec_kernel(const T* __restrict__ h, const float* __restrict__ w, float* __restrict__ state,
                                                             int64_t state_stride, int64_t off, T* __restrict__ out,
                                                             const int32_t* __restrict__ seq_first_row, const int32_t* __restrict__ seq_slot,
                                                             int width) {
    constexpr int KEPT = TAPS - 1;
    pdl_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8, seq = blockIdx.y;
    float wk[TAPS][8];
    if (c < width) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) ic_load8(w + (int64_t)j * width + c, wk[j]);
    }
    pdl_wait();
    const int row0 = seq_first_row[seq], n_tok = seq_first_row[seq + 1] - row0, slot = seq_slot[seq];
    const int t0 = blockIdx.z * IC_VEC_ROWS, t1 = min(n_tok, t0 + IC_VEC_ROWS);
    if (c >= width || t0 >= n_tok || slot < 0) return;
    float* st = state + (int64_t)slot * state_stride + off + c;
    const T* src = h + (int64_t)row0 * width + c;
    IcRaw<T> raw[IC_VEC_ROWS];
#pragma unroll
    for (int r = 0; r < IC_VEC_ROWS; ++r)
        if (t0 + r < t1) raw[r].load(src + (int64_t)(t0 + r) * width);
    float win[TAPS][8];                     // the inputs ahead of the row, oldest first, then the row's own
#pragma unroll
    for (int i = 0; i < KEPT; ++i) {
        const int at = t0 - KEPT + i;
        if (at >= 0) ic_load8(src + (int64_t)at * width, win[i]);
        else ic_load8(st + (int64_t)(at + KEPT) * width, win[i]);
    }
#pragma unroll
    for (int r = 0; r < IC_VEC_ROWS; ++r) {
        if (t0 + r >= t1) break;
        raw[r].unpack(win[KEPT]);
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc = fmaf(wk[j][e], win[j][e], acc);
            y[e] = win[KEPT][e] + acc;
        }
        ic_store8(out + (int64_t)(row0 + t0 + r) * width + c, y);
#pragma unroll
        for (int i = 0; i < KEPT; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) win[i][e] = win[i + 1][e];
    }
    if (t0 == 0) {
#pragma unroll
        for (int i = 0; i < KEPT; ++i) {
            const int at = n_tok - KEPT + i;
            float v[8];
            if (at >= 0) ic_load8(src + (int64_t)at * width, v);
            else ic_load8(st + (int64_t)(at + KEPT) * width, v);
            ic_store8(st + (int64_t)i * width, v);
        }
    }
}

X0NE_API int x0ne_input_conv_max_taps() { return IC_MAX_TAPS; }

// h, out: [rows][width] in the activation type; w: float32 [taps][width]; max_seq_rows: at least the most rows a sequence
// brings.  Rows of no sequence are not written.
X0NE_API int x0ne_input_conv(const void* h, int dt, const float* w, float* state, int64_t state_stride, int64_t off, void* out,
                             const int32_t* seq_first_row, const int32_t* seq_slot, int n_seqs, int max_seq_rows, int width, int taps,
                             cudaStream_t stream) {
    X0NE_REQUIRE(n_seqs >= 0 && n_seqs <= 65535 && width > 0 && taps >= 1 && taps <= IC_MAX_TAPS && max_seq_rows >= 0 && max_seq_rows <= 65535 * IC_VEC_ROWS,
                 "input_conv: %d sequences of up to %d rows, width %d, %d taps (at most %d)", n_seqs, max_seq_rows, width, taps, IC_MAX_TAPS);
    X0NE_REQUIRE(taps == 1 || (state != nullptr && off >= 0 && state_stride >= off + (int64_t)(taps - 1) * width), "input_conv: the state row is too short");
    X0NE_REQUIRE(h != out, "input_conv: a row's inputs are read after rows above are written, so it does not run in place");
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "input_conv: unknown dtype tag %d", dt);
    if (n_seqs == 0 || max_seq_rows == 0) return 0;
    const bool vec = width % 8 == 0 && taps <= 5 && off % 4 == 0 && state_stride % 4 == 0 &&
                     (((uintptr_t)h | (uintptr_t)out | (uintptr_t)w | (uintptr_t)state) & 15) == 0;
    if (vec) {
        const int threads = width / 8 >= 128 ? 128 : (width / 8 + 31) / 32 * 32;
        const dim3 grid((unsigned)((width / 8 + threads - 1) / threads), (unsigned)n_seqs, (unsigned)((max_seq_rows + IC_VEC_ROWS - 1) / IC_VEC_ROWS)),
            block(threads);
#define IC_VEC(K)                                                                                                                        \
        if (dt == X0NE_F32) x0ne_launch(input_conv_vec_kernel<float, K>, grid, block, 0, stream, (const float*)h, w, state, state_stride, off, (float*)out, seq_first_row, seq_slot, width); \
        else x0ne_launch(input_conv_vec_kernel<bf16, K>, grid, block, 0, stream, (const bf16*)h, w, state, state_stride, off, (bf16*)out, seq_first_row, seq_slot, width)
        switch (taps) {
            case 1: IC_VEC(1); break;
            case 2: IC_VEC(2); break;
            case 3: IC_VEC(3); break;
            case 4: IC_VEC(4); break;
            default: IC_VEC(5); break;
        }
#undef IC_VEC
        X0NE_LAUNCH_CHECK();
    }
    const int threads = width >= 128 ? 128 : (width + 31) / 32 * 32;
    const dim3 grid((unsigned)((width + threads - 1) / threads), (unsigned)n_seqs, (unsigned)((max_seq_rows + IC_ROWS - 1) / IC_ROWS));
    if (dt == X0NE_F32)
        x0ne_launch(input_conv_any_kernel<float>, grid, dim3(threads), 0, stream, (const float*)h, w, state, state_stride, off, (float*)out, seq_first_row, seq_slot, width, taps);
    else
        x0ne_launch(input_conv_any_kernel<bf16>, grid, dim3(threads), 0, stream, (const bf16*)h, w, state, state_stride, off, (bf16*)out, seq_first_row, seq_slot, width, taps);
    X0NE_LAUNCH_CHECK();
}

// ----------------------------------------------------------------------------------------
// One row per sequence:  d = norm(delta + bias_d) * w_d (delta null: nothing is added);  resid += d;
// h = T(norm(resid) * w);  out = T(h + convolution);  the kept inputs move up by one and h joins them.
// A block per row, 8 values per thread and sweep, the row in registers from the one read of it.
// ----------------------------------------------------------------------------------------
struct NormConvArgs {
    float* resid;
    const void* delta;
    const float* bias_d;
    const float* w_d;
    float eps_d;
    const float* w;
    float eps;
    const float* conv;      // [taps][width]
    float* state;
    int64_t state_stride, off;
    const int32_t* row_slot;
    int32_t width, taps;
};

template <typename T, int ITS>
__global__ void __launch_bounds__(1024) norm_conv_step_kernel(NormConvArgs a, T* __restrict__ out) {
    __shared__ float sh[32];
    pdl_launch_dependents();
    const int64_t row = blockIdx.x;
    float wv[ITS][8];
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < a.width) ic_load8(a.w + i, wv[it]);
    }
    const int slot = a.row_slot[row];
    pdl_wait();
    float* r = a.resid + row * a.width;
    const T* d = a.delta != nullptr ? (const T*)a.delta + row * a.width : nullptr;
    float v[ITS][8], dv[ITS][8];
    float dd = 0.f, ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < a.width) {
            ic_load8(r + i, v[it]);
            if (d != nullptr) {
                ic_load8(d + i, dv[it]);
                if (a.bias_d != nullptr) {
                    float bv[8];
                    ic_load8(a.bias_d + i, bv);
#pragma unroll
                    for (int k = 0; k < 8; ++k) dv[it][k] += bv[k];
                }
#pragma unroll
                for (int k = 0; k < 8; ++k) dd += dv[it][k] * dv[it][k];
            }
        }
    }
    const float scale_d = d != nullptr ? 1.0f / sqrtf(block_sum(dd, sh) / (float)a.width + a.eps_d) : 0.f;
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < a.width) {
            if (d != nullptr) {
                float wd[8];
                ic_load8(a.w_d + i, wd);
#pragma unroll
                for (int k = 0; k < 8; ++k) v[it][k] = v[it][k] + dv[it][k] * scale_d * wd[k];
                ic_store8(r + i, v[it]);
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) ss += v[it][k] * v[it][k];
        }
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, sh) / (float)a.width + a.eps);
    const int kept = a.taps - 1;
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < a.width) {
            float hv[8], acc[8], cw[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) hv[k] = to_f32(from_f32<T>(v[it][k] * scale * wv[it][k]));
#pragma unroll
            for (int k = 0; k < 8; ++k) acc[k] = 0.f;
            float* st = a.state + (slot >= 0 ? (int64_t)slot * a.state_stride : 0) + a.off + i;
            for (int j = 0; j < kept; ++j) {
                float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                ic_load8(a.conv + (int64_t)j * a.width + i, cw);
                if (slot >= 0) {
                    ic_load8(st + (int64_t)j * a.width, x);
                    if (j > 0) ic_store8(st + (int64_t)(j - 1) * a.width, x);
                }
#pragma unroll
                for (int k = 0; k < 8; ++k) acc[k] = fmaf(cw[k], x[k], acc[k]);
            }
            if (slot >= 0 && kept > 0) ic_store8(st + (int64_t)(kept - 1) * a.width, hv);
            ic_load8(a.conv + (int64_t)kept * a.width + i, cw);
            float y[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) y[k] = hv[k] + fmaf(cw[k], hv[k], acc[k]);
            ic_store8(out + row * a.width + i, y);
        }
    }
}

// Whether x0ne_norm_conv_step takes rows of this width (16-byte aligned bases are the caller's business).
X0NE_API int x0ne_norm_conv_step_takes(int width) { return width % 8 == 0 && width <= 8 * 1024 * 2; }

X0NE_API int x0ne_norm_conv_step(NormConvArgs a, void* out, int dt, int n_rows, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && a.width > 0 && a.width % 8 == 0 && a.width <= 8 * 1024 * 2 && a.taps >= 1 && a.taps <= IC_MAX_TAPS,
                 "norm_conv_step: rows %d width %d taps %d", n_rows, a.width, a.taps);
    X0NE_REQUIRE(a.taps == 1 || (a.state != nullptr && a.off >= 0 && a.off % 4 == 0 && a.state_stride % 4 == 0 && a.state_stride >= a.off + (int64_t)(a.taps - 1) * a.width),
                 "norm_conv_step: the state row is too short or misaligned");
    X0NE_REQUIRE((((uintptr_t)a.resid | (uintptr_t)a.delta | (uintptr_t)a.bias_d | (uintptr_t)a.w_d | (uintptr_t)a.w | (uintptr_t)a.conv | (uintptr_t)a.state | (uintptr_t)out) & 15) == 0 &&
                     (a.delta == nullptr || a.w_d != nullptr), "norm_conv_step: misaligned rows, or a delta without its norm's weight");
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "norm_conv_step: unknown dtype tag %d", dt);
    if (n_rows == 0) return 0;
    int threads = (a.width / 8 + 31) / 32 * 32;
    if (threads > 1024) threads = 1024;
    if (a.width / 8 > 512 && a.width / 8 <= 1024) threads = 512;
    const int sweeps = (a.width / 8 + threads - 1) / threads;
#define IC_STEP(T, ITS) x0ne_launch(norm_conv_step_kernel<T, ITS>, dim3(n_rows), dim3(threads), 0, stream, a, (T*)out)
    if (dt == X0NE_F32) { if (sweeps <= 1) IC_STEP(float, 1); else IC_STEP(float, 2); }
    else { if (sweeps <= 1) IC_STEP(bf16, 1); else IC_STEP(bf16, 2); }
#undef IC_STEP
    X0NE_LAUNCH_CHECK();
}
