// Row-wise kernels: embedding, residual add + RMSNorm, q/k head norm + RoPE + cache write,
// SwiGLU.  Each is templated on the activation type (float for the 32-bit path, bfloat16 for
// the serving path); per-channel weights are always float32.
#include <stdarg.h>
#include <stdio.h>
#include <stdlib.h>

#include "common.cuh"

static thread_local char g_error[512];

void x0ne_set_error(const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_error, sizeof g_error, fmt, ap);
    va_end(ap);
}

X0NE_API const char* x0ne_last_error() { return g_error; }

bool x0ne_pdl_enabled() {
    static int on = -1;
    if (on < 0) {
        const char* e = getenv("X0NE_PDL");
        on = (e != nullptr && e[0] == '0') ? 0 : 1;
    }
    return on == 1;
}


// ----------------------------------------------------------------------------------------
// Residual add, then RMSNorm: r = resid + f32(delta) (one IEEE add, stored back);
// out = T(r * rsqrt(mean(r^2) + eps) * w)  (x0ne-core/kernels/cuda/rmsnorm.cu:11-20; eps is
// inside the root; the weight multiplies directly).  `delta` may be null (norm only).
// `rows`, if given, lists the source rows to process; output row i then belongs to source row
// rows[i] (used to norm only the rows whose logits are wanted).
// One block per row; the sum of squares is a fixed-order block sum.
// ----------------------------------------------------------------------------------------
// General form, any width: each thread owns every blockDim-th element.  The row after the add is
// parked in shared memory between the two sweeps when it fits there (`keep` floats of dynamic
// shared memory, 0 if it does not), so the residual is read once.
template <typename T>
__global__ void add_rmsnorm_any_kernel(float* __restrict__ resid, const T* __restrict__ delta, const T* __restrict__ delta2,
                                       const float* __restrict__ w, T* __restrict__ out,
                                       const int32_t* __restrict__ rows, int hidden, float eps, int keep, int ld) {
    extern __shared__ float parked[];
    __shared__ float partial[32];
    pdl_prologue();
    // blockIdx.y: the group of `hidden` consecutive values of a row of `ld` values that this block norms by itself
    const int64_t src = rows ? rows[blockIdx.x] : blockIdx.x;
    const int64_t at = src * ld + (int64_t)blockIdx.y * hidden;
    float* r = resid + at;
    w += (int64_t)blockIdx.y * hidden;
    float sum_sq = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = r[i];
        if (delta) {
            // one IEEE add, stored back; two branches of a parallel layer are summed first
            v = v + (delta2 ? to_f32(delta[at + i]) + to_f32(delta2[at + i]) : to_f32(delta[at + i]));
            r[i] = v;
        }
        if (i < keep) parked[i] = v;
        sum_sq = fmaf(v, v, sum_sq);
    }
    const float mean_sq = block_reduce(sum_sq, partial, OpSum(), 0.f) / (float)hidden;
    const float scale = 1.0f / sqrtf(mean_sq + eps);
    T* o = out + (int64_t)blockIdx.x * ld + (int64_t)blockIdx.y * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = i < keep ? parked[i] : r[i];     // a thread reads back only what it wrote itself
        o[i] = from_f32<T>(v * scale * w[i]);
    }
}

// The same, for hidden % 8 == 0 and hidden <= 8 * 1024 * VEC_IT: 16-byte accesses, and the row stays
// in registers between the sum of squares and the scaling, so it is read once.
#define VEC_IT 4
__device__ __forceinline__ void load8(const float* p, float* v) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load8(const bf16* p, float* v) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void store8(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(bf16* p, const float* v) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = u;
}

__device__ __forceinline__ void load2(const float* p, float* v) {
    const float2 a = *reinterpret_cast<const float2*>(p);
    v[0] = a.x; v[1] = a.y;
}
__device__ __forceinline__ void load2(const bf16* p, float* v) {
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = f.x; v[1] = f.y;
}
__device__ __forceinline__ void store2(float* p, const float* v) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
__device__ __forceinline__ void store2(bf16* p, const float* v) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
}
__device__ __forceinline__ void copy16(float* d, const float* s) {    // 8 values
    reinterpret_cast<float4*>(d)[0] = reinterpret_cast<const float4*>(s)[0];
    reinterpret_cast<float4*>(d)[1] = reinterpret_cast<const float4*>(s)[1];
}
__device__ __forceinline__ void copy16(bf16* d, const bf16* s) { *reinterpret_cast<uint4*>(d) = *reinterpret_cast<const uint4*>(s); }
__device__ __forceinline__ void copy2(float* d, const float* s) { *reinterpret_cast<float2*>(d) = *reinterpret_cast<const float2*>(s); }
__device__ __forceinline__ void copy2(bf16* d, const bf16* s) { *reinterpret_cast<uint32_t*>(d) = *reinterpret_cast<const uint32_t*>(s); }

// ITS: how many sweeps of the block cover a row (1, 2 or VEC_IT).
template <typename T, int ITS>
__global__ void add_rmsnorm_vec_kernel(float* __restrict__ resid, const T* __restrict__ delta, const T* __restrict__ delta2,
                                       const float* __restrict__ w, T* __restrict__ out,
                                       const int32_t* __restrict__ rows, int hidden, float eps, int ld) {
    __shared__ float sh[32];
    // The weight and the list of rows are older than any kernel still running: they are asked for
    // before the wait for the kernel before this one, so that its end is followed by one trip to
    // memory (the row) and not by two.  (With four sweeps the weight would not fit in the registers
    // that 1,024 threads can have; it is read after the sum then.)
    constexpr bool EARLY = ITS <= 2;
    pdl_launch_dependents();
    const int64_t src = rows ? rows[blockIdx.x] : blockIdx.x;
    const int64_t col0 = (int64_t)blockIdx.y * hidden;      // the group of a row of `ld` values this block norms
    w += col0;
    float wv[EARLY ? ITS : 1][8];
    if (EARLY) {
#pragma unroll
        for (int it = 0; it < ITS; ++it) {
            const int i = (it * blockDim.x + threadIdx.x) * 8;
            if (i < hidden) load8(w + i, wv[it]);
        }
    }
    pdl_wait();
    float* r = resid + src * ld + col0;
    const T* d = delta ? delta + src * ld + col0 : nullptr;
    const T* d2 = delta && delta2 ? delta2 + src * ld + col0 : nullptr;
    T* o = out + (int64_t)blockIdx.x * ld + col0;
    float v[ITS][8];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < hidden) {
            load8(r + i, v[it]);
            if (d) {
                float dv[8];
                load8(d + i, dv);
                if (d2) {
                    float dw[8];
                    load8(d2 + i, dw);
#pragma unroll
                    for (int k = 0; k < 8; ++k) dv[k] = dv[k] + dw[k];
                }
#pragma unroll
                for (int k = 0; k < 8; ++k) v[it][k] = v[it][k] + dv[k];
                store8(r + i, v[it]);
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) ss += v[it][k] * v[it][k];
        }
    }
    const float total = block_sum(ss, sh);
    const float scale = 1.0f / sqrtf(total / (float)hidden + eps);
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < hidden) {
            float late[8], ov[8];
            if (!EARLY) load8(w + i, late);
#pragma unroll
            for (int k = 0; k < 8; ++k) ov[k] = v[it][k] * scale * (EARLY ? wv[EARLY ? it : 0][k] : late[k]);
            store8(o + i, ov);
        }
    }
}

template <typename T>
static void launch_add_rmsnorm_vec(float* resid, const T* delta, const T* delta2, const float* w, T* out, const int32_t* rows, int n_rows,
                                   int hidden, float eps, int threads, int groups, cudaStream_t stream) {
    const int sweeps = (hidden / 8 + threads - 1) / threads;
    const int ld = hidden * groups;
    if (sweeps <= 1)
        x0ne_launch(add_rmsnorm_vec_kernel<T, 1>, dim3(n_rows, groups), dim3(threads), 0, stream, resid, delta, delta2, w, out, rows, hidden, eps, ld);
    else if (sweeps == 2)
        x0ne_launch(add_rmsnorm_vec_kernel<T, 2>, dim3(n_rows, groups), dim3(threads), 0, stream, resid, delta, delta2, w, out, rows, hidden, eps, ld);
    else
        x0ne_launch(add_rmsnorm_vec_kernel<T, VEC_IT>, dim3(n_rows, groups), dim3(threads), 0, stream, resid, delta, delta2, w, out, rows, hidden, eps, ld);
}

// `delta2`, if given with `delta`, is a second branch's result: r = resid + (f32(delta) + f32(delta2)).
// `groups` > 1: a row of `width` values is `groups` equal consecutive parts, each normed by its own root mean
// square (the weight still has one value per value of the row).
X0NE_API int x0ne_add2_group_rmsnorm(float* resid, const void* delta, const void* delta2, const float* w, void* out, int dt,
                                     const int32_t* rows, int n_rows, int width, int groups, float eps, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && width > 0 && groups >= 1 && groups <= 65535 && width % groups == 0, "add_rmsnorm: rows %d width %d in %d groups", n_rows, width, groups);
    X0NE_REQUIRE(delta != nullptr || delta2 == nullptr, "add_rmsnorm: a second delta without a first");
    if (n_rows == 0) return 0;
    const int hidden = width / groups;
    if (hidden % 8 == 0 && hidden <= 8 * 1024 * VEC_IT &&
        ((((uintptr_t)resid | (uintptr_t)delta | (uintptr_t)delta2 | (uintptr_t)w | (uintptr_t)out) & 15) == 0)) {
        int threads = (hidden / 8 + 31) / 32 * 32;
        if (threads > 1024) threads = 1024;
        if (hidden / 8 > 512 && hidden / 8 <= 1024) threads = 512;   // two sweeps of 512 rather than one of 1024
        if (dt == X0NE_F32)
            launch_add_rmsnorm_vec<float>(resid, (const float*)delta, (const float*)delta2, w, (float*)out, rows, n_rows, hidden, eps, threads, groups, stream);
        else if (dt == X0NE_BF16)
            launch_add_rmsnorm_vec<bf16>(resid, (const bf16*)delta, (const bf16*)delta2, w, (bf16*)out, rows, n_rows, hidden, eps, threads, groups, stream);
        else
            X0NE_REQUIRE(false, "add_rmsnorm: unknown dtype tag %d", dt);
        X0NE_LAUNCH_CHECK();
    }
    const int block = 256;
    const int keep = hidden <= 10240 ? hidden : 0;        // up to 40 KB of dynamic shared memory
    const size_t smem = (size_t)keep * sizeof(float);
    if (dt == X0NE_F32)
        x0ne_launch(add_rmsnorm_any_kernel<float>, dim3(n_rows, groups), dim3(block), smem, stream, resid, (const float*)delta, (const float*)delta2, w, (float*)out, rows, hidden, eps, keep, width);
    else if (dt == X0NE_BF16)
        x0ne_launch(add_rmsnorm_any_kernel<bf16>, dim3(n_rows, groups), dim3(block), smem, stream, resid, (const bf16*)delta, (const bf16*)delta2, w, (bf16*)out, rows, hidden, eps, keep, width);
    else
        X0NE_REQUIRE(false, "add_rmsnorm: unknown dtype tag %d", dt);
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_add2_rmsnorm(float* resid, const void* delta, const void* delta2, const float* w, void* out, int dt,
                               const int32_t* rows, int n_rows, int hidden, float eps, cudaStream_t stream) {
    return x0ne_add2_group_rmsnorm(resid, delta, delta2, w, out, dt, rows, n_rows, hidden, 1, eps, stream);
}

X0NE_API int x0ne_add_rmsnorm(float* resid, const void* delta, const float* w, void* out, int dt,
                              const int32_t* rows, int n_rows, int hidden, float eps, cudaStream_t stream) {
    return x0ne_add2_rmsnorm(resid, delta, nullptr, w, out, dt, rows, n_rows, hidden, eps, stream);
}

// ----------------------------------------------------------------------------------------
// Residual add of a delta that is normed first, then RMSNorm (a layer with a norm after each
// sublayer as well as before it):
//   x = f32(delta) + bias_d (null: none);  d = x * rsqrt(mean(x^2) + eps_d) * w_d     (float32, never rounded)
//   r = resid + d (stored back);  out = T(r * rsqrt(mean(r^2) + eps) * w)
// Same rows / block conventions as above; both sums of squares are fixed-order block sums.
// ----------------------------------------------------------------------------------------
template <typename T>
__global__ void add_normed_rmsnorm_any_kernel(float* __restrict__ resid, const T* __restrict__ delta, const float* __restrict__ bias_d,
                                              const float* __restrict__ w_d,
                                              float eps_d, const float* __restrict__ w, T* __restrict__ out,
                                              const int32_t* __restrict__ rows, int hidden, float eps, int keep) {
    extern __shared__ float parked[];
    __shared__ float partial[32];
    pdl_prologue();
    const int64_t src = rows ? rows[blockIdx.x] : blockIdx.x;
    float* r = resid + src * hidden;
    const T* d = delta + src * hidden;
    float dd = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = to_f32(d[i]) + (bias_d != nullptr ? bias_d[i] : 0.f);
        dd = fmaf(v, v, dd);
    }
    const float scale_d = 1.0f / sqrtf(block_reduce(dd, partial, OpSum(), 0.f) / (float)hidden + eps_d);
    float sum_sq = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = r[i] + (to_f32(d[i]) + (bias_d != nullptr ? bias_d[i] : 0.f)) * scale_d * w_d[i];
        r[i] = v;
        if (i < keep) parked[i] = v;
        sum_sq = fmaf(v, v, sum_sq);
    }
    const float scale = 1.0f / sqrtf(block_reduce(sum_sq, partial, OpSum(), 0.f) / (float)hidden + eps);
    T* o = out + (int64_t)blockIdx.x * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = i < keep ? parked[i] : r[i];
        o[i] = from_f32<T>(v * scale * w[i]);
    }
}

// hidden % 8 == 0 and hidden <= 8 * 1024 * 2: 16-byte accesses, the row and the delta stay in registers.
template <typename T, int ITS>
__global__ void __launch_bounds__(1024) add_normed_rmsnorm_vec_kernel(float* __restrict__ resid, const T* __restrict__ delta, const float* __restrict__ bias_d,
                                              const float* __restrict__ w_d,
                                              float eps_d, const float* __restrict__ w, T* __restrict__ out,
                                              const int32_t* __restrict__ rows, int hidden, float eps) {
    __shared__ float sh[32];
    pdl_launch_dependents();
    const int64_t src = rows ? rows[blockIdx.x] : blockIdx.x;
    pdl_wait();
    float* r = resid + src * hidden;
    const T* d = delta + src * hidden;
    T* o = out + (int64_t)blockIdx.x * hidden;
    float dv[ITS][8], v[ITS][8];
    float dd = 0.f;
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < hidden) {
            load8(d + i, dv[it]);
            load8(r + i, v[it]);
            if (bias_d != nullptr) {
                float bv[8];
                load8(bias_d + i, bv);
#pragma unroll
                for (int k = 0; k < 8; ++k) dv[it][k] += bv[k];
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) dd += dv[it][k] * dv[it][k];
        }
    }
    const float scale_d = 1.0f / sqrtf(block_sum(dd, sh) / (float)hidden + eps_d);
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < hidden) {
            float wd[8];
            load8(w_d + i, wd);
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                v[it][k] = v[it][k] + dv[it][k] * scale_d * wd[k];
                ss += v[it][k] * v[it][k];
            }
            store8(r + i, v[it]);
        }
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, sh) / (float)hidden + eps);
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < hidden) {
            float wv[8], ov[8];
            load8(w + i, wv);
#pragma unroll
            for (int k = 0; k < 8; ++k) ov[k] = v[it][k] * scale * wv[k];
            store8(o + i, ov);
        }
    }
}

X0NE_API int x0ne_add_normed_rmsnorm(float* resid, const void* delta, const float* bias_d, const float* w_d, float eps_d, const float* w, void* out,
                                     int dt, const int32_t* rows, int n_rows, int hidden, float eps, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && hidden > 0 && delta != nullptr && w_d != nullptr, "add_normed_rmsnorm: rows %d hidden %d", n_rows, hidden);
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "add_normed_rmsnorm: unknown dtype tag %d", dt);
    if (n_rows == 0) return 0;
    if (hidden % 8 == 0 && hidden <= 8 * 1024 * 2 &&
        ((((uintptr_t)resid | (uintptr_t)delta | (uintptr_t)bias_d | (uintptr_t)w_d | (uintptr_t)w | (uintptr_t)out) & 15) == 0)) {
        int threads = (hidden / 8 + 31) / 32 * 32;
        if (threads > 1024) threads = 1024;
        if (hidden / 8 > 512 && hidden / 8 <= 1024) threads = 512;
        const int sweeps = (hidden / 8 + threads - 1) / threads;
#define X0NE_ANR(T, ITS) x0ne_launch(add_normed_rmsnorm_vec_kernel<T, ITS>, dim3(n_rows), dim3(threads), 0, stream, resid, (const T*)delta, bias_d, w_d, eps_d, w, (T*)out, rows, hidden, eps)
        if (dt == X0NE_F32) {
            if (sweeps <= 1) X0NE_ANR(float, 1); else X0NE_ANR(float, 2);
        } else {
            if (sweeps <= 1) X0NE_ANR(bf16, 1); else X0NE_ANR(bf16, 2);
        }
#undef X0NE_ANR
        X0NE_LAUNCH_CHECK();
    }
    const int keep = hidden <= 10240 ? hidden : 0;
    const size_t smem = (size_t)keep * sizeof(float);
    if (dt == X0NE_F32)
        x0ne_launch(add_normed_rmsnorm_any_kernel<float>, dim3(n_rows), dim3(256), smem, stream, resid, (const float*)delta, bias_d, w_d, eps_d, w, (float*)out, rows, hidden, eps, keep);
    else
        x0ne_launch(add_normed_rmsnorm_any_kernel<bf16>, dim3(n_rows), dim3(256), smem, stream, resid, (const bf16*)delta, bias_d, w_d, eps_d, w, (bf16*)out, rows, hidden, eps, keep);
    X0NE_LAUNCH_CHECK();
}

// ----------------------------------------------------------------------------------------
// Per-head RMSNorm of q and k (optional), rotate-half RoPE, and the K/V write into the
// paged cache (x0ne-core/kernels/cuda/rope.cu:7-47).  One warp per (row, head); the row's sines and
// cosines come from a table made at start-up (or are computed by the warp); heads
// 0..q_heads-1 are q heads, the rest k heads, whose warps also copy the v head.
//   scale = rsqrt(mean(x^2 over head_dim) + eps); n = x * scale * w
//   angle = (float)pos * inv_freq[i]; (a, b) = (n[i], n[i + rot/2])
//   out[i] = a cos - b sin; out[i + rot/2] = b cos + a sin; dims >= rot pass through.
// `norm_q`/`norm_k` null: no head norm.  rot == 0: no rotation.
// A row whose position has no page writes nothing into the cache.
// ----------------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void rope_one_head(const T* __restrict__ qkv, const float* __restrict__ norm_q,
                                              const float* __restrict__ norm_k, int rot, T* __restrict__ q_out,
                                              const PagedCache& cache, const int32_t* __restrict__ row_slot, int row, int pos,
                                              int head, int q_heads, float eps, int write_kv,
                                              const float* __restrict__ cs_tab, const float* __restrict__ sn_tab) {
    const int lane = threadIdx.x & 31;
    const int hd = cache.head_dim, half = rot >> 1;
    const int q_dim = q_heads * hd, kv_dim = cache.kv_heads * hd;
    const bool is_q = head < q_heads;
    const int kh = is_q ? 0 : head - q_heads;
    if (!is_q && !write_kv) return;
    const T* src = qkv + (int64_t)row * (q_dim + 2 * kv_dim) + (is_q ? head * hd : q_dim + kh * hd);
    const float* nw = is_q ? norm_q : norm_k;

    T* dst;
    if (is_q) {
        dst = q_out + (int64_t)row * q_dim + head * hd;
    } else {
        const int64_t off = cache_row_offset(cache, row_slot[row], pos, kh, 0);
        if (off < 0) return;
        dst = (T*)cache.base + off;
    }

    // The common shape (whole head rotated, head_dim a multiple of 4 up to 256): each lane owns the
    // pairs (i, i + half) for i = 2 lane, 2 lane + 1 (+ 64 ...), keeps them in registers between the
    // sum of squares and the rotation, and moves two values per access.
    if (rot == hd && (hd & 3) == 0 && hd <= 256) {
        float a[2][2], b[2][2];
        float ss = 0.f;
#pragma unroll
        for (int it = 0; it < 2; ++it) {
            const int i = 2 * lane + 64 * it;
            if (i < half) {
                load2(src + i, a[it]);
                load2(src + i + half, b[it]);
                ss += a[it][0] * a[it][0] + a[it][1] * a[it][1] + b[it][0] * b[it][0] + b[it][1] * b[it][1];
            }
        }
        float scale = 1.f;
        if (nw) {
            ss = warp_sum(ss);
            scale = 1.0f / sqrtf(ss / (float)hd + eps);
        }
#pragma unroll
        for (int it = 0; it < 2; ++it) {
            const int i = 2 * lane + 64 * it;
            if (i < half) {
                float ra[2], rb[2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float x = a[it][e], y = b[it][e];
                    if (nw) {
                        x = x * scale * nw[i + e];
                        y = y * scale * nw[i + e + half];
                    }
                    const float sn = sn_tab[i + e], cs = cs_tab[i + e];
                    ra[e] = x * cs - y * sn;
                    rb[e] = y * cs + x * sn;
                }
                store2(dst + i, ra);
                store2(dst + i + half, rb);
            }
        }
        if (!is_q) {
            const T* vs = src + kv_dim;
            T* vd = dst + (int64_t)cache.kv_heads * cache.page_size * hd;
            for (int i = 2 * lane; i < hd; i += 64) copy2(vd + i, vs + i);
        }
        return;
    }

    float scale = 1.f;
    if (nw) {
        float ss = 0.f;
        for (int i = lane; i < hd; i += 32) {
            const float x = to_f32(src[i]);
            ss += x * x;
        }
        ss = warp_sum(ss);
        scale = 1.0f / sqrtf(ss / (float)hd + eps);
    }
    for (int i = lane; i < half; i += 32) {
        float a = to_f32(src[i]), b = to_f32(src[i + half]);
        if (nw) {
            a = a * scale * nw[i];
            b = b * scale * nw[i + half];
        }
        const float s = sn_tab[i], c = cs_tab[i];
        dst[i] = from_f32<T>(a * c - b * s);
        dst[i + half] = from_f32<T>(b * c + a * s);
    }
    for (int i = rot + lane; i < hd; i += 32) {
        float a = to_f32(src[i]);
        if (nw) a = a * scale * nw[i];
        dst[i] = from_f32<T>(a);
    }
    if (!is_q) {
        const T* vs = src + kv_dim;
        T* vd = dst + (int64_t)cache.kv_heads * cache.page_size * hd;
        for (int i = lane; i < hd; i += 32) vd[i] = vs[i];
    }
}


template <typename T>
__global__ void qk_norm_rope_kv_write_kernel(const T* __restrict__ qkv, const float* __restrict__ norm_q,
                                             const float* __restrict__ norm_k,
                                             const float* __restrict__ inv_freq, int rot, T* __restrict__ q_out,
                                             PagedCache cache, const int32_t* __restrict__ row_slot,
                                             const int32_t* __restrict__ row_pos, int n_rows, int q_heads,
                                             float eps, int write_kv, const float* __restrict__ rope_table,
                                             int table_positions) {
    extern __shared__ float rope_cs[];          // [warps][rot]: per warp, cosines then sines (only without a table)
    pdl_prologue();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int heads = q_heads + cache.kv_heads;
    const int64_t item = (int64_t)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= (int64_t)n_rows * heads) return;
    const int row = (int)(item / heads), head = (int)(item % heads);
    const int half = rot >> 1;
    const int pos = row_pos[row];
    // The row's cosines and sines: from the table the position encoding made at start-up
    // ([position][cos..., sin...]) when it covers the position, else computed here by the warp.
    const float* cs_tab;
    const float* sn_tab;
    if (rope_table != nullptr && pos >= 0 && pos < table_positions) {
        cs_tab = rope_table + (int64_t)pos * rot;
        sn_tab = cs_tab + half;
    } else {
        float* c = rope_cs + warp * rot;
        float* sn = c + half;
        for (int i = lane; i < half; i += 32) sincosf((float)pos * inv_freq[i], &sn[i], &c[i]);
        __syncwarp();
        cs_tab = c;
        sn_tab = sn;
    }
    rope_one_head<T>(qkv, norm_q, norm_k, rot, q_out, cache, row_slot, row, pos, head, q_heads, eps, write_kv, cs_tab, sn_tab);
}

// The same for the common shapes (whole head rotated, head_dim 32, 64, 128 or 256, a table for the
// row's position): head_dim / 16 lanes per head, each owning 8 consecutive values of the first half
// and the 8 they pair with, moved 16 bytes at a time; a warp serves 512 / head_dim heads at once.
template <typename T, int HD>
__global__ void qk_norm_rope_kv_write_vec_kernel(const T* __restrict__ qkv, const float* __restrict__ norm_q,
                                                 const float* __restrict__ norm_k, T* __restrict__ q_out,
                                                 PagedCache cache, const int32_t* __restrict__ row_slot,
                                                 const int32_t* __restrict__ row_pos, int n_rows, int q_heads, float eps,
                                                 int write_kv, const float* __restrict__ rope_table, int table_positions,
                                                 const float* __restrict__ inv_freq) {
    constexpr int LPH = HD / 16;        // lanes per head
    constexpr int HPW = 32 / LPH;       // heads per warp
    constexpr int HALF = HD / 2;
    // Positions, slots, the page table, the norm weights and the rotation table are older than any
    // kernel still running; only q|k|v comes from the kernel before this one.  So everything but
    // q|k|v is asked for before the wait: the end of the product is followed by one trip to memory.
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int heads = q_heads + cache.kv_heads;
    const int64_t item = ((int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5)) * HPW + lane / LPH;
    const bool live = item < (int64_t)n_rows * heads;
    const int row = live ? (int)(item / heads) : 0, head = live ? (int)(item % heads) : 0;
    const int c = (lane % LPH) * 8;     // this lane's values: c .. c + 7 and HALF + c .. HALF + c + 7
    const int q_dim = q_heads * HD, kv_dim = cache.kv_heads * HD;
    const bool is_q = head < q_heads;
    const int kh = is_q ? 0 : head - q_heads;
    const T* src = qkv + (int64_t)row * (q_dim + 2 * kv_dim) + (is_q ? head * HD : q_dim + kh * HD);
    const float* nw = is_q ? norm_q : norm_k;
    const int pos = row_pos[row];
    const bool writes = live && (is_q || write_kv);
    T* dst = nullptr;
    if (writes) {
        if (is_q) {
            dst = q_out + (int64_t)row * q_dim + head * HD;
        } else {
            const int64_t off = cache_row_offset(cache, row_slot[row], pos, kh, 0);
            if (off >= 0) dst = (T*)cache.base + off;
        }
    }
    float wa[8], wb[8], cs[8], sn[8];
    if (nw) {
        load8(nw + c, wa);
        load8(nw + HALF + c, wb);
    }
    if (pos >= 0 && pos < table_positions) {
        load8(rope_table + (int64_t)pos * HD + c, cs);
        load8(rope_table + (int64_t)pos * HD + HALF + c, sn);
    } else {        // a position the table does not cover
#pragma unroll
        for (int k = 0; k < 8; ++k) sincosf((float)pos * inv_freq[c + k], &sn[k], &cs[k]);
    }
    pdl_wait();
    float a[8], b[8];
    load8(src + c, a);
    load8(src + HALF + c, b);
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) ss += a[k] * a[k] + b[k] * b[k];
#pragma unroll
    for (int o = 1; o < LPH; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (dst == nullptr) return;
    if (nw) {
        const float scale = 1.0f / sqrtf(ss / (float)HD + eps);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            a[k] = a[k] * scale * wa[k];
            b[k] = b[k] * scale * wb[k];
        }
    }
    float ra[8], rb[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        ra[k] = a[k] * cs[k] - b[k] * sn[k];
        rb[k] = b[k] * cs[k] + a[k] * sn[k];
    }
    store8(dst + c, ra);
    store8(dst + HALF + c, rb);
    if (!is_q) {
        const T* vs = src + kv_dim;
        T* vd = dst + (int64_t)cache.kv_heads * cache.page_size * HD;
        copy16(vd + c, vs + c);
        copy16(vd + HALF + c, vs + HALF + c);
    }
}

template <typename T>
static int launch_rope_vec(const T* qkv, const float* norm_q, const float* norm_k, T* q_out, const PagedCache& cache,
                           const int32_t* row_slot, const int32_t* row_pos, int n_rows, int q_heads, float eps, int write_kv,
                           const float* rope_table, int table_positions, const float* inv_freq, cudaStream_t stream) {
    const int hd = cache.head_dim;
    const int64_t items = (int64_t)n_rows * (q_heads + cache.kv_heads);
    const int hpw = 32 / (hd / 16), warps = 4;
    const int64_t blocks = (items + (int64_t)hpw * warps - 1) / ((int64_t)hpw * warps);
    X0NE_REQUIRE(blocks <= 0x7fffffff, "rope: too many rows");
#define X0NE_ROPE_VEC(HDV)                                                                                             \
    x0ne_launch(qk_norm_rope_kv_write_vec_kernel<T, HDV>, dim3((unsigned)blocks), dim3(warps * 32), 0, stream, qkv, norm_q, \
                norm_k, q_out, cache, row_slot, row_pos, n_rows, q_heads, eps, write_kv, rope_table, table_positions, inv_freq)
    if (hd == 32) X0NE_ROPE_VEC(32);
    else if (hd == 64) X0NE_ROPE_VEC(64);
    else if (hd == 128) X0NE_ROPE_VEC(128);
    else X0NE_ROPE_VEC(256);
#undef X0NE_ROPE_VEC
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_qk_norm_rope_kv_write(const void* qkv, int dt, const float* norm_q, const float* norm_k,
                                        const float* inv_freq, int rotary_dim, void* q_out, PagedCache cache,
                                        const int32_t* row_slot, const int32_t* row_pos, int n_rows, int q_heads,
                                        float eps, int write_kv, const float* rope_table, int table_positions,
                                        cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && q_heads > 0 && cache.kv_heads > 0 && cache.head_dim > 0, "rope: bad sizes");
    X0NE_REQUIRE(rotary_dim >= 0 && rotary_dim % 2 == 0 && rotary_dim <= cache.head_dim,
                 "rope: rotary_dim %d must be even and at most head_dim %d", rotary_dim, cache.head_dim);
    X0NE_REQUIRE(rotary_dim == 0 || inv_freq != nullptr, "rope: no inv_freq table");
    if (n_rows == 0) return 0;
    const int hd_ = cache.head_dim;
    if (rope_table != nullptr && rotary_dim == hd_ && (hd_ == 32 || hd_ == 64 || hd_ == 128 || hd_ == 256) &&
        (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)cache.base | (uintptr_t)rope_table | (uintptr_t)norm_q |
          (uintptr_t)norm_k) & 15) == 0) {
        if (dt == X0NE_F32)
            return launch_rope_vec<float>((const float*)qkv, norm_q, norm_k, (float*)q_out, cache, row_slot, row_pos, n_rows,
                                          q_heads, eps, write_kv, rope_table, table_positions, inv_freq, stream);
        if (dt == X0NE_BF16)
            return launch_rope_vec<bf16>((const bf16*)qkv, norm_q, norm_k, (bf16*)q_out, cache, row_slot, row_pos, n_rows,
                                         q_heads, eps, write_kv, rope_table, table_positions, inv_freq, stream);
    }
    // one warp per (row, head)
    const int heads = q_heads + cache.kv_heads;
    const int warps = 4;
    const int64_t items = (int64_t)n_rows * heads;
    X0NE_REQUIRE((items + warps - 1) / warps <= 0x7fffffff, "rope: too many rows");
    const dim3 grid((unsigned)((items + warps - 1) / warps));
    const size_t smem = (size_t)warps * rotary_dim * sizeof(float);
    if (dt == X0NE_F32)
        x0ne_launch(qk_norm_rope_kv_write_kernel<float>, dim3(grid), dim3(warps * 32), smem, stream, 
            (const float*)qkv, norm_q, norm_k, inv_freq, rotary_dim, (float*)q_out, cache, row_slot, row_pos, n_rows,
            q_heads, eps, write_kv, rope_table, table_positions);
    else if (dt == X0NE_BF16)
        x0ne_launch(qk_norm_rope_kv_write_kernel<bf16>, dim3(grid), dim3(warps * 32), smem, stream, 
            (const bf16*)qkv, norm_q, norm_k, inv_freq, rotary_dim, (bf16*)q_out, cache, row_slot, row_pos, n_rows,
            q_heads, eps, write_kv, rope_table, table_positions);
    else
        X0NE_REQUIRE(false, "rope: unknown dtype tag %d", dt);
    X0NE_LAUNCH_CHECK();
}

// ----------------------------------------------------------------------------------------
// SwiGLU on the packed [gate; up] row: out[i] = T(g / (1 + expf(-g)) * u), g and u with `bias` (packed alike,
// float32) added first if it is given (x0ne-core/kernels/cuda/swiglu.cu:5-11).
// ----------------------------------------------------------------------------------------
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gate_up, const float* __restrict__ bias, T* __restrict__ out, int inter) {
    pdl_prologue();
    const int i = blockIdx.x * blockDim.x + threadIdx.x, r = blockIdx.y;
    if (i >= inter) return;
    const T* row = gate_up + (int64_t)r * 2 * inter;
    float g = to_f32(row[i]), u = to_f32(row[inter + i]);
    if (bias != nullptr) {
        g += bias[i];
        u += bias[inter + i];
    }
    out[(int64_t)r * inter + i] = from_f32<T>(g / (1.0f + expf(-g)) * u);
}

// 8 values per thread with 16-byte accesses (inter % 8 == 0 and aligned rows).
template <typename T>
__global__ void swiglu_vec_kernel(const T* __restrict__ gate_up, const float* __restrict__ bias, T* __restrict__ out, int inter, int64_t total8) {
    pdl_prologue();
    const int per_row = inter / 8;
    for (int64_t e = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; e < total8; e += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = e / per_row;
        const int i = (int)(e % per_row) * 8;
        const T* row = gate_up + r * 2 * inter;
        float g[8], u[8], o[8];
        load8(row + i, g);
        load8(row + inter + i, u);
        if (bias != nullptr) {
            float b[8], c[8];
            load8(bias + i, b);
            load8(bias + inter + i, c);
#pragma unroll
            for (int k = 0; k < 8; ++k) { g[k] += b[k]; u[k] += c[k]; }
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) o[k] = g[k] / (1.0f + expf(-g[k])) * u[k];
        store8(out + r * inter + i, o);
    }
}

X0NE_API int x0ne_swiglu(const void* gate_up, const float* bias, void* out, int dt, int n_rows, int inter, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && inter > 0, "swiglu: rows %d inter %d", n_rows, inter);
    if (n_rows == 0) return 0;
    X0NE_REQUIRE(n_rows <= 65535 * 1024, "swiglu: too many rows for one launch");
    const int esize = dt == X0NE_F32 ? 4 : 2;
    if (inter % 8 == 0 && (((uintptr_t)gate_up | (uintptr_t)bias | (uintptr_t)out) & 15) == 0 && ((int64_t)inter * esize) % 16 == 0) {
        const int64_t total8 = (int64_t)n_rows * (inter / 8);
        int64_t blocks = (total8 + 255) / 256;
        if (blocks > 148 * 16) blocks = 148 * 16;
        if (dt == X0NE_F32)
            x0ne_launch(swiglu_vec_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, (const float*)gate_up, bias, (float*)out, inter, total8);
        else if (dt == X0NE_BF16)
            x0ne_launch(swiglu_vec_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, stream, (const bf16*)gate_up, bias, (bf16*)out, inter, total8);
        else
            X0NE_REQUIRE(false, "swiglu: unknown dtype tag %d", dt);
        X0NE_LAUNCH_CHECK();
    }
    for (int r0 = 0; r0 < n_rows; r0 += 65535) {
        const int nr = n_rows - r0 < 65535 ? n_rows - r0 : 65535;
        dim3 grid((inter + 255) / 256, nr);
        if (dt == X0NE_F32)
            x0ne_launch(swiglu_kernel<float>, dim3(grid), dim3(256), 0, stream, (const float*)gate_up + (int64_t)r0 * 2 * inter, bias,
                        (float*)out + (int64_t)r0 * inter, inter);
        else if (dt == X0NE_BF16)
            x0ne_launch(swiglu_kernel<bf16>, dim3(grid), dim3(256), 0, stream, (const bf16*)gate_up + (int64_t)r0 * 2 * inter, bias,
                        (bf16*)out + (int64_t)r0 * inter, inter);
        else
            X0NE_REQUIRE(false, "swiglu: unknown dtype tag %d", dt);
    }
    X0NE_LAUNCH_CHECK();
}

// ----------------------------------------------------------------------------------------
// Embedding: resid[r] = f32(table[tokens[r]]); an id outside the table gives a zero row
// (x0ne-core/kernels/cuda/embedding.cu:5-17).  The engine there copies the row and lets the
// first add-norm add it to a zeroed residual (x0ne-core/runtime/src/engine.rs:744-745); here
// the row is written straight into the float32 residual, which is the same value.
// ----------------------------------------------------------------------------------------
template <typename T>
__global__ void embedding_kernel(const T* __restrict__ table, const int32_t* __restrict__ tokens,
                                 float* __restrict__ resid, int hidden, int vocab, float scale) {
    pdl_prologue();
    const int row = blockIdx.x;
    const int t = tokens[row];
    float* dst = resid + (int64_t)row * hidden;
    if (t < 0 || t >= vocab) {
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = 0.f;
        return;
    }
    const T* src = table + (int64_t)t * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = to_f32(src[i]) * scale;
}

// The same with 16-byte accesses (hidden % 8 == 0, aligned rows): all of a row's loads are in flight
// at once, where the loop above waits for memory once per 256 values (9.5 us for 8 rows of 4,096).
template <typename T>
__global__ void embedding_vec_kernel(const T* __restrict__ table, const int32_t* __restrict__ tokens,
                                     float* __restrict__ resid, int hidden, int vocab, float scale) {
    pdl_prologue();
    const int row = blockIdx.x;
    const int t = tokens[row];
    float* dst = resid + (int64_t)row * hidden;
    const bool none = t < 0 || t >= vocab;
    const T* src = table + (int64_t)(none ? 0 : t) * hidden;
    for (int i0 = threadIdx.x * 8; i0 < hidden; i0 += 4 * blockDim.x * 8) {
        float v[4][8];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int i = i0 + u * blockDim.x * 8;
            if (i < hidden && !none) load8(src + i, v[u]);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int i = i0 + u * blockDim.x * 8;
            if (i < hidden) {
#pragma unroll
                for (int k = 0; k < 8; ++k) v[u][k] = none ? 0.f : v[u][k] * scale;
                store8(dst + i, v[u]);
            }
        }
    }
}

// `scale` multiplies every value in float32 (1: the row itself, the same bits).
X0NE_API int x0ne_embedding(const void* table, int dt, const int32_t* tokens, float* resid, int n_rows,
                            int hidden, int vocab, float scale, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && hidden > 0 && vocab > 0, "embedding: rows %d hidden %d vocab %d", n_rows, hidden, vocab);
    if (n_rows == 0) return 0;
    const int block = hidden >= 1024 ? 256 : 128;
    if (hidden % 8 == 0 && (((uintptr_t)table | (uintptr_t)resid) & 15) == 0 && (dt == X0NE_F32 || dt == X0NE_BF16)) {
        const int threads = hidden / 8 >= 256 ? 256 : (hidden / 8 + 31) / 32 * 32;
        if (dt == X0NE_F32)
            x0ne_launch(embedding_vec_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, (const float*)table, tokens, resid, hidden, vocab, scale);
        else
            x0ne_launch(embedding_vec_kernel<bf16>, dim3(n_rows), dim3(threads), 0, stream, (const bf16*)table, tokens, resid, hidden, vocab, scale);
        X0NE_LAUNCH_CHECK();
    }
    if (dt == X0NE_F32)
        x0ne_launch(embedding_kernel<float>, dim3(n_rows), dim3(block), 0, stream, (const float*)table, tokens, resid, hidden, vocab, scale);
    else if (dt == X0NE_BF16)
        x0ne_launch(embedding_kernel<bf16>, dim3(n_rows), dim3(block), 0, stream, (const bf16*)table, tokens, resid, hidden, vocab, scale);
    else
        X0NE_REQUIRE(false, "embedding: unknown dtype tag %d", dt);
    X0NE_LAUNCH_CHECK();
}


// ----------------------------------------------------------------------------------------
// The start of a pass over a run of layers that a model repeats:
//   resid[r] = ((resid[r] + delta[r]) + scale * table[token[r]]) + step[c]
// in float32, one IEEE add after the other.  `delta` (the pending result of the layer before) and the
// embedding term (`table` null: not added) are optional; `step` is one vector of the pass.
// ----------------------------------------------------------------------------------------
template <typename T, typename E>
__global__ void open_pass_kernel(float* __restrict__ resid, const T* __restrict__ delta, const E* __restrict__ table,
                                 const int32_t* __restrict__ tokens, float scale, const float* __restrict__ step, int hidden, int vocab) {
    pdl_prologue();
    const int row = blockIdx.x;
    float* r = resid + (int64_t)row * hidden;
    const int t = table != nullptr ? tokens[row] : -1;
    const E* e = (table != nullptr && t >= 0 && t < vocab) ? table + (int64_t)t * hidden : nullptr;
    const T* d = delta != nullptr ? delta + (int64_t)row * hidden : nullptr;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = r[i];
        if (d != nullptr) v = v + to_f32(d[i]);
        if (e != nullptr) v = v + to_f32(e[i]) * scale;
        if (step != nullptr) v = v + step[i];
        r[i] = v;
    }
}

X0NE_API int x0ne_open_pass(float* resid, const void* delta, int dt, const void* table, int table_dt, const int32_t* tokens, float scale,
                            const float* step, int n_rows, int hidden, int vocab, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && hidden > 0 && (table == nullptr || (tokens != nullptr && vocab > 0)), "open_pass: rows %d hidden %d", n_rows, hidden);
    X0NE_REQUIRE((dt == X0NE_F32 || dt == X0NE_BF16) && (table_dt == X0NE_F32 || table_dt == X0NE_BF16), "open_pass: unknown dtype tag");
    if (n_rows == 0) return 0;
    const int block = hidden >= 256 ? 256 : (hidden + 31) / 32 * 32;
#define X0NE_OPEN(T, E) x0ne_launch(open_pass_kernel<T, E>, dim3(n_rows), dim3(block), 0, stream, resid, (const T*)delta, (const E*)table, tokens, scale, step, hidden, vocab)
    if (dt == X0NE_F32 && table_dt == X0NE_F32) X0NE_OPEN(float, float);
    else if (dt == X0NE_F32) X0NE_OPEN(float, bf16);
    else if (table_dt == X0NE_F32) X0NE_OPEN(bf16, float);
    else X0NE_OPEN(bf16, bf16);
#undef X0NE_OPEN
    X0NE_LAUNCH_CHECK();
}

// ----------------------------------------------------------------------------------------
// Embedding as a sum of up to three rows, added in float32 in this order:
//   table[token] + pairs[(prev * mul_prev + token * mul_cur) mod buckets] + positions[pos]
// The pair row of a sequence's first token (pos 0) is number `buckets`, the last one.  The token before a row is the row
// above's where that continues the same sequence in this pass, else the one the sequence's state keeps; the block of the
// first row a sequence brings reads that and leaves the sequence's last token of the pass there (one int32 per slot,
// `state_stride` apart; no other block touches it).  `pairs` and `positions` may be null; `copy`, if given, receives the
// rows too (what later stages of the model call the embedding output).
// ----------------------------------------------------------------------------------------
struct EmbedSumArgs {
    const void* table;
    const void* pairs;
    const void* positions;
    const int32_t* tokens;
    const int32_t* row_slot;
    const int32_t* row_pos;
    const int32_t* seq_first_row;
    int32_t* last_token;            // per slot (null without `pairs`)
    int64_t state_stride;
    float* resid;
    float* copy;
    int64_t mul_prev, mul_cur, buckets;
    int32_t n_seqs, hidden, vocab, n_positions;
};

template <typename T, bool VEC>
__global__ void embed_sum_kernel(EmbedSumArgs a) {
    __shared__ int prev_s;
    pdl_prologue();
    const int row = blockIdx.x, slot = a.row_slot[row], pos = a.row_pos[row], t = a.tokens[row];
    int64_t pair = a.buckets;
    if (a.pairs != nullptr) {
        const bool above = row > 0 && slot >= 0 && a.row_slot[row - 1] == slot && a.row_pos[row - 1] == pos - 1;
        int prev = 0;
        if (above) {
            prev = a.tokens[row - 1];
        } else if (slot >= 0) {             // (the same for every thread of the block)
            if (threadIdx.x == 0) {
                int32_t* kept = a.last_token + (int64_t)slot * a.state_stride;
                prev_s = *kept;
                int lo = 0, hi = a.n_seqs - 1;          // the sequence whose first row this is: first rows ascend
                while (lo < hi) {
                    const int mid = (lo + hi + 1) / 2;
                    if (a.seq_first_row[mid] <= row) lo = mid; else hi = mid - 1;
                }
                *kept = a.tokens[a.seq_first_row[lo + 1] - 1];
            }
            __syncthreads();
            prev = prev_s;
        }
        if (pos > 0) {
            int64_t b = ((int64_t)prev * a.mul_prev + (int64_t)t * a.mul_cur) % a.buckets;
            pair = b < 0 ? b + a.buckets : b;
        }
    }
    const bool none = t < 0 || t >= a.vocab;
    const T* e = (const T*)a.table + (int64_t)(none ? 0 : t) * a.hidden;
    const T* g = a.pairs != nullptr ? (const T*)a.pairs + pair * a.hidden : nullptr;
    const T* p = a.positions != nullptr && pos >= 0 && pos < a.n_positions ? (const T*)a.positions + (int64_t)pos * a.hidden : nullptr;
    float* dst = a.resid + (int64_t)row * a.hidden;
    float* cp = a.copy != nullptr ? a.copy + (int64_t)row * a.hidden : nullptr;
    if (VEC) {
        for (int i = threadIdx.x * 8; i < a.hidden; i += blockDim.x * 8) {
            float v[8], x[8], y[8];
            load8(e + i, v);
            if (g != nullptr) load8(g + i, x);
            if (p != nullptr) load8(p + i, y);
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                if (none) v[k] = 0.f;
                if (g != nullptr) v[k] += x[k];
                if (p != nullptr) v[k] += y[k];
            }
            store8(dst + i, v);
            if (cp != nullptr) store8(cp + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {
            float v = none ? 0.f : to_f32(e[i]);
            if (g != nullptr) v += to_f32(g[i]);
            if (p != nullptr) v += to_f32(p[i]);
            dst[i] = v;
            if (cp != nullptr) cp[i] = v;
        }
    }
}

X0NE_API int x0ne_embed_sum(EmbedSumArgs a, int dt, int n_rows, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && a.hidden > 0 && a.vocab > 0 && a.n_seqs >= 0, "embed_sum: rows %d hidden %d vocab %d", n_rows, a.hidden, a.vocab);
    X0NE_REQUIRE(a.pairs == nullptr || (a.buckets > 0 && a.last_token != nullptr && a.seq_first_row != nullptr && a.n_seqs > 0), "embed_sum: pair rows need buckets, the sequences' last tokens and their rows");
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "embed_sum: unknown dtype tag %d", dt);
    if (n_rows == 0) return 0;
    const bool vec = a.hidden % 8 == 0 && (((uintptr_t)a.table | (uintptr_t)a.pairs | (uintptr_t)a.positions | (uintptr_t)a.resid | (uintptr_t)a.copy) & 15) == 0;
    const int work = vec ? a.hidden / 8 : a.hidden;
    const int threads = work >= 256 ? 256 : (work + 31) / 32 * 32;
#define X0NE_ES(T, V) x0ne_launch(embed_sum_kernel<T, V>, dim3(n_rows), dim3(threads), 0, stream, a)
    if (dt == X0NE_F32) { if (vec) X0NE_ES(float, true); else X0NE_ES(float, false); }
    else { if (vec) X0NE_ES(bf16, true); else X0NE_ES(bf16, false); }
#undef X0NE_ES
    X0NE_LAUNCH_CHECK();
}

// ----------------------------------------------------------------------------------------
// The operand of a product over two concatenated rows:  out[r] = [ x | x0[r] ]  with
//   x = resid[r] + norm(delta[r] + bias_d) * w_d      (delta null: resid alone; w_d null: delta added as it is)
// in float32, rounded once to the activation type.  The residual is only read (the product's result replaces it).
// One block per row; the sum of squares is a fixed-order block sum.
// ----------------------------------------------------------------------------------------
template <typename T>
__global__ void concat_rows_kernel(const float* __restrict__ resid, const T* __restrict__ delta, const float* __restrict__ bias_d,
                                   const float* __restrict__ w_d, float eps_d, const float* __restrict__ x0, T* __restrict__ out, int hidden) {
    __shared__ float sh[32];
    pdl_prologue();
    const int64_t row = blockIdx.x;
    const float* r = resid + row * hidden;
    const float* z = x0 + row * hidden;
    const T* d = delta != nullptr ? delta + row * hidden : nullptr;
    T* o = out + row * 2 * hidden;
    float scale = 1.f;
    if (d != nullptr && w_d != nullptr) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            const float v = to_f32(d[i]) + (bias_d != nullptr ? bias_d[i] : 0.f);
            ss = fmaf(v, v, ss);
        }
        scale = 1.0f / sqrtf(block_sum(ss, sh) / (float)hidden + eps_d);
    }
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = r[i];
        if (d != nullptr) v += (to_f32(d[i]) + (bias_d != nullptr ? bias_d[i] : 0.f)) * scale * (w_d != nullptr ? w_d[i] : 1.f);
        o[i] = from_f32<T>(v);
        o[hidden + i] = from_f32<T>(z[i]);
    }
}

X0NE_API int x0ne_concat_rows(const float* resid, const void* delta, int dt, const float* bias_d, const float* w_d, float eps_d, const float* x0,
                              void* out, int n_rows, int hidden, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && hidden > 0 && resid != nullptr && x0 != nullptr && out != nullptr, "concat_rows: rows %d hidden %d", n_rows, hidden);
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "concat_rows: unknown dtype tag %d", dt);
    if (n_rows == 0) return 0;
    const int block = hidden >= 512 ? 512 : (hidden + 31) / 32 * 32;
    if (dt == X0NE_F32)
        x0ne_launch(concat_rows_kernel<float>, dim3(n_rows), dim3(block), 0, stream, resid, (const float*)delta, bias_d, w_d, eps_d, x0, (float*)out, hidden);
    else
        x0ne_launch(concat_rows_kernel<bf16>, dim3(n_rows), dim3(block), 0, stream, resid, (const bf16*)delta, bias_d, w_d, eps_d, x0, (bf16*)out, hidden);
    X0NE_LAUNCH_CHECK();
}
