// Residual add and norm where either norm may subtract the mean (layer norm):
//   x = delta + bias_d (null: none);  d = (x - m(x)) / sqrt(mean((x - m(x))^2) + eps_d) * w_d    (w_d null: d = x as it is)
//   r = resid + d, stored back (delta null: r = resid);  out = T((r - m(r)) / sqrt(mean((r - m(r))^2) + eps) * w)
// with m(.) the mean where a norm is centred and 0 where it is not (RMS norm).  `rows` gathers source rows.  Everything is
// float32, d is never rounded; the sum of squared deviations is taken around the mean itself.  One block per row.
#include "common.cuh"

#define LN_MAX_WARPS 16

// Mean and mean squared deviation of a row whose values lie in the threads' registers (`count` of a thread's N, `total` in all).
// A warp's mean comes first, then its deviations from that; the warps' parts (count, mean, deviations) meet in shared memory,
// where every warp adds them up, one part per lane: deviations from the row's mean are those from the warp's plus count times the
// square of the means' difference.  `parts` must not be in use.
struct LnStats {
    float mean, dev2;           // dev2: mean squared deviation from the mean
};
template <int N>
__device__ __forceinline__ LnStats ln_stats(const float (&x)[N], int count, int warp_count, float4* parts, int total) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (i < count) s += x[i];
    const float n = (float)warp_count;
    const float mean_w = warp_count > 0 ? warp_sum(s) / n : 0.f;
    float d2 = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (i < count) {
            const float d = x[i] - mean_w;
            d2 = fmaf(d, d, d2);
        }
    d2 = warp_sum(d2);
    if (lane == 0) parts[warp] = make_float4(n, mean_w, d2, 0.f);
    __syncthreads();
    const float4 p = lane < (int)(blockDim.x >> 5) ? parts[lane] : make_float4(0.f, 0.f, 0.f, 0.f);
    const float mean = warp_sum(p.x * p.y) / (float)total;
    const float d = p.y - mean, dev = warp_sum(fmaf(p.x * d, d, p.z));
    return {mean, dev / (float)total};
}
// what is taken off, and what the rest is multiplied by
__device__ __forceinline__ void ln_factors(const LnStats& s, int centred, float eps, float& off, float& scale) {
    off = centred ? s.mean : 0.f;
    scale = 1.0f / sqrtf((centred ? s.dev2 : fmaf(s.mean, s.mean, s.dev2)) + eps);
}

struct LnArgs {
    float* resid;
    const void* delta;
    const float* bias_d;
    const float* w_d;
    const float* w;
    const int32_t* rows;
    float eps_d, eps;
    int32_t centred_d, centred, hidden;
};

__device__ __forceinline__ void ln_load8(const float* p, float* v) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ln_load8(const bf16* p, float* v) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void ln_store8(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void ln_store8(bf16* p, const float* v) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = u;
}

// hidden % 8 == 0, 8 values per thread and sweep, 16-byte aligned rows: row and delta stay in registers; EARLY: weights are asked
// for before the wait for the kernel before.
template <typename T, int ITS, bool EARLY>
__global__ void __launch_bounds__(512) add_norm_vec_kernel(LnArgs a, T* __restrict__ out) {
    __shared__ float4 parts[2][LN_MAX_WARPS];
    pdl_launch_dependents();
    const int64_t src = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
    const int H = a.hidden;
    float wd[EARLY ? 8 : 1], w[EARLY ? 8 : 1], bd[EARLY ? 8 : 1];
    int count = 0, warp_count = 0;              // values of this thread, and of its warp
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int at = it * (int)blockDim.x * 8, of_warp = H - at - (int)(threadIdx.x & ~31u) * 8;
        count += at + (int)threadIdx.x * 8 < H ? 8 : 0;
        warp_count += min(max(of_warp, 0), 256);
    }
    if (EARLY && count) {
        ln_load8(a.w + threadIdx.x * 8, w);
        if (a.w_d) ln_load8(a.w_d + threadIdx.x * 8, wd);
        if (a.bias_d) ln_load8(a.bias_d + threadIdx.x * 8, bd);
    }
    pdl_wait();
    float* r = a.resid + src * H;
    const T* d = a.delta ? (const T*)a.delta + src * H : nullptr;
    T* o = out + (int64_t)blockIdx.x * H;
    float v[ITS * 8], x[ITS * 8];
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < H) {
            ln_load8(r + i, v + it * 8);
            if (d) ln_load8(d + i, x + it * 8);
        }
    }
    if (d) {
        if (a.bias_d) {
#pragma unroll
            for (int it = 0; it < ITS; ++it) {
                const int i = (it * blockDim.x + threadIdx.x) * 8;
                if (i < H) {
                    float late[8];
                    if (!EARLY) ln_load8(a.bias_d + i, late);
#pragma unroll
                    for (int k = 0; k < 8; ++k) x[it * 8 + k] += EARLY ? bd[EARLY ? k : 0] : late[k];
                }
            }
        }
        if (a.w_d) {
            float off, scale;
            ln_factors(ln_stats(x, count, warp_count, parts[0], H), a.centred_d, a.eps_d, off, scale);
#pragma unroll
            for (int it = 0; it < ITS; ++it) {
                const int i = (it * blockDim.x + threadIdx.x) * 8;
                if (i < H) {
                    float late[8];
                    if (!EARLY) ln_load8(a.w_d + i, late);
#pragma unroll
                    for (int k = 0; k < 8; ++k) x[it * 8 + k] = (x[it * 8 + k] - off) * scale * (EARLY ? wd[EARLY ? k : 0] : late[k]);
                }
            }
        }
#pragma unroll
        for (int it = 0; it < ITS; ++it) {
            const int i = (it * blockDim.x + threadIdx.x) * 8;
            if (i < H) {
#pragma unroll
                for (int k = 0; k < 8; ++k) v[it * 8 + k] += x[it * 8 + k];
                ln_store8(r + i, v + it * 8);
            }
        }
    }
    float off, scale;
    ln_factors(ln_stats(v, count, warp_count, parts[1], H), a.centred, a.eps, off, scale);
#pragma unroll
    for (int it = 0; it < ITS; ++it) {
        const int i = (it * blockDim.x + threadIdx.x) * 8;
        if (i < H) {
            float late[8], y[8];
            if (!EARLY) ln_load8(a.w + i, late);
#pragma unroll
            for (int k = 0; k < 8; ++k) y[k] = (v[it * 8 + k] - off) * scale * (EARLY ? w[EARLY ? k : 0] : late[k]);
            ln_store8(o + i, y);
        }
    }
}

// Any width: rows are read again for every sweep (each thread reads back only what it wrote itself).
template <typename T, typename F>
__device__ __forceinline__ void ln_sweep_factors(F value, int H, float* sh, int centred, float eps, float& off, float& scale) {
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) s += value(i);
    const float mean = block_sum(s, sh) / (float)H;
    float d2 = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float d = value(i) - mean;
        d2 = fmaf(d, d, d2);
    }
    const LnStats st = {mean, block_sum(d2, sh) / (float)H};
    ln_factors(st, centred, eps, off, scale);
}

template <typename T>
__global__ void __launch_bounds__(256) add_norm_any_kernel(LnArgs a, T* __restrict__ out) {
    __shared__ float sh[32];
    pdl_prologue();
    const int64_t src = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
    const int H = a.hidden;
    float* r = a.resid + src * H;
    const T* d = a.delta ? (const T*)a.delta + src * H : nullptr;
    if (d) {
        auto value = [&](int i) { return to_f32(d[i]) + (a.bias_d ? a.bias_d[i] : 0.f); };
        float off = 0.f, scale = 1.f;
        if (a.w_d) ln_sweep_factors<T>(value, H, sh, a.centred_d, a.eps_d, off, scale);
        for (int i = threadIdx.x; i < H; i += blockDim.x) r[i] += a.w_d ? (value(i) - off) * scale * a.w_d[i] : value(i);
    }
    float off, scale;
    ln_sweep_factors<T>([&](int i) { return r[i]; }, H, sh, a.centred, a.eps, off, scale);
    T* o = out + (int64_t)blockIdx.x * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = from_f32<T>((r[i] - off) * scale * a.w[i]);
}

X0NE_API int x0ne_add_norm(LnArgs a, void* out, int dt, int n_rows, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && a.hidden > 0 && a.resid != nullptr && a.w != nullptr && (a.delta != nullptr || (a.w_d == nullptr && a.bias_d == nullptr)),
                 "add_norm: rows %d width %d", n_rows, a.hidden);
    X0NE_REQUIRE(dt == X0NE_F32 || dt == X0NE_BF16, "add_norm: unknown dtype tag %d", dt);
    if (n_rows == 0) return 0;
    const int H = a.hidden;
    if (H % 8 == 0 && H <= 8 * 1024 &&
        ((((uintptr_t)a.resid | (uintptr_t)a.delta | (uintptr_t)a.bias_d | (uintptr_t)a.w_d | (uintptr_t)a.w | (uintptr_t)out) & 15) == 0)) {
        const int pieces = H / 8;
        const bool two = pieces > 512;                      // two sweeps of 512 rather than one of 1,024
        int threads = two ? ((pieces + 1) / 2 + 31) / 32 * 32 : (pieces + 31) / 32 * 32;
        // few rows: the weights are asked for before the wait; many rows: fewer registers, so more rows in flight
        const bool early = !two && n_rows <= 256;
#define LN_VEC(T, ITS, EARLY) x0ne_launch(add_norm_vec_kernel<T, ITS, EARLY>, dim3(n_rows), dim3(threads), 0, stream, a, (T*)out)
#define LN_SWEEPS(T)                          \
    do {                                      \
        if (two) LN_VEC(T, 2, false);         \
        else if (early) LN_VEC(T, 1, true);   \
        else LN_VEC(T, 1, false);             \
    } while (0)
        if (dt == X0NE_F32) LN_SWEEPS(float);
        else LN_SWEEPS(bf16);
#undef LN_SWEEPS
#undef LN_VEC
        X0NE_LAUNCH_CHECK();
    }
    if (dt == X0NE_F32) x0ne_launch(add_norm_any_kernel<float>, dim3(n_rows), dim3(256), 0, stream, a, (float*)out);
    else x0ne_launch(add_norm_any_kernel<bf16>, dim3(n_rows), dim3(256), 0, stream, a, (bf16*)out);
    X0NE_LAUNCH_CHECK();
}
