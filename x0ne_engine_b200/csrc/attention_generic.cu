// Attention over the paged cache, any head size, any window: the plain kernel.
//
// It serves the 32-bit path for prefill and decode alike, and the bfloat16 path for shapes the
// tensor-core kernels do not take.  One warp per (query row, q head).  The query at position p
// of sequence slot s reads keys max(0, p - window + 1) .. p of that slot (causal by loop bound,
// no mask matrix: x0ne-core/kernels/cuda/attention.cu:21,28,102-103); q head h reads kv head
// h / (q_heads / kv_heads) (attention.cu:20).  Online softmax in float32
// (attention.cu:44-59,138-157): running max m, sum l, p_j = expf(s_j - m_new),
// alpha = expf(m - m_new), acc = acc * alpha + sum p_j v_j, out = acc / l.
//
// The order of every sum depends only on the query's position and the window: keys are taken
// in tiles of 32 starting at the first visible key, lane t owns key t of the tile, each score
// is one sequential dot product, the tile's sum is an xor-shuffle tree, and the values are
// accumulated key by key.  So the same query gives the same bits whether it arrives in a
// prompt, in a later chunk, alone or in a batch.
#include "common.cuh"

//
// Beyond that (`AttnExtra`): a chunked mask (the query sees its own chunk of positions only), a
// value width other than the keys', values read out of the key rows, a per-head sink in the
// denominator, a sigmoid gate on the output (per (row, head), or per value), a per-head slope times the
// distance i - j taken off every score, and first keys that stay visible
// whatever the window (they are taken first, in tiles of 32 from key 0, then the window's), and results written as float32
// for a caller that goes on in 32-bit; or, instead of the softmax, weights sigmoid(score + a number per head) that nothing
// normalises, results multiplied by a factor and written to rows wider than the heads.  With none of them asked for the
// operations and their order are the ones above.

#define ATT_MAX_I 16  // value width <= 32 * ATT_MAX_I

template <typename T>
__global__ void attention_rows_kernel(const T* __restrict__ q, T* __restrict__ out, PagedCache cache,
                                      const int32_t* __restrict__ row_slot, const int32_t* __restrict__ row_pos,
                                      int n_rows, int q_heads, float scale, int window, AttnExtra ex) {
    extern __shared__ float smem[];
    pdl_prologue();
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const int hd = cache.head_dim;
    const int vd = ex.v_from_k > 0 ? ex.v_from_k : cache_v_dim(cache);
    const int64_t item = (int64_t)blockIdx.x * (blockDim.x >> 5) + w;
    if (item >= (int64_t)n_rows * q_heads) return;
    const int row = (int)(item / q_heads), head = (int)(item % q_heads);
    const int kh = head / (q_heads / cache.kv_heads);
    const int pos = row_pos[row], slot = row_slot[row];
    float* qs = smem + w * hd;
    const float slope = ex.slope != nullptr ? ex.slope[head] : 0.f;
    const float sig_b = ex.sig_bias != nullptr ? ex.sig_bias[head] : 0.f;
    const T* qr = q + (int64_t)row * (ex.q_ld > 0 ? ex.q_ld : (int64_t)q_heads * hd) + (int64_t)head * hd;
    for (int d = lane; d < hd; d += 32) qs[d] = to_f32(qr[d]) * scale;
    __syncwarp();

    int j_lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (ex.chunk > 0) j_lo = max(j_lo, pos - pos % ex.chunk);
    const int64_t v_plane = (int64_t)cache.kv_heads * cache.page_size * hd;
    const T* base = (const T*)cache.base;
    float m = -INFINITY, l = 0.f;
    float acc[ATT_MAX_I];
#pragma unroll
    for (int i = 0; i < ATT_MAX_I; ++i) acc[i] = 0.f;

    // the kept first keys that lie before the window (tiles of 32 from key 0), then the window's keys
    const int kept = min(ex.keep_first, j_lo);
    for (int seg = kept > 0 ? 0 : 1; seg < 2; ++seg) {
    const int j_end = seg == 0 ? kept - 1 : pos;
    for (int j0 = seg == 0 ? 0 : j_lo; j0 <= j_end; j0 += 32) {
        const int j = j0 + lane;
        int64_t off = -1;
        float s = -INFINITY;
        if (j <= j_end) {
            off = cache_row_offset(cache, slot, j, kh, 0);
            if (off >= 0) {
                const T* kr = base + off;
                float a = 0.f;
                for (int d = 0; d < hd; ++d) a = fmaf(qs[d], to_f32(kr[d]), a);
                s = ex.slope != nullptr ? a - slope * (float)(pos - j) : a;
            }
        }
        float p, m_new = m;
        if (ex.sig_bias != nullptr) {
            p = off >= 0 ? 1.0f / (1.0f + expf(-(s + sig_b))) : 0.f;
        } else {
            m_new = fmaxf(m, warp_max(s));
            if (m_new == -INFINITY) continue;  // no readable key in this tile
            p = off >= 0 ? expf(s - m_new) : 0.f;
            const float alpha = expf(m - m_new);
            l = l * alpha + warp_sum(p);
#pragma unroll
            for (int i = 0; i < ATT_MAX_I; ++i) acc[i] *= alpha;
        }
        const int nt = min(32, j_end - j0 + 1);
        for (int t = 0; t < nt; ++t) {
            const float pt = __shfl_sync(0xffffffffu, p, t);
            const long long ot = __shfl_sync(0xffffffffu, (long long)off, t);
            if (ot < 0) continue;
            // the value row of the same position: the key row itself, or the row of the value plane
            const T* vr = ex.v_from_k > 0 ? base + ot
                                          : base + (ot - ot % cache.page_stride) + v_plane + ((ot % cache.page_stride) / hd) * vd;
#pragma unroll
            for (int i = 0; i < ATT_MAX_I; ++i) {
                const int d = lane + 32 * i;
                if (d < vd) acc[i] = fmaf(pt, to_f32(vr[d]), acc[i]);
            }
        }
        m = m_new;
    }
    }
    if (ex.sink != nullptr && slot >= 0 && ex.sig_bias == nullptr) {
        const float sk = ex.sink[head];
        const float m_new = fmaxf(m, sk);
        const float alpha = expf(m - m_new);
        l = l * alpha + expf(sk - m_new);
#pragma unroll
        for (int i = 0; i < ATT_MAX_I; ++i) acc[i] *= alpha;
    }
    const int64_t o0 = (int64_t)row * (ex.out_ld > 0 ? ex.out_ld : (int64_t)q_heads * vd) + ex.out_col + (int64_t)head * vd;
    T* o = out + o0;
    float* of = ex.out_f32 > 0 ? reinterpret_cast<float*>(out) + o0 : nullptr;
    float inv = ex.sig_bias != nullptr ? 1.f : l > 0.f ? 1.0f / l : 0.f;      // a row with no readable key (a padding row) gets zeros
    if (ex.out_scale != 0.f) inv *= ex.out_scale;
    if (ex.gate != nullptr && ex.gate_wide <= 0) inv *= 1.0f / (1.0f + expf(-to_f32(((const T*)ex.gate)[(int64_t)row * ex.gate_ld + head])));
    const T* gw = ex.gate != nullptr && ex.gate_wide > 0 ? (const T*)ex.gate + (int64_t)row * ex.gate_ld + (int64_t)head * vd : nullptr;
#pragma unroll
    for (int i = 0; i < ATT_MAX_I; ++i) {
        const int d = lane + 32 * i;
        if (d < vd) {
            const float r = gw != nullptr ? acc[i] * inv * (1.0f / (1.0f + expf(-to_f32(gw[d])))) : acc[i] * inv;
            if (of != nullptr) of[d] = r;
            else o[d] = from_f32<T>(r);
        }
    }
}

X0NE_API int x0ne_attention_rows_ex(const void* q, void* out, int dt, PagedCache cache, const int32_t* row_slot,
                                    const int32_t* row_pos, int n_rows, int q_heads, float scale, int window,
                                    AttnExtra ex, cudaStream_t stream) {
    X0NE_REQUIRE(n_rows >= 0 && q_heads > 0 && cache.kv_heads > 0 && q_heads % cache.kv_heads == 0,
                 "attention: %d q heads over %d kv heads", q_heads, cache.kv_heads);
    const int vd = ex.v_from_k > 0 ? ex.v_from_k : cache_v_dim(cache);
    X0NE_REQUIRE(cache.head_dim > 0 && cache.head_dim <= 2048 && vd > 0 && vd <= 32 * ATT_MAX_I && ex.v_from_k <= cache.head_dim,
                 "attention: keys of %d and values of %d are beyond the plain kernel's limits of 2048 and %d", cache.head_dim, vd, 32 * ATT_MAX_I);
    X0NE_REQUIRE(window >= 0 && ex.chunk >= 0 && ex.keep_first >= 0, "attention: negative window, chunk or count of kept keys");
    if (n_rows == 0) return 0;
    const int warps = 4;
    const int64_t items = (int64_t)n_rows * q_heads;
    const unsigned grid = (unsigned)((items + warps - 1) / warps);
    const size_t smem = (size_t)warps * cache.head_dim * sizeof(float);
    if (dt == X0NE_F32)
        x0ne_launch(attention_rows_kernel<float>, dim3(grid), dim3(warps * 32), smem, stream, (const float*)q, (float*)out, cache, row_slot,
                                                                       row_pos, n_rows, q_heads, scale, window, ex);
    else if (dt == X0NE_BF16)
        x0ne_launch(attention_rows_kernel<bf16>, dim3(grid), dim3(warps * 32), smem, stream, (const bf16*)q, (bf16*)out, cache, row_slot,
                                                                      row_pos, n_rows, q_heads, scale, window, ex);
    else
        X0NE_REQUIRE(false, "attention: unknown dtype tag %d", dt);
    X0NE_LAUNCH_CHECK();
}

X0NE_API int x0ne_attention_rows(const void* q, void* out, int dt, PagedCache cache, const int32_t* row_slot,
                                 const int32_t* row_pos, int n_rows, int q_heads, float scale, int window,
                                 cudaStream_t stream) {
    AttnExtra none = {};
    return x0ne_attention_rows_ex(q, out, dt, cache, row_slot, row_pos, n_rows, q_heads, scale, window, none, stream);
}
