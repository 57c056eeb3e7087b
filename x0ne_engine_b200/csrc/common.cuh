// Shared device and host helpers of every kernel file.
//
// Conventions (the same as x0ne-core/kernels/cuda/x0ne_kernels.h:1-3 states for its
// kernels): C linkage for every entry point, row-major tensors, 32-bit accumulation,
// token ids / positions / slots read from device memory, and every index checked without
// trapping: an id outside the vocabulary gives a zero row, a position with no page writes
// nothing.  Reductions run in a fixed order, so a row's result does not depend on what else
// is in the launch (x0ne-core/kernels/cuda/common.cuh:1,24-44).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

typedef __nv_bfloat16 bf16;

#define X0NE_API extern "C" __attribute__((visibility("default")))

// dtype tags of the C interface
#define X0NE_F32 0
#define X0NE_BF16 1

// Error codes of the C interface (0 = ok; positive values below 10000 are cudaError_t).
#define X0NE_ERR_ARG 10001

void x0ne_set_error(const char* fmt, ...);

#define X0NE_REQUIRE(cond, ...)            \
    do {                                   \
        if (!(cond)) {                     \
            x0ne_set_error(__VA_ARGS__);   \
            return X0NE_ERR_ARG;           \
        }                                  \
    } while (0)

#define X0NE_LAUNCH_CHECK()                                          \
    do {                                                             \
        cudaError_t e_ = cudaGetLastError();                         \
        if (e_ != cudaSuccess) {                                     \
            x0ne_set_error("%s:%d: %s", __FILE__, __LINE__, cudaGetErrorString(e_)); \
            return (int)e_;                                          \
        }                                                            \
        return 0;                                                    \
    } while (0)

// Programmatic dependent launch.  Every kernel of this library is launched so that it may start
// while the kernel before it in the stream is still running (its blocks are scheduled and run
// their prologue early); `pdl_wait` then blocks until that kernel has finished and its writes
// are visible.  A kernel calls `pdl_launch_dependents` at once, to let its own successor start
// early in turn, and `pdl_wait` before it touches anything an earlier kernel may have written,
// and before its own first write.  Only reads of weights may come before the wait.
// Set X0NE_PDL=0 in the environment to launch everything fully serialized.
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_prologue() {
    pdl_launch_dependents();
    pdl_wait();
}

bool x0ne_pdl_enabled();

// Set-up that the runtime keeps per device (a kernel's shared-memory attribute, occupancy numbers)
// is done once per device, by the first call with that device current: `need()` says whether it
// is still to do, `done()` records it.  Two host threads making the first call on a device at the
// same moment would both do it, which is harmless (the same values are set twice).
struct OncePerDevice {
    unsigned char set[64] = {};
    static int device() {
        int d = 0;
        return cudaGetDevice(&d) == cudaSuccess && d >= 0 && d < 64 ? d : -1;
    }
    bool need() const {
        const int d = device();
        return d < 0 || !set[d];
    }
    void done() {
        const int d = device();
        if (d >= 0) set[d] = 1;
    }
};

template <typename... KArgs, typename... Args>
static inline cudaError_t x0ne_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                      Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = x0ne_pdl_enabled() ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// The same with the grid cut into clusters of `cluster_x` consecutive blocks along x (grid.x must be
// a multiple of it): blocks of a cluster run at the same time and can read each other's shared memory.
template <typename... KArgs, typename... Args>
static inline cudaError_t x0ne_launch_clusters(void (*kernel)(KArgs...), dim3 grid, dim3 block, int cluster_x, size_t smem,
                                               cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cluster_x;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = x0ne_pdl_enabled() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

__device__ __forceinline__ float to_f32(float x) { return x; }
__device__ __forceinline__ float to_f32(bf16 x) { return __bfloat162float(x); }
template <typename T> __device__ __forceinline__ T from_f32(float x);
template <> __device__ __forceinline__ float from_f32<float>(float x) { return x; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float x) { return __float2bfloat16_rn(x); }

// Reductions.  One butterfly over the lanes of a warp and one two-level form over a block, both
// with the combining operation as a parameter; every lane / thread gets the result, and the order
// in which values meet depends on lane and warp numbers only, never on the data or on what else
// runs (the fixed-order rule of x0ne-core/kernels/cuda/common.cuh:1).
struct OpSum {
    template <typename V> __device__ __forceinline__ V operator()(V a, V b) const { return a + b; }
};
struct OpMax {
    __device__ __forceinline__ float operator()(float a, float b) const { return fmaxf(a, b); }
    __device__ __forceinline__ int operator()(int a, int b) const { return a > b ? a : b; }
    __device__ __forceinline__ unsigned long long operator()(unsigned long long a, unsigned long long b) const {
        return a > b ? a : b;
    }
};

template <typename V, typename Op>
__device__ __forceinline__ V warp_reduce(V v, Op op) {
#pragma unroll
    for (int width = 32; width > 1; width >>= 1) v = op(v, __shfl_xor_sync(0xffffffffu, v, width >> 1));
    return v;
}

// Over the block (blockDim.x a multiple of 32, at most 1024).  `sh` holds 32 values of V;
// `neutral` fills the places of warps the block does not have.
template <typename V, typename Op>
__device__ __forceinline__ V block_reduce(V v, V* sh, Op op, V neutral) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    v = warp_reduce(v, op);
    __syncthreads();              // `sh` may still be read by a reduction before this one
    if (lane == 0) sh[warp] = v;
    __syncthreads();
    return warp_reduce(lane < n_warps ? sh[lane] : neutral, op);
}

__device__ __forceinline__ float warp_sum(float v) { return warp_reduce(v, OpSum()); }
__device__ __forceinline__ float warp_max(float v) { return warp_reduce(v, OpMax()); }
__device__ __forceinline__ float block_sum(float v, float* sh) { return block_reduce(v, sh, OpSum(), 0.f); }
__device__ __forceinline__ float block_max(float v, float* sh) { return block_reduce(v, sh, OpMax(), -INFINITY); }

// The paged cache of one run-order entry.  A page holds `page_size` positions of every kv
// head, K then V: [kv_heads][page_size][head_dim] keys, then [kv_heads][page_size][v width]
// values.  The values are as wide as the keys unless `v_dim` says otherwise (0: as wide as the
// keys; negative: the page holds no values, a mixer whose values are a part of its keys).  A
// sequence's logical page (pos / page_size) % ring_pages is found in its row of the page table.
struct PagedCache {
    void* base;                 // first page of this entry
    const int32_t* page_table;  // [slots][table_stride]
    int64_t page_stride;        // elements between consecutive pages
    int32_t table_stride;
    int32_t ring_pages;         // logical pages wrap at this count (= table_stride for a full cache)
    int32_t page_size;
    int32_t kv_heads;
    int32_t head_dim;
    int32_t n_pages;            // pages in the pool, for the bounds check
    int32_t v_dim;              // width of a value row: 0 = head_dim, negative = no values are kept
};

__host__ __device__ __forceinline__ int cache_v_dim(const PagedCache& c) { return c.v_dim == 0 ? c.head_dim : (c.v_dim > 0 ? c.v_dim : 0); }

// The gated activation a product's epilogue applies to a (gate, up) pair.  limit <= 0: silu(g) u.  Else the
// clipped unit: g = min(g, limit), u = clamp(u, -limit, limit), g sigmoid(slope g) (u + shift).  `bias`, if given, holds
// the gate's biases and then the up branch's (float32, one per output each), added before the activation.
struct GluParams {
    float limit, slope, shift;
    const float* bias;
    int32_t out_act;            // products without a gate: what the epilogue does to a result (X0NE_OUT_*)
};
__device__ __forceinline__ float glu_act(float g, float u, const GluParams& p) {
    if (p.limit > 0.f) {
        g = fminf(g, p.limit);
        u = fminf(fmaxf(u, -p.limit), p.limit);
        return g / (1.0f + expf(-p.slope * g)) * (u + p.shift);
    }
    return g / (1.0f + expf(-g)) * u;
}
// the same for output n of N
__device__ __forceinline__ float glu_act_at(float g, float u, int n, int N, const GluParams& p) {
    if (p.bias != nullptr) {
        const int at = n < N ? n : N - 1;
        g += __ldg(p.bias + at);
        u += __ldg(p.bias + N + at);
    }
    return glu_act(g, u, p);
}

// What a plain product's epilogue may do to a result before it is stored.
#define X0NE_OUT_AS_IT_IS 0
#define X0NE_OUT_RELU2 1        // max(v, 0)^2
#define X0NE_OUT_SOFT_CAP 2     // limit * tanh(v / limit)
__device__ __forceinline__ float soft_capped(float v, float cap) { return cap * tanhf(v / cap); }
__device__ __forceinline__ float out_act(float v, const GluParams& p) {
    if (p.out_act == X0NE_OUT_RELU2) {
        v = fmaxf(v, 0.f);
        return v * v;
    }
    return p.out_act == X0NE_OUT_SOFT_CAP ? soft_capped(v, p.limit) : v;
}

// What an attention kernel may be asked for beyond causal softmax over a window.  All zero: nothing.
struct AttnExtra {
    int32_t chunk;        // > 0: a query sees the keys of its own chunk of this many positions only
    int32_t v_from_k;     // > 0: the values are the first v_from_k values of the key rows (no value plane is read)
    const float* sink;    // per q head, or null: exp(sink) joins the softmax denominator once (no key, no value, unscaled)
    const void* gate;     // per (row, q head) in the activation type, or null: the head's output is multiplied by sigmoid(gate)
    int64_t gate_ld;      // values between the gates of consecutive rows
    int64_t q_ld;         // values between consecutive query rows (0: q heads x head_dim)
    int32_t keep_first;   // > 0: besides its window or chunk a query sees the keys at positions below this (at their true positions)
    int32_t gate_wide;    // > 0: `gate` holds one value per (row, q head, value) at row * gate_ld + head * value width + value
    const float* slope;   // per q head, or null: slope[h] * (i - j) is taken off the scaled score of query i and key j
    int32_t out_f32;      // > 0: the results are written as float32 whatever the activation type (same places, counted in values)
    const float* sig_bias;   // per q head, or null: no softmax; key j weighs sigmoid(score + sig_bias[h]), nothing is normalised over keys
    int64_t out_ld;       // values between consecutive result rows (0: q heads x value width)
    float out_scale;      // the results are multiplied by it (0: by one)
    int32_t out_col;      // where the heads start in a result row
};

// Element offset of (slot, pos, kv head, which = 0 for K / 1 for V); -1 if there is no page, or if
// the slot is negative (a padding row that belongs to no sequence).
__device__ __forceinline__ int64_t cache_row_offset(const PagedCache& c, int slot, int pos, int kv_head, int which) {
    if (slot < 0 || pos < 0) return -1;
    const int lp = (pos / c.page_size) % c.ring_pages;
    const int page = c.page_table[(int64_t)slot * c.table_stride + lp];
    if (page < 0 || page >= c.n_pages) return -1;
    if (which == 0) return (int64_t)page * c.page_stride + ((int64_t)kv_head * c.page_size + (pos % c.page_size)) * c.head_dim;
    return (int64_t)page * c.page_stride + (int64_t)c.kv_heads * c.page_size * c.head_dim +
           ((int64_t)kv_head * c.page_size + (pos % c.page_size)) * cache_v_dim(c);
}
