// Shared helpers of the hand-written sm_100a kernels.
//
// Every exported entry point is `extern "C"`, takes raw device pointers, sizes and a
// cudaStream_t, launches on that stream and returns a cudaError_t-compatible int
// (0 = launched).  Sizes a kernel cannot take are refused on the host side with
// OE_ERR_UNSUPPORTED before anything is launched; nothing falls back to another path.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>
#include <stdlib.h>

#define OE_ERR_UNSUPPORTED 100001   // size or option outside what the kernel takes
#define OE_PAGE 64                  // tokens per cache page

typedef __nv_bfloat16 bf16;

// ---------------------------------------------------------------------------------------
// Programmatic dependent launch.  Every kernel of this library is launched with the
// programmatic-stream-serialization attribute: it may start while the kernel before it in
// the stream is still draining, does whatever does not depend on that kernel (set-up,
// prefetch of weights), and calls pdl_wait() before it first touches memory that an
// earlier kernel of the stream may have written (or may still read, for buffers it
// overwrites).  pdl_wait() returns when every earlier kernel has completed and its
// writes are visible.  Every kernel calls it, so completion is transitive along the
// stream.  pdl_launch_dependents() lets the next kernel be scheduled early.
// A kernel that starts early must read what earlier kernels wrote through the coherent path:
// pointers to such data are NOT `const __restrict__` (which lets the compiler use the read-only
// cache, valid only for data that does not change while the kernel is resident); weights and
// the step's integer tables, written before the step's first kernel, may be.
// Set OE_PDL=0 in the environment to launch without the attribute.
// ---------------------------------------------------------------------------------------
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

#ifndef __CUDA_ARCH__
static inline int oe_pdl_enabled() {
    static int v = -1;
    if (v < 0) {
        const char* e = getenv("OE_PDL");
        v = (e != nullptr && e[0] == '0') ? 0 : 1;
    }
    return v;
}
#endif

// The attribute can also be switched at run time, per library (every library is one translation unit and exports its
// own oe_pdl_set): the step function launches large prompt steps without it (engine/step.py says why).
#ifndef __CUDA_ARCH__
static int oe_pdl_runtime_flag = 1;
extern "C" __attribute__((visibility("default"))) void oe_pdl_set(int on) { oe_pdl_runtime_flag = on ? 1 : 0; }
static inline int oe_pdl_now() { return oe_pdl_enabled() && oe_pdl_runtime_flag; }
#endif

template <typename... KArgs, typename... Args>
static inline int oe_launch_ex(bool early, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st,
                               Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
#ifndef __CUDA_ARCH__
    attr[0].val.programmaticStreamSerializationAllowed = early ? oe_pdl_now() : 0;
#endif
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

// The same with clusters of cluster_x consecutive CTAs along x (the grid's x is a multiple of it).
template <typename... KArgs, typename... Args>
static inline int oe_launch_cluster(void (*kernel)(KArgs...), unsigned cluster_x, dim3 grid, dim3 block, size_t smem,
                                    cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
#ifndef __CUDA_ARCH__
    attr[0].val.programmaticStreamSerializationAllowed = oe_pdl_now();
#endif
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster_x;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    return (int)cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

// early = true: the kernel may start before the one before it has finished (see above).
template <typename... KArgs, typename... Args>
static inline int oe_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args... args) {
    return oe_launch_ex(true, kernel, grid, block, smem, st, args...);
}

// The first key a query at position `pos` sees; its last one is its own.  `span` is what the attention entry points
// call `window`: 0, every key of the sequence; n > 0, the last n keys (pos - n < key); -n < 0, the keys of the query's own
// chunk, positions being cut into chunks of n from position 0 of the sequence on (key / n == pos / n).
__device__ __forceinline__ int oe_first_key(int pos, int span) {
    if (span > 0) return pos >= span ? pos - span + 1 : 0;
    if (span < 0) return pos - pos % -span;
    return 0;
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// An output gate of an attention: what head h's result of token t is multiplied by at column d, sigmoid of the row's value
// for that column (OE_GATE_VALUE, rows of H dv values) or of the head's value (OE_GATE_HEAD, rows of H values).
#define OE_GATE_VALUE 1
#define OE_GATE_HEAD 2
__device__ __forceinline__ float oe_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
template <typename T>
__device__ __forceinline__ float oe_sigmoid_gate(const T* gate, long long stride, int mode, long long t, int h, int H, int dv, int d) {
    return oe_sigmoid(to_f32(gate[t * stride + (mode == OE_GATE_HEAD ? h : (long long)h * dv + d)]));
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// z times the normal distribution function: the exact gelu.
__device__ __forceinline__ float oe_gelu(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }

// What a product does to its float32 sums before it stores them as bfloat16: the features (weight rows) from `from` on
// go through `act` and are then multiplied by a per-token weight of their group of `ff` features, w[token * ld +
// (feature - from) / ff] (w null: by nothing); the features before `from` are stored as they are.
struct OeEpilogue {
    int act;                   // 0 none, 1 exact gelu, 2 squared ReLU
    int from, ff;
    long long ld;
    const float* w;            // written by an earlier kernel of the stream: read only behind pdl_wait()
};
// The exact gelu for a result that is rounded to bfloat16, without branches, so that the values of a row overlap:
// 1 - erf(x) by formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions (absolute error 1.5e-7).
__device__ __forceinline__ float oe_gelu_bf16(float z) {
    const float x = fabsf(z) * 0.70710678118654752f;
    const float t = __fdividef(1.f, fmaf(0.3275911f, x, 1.f));
    float p = fmaf(1.061405429f, t, -1.453152027f);
    p = fmaf(p, t, 1.421413741f);
    p = fmaf(p, t, -0.284496736f);
    p = fmaf(p, t, 0.254829592f);
    const float h = 0.5f * z * (p * t * __expf(-x * x));          // z times half of what lies beyond |z|
    return z >= 0.f ? z - h : h;
}
template <int N>
__device__ __forceinline__ void oe_activate(int act, float (&v)[N]) {
    if (act == 1) {
#pragma unroll
        for (int j = 0; j < N; j++) v[j] = oe_gelu_bf16(v[j]);
    } else {
#pragma unroll
        for (int j = 0; j < N; j++) { const float r = fmaxf(v[j], 0.f); v[j] = r * r; }
    }
}
// A token's weight of the group that holds the features [lo, hi) behind `from`: kept while a thread walks along a row.
struct OeGroupWeight {
    int lo = 0, hi = 0;
    float w = 0.f;
};
// N consecutive features of one token, feature0 .. feature0 + N - 1; those from n_features on are not stored.
template <int N>
__device__ __forceinline__ void oe_epilogue_row(const OeEpilogue& e, float (&v)[N], int token, int feature0, int n_features,
                                                OeGroupWeight& kept) {
    if (feature0 + N <= e.from) return;
    const int b0 = feature0 - e.from;
    if (b0 >= 0 && e.w == nullptr) {
        oe_activate(e.act, v);
        return;
    }
    const float* row = e.w + (long long)token * e.ld;
    if (b0 >= 0 && (b0 < kept.lo || b0 + N > kept.hi) && feature0 < n_features) {
        const int group = b0 / e.ff;
        if (b0 + N <= (group + 1) * e.ff) {
            kept.lo = group * e.ff;
            kept.hi = kept.lo + e.ff;
            kept.w = row[group];
        }
    }
    if (b0 >= 0 && b0 >= kept.lo && b0 + N <= kept.hi) {
        oe_activate(e.act, v);
#pragma unroll
        for (int j = 0; j < N; j++) v[j] *= kept.w;
        return;
    }
    // the features lie on both sides of `from` or of a group's edge
    float u[N];
#pragma unroll
    for (int j = 0; j < N; j++) u[j] = v[j];
    oe_activate(e.act, u);
#pragma unroll
    for (int j = 0; j < N; j++)
        if (b0 + j >= 0 && feature0 + j < n_features) v[j] = e.w == nullptr ? u[j] : u[j] * row[(b0 + j) / e.ff];
}
__device__ __forceinline__ float oe_epilogue_one(const OeEpilogue& e, float v, int token, int feature) {
    if (feature < e.from) return v;
    float u[1] = {v};
    oe_activate(e.act, u);
    return e.w == nullptr ? u[0] : u[0] * e.w[(long long)token * e.ld + (feature - e.from) / e.ff];
}
// The host side of the four arguments: false if they make no sense.
static inline bool oe_epilogue_ok(const OeEpilogue& e, int out_kind, int n_features) {
    if (e.act == 0) return e.w == nullptr;
    return (e.act == 1 || e.act == 2) && out_kind == 0 && e.from >= 0 && e.from <= n_features &&
           (e.w == nullptr || (e.ff > 0 && e.ld >= (n_features - e.from + e.ff - 1) / e.ff));
}

// Sum over a block in a fixed order (warp shuffles, then warp 0 over the warp totals);
// every thread gets the result.  `red` holds 32 floats of shared memory.
__device__ __forceinline__ float block_sum(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = (lane < nwarps) ? red[lane] : 0.f;
    t = warp_sum(t);
    return t;
}
__device__ __forceinline__ float block_max(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = (lane < nwarps) ? red[lane] : -INFINITY;
    t = warp_max(t);
    return t;
}

// Address of token `pos` of one (cache entry, K-or-V, kv head) in the paged cache.
// Storage of one cache entry: [n_pages][2][kv_heads][OE_PAGE][head_dim].
// Returns the element offset from the entry's base, or -1 if the page is not mapped.
__device__ __forceinline__ long long page_row_offset(const int* __restrict__ table_row, int pos,
                                                     int which, int kvh, int kv_heads, int head_dim) {
    const int page = table_row[pos / OE_PAGE];
    if (page < 0) return -1;
    return ((((long long)page * 2 + which) * kv_heads + kvh) * OE_PAGE + (pos % OE_PAGE)) * head_dim;
}
