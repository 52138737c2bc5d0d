// Routing of a mixture of experts, and the activation of its experts computed side by side.
//
//   moe_route       one warp per token.  z [T, ldz] float32 holds the router's logits of E experts (and, when
//                   has_gate, one more column: the logit of the shared expert's gate).  The `top` largest logits
//                   choose the experts (of equal logits the lower index first); their weights are the softmax
//                   over the chosen logits alone.  Written: idx [T, top] and wt [T, top] (either may be null), and
//                   dense [T, E + (has_gate != 0)]: an expert's weight where it was chosen, zero elsewhere, and
//                   in the last column sigmoid(gate logit) (has_gate 1) or one (has_gate 2: a shared expert without
//                   a gate; z then holds no column for it).  mode 1: the weight of a chosen expert is the sigmoid
//                   of its own logit, not renormalised (the choice is by the same order).  With `bias` (one float32
//                   per expert) in mode 1 the choice is by sigmoid(z) + bias and the weight stays sigmoid(z); in modes 0
//                   and 2 the bias is part of the logits: choice and weights are those of z + bias.
//                   mode 2: the scores are the softmax over ALL experts, the weights the chosen scores over (their sum
//                   + 1e-20).  n_groups > 0: the experts stand in n_groups equal runs, a run's score is its best
//                   expert's, and only experts of the `keep` best runs can be chosen.
//   moe_router      the router's product with bfloat16 inputs and moe_route in one launch (up to 64 rows of weights).
//   moe_dense_act   gu [T, 2 F] holds, for F = E ff + shared_ff columns, the gate rows and, F columns further, the
//                   up rows of all experts (expert e owns columns e ff .. (e + 1) ff - 1, the shared expert the last
//                   shared_ff).  a[t, c] = silu(gate) * up * dense[t, expert of c]: the experts a token did not
//                   choose contribute zeros to the one product with all down matrices that follows.  scale_input:
//                   the weight multiplies the expert's input instead of its output, a = silu(w gate) * (w up).
//   moe_dense_relu2   the same for experts without a gate, in place: u[t, c] = max(u[t, c], 0)^2 * dense[t, c / ff].
#include "common.cuh"

namespace {

// One warp routes token t, whose logits are zr (global or shared memory); `kept` is the warp's own 32 words of shared
// memory (bit g: run g stays in the race).
__device__ __forceinline__ void route_token(const float* zr, int t, int lane, int E, int top, int has_gate, int mode, int* idx,
                                            float* wt, float* dense, const int* __restrict__ tok_seq,
                                            const float* __restrict__ bias, int n_groups, int keep, unsigned* kept) {
    const int W = E + (has_gate ? 1 : 0);
    float* drow = dense + (size_t)t * W;
    for (int e = lane; e < W; e += 32) drow[e] = 0.f;
    if (tok_seq[t] < 0) {
        for (int j = lane; j < top; j += 32) {
            if (idx) idx[(size_t)t * top + j] = 0;
            if (wt) wt[(size_t)t * top + j] = 0.f;
        }
        return;
    }
    __syncwarp();
    // what the choice goes by: a logit (its order is the softmax's), or sigmoid + bias
    auto score = [&](int e) {
        if (!bias) return zr[e];
        return (mode == 1 ? 1.f / (1.f + expf(-zr[e])) : zr[e]) + bias[e];
    };
    const int per_run = n_groups > 0 ? E / n_groups : E;
    if (n_groups > 0) {
        kept[lane] = 0u;
        __syncwarp();
        for (int j = 0; j < keep; j++) {
            float best = -INFINITY;
            int bg = 0x7fffffff;
            for (int g = lane; g < n_groups; g += 32) {
                if (kept[g >> 5] >> (g & 31) & 1u) continue;
                float v = -INFINITY;
                for (int e = g * per_run; e < (g + 1) * per_run; e++) v = fmaxf(v, score(e));
                if (v > best || (v == best && g < bg)) { best = v; bg = g; }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int og = __shfl_xor_sync(0xffffffffu, bg, o);
                if (ov > best || (ov == best && og < bg)) { best = ov; bg = og; }
            }
            if (bg == 0x7fffffff) break;
            __syncwarp();
            if (lane == 0) kept[bg >> 5] |= 1u << (bg & 31);
            __syncwarp();
        }
    }
    unsigned taken = 0;                      // bit i: this lane's element lane + 32 i is chosen already
    float zmax = 0.f, sum = 0.f;
    // pass 1: choose; the first chosen logit is the largest and anchors the exponentials
    for (int j = 0; j < top; j++) {
        float best = -INFINITY;
        int bi = 0x7fffffff;
        for (int i = 0, e = lane; e < E; e += 32, i++) {
            if (taken >> i & 1u) continue;
            if (n_groups > 0 && !(kept[(e / per_run) >> 5] >> ((e / per_run) & 31) & 1u)) continue;
            const float v = score(e);
            if (v > best || (v == best && e < bi)) { best = v; bi = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        if (bi == 0x7fffffff) break;         // fewer experts than `top`
        if ((bi & 31) == lane) taken |= 1u << (bi >> 5);
        if (j == 0) zmax = best;
        const float p = mode == 1 ? 1.f / (1.f + expf(-(bias ? zr[bi] : best))) : expf(best - zmax);
        sum += p;
        if (lane == 0) {
            if (idx) idx[(size_t)t * top + j] = bi;
            drow[bi] = p;
            if (wt) wt[(size_t)t * top + j] = p;
        }
    }
    __syncwarp();
    float inv = mode == 1 ? 1.f : 1.f / sum;
    if (mode == 2) {
        // zmax is the largest logit of all: the best run holds it.  With Z = sum_all exp(z - zmax) a score is
        // p / Z, and p / Z / (sum / Z + 1e-20) is the weight.
        float total = 0.f;
        for (int e = lane; e < E; e += 32) total += expf(score(e) - zmax);
        total = warp_sum(total);
        inv = 1.f / total / (sum / total + 1e-20f);
    }
    for (int i = 0, e = lane; e < E; e += 32, i++)
        if (taken >> i & 1u) drow[e] *= inv;
    if (wt) for (int j = lane; j < top; j += 32) wt[(size_t)t * top + j] *= inv;
    if (has_gate && lane == 0) drow[E] = has_gate == 2 ? 1.f : 1.f / (1.f + expf(-zr[E]));
}

__global__ void __launch_bounds__(128)
moe_route_kernel(const float* z, long long ldz, int E, int top, int has_gate, int mode, int* idx, float* wt, float* dense,
                 const int* __restrict__ tok_seq, int n_tokens, const float* __restrict__ bias, int n_groups, int keep) {
    __shared__ unsigned kept_runs[4][32];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * 4 + warp;
    if (t >= n_tokens) return;
    route_token(z + (size_t)t * ldz, t, lane, E, top, has_gate, mode, idx, wt, dense, tok_seq, bias, n_groups, keep, kept_runs[warp]);
}

// The router's product and the routing in one launch, for bfloat16 inputs and up to ROWS (8, 16, 32 or 64) rows of router
// weights [R, D] (the experts', and the shared expert's gate behind them).  A block takes TOK tokens; its 8 warps share
// the columns, 256 a warp and turn, a lane 8 of them (16 bytes) of every token and every row; float32 sums, added over
// the lanes and then over the warps in their order, so that a token's logits do not depend on its neighbours.
constexpr int ROUTER_WARPS = 8;
template <int ROWS, int TOK>
__global__ void __launch_bounds__(ROUTER_WARPS * 32)
moe_router_kernel(const bf16* h, long long ldh, const bf16* __restrict__ w, int R, int D, int E, int top, int has_gate,
                  int mode, float* dense, const int* __restrict__ tok_seq, int n_tokens, const float* __restrict__ bias,
                  int n_groups, int keep) {
    __shared__ float part[ROUTER_WARPS][TOK][ROWS];
    __shared__ float z[TOK][ROWS];
    __shared__ unsigned kept_runs[TOK][32];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = blockIdx.x * TOK;
    float acc[TOK][ROWS];
#pragma unroll
    for (int i = 0; i < TOK; i++)
#pragma unroll
        for (int r = 0; r < ROWS; r++) acc[i][r] = 0.f;
    for (int c = (warp * 32 + lane) * 8; c < D; c += ROUTER_WARPS * 256) {
        float x[TOK][8];
#pragma unroll
        for (int i = 0; i < TOK; i++) {
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (t0 + i < n_tokens) v = *reinterpret_cast<const uint4*>(h + (size_t)(t0 + i) * ldh + c);
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
            for (int j = 0; j < 4; j++) { const float2 f = __bfloat1622float2(p[j]); x[i][2 * j] = f.x; x[i][2 * j + 1] = f.y; }
        }
#pragma unroll
        for (int r = 0; r < ROWS; r++) {
            if (r >= R) break;
            const uint4 v = *reinterpret_cast<const uint4*>(w + (size_t)r * D + c);
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const float2 f = __bfloat1622float2(p[j]);
#pragma unroll
                for (int i = 0; i < TOK; i++) acc[i][r] = fmaf(x[i][2 * j + 1], f.y, fmaf(x[i][2 * j], f.x, acc[i][r]));
            }
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; r++) {
        if (r >= R) break;
#pragma unroll
        for (int i = 0; i < TOK; i++) {
            const float s = warp_sum(acc[i][r]);
            if (lane == 0) part[warp][i][r] = s;
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < TOK * R; e += blockDim.x) {
        float s = 0.f;
#pragma unroll
        for (int q = 0; q < ROUTER_WARPS; q++) s += part[q][e / R][e % R];
        z[e / R][e % R] = s;
    }
    __syncthreads();
    if (warp < TOK && t0 + warp < n_tokens)
        route_token(z[warp], t0 + warp, lane, E, top, has_gate, mode, nullptr, nullptr, dense, tok_seq, bias, n_groups, keep,
                    kept_runs[warp]);
}

// One thread takes 8 consecutive columns of one token (16 bytes of bfloat16) where an expert's columns come in
// multiples of 8, else one column; the columns of an expert the token did not choose are written as zeros without
// their gate and up values being read.
template <typename T, int V>
__global__ void __launch_bounds__(256)
moe_dense_act_kernel(T* a, const T* gu, const float* dense, int n_tokens, int F, int E, int ff, int W, int scale_input,
                     int act, float limit) {
    pdl_launch_dependents();
    pdl_wait();
    const int per_row = F / V;
    const size_t total = (size_t)n_tokens * per_row;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / per_row;
        const int c = (int)(e % per_row) * V;
        int grp = c / ff;
        if (grp > E) grp = E;
        const float w = grp < W ? dense[t * W + grp] : 0.f;
        T out[V];
        if (w != 0.f) {
            T g[V], u[V];
            if (V == 8) {
                *reinterpret_cast<uint4*>(g) = *reinterpret_cast<const uint4*>(gu + t * 2 * F + c);
                *reinterpret_cast<uint4*>(u) = *reinterpret_cast<const uint4*>(gu + t * 2 * F + F + c);
            } else {
                g[0] = gu[t * 2 * F + c];
                u[0] = gu[t * 2 * F + F + c];
            }
#pragma unroll
            for (int i = 0; i < V; i++) {
                if (act == 1) {
                    const float gf = fminf(to_f32(g[i]), limit);
                    const float uf = fminf(fmaxf(to_f32(u[i]), -limit), limit);
                    out[i] = from_f32<T>(gf / (1.f + expf(-1.702f * gf)) * (uf + 1.f) * w);
                } else if (scale_input) {
                    const float gf = to_f32(g[i]) * w;
                    out[i] = from_f32<T>(gf / (1.f + expf(-gf)) * (to_f32(u[i]) * w));
                } else {
                    const float gf = to_f32(g[i]);
                    out[i] = from_f32<T>(gf / (1.f + expf(-gf)) * to_f32(u[i]) * w);
                }
            }
        } else {
#pragma unroll
            for (int i = 0; i < V; i++) out[i] = from_f32<T>(0.f);
        }
        if (V == 8) *reinterpret_cast<uint4*>(a + t * F + c) = *reinterpret_cast<uint4*>(out);
        else a[t * F + c] = out[0];
    }
}

// In place; a thread takes 8 consecutive columns (16 bytes of bfloat16) or one; the columns of an expert the token did
// not choose become zero unread.
template <typename T, int V>
__global__ void __launch_bounds__(256)
moe_dense_relu2_kernel(T* u, const float* dense, int n_tokens, int F, int ff, int W) {
    pdl_launch_dependents();
    pdl_wait();
    const int per_row = F / V;
    const size_t total = (size_t)n_tokens * per_row;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / per_row;
        const int c = (int)(e % per_row) * V;
        const float w = dense[t * W + c / ff];
        T v[V];
        if (w != 0.f) {
            if (V == 8) *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(u + t * F + c);
            else v[0] = u[t * F + c];
#pragma unroll
            for (int i = 0; i < V; i++) {
                const float r = fmaxf(to_f32(v[i]), 0.f);
                v[i] = from_f32<T>(r * r * w);
            }
        } else {
#pragma unroll
            for (int i = 0; i < V; i++) v[i] = from_f32<T>(0.f);
        }
        if (V == 8) *reinterpret_cast<uint4*>(u + t * F + c) = *reinterpret_cast<uint4*>(v);
        else u[t * F + c] = v[0];
    }
}

template <typename T>
int launch_relu2(T* u, const float* dense, int n_tokens, int F, int ff, int W, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (F < 1 || ff < 1 || F % ff || W < F / ff) return OE_ERR_UNSUPPORTED;
    const bool vec = sizeof(T) == 2 && ff % 8 == 0 && !((uintptr_t)u & 15);
    const size_t total = (size_t)n_tokens * (vec ? F / 8 : F);
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (vec) return oe_launch(moe_dense_relu2_kernel<T, 8>, dim3((unsigned)blocks), dim3(256), 0, st, u, dense, n_tokens, F, ff, W);
    return oe_launch(moe_dense_relu2_kernel<T, 1>, dim3((unsigned)blocks), dim3(256), 0, st, u, dense, n_tokens, F, ff, W);
}

template <typename T>
int launch_act(T* a, const T* gu, const float* dense, int n_tokens, int F, int E, int ff, int W, int scale_input,
               int act, float limit, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (F < 1 || ff < 1 || E < 0 || act < 0 || act > 1 || (act == 1 && scale_input)) return OE_ERR_UNSUPPORTED;
    // 16-byte pieces: bfloat16, every expert's columns and the row a multiple of 8, aligned pointers
    const bool vec = sizeof(T) == 2 && ff % 8 == 0 && F % 8 == 0 && !(((uintptr_t)a | (uintptr_t)gu) & 15);
    const size_t total = (size_t)n_tokens * (vec ? F / 8 : F);
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (vec)
        return oe_launch(moe_dense_act_kernel<T, 8>, dim3((unsigned)blocks), dim3(256), 0, st, a, gu, dense, n_tokens, F, E, ff, W, scale_input, act, limit);
    return oe_launch(moe_dense_act_kernel<T, 1>, dim3((unsigned)blocks), dim3(256), 0, st, a, gu, dense, n_tokens, F, E, ff, W, scale_input, act, limit);
}

}  // namespace

extern "C" {

int oe_moe_route(const float* z, long long ldz, int E, int top, int has_gate, int mode, int* idx, float* wt, float* dense,
                 const int* tok_seq, int n_tokens, const float* bias, int n_groups, int keep, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (E < 1 || E > 1024 || top < 1 || mode < 0 || mode > 2) return OE_ERR_UNSUPPORTED;
    if (n_groups < 0 || (n_groups > 0 && (E % n_groups || keep < 1 || keep > n_groups))) return OE_ERR_UNSUPPORTED;
    return oe_launch(moe_route_kernel, dim3((n_tokens + 3) / 4), dim3(128), 0, st, z, ldz, E, top, has_gate, mode, idx, wt, dense,
                     tok_seq, n_tokens, bias, n_groups, keep);
}
// h [T, D] bfloat16 (rows of ldh), w [R, D] bfloat16 with R = E rows, one more when has_gate is 1.
int oe_moe_router(const bf16* h, long long ldh, const bf16* w, int D, int E, int top, int has_gate, int mode, float* dense,
                  const int* tok_seq, int n_tokens, const float* bias, int n_groups, int keep, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    const int R = E + (has_gate == 1 ? 1 : 0);
    if (E < 1 || R > 64 || top < 1 || mode < 0 || mode > 2) return OE_ERR_UNSUPPORTED;
    if (n_groups < 0 || (n_groups > 0 && (E % n_groups || keep < 1 || keep > n_groups))) return OE_ERR_UNSUPPORTED;
    if (D % 8 || ldh % 8 || (((uintptr_t)h | (uintptr_t)w) & 15)) return OE_ERR_UNSUPPORTED;
#define OE_ROUTER(ROWS, TOK)                                                                                              \
    return oe_launch(moe_router_kernel<ROWS, TOK>, dim3((n_tokens + TOK - 1) / TOK), dim3(ROUTER_WARPS * 32), 0, st, h, ldh, w, \
                     R, D, E, top, has_gate, mode, dense, tok_seq, n_tokens, bias, n_groups, keep)
    // few tokens: a block each; many: the weights' loads serve several
    if (R <= 8) { if (n_tokens <= 296) OE_ROUTER(8, 1); OE_ROUTER(8, 4); }
    if (R <= 16) { if (n_tokens <= 296) OE_ROUTER(16, 1); OE_ROUTER(16, 4); }
    if (R <= 32) OE_ROUTER(32, 1);
    OE_ROUTER(64, 1);
#undef OE_ROUTER
}
int oe_moe_dense_relu2_f32(float* u, const float* dense, int n_tokens, int F, int ff, int W, cudaStream_t st) {
    return launch_relu2<float>(u, dense, n_tokens, F, ff, W, st);
}
int oe_moe_dense_relu2_bf16(bf16* u, const float* dense, int n_tokens, int F, int ff, int W, cudaStream_t st) {
    return launch_relu2<bf16>(u, dense, n_tokens, F, ff, W, st);
}
int oe_moe_dense_act_f32(float* a, const float* gu, const float* dense, int n_tokens, int F, int E, int ff, int W,
                         int scale_input, int act, float limit, cudaStream_t st) {
    return launch_act<float>(a, gu, dense, n_tokens, F, E, ff, W, scale_input, act, limit, st);
}
int oe_moe_dense_act_bf16(bf16* a, const bf16* gu, const float* dense, int n_tokens, int F, int E, int ff, int W,
                          int scale_input, int act, float limit, cudaStream_t st) {
    return launch_act<bf16>(a, gu, dense, n_tokens, F, E, ff, W, scale_input, act, limit, st);
}

}  // extern "C"
