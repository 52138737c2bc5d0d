// Selective scan: a recurrence with a state of N values per channel whose decay, input and read-out depend on the token.
//
//   causal_conv       out[t, c] = silu(sum_j w[j][c] x[t - (taps - 1) + j, c] + b[c]) per sequence: rows before a step's first
//                     token come from the sequence's kept rows [taps - 1, C] (float32, zeros at its start).  In a step of
//                     one token per sequence the same kernel shifts the kept rows.
//   conv_rows_state   the kept rows after a step of any other kind.
//   thin_cast         columns of a float32 product in bfloat16 (the operand of the step sizes' product).
//   selective_scan    dt_c = softplus(zdt_c + bias_c);  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c b_n;
//                     y_c = (sum_n S[c, n] c_n + D_c u_c) * silu(z_c)                                  everything in float32
//   selective_step    the same for one token per sequence, with the step sizes' product inside: zdt_c = sum_j W[c, j] r_j.
//
// A channel's N states belong to L adjacent lanes (which may own a second channel), lane l keeping states l PER .. l PER + PER - 1 in registers for all
// tokens of the step; b and c, which every channel reads, go through shared memory a few tokens at a time.  The decay is
// 2^(dt A2) with A2 = A log2(e) made once.  Without segments a step's tokens of one sequence are walked in order,
// whatever their number: the cut of a sequence into steps changes no bit.
//
// A long prompt in segments (oe_selective_scan_segments): the recurrence is linear in the state, so a sequence's tokens are
// cut into segments of seg_len that run side by side.  Pass 1 walks every segment but a sequence's last from a zero state
// and keeps its end state L_g and the sum s_g of its step sizes (the product of a segment's decays is 2^(s_g A2));
// selective_join_kernel makes every segment's true entering state, E_0 = S, E_(g+1) = 2^(s_g A2) E_g + L_g; pass 2
// walks every segment from its E_g and writes the outputs, a sequence's last segment also the state.
#include "common.cuh"

namespace {

constexpr int MAX_TAPS = 32;
constexpr int CHUNK = 16;        // tokens whose b and c are staged at once
constexpr int THREADS = 128;

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// silu of a result that is rounded to bfloat16 by the hardware's exponential and division.
template <typename T>
__device__ __forceinline__ float gate_silu(float z) {
    if (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
    return silu_f(z);
}
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// V consecutive values in pieces of 16 (or once 8) bytes; one value as it is.
template <typename T, int V>
__device__ __forceinline__ void load_vec(float (&o)[V], const T* p) {
    if constexpr (V == 1) {
        o[0] = to_f32(p[0]);
    } else {
        __align__(16) T t[V];
        if constexpr (V * sizeof(T) == 8) {
            *reinterpret_cast<uint2*>(t) = *reinterpret_cast<const uint2*>(p);
        } else {
            static_assert(V * sizeof(T) % 16 == 0, "pieces of 16 bytes");
#pragma unroll
            for (int i = 0; i < V * (int)sizeof(T) / 16; i++) reinterpret_cast<uint4*>(t)[i] = reinterpret_cast<const uint4*>(p)[i];
        }
#pragma unroll
        for (int i = 0; i < V; i++) o[i] = to_f32(t[i]);
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_vec(T* p, const float (&o)[V]) {
    if constexpr (V == 1) {
        p[0] = from_f32<T>(o[0]);
    } else {
        __align__(16) T t[V];
#pragma unroll
        for (int i = 0; i < V; i++) t[i] = from_f32<T>(o[i]);
        if constexpr (V * sizeof(T) == 8) {
            *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(t);
        } else {
#pragma unroll
            for (int i = 0; i < V * (int)sizeof(T) / 16; i++) reinterpret_cast<uint4*>(p)[i] = reinterpret_cast<uint4*>(t)[i];
        }
    }
}

// grid (token tiles of PT, channel tiles).  A thread owns V adjacent channels and takes the tile's tokens with the window of
// the last TAPS rows in registers.  A tile inside one sequence, its first window included, asks for all its rows at once;
// any other goes token by token and fills the window anew at a sequence's first token of the step, from the kept rows.
// `shift`: every sequence brings one token, its thread also moves the kept rows on.  w [taps, C].
template <typename T, int TAPS, int V, int PT>
__global__ void __launch_bounds__(THREADS)
causal_conv_kernel(T* out, const T* x, long long ldx, const float* __restrict__ w, const float* __restrict__ bias, float* state,
                   const int* __restrict__ tok_seq, const int* __restrict__ seq_slot, const int* __restrict__ cu_q,
                   int n_tokens, int C, int shift) {
    const int c = (blockIdx.y * THREADS + threadIdx.x) * V;
    float k[TAPS][V], b[V];
    if (c < C) {
#pragma unroll
        for (int j = 0; j < TAPS; j++) load_vec<float, V>(k[j], w + (size_t)j * C + c);
#pragma unroll
        for (int i = 0; i < V; i++) b[i] = 0.f;
        if (bias) load_vec<float, V>(b, bias + c);
    }
    pdl_launch_dependents();
    pdl_wait();
    if (c >= C) return;
    const int t0 = blockIdx.x * PT;
    if (PT > 1 && t0 + PT <= n_tokens) {
        const int s = tok_seq[t0];
        if (s >= 0 && s == tok_seq[t0 + PT - 1] && t0 - cu_q[s] >= TAPS - 1) {
            float rows[PT + TAPS - 1][V];
#pragma unroll
            for (int r = 0; r < PT + TAPS - 1; r++) load_vec<T, V>(rows[r], x + (size_t)(t0 - (TAPS - 1) + r) * ldx + c);
#pragma unroll
            for (int t = 0; t < PT; t++) {
                float y[V];
#pragma unroll
                for (int i = 0; i < V; i++) {
                    float a = b[i];
#pragma unroll
                    for (int j = 0; j < TAPS; j++) a = fmaf(k[j][i], rows[t + j][i], a);
                    y[i] = gate_silu<T>(a);
                }
                store_vec<T, V>(out + (size_t)(t0 + t) * C + c, y);
            }
            return;
        }
    }
    float win[TAPS][V];
    const int t_end = min(n_tokens, t0 + PT);
    int prev_seq = -1;
    for (int t = t0; t < t_end; t++) {
        const int s = tok_seq[t];
        if (s < 0) { prev_seq = -1; continue; }
        const int rel = t - cu_q[s];
        float* st = state + (size_t)seq_slot[s] * (TAPS - 1) * C;
        if (s != prev_seq) {
#pragma unroll
            for (int j = 0; j < TAPS - 1; j++) {
                const int r = rel - (TAPS - 1) + j;
                if (r >= 0) load_vec<T, V>(win[j + 1], x + (size_t)(t - rel + r) * ldx + c);
                else load_vec<float, V>(win[j + 1], st + (size_t)(rel + j) * C + c);
            }
            prev_seq = s;
        }
#pragma unroll
        for (int j = 0; j < TAPS - 1; j++)
#pragma unroll
            for (int i = 0; i < V; i++) win[j][i] = win[j + 1][i];
        load_vec<T, V>(win[TAPS - 1], x + (size_t)t * ldx + c);
        float y[V];
#pragma unroll
        for (int i = 0; i < V; i++) {
            float a = b[i];
#pragma unroll
            for (int j = 0; j < TAPS; j++) a = fmaf(k[j][i], win[j][i], a);
            y[i] = gate_silu<T>(a);
        }
        store_vec<T, V>(out + (size_t)t * C + c, y);
        if (shift)
#pragma unroll
            for (int j = 0; j < TAPS - 1; j++) store_vec<float, V>(st + (size_t)j * C + c, win[j + 1]);
    }
}

// Any number of taps: grid (tokens, channel tiles), a thread per channel.
template <typename T>
__global__ void __launch_bounds__(THREADS)
causal_conv_any_kernel(T* out, const T* x, long long ldx, const float* __restrict__ w, const float* __restrict__ bias, int taps,
                       const float* state, const int* __restrict__ tok_seq, const int* __restrict__ seq_slot,
                       const int* __restrict__ cu_q, int C) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, c = blockIdx.y * THREADS + threadIdx.x;
    const int s = tok_seq[t];
    if (s < 0 || c >= C) return;
    const int rel = t - cu_q[s];
    const float* st = state + (size_t)seq_slot[s] * (taps - 1) * C;
    float a = bias ? bias[c] : 0.f;
    for (int j = 0; j < taps; j++) {
        const int r = rel - (taps - 1) + j;
        const float v = r >= 0 ? to_f32(x[(size_t)(t - rel + r) * ldx + c]) : st[(size_t)(rel + j) * C + c];
        a = fmaf(w[(size_t)j * C + c], v, a);
    }
    out[(size_t)t * C + c] = from_f32<T>(gate_silu<T>(a));
}

// grid (sequences, channel tiles); a thread owns a channel, so it reads its old rows before it writes them.
template <typename T>
__global__ void __launch_bounds__(THREADS)
conv_rows_state_kernel(float* state, const T* x, long long ldx, int C, int taps, const int* __restrict__ seq_slot,
                       const int* __restrict__ cu_q) {
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.x, c = blockIdx.y * THREADS + threadIdx.x;
    const int slot = seq_slot[b], row0 = cu_q[b], n = cu_q[b + 1] - row0;
    if (slot < 0 || n <= 0 || c >= C) return;
    float* st = state + (size_t)slot * (taps - 1) * C;
    // row i of the new ones is old row n + i as long as that exists: in rising order nothing is overwritten unread
    for (int i = 0; i < taps - 1; i++) {
        const int r = n - (taps - 1) + i;
        st[(size_t)i * C + c] = r >= 0 ? to_f32(x[(size_t)(row0 + r) * ldx + c]) : st[(size_t)(n + i) * C + c];
    }
}

__global__ void __launch_bounds__(256)
thin_cast_kernel(bf16* out, const float* in, long long ld, int n_tokens, int n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t total = (size_t)n_tokens * n;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x)
        out[e] = __float2bfloat16_rn(in[(e / n) * ld + e % n]);
}

template <typename T>
struct ScanArgs {
    T* y;                                   // [T, C]
    float* state;                           // [slots, C, N]
    const T* u;                             // [T, C]
    const float* zdt;                       // [T, C], before bias and softplus
    const float* dt_bias;                   // [C]
    const float* thin; long long ldthin;    // float32 rows; b at column off_b, c at off_c
    int off_b, off_c;
    const float* A2;                        // [C, N]: A log2(e)
    const float* Dw;                        // [C]
    const T* z; long long ldz;              // gate rows
    const int* seq_slot; const int* cu_q;
    int C, N;
    int seg_len; float* seg_state; float* seg_dt;      // segments: [n_seqs, n_seg, C, N] and [n_seqs, n_seg, C]
};

// Two neighbouring states in one register pair: sm_100 multiplies and adds such pairs in one instruction.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pair_of(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 parts_of(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 pair_mul(f32x2 x, f32x2 y) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(x), "l"(y));
    return r;
}
__device__ __forceinline__ f32x2 pair_fma(f32x2 x, f32x2 y, f32x2 z) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(x), "l"(y), "l"(z));
    return r;
}

// PER (a multiple of 4) states from `first` on; zeros behind the N-th.
template <int PER>
__device__ __forceinline__ void load_states(f32x2 (&s)[PER / 2], const float* p, int first, int N, bool vec) {
#pragma unroll
    for (int i = 0; i < PER; i += 4) {
        float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
        if (vec) {
            if (first + i < N) q = *reinterpret_cast<const float4*>(p + first + i);
        } else {
            if (first + i < N) q.x = p[first + i];
            if (first + i + 1 < N) q.y = p[first + i + 1];
            if (first + i + 2 < N) q.z = p[first + i + 2];
            if (first + i + 3 < N) q.w = p[first + i + 3];
        }
        s[i / 2] = pair_of(q.x, q.y);
        s[i / 2 + 1] = pair_of(q.z, q.w);
    }
}
template <int PER>
__device__ __forceinline__ void store_states(float* p, const f32x2 (&s)[PER / 2], int first, int N, bool vec) {
#pragma unroll
    for (int i = 0; i < PER; i += 4) {
        const float2 x = parts_of(s[i / 2]), y = parts_of(s[i / 2 + 1]);
        if (vec) {
            if (first + i < N) *reinterpret_cast<float4*>(p + first + i) = make_float4(x.x, x.y, y.x, y.y);
        } else {
            if (first + i < N) p[first + i] = x.x;
            if (first + i + 1 < N) p[first + i + 1] = x.y;
            if (first + i + 2 < N) p[first + i + 2] = y.x;
            if (first + i + 3 < N) p[first + i + 3] = y.y;
        }
    }
}

// 2^x by the hardware's instruction; a result too small for a normal number is zero (a decay: the state is gone).
__device__ __forceinline__ float decay_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int L>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = 1; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// One token of NC channels: their states move on, acc receives the read-outs' shares of this lane's states.  sb, sc: this
// lane's part of the token's b and c, PER values each, padded with zeros, read once for all NC channels.
template <int NC, int PER, bool OUT>
__device__ __forceinline__ void scan_token(f32x2 (&s)[NC][PER / 2], const f32x2 (&a2)[NC][PER / 2], const float (&dt)[NC],
                                           const float (&du)[NC], const float* sb, const float* sc, float (&acc)[NC]) {
    f32x2 sum[NC][2], dt2[NC], du2[NC];
#pragma unroll
    for (int k = 0; k < NC; k++) {
        sum[k][0] = sum[k][1] = 0ull;
        dt2[k] = pair_of(dt[k], dt[k]);
        du2[k] = pair_of(du[k], du[k]);
    }
#pragma unroll
    for (int i = 0; i < PER / 2; i += 2) {
        const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(sb + 2 * i);
        ulonglong2 c = make_ulonglong2(0ull, 0ull);
        if (OUT) c = *reinterpret_cast<const ulonglong2*>(sc + 2 * i);
#pragma unroll
        for (int k = 0; k < NC; k++) {
            const float2 x = parts_of(pair_mul(dt2[k], a2[k][i])), y = parts_of(pair_mul(dt2[k], a2[k][i + 1]));
            s[k][i] = pair_fma(pair_of(decay_exp2(x.x), decay_exp2(x.y)), s[k][i], pair_mul(du2[k], b.x));
            s[k][i + 1] = pair_fma(pair_of(decay_exp2(y.x), decay_exp2(y.y)), s[k][i + 1], pair_mul(du2[k], b.y));
            if (OUT) {
                sum[k][0] = pair_fma(s[k][i], c.x, sum[k][0]);
                sum[k][1] = pair_fma(s[k][i + 1], c.y, sum[k][1]);
            }
        }
    }
#pragma unroll
    for (int k = 0; k < NC; k++) {
        const float2 x = parts_of(sum[k][0]), y = parts_of(sum[k][1]);
        acc[k] = (x.x + x.y) + (y.x + y.y);
    }
}

template <typename T, int NC>
__device__ __forceinline__ void load_channels(float (&o)[NC], const T* p) {
    if constexpr (NC == 2 && sizeof(T) == 2) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        o[0] = f.x;
        o[1] = f.y;
    } else if constexpr (NC == 2) {
        const float2 f = *reinterpret_cast<const float2*>(p);
        o[0] = f.x;
        o[1] = f.y;
    } else {
        o[0] = to_f32(p[0]);
    }
}

// grid (channel tiles, sequences[, segments]).  MODE 0: one walk; 1 and 2: the two passes over segments.  A group of L lanes
// owns NC adjacent channels (NC 2: C and ldz even, rows aligned for pairs).
template <typename T, int PER, int L, int MODE, int NC>
__global__ void __launch_bounds__(THREADS, NC == 2 ? 4 : 1)
selective_scan_kernel(const ScanArgs<T> a) {
    constexpr int CPB = THREADS / L * NC, NP = PER * L;     // channels per block, states padded
    constexpr bool OUT = MODE != 1;
    constexpr int AHEAD = 4;                                // tokens whose channel values are asked for at once
    __shared__ __align__(16) float stage[2][CHUNK][NP];
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.y;
    const int slot = a.seq_slot[b], row0 = a.cu_q[b];
    int n = a.cu_q[b + 1] - row0;
    if (slot < 0 || n <= 0) return;
    int first = 0;
    bool last = true;
    const int g = MODE ? blockIdx.z : 0, n_seg = MODE ? gridDim.z : 1;
    if (MODE) {
        first = g * a.seg_len;
        if (first >= n) return;
        last = first + a.seg_len >= n;
        if (MODE == 1 && last) return;                      // nothing comes after it
        n = min(n, first + a.seg_len);
    }
    const int l = threadIdx.x % L, c = blockIdx.x * CPB + threadIdx.x / L * NC;
    const bool mine = c < a.C;
    const int cc = mine ? c : a.C - NC;
    const bool vec = a.N % 4 == 0;
    f32x2 s[NC][PER / 2], a2[NC][PER / 2];
    float bias[NC], dw[NC], dt_sum[NC];
#pragma unroll
    for (int k = 0; k < NC; k++) {
        load_states<PER>(a2[k], a.A2 + (size_t)(cc + k) * a.N, l * PER, a.N, vec);
        const float* enter = MODE == 2 && g > 0 ? a.seg_state + (((size_t)b * n_seg + g - 1) * a.C + cc + k) * a.N
                                                : a.state + ((size_t)slot * a.C + cc + k) * a.N;
        if (MODE == 1) {
#pragma unroll
            for (int i = 0; i < PER / 2; i++) s[k][i] = 0ull;
        } else {
            load_states<PER>(s[k], enter, l * PER, a.N, vec);
        }
        bias[k] = a.dt_bias[cc + k];
        dw[k] = a.Dw[cc + k];
        dt_sum[k] = 0.f;
    }
    float dt[AHEAD][NC], u[AHEAD][NC], z[AHEAD][NC];
    auto fetch = [&](int t0) {                              // tokens t0 .. t0 + AHEAD - 1 of the sequence (clamped to n - 1)
#pragma unroll
        for (int k = 0; k < AHEAD; k++) {
            const size_t row = (size_t)(row0 + min(t0 + k, n - 1));
            load_channels<float, NC>(dt[k], a.zdt + row * a.C + cc);
            load_channels<T, NC>(u[k], a.u + row * a.C + cc);
            if (OUT) load_channels<T, NC>(z[k], a.z + row * a.ldz + cc);
        }
    };
    fetch(first);
    for (int c0 = first; c0 < n; c0 += CHUNK) {
        const int cn = min(CHUNK, n - c0);
        __syncthreads();
        for (int e = threadIdx.x; e < cn * NP; e += THREADS) {
            const int tt = e / NP, i = e % NP;
            const float* row = a.thin + (size_t)(row0 + c0 + tt) * a.ldthin;
            stage[0][tt][i] = i < a.N ? row[a.off_b + i] : 0.f;
            if (OUT) stage[1][tt][i] = i < a.N ? row[a.off_c + i] : 0.f;
        }
        __syncthreads();
        for (int t4 = 0; t4 < cn; t4 += AHEAD) {
            // what does not depend on the state comes first, for all of these tokens
            float d_all[AHEAD][NC], u_now[AHEAD][NC], gate[AHEAD][NC];
#pragma unroll
            for (int k = 0; k < AHEAD; k++)
#pragma unroll
                for (int e = 0; e < NC; e++) {
                    d_all[k][e] = softplus_f(dt[k][e] + bias[e]);
                    u_now[k][e] = u[k][e];
                    if (OUT) gate[k][e] = gate_silu<T>(z[k][e]);
                }
            if (c0 + t4 + AHEAD < n) fetch(c0 + t4 + AHEAD);
#pragma unroll
            for (int k = 0; k < AHEAD; k++) {
                if (t4 + k < cn) {
                    float d[NC], du[NC], y[NC];
#pragma unroll
                    for (int e = 0; e < NC; e++) {
                        d[e] = d_all[k][e];
                        du[e] = d[e] * u_now[k][e];
                        if (MODE == 1) dt_sum[e] += d[e];
                    }
                    scan_token<NC, PER, OUT>(s, a2, d, du, &stage[0][t4 + k][l * PER], &stage[1][t4 + k][l * PER], y);
                    if (OUT) {
#pragma unroll
                        for (int e = 0; e < NC; e++) y[e] = fmaf(dw[e], u_now[k][e], lanes_sum<L>(y[e])) * gate[k][e];
                        T* dst = a.y + (size_t)(row0 + c0 + t4 + k) * a.C + c;
                        if (mine && l == 0) {
                            if constexpr (NC == 2 && sizeof(T) == 2) *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(y[0], y[1]);
                            else
#pragma unroll
                                for (int e = 0; e < NC; e++) dst[e] = from_f32<T>(y[e]);
                        }
                    }
                }
            }
        }
    }
    if (!mine) return;
#pragma unroll
    for (int k = 0; k < NC; k++) {
        if (MODE == 1) {
            store_states<PER>(a.seg_state + (((size_t)b * n_seg + g) * a.C + c + k) * a.N, s[k], l * PER, a.N, vec);
            if (l == 0) a.seg_dt[((size_t)b * n_seg + g) * a.C + c + k] = dt_sum[k];
        } else if (last) {
            store_states<PER>(a.state + ((size_t)slot * a.C + c + k) * a.N, s[k], l * PER, a.N, vec);
        }
    }
}

// seg_state[b][g] becomes what segment g + 1 starts from.  One thread per (channel, state); grid (blocks, sequences).
__global__ void __launch_bounds__(256)
selective_join_kernel(const float* state, float* seg_state, const float* seg_dt, const float* __restrict__ A2,
                      const int* __restrict__ seq_slot, const int* __restrict__ cu_q, int C, int N, int seg_len, int n_seg) {
    pdl_launch_dependents();
    pdl_wait();
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x, CN = (long long)C * N;
    const int b = blockIdx.y;
    const int slot = seq_slot[b], n = cu_q[b + 1] - cu_q[b];
    if (slot < 0 || e >= CN) return;
    const int c = (int)(e / N);
    const float a2 = A2[e];
    float s = state[(long long)slot * CN + e];
    for (int g = 0; (g + 1) * seg_len < n; g++) {
        const size_t at = (size_t)b * n_seg + g;
        s = fmaf(decay_exp2(seg_dt[at * C + c] * a2), s, seg_state[at * CN + e]);
        seg_state[at * CN + e] = s;
    }
}

// One token per sequence.  grid (channel tiles, groups of SG sequences): the weights of the step sizes are read once for a
// group's sequences.  W [C, ldw], ldw a multiple of 8 (zeros behind the rank), r at column off_r of `thin`.
template <typename T, int PER, int L, int SG>
__global__ void __launch_bounds__(THREADS)
selective_step_kernel(const ScanArgs<T> a, const T* __restrict__ W, int ldw, int off_r, int rank, int n_seqs) {
    constexpr int CPB = THREADS / L, NP = PER * L;
    extern __shared__ __align__(16) float staged[];         // per sequence: r [ldw], b [NP], c [NP]
    pdl_launch_dependents();
    pdl_wait();
    const int l = threadIdx.x % L, c = blockIdx.x * CPB + threadIdx.x / L;
    const bool mine = c < a.C;
    const int cc = mine ? c : a.C - 1;
    const bool vec = a.N % 4 == 0;
    const int per_seq = ldw + 2 * NP;
    int slot[SG], row[SG];
#pragma unroll
    for (int k = 0; k < SG; k++) {
        const int b = blockIdx.y * SG + k;
        slot[k] = b < n_seqs ? a.seq_slot[b] : -1;
        row[k] = b < n_seqs ? a.cu_q[b] : 0;
        if (slot[k] >= 0 && a.cu_q[b + 1] <= row[k]) slot[k] = -1;
    }
    f32x2 s[SG][1][PER / 2], a2[1][PER / 2];
    float u[SG], z[SG];
    load_states<PER>(a2[0], a.A2 + (size_t)cc * a.N, l * PER, a.N, vec);
#pragma unroll
    for (int k = 0; k < SG; k++) {
        u[k] = z[k] = 0.f;
        if (slot[k] < 0) continue;
        load_states<PER>(s[k][0], a.state + ((size_t)slot[k] * a.C + cc) * a.N, l * PER, a.N, vec);
        u[k] = to_f32(a.u[(size_t)row[k] * a.C + cc]);
        z[k] = to_f32(a.z[(size_t)row[k] * a.ldz + cc]);
        const float* tr = a.thin + (size_t)row[k] * a.ldthin;
        float* dst = staged + k * per_seq;
        for (int i = threadIdx.x; i < ldw; i += THREADS) dst[i] = i < rank ? tr[off_r + i] : 0.f;
        for (int i = threadIdx.x; i < NP; i += THREADS) {
            dst[ldw + i] = i < a.N ? tr[a.off_b + i] : 0.f;
            dst[ldw + NP + i] = i < a.N ? tr[a.off_c + i] : 0.f;
        }
    }
    __syncthreads();
    float zd[SG];
#pragma unroll
    for (int k = 0; k < SG; k++) zd[k] = 0.f;
    for (int j = l * 8; j < ldw; j += L * 8) {
        float w[8];
        load_vec<T, 8>(w, W + (size_t)cc * ldw + j);
#pragma unroll
        for (int k = 0; k < SG; k++) {
            const float4 p = *reinterpret_cast<const float4*>(staged + k * per_seq + j);
            const float4 q = *reinterpret_cast<const float4*>(staged + k * per_seq + j + 4);
            if (slot[k] < 0) continue;
            float d = zd[k];
            d = fmaf(w[0], p.x, d); d = fmaf(w[1], p.y, d); d = fmaf(w[2], p.z, d); d = fmaf(w[3], p.w, d);
            d = fmaf(w[4], q.x, d); d = fmaf(w[5], q.y, d); d = fmaf(w[6], q.z, d); d = fmaf(w[7], q.w, d);
            zd[k] = d;
        }
    }
    const float bias = a.dt_bias[cc], dw = a.Dw[cc];
#pragma unroll
    for (int k = 0; k < SG; k++) {
        if (slot[k] < 0) continue;                          // the same for the whole block
        const float dt = softplus_f(lanes_sum<L>(zd[k]) + bias);
        const float* st = staged + k * per_seq + ldw + l * PER;
        const float d[1] = {dt}, du[1] = {dt * u[k]};
        float y[1];
        scan_token<1, PER, true>(s[k], a2, d, du, st, st + NP, y);
        y[0] = lanes_sum<L>(y[0]);
        if (!mine) continue;
        if (l == 0) a.y[(size_t)row[k] * a.C + c] = from_f32<T>(fmaf(dw, u[k], y[0]) * gate_silu<T>(z[k]));
        store_states<PER>(a.state + ((size_t)slot[k] * a.C + c) * a.N, s[k][0], l * PER, a.N, vec);
    }
}

inline int lanes_for(int N, int per) {
    int L = 1;
    while (L * per < N) L *= 2;
    return L;
}

template <typename T>
int launch_conv(T* out, const T* x, long long ldx, const float* w, const float* bias, int taps, float* state,
                const int* tok_seq, const int* seq_slot, const int* cu_q, int n_tokens, int n_seqs, int C, int one_each,
                cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (taps < 1 || taps > MAX_TAPS || C < 1) return OE_ERR_UNSUPPORTED;
    if (taps < 2 || taps > 4) {
        const dim3 grid(n_tokens, (C + THREADS - 1) / THREADS);
        if (grid.y > 65535) return OE_ERR_UNSUPPORTED;
        return oe_launch(causal_conv_any_kernel<T>, grid, dim3(THREADS), 0, st, out, x, ldx, w, bias, taps, (const float*)state, tok_seq, seq_slot, cu_q, C);
    }
    // four channels a thread where the rows allow it and there are enough tokens; few tokens: a thread per channel
    constexpr int V = 4;
    constexpr int PT = 8;
    const bool vec = C % V == 0 && ldx % V == 0 && !one_each &&
                     !(((uintptr_t)out | (uintptr_t)x | (uintptr_t)state | (uintptr_t)w | (uintptr_t)bias) & 15) &&
                     (long long)n_tokens * C >= (1LL << 20);
    const int width = THREADS * (vec ? V : 1);
    const dim3 grid(vec ? (n_tokens + PT - 1) / PT : n_tokens, (C + width - 1) / width);
    if (grid.y > 65535) return OE_ERR_UNSUPPORTED;
#define OE_CONV(TAPS)                                                                                                          \
    if (taps == TAPS) {                                                                                                        \
        if (vec) return oe_launch(causal_conv_kernel<T, TAPS, V, PT>, grid, dim3(THREADS), 0, st, out, x, ldx, w, bias, state, \
                                  tok_seq, seq_slot, cu_q, n_tokens, C, one_each);                                             \
        return oe_launch(causal_conv_kernel<T, TAPS, 1, 1>, grid, dim3(THREADS), 0, st, out, x, ldx, w, bias, state, tok_seq,  \
                         seq_slot, cu_q, n_tokens, C, one_each);                                                               \
    }
    OE_CONV(2) OE_CONV(3) OE_CONV(4)
#undef OE_CONV
    return OE_ERR_UNSUPPORTED;
}

template <typename T>
int launch_rows_state(float* state, const T* x, long long ldx, int C, int taps, const int* seq_slot, const int* cu_q, int n_seqs,
                      cudaStream_t st) {
    if (n_seqs <= 0 || taps <= 1) return 0;
    if (taps > MAX_TAPS || C < 1) return OE_ERR_UNSUPPORTED;
    return oe_launch(conv_rows_state_kernel<T>, dim3(n_seqs, (C + THREADS - 1) / THREADS), dim3(THREADS), 0, st, state, x, ldx, C,
                     taps, seq_slot, cu_q);
}

constexpr long long BUSY_THREADS = 148LL * 1024;        // threads that keep the GPU busy

template <typename T>
int launch_scan(const ScanArgs<T>& a, int n_seqs, cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    if (a.C < 1 || a.N < 1 || a.N > 256 || n_seqs > 65535) return OE_ERR_UNSUPPORTED;
    // few channels and sequences: a channel's states over more lanes.  float32: the same lanes whatever the batch, so that
    // the order of a read-out's sum is always the same
    const long long pairs = (sizeof(T) == 4 ? 1LL : (long long)n_seqs) * a.C;
    int per = 4;
    while (per < 16 && per < a.N && (lanes_for(a.N, per) > 32 || pairs * lanes_for(a.N, per) > BUSY_THREADS)) per *= 2;
    const int L = lanes_for(a.N, per);
    const dim3 grid((a.C + THREADS / L - 1) / (THREADS / L), n_seqs);
#define OE_SCAN(P, LL) if (per == P && L == LL) return oe_launch(selective_scan_kernel<T, P, LL, 0, 1>, grid, dim3(THREADS), 0, st, a);
    OE_SCAN(4, 1) OE_SCAN(4, 2) OE_SCAN(4, 4) OE_SCAN(4, 8) OE_SCAN(4, 16) OE_SCAN(4, 32)
    OE_SCAN(8, 1) OE_SCAN(8, 2) OE_SCAN(8, 4) OE_SCAN(8, 8) OE_SCAN(8, 16) OE_SCAN(8, 32)
    OE_SCAN(16, 1) OE_SCAN(16, 2) OE_SCAN(16, 4) OE_SCAN(16, 8) OE_SCAN(16, 16)
#undef OE_SCAN
    return OE_ERR_UNSUPPORTED;
}

int launch_segments(const ScanArgs<bf16>& a, int n_seqs, int n_seg, cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    if (a.C < 1 || a.N < 1 || a.N > 256 || n_seqs > 65535 || n_seg < 1 || n_seg > 65535 || a.seg_len < 1 ||
        a.seg_state == nullptr || a.seg_dt == nullptr)
        return OE_ERR_UNSUPPORTED;
    int per = 8;
    while (per < 16 && per < a.N && (lanes_for(a.N, per) > 32 || (long long)n_seqs * n_seg * a.C * lanes_for(a.N, per) > BUSY_THREADS)) per *= 2;
    const int L = lanes_for(a.N, per);
    // two channels a lane, so that what is read of b and c serves both
    const bool two = a.C % 2 == 0 && a.ldz % 2 == 0 && !(((uintptr_t)a.u | (uintptr_t)a.z | (uintptr_t)a.y) & 3) && !((uintptr_t)a.zdt & 7);
    const int cpb = THREADS / L * (two ? 2 : 1);
    const dim3 grid((a.C + cpb - 1) / cpb, n_seqs, n_seg);
    const long long blocks = ((long long)a.C * a.N + 255) / 256;
#define OE_SCAN(P, LL)                                                                                                         \
    if (per == P && L == LL) {                                                                                                 \
        int rc = two ? oe_launch(selective_scan_kernel<bf16, P, LL, 1, 2>, grid, dim3(THREADS), 0, st, a)                      \
                     : oe_launch(selective_scan_kernel<bf16, P, LL, 1, 1>, grid, dim3(THREADS), 0, st, a);                     \
        if (rc) return rc;                                                                                                     \
        rc = oe_launch(selective_join_kernel, dim3((unsigned)blocks, n_seqs), dim3(256), 0, st, (const float*)a.state, a.seg_state, \
                       (const float*)a.seg_dt, a.A2, a.seq_slot, a.cu_q, a.C, a.N, a.seg_len, n_seg);                          \
        if (rc) return rc;                                                                                                     \
        if (two) return oe_launch(selective_scan_kernel<bf16, P, LL, 2, 2>, grid, dim3(THREADS), 0, st, a);                    \
        return oe_launch(selective_scan_kernel<bf16, P, LL, 2, 1>, grid, dim3(THREADS), 0, st, a);                             \
    }
    OE_SCAN(8, 1) OE_SCAN(8, 2) OE_SCAN(8, 4) OE_SCAN(8, 8) OE_SCAN(8, 16) OE_SCAN(8, 32)
    OE_SCAN(16, 1) OE_SCAN(16, 2) OE_SCAN(16, 4) OE_SCAN(16, 8) OE_SCAN(16, 16)
#undef OE_SCAN
    return OE_ERR_UNSUPPORTED;
}

template <typename T>
int launch_step(const ScanArgs<T>& a, const T* W, int ldw, int off_r, int rank, int n_seqs, cudaStream_t st) {
    if (n_seqs <= 0) return 0;
    if (a.C < 1 || a.N < 1 || a.N > 256 || ldw < rank || ldw % 8 || rank < 1 || ((uintptr_t)W & 15)) return OE_ERR_UNSUPPORTED;
    const int per = a.N <= 128 ? 4 : 8, L = lanes_for(a.N, per);
    const int tiles = (a.C + THREADS / L - 1) / (THREADS / L);
    // groups of sequences where enough blocks are left to fill the GPU and the groups' rows fit
    const int sg = (long long)tiles * n_seqs > 4 * 148 * 4 && (size_t)4 * (ldw + 2 * per * L) * sizeof(float) <= 48 * 1024 ? 4 : 1;
    const dim3 grid(tiles, (n_seqs + sg - 1) / sg);
    const size_t smem = (size_t)sg * (ldw + 2 * per * L) * sizeof(float);
    if (grid.y > 65535 || smem > 48 * 1024) return OE_ERR_UNSUPPORTED;
#define OE_STEP(P, LL)                                                                                                         \
    if (per == P && L == LL) {                                                                                                 \
        if (sg == 1) return oe_launch(selective_step_kernel<T, P, LL, 1>, grid, dim3(THREADS), smem, st, a, W, ldw, off_r, rank, n_seqs); \
        return oe_launch(selective_step_kernel<T, P, LL, 4>, grid, dim3(THREADS), smem, st, a, W, ldw, off_r, rank, n_seqs);   \
    }
    OE_STEP(4, 1) OE_STEP(4, 2) OE_STEP(4, 4) OE_STEP(4, 8) OE_STEP(4, 16) OE_STEP(4, 32) OE_STEP(8, 32)
#undef OE_STEP
    return OE_ERR_UNSUPPORTED;
}

template <typename T>
ScanArgs<T> make_args(T* y, float* state, const T* u, const float* zdt, const float* dt_bias, const float* thin, long long ldthin,
                      int off_b, int off_c, const float* A2, const float* Dw, const T* z, long long ldz, const int* seq_slot,
                      const int* cu_q, int C, int N) {
    ScanArgs<T> a;
    a.y = y; a.state = state; a.u = u; a.zdt = zdt; a.dt_bias = dt_bias; a.thin = thin; a.ldthin = ldthin; a.off_b = off_b;
    a.off_c = off_c; a.A2 = A2; a.Dw = Dw; a.z = z; a.ldz = ldz; a.seq_slot = seq_slot; a.cu_q = cu_q; a.C = C; a.N = N;
    a.seg_len = 0; a.seg_state = nullptr; a.seg_dt = nullptr;
    return a;
}

}  // namespace

extern "C" {

int oe_thin_cast(bf16* out, const float* in, long long ld, int n_tokens, int n, cudaStream_t st) {
    if (n_tokens <= 0 || n <= 0) return 0;
    const size_t total = (size_t)n_tokens * n;
    const size_t blocks = (total + 255) / 256;
    return oe_launch(thin_cast_kernel, dim3((unsigned)(blocks < 148 * 16 ? blocks : 148 * 16)), dim3(256), 0, st, out, in, ld, n_tokens, n);
}

#define OE_TYPED(SUFFIX, T)                                                                                                    \
    int oe_causal_conv_##SUFFIX(T* out, const T* x, long long ldx, const float* w, const float* bias, int taps, float* state,  \
                                const int* tok_seq, const int* seq_slot, const int* cu_q, int n_tokens, int n_seqs, int C,     \
                                int one_each, cudaStream_t st) {                                                               \
        return launch_conv<T>(out, x, ldx, w, bias, taps, state, tok_seq, seq_slot, cu_q, n_tokens, n_seqs, C, one_each, st);   \
    }                                                                                                                          \
    int oe_conv_rows_state_##SUFFIX(float* state, const T* x, long long ldx, int C, int taps, const int* seq_slot,             \
                                    const int* cu_q, int n_seqs, cudaStream_t st) {                                            \
        return launch_rows_state<T>(state, x, ldx, C, taps, seq_slot, cu_q, n_seqs, st);                                       \
    }                                                                                                                          \
    int oe_selective_scan_##SUFFIX(T* y, float* state, const T* u, const float* zdt, const float* dt_bias, const float* thin,  \
                                   long long ldthin, int off_b, int off_c, const float* A2, const float* Dw, const T* z,       \
                                   long long ldz, const int* seq_slot, const int* cu_q, int n_seqs, int C, int N,              \
                                   cudaStream_t st) {                                                                          \
        return launch_scan<T>(make_args<T>(y, state, u, zdt, dt_bias, thin, ldthin, off_b, off_c, A2, Dw, z, ldz, seq_slot,    \
                                           cu_q, C, N), n_seqs, st);                                                           \
    }                                                                                                                          \
    int oe_selective_step_##SUFFIX(T* y, float* state, const T* u, const T* W, int ldw, int off_r, int rank,                   \
                                   const float* dt_bias, const float* thin, long long ldthin, int off_b, int off_c,            \
                                   const float* A2, const float* Dw, const T* z, long long ldz, const int* seq_slot,           \
                                   const int* cu_q, int n_seqs, int C, int N, cudaStream_t st) {                               \
        return launch_step<T>(make_args<T>(y, state, u, nullptr, dt_bias, thin, ldthin, off_b, off_c, A2, Dw, z, ldz,          \
                                           seq_slot, cu_q, C, N), W, ldw, off_r, rank, n_seqs, st);                            \
    }
OE_TYPED(f32, float)
OE_TYPED(bf16, bf16)
#undef OE_TYPED

// seg_state [n_seqs, n_seg, C, N] and seg_dt [n_seqs, n_seg, C] are scratch; sequences bring up to n_seg * seg_len tokens.
int oe_selective_scan_segments(bf16* y, float* state, const bf16* u, const float* zdt, const float* dt_bias, const float* thin,
                               long long ldthin, int off_b, int off_c, const float* A2, const float* Dw, const bf16* z,
                               long long ldz, const int* seq_slot, const int* cu_q, int n_seqs, int C, int N, int seg_len,
                               int n_seg, float* seg_state, float* seg_dt, cudaStream_t st) {
    ScanArgs<bf16> a = make_args<bf16>(y, state, u, zdt, dt_bias, thin, ldthin, off_b, off_c, A2, Dw, z, ldz, seq_slot, cu_q, C, N);
    a.seg_len = seg_len; a.seg_state = seg_state; a.seg_dt = seg_dt;
    return launch_segments(a, n_seqs, n_seg, st);
}

}  // extern "C"
