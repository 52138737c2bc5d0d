// What an attention with normed, turned queries, keys AND values does around its softmax.
//
//   qkv_norm_rot_write   one warp per (token, head) of the float32 projection row [q: H dk | k: G dk | v: G dv]:
//                        + bias;  q and k heads: / sqrt(mean(.^2) + eps) * weight (a weight of dk values shared by the
//                        heads), then the first `rot` dimensions turned by the token's position (i paired with
//                        i + rot/2, cosine and sine from a float32 table [positions, rot/2]);  v heads: / sqrt(mean(.^2)
//                        + eps) without a weight, then ALL dv dimensions turned by the position (m paired with m + dv/2,
//                        a table [positions, dv/2] of its own).  q goes to a contiguous [T, H dk] tensor of the compute
//                        type, k and v to the token's rows of the paged cache [pages, G, PAGE, dk] / [pages, G, PAGE, dv].
//                        Each of bias, norm, key rotation, value norm and value rotation can be absent.
//   unrotate_heads       every head of o [T, H dv] turned back by its own token's position (angle -pos * f_m), in place:
//                        with values stored turned by the key's position, a softmax-weighted sum turned back by the
//                        query's position depends on the values through relative positions only.
//   qkv_row_norm_rot_write   one block per token of the row [q: H dk | k: G dk | v: G dv | ...] (float32 or bfloat16): q
//                        divided by the root mean square of ALL its H dk values and times a weight of that size, k likewise
//                        over its G dk values (the norm may be absent); then the first `rot` dimensions of every head
//                        turned by the token's position, 2i paired with 2i + 1 or i with i + rot/2.  q goes back in place, k
//                        and v to the token's cache rows.
// All arithmetic is float32.
#include "common.cuh"

namespace {

constexpr int MAX_D = 256;
constexpr int WARPS = 4;

struct PrepArgs {
    const float* proj; long long ld;
    const float* qb; const float* kb; const float* vb;        // biases [H dk], [G dk], [G dv] or null
    const float* qw; const float* kw;                          // norm weights [dk] or null (null: no norm of q / k)
    float eps;
    const float* cos_k; const float* sin_k; int rot;           // key rotation table [positions, rot/2]; rot 0: none
    const float* cos_v; const float* sin_v;                    // value rotation table [positions, dv/2] or null
    int v_norm;
    const int* tables; int max_pages;
    const int* tok_seq; const int* tok_pos;
    int n_tokens, H, G, dk, dv;
};

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
qkv_norm_rot_write_kernel(T* q_out, T* kcache, T* vcache, const PrepArgs a) {
    __shared__ float stage[WARPS][MAX_D];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int heads = a.H + 2 * a.G;
    const long long item = (long long)blockIdx.x * WARPS + warp;
    if (item >= (long long)a.n_tokens * heads) return;
    const int t = (int)(item / heads), hh = (int)(item % heads);
    const int b = a.tok_seq[t];
    if (b < 0) return;
    const int pos = a.tok_pos[t];
    const int kind = hh < a.H ? 0 : (hh < a.H + a.G ? 1 : 2);            // q, k, v
    const int head = kind == 0 ? hh : (kind == 1 ? hh - a.H : hh - a.H - a.G);
    const int d = kind == 2 ? a.dv : a.dk;
    const long long col0 = kind == 0 ? (long long)head * a.dk
                         : (kind == 1 ? (long long)a.H * a.dk + (long long)head * a.dk
                                      : (long long)(a.H + a.G) * a.dk + (long long)head * a.dv);
    const float* src = a.proj + (size_t)t * a.ld + col0;
    const float* bias = kind == 0 ? a.qb : (kind == 1 ? a.kb : a.vb);
    const float* w = kind == 0 ? a.qw : (kind == 1 ? a.kw : nullptr);
    const bool normed = kind == 2 ? a.v_norm != 0 : w != nullptr;
    // everything a lane loads is asked for before the sums: the row's values, the bias, the norm weight and the angles
    const int rot = kind == 2 ? (a.cos_v ? a.dv : 0) : a.rot;
    const int half = rot / 2;
    const float* cr = (kind == 2 ? a.cos_v : a.cos_k) + (size_t)pos * half;
    const float* sr = (kind == 2 ? a.sin_v : a.sin_k) + (size_t)pos * half;
    const int page = kind == 0 ? 0 : a.tables[(size_t)b * a.max_pages + pos / OE_PAGE];
    float v[MAX_D / 32], wn[MAX_D / 32], cs[MAX_D / 32], sn[MAX_D / 32];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < MAX_D / 32; j++) {
        const int i = lane + 32 * j;
        v[j] = 0.f; wn[j] = 1.f; cs[j] = 1.f; sn[j] = 0.f;
        if (i < d) {
            v[j] = src[i] + (bias ? bias[(kind == 2 ? (long long)head * a.dv : (long long)head * a.dk) + i] : 0.f);
            if (w) wn[j] = w[i];
            if (i < rot) { const int m = i < half ? i : i - half; cs[j] = cr[m]; sn[j] = sr[m]; }
        }
    }
#pragma unroll
    for (int j = 0; j < MAX_D / 32; j++) ss = fmaf(v[j], v[j], ss);
    ss = warp_sum(ss);
    const float s = normed ? 1.f / sqrtf(ss / (float)d + a.eps) : 1.f;
    float* sm = stage[warp];
#pragma unroll
    for (int j = 0; j < MAX_D / 32; j++) {
        const int i = lane + 32 * j;
        v[j] = (v[j] * s) * wn[j];
        if (i < rot) sm[i] = v[j];               // only the turned dimensions need their partner
    }
    __syncwarp();
    T* dst;
    if (kind == 0) {
        dst = q_out + ((size_t)t * a.H + head) * a.dk;
    } else {
        if (page < 0) return;
        dst = (kind == 1 ? kcache : vcache) + (((size_t)page * a.G + head) * OE_PAGE + (pos % OE_PAGE)) * d;
    }
#pragma unroll
    for (int j = 0; j < MAX_D / 32; j++) {
        const int i = lane + 32 * j;
        if (i >= d) continue;
        float r = v[j];
        if (i < half) r = v[j] * cs[j] - sm[i + half] * sn[j];
        else if (i < rot) r = v[j] * cs[j] + sm[i - half] * sn[j];
        dst[i] = from_f32<T>(r);
    }
}

struct RowPrepArgs {
    long long ld;
    const float* qw; const float* kw; float eps;
    const float* cos_t; const float* sin_t; int rot, halves;
    const int* tables; int max_pages;
    const int* tok_seq; const int* tok_pos;
    int n_tokens, H, G, dk, dv;
};

constexpr int ROW_THREADS = 256;

// A turned pair of head values: where its two values lie behind the first column of the head.
__device__ __forceinline__ void pair_columns(int i, int rot, int halves, int& first, int& second) {
    if (halves) { first = i; second = i + rot / 2; }
    else { first = 2 * i; second = 2 * i + 1; }
}

// bfloat16 rows in 16-byte pieces: dk, dv and rot multiples of 8, pairs interleaved, so that a piece holds four pairs of one
// head or eight values that pass.  The row's pieces stay in registers between the sums and the turn.
template <int KEEP>
__global__ void __launch_bounds__(ROW_THREADS)
qkv_row_norm_rot_write_vec_kernel(bf16* qkv, bf16* kcache, bf16* vcache, const RowPrepArgs a) {
    __shared__ float red[2][32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int b = a.tok_seq[t];
    if (b < 0) return;
    const int pos = a.tok_pos[t];
    const int page = a.tables[(size_t)b * a.max_pages + pos / OE_PAGE];
    bf16* row = qkv + (size_t)t * a.ld;
    const int qp = a.H * a.dk / 8, kp = a.G * a.dk / 8, vp = a.G * a.dv / 8;
    uint4 keep[KEEP];
    float s = 0.f, u = 0.f;
#pragma unroll
    for (int j = 0; j < KEEP; j++) {
        const int e = threadIdx.x + j * ROW_THREADS;
        keep[j] = make_uint4(0u, 0u, 0u, 0u);
        if (e < qp + kp + vp) keep[j] = reinterpret_cast<const uint4*>(row)[e];
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&keep[j]);
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 4; i++) { const float2 f = __bfloat1622float2(p[i]); ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss)); }
        if (e < qp) s += ss;
        else if (e < qp + kp) u += ss;
    }
    float sq = 1.f, sk = 1.f;
    if (a.qw) {
        s = block_sum(s, red[0]);
        u = block_sum(u, red[1]);
        sq = 1.f / sqrtf(s / (float)(a.H * a.dk) + a.eps);
        sk = 1.f / sqrtf(u / (float)(a.G * a.dk) + a.eps);
    }
    const float* cr = a.cos_t + (size_t)pos * (a.rot / 2);
    const float* sr = a.sin_t + (size_t)pos * (a.rot / 2);
#pragma unroll
    for (int j = 0; j < KEEP; j++) {
        const int e = threadIdx.x + j * ROW_THREADS;
        if (e >= qp + kp + vp) continue;
        if (e >= qp && page < 0) continue;
        if (e >= qp + kp) {
            const int c = (e - qp - kp) * 8, head = c / a.dv;
            *reinterpret_cast<uint4*>(vcache + (((size_t)page * a.G + head) * OE_PAGE + (pos % OE_PAGE)) * a.dv + (c - head * a.dv)) = keep[j];
            continue;
        }
        const bool key = e >= qp;
        const int c = (key ? e - qp : e) * 8, head = c / a.dk, d = c - head * a.dk;
        const float sc = key ? sk : sq;
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&keep[j]);
        float v[8];
#pragma unroll
        for (int i = 0; i < 4; i++) { const float2 f = __bfloat1622float2(p[i]); v[2 * i] = f.x * sc; v[2 * i + 1] = f.y * sc; }
        if (a.qw) {
            const float4* w = reinterpret_cast<const float4*>((key ? a.kw : a.qw) + c);
            const float4 w0 = w[0], w1 = w[1];
            v[0] *= w0.x; v[1] *= w0.y; v[2] *= w0.z; v[3] *= w0.w; v[4] *= w1.x; v[5] *= w1.y; v[6] *= w1.z; v[7] *= w1.w;
        }
        if (d < a.rot) {
            const float4 cs = *reinterpret_cast<const float4*>(cr + d / 2), sn = *reinterpret_cast<const float4*>(sr + d / 2);
            const float cc[4] = {cs.x, cs.y, cs.z, cs.w}, ss[4] = {sn.x, sn.y, sn.z, sn.w};
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float x = v[2 * i], y = v[2 * i + 1];
                v[2 * i] = x * cc[i] - y * ss[i];
                v[2 * i + 1] = y * cc[i] + x * ss[i];
            }
        }
        __nv_bfloat162 o[4];
#pragma unroll
        for (int i = 0; i < 4; i++) o[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        bf16* dst = key ? kcache + (((size_t)page * a.G + head) * OE_PAGE + (pos % OE_PAGE)) * a.dk + d : row + c;
        *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(o);
    }
}

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
qkv_row_norm_rot_write_kernel(T* qkv, T* kcache, T* vcache, const RowPrepArgs a) {
    __shared__ float red[2][32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int b = a.tok_seq[t];
    if (b < 0) return;
    const int pos = a.tok_pos[t];
    const int page = a.tables[(size_t)b * a.max_pages + pos / OE_PAGE];
    T* row = qkv + (size_t)t * a.ld;
    const int qn = a.H * a.dk, kn = a.G * a.dk, vn = a.G * a.dv;
    T* krow = row + qn;
    const T* vrow = krow + kn;
    float sq = 1.f, sk = 1.f;
    if (a.qw) {
        float s = 0.f, u = 0.f;
        for (int i = threadIdx.x; i < qn; i += ROW_THREADS) { const float v = to_f32(row[i]); s = fmaf(v, v, s); }
        for (int i = threadIdx.x; i < kn; i += ROW_THREADS) { const float v = to_f32(krow[i]); u = fmaf(v, v, u); }
        s = block_sum(s, red[0]);
        u = block_sum(u, red[1]);
        sq = 1.f / sqrtf(s / (float)qn + a.eps);
        sk = 1.f / sqrtf(u / (float)kn + a.eps);
    }
    const int half = a.rot / 2;
    const float* cr = a.cos_t + (size_t)pos * half;
    const float* sr = a.sin_t + (size_t)pos * half;
    const int rest = a.dk - half;                 // what a head takes: `half` pairs, then the dimensions that pass
    // q and k heads: a thread owns whole pairs, so that it may write where it read
    for (int e = threadIdx.x; e < (a.H + a.G) * rest; e += ROW_THREADS) {
        const int hh = e / rest, i = e % rest;
        const bool key = hh >= a.H;
        const int head = key ? hh - a.H : hh;
        if (key && page < 0) continue;
        const T* src = (key ? krow : row) + (size_t)head * a.dk;
        T* dst = key ? kcache + (((size_t)page * a.G + head) * OE_PAGE + (pos % OE_PAGE)) * a.dk : row + (size_t)head * a.dk;
        const float* w = a.qw ? (key ? a.kw : a.qw) + (size_t)head * a.dk : nullptr;
        const float s = key ? sk : sq;
        if (i < half) {
            int c0, c1;
            pair_columns(i, a.rot, a.halves, c0, c1);
            const float u = to_f32(src[c0]) * s * (w ? w[c0] : 1.f), v = to_f32(src[c1]) * s * (w ? w[c1] : 1.f);
            dst[c0] = from_f32<T>(u * cr[i] - v * sr[i]);
            dst[c1] = from_f32<T>(v * cr[i] + u * sr[i]);
        } else {
            const int c = i + half;
            dst[c] = from_f32<T>(to_f32(src[c]) * s * (w ? w[c] : 1.f));
        }
    }
    if (page < 0) return;
    for (int e = threadIdx.x; e < vn; e += ROW_THREADS)
        vcache[(((size_t)page * a.G + e / a.dv) * OE_PAGE + (pos % OE_PAGE)) * a.dv + e % a.dv] = vrow[e];
}

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
unrotate_heads_kernel(T* o, const float* __restrict__ cos_v, const float* __restrict__ sin_v,
                      const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, int n_tokens, int H, int dv) {
    __shared__ float stage[WARPS][MAX_D];
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * WARPS + warp;
    if (item >= (long long)n_tokens * H) return;
    const int t = (int)(item / H);
    if (tok_seq[t] < 0) return;
    const int pos = tok_pos[t];
    const int half = dv / 2;
    T* row = o + (size_t)item * dv;
    float* sm = stage[warp];
    for (int i = lane; i < dv; i += 32) sm[i] = to_f32(row[i]);
    __syncwarp();
    const float* cr = cos_v + (size_t)pos * half;
    const float* sr = sin_v + (size_t)pos * half;
    for (int i = lane; i < 2 * half; i += 32) {
        // the turn by -angle: (u, v) -> (u c + v s, v c - u s)
        const float r = i < half ? sm[i] * cr[i] + sm[i + half] * sr[i] : sm[i] * cr[i - half] - sm[i - half] * sr[i - half];
        row[i] = from_f32<T>(r);
    }
}

template <typename T>
int launch_prep(T* q_out, T* kcache, T* vcache, const PrepArgs& a, cudaStream_t st) {
    if (a.n_tokens <= 0) return 0;
    if (a.dk < 1 || a.dk > MAX_D || a.dv < 1 || a.dv > MAX_D || a.H < 1 || a.G < 1 || a.rot < 0 || a.rot % 2 || a.rot > a.dk
        || (a.cos_v && a.dv % 2))
        return OE_ERR_UNSUPPORTED;
    const long long items = (long long)a.n_tokens * (a.H + 2 * a.G);
    const long long blocks = (items + WARPS - 1) / WARPS;
    if (blocks > 2147483647LL) return OE_ERR_UNSUPPORTED;
    return oe_launch(qkv_norm_rot_write_kernel<T>, dim3((unsigned)blocks), dim3(WARPS * 32), 0, st, q_out, kcache, vcache, a);
}

template <typename T>
int launch_row_prep(T* qkv, long long ld, T* kcache, T* vcache, const float* qw, const float* kw, float eps, const float* cos_t,
                    const float* sin_t, int rot, int halves, const int* tables, int max_pages, const int* tok_seq,
                    const int* tok_pos, int n_tokens, int H, int G, int dk, int dv, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (H < 1 || G < 1 || dk < 1 || dv < 1 || rot < 0 || rot % 2 || rot > dk || (qw == nullptr) != (kw == nullptr) ||
        (rot && (cos_t == nullptr || sin_t == nullptr)))
        return OE_ERR_UNSUPPORTED;
    RowPrepArgs a;
    a.ld = ld; a.qw = qw; a.kw = kw; a.eps = eps; a.cos_t = cos_t; a.sin_t = sin_t; a.rot = rot; a.halves = halves;
    a.tables = tables; a.max_pages = max_pages; a.tok_seq = tok_seq; a.tok_pos = tok_pos;
    a.n_tokens = n_tokens; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
    if constexpr (sizeof(T) == 2) {
        const bool vec = dk % 8 == 0 && dv % 8 == 0 && rot % 8 == 0 && (rot == 0 || !halves) && ld % 8 == 0 &&
                         !(((uintptr_t)qkv | (uintptr_t)kcache | (uintptr_t)vcache | (uintptr_t)qw | (uintptr_t)kw | (uintptr_t)cos_t |
                            (uintptr_t)sin_t) & 15);
        const int pieces = (H * dk + G * dk + G * dv) / 8;
        if (vec && pieces <= 2 * ROW_THREADS)
            return oe_launch(qkv_row_norm_rot_write_vec_kernel<2>, dim3(n_tokens), dim3(ROW_THREADS), 0, st, qkv, kcache, vcache, a);
        if (vec && pieces <= 8 * ROW_THREADS)
            return oe_launch(qkv_row_norm_rot_write_vec_kernel<8>, dim3(n_tokens), dim3(ROW_THREADS), 0, st, qkv, kcache, vcache, a);
    }
    return oe_launch(qkv_row_norm_rot_write_kernel<T>, dim3(n_tokens), dim3(ROW_THREADS), 0, st, qkv, kcache, vcache, a);
}

template <typename T>
int launch_unrot(T* o, const float* cos_v, const float* sin_v, const int* tok_seq, const int* tok_pos, int n_tokens, int H,
                 int dv, cudaStream_t st) {
    if (n_tokens <= 0) return 0;
    if (dv < 2 || dv > MAX_D || dv % 2 || H < 1) return OE_ERR_UNSUPPORTED;
    const long long blocks = ((long long)n_tokens * H + WARPS - 1) / WARPS;
    if (blocks > 2147483647LL) return OE_ERR_UNSUPPORTED;
    return oe_launch(unrotate_heads_kernel<T>, dim3((unsigned)blocks), dim3(WARPS * 32), 0, st, o, cos_v, sin_v, tok_seq,
                     tok_pos, n_tokens, H, dv);
}

PrepArgs make_args(const float* proj, long long ld, const float* qb, const float* kb, const float* vb, const float* qw,
                   const float* kw, float eps, const float* cos_k, const float* sin_k, int rot, const float* cos_v,
                   const float* sin_v, int v_norm, const int* tables, int max_pages, const int* tok_seq, const int* tok_pos,
                   int n_tokens, int H, int G, int dk, int dv) {
    PrepArgs a;
    a.proj = proj; a.ld = ld; a.qb = qb; a.kb = kb; a.vb = vb; a.qw = qw; a.kw = kw; a.eps = eps;
    a.cos_k = cos_k; a.sin_k = sin_k; a.rot = (cos_k && sin_k) ? rot : 0; a.cos_v = (cos_v && sin_v) ? cos_v : nullptr;
    a.sin_v = sin_v; a.v_norm = v_norm; a.tables = tables; a.max_pages = max_pages; a.tok_seq = tok_seq; a.tok_pos = tok_pos;
    a.n_tokens = n_tokens; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
    return a;
}

}  // namespace

extern "C" {

int oe_qkv_norm_rot_write_f32(float* q_out, float* kcache, float* vcache, const float* proj, long long ld, const float* qb,
                              const float* kb, const float* vb, const float* qw, const float* kw, float eps,
                              const float* cos_k, const float* sin_k, int rot, const float* cos_v, const float* sin_v,
                              int v_norm, const int* tables, int max_pages, const int* tok_seq, const int* tok_pos,
                              int n_tokens, int H, int G, int dk, int dv, cudaStream_t st) {
    return launch_prep<float>(q_out, kcache, vcache, make_args(proj, ld, qb, kb, vb, qw, kw, eps, cos_k, sin_k, rot, cos_v, sin_v,
                                                               v_norm, tables, max_pages, tok_seq, tok_pos, n_tokens, H, G, dk, dv), st);
}
int oe_qkv_norm_rot_write_bf16(bf16* q_out, bf16* kcache, bf16* vcache, const float* proj, long long ld, const float* qb,
                               const float* kb, const float* vb, const float* qw, const float* kw, float eps,
                               const float* cos_k, const float* sin_k, int rot, const float* cos_v, const float* sin_v,
                               int v_norm, const int* tables, int max_pages, const int* tok_seq, const int* tok_pos,
                               int n_tokens, int H, int G, int dk, int dv, cudaStream_t st) {
    return launch_prep<bf16>(q_out, kcache, vcache, make_args(proj, ld, qb, kb, vb, qw, kw, eps, cos_k, sin_k, rot, cos_v, sin_v,
                                                              v_norm, tables, max_pages, tok_seq, tok_pos, n_tokens, H, G, dk, dv), st);
}
int oe_qkv_row_norm_rot_write_f32(float* qkv, long long ld, float* kcache, float* vcache, const float* qw, const float* kw,
                                  float eps, const float* cos_t, const float* sin_t, int rot, int halves, const int* tables,
                                  int max_pages, const int* tok_seq, const int* tok_pos, int n_tokens, int H, int G, int dk,
                                  int dv, cudaStream_t st) {
    return launch_row_prep<float>(qkv, ld, kcache, vcache, qw, kw, eps, cos_t, sin_t, rot, halves, tables, max_pages, tok_seq,
                                  tok_pos, n_tokens, H, G, dk, dv, st);
}
int oe_qkv_row_norm_rot_write_bf16(bf16* qkv, long long ld, bf16* kcache, bf16* vcache, const float* qw, const float* kw,
                                   float eps, const float* cos_t, const float* sin_t, int rot, int halves, const int* tables,
                                   int max_pages, const int* tok_seq, const int* tok_pos, int n_tokens, int H, int G, int dk,
                                   int dv, cudaStream_t st) {
    return launch_row_prep<bf16>(qkv, ld, kcache, vcache, qw, kw, eps, cos_t, sin_t, rot, halves, tables, max_pages, tok_seq,
                                 tok_pos, n_tokens, H, G, dk, dv, st);
}
int oe_unrotate_heads_f32(float* o, const float* cos_v, const float* sin_v, const int* tok_seq, const int* tok_pos,
                          int n_tokens, int H, int dv, cudaStream_t st) {
    return launch_unrot<float>(o, cos_v, sin_v, tok_seq, tok_pos, n_tokens, H, dv, st);
}
int oe_unrotate_heads_bf16(bf16* o, const float* cos_v, const float* sin_v, const int* tok_seq, const int* tok_pos,
                           int n_tokens, int H, int dv, cudaStream_t st) {
    return launch_unrot<bf16>(o, cos_v, sin_v, tok_seq, tok_pos, n_tokens, H, dv, st);
}

}  // extern "C"
