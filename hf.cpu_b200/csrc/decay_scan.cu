// Linear recurrences whose decay is one number per head and token:
//     S <- a_t S + c_t k_t u_t^T,   o_t = S^T q_t + D_h u_t          a_t = exp(la_t),  S [d, dv] per head
// (a fixed decay per head: retention; a decay and a step size c_t made from the token: Mamba-2's state-space form), what
// makes their operands from the products' float32 sums, and what stands behind them.
//
// The state is float32 and lives in a request's slot between steps, [H][dvp][dp] (a column of S, one value channel, is
// contiguous).  dp and dvp are d and dv rounded up to a multiple of 16; the operands q, k [T][heads][dp] and u
// [T][H][dvp] are stored the same way with zeros in the padding, so the padding of the state stays zero and every
// access below is a whole aligned vector.  q, k and u are in the run's type, la and c are float32.
//
// Two forms of the same recurrence:
//  * the walk (decay_walk_kernel): token by token, float32 multiply-adds, any number of tokens per request.  Columns of S
//    are independent, so (request, head, columns) spread over the grid.  Steps of single tokens, short portions, the
//    float32 run.
//  * chunks of CH tokens (three kernels, bf16 operands on mma.sync with float32 sums): with L_t the sum of la over the
//    chunk's tokens up to t,
//        o_t = exp(L_t) S_start^T q_t + sum_{s <= t} (q_t . k_s) exp(L_t - L_s) c_s u_s (+ D_h u_t)
//        S_end = exp(L_end) S_start + sum_s exp(L_end - L_s) c_s k_s u_s^T
//    decay_chunk_state_kernel: the sum in S_end, all chunks side by side; decay_chunk_pass_kernel: S_start of every chunk,
//    chunk after chunk per state element; decay_chunk_out_kernel: the outputs, all chunks side by side.  Operands that are
//    float32 by nature (the state, the weights (q . k) exp() c, and exp() c u) enter the products as a bfloat16 value
//    plus the bfloat16 of what is left, two products each, so what is lost is below 2^-16 of an operand; q, k and u are
//    bfloat16 in the walk too.  The decays multiply float32 values only.
#include "common.cuh"

static thread_local cudaError_t g_launch_err = cudaSuccess;      // what the last launch_pdl returned

namespace hfb {
int *error_word();

constexpr int DS_CH = 64;             // tokens of a chunk
constexpr int DS_DVT = 64;            // value channels of a block
constexpr int DS_MAX_CHUNK_D = 256;   // largest padded key head of the chunk form
constexpr int DS_MAX_D = 512;         // ... and of the walk
constexpr int DS_MAX_TAPS = 16;

static bool aligned16(const void *p) { return ((uintptr_t)p & 15) == 0; }

template <typename T> struct Pack4;
template <> struct Pack4<float> {
    static __device__ __forceinline__ float4 load(const float *p) { return *(const float4 *)p; }
};
template <> struct Pack4<__nv_bfloat16> {
    static __device__ __forceinline__ float4 load(const __nv_bfloat16 *p)
    {
        const uint2 u = *(const uint2 *)p;
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162 *)&u.x), b = __bfloat1622float2(*(const __nv_bfloat162 *)&u.y);
        return make_float4(a.x, a.y, b.x, b.y);
    }
};

// exp and z * sigmoid(z): from the special-function unit where the result is rounded to bfloat16 behind it, else CUDA's
// full-accuracy functions.
template <typename TO> __device__ __forceinline__ float silu_for(float z)
{
    if constexpr (sizeof(TO) == 4) return z / (1.0f + expf(-z));
    else return __fdividef(z, 1.0f + __expf(-z));
}

template <typename TO> __device__ __forceinline__ float sigmoid_for(float z)
{
    if constexpr (sizeof(TO) == 4) return 1.0f / (1.0f + expf(-z));
    else return __fdividef(1.0f, 1.0f + __expf(-z));
}

__device__ __forceinline__ void store2(float *p, float a, float b) { *(float2 *)p = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16 *p, float a, float b) { *(__nv_bfloat162 *)p = __floats2bfloat162_rn(a, b); }

// ---- operands of retention --------------------------------------------------------------------------------------
template <typename TO, bool SILU> __device__ __forceinline__ float head_in(const float *p, int splits, size_t plane)
{
    const float v = plane_sum(p, splits, plane);
    return SILU ? silu_for<TO>(v) : v;
}
template <typename TO, bool SILU> __device__ __forceinline__ float2 head_in2(const float *p, int splits, size_t plane)
{
    const float2 v = plane_sum2(p, splits, plane);
    return SILU ? make_float2(silu_for<TO>(v.x), silu_for<TO>(v.y)) : v;
}

// One warp per (token, head) of the rows [H query heads of d | H key heads of d | H value heads of dv | ...] (row_stride
// floats, `splits` planes): rotation of the first n_rot dimensions of queries and keys (pairs i, i + n_rot/2), keys times
// k_scale, everything to its padded place.  SILU: queries, keys and values pass silu first.
template <typename TO, bool SILU>
__global__ void __launch_bounds__(128)
rotate_heads_kernel(const float *src, int splits, int row_stride, const float *cos_sin, int n_rot, int n_positions,
                    const int32_t *positions, float k_scale, TO *q, TO *k, TO *u, int T, int H, int d, int dv, int dp, int dvp, int pairs,
                    int *err)
{
    pdl_entry();
    pdl_sync_small();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, h = blockIdx.y * 4 + warp;
    if (h >= H) return;
    const size_t plane = (size_t)T * row_stride;
    const float *row = src + (size_t)t * row_stride;
    const int half = n_rot / 2;
    int pos = 0;
    if (half > 0) {
        pos = positions[t];
        if (pos < 0 || pos >= n_positions) { if (lane == 0) atomicOr(err, HFB_ERR_POSITION); pos = 0; }
    }
    const float *cs = cos_sin + (size_t)pos * n_rot;
    const float *qr = row + h * d, *kr = qr + H * d, *vr = row + 2 * H * d + h * dv;
    TO *qd = q + ((size_t)t * H + h) * dp, *kd = k + ((size_t)t * H + h) * dp, *ud = u + ((size_t)t * H + h) * dvp;
    if (pairs) {
        // two neighbouring dimensions a lane: everything of the head is even and aligned to two
        for (int i = 2 * lane; i < half; i += 64) {
            const float4 c = *(const float4 *)(cs + 2 * i);
            const float2 qa = head_in2<TO, SILU>(qr + i, splits, plane), qb = head_in2<TO, SILU>(qr + i + half, splits, plane);
            const float2 ka = head_in2<TO, SILU>(kr + i, splits, plane), kb = head_in2<TO, SILU>(kr + i + half, splits, plane);
            float lo0, hi0, lo1, hi1;
            rope_pair(qa.x, qb.x, c.x, c.y, lo0, hi0);
            rope_pair(qa.y, qb.y, c.z, c.w, lo1, hi1);
            store2(qd + i, lo0, lo1);
            store2(qd + i + half, hi0, hi1);
            rope_pair(ka.x, kb.x, c.x, c.y, lo0, hi0);
            rope_pair(ka.y, kb.y, c.z, c.w, lo1, hi1);
            store2(kd + i, lo0 * k_scale, lo1 * k_scale);
            store2(kd + i + half, hi0 * k_scale, hi1 * k_scale);
        }
        for (int i = n_rot + 2 * lane; i < dp; i += 64) {
            const float2 a = i < d ? head_in2<TO, SILU>(qr + i, splits, plane) : make_float2(0.f, 0.f);
            const float2 b = i < d ? head_in2<TO, SILU>(kr + i, splits, plane) : make_float2(0.f, 0.f);
            store2(qd + i, a.x, a.y);
            store2(kd + i, b.x * k_scale, b.y * k_scale);
        }
        for (int i = 2 * lane; i < dvp; i += 64) {
            const float2 a = i < dv ? head_in2<TO, SILU>(vr + i, splits, plane) : make_float2(0.f, 0.f);
            store2(ud + i, a.x, a.y);
        }
        return;
    }
#pragma unroll 1
    for (int part = 0; part < 2; part++) {
        const float *p = part ? kr : qr;
        TO *dst = part ? kd : qd;
        const float f = part ? k_scale : 1.0f;
        for (int i = lane; i < half; i += 32) {
            float lo, hi;
            rope_pair(head_in<TO, SILU>(p + i, splits, plane), head_in<TO, SILU>(p + i + half, splits, plane), cs[2 * i], cs[2 * i + 1], lo, hi);
            dst[i] = from_f32<TO>(lo * f);
            dst[i + half] = from_f32<TO>(hi * f);
        }
        for (int i = n_rot + lane; i < dp; i += 32) dst[i] = from_f32<TO>(i < d ? head_in<TO, SILU>(p + i, splits, plane) * f : 0.f);
    }
    for (int i = lane; i < dvp; i += 32) ud[i] = from_f32<TO>(i < dv ? head_in<TO, SILU>(vr + i, splits, plane) : 0.f);
}

// ---- operands of the state-space form ---------------------------------------------------------------------------
// Rows (row_stride floats, `splits` planes): [z: H dv | x: H dv | B: G d | C: G d | dt: H | ...].  x, B and C pass a causal
// convolution per channel (w [CC, taps], last column the current token's; bias [CC]) and silu: x to u, B to k, C to q.  A
// thread takes V neighbouring channels.
// step[t, h] = softplus(dt + dt_bias), la[t, h] = -rate[h] * step.  Blocks: `tt` tokens x 128 V channels, a thread
// slides a window of taps along the tokens; the last blocks in x make step and la.  Inputs before a request's first
// token of this step come from its slot, carried [taps - 1][CC] oldest first (zeros for a new request).  `single`: every
// request brings one token, and the thread brings its channel of the slot up to date itself (else conv_carry does).
template <int TAPS, int V, typename TO>
__global__ void __launch_bounds__(128)
state_space_operands_kernel(const float *src, int splits, int row_stride, const void *w, int w_dt, const void *bias, int bias_dt, int taps,
                            const void *dt_bias, int dtb_dt, const float *rate, float *carried, size_t slot_stride,
                            const int32_t *token_seq, const int32_t *cu_tokens, const int32_t *seq_slots, int n_slots, int single,
                            TO *q, TO *k, TO *u, float *step, float *la, int T, int H, int G, int d, int dv, int dp, int dvp, int tt,
                            int *err)
{
    pdl_entry();
    pdl_sync_small();
    const int inner = H * dv, CC = inner + 2 * G * d;
    const int conv_blocks = (CC + 128 * V - 1) / (128 * V);
    const size_t plane = (size_t)T * row_stride;
    const int tb = blockIdx.y * tt, te = min(T, tb + tt);
    if ((int)blockIdx.x >= conv_blocks) {
        const int h = ((int)blockIdx.x - conv_blocks) * 128 + threadIdx.x;
        if (h >= H) return;
        const float b = load_any(dt_bias, dtb_dt, h), r = rate[h];
#pragma unroll 4
        for (int t = tb; t < te; t++) {
            const float *p = src + (size_t)t * row_stride + 2 * inner + 2 * G * d + h;
            const float z = plane_sum(p, splits, plane) + b;
            const float v = z > 20.f ? z : log1pf(expf(z));
            step[(size_t)t * H + h] = v;
            la[(size_t)t * H + h] = -r * v;
        }
        return;
    }
    constexpr int W = TAPS ? TAPS : DS_MAX_TAPS;
    const int ch = (blockIdx.x * 128 + threadIdx.x) * V;
    if (ch >= CC) return;
    const int n_taps = TAPS ? TAPS : taps, K = n_taps - 1;
    // the window holds the last n_taps inputs in its last n_taps places; weights likewise
    float wv[V][W], win[V][W], b[V];
#pragma unroll
    for (int c = 0; c < V; c++) {
#pragma unroll
        for (int j = 0; j < W; j++) {
            const int i = j - (W - n_taps);
            wv[c][j] = i >= 0 ? load_any(w, w_dt, (size_t)(ch + c) * n_taps + i) : 0.f;
            win[c][j] = 0.f;
        }
        b[c] = load_any(bias, bias_dt, ch + c);
    }
    // where this thread's channels go (V = 2: heads of even size, so both belong to one)
    TO *dst;
    size_t dst_stride;
    int pad = 0;                                     // zeros behind a head's last channel
    if (ch < inner) {
        const int h = ch / dv, i = ch % dv;
        dst = u + (size_t)h * dvp + i;
        dst_stride = (size_t)H * dvp;
        if (i + V == dv) pad = dvp - dv;
    } else {
        const int c = ch - inner, which = c / (G * d), g = c % (G * d) / d, i = c % d;
        dst = (which ? q : k) + (size_t)g * dp + i;
        dst_stride = (size_t)G * dp;
        if (i + V == d) pad = dp - d;
    }
    const float *x = src + inner + ch;
    auto input = [&](int t, float *v) {
        if constexpr (V == 2) {
            const float2 a = plane_sum2(x + (size_t)t * row_stride, splits, plane);
            v[0] = a.x;
            v[1] = a.y;
        } else {
            v[0] = plane_sum(x + (size_t)t * row_stride, splits, plane);
        }
    };
    // a request's tokens of the tile at a time: the window before the first of them, then eight tokens in flight
    for (int t = tb; t < te;) {
        const int seq = token_seq[t], t0 = cu_tokens[seq], t1 = min(te, cu_tokens[seq + 1]), slot = seq_slots[seq];
        if (slot < 0 || slot >= n_slots) { if (threadIdx.x == 0) atomicOr(err, HFB_ERR_SLOT); return; }
        float *old = carried + (size_t)slot * slot_stride + ch;
#pragma unroll
        for (int i = 0; i < W; i++) {
            // place i holds the input W - i tokens back; the shift below brings it to place i - 1
            const int back = W - i, tp = t - back;
            if (back <= K) {
                float v[V];
                if (tp >= t0) {
                    input(tp, v);
                } else {
#pragma unroll
                    for (int c = 0; c < V; c++) v[c] = old[(size_t)(tp - t0 + K) * CC + c];
                }
#pragma unroll
                for (int c = 0; c < V; c++) win[c][i] = v[c];
            }
        }
        for (; t < t1; t += 8) {
            float xin[8][V];
            if (splits == 1) {                           // (all eight reads in flight)
#pragma unroll
                for (int j = 0; j < 8; j++) {
                    if (t + j < t1) {
                        const float *p = x + (size_t)(t + j) * row_stride;
                        if constexpr (V == 2) { const float2 a = *(const float2 *)p; xin[j][0] = a.x; xin[j][1] = a.y; }
                        else xin[j][0] = p[0];
                    }
                }
            } else {
#pragma unroll 1
                for (int j = 0; j < 8 && t + j < t1; j++) {
                    float v[V];
                    input(t + j, v);
#pragma unroll
                    for (int jj = 0; jj < 8; jj++)
                        if (jj == j)
#pragma unroll
                            for (int c = 0; c < V; c++) xin[jj][c] = v[c];
                }
            }
#pragma unroll
            for (int j = 0; j < 8; j++) {
                if (t + j < t1) {
                    float y[V];
#pragma unroll
                    for (int c = 0; c < V; c++) {
#pragma unroll
                        for (int i = 0; i + 1 < W; i++) win[c][i] = win[c][i + 1];
                        win[c][W - 1] = xin[j][c];
                        float acc = b[c];
#pragma unroll
                        for (int i = 0; i < W; i++) acc = fmaf(wv[c][i], win[c][i], acc);
                        y[c] = silu_for<TO>(acc);
                    }
                    TO *o = dst + (size_t)(t + j) * dst_stride;
                    if constexpr (V == 2) store2(o, y[0], y[1]);
                    else o[0] = from_f32<TO>(y[0]);
                    for (int i = V; i < V + pad; i++) o[i] = from_f32<TO>(0.f);
                }
            }
        }
        t = t1;
        if (single) {
#pragma unroll
            for (int i = 0; i < W; i++) {
                const int back = W - 1 - i;                  // 0: the token itself
                if (back < K) {
#pragma unroll
                    for (int c = 0; c < V; c++) old[(size_t)(K - 1 - back) * CC + c] = win[c][i];
                }
            }
        }
    }
}

// ---- the walk ---------------------------------------------------------------------------------------------------
// L lanes share a column of S, each holding J vectors of four of its entries; a group of L lanes takes DS_COLS columns.
// Where the decay is the same for every token, `fixed` [H] holds it as it is: an exponential made from its rounded logarithm
// may be off by an ulp, the same way at every token, and a thousand tokens add that up.
constexpr int DS_COLS = 4;

template <typename TI, int L, int J>
__global__ void __launch_bounds__(128)
decay_walk_kernel(const TI *q, const TI *k, const TI *u, const float *la, int la_stride, const float *fixed, const float *step, const float *skip,
                  float *state, size_t slot_stride, const int32_t *cu_tokens, const int32_t *seq_slots, int n_slots, float *o, int H,
                  int Hq, int dp, int dv, int dvp, int *err)
{
    pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, hq = h / (H / Hq);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane % L;
    const int c0 = ((blockIdx.z * 4 + warp) * (32 / L) + lane / L) * DS_COLS;
    const int slot = seq_slots[seq];
    if (slot < 0 || slot >= n_slots) { if (threadIdx.x == 0) atomicOr(err, HFB_ERR_SLOT); return; }
    const int t0 = cu_tokens[seq], t1 = cu_tokens[seq + 1];
    float *sp = state + (size_t)slot * slot_stride + (size_t)h * dvp * dp;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 S[DS_COLS][J];
#pragma unroll
    for (int c = 0; c < DS_COLS; c++)
#pragma unroll
        for (int j = 0; j < J; j++) {
            const int i = (part + j * L) * 4;
            S[c][j] = (c0 + c < dvp && i < dp) ? *(const float4 *)(sp + (size_t)(c0 + c) * dp + i) : zero;
        }
    const float dsk = skip ? skip[h] : 0.f, a_fixed = fixed ? fixed[h] : 0.f;
    float4 qn[J], kn[J];
    float un[DS_COLS], an, cn;
    auto fetch = [&](int t) {
#pragma unroll
        for (int j = 0; j < J; j++) {
            const int i = (part + j * L) * 4;
            const size_t at = ((size_t)t * Hq + hq) * dp + i;
            qn[j] = i < dp ? Pack4<TI>::load(q + at) : zero;
            kn[j] = i < dp ? Pack4<TI>::load(k + at) : zero;
        }
#pragma unroll
        for (int c = 0; c < DS_COLS; c++) un[c] = c0 + c < dvp ? to_f32(u[((size_t)t * H + h) * dvp + c0 + c]) : 0.f;
        an = la[(size_t)t * la_stride + h];
        cn = step ? step[(size_t)t * H + h] : 1.0f;
    };
    if (t0 < t1) fetch(t0);
    for (int t = t0; t < t1; t++) {
        float4 qa[J], ka[J];
        float ua[DS_COLS];
#pragma unroll
        for (int j = 0; j < J; j++) { qa[j] = qn[j]; ka[j] = kn[j]; }
#pragma unroll
        for (int c = 0; c < DS_COLS; c++) ua[c] = un[c];
        const float a = fixed ? a_fixed : expf(an), cs = cn;
        if (t + 1 < t1) fetch(t + 1);
        float dot[DS_COLS];
#pragma unroll
        for (int c = 0; c < DS_COLS; c++) {
            const float uc = ua[c] * cs;
            float x = 0.f, y = 0.f;
#pragma unroll
            for (int j = 0; j < J; j++) {
                float4 &s = S[c][j];
                s.x = fmaf(a, s.x, ka[j].x * uc); s.y = fmaf(a, s.y, ka[j].y * uc);
                s.z = fmaf(a, s.z, ka[j].z * uc); s.w = fmaf(a, s.w, ka[j].w * uc);
                x = fmaf(s.x, qa[j].x, x); y = fmaf(s.y, qa[j].y, y);
                x = fmaf(s.z, qa[j].z, x); y = fmaf(s.w, qa[j].w, y);
            }
            dot[c] = x + y;
        }
#pragma unroll
        for (int m = L / 2; m > 0; m >>= 1)
#pragma unroll
            for (int c = 0; c < DS_COLS; c++) dot[c] += __shfl_xor_sync(0xffffffffu, dot[c], m);
        if (part == 0) {
#pragma unroll
            for (int c = 0; c < DS_COLS; c++)
                if (c0 + c < dv) o[((size_t)t * H + h) * dv + c0 + c] = fmaf(dsk, ua[c], dot[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < DS_COLS; c++)
#pragma unroll
        for (int j = 0; j < J; j++) {
            const int i = (part + j * L) * 4;
            if (c0 + c < dvp && i < dp) *(float4 *)(sp + (size_t)(c0 + c) * dp + i) = S[c][j];
        }
}

// ---- chunks -----------------------------------------------------------------------------------------------------
__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t *r, uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t *r, uint32_t addr)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float *c, const uint32_t *a, uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(void *dst, const void *src)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_wait_all() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory"); }

// two float32 as a pair of bfloat16 and the pair of what is left
__device__ __forceinline__ void split2(float a, float b, uint32_t &hi, uint32_t &lo)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 back = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - back.x, b - back.y);
    hi = *(const uint32_t *)&h;
    lo = *(const uint32_t *)&l;
}

// `rows` x COLS values of shared memory (rows COLS + 8 values apart) from n rows of `cols` values, row_stride apart, zeros
// beyond them.
template <int COLS>
__device__ __forceinline__ void stage_rows(__nv_bfloat16 *dst, const __nv_bfloat16 *src, size_t row_stride, int n, int rows, int cols)
{
    constexpr int PER = COLS / 8;
#pragma unroll 4
    for (int idx = threadIdx.x; idx < rows * PER; idx += 128) {
        const int r = idx / PER, c = idx % PER * 8;
        __nv_bfloat16 *to = dst + r * (COLS + 8) + c;
        if (r < n && c < cols) cp16(to, src + (size_t)r * row_stride + c);
        else *(uint4 *)to = make_uint4(0, 0, 0, 0);
    }
}

// Decays of a chunk, by the first warp: two tokens' la and step size a lane (1 where there are no step sizes, 0 beyond n),
// then L[i] = la summed over the tokens 0 .. i (tokens beyond n repeat the last sum) and c[i] = step sizes.
struct ChunkDecays {
    float a, b, ca, cb;
    __device__ __forceinline__ void fetch(const float *la, int la_stride, const float *step, int H, int h, int t0, int n)
    {
        const int i = threadIdx.x * 2;
        a = i < n ? la[(size_t)(t0 + i) * la_stride + h] : 0.f;
        b = i + 1 < n ? la[(size_t)(t0 + i + 1) * la_stride + h] : 0.f;
        ca = i < n ? (step ? step[(size_t)(t0 + i) * H + h] : 1.0f) : 0.f;
        cb = i + 1 < n ? (step ? step[(size_t)(t0 + i + 1) * H + h] : 1.0f) : 0.f;
    }
    __device__ __forceinline__ void finish(float *Ls, float *cs) const
    {
        const int i = threadIdx.x * 2;
        const float both = a + b;
        float run = both;
#pragma unroll
        for (int m = 1; m < 32; m <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, run, m);
            if ((int)threadIdx.x >= m) run += v;
        }
        const float before = __shfl_up_sync(0xffffffffu, run, 1);
        const float base = threadIdx.x ? before : 0.f;
        Ls[i] = base + a;
        Ls[i + 1] = base + both;
        cs[i] = ca;
        cs[i + 1] = cb;
    }
};

// What a chunk adds to the state: dS[chunk][h][dvp][dp] = sum_s exp(L_end - L_s) c_s u_s k_s^T, and the chunk's L_end.
// Block: chunk x head x (64 value channels, 128 key channels); a warp takes 16 value channels.
template <int KT>                        // key channels of a block
__global__ void __launch_bounds__(128)
decay_chunk_state_kernel(const __nv_bfloat16 *k, const __nv_bfloat16 *u, const float *la, int la_stride, const float *step,
                         const int32_t *chunk_t0, const int32_t *chunk_n, float *dS, float *l_end, int H, int Hq, int dp, int dvp)
{
    pdl_wait();
    __shared__ __align__(16) __nv_bfloat16 us[DS_CH * (DS_DVT + 8)], ks[DS_CH * (KT + 8)];
    __shared__ float Ls[DS_CH], cs[DS_CH];
    const int chunk = blockIdx.x, h = blockIdx.y, hq = h / (H / Hq);
    const int d_tiles = (dp + KT - 1) / KT;
    const int v0 = (int)blockIdx.z / d_tiles * DS_DVT, d0 = (int)blockIdx.z % d_tiles * KT;
    const int vt = min(DS_DVT, dvp - v0), kt = min(KT, dp - d0);
    const int t0 = chunk_t0[chunk], n = chunk_n[chunk];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    ChunkDecays dec;
    if (warp == 0) dec.fetch(la, la_stride, step, H, h, t0, n);
    stage_rows<DS_DVT>(us, u + ((size_t)t0 * H + h) * dvp + v0, (size_t)H * dvp, n, DS_CH, vt);
    stage_rows<KT>(ks, k + ((size_t)t0 * Hq + hq) * dp + d0, (size_t)Hq * dp, n, DS_CH, kt);
    if (warp == 0) dec.finish(Ls, cs);
    cp_wait_all();
    __syncthreads();
    const float lend = Ls[n - 1];
    if (blockIdx.z == 0 && threadIdx.x == 0) l_end[(size_t)chunk * H + h] = lend;
    if (warp * 16 >= vt) return;
    constexpr int NT = KT / 8, KP = KT + 8;
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    const uint32_t ua = smem_addr(us) + (((lane & 7) + (lane >> 4) * 8) * (DS_DVT + 8) + warp * 16 + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t ka = smem_addr(ks) + (((lane & 7) + ((lane >> 3) & 1) * 8) * KP + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int kk = 0; kk < DS_CH / 16; kk++) {
        uint32_t raw[4], hi[4], lo[4];
        ldsm4_t(raw, ua + kk * 16 * (DS_DVT + 8) * 2);
        const int ta = kk * 16 + (lane & 3) * 2;
        float wgt[4];                                                        // tokens ta, ta + 1, ta + 8, ta + 9
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float2 L = *(const float2 *)&Ls[ta + 8 * i], c = *(const float2 *)&cs[ta + 8 * i];
            wgt[2 * i] = __expf(lend - L.x) * c.x;
            wgt[2 * i + 1] = __expf(lend - L.y) * c.y;
        }
#pragma unroll
        for (int i = 0; i < 4; i++) {                                        // registers: (rows, tokens ta..), (rows + 8, ..), (rows, ta + 8..), ..
            const float2 f = __bfloat1622float2(*(const __nv_bfloat162 *)&raw[i]);
            split2(f.x * wgt[(i >> 1) * 2], f.y * wgt[(i >> 1) * 2 + 1], hi[i], lo[i]);
        }
#pragma unroll
        for (int nt = 0; nt < NT / 2; nt++) {
            uint32_t b[4];
            ldsm4_t(b, ka + (kk * 16 * KP + nt * 16) * 2);
            mma16816(acc[2 * nt], hi, b[0], b[1]);
            mma16816(acc[2 * nt + 1], hi, b[2], b[3]);
            mma16816(acc[2 * nt], lo, b[0], b[1]);
            mma16816(acc[2 * nt + 1], lo, b[2], b[3]);
        }
    }
    float *out = dS + (((size_t)chunk * H + h) * dvp + v0 + warp * 16 + (lane >> 2)) * dp + d0 + (lane & 3) * 2;
#pragma unroll
    for (int nt = 0; nt < NT; nt++) {
        if (nt * 8 < kt) {
            *(float2 *)(out + nt * 8) = make_float2(acc[nt][0], acc[nt][1]);
            *(float2 *)(out + (size_t)8 * dp + nt * 8) = make_float2(acc[nt][2], acc[nt][3]);
        }
    }
}

// The state at every chunk's start, chunk after chunk; a thread per four state elements of a request.  start
// [chunk][h][2][dvp][dp]: the bfloat16 of the state and the bfloat16 of what is left.
__global__ void __launch_bounds__(256)
decay_chunk_pass_kernel(const float *__restrict__ dS, const float *__restrict__ l_end, float *state, size_t slot_stride,
                        const int32_t *chunk_first, const int32_t *seq_slots, int n_slots, __nv_bfloat16 *__restrict__ start, int H, int dp,
                        int dvp, int *err)
{
    pdl_wait();
    const int seq = blockIdx.y;
    const size_t per_head = (size_t)dvp * dp, total = (size_t)H * per_head;
    const size_t e = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
    if (e >= total) return;
    const int slot = seq_slots[seq];
    if (slot < 0 || slot >= n_slots) { if (threadIdx.x == 0) atomicOr(err, HFB_ERR_SLOT); return; }
    const int h = (int)(e / per_head);
    const size_t in_head = e - (size_t)h * per_head;
    float4 *st = (float4 *)(state + (size_t)slot * slot_stride + e);
    float4 S = *st;
    const int c1 = chunk_first[seq + 1];
    for (int c = chunk_first[seq]; c < c1; c += 8) {
        float4 add[8];
        float dec[8];
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (c + j < c1) {
                add[j] = *(const float4 *)(dS + (size_t)(c + j) * total + e);
                dec[j] = l_end[(size_t)(c + j) * H + h];
            }
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (c + j < c1) {
                uint2 hi, lo;
                split2(S.x, S.y, hi.x, lo.x);
                split2(S.z, S.w, hi.y, lo.y);
                __nv_bfloat16 *p = start + ((size_t)(c + j) * H + h) * 2 * per_head + in_head;
                *(uint2 *)p = hi;
                *(uint2 *)(p + per_head) = lo;
                const float a = expf(dec[j]);
                S.x = fmaf(a, S.x, add[j].x); S.y = fmaf(a, S.y, add[j].y);
                S.z = fmaf(a, S.z, add[j].z); S.w = fmaf(a, S.w, add[j].w);
            }
    }
    *st = S;
}

// The outputs of a chunk.  A block takes one chunk and one query/key head, whose queries it holds in registers (NK tiles of
// 16 key channels) and whose scores q . k it computes once; then it walks its share of the (head, 64 value channels) items
// that read this query/key head, the next item's state and values on their way while it works on one.  A warp takes 16
// tokens.
template <int NK>
__global__ void __launch_bounds__(128)
decay_chunk_out_kernel(const __nv_bfloat16 *q, const __nv_bfloat16 *k, const __nv_bfloat16 *u, const float *la, int la_stride,
                       const float *step, const float *skip, const __nv_bfloat16 *start, const int32_t *chunk_t0, const int32_t *chunk_n,
                       float *o, int H, int Hq, int dp, int dv, int dvp, int v_tiles, int per_block)
{
    pdl_wait();
    extern __shared__ __align__(16) uint8_t ds_smem[];
    constexpr int D = NK * 16, P = D + 8, STAGE = 2 * DS_DVT * P + DS_CH * (DS_DVT + 8);
    __nv_bfloat16 *ks = (__nv_bfloat16 *)ds_smem;                            // [CH][P]
    __nv_bfloat16 *stages = ks + DS_CH * P;                                  // per stage: sh, sl [DVT][P], us [CH][DVT + 8]
    __shared__ float Ls[2][DS_CH], cs[2][DS_CH];
    const int chunk = blockIdx.x, rep = H / Hq, items = rep * v_tiles, shares = (items + per_block - 1) / per_block;
    const int hq = blockIdx.y / shares, i0 = (blockIdx.y % shares) * per_block, i1 = min(items, i0 + per_block);
    const int t0 = chunk_t0[chunk], n = chunk_n[chunk];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    ChunkDecays dec;                                                         // (the first warp's, fetched an item ahead)

    auto issue = [&](int item, int stage) {
        const int h = hq * rep + item / v_tiles, v0 = item % v_tiles * DS_DVT, vt = min(DS_DVT, dvp - v0);
        __nv_bfloat16 *sh = stages + stage * STAGE, *sl = sh + DS_DVT * P, *us = sl + DS_DVT * P;
        const __nv_bfloat16 *sp = start + ((size_t)chunk * H + h) * 2 * dvp * dp + (size_t)v0 * dp;
        stage_rows<D>(sh, sp, dp, vt, DS_DVT, dp);
        stage_rows<D>(sl, sp + (size_t)dvp * dp, dp, vt, DS_DVT, dp);
        stage_rows<DS_DVT>(us, u + ((size_t)t0 * H + h) * dvp + v0, (size_t)H * dvp, n, DS_CH, vt);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (warp == 0) {
            dec.finish(Ls[stage], cs[stage]);
            if (item + 1 < i1) dec.fetch(la, la_stride, step, H, hq * rep + (item + 1) / v_tiles, t0, n);
        }
    };
    if (warp == 0) dec.fetch(la, la_stride, step, H, hq * rep + i0 / v_tiles, t0, n);
    stage_rows<D>(ks, k + ((size_t)t0 * Hq + hq) * dp, (size_t)Hq * dp, n, DS_CH, dp);
    const int r0 = warp * 16 + (lane >> 2), r1 = r0 + 8;                    // this thread's two tokens
    uint32_t qf[NK][4];
    {
        const __nv_bfloat16 *q0 = q + ((size_t)(t0 + min(r0, n - 1)) * Hq + hq) * dp + (lane & 3) * 2;
        const __nv_bfloat16 *q1 = q + ((size_t)(t0 + min(r1, n - 1)) * Hq + hq) * dp + (lane & 3) * 2;
#pragma unroll
        for (int kk = 0; kk < NK; kk++) {
            const bool in = kk * 16 < dp;
            qf[kk][0] = in ? *(const uint32_t *)(q0 + kk * 16) : 0u;
            qf[kk][1] = in ? *(const uint32_t *)(q1 + kk * 16) : 0u;
            qf[kk][2] = in ? *(const uint32_t *)(q0 + kk * 16 + 8) : 0u;
            qf[kk][3] = in ? *(const uint32_t *)(q1 + kk * 16 + 8) : 0u;
        }
    }
    issue(i0, 0);
    const uint32_t nk = (((lane & 7) + (lane >> 4) * 8) * P + ((lane >> 3) & 1) * 8) * 2;      // [n][k] operands
    const uint32_t ka = smem_addr(ks) + nk;
    const bool works = warp * 16 < n;
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) s[i][j] = 0.f;
    for (int item = i0; item < i1; item++) {
        const int stage = (item - i0) & 1;
        if (item + 1 < i1) {
            issue(item + 1, stage ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if (works) {
            if (item == i0) {
#pragma unroll
                for (int kt = 0; kt < 4; kt++) {
                    if (kt <= warp) {
#pragma unroll
                        for (int kk = 0; kk < NK; kk++) {
                            uint32_t b[4];
                            ldsm4(b, ka + kt * 16 * P * 2 + kk * 32);
                            mma16816(s[2 * kt], qf[kk], b[0], b[1]);
                            mma16816(s[2 * kt + 1], qf[kk], b[2], b[3]);
                        }
                    }
                }
            }
            const int h = hq * rep + item / v_tiles, v0 = item % v_tiles * DS_DVT, vt = min(DS_DVT, dvp - v0);
            const __nv_bfloat16 *sh = stages + stage * STAGE, *sl = sh + DS_DVT * P, *us = sl + DS_DVT * P;
            const uint32_t ha = smem_addr(sh) + nk, lo_a = smem_addr(sl) + nk;
            const uint32_t ua = smem_addr(us) + (((lane & 7) + ((lane >> 3) & 1) * 8) * (DS_DVT + 8) + (lane >> 4) * 8) * 2;
            const float dsk = skip ? skip[h] : 0.f;
            float acc[8][4];
#pragma unroll
            for (int i = 0; i < 8; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
            // what the state at the chunk's start gives
#pragma unroll
            for (int kk = 0; kk < NK; kk++) {
                uint32_t b[4][4];
#pragma unroll
                for (int nt = 0; nt < 4; nt++) ldsm4(b[nt], ha + nt * 16 * P * 2 + kk * 32);
#pragma unroll
                for (int nt = 0; nt < 4; nt++) {
                    mma16816(acc[2 * nt], qf[kk], b[nt][0], b[nt][1]);
                    mma16816(acc[2 * nt + 1], qf[kk], b[nt][2], b[nt][3]);
                }
#pragma unroll
                for (int nt = 0; nt < 4; nt++) ldsm4(b[nt], lo_a + nt * 16 * P * 2 + kk * 32);
#pragma unroll
                for (int nt = 0; nt < 4; nt++) {
                    mma16816(acc[2 * nt], qf[kk], b[nt][0], b[nt][1]);
                    mma16816(acc[2 * nt + 1], qf[kk], b[nt][2], b[nt][3]);
                }
            }
            const float L0 = Ls[stage][r0], L1 = Ls[stage][r1];
            {
                const float e0 = __expf(L0), e1 = __expf(L1);
#pragma unroll
                for (int i = 0; i < 8; i++) { acc[i][0] *= e0; acc[i][1] *= e0; acc[i][2] *= e1; acc[i][3] *= e1; }
            }
            // what the chunk's own tokens give
#pragma unroll
            for (int kt = 0; kt < 4; kt++) {
                if (kt <= warp) {
                    uint32_t hi[4], lo[4];
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const int key = kt * 16 + half * 8 + (lane & 3) * 2;
                        const float2 Lk = *(const float2 *)&Ls[stage][key], ck = *(const float2 *)&cs[stage][key];
                        float w[4];
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            const int ky = key + (i & 1), r = i < 2 ? r0 : r1;
                            const float L = (i < 2 ? L0 : L1) - (i & 1 ? Lk.y : Lk.x);
                            float v = ky <= r ? s[2 * kt + half][i] * __expf(fminf(L, 0.f)) * (i & 1 ? ck.y : ck.x) : 0.f;
                            if (ky == r) v += dsk;
                            w[i] = v;
                        }
                        split2(w[0], w[1], hi[2 * half], lo[2 * half]);
                        split2(w[2], w[3], hi[2 * half + 1], lo[2 * half + 1]);
                    }
#pragma unroll
                    for (int nt = 0; nt < 4; nt++) {
                        uint32_t b[4];
                        ldsm4_t(b, ua + (kt * 16 * (DS_DVT + 8) + nt * 16) * 2);
                        mma16816(acc[2 * nt], hi, b[0], b[1]);
                        mma16816(acc[2 * nt + 1], hi, b[2], b[3]);
                        mma16816(acc[2 * nt], lo, b[0], b[1]);
                        mma16816(acc[2 * nt + 1], lo, b[2], b[3]);
                    }
                }
            }
            const bool even = (dv & 1) == 0;
#pragma unroll
            for (int nt = 0; nt < 8; nt++) {
                const int c = v0 + nt * 8 + (lane & 3) * 2;
                if (nt * 8 < vt && c < dv) {
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const int r = half ? r1 : r0;
                        if (r < n) {
                            float *p = o + ((size_t)(t0 + r) * H + h) * dv + c;
                            if (even) *(float2 *)p = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
                            else { p[0] = acc[nt][2 * half]; if (c + 1 < dv) p[1] = acc[nt][2 * half + 1]; }
                        }
                    }
                }
            }
        }
        __syncthreads();                                                     // the stage is free for the item after the next
    }
}

// ---- behind the recurrence --------------------------------------------------------------------------------------
// A row of o [T, C] in parts of n values, each divided by its own root mean square; the gate, silu(g) or (SIGMOID) sigmoid(g),
// multiplies before the norm (gate_first) or after it; times a weight [C] where there is one.  g is the sum of `splits` planes [T, g_stride] read
// from column g_col0 on.  TH threads per part, at most 16 values a thread, V at a time.
template <typename TO, int TH, int V, int N, bool SIGMOID>
__global__ void __launch_bounds__(TH < 128 ? 128 : TH)
part_norm_gate_kernel(const float *o, const float *g, int splits, int g_stride, int g_col0, const float *w, float eps, int gate_first,
                      TO *out, size_t out_stride, int T, int C, int n, int parts)
{
    pdl_entry();
    pdl_sync_small();
    constexpr int PER_BLOCK = TH < 128 ? 128 / TH : 1;
    const int lane = threadIdx.x % TH, p = blockIdx.y * PER_BLOCK + threadIdx.x / TH, t = blockIdx.x;
    __shared__ float red[32];
    if (PER_BLOCK > 1 && p >= parts) return;
    const size_t plane = (size_t)T * g_stride;
    const float *op = o + (size_t)t * C + (size_t)p * n, *gp = g + (size_t)t * g_stride + g_col0 + (size_t)p * n;
    float v[N * V], gate[N * V];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < N; j++) {
        const int c = (lane + j * TH) * V;
        if (c < n) {
            if constexpr (V == 4) {
                const float4 a = *(const float4 *)(op + c), z = plane_sum4(gp + c, splits, plane);
                v[4 * j] = a.x; v[4 * j + 1] = a.y; v[4 * j + 2] = a.z; v[4 * j + 3] = a.w;
                gate[4 * j] = z.x; gate[4 * j + 1] = z.y; gate[4 * j + 2] = z.z; gate[4 * j + 3] = z.w;
            } else {
                v[j] = op[c];
                gate[j] = plane_sum(gp + c, splits, plane);
            }
        } else {
#pragma unroll
            for (int i = 0; i < V; i++) { v[V * j + i] = 0.f; gate[V * j + i] = 0.f; }
        }
    }
#pragma unroll
    for (int j = 0; j < N * V; j++) {
        gate[j] = SIGMOID ? sigmoid_for<TO>(gate[j]) : silu_for<TO>(gate[j]);
        if (gate_first) v[j] *= gate[j];
        ss = fmaf(v[j], v[j], ss);
    }
    ss = warp_sum(ss);
    if (TH > 32) {
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
        __syncthreads();
        ss = warp_sum((threadIdx.x & 31) < TH / 32 ? red[threadIdx.x & 31] : 0.f);
    }
    const float r = 1.0f / sqrtf(ss / (float)n + eps);
    TO *dst = out + (size_t)t * out_stride + (size_t)p * n;
#pragma unroll
    for (int j = 0; j < N; j++) {
        const int c = (lane + j * TH) * V;
        if (c >= n) continue;
#pragma unroll
        for (int i = 0; i < V; i++) {
            float y = v[V * j + i] * r;
            if (w) y *= w[(size_t)p * n + c + i];
            if (!gate_first) y *= gate[V * j + i];
            v[V * j + i] = y;
        }
        if constexpr (V == 4) {
            store2(dst + c, v[4 * j], v[4 * j + 1]);
            store2(dst + c + 2, v[4 * j + 2], v[4 * j + 3]);
        } else {
            dst[c] = from_f32<TO>(v[j]);
        }
    }
}

}  // namespace hfb

using namespace hfb;

static int bad_sizes(const char *who, int H, int Hq, int d, int dv, int dp, int dvp)
{
    if (H <= 0 || Hq <= 0 || H % Hq || d <= 0 || dv <= 0 || dp < d || dvp < dv || (dp & 15) || (dvp & 15))
        return fail(HFB_EINVAL, "%s: bad sizes (H=%d Hq=%d d=%d/%d dv=%d/%d)", who, H, Hq, d, dp, dv, dvp);
    if (dp > DS_MAX_D) return fail(HFB_ENOTSUP, "%s: key heads above %d are not supported", who, DS_MAX_D);
    if (H > 65535) return fail(HFB_ENOTSUP, "%s: %d heads exceed the grid limit", who, H);
    return HFB_OK;
}

extern "C" int hfb_rotate_heads(const float *src, int splits, int row_stride, const float *cos_sin, int n_rot, int n_positions,
                                const int32_t *positions, float k_scale, void *q, void *k, void *u, int out_dt, int T, int H, int d, int dv,
                                int dp, int dvp, int silu, hfb_stream s)
{
    if (T <= 0) return HFB_OK;
    int rc = bad_sizes("rotate_heads", H, H, d, dv, dp, dvp);
    if (rc != HFB_OK) return rc;
    if (!src || splits < 1 || row_stride < H * (2 * d + dv) || n_rot < 0 || n_rot > d || (n_rot & 1) || (n_rot && (!cos_sin || !positions)) ||
        !q || !k || !u || !valid_dt(out_dt))
        return fail(HFB_EINVAL, "rotate_heads: bad arguments (n_rot=%d)", n_rot);
    const dim3 grid(T, (H + 3) / 4);
    // (dp and dvp are multiples of 16, the outputs' heads therefore aligned)
    const int pairs = (d & 1) == 0 && (dv & 1) == 0 && (row_stride & 1) == 0 && (n_rot & 3) == 0 && ((uintptr_t)src & 7) == 0 && aligned16(cos_sin) &&
                      aligned16(q) && aligned16(k) && aligned16(u);
#define HFB_ROT(TY, SILU) \
    g_launch_err = launch_pdl(rotate_heads_kernel<TY, SILU>, grid, dim3(128), 0, (cudaStream_t)s, src, splits, row_stride, cos_sin, n_rot, n_positions, \
                              positions, k_scale, (TY *)q, (TY *)k, (TY *)u, T, H, d, dv, dp, dvp, pairs, error_word())
    if (out_dt == HFB_F32) { if (silu) HFB_ROT(float, true); else HFB_ROT(float, false); }
    else { if (silu) HFB_ROT(__nv_bfloat16, true); else HFB_ROT(__nv_bfloat16, false); }
#undef HFB_ROT
    return check_pdl_launch(g_launch_err, "rotate_heads");
}

extern "C" int hfb_state_space_operands(const float *src, int splits, int row_stride, const void *w, int w_dt, const void *bias, int bias_dt,
                                        int taps, const void *dt_bias, int dtb_dt, const float *rate, float *carried, int64_t slot_stride,
                                        const int32_t *token_seq, const int32_t *cu_tokens, const int32_t *seq_slots, int n_slots, int S,
                                        void *q, void *k, void *u, int out_dt, float *step, float *la, int T, int H, int G, int d, int dv,
                                        int dp, int dvp, hfb_stream s)
{
    if (T <= 0 || S <= 0) return HFB_OK;
    int rc = bad_sizes("state_space_operands", H, G, d, dv, dp, dvp);
    if (rc != HFB_OK) return rc;
    const int CC = H * dv + 2 * G * d;
    if (!src || splits < 1 || row_stride < H * dv + CC + H || !w || !valid_dt(w_dt) || !bias || !valid_dt(bias_dt) || !dt_bias || !valid_dt(dtb_dt) ||
        !rate || !carried || !token_seq || !cu_tokens || !seq_slots || !q || !k || !u || !valid_dt(out_dt) || !step || !la || taps < 1)
        return fail(HFB_EINVAL, "state_space_operands: bad arguments (taps=%d)", taps);
    if (taps > DS_MAX_TAPS) return fail(HFB_ENOTSUP, "state_space_operands: %d taps exceed %d", taps, DS_MAX_TAPS);
    const int single = T == S;                           // every request brings one token
    const bool two = (d & 1) == 0 && (dv & 1) == 0 && (row_stride & 1) == 0 && ((uintptr_t)src & 7) == 0 && aligned16(q) && aligned16(k) && aligned16(u);
    const int per = two ? 256 : 128;
    const int blocks_x = (CC + per - 1) / per + (H + 127) / 128;
    int tt = 32;                                         // tokens of a block: fewer where that leaves SMs idle
    while (tt > 1 && (long)blocks_x * ((T + tt - 1) / tt) < 148 * 8) tt >>= 1;
    if ((T + tt - 1) / tt > 65535) tt = (T + 65534) / 65535;
    const dim3 grid(blocks_x, (T + tt - 1) / tt);
#define HFB_SSO(TAPS, V, TY) \
    g_launch_err = launch_pdl(state_space_operands_kernel<TAPS, V, TY>, grid, dim3(128), 0, (cudaStream_t)s, src, splits, row_stride, w, w_dt, bias, bias_dt, \
                              taps, dt_bias, dtb_dt, rate, carried, (size_t)slot_stride, token_seq, cu_tokens, seq_slots, n_slots, single, (TY *)q, \
                              (TY *)k, (TY *)u, step, la, T, H, G, d, dv, dp, dvp, tt, error_word())
#define HFB_SSOT(TY) do { if (taps == 4 && two) HFB_SSO(4, 2, TY); else if (taps == 4) HFB_SSO(4, 1, TY); else if (two) HFB_SSO(0, 2, TY); else HFB_SSO(0, 1, TY); } while (0)
    if (out_dt == HFB_F32) HFB_SSOT(float);
    else HFB_SSOT(__nv_bfloat16);
#undef HFB_SSOT
#undef HFB_SSO
    rc = check_pdl_launch(g_launch_err, "state_space_operands");
    if (rc != HFB_OK || single) return rc;
    return hfb_conv_carry(src, splits, row_stride, H * dv, taps, carried, slot_stride, cu_tokens, seq_slots, n_slots, S, T, CC, s);
}

extern "C" int hfb_decay_walk(const void *q, const void *k, const void *u, int dt, const float *la, int la_stride, const float *fixed,
                              const float *step, const float *skip, float *state, int64_t slot_stride, const int32_t *cu_tokens, const int32_t *seq_slots,
                              int n_slots, int S, float *o, int H, int Hq, int d, int dv, int dp, int dvp, hfb_stream s)
{
    if (S <= 0) return HFB_OK;
    int rc = bad_sizes("decay_walk", H, Hq, d, dv, dp, dvp);
    if (rc != HFB_OK) return rc;
    if (!q || !k || !u || !valid_dt(dt) || !la || (la_stride != 0 && la_stride != H) || !state || !cu_tokens || !seq_slots || !o ||
        slot_stride < (int64_t)H * dvp * dp || (slot_stride & 3) || !aligned16(state) || !aligned16(q) || !aligned16(k))
        return fail(HFB_EINVAL, "decay_walk: bad arguments");
#define HFB_WALK(TY, L, J) do { \
        const int cols = 4 * (32 / L) * DS_COLS; \
        g_launch_err = launch_pdl(decay_walk_kernel<TY, L, J>, dim3(S, H, (dvp + cols - 1) / cols), dim3(128), 0, (cudaStream_t)s, (const TY *)q, \
            (const TY *)k, (const TY *)u, la, la_stride, fixed, step, skip, state, (size_t)slot_stride, cu_tokens, seq_slots, n_slots, o, H, Hq, dp, dv, dvp, \
            error_word()); \
    } while (0)
#define HFB_WALKS(TY) do { \
        if (dp <= 32) HFB_WALK(TY, 8, 1); \
        else if (dp <= 64) HFB_WALK(TY, 16, 1); \
        else if (dp <= 128) HFB_WALK(TY, 32, 1); \
        else if (dp <= 256) HFB_WALK(TY, 32, 2); \
        else HFB_WALK(TY, 32, 4); \
    } while (0)
    if (dt == HFB_F32) HFB_WALKS(float);
    else HFB_WALKS(__nv_bfloat16);
#undef HFB_WALKS
#undef HFB_WALK
    return check_pdl_launch(g_launch_err, "decay_walk");
}

// Bytes of scratch hfb_decay_chunks needs for `chunks` chunks (0: these sizes have no chunk form).
extern "C" size_t hfb_decay_chunks_scratch(int chunks, int H, int dp, int dvp)
{
    if (dp > DS_MAX_CHUNK_D) return 0;
    const size_t state = (size_t)H * dp * dvp;
    return (size_t)chunks * (state * 8 + (((size_t)H * 4 + 15) & ~(size_t)15)) + 16;
}

extern "C" int hfb_decay_chunk_tokens(void) { return DS_CH; }

// All of a step's tokens in chunks: chunk c is tokens chunk_t0[c] .. + chunk_n[c] - 1 of one request (at most DS_CH), the
// chunks of request s are chunk_first[s] .. chunk_first[s + 1] - 1 in order.  bfloat16 operands.
extern "C" int hfb_decay_chunks(const void *q, const void *k, const void *u, const float *la, int la_stride, const float *step,
                                const float *skip, float *state, int64_t slot_stride, const int32_t *chunk_t0, const int32_t *chunk_n,
                                const int32_t *chunk_first, int chunks, const int32_t *seq_slots, int n_slots, int S, void *scratch,
                                size_t scratch_bytes, float *o, int H, int Hq, int d, int dv, int dp, int dvp, hfb_stream s)
{
    if (S <= 0 || chunks <= 0) return HFB_OK;
    int rc = bad_sizes("decay_chunks", H, Hq, d, dv, dp, dvp);
    if (rc != HFB_OK) return rc;
    if (dp > DS_MAX_CHUNK_D) return fail(HFB_ENOTSUP, "decay_chunks: key heads above %d have no chunk form", DS_MAX_CHUNK_D);
    if (!q || !k || !u || !la || (la_stride != 0 && la_stride != H) || !state || !chunk_t0 || !chunk_n || !chunk_first || !seq_slots || !o ||
        slot_stride < (int64_t)H * dvp * dp || (slot_stride & 3) || !aligned16(state) || !aligned16(q) || !aligned16(k) || !aligned16(u) ||
        !aligned16(scratch) || scratch_bytes < hfb_decay_chunks_scratch(chunks, H, dp, dvp) || S > 65535)
        return fail(HFB_EINVAL, "decay_chunks: bad arguments");
    const size_t st = (size_t)H * dp * dvp;
    float *dS = (float *)scratch;
    __nv_bfloat16 *start = (__nv_bfloat16 *)(dS + (size_t)chunks * st);
    float *l_end = (float *)(start + (size_t)chunks * st * 2);
    const int v_tiles = (dvp + DS_DVT - 1) / DS_DVT;
#define HFB_CHUNK_STATE(KT) \
    g_launch_err = launch_pdl(decay_chunk_state_kernel<KT>, dim3(chunks, H, v_tiles * ((dp + KT - 1) / KT)), dim3(128), 0, (cudaStream_t)s, \
                              (const __nv_bfloat16 *)k, (const __nv_bfloat16 *)u, la, la_stride, step, chunk_t0, chunk_n, dS, l_end, H, Hq, dp, dvp)
    if (dp <= 64) HFB_CHUNK_STATE(64);
    else HFB_CHUNK_STATE(128);
#undef HFB_CHUNK_STATE
    if ((rc = check_pdl_launch(g_launch_err, "decay_chunk_state")) != HFB_OK) return rc;
    g_launch_err = launch_pdl(decay_chunk_pass_kernel, dim3((unsigned)((st / 4 + 255) / 256), S), dim3(256), 0, (cudaStream_t)s, dS, l_end, state,
                              (size_t)slot_stride, chunk_first, seq_slots, n_slots, start, H, dp, dvp, error_word());
    if ((rc = check_pdl_launch(g_launch_err, "decay_chunk_pass")) != HFB_OK) return rc;
    // a block's share of the items that read one query/key head: the one with the fewest rounds over the SMs, a block's start
    // (keys, queries, the first item's state) counted as one item more
    const int items = H / Hq * v_tiles, resident = 148 * (dp <= 128 ? 2 : 1);
    int per_block = 1;
    long best = -1;
    for (int p = 1; p <= items && p <= 32; p++) {
        const long blocks = (long)chunks * Hq * ((items + p - 1) / p), cost = (blocks + resident - 1) / resident * (p + 1);
        if (best < 0 || cost < best) { best = cost; per_block = p; }
    }
    const int shares = (items + per_block - 1) / per_block;
    if ((long)Hq * shares > 65535) return fail(HFB_ENOTSUP, "decay_chunks: %d heads exceed the grid limit", H);
#define HFB_CHUNK_OUT(NK) do { \
        const int smem_c = (DS_CH * (NK * 16 + 8) + 2 * (2 * DS_DVT * (NK * 16 + 8) + DS_CH * (DS_DVT + 8))) * 2; \
        static bool opted[64] = {false}; \
        const int dev = current_device(); \
        if (!opted[dev]) { \
            cudaError_t e = cudaFuncSetAttribute(decay_chunk_out_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_c); \
            if (e != cudaSuccess) return fail(HFB_ECUDA, "decay_chunks: %s", cudaGetErrorString(e)); \
            opted[dev] = true; \
        } \
        g_launch_err = launch_pdl(decay_chunk_out_kernel<NK>, dim3(chunks, Hq * shares), dim3(128), smem_c, (cudaStream_t)s, (const __nv_bfloat16 *)q, \
                                  (const __nv_bfloat16 *)k, (const __nv_bfloat16 *)u, la, la_stride, step, skip, start, chunk_t0, chunk_n, o, H, Hq, \
                                  dp, dv, dvp, v_tiles, per_block); \
    } while (0)
    if (dp <= 64) HFB_CHUNK_OUT(4);
    else if (dp <= 128) HFB_CHUNK_OUT(8);
    else HFB_CHUNK_OUT(16);
#undef HFB_CHUNK_OUT
    return check_pdl_launch(g_launch_err, "decay_chunk_out");
}

extern "C" int hfb_part_norm_gate(const float *o, const float *g, int splits, int g_stride, int g_col0, const float *w, float eps,
                                  int gate_first, int sigmoid, void *out, int out_dt, int64_t out_stride, int T, int C, int parts,
                                  hfb_stream s)
{
    if (T <= 0) return HFB_OK;
    if (!o || !g || splits < 1 || C <= 0 || parts < 1 || C % parts || g_col0 < 0 || g_col0 + C > g_stride || !out || !valid_dt(out_dt) || out_stride < C)
        return fail(HFB_EINVAL, "part_norm_gate: bad arguments (C=%d parts=%d)", C, parts);
    const int n = C / parts, esz = out_dt == HFB_F32 ? 4 : 2;
    if (n > 16 * 1024) return fail(HFB_ENOTSUP, "part_norm_gate: parts of %d values exceed %d", n, 16 * 1024);
    if (parts > 65535) return fail(HFB_ENOTSUP, "part_norm_gate: %d parts exceed the grid limit", parts);
    const bool vec = (n & 3) == 0 && (g_stride & 3) == 0 && (g_col0 & 3) == 0 && aligned16(o) && aligned16(g) && (out_stride & 3) == 0 &&
                     ((uintptr_t)out & (4 * esz - 1)) == 0;
#define HFB_PNG(TY, TH, V, N, SG) \
    g_launch_err = launch_pdl(part_norm_gate_kernel<TY, TH, V, N, SG>, dim3(T, TH < 128 ? (parts + 128 / TH - 1) / (128 / TH) : parts), dim3(TH < 128 ? 128 : TH), \
                              0, (cudaStream_t)s, o, g, splits, g_stride, g_col0, w, eps, gate_first, (TY *)out, (size_t)out_stride, T, C, n, parts)
    // a warp for parts of up to 128, 256 or 512 values, else a block
#define HFB_PNGT(TY, SG) do { \
        if (vec) { \
            if (n <= 128) HFB_PNG(TY, 32, 4, 1, SG); else if (n <= 256) HFB_PNG(TY, 32, 4, 2, SG); else if (n <= 512) HFB_PNG(TY, 32, 4, 4, SG); \
            else if (n <= 2048) HFB_PNG(TY, 256, 4, 2, SG); else if (n <= 4096) HFB_PNG(TY, 256, 4, 4, SG); else HFB_PNG(TY, 1024, 4, 4, SG); \
        } else { \
            if (n <= 512) HFB_PNG(TY, 32, 1, 16, SG); else if (n <= 4096) HFB_PNG(TY, 256, 1, 16, SG); else HFB_PNG(TY, 1024, 1, 16, SG); \
        } \
    } while (0)
    if (out_dt == HFB_F32) { if (sigmoid) HFB_PNGT(float, true); else HFB_PNGT(float, false); }
    else { if (sigmoid) HFB_PNGT(__nv_bfloat16, true); else HFB_PNGT(__nv_bfloat16, false); }
#undef HFB_PNGT
#undef HFB_PNG
    return check_pdl_launch(g_launch_err, "part_norm_gate");
}
