// What ends a sublayer whose output is normed before it joins the stream, and a step between layers, in one pass over
// the float32 stream.  Per row:
//
//     v = sum of a product's `splits` partial sums (+ bias) (+ sum_j mix_w[j] mix_y[j], j in order)
//     v = v / sqrt(mean(v^2) + eps) * post_w              (where post_w is given)
//     x = base + v                                        (base: the stream itself where none is given)
//     out = x / sqrt(mean(x^2) + eps) * next_w            (next_w given), or x as it is (else; `out` may be null)
//
// One block per row with the row's values in registers, so both norms and the next product's operand cost one read of the
// sums and of the stream and one write each.  The number of threads goes with the row's width only: the order in which
// squares are summed does not depend on what else the step holds.  Everything is float32 but `out` in the run's type.
#include "common.cuh"

static thread_local cudaError_t g_launch_err = cudaSuccess;      // what the last launch_pdl returned

namespace hfb {

// Sum over the block, the same value in every thread; `red` holds one float per warp and is not shared between two sums.
__device__ __forceinline__ float rt_block_sum(float v, float *red)
{
    v = warp_sum(v);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (lane == 0) red[warp] = v;
    __syncthreads();
    return warp_sum(lane < (int)(blockDim.x >> 5) ? red[lane] : 0.f);
}

template <int V> struct RtVec;
template <> struct RtVec<1> {
    float v[1];
    __device__ __forceinline__ void load(const float *p) { v[0] = p[0]; }
    __device__ __forceinline__ void store(float *p) const { p[0] = v[0]; }
};
template <> struct RtVec<4> {
    float v[4];
    __device__ __forceinline__ void load(const float *p)
    {
        const float4 a = *(const float4 *)p;
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    }
    __device__ __forceinline__ void store(float *p) const { *(float4 *)p = make_float4(v[0], v[1], v[2], v[3]); }
};

// V consecutive elements of a vector of either type; 16-byte (8-byte) reads where V is 4 (the caller checks alignment)
template <int V> __device__ __forceinline__ void rt_load_any(const void *p, int dt, int i, float *w)
{
    if constexpr (V == 4) {
        if (dt == HFB_F32) {
            const float4 a = *(const float4 *)((const float *)p + i);
            w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w;
        } else {
            const uint2 u = *(const uint2 *)((const __nv_bfloat16 *)p + i);
            const float2 a = __bfloat1622float2(*(const __nv_bfloat162 *)&u.x), b = __bfloat1622float2(*(const __nv_bfloat162 *)&u.y);
            w[0] = a.x; w[1] = a.y; w[2] = b.x; w[3] = b.y;
        }
    } else {
        w[0] = load_any(p, dt, i);
    }
}

template <int V> __device__ __forceinline__ void rt_store_out(void *p, int dt, size_t i, const float *v)
{
    if constexpr (V == 4) {
        if (dt == HFB_F32) {
            *(float4 *)((float *)p + i) = make_float4(v[0], v[1], v[2], v[3]);
        } else {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
            *(uint2 *)((__nv_bfloat16 *)p + i) = make_uint2(*(const uint32_t *)&a, *(const uint32_t *)&b);
        }
    } else {
        store_any(p, dt, i, v[0]);
    }
}

struct RtArgs {
    const float *y;
    int splits;
    const void *bias;
    int bias_dt;
    const float *mix_y, *mix_w;
    int top;
    const void *post_w;
    int post_dt;
    float post_eps;
    const float *base;
    float *residual;
    const void *next_w;
    int next_dt;
    float next_eps;
    void *out;
    int out_dt, M, N;
};

template <int V, int PER, int TH>
__global__ void __launch_bounds__(TH)
rms_tail_kernel(RtArgs a)
{
    pdl_entry();
    __shared__ float red[2][32];
    const int m = blockIdx.x, N = a.N;
    const size_t MN = (size_t)a.M * N, row = (size_t)m * N;
    // what the kernel in front does not write is fetched while it finishes (rows of one vector a thread; wider ones read it
    // where it is used, for want of registers)
    constexpr bool EARLY = PER == 1;
    float pw[EARLY ? V : 1], nw[EARLY ? V : 1], bv[EARLY ? V : 1];
    const int i0 = threadIdx.x * V;
    if (EARLY && i0 < N) {
        if (a.post_w) rt_load_any<V>(a.post_w, a.post_dt, i0, pw);
        if (a.next_w) rt_load_any<V>(a.next_w, a.next_dt, i0, nw);
        if (a.bias) rt_load_any<V>(a.bias, a.bias_dt, i0, bv);
    }
    pdl_sync_small();
    const bool sums = a.splits > 0 || a.mix_y;
    const float *base = (a.base ? a.base : a.residual) + row;
    RtVec<V> v[PER], x[PER];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; j++) {
        const int i = (threadIdx.x + j * TH) * V;
#pragma unroll
        for (int e = 0; e < V; e++) v[j].v[e] = x[j].v[e] = 0.f;
        if (i >= N) continue;
        x[j].load(base + i);
        if (!sums) continue;
        // eight planes (four rows of the mix) in flight: their latency is what a step of few tokens waits for
        for (int s0 = 0; s0 < a.splits; s0 += 8) {
            RtVec<V> q[8];
#pragma unroll
            for (int k = 0; k < 8; k++) {
                if (s0 + k < a.splits) q[k].load(a.y + (size_t)(s0 + k) * MN + row + i);
                else
#pragma unroll
                    for (int e = 0; e < V; e++) q[k].v[e] = 0.f;
            }
#pragma unroll
            for (int k = 0; k < 8; k++)
#pragma unroll
                for (int e = 0; e < V; e++) v[j].v[e] += q[k].v[e];
        }
        if (a.bias) {
            float b[V];
            if (EARLY) {
#pragma unroll
                for (int e = 0; e < V; e++) b[e] = bv[EARLY ? e : 0];
            } else {
                rt_load_any<V>(a.bias, a.bias_dt, i, b);
            }
#pragma unroll
            for (int e = 0; e < V; e++) v[j].v[e] += b[e];
        }
        if (a.mix_y) {
            RtVec<V> acc;
#pragma unroll
            for (int e = 0; e < V; e++) acc.v[e] = 0.f;
            for (int k0 = 0; k0 < a.top; k0 += 4) {
                RtVec<V> q[4];
                float w[4];
#pragma unroll
                for (int k = 0; k < 4; k++) {
                    const size_t p = (size_t)m * a.top + k0 + k;
                    w[k] = 0.f;
#pragma unroll
                    for (int e = 0; e < V; e++) q[k].v[e] = 0.f;
                    if (k0 + k < a.top) { q[k].load(a.mix_y + p * N + i); w[k] = a.mix_w[p]; }
                }
#pragma unroll
                for (int k = 0; k < 4; k++)
#pragma unroll
                    for (int e = 0; e < V; e++) acc.v[e] = fmaf(w[k], q[k].v[e], acc.v[e]);
            }
#pragma unroll
            for (int e = 0; e < V; e++) v[j].v[e] += acc.v[e];
        }
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(v[j].v[e], v[j].v[e], ss);
    }
    const float r = a.post_w ? 1.0f / sqrtf(rt_block_sum(ss, red[0]) / (float)N + a.post_eps) : 1.0f;
    float s2 = 0.f;
#pragma unroll
    for (int j = 0; j < PER; j++) {
        const int i = (threadIdx.x + j * TH) * V;
        if (i >= N) continue;
        float w[V];
        if (a.post_w) {
            if (EARLY) {
#pragma unroll
                for (int e = 0; e < V; e++) w[e] = pw[EARLY ? e : 0];
            } else {
                rt_load_any<V>(a.post_w, a.post_dt, i, w);
            }
        }
#pragma unroll
        for (int e = 0; e < V; e++) {
            x[j].v[e] += a.post_w ? v[j].v[e] * r * w[e] : v[j].v[e];
            s2 = fmaf(x[j].v[e], x[j].v[e], s2);
        }
        if (sums) x[j].store(a.residual + row + i);
    }
    if (!a.out) return;
    const float rn = a.next_w ? 1.0f / sqrtf(rt_block_sum(s2, red[1]) / (float)N + a.next_eps) : 1.0f;
#pragma unroll
    for (int j = 0; j < PER; j++) {
        const int i = (threadIdx.x + j * TH) * V;
        if (i >= N) continue;
        float y[V];
        if (a.next_w) {
            float w[V];
            if (EARLY) {
#pragma unroll
                for (int e = 0; e < V; e++) w[e] = nw[EARLY ? e : 0];
            } else {
                rt_load_any<V>(a.next_w, a.next_dt, i, w);
            }
#pragma unroll
            for (int e = 0; e < V; e++) y[e] = (x[j].v[e] * rn) * w[e];
        } else {
#pragma unroll
            for (int e = 0; e < V; e++) y[e] = x[j].v[e];
        }
        rt_store_out<V>(a.out, a.out_dt, row + i, y);
    }
}

}  // namespace hfb

using namespace hfb;

extern "C" int hfb_rms_tail(const float *y, int splits, const void *bias, int bias_dt, const float *mix_y, const float *mix_w, int top,
                            const void *post_w, int post_dt, float post_eps, const float *base, float *residual, const void *next_w,
                            int next_dt, float next_eps, void *out, int out_dt, int M, int N, hfb_stream s)
{
    if (M <= 0) return HFB_OK;
    const bool sums = splits > 0 || mix_y;
    if (N <= 0 || !residual || splits < 0 || (splits > 0 && !y) || (mix_y && (!mix_w || top < 1)) || (!sums && (post_w || bias || base)) ||
        (bias && !valid_dt(bias_dt)) || (post_w && !valid_dt(post_dt)) || (next_w && (!out || !valid_dt(next_dt))) ||
        (out && !valid_dt(out_dt)) || (!sums && !out))
        return fail(HFB_EINVAL, "rms_tail: bad arguments (M=%d N=%d splits=%d)", M, N, splits);
    if (N > 16384) return fail(HFB_ENOTSUP, "rms_tail: rows above 16384 values are not supported (%d)", N);
    RtArgs a{splits > 0 ? y : nullptr, splits, bias, bias_dt, mix_y, mix_w, top, post_w, post_dt, post_eps, base, residual, next_w, next_dt, next_eps, out, out_dt, M, N};
    auto al = [](const void *p, size_t n) { return ((uintptr_t)p & (n - 1)) == 0; };
    auto al_dt = [&](const void *p, int dt) { return !p || al(p, dt == HFB_F32 ? 16 : 8); };
    const bool vec = (N & 3) == 0 && al(a.y, 16) && al(mix_y, 16) && al(base, 16) && al(residual, 16) && al_dt(bias, bias_dt) &&
                     al_dt(post_w, post_dt) && al_dt(next_w, next_dt) && al_dt(out, out_dt);
    cudaStream_t st = (cudaStream_t)s;
#define HFB_RT(V, PER, TH) g_launch_err = launch_pdl(rms_tail_kernel<V, PER, TH>, dim3(M), dim3(TH), 0, st, a)
    if (vec) {
        if (N <= 512) HFB_RT(4, 1, 128);
        else if (N <= 1024) HFB_RT(4, 1, 256);
        else if (N <= 2048) HFB_RT(4, 1, 512);
        else if (N <= 4096) HFB_RT(4, 1, 1024);
        else if (N <= 8192) HFB_RT(4, 2, 1024);
        else HFB_RT(4, 4, 1024);
    } else {
        if (N <= 512) HFB_RT(1, 2, 256);
        else if (N <= 2048) HFB_RT(1, 4, 512);
        else HFB_RT(1, 16, 1024);
    }
#undef HFB_RT
    return check_pdl_launch(g_launch_err, "rms_tail");
}
