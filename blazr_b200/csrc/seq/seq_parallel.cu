// seq_parallel.cu -- the residual path of parallel layers: one norm per layer whose output both the mixer and the feed-forward read,
// x <- x + mult * (mixer(h) + ff(h)).  Between two layers ONE kernel: the mixer's branches with their norms (or the deferred norm of a linear attention),
// the weighted sum of the experts' rows, the residual sum, the row added in front of a pass, the next layer's norm and its input in the activation
// type.  All arithmetic in f32.
#include "seq_common.cuh"

namespace b200seq {

// two sums over the block at once; red: >= 66 floats.  Fixed order: deterministic.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    a = warp_sum(a), b = warp_sum(b);
    __syncthreads();
    if (lane == 0) red[wid] = a, red[33 + wid] = b;
    __syncthreads();
    if (wid == 0) {
        a = warp_sum(lane < nw ? red[lane] : 0.f), b = warp_sum(lane < nw ? red[33 + lane] : 0.f);
        if (lane == 0) red[32] = a, red[65] = b;
    }
    __syncthreads();
    return make_float2(red[32], red[65]);
}

template <int VW>
struct Vec {
    float v[VW];
};
template <int VW>
__device__ __forceinline__ Vec<VW> ldv(const float* p) {
    Vec<VW> r;
    if (VW == 4) {
        const float4 q = ld4(p);
        r.v[0] = q.x, r.v[1 % VW] = q.y, r.v[2 % VW] = q.z, r.v[3 % VW] = q.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}

// one block per row; a thread keeps EPT groups of VW neighbouring elements in registers (W <= VW * EPT * blockDim.x; VW = 4: W % 4 == 0, 16-byte aligned rows)
template <int VW, int EPT>
__global__ void __launch_bounds__(512) parallel_close_kernel(const b200seq_parallel_desc a) {
    __shared__ float red[66];
    const int r = blockIdx.x, W = a.W, nt = blockDim.x;
    const int64_t t = a.rows ? a.rows[r] : r;
    Vec<VW> x[EPT], y1[EPT], y2[EPT];
    float ss1 = 0.f, ss2 = 0.f;
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = VW * (threadIdx.x + k * nt);
        const bool in = i < W;
#pragma unroll
        for (int u = 0; u < VW; ++u) x[k].v[u] = y1[k].v[u] = y2[k].v[u] = 0.f;
        if (!in) continue;
        x[k] = ldv<VW>(a.x + t * W + i), y1[k] = ldv<VW>(a.y1 + t * W + i);
        if (a.y2) y2[k] = ldv<VW>(a.y2 + t * W + i);
    }
#pragma unroll
    for (int k = 0; k < EPT; ++k)
#pragma unroll
        for (int u = 0; u < VW; ++u) ss1 = fmaf(y1[k].v[u], y1[k].v[u], ss1), ss2 = fmaf(y2[k].v[u], y2[k].v[u], ss2);
    float r1 = 1.f, r2 = 1.f;
    if (a.ss1) {        // deferred norm: the partial sums are in memory
        ss1 = 0.f;
        for (int i = threadIdx.x; i < a.ss_n; i += nt) ss1 += a.ss1[t * a.ss_n + i];
    }
    if (a.w_b1 || a.w_b2 || a.ss1) {
        const float2 s = block_sum2(ss1, ss2, red);
        if (a.ss1) r1 = 1.0f / sqrtf(s.x / (float)a.ss_count + a.eps);
        else if (a.w_b1) r1 = 1.0f / sqrtf(s.x / (float)W + a.eps);
        if (a.w_b2) r2 = 1.0f / sqrtf(s.y / (float)W + a.eps);
    }
    const float m1 = a.s1 * r1, m2 = a.s2 * r2;
    float sf = 0.f;
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = VW * (threadIdx.x + k * nt);
        if (i >= W) continue;
        Vec<VW> b;
#pragma unroll
        for (int u = 0; u < VW; ++u) b.v[u] = m1 * y1[k].v[u];
        if (a.w_b1) {
            const Vec<VW> w = ldv<VW>(a.w_b1 + i);
#pragma unroll
            for (int u = 0; u < VW; ++u) b.v[u] *= w.v[u];
        }
        if (a.y2) {
            Vec<VW> c = y2[k];
            if (a.w_b2) {
                const Vec<VW> w = ldv<VW>(a.w_b2 + i);
#pragma unroll
                for (int u = 0; u < VW; ++u) c.v[u] *= w.v[u];
            }
#pragma unroll
            for (int u = 0; u < VW; ++u) b.v[u] = fmaf(m2, c.v[u], b.v[u]);
        }
        if (a.ys) {
            for (int j = 0; j < a.top; ++j) {
                const int64_t p = t * a.top + j;
                const int64_t s = a.slot_of ? a.slot_of[p] : p;
                const Vec<VW> f = ldv<VW>(a.ys + s * W + i);
                const float wt = a.wts[p];
#pragma unroll
                for (int u = 0; u < VW; ++u) b.v[u] = fmaf(wt, f.v[u], b.v[u]);
            }
        } else if (a.y3) {
            const Vec<VW> f = ldv<VW>(a.y3 + t * W + i);
#pragma unroll
            for (int u = 0; u < VW; ++u) b.v[u] += f.v[u];
        }
#pragma unroll
        for (int u = 0; u < VW; ++u) x[k].v[u] = fmaf(a.mult, b.v[u], x[k].v[u]);
        if (a.add_vec) {
            const Vec<VW> w = ldv<VW>(a.add_vec + i);
#pragma unroll
            for (int u = 0; u < VW; ++u) x[k].v[u] += w.v[u];
        }
#pragma unroll
        for (int u = 0; u < VW; ++u) sf = fmaf(x[k].v[u], x[k].v[u], sf);
        if (a.x_out) {
            if (VW == 4) *reinterpret_cast<float4*>(a.x_out + t * W + i) = make_float4(x[k].v[0], x[k].v[1 % VW], x[k].v[2 % VW], x[k].v[3 % VW]);
            else a.x_out[t * W + i] = x[k].v[0];
        }
    }
    if (!a.a_out) return;
    float rf = 1.f;
    if (a.fin_w) rf = 1.0f / sqrtf(block_sum(sf, red) / (float)W + a.eps);
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = VW * (threadIdx.x + k * nt);
        if (i >= W) continue;
        Vec<VW> n = x[k];
        if (a.fin_w) {
            const Vec<VW> w = ldv<VW>(a.fin_w + i);
#pragma unroll
            for (int u = 0; u < VW; ++u) n.v[u] *= rf * w.v[u];
        }
        if (VW == 4) store_act4(a.a_out, a.out_dtype, (int64_t)r * W + i, make_float4(n.v[0], n.v[1 % VW], n.v[2 % VW], n.v[3 % VW]));
        else store_act(a.a_out, a.out_dtype, (int64_t)r * W + i, n.v[0]);
    }
}

template <int VW>
static bool launch_close(const b200seq_parallel_desc& d, cudaStream_t cs) {
    const int groups = (d.W + VW - 1) / VW;
    int nt = ((groups + 31) / 32) * 32;
    if (nt > 512) nt = 512;
    if (nt == 512 && groups <= 1024) nt = ((groups + 1) / 2 + 31) / 32 * 32;   // two groups per thread: fewer idle lanes
    const int ept = (groups + nt - 1) / nt;
    if (ept <= 1) parallel_close_kernel<VW, 1><<<d.R, nt, 0, cs>>>(d);
    else if (ept <= 2) parallel_close_kernel<VW, 2><<<d.R, nt, 0, cs>>>(d);
    else if (ept <= 4) parallel_close_kernel<VW, 4><<<d.R, nt, 0, cs>>>(d);
    else if (ept <= 8) parallel_close_kernel<VW, 8><<<d.R, nt, 0, cs>>>(d);
    else return false;
    return true;
}

}  // namespace b200seq

using namespace b200seq;

extern "C" int b200seq_parallel_close(const b200seq_parallel_desc* d, void* stream) {
    if (!d || !d->x || !d->y1 || d->W < 1 || d->R < 0 || (d->w_b2 && !d->y2) || (d->ss1 && (d->w_b1 || d->ss_n < 1 || d->ss_count < 1)) || (d->ys && (!d->wts || d->top < 1)) ||
        (d->ys && d->y3) || (d->a_out && d->out_dtype != B200SEQ_F32 && d->out_dtype != B200SEQ_BF16))
        return fail(B200SEQ_ERR_INVALID_ARG, "parallel_close: bad arguments");
    if (d->R == 0) return 0;
    const void* ps[] = {d->x, d->y1, d->w_b1, d->y2, d->w_b2, d->y3, d->ys, d->add_vec, d->x_out, d->a_out, d->fin_w};
    bool vec = d->W % 4 == 0;
    for (const void* p : ps) vec = vec && (reinterpret_cast<uintptr_t>(p) & 15) == 0;
    if (!(vec ? launch_close<4>(*d, (cudaStream_t)stream) : launch_close<1>(*d, (cudaStream_t)stream)))
        return fail(B200SEQ_ERR_UNSUPPORTED, "parallel_close: width %d too large", d->W);
    SEQ_LAUNCH_CHECK("parallel_close");
    return 0;
}
