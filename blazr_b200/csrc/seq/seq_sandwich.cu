// seq_sandwich.cu -- the residual path of layers whose sublayers are normed on both sides, x <- x + rms(f(rms(x) * w_in)) * w_out, with
// positions that enter as a sinusoid at the embedding, rows added in front of a looped span of layers, and an addition per layer that
// depends on the token id.  Between two sublayers ONE kernel: norm of the sublayer's result, residual sum, additions, the next sublayer's
// norm, its input in the activation type.  All arithmetic in f32.
#include <cooperative_groups.h>

#include "seq_common.cuh"

namespace b200seq {

__device__ __forceinline__ float4 add4(const float4 a, const float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float sq4(const float4 a, float acc) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, fmaf(a.w, a.w, acc)))); }

// pos * f with f = hi + lo carried in two floats: the product's rounding error joins the small part, sin and cos follow to first order
__device__ __forceinline__ void sincos_pos(float pos, float hi, float lo, float& sn, float& cs) {
    const float p = pos * hi;
    const float err = fmaf(pos, hi, -p) + pos * lo;
    float s, c;
    sincosf(p, &s, &c);
    sn = fmaf(c, err, s), cs = fmaf(-s, err, c);
}

// ---- embedding + sinusoid (+ a vector, + the first norm) -------------------------------------------------------------------------------------
// grid (T); freq: [2][(W + 1) / 2] high and low parts of the pair frequencies, or null (no positions)
struct EmbedPos {
    const __nv_bfloat16* table;
    const int32_t* ids;
    const float* freq;
    float scale;
    int W;
    float* x0;              // the embedding output itself, or null
    const float* add_vec;   // [W] or null
    float* x;
    const float* fin_w;     // norm of the first sublayer, or null: a = x
    float eps;
    void* a;                // or null
    int a_dtype;
    int pairs;
};
__global__ void embed_pos_kernel(const EmbedPos p, const b200seq_step st) {
    extern __shared__ __align__(16) float row[];   // [W] | 40 of reduction scratch
    const int t = blockIdx.x, W = p.W, np = (W + 1) >> 1;
    const __nv_bfloat16* src = p.table + (int64_t)p.ids[t] * W;
    const float pos = (float)st.tok_pos[t];
    float ss = 0.f;
    for (int i = threadIdx.x; i < np; i += blockDim.x) {
        float sn = 0.f, cs = 0.f;
        if (p.freq) sincos_pos(pos, p.freq[i], p.freq[np + i], sn, cs);
        if (p.pairs) {   // even width, aligned rows: both elements of a pair in one access
            const float2 tv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + 2 * i));
            float2 v = make_float2(fmaf(tv.x, p.scale, sn), fmaf(tv.y, p.scale, cs));
            const int64_t o = (int64_t)t * W + 2 * i;
            if (p.x0) *reinterpret_cast<float2*>(p.x0 + o) = v;
            if (p.add_vec) v.x += p.add_vec[2 * i], v.y += p.add_vec[2 * i + 1];
            *reinterpret_cast<float2*>(p.x + o) = v;
            *reinterpret_cast<float2*>(row + 2 * i) = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, ss));
            continue;
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int j = 2 * i + k;
            if (j >= W) continue;
            float v = fmaf(__bfloat162float(src[j]), p.scale, k ? cs : sn);
            if (p.x0) p.x0[(int64_t)t * W + j] = v;
            if (p.add_vec) v += p.add_vec[j];
            p.x[(int64_t)t * W + j] = v;
            row[j] = v;
            ss = fmaf(v, v, ss);
        }
    }
    if (!p.a) return;
    float rinv = 1.f;
    if (p.fin_w) rinv = 1.0f / sqrtf(block_sum(ss, row + W) / (float)W + p.eps);
    __syncthreads();
    for (int j = threadIdx.x; j < W; j += blockDim.x) store_act(p.a, p.a_dtype, (int64_t)t * W + j, p.fin_w ? row[j] * rinv * p.fin_w[j] : row[j]);
}

// the same without positions, the row in registers (W % 4 == 0, W <= 4 * EPT * blockDim.x, 16-byte aligned rows)
template <int EPT>
__global__ void __launch_bounds__(512) embed_reg_kernel(const EmbedPos p) {
    __shared__ float red[40];
    const int t = blockIdx.x, W = p.W, nt = blockDim.x;
    const __nv_bfloat16* src = p.table + (int64_t)p.ids[t] * W;
    float4 v[EPT];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = 4 * (threadIdx.x + k * nt);
        v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i >= W) continue;
        const uint2 r = *reinterpret_cast<const uint2*>(src + i);
        v[k] = make_float4(__uint_as_float(r.x << 16) * p.scale, __uint_as_float(r.x & 0xffff0000u) * p.scale, __uint_as_float(r.y << 16) * p.scale,
                           __uint_as_float(r.y & 0xffff0000u) * p.scale);
        if (p.x0) *reinterpret_cast<float4*>(p.x0 + (int64_t)t * W + i) = v[k];
        if (p.add_vec) v[k] = add4(v[k], ld4(p.add_vec + i));
        *reinterpret_cast<float4*>(p.x + (int64_t)t * W + i) = v[k];
        ss = sq4(v[k], ss);
    }
    if (!p.a) return;
    float rinv = 1.f;
    if (p.fin_w) rinv = 1.0f / sqrtf(block_sum(ss, red) / (float)W + p.eps);
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = 4 * (threadIdx.x + k * nt);
        if (i >= W) continue;
        float4 n = v[k];
        if (p.fin_w) {
            const float4 f = ld4(p.fin_w + i);
            n = make_float4(n.x * rinv * f.x, n.y * rinv * f.y, n.z * rinv * f.z, n.w * rinv * f.w);
        }
        store_act4(p.a, p.a_dtype, (int64_t)t * W + i, n);
    }
}

// ---- norm of a sublayer's result + residual + additions + next norm ----------------------------------------------------------------------------
struct SandwichArgs {
    const float *x, *y, *w;
    float eps;
    const float *add_row, *add_vec;
    int W;
    const int32_t* rows;
    float* x_out;
    void* a_out;
    int out_dtype;
    const float* fin_w;
};

// one block per row; dynamic shared memory: W floats + 40 of reduction scratch
__global__ void sandwich_norm_kernel(const SandwichArgs a) {
    extern __shared__ __align__(16) float v[];
    float* red = v + a.W;
    const int r = blockIdx.x, W = a.W;
    const int64_t t = a.rows ? a.rows[r] : r;
    const float* y = a.y ? a.y + t * W : nullptr;
    float rn = 0.f;
    if (y) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < W; i += blockDim.x) ss = fmaf(y[i], y[i], ss);
        rn = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
    }
    float sf = 0.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        float xn = a.x[t * W + i];
        if (y) xn += y[i] * rn * a.w[i];
        if (a.add_row) xn += a.add_row[t * W + i];
        if (a.add_vec) xn += a.add_vec[i];
        v[i] = xn;
        sf = fmaf(xn, xn, sf);
        if (a.x_out) a.x_out[t * W + i] = xn;
    }
    if (!a.a_out) return;
    float rf = 1.f;
    if (a.fin_w) rf = 1.0f / sqrtf(block_sum(sf, red) / (float)W + a.eps);
    for (int i = threadIdx.x; i < W; i += blockDim.x) store_act(a.a_out, a.out_dtype, (int64_t)r * W + i, a.fin_w ? v[i] * rf * a.fin_w[i] : v[i]);   // own elements only
}

// the row in registers (W % 4 == 0, W <= 4 * EPT * blockDim.x, 16-byte aligned rows).  PRE (few rows): the weights are requested with the rows.
template <int EPT, bool PRE>
__global__ void __launch_bounds__(512) sandwich_norm_reg_kernel(const SandwichArgs a) {
    __shared__ float red[40];
    const int r = blockIdx.x, W = a.W, nt = blockDim.x;
    const int64_t t = a.rows ? a.rows[r] : r;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 xv[EPT], yv[EPT], wv[EPT], fv[EPT];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = 4 * (threadIdx.x + k * nt);
        const bool in = i < W;
        xv[k] = in ? ld4(a.x + t * W + i) : zero;
        yv[k] = (in && a.y) ? ld4(a.y + t * W + i) : zero;
        if (in && a.add_row) xv[k] = add4(xv[k], ld4(a.add_row + t * W + i));
        if (in && a.add_vec) xv[k] = add4(xv[k], ld4(a.add_vec + i));
        if (PRE) {
            wv[k] = (in && a.w) ? ld4(a.w + i) : zero;
            fv[k] = (in && a.fin_w) ? ld4(a.fin_w + i) : zero;
        }
    }
    float rn = 0.f;
    if (a.y) {
#pragma unroll
        for (int k = 0; k < EPT; ++k) ss = sq4(yv[k], ss);
        rn = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
    }
    float sf = 0.f;
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = 4 * (threadIdx.x + k * nt);
        if (i >= W) continue;
        if (a.y) {
            const float4 w = PRE ? wv[k] : ld4(a.w + i);
            xv[k].x += yv[k].x * rn * w.x, xv[k].y += yv[k].y * rn * w.y, xv[k].z += yv[k].z * rn * w.z, xv[k].w += yv[k].w * rn * w.w;
        }
        sf = sq4(xv[k], sf);
        if (a.x_out) *reinterpret_cast<float4*>(a.x_out + t * W + i) = xv[k];
    }
    if (!a.a_out) return;
    float rf = 1.f;
    if (a.fin_w) rf = 1.0f / sqrtf(block_sum(sf, red) / (float)W + a.eps);
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int i = 4 * (threadIdx.x + k * nt);
        if (i >= W) continue;
        float4 n = xv[k];
        if (a.fin_w) {
            const float4 f = PRE ? fv[k] : ld4(a.fin_w + i);
            n = make_float4(n.x * rf * f.x, n.y * rf * f.y, n.z * rf * f.z, n.w * rf * f.w);
        }
        store_act4(a.a_out, a.out_dtype, (int64_t)r * W + i, n);
    }
}

// ---- the addition that depends on the token id ---------------------------------------------------------------------------------------------------
// g[t][j] = gelu_tanh(z[t][j]) * table[ids[t]][col + j]
// grid (T)
__global__ void token_gate_kernel(const float* __restrict__ z, int64_t ldz, int dim, const __nv_bfloat16* __restrict__ table, int64_t ldt, int col,
                                  const int32_t* __restrict__ ids, void* __restrict__ out, int out_dtype) {
    const int t = blockIdx.x;
    const __nv_bfloat16* row = table + (int64_t)ids[t] * ldt + col;
    for (int j = threadIdx.x; j < dim; j += blockDim.x) store_act(out, out_dtype, (int64_t)t * dim + j, gelu_tanhf_acc(z[t * ldz + j]) * __bfloat162float(row[j]));
}

// Steps of few tokens: the norm of the sublayer's result, the residual sum, the token's addition and the next norm in one kernel.  Any sizes: a block per row r
// (token t = rows ? rows[r] : r).  Dynamic shared memory: x [W] | projected addition [W] | gated [dim] | 40
struct SideArgs {
    SandwichArgs s;                   // x, y, w: the sublayer this closes; add_row / add_vec / fin_w / outputs: after the addition
    const __nv_bfloat16 *gate, *proj; // [dim][W], [W][dim]
    const __nv_bfloat16* table;
    int64_t ldt;
    int col, dim;
    const int32_t* ids;
    const float* side_w;
};
__device__ __forceinline__ void bf8(const uint4 v, float* f) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) f[2 * i] = __uint_as_float(u[i] << 16), f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
}
__global__ void __launch_bounds__(1024) side_close_kernel(const SideArgs p) {
    extern __shared__ __align__(16) float sm[];
    const SandwichArgs& a = p.s;
    const int W = a.W, dim = p.dim, tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, wid = tid >> 5, nw = nt >> 5;
    float *x = sm, *y2 = x + W, *g = y2 + W, *red = g + ((dim + 3) & ~3);
    const int r = blockIdx.x;
    const int64_t t = a.rows ? a.rows[r] : r;
    const float* y = a.y + t * W;
    float ss = 0.f;
    for (int i = tid; i < W; i += nt) {
        const float v = y[i];
        y2[i] = v, x[i] = a.x[t * W + i];
        ss = fmaf(v, v, ss);
    }
    const float rn = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
    for (int i = tid; i < W; i += nt) x[i] += y2[i] * rn * a.w[i];
    __syncthreads();
    const __nv_bfloat16* tab = p.table + (int64_t)p.ids[t] * p.ldt + p.col;
    for (int j = wid; j < dim; j += nw) {
        const __nv_bfloat16* wr = p.gate + (int64_t)j * W;
        float acc = 0.f;
        for (int k = lane; k < W; k += 32) acc = fmaf(__bfloat162float(wr[k]), x[k], acc);
        acc = warp_sum(acc);
        if (lane == 0) g[j] = gelu_tanhf_acc(acc) * __bfloat162float(tab[j]);
    }
    __syncthreads();
    ss = 0.f;
    for (int i = tid; i < W; i += nt) {
        const __nv_bfloat16* wr = p.proj + (int64_t)i * dim;
        float acc = 0.f;
        for (int j = 0; j < dim; ++j) acc = fmaf(__bfloat162float(wr[j]), g[j], acc);
        y2[i] = acc;
        ss = fmaf(acc, acc, ss);
    }
    const float r2 = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
    float sf = 0.f;
    for (int i = tid; i < W; i += nt) {
        float xn = x[i] + y2[i] * r2 * p.side_w[i];
        if (a.add_row) xn += a.add_row[t * W + i];
        if (a.add_vec) xn += a.add_vec[i];
        x[i] = xn;
        sf = fmaf(xn, xn, sf);
        if (a.x_out) a.x_out[t * W + i] = xn;
    }
    if (!a.a_out) return;
    float rf = 1.f;
    if (a.fin_w) rf = 1.0f / sqrtf(block_sum(sf, red) / (float)W + a.eps);
    for (int i = tid; i < W; i += nt) store_act(a.a_out, a.out_dtype, (int64_t)r * W + i, a.fin_w ? x[i] * rf * a.fin_w[i] : x[i]);
}

// The same with a cluster of SC_CL blocks per row, each of which streams its share of both projections: the gate's rows are dealt to the blocks (their
// results go to every block's shared memory), then every block has a slice of the model width.  W % 8 == 0 and dim % 8 == 0.
// Dynamic shared memory: x [W] | projected addition [slice] | gated [dim] | partial sums 2 x [SC_CL] | 40
constexpr int SC_CL = 8, SC_NT = 512;
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }
__host__ __device__ constexpr int side_slice(int W) { return (W + SC_CL * 8 - 1) / (SC_CL * 8) * 8; }
__global__ void __launch_bounds__(SC_NT) side_close_cluster_kernel(const SideArgs p) {
    extern __shared__ __align__(16) float sm[];
    namespace cg = cooperative_groups;
    cg::cluster_group cl = cg::this_cluster();
    const SandwichArgs& a = p.s;
    const int W = a.W, dim = p.dim, tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
    const int cr = (int)cl.block_rank(), ws = side_slice(W), w0 = cr * ws, w1 = min(W, w0 + ws);
    float *x = sm, *y2 = x + W, *g = y2 + ws, *part = g + dim, *red = part + 2 * SC_CL;
    const int r = blockIdx.x / SC_CL;
    const int64_t t = a.rows ? a.rows[r] : r;
    // the weights do not depend on what runs before: the block's share of them is on its way to L2 while the norm is computed
    const __nv_bfloat16* tab = p.table + (int64_t)p.ids[t] * p.ldt + p.col;
    for (int j = cr * (SC_NT / 32) + wid; j < dim; j += SC_CL * (SC_NT / 32)) {
        for (int k = lane * 64; k < W; k += 2048) prefetch_l2(p.gate + (int64_t)j * W + k);
        if (lane == 0) prefetch_l2(tab + j);
    }
    for (int64_t k = (int64_t)w0 * dim + tid * 64; k < (int64_t)w1 * dim; k += SC_NT * 64) prefetch_l2(p.proj + k);
    const float* y = a.y + t * W;
    float ss = 0.f;
    for (int i = tid * 4; i < W; i += SC_NT * 4) ss = sq4(ld4(y + i), ss);
    const float rn = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
    for (int i = tid * 4; i < W; i += SC_NT * 4) {
        const float4 yv = ld4(y + i), w = ld4(a.w + i);
        float4 xv = ld4(a.x + t * W + i);
        xv.x += yv.x * rn * w.x, xv.y += yv.y * rn * w.y, xv.z += yv.z * rn * w.z, xv.w += yv.w * rn * w.w;
        *reinterpret_cast<float4*>(x + i) = xv;
    }
    __syncthreads();
    cl.sync();   // every block of the cluster runs: its shared memory may be written from now on (and no block has read this row's x_out place after it changed)
    for (int j = cr * (SC_NT / 32) + wid; j < dim; j += SC_CL * (SC_NT / 32)) {
        const __nv_bfloat16* wr = p.gate + (int64_t)j * W;
        const float tv = __bfloat162float(tab[j]);
        float acc = 0.f;
#pragma unroll 8
        for (int k = lane * 8; k < W; k += 256) {
            float f[8];
            bf8(__ldg(reinterpret_cast<const uint4*>(wr + k)), f);
            const float4 u0 = ld4(x + k), u1 = ld4(x + k + 4);
            acc = fmaf(f[0], u0.x, fmaf(f[1], u0.y, fmaf(f[2], u0.z, fmaf(f[3], u0.w, acc))));
            acc = fmaf(f[4], u1.x, fmaf(f[5], u1.y, fmaf(f[6], u1.z, fmaf(f[7], u1.w, acc))));
        }
        acc = warp_sum(acc);
        const float v = gelu_tanhf_acc(acc) * tv;
        if (lane < SC_CL) cl.map_shared_rank(g, lane)[j] = v;
    }
    cl.sync();
    // eight lanes per row of the projection, four rows per lane at a time
    const int sub = lane & 7;
    ss = 0.f;
    for (int i0 = w0 + wid * 16 + (lane >> 3); i0 - (lane >> 3) < w1; i0 += SC_NT / 32 * 16) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 2
        for (int j = sub * 8; j < dim; j += 64) {
            uint4 v[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) v[q] = i0 + 4 * q < w1 ? __ldg(reinterpret_cast<const uint4*>(p.proj + (int64_t)(i0 + 4 * q) * dim + j)) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                float f[8];
                bf8(v[q], f);
#pragma unroll
                for (int u = 0; u < 8; ++u) acc[q] = fmaf(f[u], g[j + u], acc[q]);
            }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            acc[q] += __shfl_xor_sync(0xffffffffu, acc[q], 1);
            acc[q] += __shfl_xor_sync(0xffffffffu, acc[q], 2);
            acc[q] += __shfl_xor_sync(0xffffffffu, acc[q], 4);
            if (i0 + 4 * q < w1 && sub == 0) {
                y2[i0 + 4 * q - w0] = acc[q];
                ss = fmaf(acc[q], acc[q], ss);
            }
        }
    }
    ss = block_sum(ss, red);
    if (tid < SC_CL) cl.map_shared_rank(part, tid)[cr] = ss;
    cl.sync();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < SC_CL; ++i) ss += part[i];
    const float r2 = 1.0f / sqrtf(ss / (float)W + a.eps);
    float sf = 0.f;
    for (int i = w0 + tid; i < w1; i += SC_NT) {
        float xn = x[i] + y2[i - w0] * r2 * p.side_w[i];
        if (a.add_row) xn += a.add_row[t * W + i];
        if (a.add_vec) xn += a.add_vec[i];
        x[i] = xn;
        sf = fmaf(xn, xn, sf);
        if (a.x_out) a.x_out[t * W + i] = xn;
    }
    if (!a.a_out) return;
    float rf = 1.f;
    if (a.fin_w) {
        sf = block_sum(sf, red);
        if (tid < SC_CL) cl.map_shared_rank(part, tid)[SC_CL + cr] = sf;
        cl.sync();
        sf = 0.f;
#pragma unroll
        for (int i = 0; i < SC_CL; ++i) sf += part[SC_CL + i];
        rf = 1.0f / sqrtf(sf / (float)W + a.eps);
    }
    for (int i = w0 + tid; i < w1; i += SC_NT) store_act(a.a_out, a.out_dtype, (int64_t)r * W + i, a.fin_w ? x[i] * rf * a.fin_w[i] : x[i]);   // own elements only
}

}  // namespace b200seq

using namespace b200seq;

static bool act_ok(int d) { return d == B200SEQ_F32 || d == B200SEQ_BF16; }

extern "C" {

int b200seq_embed_pos(const void* table_bf16, const int32_t* ids, const b200seq_step* st, float scale, const float* freq, int W, float* x0, const float* add_vec, float* x,
                      const float* fin_w, float eps, void* a, int a_dtype, void* stream) {
    if (!table_bf16 || !ids || !st || !x || W < 1 || !act_ok(a_dtype)) return fail(B200SEQ_ERR_INVALID_ARG, "embed_pos: bad arguments");
    if (st->T == 0) return 0;
    const size_t smem = ((size_t)W + 40) * sizeof(float);
    if (smem > 200 * 1024) return fail(B200SEQ_ERR_UNSUPPORTED, "embed_pos: width %d too large", W);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(embed_pos_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return cuda_status(e, "embed_pos attribute");
    }
    const EmbedPos p{(const __nv_bfloat16*)table_bf16, ids, freq, scale, W, x0, add_vec, x, fin_w, eps, a, a_dtype,
                     W % 2 == 0 && ((reinterpret_cast<uintptr_t>(table_bf16) & 3) | (reinterpret_cast<uintptr_t>(x) & 7) | (reinterpret_cast<uintptr_t>(x0) & 7)) == 0};
    auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    if (!freq && W % 4 == 0 && W <= 8192 && (reinterpret_cast<uintptr_t>(table_bf16) & 7) == 0 && al(x0) && al(add_vec) && al(x) && al(fin_w) && al(a)) {
        const int q = W / 4, nt = q <= 64 ? 64 : (q <= 256 ? 128 : (q <= 1024 ? 256 : 512));
        const int ept = (q + nt - 1) / nt;
        if (ept <= 1) embed_reg_kernel<1><<<st->T, nt, 0, (cudaStream_t)stream>>>(p);
        else if (ept <= 2) embed_reg_kernel<2><<<st->T, nt, 0, (cudaStream_t)stream>>>(p);
        else embed_reg_kernel<4><<<st->T, nt, 0, (cudaStream_t)stream>>>(p);
        SEQ_LAUNCH_CHECK("embed_pos");
        return 0;
    }
    embed_pos_kernel<<<st->T, W >= 1024 ? 512 : 128, smem, (cudaStream_t)stream>>>(p, *st);
    SEQ_LAUNCH_CHECK("embed_pos");
    return 0;
}

int b200seq_sandwich_norm(const float* x, const float* y, const float* w, float eps, const float* add_row, const float* add_vec, int W, const int32_t* rows, int R,
                          float* x_out, void* a_out, int out_dtype, const float* fin_w, void* stream) {
    if (!x || W < 1 || R < 0 || (y && !w) || (!x_out && !a_out) || !act_ok(out_dtype)) return fail(B200SEQ_ERR_INVALID_ARG, "sandwich_norm: bad arguments");
    if (R == 0) return 0;
    const SandwichArgs a{x, y, w, eps, add_row, add_vec, W, rows, x_out, a_out, out_dtype, fin_w};
    cudaStream_t cs = (cudaStream_t)stream;
    auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (W <= 8192 && W % 4 == 0 && al(x) && al(y) && al(w) && al(add_row) && al(add_vec) && al(x_out) && al(a_out) && al(fin_w)) {
        const int q = W / 4;
        const int nt = q <= 64 ? 64 : (q <= 128 ? 128 : (q <= 512 ? 256 : 512));
        const int ept = (q + nt - 1) / nt;
        const bool pre = R <= 64;
#define SANDWICH_LAUNCH(E_)                                                    \
    do {                                                                       \
        if (pre) sandwich_norm_reg_kernel<E_, true><<<R, nt, 0, cs>>>(a);      \
        else sandwich_norm_reg_kernel<E_, false><<<R, nt, 0, cs>>>(a);         \
    } while (0)
        if (ept <= 1) SANDWICH_LAUNCH(1);
        else if (ept <= 2) SANDWICH_LAUNCH(2);
        else SANDWICH_LAUNCH(4);
#undef SANDWICH_LAUNCH
        SEQ_LAUNCH_CHECK("sandwich_norm");
        return 0;
    }
    const size_t smem = ((size_t)W + 40) * sizeof(float);
    if (smem > 200 * 1024) return fail(B200SEQ_ERR_UNSUPPORTED, "sandwich_norm: width %d too large", W);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(sandwich_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return cuda_status(e, "sandwich_norm attribute");
    }
    sandwich_norm_kernel<<<R, W >= 512 ? 512 : 128, smem, cs>>>(a);
    SEQ_LAUNCH_CHECK("sandwich_norm");
    return 0;
}

int b200seq_token_gate(const float* z, int64_t ldz, int T, int dim, const void* table_bf16, int64_t ldt, int col, const int32_t* ids, void* out, int out_dtype,
                       void* stream) {
    if (!z || !table_bf16 || !ids || !out || T < 0 || dim < 1 || col < 0 || ldz < dim || ldt < col + dim || !act_ok(out_dtype))
        return fail(B200SEQ_ERR_INVALID_ARG, "token_gate: bad arguments");
    if (T == 0) return 0;
    token_gate_kernel<<<T, dim <= 64 ? 64 : 128, 0, (cudaStream_t)stream>>>(z, ldz, dim, (const __nv_bfloat16*)table_bf16, ldt, col, ids, out, out_dtype);
    SEQ_LAUNCH_CHECK("token_gate");
    return 0;
}

int b200seq_side_close(const float* x, const float* y, const float* w, float eps, const void* gate_bf16, const void* proj_bf16, const void* table_bf16, int64_t ldt, int col,
                       int dim, const int32_t* ids, const float* side_w, const float* add_row, const float* add_vec, int W, const int32_t* rows, int R,
                       float* x_out, void* a_out, int out_dtype, const float* fin_w, void* stream) {
    if (!x || !y || !w || !gate_bf16 || !proj_bf16 || !table_bf16 || !ids || !side_w || W < 1 || R < 0 || dim < 1 || col < 0 || ldt < col + dim || (!x_out && !a_out) ||
        !act_ok(out_dtype))
        return fail(B200SEQ_ERR_INVALID_ARG, "side_close: bad arguments");
    if (R == 0) return 0;
    const size_t smem = ((size_t)2 * W + dim + 48) * sizeof(float);
    if (smem > 200 * 1024) return fail(B200SEQ_ERR_UNSUPPORTED, "side_close: width %d too large", W);
    const SideArgs p{SandwichArgs{x, y, w, eps, add_row, add_vec, W, rows, x_out, a_out, out_dtype, fin_w}, (const __nv_bfloat16*)gate_bf16,
                     (const __nv_bfloat16*)proj_bf16, (const __nv_bfloat16*)table_bf16, ldt, col, dim, ids, side_w};
    const bool vec = W % 8 == 0 && dim % 8 == 0 && ((reinterpret_cast<uintptr_t>(gate_bf16) | reinterpret_cast<uintptr_t>(proj_bf16)) & 15) == 0;
    auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    if (vec && R <= 65535 / SC_CL && al(x) && al(y) && al(w)) {
        const size_t cs = ((size_t)W + side_slice(W) + dim + 2 * SC_CL + 40) * sizeof(float);
        if (cs > 48 * 1024) {
            const cudaError_t e = cudaFuncSetAttribute(side_close_cluster_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)cs);
            if (e != cudaSuccess) return cuda_status(e, "side_close attribute");
        }
        cudaLaunchConfig_t cfg{};
        cudaLaunchAttribute at{};
        at.id = cudaLaunchAttributeClusterDimension;
        at.val.clusterDim.x = SC_CL, at.val.clusterDim.y = 1, at.val.clusterDim.z = 1;
        cfg.gridDim = dim3(R * SC_CL), cfg.blockDim = dim3(SC_NT), cfg.dynamicSmemBytes = cs, cfg.stream = (cudaStream_t)stream, cfg.attrs = &at, cfg.numAttrs = 1;
        const cudaError_t e = cudaLaunchKernelEx(&cfg, side_close_cluster_kernel, p);
        if (e != cudaSuccess) return cuda_status(e, "side_close");
        count_launch();
        return 0;
    }
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(side_close_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return cuda_status(e, "side_close attribute");
    }
    const int nt = W >= 1024 ? 1024 : (W >= 512 ? 512 : 256);
    side_close_kernel<<<R, nt, smem, (cudaStream_t)stream>>>(p);
    SEQ_LAUNCH_CHECK("side_close");
    return 0;
}

}  // extern "C"
