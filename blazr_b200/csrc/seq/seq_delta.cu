// seq_delta.cu -- delta-rule recurrence with a decay per key channel over a flat mixed batch.  Per head (key size D, value size V), with the
// state S [D][V] carried per sequence in f32, and per token r, k [D], v [V], decay w [D], removal rate a [D]:
//     u = k / sqrt(sum k^2 + unit_eps),     S_t = diag(w) S_(t-1) - (a * u) (u^T S_(t-1)) + k v^T,     o_t = S_t^T r
// followed by the division of every head's o_t by its root mean square, a weight per channel and a sigmoid gate.
// w = exp(-decay_scale * sigmoid(z + w0)) with z from a low-rank branch, a = sigmoid(az + a_b).  Everything here is f32.
//
// Steps in which every entry brings ONE token (decode): one kernel per (entry, head) -- second half of the low-rank branch, decay, removal rate,
// unit key, state update, output, unit norm, weight and gate.
// Other steps: the portions are cut into chunks of DL_C tokens (from the portion's first token) that run in parallel.  With W_i the product of the
// decays of the chunk's tokens up to i, S_i = diag(W_i) Z_i turns the recurrence into
//     Z_i = Z_(i-1) - beta_i (p_i^T Z_(i-1)) + kappa_i v_i^T,   p_i = u_i * W_(i-1),  beta_i = a_i u_i / W_i,  kappa_i = k_i / W_i,  rho_i = r_i * W_i
// so that with the removed rows y_i = p_i^T Z_(i-1) (Z_0 = S before the chunk):
//     (I + L) Y = P Z_0 + M V,   L = [p_i . beta_j]_(j < i),  M = [p_i . kappa_j]_(j < i),    O = rho Z_0 + E V - F Y,   E, F = [rho_i . kappa_j, beta_j]_(j <= i)
//   A  per chunk and head: the four score matrices, then by forward substitution P' = (I + L)^-1 P and Y0 = (I + L)^-1 M V, R' = rho - F P',
//      O0 = E V - F Y0, U = diag(W_C) (kappa^T V - beta^T Y0)
//   B  in chunk order per entry, head and value tile:  start_c = S;  S = diag(W_C) S + U - (beta W_C)^T (P' S); the last S goes to the slot
//   C  O = R' start_c + O0, unit norm, weight, gate, written in the activation type
// All ratios of decay products that enter have their later index on top, so no term grows; W_i stays above exp(-decay_scale * DL_C), far from
// the end of the f32 range.  W is a running product (not the exponential of a sum of logarithms): a ratio W_i / W_j carries the rounding
// of the steps between j and i only.
#include "seq_common.cuh"

namespace b200seq {

constexpr int DL_C = 32;     // tokens per chunk
constexpr int DL_NT = 256;
constexpr int DL_AS = DL_C + 4;   // row stride of the score matrices
constexpr int DL_VT = 16;    // value columns per block of pass B
constexpr int DL_SS = 18;    // row stride of pass B's state tile

struct DeltaArgs {
    const float* proj;
    int64_t ld;
    int r_col, k_col, v_col, g_col, a_col, w_col, rank;
    const float* wz;             // portions: [T][H * D] low-rank branch output
    int64_t ldw;
    const __nv_bfloat16* w2;     // single tokens: [H * D][rank], applied to tanh of the projection row's `rank` columns at w_col
    const float *w0, *a_b, *norm_w;
    float decay_scale, unit_eps, eps;
    int H, D, V;
    float* state;                // [slots][H][D][V]
    float* chunk;                // work area, one record per (chunk, head)
    void* out;
    int out_dtype;
};

// record of one (chunk, head): P' [C][Dp] | beta W_C [C][Dp] | R' [C][Dp] | W_C [Dp] | U, then the start state [Dp][Vp] | O0 [C][Vp]
struct DeltaRec {
    int Dp, Vp;
    __host__ __device__ DeltaRec(int D, int V) : Dp((D + 3) & ~3), Vp((V + 3) & ~3) {}
    __host__ __device__ int64_t p() const { return 0; }
    __host__ __device__ int64_t b() const { return (int64_t)DL_C * Dp; }
    __host__ __device__ int64_t r() const { return (int64_t)2 * DL_C * Dp; }
    __host__ __device__ int64_t w() const { return (int64_t)3 * DL_C * Dp; }
    __host__ __device__ int64_t u() const { return w() + Dp; }
    __host__ __device__ int64_t o() const { return u() + (int64_t)Dp * Vp; }
    __host__ __device__ int64_t size() const { return o() + (int64_t)DL_C * Vp; }
};

__device__ __forceinline__ float delta_decay(float z, float scale) { return expf(-scale * sigmoidf_acc(z)); }

// ---- decode: grid (B, H) ----------------------------------------------------------------------------------------------------------------
// thread = (value column of a tile of 64, one of 4 groups of key channels); EPT: state elements a thread keeps in registers (D <= 4 * EPT), 0: any D,
// the state is read twice.  Dynamic shared memory: u | a u | k | r | w [D each] | tanh [rank] | partial sums 2 x [4][64] | o [V] | 40
template <int EPT>
__global__ void __launch_bounds__(DL_NT) delta_step_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int D = a.D, V = a.V, H = a.H;
    float *us = sm, *bs = us + D, *ks = bs + D, *rs = ks + D, *ws = rs + D, *tw = ws + D;
    float *py = tw + a.rank, *po = py + 256, *os = po + 256, *red = os + V;
    const int e = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int t = st.ent_start[e];
    const float* row = a.proj + (int64_t)t * a.ld;
    float* S = a.state + ((int64_t)st.ent_slot[e] * H + h) * D * V;
    const bool fresh = st.ent_pos0[e] == 0;
    const int vt = tid & 63, dg = tid >> 6;
    constexpr int NE = EPT > 0 ? EPT : 1;
    float s[NE];
    if (EPT > 0) {   // the first value tile's state is requested before anything is waited for
#pragma unroll
        for (int j = 0; j < NE; ++j) {
            const int d = dg + 4 * j;
            s[j] = (!fresh && d < D && vt < V) ? S[(int64_t)d * V + vt] : 0.f;
        }
    }
    for (int i = tid; i < a.rank; i += DL_NT) tw[i] = tanhf(row[a.w_col + i]);
    float ss = 0.f;
    for (int d = tid; d < D; d += DL_NT) {
        const float k = row[a.k_col + h * D + d];
        ks[d] = k, rs[d] = row[a.r_col + h * D + d];
        ss = fmaf(k, k, ss);
    }
    const float uinv = 1.0f / sqrtf(block_sum(ss, red) + a.unit_eps);   // its barriers also publish ks, rs, tw
    for (int d0 = 0; d0 < D; d0 += 64) {
        const int d = d0 + (tid >> 2), sub = tid & 3;
        float z = 0.f;
        if (d < D) {
            const __nv_bfloat16* w2 = a.w2 + (int64_t)(h * D + d) * a.rank;
            for (int i = sub; i < a.rank; i += 4) z = fmaf(__bfloat162float(w2[i]), tw[i], z);
        }
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        z += __shfl_xor_sync(0xffffffffu, z, 2);
        if (sub == 0 && d < D) {
            const int c = h * D + d;
            const float u = ks[d] * uinv;
            us[d] = u;
            bs[d] = sigmoidf_acc(row[a.a_col + c] + a.a_b[c]) * u;
            ws[d] = delta_decay(z + a.w0[c], a.decay_scale);
        }
    }
    __syncthreads();
    for (int v0 = 0; v0 < V; v0 += 64) {
        const int v = v0 + vt;
        const bool in = v < V;
        float y = 0.f;
        if (EPT > 0) {
            if (v0 > 0) {
#pragma unroll
                for (int j = 0; j < NE; ++j) {
                    const int d = dg + 4 * j;
                    s[j] = (!fresh && d < D && in) ? S[(int64_t)d * V + v] : 0.f;
                }
            }
#pragma unroll
            for (int j = 0; j < NE; ++j)
                if (dg + 4 * j < D) y = fmaf(us[dg + 4 * j], s[j], y);
        } else if (in && !fresh) {
            for (int d = dg; d < D; d += 4) y = fmaf(us[d], S[(int64_t)d * V + v], y);
        }
        py[dg * 64 + vt] = y;
        __syncthreads();
        y = (py[vt] + py[64 + vt]) + (py[128 + vt] + py[192 + vt]);
        float o = 0.f;
        if (in) {
            const float vv = row[a.v_col + h * V + v];
            if (EPT > 0) {
#pragma unroll
                for (int j = 0; j < NE; ++j) {
                    const int d = dg + 4 * j;
                    if (d < D) {
                        const float n = fmaf(ks[d], vv, fmaf(-bs[d], y, ws[d] * s[j]));
                        S[(int64_t)d * V + v] = n;
                        o = fmaf(rs[d], n, o);
                    }
                }
            } else {
                for (int d = dg; d < D; d += 4) {
                    const float old = fresh ? 0.f : S[(int64_t)d * V + v];
                    const float n = fmaf(ks[d], vv, fmaf(-bs[d], y, ws[d] * old));
                    S[(int64_t)d * V + v] = n;
                    o = fmaf(rs[d], n, o);
                }
            }
        }
        po[dg * 64 + vt] = o;
        __syncthreads();   // also: every thread is done with py before the next tile rewrites it
        if (dg == 0 && in) os[v] = (po[vt] + po[64 + vt]) + (po[128 + vt] + po[192 + vt]);
    }
    __syncthreads();
    float sq = 0.f;
    for (int v = tid; v < V; v += DL_NT) sq = fmaf(os[v], os[v], sq);
    const float rinv = 1.0f / sqrtf(block_sum(sq, red) / (float)V + a.eps);
    for (int v = tid; v < V; v += DL_NT) {
        const int c = h * V + v;
        store_act(a.out, a.out_dtype, (int64_t)t * H * V + c, os[v] * rinv * a.norm_w[c] * sigmoidf_acc(row[a.g_col + c]));
    }
}

// ---- pass A: grid (chunks, H) -----------------------------------------------------------------------------------------------------------
// Dynamic shared memory: P | R | B | K [C][Ds] (B and K next to each other: one operand of 2 C rows; P and R likewise) | four transposed score
// matrices [C (j)][AS] | decays [C][Ds] in the same place as V and Y tiles 2 x [C][68] | products of the decays per segment [4][Dp] | W_C [Dp]
__host__ __device__ inline int delta_ds(int D) { return ((D + 3) & ~3) + 4; }
__host__ __device__ inline int delta_local_floats(int D) {
    const int Ds = delta_ds(D), Dp = (D + 3) & ~3;
    const int wd = DL_C * Ds, vy = 2 * DL_C * 68;
    return 4 * DL_C * Ds + 4 * DL_C * DL_AS + (wd > vy ? wd : vy) + 5 * Dp;
}

__global__ void __launch_bounds__(DL_NT, 2) delta_local_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int D = a.D, V = a.V, H = a.H, Ds = delta_ds(D), Dp = (D + 3) & ~3;
    float *P = sm, *R = P + DL_C * Ds, *B = R + DL_C * Ds, *K = B + DL_C * Ds;
    float *AL = K + DL_C * Ds, *AM = AL + DL_C * DL_AS, *AF = AM + DL_C * DL_AS, *AE = AF + DL_C * DL_AS;
    float* Wd = AE + DL_C * DL_AS;
    float *Vs = Wd, *Ys = Wd + DL_C * 68;
    const int wd = DL_C * Ds, vy = 2 * DL_C * 68;
    float* segp = Wd + (wd > vy ? wd : vy);
    float* wc = segp + 4 * Dp;
    const int c = blockIdx.x, h = blockIdx.y;
    int e, row0, len;
    if (!find_chunk(st, c, DL_C, e, row0, len)) return;
    const DeltaRec rec(D, V);
    float* out = a.chunk + ((int64_t)c * H + h) * rec.size();
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
    // the tokens' rows: a warp takes four tokens
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const int i = wid * 4 + q;
        const bool in = i < len;
        const float* row = a.proj + (int64_t)(row0 + i) * a.ld;
        float ss = 0.f;
        for (int d = lane; d < Dp; d += 32) {
            float k = 0.f, r = 0.f, av = 0.f, w = 1.f;
            if (in && d < D) {
                const int cc = h * D + d;
                k = row[a.k_col + cc], r = row[a.r_col + cc];
                av = sigmoidf_acc(row[a.a_col + cc] + a.a_b[cc]);
                w = delta_decay(a.wz[(int64_t)(row0 + i) * a.ldw + cc] + a.w0[cc], a.decay_scale);
            }
            ss = fmaf(k, k, ss);
            K[i * Ds + d] = k, R[i * Ds + d] = r, B[i * Ds + d] = av, Wd[i * Ds + d] = w;
        }
        const float uinv = 1.0f / sqrtf(warp_sum(ss) + a.unit_eps);
        for (int d = lane; d < Dp; d += 32) {
            const float u = K[i * Ds + d] * uinv;
            P[i * Ds + d] = u, B[i * Ds + d] *= u;
        }
    }
    __syncthreads();
    // running products of the decays: four segments of eight tokens per channel
    for (int it = tid; it < 4 * Dp; it += DL_NT) {
        const int sg = it / Dp, d = it - sg * Dp;
        float p = 1.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) p *= Wd[(sg * 8 + i) * Ds + d];
        segp[it] = p;
    }
    __syncthreads();
    for (int it = tid; it < 4 * Dp; it += DL_NT) {
        const int sg = it / Dp, d = it - sg * Dp;
        float W = 1.f;
        for (int s = 0; s < sg; ++s) W *= segp[s * Dp + d];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int o = (sg * 8 + i) * Ds + d;
            P[o] *= W;
            W *= Wd[o];
            const float inv = 1.0f / W;
            R[o] *= W, B[o] *= inv, K[o] *= inv;
        }
        if (sg == 3) {
            wc[d] = W;
            out[rec.w() + d] = W;
        }
    }
    __syncthreads();
    // scores: rows p_0 .. p_31, rho_0 .. rho_31 against beta_0 .. , kappa_0 ..; thread (ty, tx): rows ty * 4 + i, columns tx + 16 j
    {
        const int tx = tid & 15, ty = tid >> 4;
        float s[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
        for (int d = 0; d < Dp; d += 4) {
            float4 q[4], k[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) q[i] = *reinterpret_cast<const float4*>(P + (ty * 4 + i) * Ds + d);
#pragma unroll
            for (int j = 0; j < 4; ++j) k[j] = *reinterpret_cast<const float4*>(B + (tx + 16 * j) * Ds + d);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    s[i][j] = fmaf(q[i].x, k[j].x, s[i][j]), s[i][j] = fmaf(q[i].y, k[j].y, s[i][j]);
                    s[i][j] = fmaf(q[i].z, k[j].z, s[i][j]), s[i][j] = fmaf(q[i].w, k[j].w, s[i][j]);
                }
        }
        const bool isp = ty < 8;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int ri = (ty & 7) * 4 + i;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int cj = tx + 16 * (j & 1);
                float* m = isp ? (j < 2 ? AL : AM) : (j < 2 ? AF : AE);
                m[cj * DL_AS + ri] = (isp ? cj < ri : cj <= ri) ? s[i][j] : 0.f;
            }
        }
    }
    __syncthreads();
    // value tiles of 64 columns: Y0 and O0 (one column per thread), then U
    for (int v0 = 0; v0 < V; v0 += 64) {
        __syncthreads();   // the decays (first tile) or the previous tile are done with
        for (int it = tid; it < DL_C * 64; it += DL_NT) {
            const int i = it >> 6, cc = it & 63;
            Vs[i * 68 + cc] = (i < len && v0 + cc < V) ? a.proj[(int64_t)(row0 + i) * a.ld + a.v_col + (int64_t)h * V + v0 + cc] : 0.f;
        }
        __syncthreads();
        if (v0 == 0 && tid < Dp) {   // P' and R', one column (key channel) per thread (D <= the block's threads)
            const int d = tid;
            float x[DL_C], r[DL_C];
    #pragma unroll
            for (int i = 0; i < DL_C; ++i) x[i] = P[i * Ds + d], r[i] = R[i * Ds + d];
    #pragma unroll
            for (int j = 0; j < DL_C; ++j) {
                const float y = x[j];
    #pragma unroll
                for (int i4 = j & ~3; i4 < DL_C; i4 += 4) {
                    const float4 l = *reinterpret_cast<const float4*>(AL + j * DL_AS + i4), f = *reinterpret_cast<const float4*>(AF + j * DL_AS + i4);
                    x[i4] = fmaf(-l.x, y, x[i4]), x[i4 + 1] = fmaf(-l.y, y, x[i4 + 1]), x[i4 + 2] = fmaf(-l.z, y, x[i4 + 2]), x[i4 + 3] = fmaf(-l.w, y, x[i4 + 3]);
                    r[i4] = fmaf(-f.x, y, r[i4]), r[i4 + 1] = fmaf(-f.y, y, r[i4 + 1]), r[i4 + 2] = fmaf(-f.z, y, r[i4 + 2]), r[i4 + 3] = fmaf(-f.w, y, r[i4 + 3]);
                }
            }
    #pragma unroll
            for (int i = 0; i < DL_C; ++i) {
                out[rec.p() + (int64_t)i * Dp + d] = x[i];
                out[rec.r() + (int64_t)i * Dp + d] = r[i];
            }
        }
        // Y0 and O0, one value column per thread: the block's last two warps, beside the P' columns of its first ones
        if (tid >= DL_NT - 64) {
            const int cc = tid - (DL_NT - 64);
            float x[DL_C], o[DL_C];
#pragma unroll
            for (int i = 0; i < DL_C; ++i) x[i] = 0.f, o[i] = 0.f;
#pragma unroll
            for (int j = 0; j < DL_C; ++j) {
                const float y = x[j], vv = Vs[j * 68 + cc];
#pragma unroll
                for (int i4 = j & ~3; i4 < DL_C; i4 += 4) {
                    const float4 l = *reinterpret_cast<const float4*>(AL + j * DL_AS + i4), m = *reinterpret_cast<const float4*>(AM + j * DL_AS + i4);
                    const float4 f = *reinterpret_cast<const float4*>(AF + j * DL_AS + i4), g = *reinterpret_cast<const float4*>(AE + j * DL_AS + i4);
                    x[i4] = fmaf(m.x, vv, fmaf(-l.x, y, x[i4])), x[i4 + 1] = fmaf(m.y, vv, fmaf(-l.y, y, x[i4 + 1]));
                    x[i4 + 2] = fmaf(m.z, vv, fmaf(-l.z, y, x[i4 + 2])), x[i4 + 3] = fmaf(m.w, vv, fmaf(-l.w, y, x[i4 + 3]));
                    o[i4] = fmaf(g.x, vv, fmaf(-f.x, y, o[i4])), o[i4 + 1] = fmaf(g.y, vv, fmaf(-f.y, y, o[i4 + 1]));
                    o[i4 + 2] = fmaf(g.z, vv, fmaf(-f.z, y, o[i4 + 2])), o[i4 + 3] = fmaf(g.w, vv, fmaf(-f.w, y, o[i4 + 3]));
                }
            }
            const bool in = v0 + cc < rec.Vp;
#pragma unroll
            for (int i = 0; i < DL_C; ++i) {
                Ys[i * 68 + cc] = x[i];
                if (in) out[rec.o() + (int64_t)i * rec.Vp + v0 + cc] = o[i];
            }
        }
        for (int it = v0 == 0 ? tid : DL_C * Dp; it < DL_C * Dp; it += DL_NT) {
            const int i = it / Dp, d = it - i * Dp;
            out[rec.b() + it] = B[i * Ds + d] * wc[d];
        }
        __syncthreads();
        const int tx = tid & 15, ty = tid >> 4;
        for (int d0 = 0; d0 < Dp; d0 += 64) {
            const int d = d0 + ty * 4;
            if (d >= Dp) break;
            float acc[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) acc[i][u] = 0.f;
#pragma unroll 4
            for (int j = 0; j < DL_C; ++j) {
                const float4 k = *reinterpret_cast<const float4*>(K + j * Ds + d), b = *reinterpret_cast<const float4*>(B + j * Ds + d);
                const float4 v = *reinterpret_cast<const float4*>(Vs + j * 68 + tx * 4), y = *reinterpret_cast<const float4*>(Ys + j * 68 + tx * 4);
                const float kk[4] = {k.x, k.y, k.z, k.w}, bb[4] = {b.x, b.y, b.z, b.w}, vv[4] = {v.x, v.y, v.z, v.w}, yy[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int u = 0; u < 4; ++u) acc[i][u] = fmaf(kk[i], vv[u], fmaf(-bb[i], yy[u], acc[i][u]));
            }
            if (v0 + tx * 4 < rec.Vp) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float w = wc[d + i];
                    *reinterpret_cast<float4*>(out + rec.u() + (int64_t)(d + i) * rec.Vp + v0 + tx * 4) = make_float4(acc[i][0] * w, acc[i][1] * w, acc[i][2] * w, acc[i][3] * w);
                }
            }
        }
    }
}

// ---- pass B: grid (value tiles of DL_VT, H, B) -------------------------------------------------------------------------------------------
// Dynamic shared memory: S [Dp][DL_SS] | two stages of (P' [C][Ds] | beta W_C [C][Ds] | W_C [Dp]) | Y [C][20]
__host__ __device__ inline int delta_scan_floats(int D) {
    const int Ds = delta_ds(D), Dp = (D + 3) & ~3;
    return ((Dp * DL_SS + 3) & ~3) + 2 * (2 * DL_C * Ds + Dp) + DL_C * 20;
}

__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(src));
}

template <int NU>   // key channels per thread row group: D <= 64 * NU
__global__ void __launch_bounds__(DL_NT) delta_scan_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int D = a.D, V = a.V, H = a.H, Ds = delta_ds(D), Dp = (D + 3) & ~3;
    const DeltaRec rec(D, V);
    const int stage = 2 * DL_C * Ds + Dp;
    float* S = sm;
    float* buf = S + ((Dp * DL_SS + 3) & ~3);
    float* Y = buf + 2 * stage;
    const int v0 = blockIdx.x * DL_VT, h = blockIdx.y, e = blockIdx.z, tid = threadIdx.x;
    int c0 = 0;
    for (int i = 0; i < e; ++i) c0 += (st.ent_start[i + 1] - st.ent_start[i] + DL_C - 1) / DL_C;
    const int nc = (st.ent_start[e + 1] - st.ent_start[e] + DL_C - 1) / DL_C;
    if (nc == 0) return;
    float* slot = a.state + ((int64_t)st.ent_slot[e] * H + h) * D * V;
    const bool fresh = st.ent_pos0[e] == 0;
    for (int it = tid; it < Dp * DL_VT; it += DL_NT) {
        const int d = it / DL_VT, cc = it - d * DL_VT;
        S[d * DL_SS + cc] = (!fresh && d < D && v0 + cc < V) ? slot[(int64_t)d * V + v0 + cc] : 0.f;
    }
    auto fetch = [&](int c, int s) {
        const float* g = a.chunk + ((int64_t)(c0 + c) * H + h) * rec.size();
        float* b = buf + s * stage;
        const int q = Dp >> 2;
        for (int it = tid; it < 2 * DL_C * q; it += DL_NT) {   // P' rows, then beta W_C rows: adjacent in the record
            const int i = it / q, d4 = it - i * q;
            cp_async16(b + i * Ds + 4 * d4, g + (int64_t)i * Dp + 4 * d4);
        }
        for (int it = tid; it < q; it += DL_NT) cp_async16(b + 2 * DL_C * Ds + 4 * it, g + rec.w() + 4 * it);
        asm volatile("cp.async.commit_group;\n");
    };
    // this thread's part of the update: channels dgr * 4 + kq (+ 64 per step), value columns vg * 4 .. + 3
    const int kq = tid & 3, rest = tid >> 2, dgr = rest >> 2, vg = rest & 3;
    const int rg = rest >> 3, cg = rest & 7;
    const bool vin = v0 + vg * 4 < rec.Vp;
    float4 un[NU];
    auto load_u = [&](int c) {
        const float* g = a.chunk + ((int64_t)(c0 + c) * H + h) * rec.size() + rec.u() + v0 + vg * 4;
#pragma unroll
        for (int n = 0; n < NU; ++n) {
            const int d = n * 64 + dgr * 4 + kq;
            un[n] = (vin && d < Dp) ? *reinterpret_cast<const float4*>(g + (int64_t)d * rec.Vp) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    fetch(0, 0);
    load_u(0);
    for (int c = 0; c < nc; ++c) {
        float4 uc[NU];
#pragma unroll
        for (int n = 0; n < NU; ++n) uc[n] = un[n];
        if (c + 1 < nc) {
            fetch(c + 1, (c + 1) & 1);
            load_u(c + 1);
            asm volatile("cp.async.wait_group 1;\n");
        } else {
            asm volatile("cp.async.wait_group 0;\n");
        }
        __syncthreads();   // stage c is in place, S is the state in front of chunk c
        const float* Pm = buf + (c & 1) * stage;
        const float* Bm = Pm + DL_C * Ds;
        const float* wc = Bm + DL_C * Ds;
        {   // Y = P' S: rows rg * 4 + i, columns cg * 2 + u, key channels dealt to the four lanes kq
            float acc[4][2];
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0.f;
            for (int d = kq * 4; d < Dp; d += 16) {
                float4 p[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) p[i] = *reinterpret_cast<const float4*>(Pm + (rg * 4 + i) * Ds + d);
#pragma unroll
                for (int dd = 0; dd < 4; ++dd) {
                    const float2 s = *reinterpret_cast<const float2*>(S + (d + dd) * DL_SS + cg * 2);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float pv = dd == 0 ? p[i].x : dd == 1 ? p[i].y : dd == 2 ? p[i].z : p[i].w;
                        acc[i][0] = fmaf(pv, s.x, acc[i][0]), acc[i][1] = fmaf(pv, s.y, acc[i][1]);
                    }
                }
            }
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    acc[i][u] += __shfl_xor_sync(0xffffffffu, acc[i][u], 1);
                    acc[i][u] += __shfl_xor_sync(0xffffffffu, acc[i][u], 2);
                }
                if (kq == i) y0 = acc[i][0], y1 = acc[i][1];
            }
            *reinterpret_cast<float2*>(Y + (rg * 4 + kq) * 20 + cg * 2) = make_float2(y0, y1);
        }
        __syncthreads();
        float* gz = a.chunk + ((int64_t)(c0 + c) * H + h) * rec.size() + rec.u() + v0 + vg * 4;
#pragma unroll
        for (int n = 0; n < NU; ++n) {   // S = W_C S + U - (beta W_C)^T Y; the old S takes U's place in the record
            const int db = n * 64 + dgr * 4;
            const bool dok = db < Dp;    // Dp is a multiple of 4: all four channels or none (the same for the four lanes kq)
            float acc[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) acc[i][u] = 0.f;
            if (dok) {
#pragma unroll
                for (int j = kq; j < DL_C; j += 4) {
                    const float4 b = *reinterpret_cast<const float4*>(Bm + j * Ds + db), y = *reinterpret_cast<const float4*>(Y + j * 20 + vg * 4);
                    const float bb[4] = {b.x, b.y, b.z, b.w}, yy[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i)
#pragma unroll
                        for (int u = 0; u < 4; ++u) acc[i][u] = fmaf(bb[i], yy[u], acc[i][u]);
                }
            }
            // sum over the four lanes; lane kq keeps channel kq of the group
            float m[2][4], f[4];
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const float send = (kq & 2) ? acc[i][u] : acc[i + 2][u], mine = (kq & 2) ? acc[i + 2][u] : acc[i][u];
                    m[i][u] = mine + __shfl_xor_sync(0xffffffffu, send, 2);
                }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float send = (kq & 1) ? m[0][u] : m[1][u], mine = (kq & 1) ? m[1][u] : m[0][u];
                f[u] = mine + __shfl_xor_sync(0xffffffffu, send, 1);
            }
            if (dok) {
                const int d = db + kq;
                float2* sp = reinterpret_cast<float2*>(S + d * DL_SS + vg * 4);
                const float2 s0 = sp[0], s1 = sp[1];
                if (vin) *reinterpret_cast<float4*>(gz + (int64_t)d * rec.Vp) = make_float4(s0.x, s0.y, s1.x, s1.y);
                const float w = wc[d];
                sp[0] = make_float2(fmaf(w, s0.x, uc[n].x - f[0]), fmaf(w, s0.y, uc[n].y - f[1]));
                sp[1] = make_float2(fmaf(w, s1.x, uc[n].z - f[2]), fmaf(w, s1.y, uc[n].w - f[3]));
            }
        }
        __syncthreads();   // S is complete; the stage of chunk c may be refilled
    }
    for (int it = tid; it < D * DL_VT; it += DL_NT) {
        const int d = it / DL_VT, cc = it - d * DL_VT;
        if (v0 + cc < V) slot[(int64_t)d * V + v0 + cc] = S[d * DL_SS + cc];
    }
}

// ---- pass C: grid (chunks, H), 128 threads; thread (ty, tx): tokens ty * 4 + i, value columns tx * 4 + u of a tile of 64 --------------------
// Dynamic shared memory: R' [C][Ds] | slab of the start state [32][68] | o [C][Vp + 4]
constexpr int DL_NC = 128;
__host__ __device__ inline int delta_out_floats(int D, int V) { return DL_C * delta_ds(D) + 32 * 68 + DL_C * (((V + 3) & ~3) + 4); }

__global__ void __launch_bounds__(DL_NC) delta_out_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int D = a.D, V = a.V, H = a.H, Ds = delta_ds(D), Dp = (D + 3) & ~3;
    const DeltaRec rec(D, V);
    const int Os = rec.Vp + 4;
    float *R = sm, *Z = R + DL_C * Ds, *O = Z + 32 * 68;
    const int c = blockIdx.x, h = blockIdx.y;
    int e, row0, len;
    if (!find_chunk(st, c, DL_C, e, row0, len)) return;
    const float* g = a.chunk + ((int64_t)c * H + h) * rec.size();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int q = Dp >> 2;
    for (int it = tid; it < DL_C * q; it += DL_NC) {
        const int i = it / q, d4 = it - i * q;
        *reinterpret_cast<float4*>(R + i * Ds + 4 * d4) = *reinterpret_cast<const float4*>(g + rec.r() + (int64_t)i * Dp + 4 * d4);
    }
    for (int v0 = 0; v0 < V; v0 += 64) {
        float acc[4][4];
        const bool vin = v0 + tx * 4 < rec.Vp;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float4 o = vin ? *reinterpret_cast<const float4*>(g + rec.o() + (int64_t)(ty * 4 + i) * rec.Vp + v0 + tx * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            acc[i][0] = o.x, acc[i][1] = o.y, acc[i][2] = o.z, acc[i][3] = o.w;
        }
        for (int d0 = 0; d0 < Dp; d0 += 32) {
            __syncthreads();
            for (int it = tid; it < 32 * 16; it += DL_NC) {
                const int dd = it >> 4, c4 = it & 15;
                *reinterpret_cast<float4*>(Z + dd * 68 + 4 * c4) = (d0 + dd < Dp && v0 + 4 * c4 < rec.Vp)
                    ? *reinterpret_cast<const float4*>(g + rec.u() + (int64_t)(d0 + dd) * rec.Vp + v0 + 4 * c4) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
            __syncthreads();
            const int dn = min(32, Dp - d0);
            for (int dd = 0; dd < dn; dd += 4) {
                float4 r[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) r[i] = *reinterpret_cast<const float4*>(R + (ty * 4 + i) * Ds + d0 + dd);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const float4 z = *reinterpret_cast<const float4*>(Z + (dd + k) * 68 + tx * 4);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float rv = k == 0 ? r[i].x : k == 1 ? r[i].y : k == 2 ? r[i].z : r[i].w;
                        acc[i][0] = fmaf(rv, z.x, acc[i][0]), acc[i][1] = fmaf(rv, z.y, acc[i][1]);
                        acc[i][2] = fmaf(rv, z.z, acc[i][2]), acc[i][3] = fmaf(rv, z.w, acc[i][3]);
                    }
                }
            }
        }
        if (vin) {
#pragma unroll
            for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(O + (ty * 4 + i) * Os + v0 + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        }
    }
    __syncthreads();
    const int lane = tid & 31, wid = tid >> 5;
    for (int i = wid; i < len; i += DL_NC / 32) {
        const float* o = O + i * Os;
        float ss = 0.f;
        for (int v = lane; v < V; v += 32) ss = fmaf(o[v], o[v], ss);
        const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)V + a.eps);
        const int64_t t = row0 + i;
        const float* gate = a.proj + t * a.ld + a.g_col + (int64_t)h * V;
        const float* nw = a.norm_w + (int64_t)h * V;
        for (int v = lane; v < V; v += 32) store_act(a.out, a.out_dtype, (t * H + h) * V + v, o[v] * rinv * nw[v] * sigmoidf_acc(gate[v]));
    }
}

}  // namespace b200seq

using namespace b200seq;

extern "C" size_t b200seq_delta_scratch_floats(int T, int B, int H, int D, int V) {
    if (T < 1 || B < 1 || T == B) return 0;
    const size_t chunks = (size_t)(T + DL_C - 1) / DL_C + (size_t)B;
    return chunks * H * (size_t)DeltaRec(D, V).size();
}

extern "C" int b200seq_delta(const float* proj, int64_t ld, const b200seq_step* st, const b200seq_delta_desc* d, const float* wz, int64_t ldw, float* state, void* out,
                             int out_dtype, float* scratch, size_t scratch_floats, void* stream) {
    if (!proj || !st || !d || !state || !out || d->H < 1 || d->D < 1 || d->V < 1 || d->r_col < 0 || d->k_col < 0 || d->v_col < 0 || d->g_col < 0 || d->a_col < 0 ||
        d->w_col < 0 || d->rank < 1 || !d->w2 || !d->w0 || !d->a_b || !d->norm_w)
        return fail(B200SEQ_ERR_INVALID_ARG, "delta: bad arguments");
    if (out_dtype != B200SEQ_F32 && out_dtype != B200SEQ_BF16) return fail(B200SEQ_ERR_INVALID_ARG, "delta: output dtype");
    if (!(d->decay_scale >= 0.f) || d->decay_scale * DL_C > 60.f)   // products of a chunk's decays stay inside the f32 range
        return fail(B200SEQ_ERR_UNSUPPORTED, "delta: decay scale outside [0, %.2f]", 60.0 / DL_C);
    if (st->T == 0 || st->B == 0) return 0;
    if (st->B > 65535 || d->H > 65535) return fail(B200SEQ_ERR_UNSUPPORTED, "delta: too many entries or heads");
    cudaStream_t cs = (cudaStream_t)stream;
    DeltaArgs a{proj, ld, d->r_col, d->k_col, d->v_col, d->g_col, d->a_col, d->w_col, d->rank, wz, ldw, (const __nv_bfloat16*)d->w2, d->w0, d->a_b, d->norm_w,
                d->decay_scale, d->unit_eps, d->eps, d->H, d->D, d->V, state, scratch, out, out_dtype};
    if (st->T == st->B) {
        const size_t smem = ((size_t)5 * d->D + d->rank + 512 + d->V + 40) * sizeof(float);
        if (smem > 48 * 1024) return fail(B200SEQ_ERR_UNSUPPORTED, "delta: head sizes too large");
        const dim3 grid(st->B, d->H);
        if (d->D <= 32) delta_step_kernel<8><<<grid, DL_NT, smem, cs>>>(a, *st);
        else if (d->D <= 64) delta_step_kernel<16><<<grid, DL_NT, smem, cs>>>(a, *st);
        else if (d->D <= 128) delta_step_kernel<32><<<grid, DL_NT, smem, cs>>>(a, *st);
        else delta_step_kernel<0><<<grid, DL_NT, smem, cs>>>(a, *st);
        SEQ_LAUNCH_CHECK("delta step");
        return 0;
    }
    const size_t need = b200seq_delta_scratch_floats(st->T, st->B, d->H, d->D, d->V);
    if (!wz || ldw < (int64_t)d->H * d->D) return fail(B200SEQ_ERR_INVALID_ARG, "delta: a step of portions needs the low-rank branch's rows");
    if (!scratch || scratch_floats < need || (reinterpret_cast<uintptr_t>(scratch) & 15)) return fail(B200SEQ_ERR_INVALID_ARG, "delta: a step of portions needs %zu floats of 16-byte aligned work area", need);
    const int chunks = (st->T + DL_C - 1) / DL_C + st->B;   // upper bound of the step's chunk count
    const size_t sa = (size_t)delta_local_floats(d->D) * sizeof(float), sb = (size_t)delta_scan_floats(d->D) * sizeof(float), sc = (size_t)delta_out_floats(d->D, d->V) * sizeof(float);
    if (d->D > 256 || sa > 220 * 1024 || sb > 220 * 1024 || sc > 220 * 1024) return fail(B200SEQ_ERR_UNSUPPORTED, "delta: head sizes too large");
    cudaError_t err = cudaSuccess;
    static size_t set_a = 48 * 1024, set_c = 48 * 1024;
    if (sa > set_a) err = cudaFuncSetAttribute(delta_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sa), set_a = sa;
    if (err == cudaSuccess && sc > set_c) err = cudaFuncSetAttribute(delta_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sc), set_c = sc;
    if (err != cudaSuccess) return cuda_status(err, "delta attribute");
    delta_local_kernel<<<dim3(chunks, d->H), DL_NT, sa, cs>>>(a, *st);
    SEQ_LAUNCH_CHECK("delta local pass");
    const dim3 gb((d->V + DL_VT - 1) / DL_VT, d->H, st->B);
#define DELTA_SCAN(NU_)                                                                                                          \
    do {                                                                                                                         \
        static size_t set_ = 48 * 1024;                                                                                          \
        if (sb > set_) err = cudaFuncSetAttribute(delta_scan_kernel<NU_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sb), set_ = sb; \
        if (err == cudaSuccess) delta_scan_kernel<NU_><<<gb, DL_NT, sb, cs>>>(a, *st);                                           \
    } while (0)
    if (d->D <= 64) DELTA_SCAN(1);
    else if (d->D <= 128) DELTA_SCAN(2);
    else DELTA_SCAN(4);
#undef DELTA_SCAN
    if (err != cudaSuccess) return cuda_status(err, "delta attribute");
    SEQ_LAUNCH_CHECK("delta scan pass");
    delta_out_kernel<<<dim3(chunks, d->H), DL_NC, sc, cs>>>(a, *st);
    SEQ_LAUNCH_CHECK("delta output pass");
    return 0;
}
