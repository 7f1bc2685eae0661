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
constexpr int DL_AS = DL_C + 4;       // row stride of a 32 x 32 matrix
constexpr int DL_MS = 2 * DL_C + 4;   // row stride of two of them side by side
constexpr int DL_VS = 68;             // row stride of a tile of 64 value columns

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

// record of one (chunk, head): P' [C][Ds] | beta W_C [C][Ds] | W_C [Dp] | R' [C][Ds] | U, then the start state [Dp][Vp] | O0 [C][Vp].  Rows of key
// channels keep the row stride they have in shared memory, so that a block copies them as they lie.
__host__ __device__ constexpr int delta_up4(int n) { return (n + 3) & ~3; }
__host__ __device__ constexpr int delta_ds(int D) { return delta_up4(D) + 4; }
struct DeltaRec {
    int Ds, Dp, Vp;
    __host__ __device__ constexpr DeltaRec(int D, int V) : Ds(delta_ds(D)), Dp(delta_up4(D)), Vp(delta_up4(V)) {}
    __host__ __device__ constexpr int b() const { return DL_C * Ds; }
    __host__ __device__ constexpr int w() const { return 2 * DL_C * Ds; }
    __host__ __device__ constexpr int r() const { return w() + Dp; }
    __host__ __device__ constexpr int u() const { return r() + DL_C * Ds; }
    __host__ __device__ constexpr int o() const { return u() + Dp * Vp; }
    __host__ __device__ constexpr int size() const { return o() + DL_C * Vp; }
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

// The passes are compiled for D = V = TD (64, 128) and in a general form (TD = 0).
// ---- pass A: grid (chunks, H) -----------------------------------------------------------------------------------------------------------
// Dynamic shared memory: P | R | B | K [C][Ds] (P and R, B and K next to each other: operands of 2 C rows) | T: L transposed, then (I + L)^-1
// transposed [C][AS] | F transposed [C][AS] | M | E transposed [C][MS] | decays [C][Ds] in the same place as V and Y tiles 2 x [C][VS] |
// products of the decays per segment [4][Dp] | W_C [Dp]
__host__ __device__ constexpr int delta_local_floats(int D) {
    const int wd = DL_C * delta_ds(D), vy = 2 * DL_C * DL_VS;
    return 4 * DL_C * delta_ds(D) + 2 * DL_C * DL_AS + DL_C * DL_MS + (wd > vy ? wd : vy) + 5 * delta_up4(D);
}

// acc[8][4] += A^T[0 .. kn)[8 rows] * B[0 .. kn)[4 columns]
template <int SIGN>
__device__ __forceinline__ void delta_mm84(float (&acc)[8][4], const float* A, int as, const float* B, int bs, int kn) {
#pragma unroll 4
    for (int k = 0; k < kn; ++k) {
        const float4 a0 = ld4(A + k * as), a1 = ld4(A + k * as + 4), b = ld4(B + k * bs);
        const float av[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float x = SIGN > 0 ? av[i] : -av[i];
            acc[i][0] = fmaf(x, b.x, acc[i][0]), acc[i][1] = fmaf(x, b.y, acc[i][1]), acc[i][2] = fmaf(x, b.z, acc[i][2]), acc[i][3] = fmaf(x, b.w, acc[i][3]);
        }
    }
}

template <int TD>
__global__ void __launch_bounds__(DL_NT, TD == 64 ? 3 : (TD == 128 ? 2 : 1)) delta_local_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int D = TD ? TD : a.D, V = TD ? TD : a.V, H = a.H;
    const DeltaRec rec(D, V);
    const int Ds = rec.Ds, Dp = rec.Dp, Vp = rec.Vp;
    float *P = sm, *R = P + DL_C * Ds, *B = R + DL_C * Ds, *K = B + DL_C * Ds;
    float *AT = K + DL_C * Ds, *AF = AT + DL_C * DL_AS, *ME = AF + DL_C * DL_AS;
    float* Wd = ME + DL_C * DL_MS;
    float *Vs = Wd, *Ys = Wd + DL_C * DL_VS;
    const int wd = DL_C * Ds, vy = 2 * DL_C * DL_VS;
    float* segp = Wd + (wd > vy ? wd : vy);
    float* wc = segp + 4 * Dp;
    const int c = blockIdx.x, h = blockIdx.y;
    int e, row0, len;
    if (!find_chunk(st, c, DL_C, e, row0, len)) return;
    float* out = a.chunk + ((int64_t)c * H + h) * rec.size();
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
    // the tokens' rows: a warp takes four tokens
#pragma unroll
    for (int q = 0; q < 4; ++q) {
        const int i = wid * 4 + q;
        const bool in = i < len;
        const float* row = a.proj + (int64_t)(row0 + i) * a.ld;
        float ss = 0.f;
#pragma unroll
        for (int d0 = 0; d0 < Dp; d0 += 32) {
            const int d = d0 + lane;
            float k = 0.f, r = 0.f, av = 0.f, w = 1.f;
            if (in && d < D) {
                const int cc = h * D + d;
                k = row[a.k_col + cc], r = row[a.r_col + cc];
                av = sigmoidf_acc(row[a.a_col + cc] + a.a_b[cc]);
                w = delta_decay(a.wz[(int64_t)(row0 + i) * a.ldw + cc] + a.w0[cc], a.decay_scale);
            }
            ss = fmaf(k, k, ss);
            if (d < Dp) K[i * Ds + d] = k, R[i * Ds + d] = r, B[i * Ds + d] = av, Wd[i * Ds + d] = w;
        }
        const float uinv = 1.0f / sqrtf(warp_sum(ss) + a.unit_eps);
#pragma unroll
        for (int d0 = 0; d0 < Dp; d0 += 32) {
            const int d = d0 + lane;
            if (d >= Dp) break;
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
#pragma unroll 2
        for (int d = 0; d < Dp; d += 4) {
            float4 q[4], k[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) q[i] = ld4(P + (ty * 4 + i) * Ds + d);
#pragma unroll
            for (int j = 0; j < 4; ++j) k[j] = ld4(B + (tx + 16 * j) * Ds + d);
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
                const float v = (isp ? cj < ri : cj <= ri) ? s[i][j] : 0.f;
                if (j < 2) (isp ? AT : AF)[cj * DL_AS + ri] = v;
                else ME[cj * DL_MS + (isp ? 0 : DL_C) + ri] = v;
            }
        }
    }
    __syncthreads();
    const int rg = wid & 3;            // products of 32 rows: a warp takes eight rows, a lane four columns; rows before the group's last one enter only
    const int kn = 8 * (rg + 1);
    for (int v0 = 0; v0 < V; v0 += 64) {
        for (int it = tid; it < DL_C * 64; it += DL_NT) {      // (the scores' barrier, or the end of the previous tile, freed the place)
            const int i = it >> 6, cc = it & 63;
            Vs[i * DL_VS + cc] = (i < len && v0 + cc < V) ? a.proj[(int64_t)(row0 + i) * a.ld + a.v_col + (int64_t)h * V + v0 + cc] : 0.f;
        }
        __syncthreads();
        const int nc = (v0 == 0 ? Dp : 0) + 64;                // columns of [P | M V]: P with the first tile only
        const int pc = v0 == 0 ? Dp : 0;
        if (wid >= 4) {                                        // M V to the Y tile, E V to the record: 64 rows, the warp's lanes cover 16 column groups of two row groups
            const int t2 = tid - 128, cg = t2 & 15, rr = t2 >> 4;
            float acc[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) acc[i][u] = 0.f;
            delta_mm84<1>(acc, ME + rr * 8, DL_MS, Vs + cg * 4, DL_VS, DL_C);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float4 v = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
                if (rr < 4) *reinterpret_cast<float4*>(Ys + (rr * 8 + i) * DL_VS + cg * 4) = v;
                else if (v0 + cg * 4 < Vp) *reinterpret_cast<float4*>(out + rec.o() + ((rr - 4) * 8 + i) * Vp + v0 + cg * 4) = v;
            }
        } else if (wid == 0 && v0 == 0) {                      // (I + L)^-1: lane = column, forward substitution
            float x[DL_C];
#pragma unroll
            for (int i = 0; i < DL_C; ++i) x[i] = i == lane ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < DL_C; ++j) {
                const float y = x[j];
#pragma unroll
                for (int i4 = j & ~3; i4 < DL_C; i4 += 4) {
                    const float4 l = ld4(AT + j * DL_AS + i4);
                    x[i4] = fmaf(-l.x, y, x[i4]), x[i4 + 1] = fmaf(-l.y, y, x[i4 + 1]), x[i4 + 2] = fmaf(-l.z, y, x[i4 + 2]), x[i4 + 3] = fmaf(-l.w, y, x[i4 + 3]);
                }
            }
            __syncwarp();
#pragma unroll
            for (int i4 = 0; i4 < DL_C; i4 += 4) *reinterpret_cast<float4*>(AT + lane * DL_AS + i4) = make_float4(x[i4], x[i4 + 1], x[i4 + 2], x[i4 + 3]);
        } else if (v0 == 0) {                                  // beta W_C to the record
            for (int it = tid - 32; it < DL_C * (Dp >> 2); it += 96) {
                const int i = it / (Dp >> 2), d = 4 * (it - i * (Dp >> 2));
                const float4 b = ld4(B + i * Ds + d), w = ld4(wc + d);
                *reinterpret_cast<float4*>(out + rec.b() + i * Ds + d) = make_float4(b.x * w.x, b.y * w.y, b.z * w.z, b.w * w.w);
            }
        }
        __syncthreads();
        // [P' | Y0] = (I + L)^-1 [P | M V], in place: column groups dealt to the two halves of the block, results held back until every warp has read
        constexpr int NG = TD ? (TD + 64 + 255) / 256 : 2;     // column groups a lane may have (D <= 256)
        float acc[NG][8][4];
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            const int col = 4 * (lane + 32 * ((wid >> 2) + 2 * g));
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) acc[g][i][u] = 0.f;
            if (col < pc) delta_mm84<1>(acc[g], AT + rg * 8, DL_AS, P + col, Ds, kn);
            else if (col < nc) delta_mm84<1>(acc[g], AT + rg * 8, DL_AS, Ys + col - pc, DL_VS, kn);
        }
        __syncthreads();
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            const int col = 4 * (lane + 32 * ((wid >> 2) + 2 * g));
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float4 v = make_float4(acc[g][i][0], acc[g][i][1], acc[g][i][2], acc[g][i][3]);
                const int r = rg * 8 + i;
                if (col < pc) {
                    *reinterpret_cast<float4*>(P + r * Ds + col) = v;
                    *reinterpret_cast<float4*>(out + r * Ds + col) = v;
                } else if (col < nc) {
                    *reinterpret_cast<float4*>(Ys + r * DL_VS + col - pc) = v;
                }
            }
        }
        __syncthreads();
        // R' = rho - F P', O0 = E V - F Y0
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            const int col = 4 * (lane + 32 * ((wid >> 2) + 2 * g));
            const bool isp = col < pc;
            if (col >= nc || (!isp && v0 + col - pc >= Vp)) continue;
            float* dst = isp ? out + rec.r() + rg * 8 * Ds + col : out + rec.o() + rg * 8 * Vp + v0 + col - pc;
            const int ds = isp ? Ds : Vp;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float4 v = isp ? ld4(R + (rg * 8 + i) * Ds + col) : ld4(dst + i * Vp);
                acc[g][i][0] = v.x, acc[g][i][1] = v.y, acc[g][i][2] = v.z, acc[g][i][3] = v.w;
            }
            if (isp) delta_mm84<-1>(acc[g], AF + rg * 8, DL_AS, P + col, Ds, kn);
            else delta_mm84<-1>(acc[g], AF + rg * 8, DL_AS, Ys + col - pc, DL_VS, kn);
#pragma unroll
            for (int i = 0; i < 8; ++i) *reinterpret_cast<float4*>(dst + i * ds) = make_float4(acc[g][i][0], acc[g][i][1], acc[g][i][2], acc[g][i][3]);
        }
        // U = W_C (kappa^T V - beta^T Y0): thread (ty, tx): channels ty * 4 + i, value columns tx * 4 + u
        const int tx = tid & 15, ty = tid >> 4;
#pragma unroll
        for (int d0 = 0; d0 < Dp; d0 += 64) {
            const int d = d0 + ty * 4;
            if (d >= Dp) break;
            float s[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) s[i][u] = 0.f;
#pragma unroll 2
            for (int j = 0; j < DL_C; ++j) {
                const float4 k = ld4(K + j * Ds + d), b = ld4(B + j * Ds + d), v = ld4(Vs + j * DL_VS + tx * 4), y = ld4(Ys + j * DL_VS + tx * 4);
                const float kk[4] = {k.x, k.y, k.z, k.w}, bb[4] = {b.x, b.y, b.z, b.w}, vv[4] = {v.x, v.y, v.z, v.w}, yy[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int u = 0; u < 4; ++u) s[i][u] = fmaf(kk[i], vv[u], fmaf(-bb[i], yy[u], s[i][u]));
            }
            if (v0 + tx * 4 < Vp) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float w = wc[d + i];
                    *reinterpret_cast<float4*>(out + rec.u() + (d + i) * Vp + v0 + tx * 4) = make_float4(s[i][0] * w, s[i][1] * w, s[i][2] * w, s[i][3] * w);
                }
            }
        }
        __syncthreads();
    }
}

// ---- pass B: grid (value tiles of VT, H, B), 16 * VT threads ------------------------------------------------------------------------------------
// Dynamic shared memory: S [Dp][VT + 2] | Y [C][YS] | NST stages of (P' [C][Ds] | beta W_C [C][Ds] | W_C [Dp] | the thread's own pieces of U)
__host__ __device__ constexpr int delta_stage_floats(int D, int VT) { return 2 * DL_C * delta_ds(D) + delta_up4(D) + (delta_up4(D) + 63) / 64 * 64 * VT; }
__host__ __device__ constexpr int delta_scan_floats(int D, int VT, int nst) { return delta_up4(delta_up4(D) * (VT + 2)) + DL_C * (VT == 16 ? 24 : 8) + nst * delta_stage_floats(D, VT); }

__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(src));
}

template <int TD, int VT, int NST>
__global__ void __launch_bounds__(16 * VT) delta_scan_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NT = 16 * VT, SS = VT + 2, YS = VT == 16 ? 24 : 8;
    const int D = TD ? TD : a.D, V = TD ? TD : a.V, H = a.H;
    const DeltaRec rec(D, V);
    const int Ds = rec.Ds, Dp = rec.Dp, Vp = rec.Vp;
    const int nu = (Dp + 63) >> 6;                  // groups of 64 key channels
    const int stage = 2 * DL_C * Ds + Dp + nu * 64 * VT;
    float* S = sm;
    float* Y = S + ((Dp * SS + 3) & ~3);
    float* buf = Y + DL_C * YS;
    const int v0 = blockIdx.x * VT, h = blockIdx.y, e = blockIdx.z, tid = threadIdx.x;
    int c0 = 0;
    for (int i = 0; i < e; ++i) c0 += (st.ent_start[i + 1] - st.ent_start[i] + DL_C - 1) / DL_C;
    const int nc = (st.ent_start[e + 1] - st.ent_start[e] + DL_C - 1) / DL_C;
    if (nc == 0) return;
    float* slot = a.state + ((int64_t)st.ent_slot[e] * H + h) * D * V;
    const bool fresh = st.ent_pos0[e] == 0;
    for (int it = tid; it < Dp * VT; it += NT) {
        const int d = it / VT, cc = it - d * VT;
        S[d * SS + cc] = (!fresh && d < D && v0 + cc < V) ? slot[(int64_t)d * V + v0 + cc] : 0.f;
    }
    // Y = P' S: rows rg * 4 + i, columns cg * 2 + u; update: channels dgr * 4 + i (+ 64 n), columns vg * 4 + u; the four lanes kq share out the sums
    const int kq = tid & 3, rest = tid >> 2, dgr = rest / (VT / 4), vg = rest % (VT / 4), rg = rest / (VT / 2), cg = rest % (VT / 2);
    const bool vin = v0 + vg * 4 < Vp;
    float* rec0 = a.chunk + ((int64_t)c0 * H + h) * rec.size();
    const int64_t rstep = (int64_t)H * rec.size();
    const int mine = (dgr * 4 + kq) * Vp + v0 + vg * 4;      // this thread's piece of U (channel dgr * 4 + kq + 64 n)
    auto fetch = [&](int c) {
        if (c < nc) {
            const float* g = rec0 + c * rstep;
            float* b = buf + (c % NST) * stage;
            const int n16 = (2 * DL_C * Ds + Dp) >> 2;
            for (int it = tid; it < n16; it += NT) cp_async16(b + 4 * it, g + 4 * it);
            float* ub = b + 4 * n16;
            for (int n = 0; n < nu; ++n)
                if (vin && n * 64 + dgr * 4 < Dp) cp_async16(ub + 4 * (n * NT + tid), g + rec.u() + mine + n * 64 * Vp);
        }
        asm volatile("cp.async.commit_group;\n");
    };
#pragma unroll
    for (int i = 0; i < NST - 1; ++i) fetch(i);
    for (int c = 0; c < nc; ++c) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(NST - 2));
        __syncthreads();   // stage c is in place, S is the state in front of chunk c, the stage of chunk c - 1 is free
        fetch(c + NST - 1);
        const float* Pm = buf + (c % NST) * stage;
        const float* Bm = Pm + DL_C * Ds;
        const float* wc = Bm + DL_C * Ds;
        const float* ub = wc + Dp;
        {
            float acc[4][2];
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0.f;
#pragma unroll 4
            for (int d = kq * 4; d < Dp; d += 16) {
                float4 p[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) p[i] = ld4(Pm + (rg * 4 + i) * Ds + d);
#pragma unroll
                for (int dd = 0; dd < 4; ++dd) {
                    const float2 s = *reinterpret_cast<const float2*>(S + (d + dd) * SS + cg * 2);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float pv = dd == 0 ? p[i].x : dd == 1 ? p[i].y : dd == 2 ? p[i].z : p[i].w;
                        acc[i][0] = fmaf(pv, s.x, acc[i][0]), acc[i][1] = fmaf(pv, s.y, acc[i][1]);
                    }
                }
            }
            // sum over the four lanes; lane kq keeps row kq
            float m[2][2], f[2];
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const float send = (kq & 2) ? acc[i][u] : acc[i + 2][u], keep = (kq & 2) ? acc[i + 2][u] : acc[i][u];
                    m[i][u] = keep + __shfl_xor_sync(0xffffffffu, send, 2);
                }
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float send = (kq & 1) ? m[0][u] : m[1][u], keep = (kq & 1) ? m[1][u] : m[0][u];
                f[u] = keep + __shfl_xor_sync(0xffffffffu, send, 1);
            }
            *reinterpret_cast<float2*>(Y + (rg * 4 + kq) * YS + cg * 2) = make_float2(f[0], f[1]);
        }
        __syncthreads();
        float* gz = rec0 + c * rstep + rec.u() + mine;
#pragma unroll
        for (int n = 0; n < (TD ? TD / 64 : 4); ++n) {   // S = W_C S + U - (beta W_C)^T Y; the old S takes U's place in the record
            if (n >= nu) break;
            const int db = n * 64 + dgr * 4;
            const bool dok = db < Dp;    // Dp is a multiple of 4: all four channels or none (the same for the four lanes kq)
            float acc[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int u = 0; u < 4; ++u) acc[i][u] = 0.f;
            if (dok) {
#pragma unroll
                for (int jj = 0; jj < DL_C / 4; ++jj) {
                    const int j = 4 * jj + kq;
                    const float4 b = ld4(Bm + j * Ds + db), y = ld4(Y + j * YS + vg * 4);
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
                    const float send = (kq & 2) ? acc[i][u] : acc[i + 2][u], keep = (kq & 2) ? acc[i + 2][u] : acc[i][u];
                    m[i][u] = keep + __shfl_xor_sync(0xffffffffu, send, 2);
                }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float send = (kq & 1) ? m[0][u] : m[1][u], keep = (kq & 1) ? m[1][u] : m[0][u];
                f[u] = keep + __shfl_xor_sync(0xffffffffu, send, 1);
            }
            if (dok) {
                const int d = db + kq;
                float2* sp = reinterpret_cast<float2*>(S + d * SS + vg * 4);
                const float2 s0 = sp[0], s1 = sp[1];
                float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
                if (vin) {
                    u = ld4(ub + 4 * (n * NT + tid));
                    *reinterpret_cast<float4*>(gz + n * 64 * Vp) = make_float4(s0.x, s0.y, s1.x, s1.y);
                }
                const float w = wc[d];
                sp[0] = make_float2(fmaf(w, s0.x, u.x - f[0]), fmaf(w, s0.y, u.y - f[1]));
                sp[1] = make_float2(fmaf(w, s1.x, u.z - f[2]), fmaf(w, s1.y, u.w - f[3]));
            }
        }
    }
    __syncthreads();
    for (int it = tid; it < D * VT; it += NT) {
        const int d = it / VT, cc = it - d * VT;
        if (v0 + cc < V) slot[(int64_t)d * V + v0 + cc] = S[d * SS + cc];
    }
}

// ---- pass C: grid (chunks, H), 128 threads; thread (ty, tx): tokens ty * 4 + i, value columns tx * 4 + u of a tile of 64 --------------------
// Dynamic shared memory: R' [C][Ds] | slab of the start state [64][VS] | o [C][Vp + 4]
constexpr int DL_NC = 128, DL_ZS = 64;
__host__ __device__ constexpr int delta_out_floats(int D, int V) { return DL_C * delta_ds(D) + DL_ZS * DL_VS + DL_C * (delta_up4(V) + 4); }

template <int TD>
__global__ void __launch_bounds__(DL_NC) delta_out_kernel(const DeltaArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int D = TD ? TD : a.D, V = TD ? TD : a.V, H = a.H;
    const DeltaRec rec(D, V);
    const int Ds = rec.Ds, Dp = rec.Dp, Vp = rec.Vp, Os = Vp + 4;
    float *R = sm, *Z = R + DL_C * Ds, *O = Z + DL_ZS * DL_VS;
    const int c = blockIdx.x, h = blockIdx.y;
    int e, row0, len;
    if (!find_chunk(st, c, DL_C, e, row0, len)) return;
    const float* g = a.chunk + ((int64_t)c * H + h) * rec.size();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    for (int it = tid; it < DL_C * Ds / 4; it += DL_NC) cp_async16(R + 4 * it, g + rec.r() + 4 * it);
    for (int v0 = 0; v0 < V; v0 += 64) {
        float acc[4][4];
        const bool vin = v0 + tx * 4 < Vp;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float4 o = vin ? ld4(g + rec.o() + (ty * 4 + i) * Vp + v0 + tx * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            acc[i][0] = o.x, acc[i][1] = o.y, acc[i][2] = o.z, acc[i][3] = o.w;
        }
        for (int d0 = 0; d0 < Dp; d0 += DL_ZS) {
            __syncthreads();
            for (int it = tid; it < DL_ZS * 16; it += DL_NC) {
                const int dd = it >> 4, c4 = it & 15;
                if (d0 + dd < Dp && v0 + 4 * c4 < Vp) cp_async16(Z + dd * DL_VS + 4 * c4, g + rec.u() + (d0 + dd) * Vp + v0 + 4 * c4);
            }
            asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n");
            __syncthreads();
            if (!vin) continue;          // (columns beyond the last are neither copied nor used)
            const int dn = min(DL_ZS, Dp - d0);
#pragma unroll 2
            for (int dd = 0; dd < dn; dd += 4) {
                float4 r[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) r[i] = ld4(R + (ty * 4 + i) * Ds + d0 + dd);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const float4 z = ld4(Z + (dd + k) * DL_VS + tx * 4);
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

template <typename K>
static cudaError_t delta_smem(K kernel, size_t bytes) {
    return bytes > 48 * 1024 ? cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) : cudaSuccess;
}

template <int TD, int VT, int NST>
static cudaError_t delta_scan_launch(const DeltaArgs& a, const b200seq_step& st, cudaStream_t cs) {
    const size_t sb = (size_t)delta_scan_floats(a.D, VT, NST) * sizeof(float);
    const cudaError_t e = delta_smem(delta_scan_kernel<TD, VT, NST>, sb);
    if (e == cudaSuccess) delta_scan_kernel<TD, VT, NST><<<dim3((a.V + VT - 1) / VT, a.H, st.B), 16 * VT, sb, cs>>>(a, st);
    return e;
}

template <int TD>
static int delta_portions(const DeltaArgs& a, const b200seq_step& st, cudaStream_t cs) {
    const int chunks = (st.T + DL_C - 1) / DL_C + st.B;   // upper bound of the step's chunk count
    const size_t sa = (size_t)delta_local_floats(a.D) * sizeof(float), sc = (size_t)delta_out_floats(a.D, a.V) * sizeof(float);
    cudaError_t err = delta_smem(delta_local_kernel<TD>, sa);
    if (err == cudaSuccess) err = delta_smem(delta_out_kernel<TD>, sc);
    if (err != cudaSuccess) return cuda_status(err, "delta attribute");
    delta_local_kernel<TD><<<dim3(chunks, a.H), DL_NT, sa, cs>>>(a, st);
    SEQ_LAUNCH_CHECK("delta local pass");
    // narrower value tiles while the wider ones would leave SMs idle
    const bool narrow = (int64_t)a.H * st.B * ((a.V + 15) / 16) < 128;
    if (TD == 0) err = a.D <= 128 ? delta_scan_launch<TD, 16, 3>(a, st, cs) : delta_scan_launch<TD, 16, 2>(a, st, cs);
    else err = narrow ? delta_scan_launch<TD, 8, 3>(a, st, cs) : delta_scan_launch<TD, 16, 3>(a, st, cs);
    if (err != cudaSuccess) return cuda_status(err, "delta attribute");
    SEQ_LAUNCH_CHECK("delta scan pass");
    delta_out_kernel<TD><<<dim3(chunks, a.H), DL_NC, sc, cs>>>(a, st);
    SEQ_LAUNCH_CHECK("delta output pass");
    return 0;
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
    if (d->D > 256 || (size_t)delta_local_floats(d->D) * 4 > 220 * 1024 || (size_t)delta_out_floats(d->D, d->V) * 4 > 220 * 1024)
        return fail(B200SEQ_ERR_UNSUPPORTED, "delta: head sizes too large");
    if (d->D == 64 && d->V == 64) return delta_portions<64>(a, *st, cs);
    if (d->D == 128 && d->V == 128) return delta_portions<128>(a, *st, cs);
    return delta_portions<0>(a, *st, cs);
}
