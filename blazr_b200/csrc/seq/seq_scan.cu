// seq_scan.cu -- selective scan over a flat mixed batch: a decay per channel and state, S [C][N] carried per sequence in f32,
//     dt = softplus(z + b),   S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c u_c B[n],   y_c = sum_n S[c][n] C[n] + D_c u_c,   out = y * gate
// Step sizes, decays, state and sums are f32.  A comes as A * log2(e), so that a decay is one exp2.
//
// Steps in which every entry brings ONE token: SS_L lanes per channel; the lanes share out the states and the products of the channel's step-size
// projection w_dt . low.
// Other steps: a thread owns a channel (large states: NL lanes of a warp share it), its states stay in registers, and it walks the tokens of a segment
// in order; B and C of a tile of tokens are staged in shared memory, u, dt and gate are read coalesced along the channels.
//   T <= SS_SEG   one launch, a segment is an entry's whole portion
//   longer        every portion is cut into segments of SS_SEG tokens (from its first token) that run in parallel:
//     A  each segment from a zero state -> its end state E and the sum of its dt; dt replaces z in memory
//     B  per entry, in order: start[s] = S;  S = exp(A sum dt) S + E[s];  the last S goes to the slot
//     C  each segment again from start[s], with the outputs
#include "seq_common.cuh"

namespace b200seq {

constexpr int SS_SEG = 64;    // tokens per segment
constexpr int SS_TT = 16;     // tokens per staged tile
constexpr int SS_NT = 128;
constexpr int SS_L = 4;       // lanes per channel in steps of single tokens
enum { SS_DIRECT = 0, SS_LOCAL = 1, SS_FINAL = 2 };

struct ScanArgs {
    const void* u;
    const float* dbc;
    int64_t ldd;
    float* dtz;
    const float* gate;
    int64_t ldg;
    int C, N, R;
    const float *a2, *Dp, *dt_b;
    const __nv_bfloat16* w_dt;
    float* state;       // [slots][C][N]
    float* seg_state;   // [segments][C][N]: E after pass A, the start state after pass B
    float* seg_dt;      // [segments][C]
    void* out;
    int out_dtype;
};

__device__ __forceinline__ float ex2f(float x) {   // 2^x for x <= 0; results below the normal range are zero
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
template <typename UT>
__device__ __forceinline__ float ld_u(const void* p, int64_t i);
template <>
__device__ __forceinline__ float ld_u<float>(const void* p, int64_t i) { return reinterpret_cast<const float*>(p)[i]; }
template <>
__device__ __forceinline__ float ld_u<__nv_bfloat16>(const void* p, int64_t i) { return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]); }

// ---- one token per entry: grid (tiles of SS_NT / SS_L channels, B) ------------------------------------------------------------------------------------
// dynamic shared memory: low [R] | B [N] | C [N] of the entry's row
template <typename UT, bool V4>
__global__ void __launch_bounds__(SS_NT) scan_token_kernel(const ScanArgs a, const b200seq_step st) {
    extern __shared__ __align__(16) float sm[];
    const int N = a.N, R = a.R;
    const int e = blockIdx.y, sub = threadIdx.x % SS_L;
    const int c = blockIdx.x * (SS_NT / SS_L) + threadIdx.x / SS_L;
    const bool live = c < a.C;
    const int cc = live ? c : a.C - 1;
    const int t = st.ent_start[e];
    const bool fresh = st.ent_pos0[e] == 0;
    float* S = a.state + ((int64_t)st.ent_slot[e] * a.C + cc) * N;
    const float* A = a.a2 + (int64_t)cc * N;
    const float* row = a.dbc + (int64_t)t * a.ldd;
    const int n4 = V4 ? (N & ~(4 * SS_L - 1)) : 0;    // states taken four at a time, the rest one at a time
    float4 s4 = make_float4(0.f, 0.f, 0.f, 0.f), a4 = s4;
    if (n4 > 0) {                                      // the first states are requested before anything is waited for
        if (!fresh) s4 = ld4(S + 4 * sub);
        a4 = ld4(A + 4 * sub);
    }
    const float u = ld_u<UT>(a.u, (int64_t)t * a.C + cc), gate = a.gate[(int64_t)t * a.ldg + cc], dtb = a.dt_b[cc], dc = a.Dp[cc];
    for (int i = threadIdx.x; i < R + 2 * N; i += SS_NT) sm[i] = row[i];
    __syncthreads();
    const float *Bs = sm + R, *Cs = Bs + N;
    float z = 0.f;
    const __nv_bfloat16* wd = a.w_dt + (int64_t)cc * R;
    if ((R & 7) == 0) {
        for (int r = sub * 8; r < R; r += 8 * SS_L) {
            const uint4 w = *reinterpret_cast<const uint4*>(wd + r);
            const uint32_t wu[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                z = fmaf(__uint_as_float(wu[i] << 16), sm[r + 2 * i], z);
                z = fmaf(__uint_as_float(wu[i] & 0xffff0000u), sm[r + 2 * i + 1], z);
            }
        }
    } else {
        for (int r = sub; r < R; r += SS_L) z = fmaf(__bfloat162float(wd[r]), sm[r], z);
    }
#pragma unroll
    for (int o = 1; o < SS_L; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
    const float dt = softplusf_acc(z + dtb), dtu = dt * u;
    float y = 0.f;
    for (int n = 4 * sub; n < n4; n += 4 * SS_L) {
        if (n >= 4 * SS_L) {
            s4 = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : ld4(S + n);
            a4 = ld4(A + n);
        }
        s4.x = fmaf(ex2f(dt * a4.x), s4.x, dtu * Bs[n]), s4.y = fmaf(ex2f(dt * a4.y), s4.y, dtu * Bs[n + 1]);
        s4.z = fmaf(ex2f(dt * a4.z), s4.z, dtu * Bs[n + 2]), s4.w = fmaf(ex2f(dt * a4.w), s4.w, dtu * Bs[n + 3]);
        y = fmaf(s4.x, Cs[n], y), y = fmaf(s4.y, Cs[n + 1], y), y = fmaf(s4.z, Cs[n + 2], y), y = fmaf(s4.w, Cs[n + 3], y);
        if (live) *reinterpret_cast<float4*>(S + n) = s4;
    }
    for (int n = n4 + sub; n < N; n += SS_L) {
        const float s = fmaf(ex2f(dt * A[n]), fresh ? 0.f : S[n], dtu * Bs[n]);
        y = fmaf(s, Cs[n], y);
        if (live) S[n] = s;
    }
#pragma unroll
    for (int o = 1; o < SS_L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (live && sub == 0) store_act(a.out, a.out_dtype, (int64_t)t * a.C + c, fmaf(dc, u, y) * gate);
}

// ---- portions: grid (channel tiles, segments or entries) ------------------------------------------------------------------------------------------------
// NPL: states per lane (lane `sub` of the NL lanes of a channel holds n = sub * NPL + i); a warp covers 32 / NL channels
template <typename UT, int NPL, int MODE>
__global__ void __launch_bounds__(SS_NT) scan_kernel(const ScanArgs a, const b200seq_step st, int NL) {
    extern __shared__ __align__(16) float sm[];   // B [SS_TT][NL * NPL] | C the same
    const int N = a.N, C = a.C, nrow = NL * NPL;
    float *Bs = sm, *Cs = sm + SS_TT * nrow;
    const int cpw = 32 / NL, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane / cpw;
    const int c = (blockIdx.x * (SS_NT / 32) + warp) * cpw + lane % cpw;
    const bool live = c < C;
    const int cc = live ? c : C - 1;
    int e, row0, len;
    if (MODE == SS_DIRECT) {
        e = blockIdx.y;
        row0 = st.ent_start[e], len = st.ent_start[e + 1] - row0;
    } else if (!find_chunk(st, blockIdx.y, SS_SEG, e, row0, len)) {
        return;
    }
    const float* init = nullptr;
    if (MODE == SS_DIRECT && st.ent_pos0[e] != 0) init = a.state + ((int64_t)st.ent_slot[e] * C + cc) * N;
    if (MODE == SS_FINAL) init = a.seg_state + ((int64_t)blockIdx.y * C + cc) * N;
    float S[NPL], A[NPL];
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        const int n = sub * NPL + i;
        S[i] = (init && n < N) ? init[n] : 0.f;
        A[i] = n < N ? a.a2[(int64_t)cc * N + n] : 0.f;
    }
    const float dtb = a.dt_b[cc], dc = a.Dp[cc];
    float dtsum = 0.f;
    for (int i0 = 0; i0 < len; i0 += SS_TT) {
        const int nt = min(SS_TT, len - i0);
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * nrow; idx += SS_NT) {
            const int tt = idx / nrow, n = idx - tt * nrow;
            const float* r = a.dbc + (int64_t)(row0 + i0 + tt) * a.ldd + a.R + n;
            Bs[idx] = n < N ? r[0] : 0.f;
            if (MODE != SS_LOCAL) Cs[idx] = n < N ? r[N] : 0.f;
        }
        __syncthreads();
        constexpr int TU = 4;    // the inputs of four tokens are in flight together
        for (int t4 = 0; t4 < nt; t4 += TU) {
            float uu[TU], dd[TU], gg[TU];
#pragma unroll
            for (int k = 0; k < TU; ++k) {
                const int64_t t = row0 + i0 + min(t4 + k, nt - 1);
                uu[k] = ld_u<UT>(a.u, t * C + cc);
                dd[k] = a.dtz[t * C + cc];
                gg[k] = MODE != SS_LOCAL ? a.gate[t * a.ldg + cc] : 0.f;
            }
            if (MODE != SS_FINAL) {
#pragma unroll
                for (int k = 0; k < TU; ++k) dd[k] = softplusf_acc(dd[k] + dtb);
            }
            if (MODE == SS_LOCAL) {
                __syncwarp();    // every lane of a channel has read z before one of them puts dt in its place
#pragma unroll
                for (int k = 0; k < TU; ++k)
                    if (t4 + k < nt && live && sub == 0) a.dtz[(int64_t)(row0 + i0 + t4 + k) * C + cc] = dd[k];
            }
#pragma unroll
            for (int k = 0; k < TU; ++k) {
                if (t4 + k >= nt) break;
                const float dt = dd[k], dtu = dt * uu[k];
                const float* Bt = Bs + (t4 + k) * nrow + sub * NPL;
                const float* Ct = Cs + (t4 + k) * nrow + sub * NPL;
                float y0 = 0.f, y1 = 0.f;
#pragma unroll
                for (int i = 0; i < NPL; i += 4) {
                    const float4 b = ld4(Bt + i);
                    S[i] = fmaf(ex2f(dt * A[i]), S[i], dtu * b.x), S[i + 1] = fmaf(ex2f(dt * A[i + 1]), S[i + 1], dtu * b.y);
                    S[i + 2] = fmaf(ex2f(dt * A[i + 2]), S[i + 2], dtu * b.z), S[i + 3] = fmaf(ex2f(dt * A[i + 3]), S[i + 3], dtu * b.w);
                    if (MODE != SS_LOCAL) {
                        const float4 q = ld4(Ct + i);
                        y0 = fmaf(S[i], q.x, y0), y1 = fmaf(S[i + 1], q.y, y1), y0 = fmaf(S[i + 2], q.z, y0), y1 = fmaf(S[i + 3], q.w, y1);
                    }
                }
                if (MODE == SS_LOCAL) {
                    dtsum += dt;
                } else {
                    float y = y0 + y1;
                    for (int o = cpw; o < 32; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
                    if (live && sub == 0) store_act(a.out, a.out_dtype, (int64_t)(row0 + i0 + t4 + k) * C + cc, fmaf(dc, uu[k], y) * gg[k]);
                }
            }
        }
    }
    if (MODE == SS_FINAL || !live) return;
    float* dst = MODE == SS_DIRECT ? a.state + ((int64_t)st.ent_slot[e] * C + c) * N : a.seg_state + ((int64_t)blockIdx.y * C + c) * N;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        const int n = sub * NPL + i;
        if (n < N) dst[n] = S[i];
    }
    if (MODE == SS_LOCAL && sub == 0) a.seg_dt[(int64_t)blockIdx.y * C + c] = dtsum;
}

// pass B: one thread per (entry, channel, state); the segments' end states do not depend on the walk, so a batch of them is fetched ahead of the chain
__global__ void scan_combine_kernel(const ScanArgs a, const b200seq_step st) {
    const int64_t per = (int64_t)a.C * a.N;
    const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    const int e = blockIdx.y;
    if (idx >= per) return;
    const int c = (int)(idx / a.N);
    int s0 = 0;
    for (int i = 0; i < e; ++i) s0 += (st.ent_start[i + 1] - st.ent_start[i] + SS_SEG - 1) / SS_SEG;
    const int ns = (st.ent_start[e + 1] - st.ent_start[e] + SS_SEG - 1) / SS_SEG;
    float* slot = a.state + (int64_t)st.ent_slot[e] * per + idx;
    float S = st.ent_pos0[e] == 0 ? 0.f : *slot;
    const float A = a.a2[idx];
    constexpr int AHEAD = 8;
    for (int sb = 0; sb < ns; sb += AHEAD) {
        float E[AHEAD], d[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const bool in = sb + j < ns;
            E[j] = in ? a.seg_state[(int64_t)(s0 + sb + j) * per + idx] : 0.f;
            d[j] = in ? a.seg_dt[(int64_t)(s0 + sb + j) * a.C + c] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (sb + j >= ns) break;
            a.seg_state[(int64_t)(s0 + sb + j) * per + idx] = S;
            S = fmaf(ex2f(A * d[j]), S, E[j]);
        }
    }
    *slot = S;
}

template <typename UT, int NPL, int MODE>
static void scan_launch(const ScanArgs& a, const b200seq_step& st, int NL, int ny, cudaStream_t cs) {
    const int ch = SS_NT / NL;
    scan_kernel<UT, NPL, MODE><<<dim3((a.C + ch - 1) / ch, ny), SS_NT, (size_t)2 * SS_TT * NL * NPL * sizeof(float), cs>>>(a, st, NL);
}

template <typename UT, int NPL>
static int scan_portions(const ScanArgs& a, const b200seq_step* st, int NL, int segs, cudaStream_t cs) {
    if (segs == 0) {
        scan_launch<UT, NPL, SS_DIRECT>(a, *st, NL, st->B, cs);
        SEQ_LAUNCH_CHECK("selective_scan");
        return 0;
    }
    scan_launch<UT, NPL, SS_LOCAL>(a, *st, NL, segs, cs);
    SEQ_LAUNCH_CHECK("selective_scan local pass");
    const int64_t per = (int64_t)a.C * a.N;
    scan_combine_kernel<<<dim3((unsigned)((per + 127) / 128), st->B), 128, 0, cs>>>(a, *st);
    SEQ_LAUNCH_CHECK("selective_scan combine pass");
    scan_launch<UT, NPL, SS_FINAL>(a, *st, NL, segs, cs);
    SEQ_LAUNCH_CHECK("selective_scan final pass");
    return 0;
}

template <typename UT>
static int scan_run(const ScanArgs& a, const b200seq_step* st, int segs, cudaStream_t cs) {
    if (st->T == st->B) {
        const size_t smem = (size_t)(a.R + 2 * a.N) * sizeof(float);
        const dim3 grid((a.C + SS_NT / SS_L - 1) / (SS_NT / SS_L), st->B);
        if (a.N % 4 == 0 && a.N >= 4 * SS_L) scan_token_kernel<UT, true><<<grid, SS_NT, smem, cs>>>(a, *st);
        else scan_token_kernel<UT, false><<<grid, SS_NT, smem, cs>>>(a, *st);
        SEQ_LAUNCH_CHECK("selective_scan single tokens");
        return 0;
    }
    int NL = 1;
    while (32 * NL < a.N) NL *= 2;
    const int npl = (a.N + NL - 1) / NL;
    if (npl <= 8) return scan_portions<UT, 8>(a, st, NL, segs, cs);
    if (npl <= 16) return scan_portions<UT, 16>(a, st, NL, segs, cs);
    if (npl <= 24) return scan_portions<UT, 24>(a, st, NL, segs, cs);
    return scan_portions<UT, 32>(a, st, NL, segs, cs);
}

}  // namespace b200seq

using namespace b200seq;

extern "C" size_t b200seq_scan_scratch_floats(int T, int B, int C, int N) {
    if (T < 1 || B < 1 || T == B || T <= SS_SEG) return 0;
    const size_t segs = (size_t)(T + SS_SEG - 1) / SS_SEG + (size_t)B;
    return segs * ((size_t)C * N + C);
}

extern "C" int b200seq_selective_scan(const void* u, int u_dtype, const float* dbc, int64_t ldd, float* dtz, const float* gate, int64_t ldg, const b200seq_step* st,
                                      const b200seq_scan_desc* d, float* state, void* out, int out_dtype, float* scratch, size_t scratch_floats, void* stream) {
    if (!u || !dbc || !gate || !st || !d || !state || !out || d->C < 1 || d->N < 1 || d->R < 1 || !d->a2 || !d->D || !d->dt_b || !d->w_dt || ldd < d->R + 2 * d->N || ldg < d->C)
        return fail(B200SEQ_ERR_INVALID_ARG, "selective_scan: bad arguments");
    if ((u_dtype != B200SEQ_F32 && u_dtype != B200SEQ_BF16) || (out_dtype != B200SEQ_F32 && out_dtype != B200SEQ_BF16))
        return fail(B200SEQ_ERR_INVALID_ARG, "selective_scan: dtype");
    if (d->N > 256 || d->R + 2 * d->N > 8192) return fail(B200SEQ_ERR_UNSUPPORTED, "selective_scan: state size %d > 256 or step-size rank too large", d->N);
    if ((reinterpret_cast<uintptr_t>(d->a2) & 15) || (reinterpret_cast<uintptr_t>(state) & 15) || (reinterpret_cast<uintptr_t>(d->w_dt) & 15))
        return fail(B200SEQ_ERR_INVALID_ARG, "selective_scan: 16-byte aligned state and weights");
    if (st->T == 0 || st->B == 0) return 0;
    if (st->B > 65535) return fail(B200SEQ_ERR_UNSUPPORTED, "selective_scan: too many entries");
    if (st->T != st->B && !dtz) return fail(B200SEQ_ERR_INVALID_ARG, "selective_scan: a step of portions needs the step-size projection");
    const size_t need = b200seq_scan_scratch_floats(st->T, st->B, d->C, d->N);
    if (need && (!scratch || scratch_floats < need)) return fail(B200SEQ_ERR_INVALID_ARG, "selective_scan: the step needs %zu floats of work area", need);
    ScanArgs a{u, dbc, ldd, dtz, gate, ldg, d->C, d->N, d->R, d->a2, d->D, d->dt_b, (const __nv_bfloat16*)d->w_dt, state, nullptr, nullptr, out, out_dtype};
    int segs = 0;
    if (need) {
        segs = (st->T + SS_SEG - 1) / SS_SEG + st->B;   // upper bound of the step's segment count
        if (segs > 65535) return fail(B200SEQ_ERR_UNSUPPORTED, "selective_scan: too many segments in one step");
        a.seg_state = scratch;
        a.seg_dt = scratch + (size_t)segs * d->C * d->N;
    }
    return u_dtype == B200SEQ_F32 ? scan_run<float>(a, st, segs, (cudaStream_t)stream) : scan_run<__nv_bfloat16>(a, st, segs, (cudaStream_t)stream);
}
