"""The operators the Zetunex design added to libb200seq or extended, each alone, against the plain float64 restatement in
tests/zetunex_oracle.py: linear attention with one norm over all heads (chunked and single-token forms, reused slots, a far memory), the
selective scan (segments, portions, single tokens, every state size class, extreme step sizes, a far memory), silu on a range of projected
columns on every path, the router's groups and weights, the residual of parallel layers in its forms, the embedding without positions,
windowed attention with biases over scattered pages."""
import math

import numpy as np
import pytest
import torch

import zetunex_oracle as O

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def ops():
    if not torch.cuda.is_available():
        pytest.skip("no GPU")
    from blazr_b200 import seqops
    seqops.lib()
    return seqops


def dev_step(ops, entries, block_size=16):
    """entries: [(n_tokens, pos0, slot, block_table)] -> (StepDesc, keep-alive tensors)"""
    from blazr_b200.batch import StepEntry, build_step
    sa = build_step([StepEntry([0] * n, p0, slot, bt) for n, p0, slot, bt in entries], block_size)
    t = {k: torch.from_numpy(np.ascontiguousarray(getattr(sa, k))).to(DEV) for k in ("tok_ent", "tok_pos", "ent_start", "ent_slot", "ent_pos0", "block_table")}
    d = ops.StepDesc(t["tok_ent"].data_ptr(), t["tok_pos"].data_ptr(), t["ent_start"].data_ptr(), t["ent_slot"].data_ptr(), t["ent_pos0"].data_ptr(),
                     t["block_table"].data_ptr(), sa.T, sa.B, sa.block_table.shape[1], block_size)
    return d, t


def pages_for(n, block_size=16, first=0):
    return list(range(first, first + -(-n // block_size)))


def close(got, ref, tol):
    ref = ref.double()
    err = (got.double().cpu() - ref).abs().max().item() / max(ref.abs().max().item(), 1e-30)
    assert err < tol, f"relative error {err:.3e} >= {tol}"


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def bf(t):
    return t.to(torch.bfloat16)


# ---- linear attention with one norm over all heads ----------------------------------------------------------------------------------------
class Lin:
    """a layer's constants and its reference from a projection row q | k | v | gate (q, k, v already activated)"""

    def __init__(self, ops, H, D, V, decay, seed=0, eps=1e-5):
        self.ops, self.H, self.D, self.V, self.eps, self.decay = ops, H, D, V, eps, decay
        self.nw = 1 + 0.3 * rnd(H * V, seed=seed)
        self.dec = torch.tensor([decay, [math.log2(d) for d in decay]], dtype=F64).float().to(DEV)
        self.nwd = self.nw.to(DEV)
        self.desc = ops.retention_desc(H, D, V, self.dec, eps, 1.0, norm_w=self.nwd, gate_sigmoid=True)

    def ref(self, proj):
        H, D, V = self.H, self.D, self.V
        x = proj.double()
        q, k, v = x[:, :H * D].reshape(-1, H, D), x[:, H * D:2 * H * D].reshape(-1, H, D), x[:, 2 * H * D:2 * H * D + H * V].reshape(-1, H, V)
        o = O.decayed_linear_attention(q, k, v, self.decay).reshape(-1, H * V)
        return O.rms_norm(o, self.eps, self.nw.double()) * torch.sigmoid(x[:, 2 * H * D + H * V:])

    def run(self, entries, proj, state, dtype=torch.float32):
        """the operator's result with the deferred division applied"""
        ops, H, V = self.ops, self.H, self.V
        st, keep = dev_step(ops, entries)
        p = proj.to(DEV).contiguous()
        T = p.shape[0]
        out = torch.full((T, H * V), float("nan"), device=DEV, dtype=dtype)
        P = ops.retention_partials(st.T, st.B, H, V)
        ss = torch.full((T, P), float("nan"), device=DEV)
        n = ops.retention_scratch_floats(st.T, st.B, H, self.D, V)
        scratch = torch.full((max(n, 1),), float("nan"), device=DEV)
        ops.retention(p, st, self.desc, state, out, scratch, sumsq=ss)
        return out.float().cpu() / torch.sqrt(ss.sum(1, keepdim=True) / (H * V) + self.eps).cpu()


@pytest.mark.parametrize("H,D,V", [(2, 64, 64), (3, 5, 7), (1, 96, 40), (5, 16, 130), (2, 128, 128), (1, 200, 33), (2, 300, 8), (1, 1, 1)])
def test_linear_attention_over_portions_and_single_tokens(ops, H, D, V):
    """two sequences share the steps, their slots hold another sequence's leftovers; portions around the chunk size, of one and of two tokens"""
    L = Lin(ops, H, D, V, [0.4, 0.97, 0.9999, 1.0, 0.8][:H], seed=1)
    n = {"a": 203, "b": 75}
    X = {s: rnd(k, L.desc.width, seed=5 + i) for i, (s, k) in enumerate(n.items())}
    ref = {s: L.ref(X[s]) for s in n}
    state = torch.full((3, H, D, V), 5.0, device=DEV)
    slot = {"a": 2, "b": 0}
    plan = [[("a", 65), ("b", 2)], [("b", 1), ("a", 1)], [("a", 2), ("b", 63)], [("b", 2), ("a", 1)], [("a", 64)], [("a", 1), ("b", 1)], [("a", 1)], [("b", 6), ("a", 68)]]
    fed = {"a": 0, "b": 0}
    for step in plan:
        got = L.run([(k, fed[s], slot[s], pages_for(fed[s] + k)) for s, k in step], torch.cat([X[s][fed[s]:fed[s] + k] for s, k in step]), state)
        o = 0
        for s, k in step:
            close(got[o:o + k], ref[s][fed[s]:fed[s] + k], 3e-5)
            fed[s] += k
            o += k
    assert fed == n and (state[1] == 5.0).all() and ops.error_flags() == 0


@pytest.mark.parametrize("cut", [[900], [64, 2, 33, 600, 201], [899, 1], [1] + [128] * 7 + [3]])
def test_linear_attention_far_memory(ops, cut):
    """one key of its own 900 tokens back under a decay of 0.9995: the last query reads that value and nothing else"""
    H, D, V, T = 1, 24, 16, 900
    L = Lin(ops, H, D, V, [0.9995], seed=2)
    x = rnd(T, L.desc.width, seed=3) * 0.3
    x[:, D] = 0.0                                  # key dimension 0 belongs to the first token alone
    x[0, D:2 * D] = 0.0
    x[0, D], x[T - 1, :D] = 4.0, 0.0
    x[T - 1, 0] = 3.0
    x[0, 2 * D:2 * D + V] = torch.linspace(-2, 2, V)
    ref = L.ref(x)
    want = torch.linspace(-2, 2, V, dtype=F64)
    assert torch.nn.functional.cosine_similarity(ref[-1] / L.nw.double() / torch.sigmoid(x[-1, 2 * D + V:].double()), want, 0) > 0.999
    state = torch.full((2, H, D, V), 3.0, device=DEV)
    lo = 0
    for n in cut:
        close(L.run([(n, lo, 1, pages_for(lo + n))], x[lo:lo + n], state), ref[lo:lo + n], 3e-5)
        lo += n
    assert lo == T


def test_linear_attention_activation_type_and_refusals(ops):
    L = Lin(ops, 3, 32, 48, [0.9, 0.99, 0.999], seed=4)
    x = rnd(70, L.desc.width, seed=5)
    ref = L.ref(x)
    state = torch.zeros(1, 3, 32, 48, device=DEV)
    close(L.run([(69, 0, 0, pages_for(69))], x[:69], state, torch.bfloat16), ref[:69], 8e-3)
    close(L.run([(1, 69, 0, pages_for(70))], x[69:], state, torch.bfloat16), ref[69:], 8e-3)
    st, keep = dev_step(ops, [(1, 0, 0, [0])])
    with pytest.raises(ops.SeqError, match="sums of squares"):
        ops.retention(x[:1].to(DEV), st, L.desc, state, torch.empty(1, 144, device=DEV), None)


# ---- selective scan ---------------------------------------------------------------------------------------------------------------------------
class Scan:
    def __init__(self, ops, C, N, R, seed=0, dt_mean=-2.0):
        self.ops, self.C, self.N, self.R = ops, C, N, R
        self.A = -torch.exp(torch.log(torch.arange(1, N + 1).float())[None] + 0.3 * rnd(C, N, seed=seed))
        self.D, self.dt_b, self.w_dt = rnd(C, seed=seed + 1), rnd(C, seed=seed + 2) + dt_mean, bf(rnd(C, R, seed=seed + 3, scale=R ** -0.5))
        self.dev = [(self.A.double() * math.log2(math.e)).float().to(DEV), self.D.to(DEV), self.dt_b.to(DEV), self.w_dt.to(DEV)]
        self.desc = ops.scan_desc(*self.dev)

    def inputs(self, T, seed):
        """u, [low | B | C] rows, gate"""
        return rnd(T, self.C, seed=seed), rnd(T, self.R + 2 * self.N, seed=seed + 1), rnd(T, self.C, seed=seed + 2)

    def ref(self, u, dbc, gate):
        R, N = self.R, self.N
        d = dbc.double()
        dt = torch.nn.functional.softplus(d[:, :R] @ self.w_dt.double().T + self.dt_b.double())
        return O.selective_scan(u.double(), dt, self.A.double(), d[:, R:R + N], d[:, R + N:], self.D.double()) * gate.double()

    def run(self, entries, u, dbc, gate, state, dtype=torch.float32):
        ops = self.ops
        st, keep = dev_step(ops, entries)
        T = u.shape[0]
        u, dbc = u.to(DEV).to(dtype).contiguous(), dbc.to(DEV).contiguous()
        wide = torch.full((T, self.C + 5), float("nan"), device=DEV)      # the gate is a part of a wider row
        wide[:, 3:3 + self.C] = gate.to(DEV)
        dtz = None
        if st.T != st.B:
            dtz = torch.empty(T, self.C, device=DEV)
            ops.linear(dbc[:, :self.R].contiguous(), self.dev[3], dtz)
        out = torch.full((T, self.C), float("nan"), device=DEV, dtype=dtype)
        scratch = torch.full((max(1, ops.scan_scratch_floats(st.T, st.B, self.C, self.N)),), float("nan"), device=DEV)
        ops.selective_scan(u, dbc, dtz, wide[:, 3:3 + self.C], st, self.desc, state, out, scratch)
        return out.float().cpu()


@pytest.mark.parametrize("C,N,R", [(64, 16, 8), (40, 24, 5), (130, 7, 3), (33, 1, 1), (96, 40, 16), (50, 64, 24), (20, 100, 8), (8, 256, 2), (256, 32, 32), (37, 12, 40)])
def test_scan_over_portions_and_single_tokens(ops, C, N, R):
    """two sequences share the steps, their slots hold another sequence's leftovers; portions around the segment size, of one and of two tokens"""
    S = Scan(ops, C, N, R, seed=10)
    n = {"a": 270, "b": 75}
    X = {s: S.inputs(k, 20 + 5 * i) for i, (s, k) in enumerate(n.items())}
    ref = {s: S.ref(*X[s]) for s in n}
    state = torch.full((3, C, N), 7.0, device=DEV)
    slot = {"a": 2, "b": 0}
    plan = [[("a", 65), ("b", 2)], [("b", 1), ("a", 1)], [("a", 2), ("b", 62)], [("b", 2), ("a", 1)], [("a", 64)], [("a", 1), ("b", 1)], [("a", 1)], [("b", 7), ("a", 135)]]
    fed = {"a": 0, "b": 0}
    for step in plan:
        cat = [torch.cat([X[s][j][fed[s]:fed[s] + k] for s, k in step]) for j in range(3)]
        got = S.run([(k, fed[s], slot[s], pages_for(fed[s] + k)) for s, k in step], *cat, state)
        o = 0
        for s, k in step:
            close(got[o:o + k], ref[s][fed[s]:fed[s] + k], 3e-5)
            fed[s] += k
            o += k
    assert fed == n and (state[1] == 7.0).all() and ops.error_flags() == 0


@pytest.mark.parametrize("dt_mean", [-9.0, 3.0, 25.0])
def test_scan_at_the_ends_of_the_step_size(ops, dt_mean):
    """steps so small that nothing decays over the sequence, and so large that every state but the newest is gone (beyond the range where softplus is the identity)"""
    S = Scan(ops, 48, 16, 8, seed=30, dt_mean=dt_mean)
    u, dbc, gate = S.inputs(150, 31)
    ref = S.ref(u, dbc, gate)
    state = torch.zeros(1, 48, 16, device=DEV)
    close(S.run([(131, 0, 0, pages_for(131))], u[:131], dbc[:131], gate[:131], state), ref[:131], 5e-5)
    for i in range(131, 150):
        close(S.run([(1, i, 0, pages_for(i + 1))], u[i:i + 1], dbc[i:i + 1], gate[i:i + 1], state), ref[i:i + 1], 5e-5)


@pytest.mark.parametrize("cut", [[700], [64, 2, 33, 400, 201], [699, 1]])
def test_scan_far_memory(ops, cut):
    """state 0 is written by the first token alone and read by the last alone, 700 tokens later, under a decay next to one"""
    C, N, R, T = 32, 8, 4, 700
    S = Scan(ops, C, N, R, seed=40, dt_mean=-4.0)
    S.A[:, 0] = -0.02
    S.dev[0].copy_((S.A.double() * math.log2(math.e)).float())
    S.D.zero_(), S.dev[1].zero_()
    u, dbc, gate = S.inputs(T, 41)
    dbc[1:, R] = 0.0
    dbc[0, R] = 300.0
    dbc[T - 1, R + N:] = 0.0
    dbc[T - 1, R + N] = 5.0
    ref = S.ref(u, dbc, gate)
    z = dbc[:1, :R].double() @ S.w_dt.double().T + S.dt_b.double()
    first = (torch.nn.functional.softplus(z) * u[:1].double())[0]
    assert torch.nn.functional.cosine_similarity(ref[-1] / gate[-1].double(), first, 0) > 0.9
    state = torch.full((2, C, N), 3.0, device=DEV)
    lo = 0
    for n in cut:
        close(S.run([(n, lo, 1, pages_for(lo + n))], u[lo:lo + n], dbc[lo:lo + n], gate[lo:lo + n], state), ref[lo:lo + n], 5e-5)
        lo += n


def test_scan_many_entries_and_activation_type(ops):
    S = Scan(ops, 72, 20, 6, seed=50)
    B = 9
    X = [S.inputs(9 + 3 * b, 51 + 7 * b) for b in range(B)]
    X = [(bf(u).float(), d, g) for u, d, g in X]
    state = torch.full((B, 72, 20), 2.0, device=DEV)
    out = S.run([(8 + 3 * b, 0, B - 1 - b, pages_for(9 + 3 * b)) for b in range(B)], *[torch.cat([x[j][:-1] for x in X]) for j in range(3)], state, torch.bfloat16)
    last = S.run([(1, 8 + 3 * b, B - 1 - b, pages_for(9 + 3 * b)) for b in range(B)], *[torch.cat([x[j][-1:] for x in X]) for j in range(3)], state, torch.bfloat16)
    o = 0
    for b in range(B):
        ref, k = S.ref(*X[b]), 8 + 3 * b
        close(out[o:o + k], ref[:-1], 6e-3)
        close(last[b:b + 1], ref[-1:], 6e-3)
        o += k


def test_scan_rejects_what_it_cannot_hold(ops):
    S = Scan(ops, 8, 4, 2)
    u, dbc, gate = (t.to(DEV) for t in S.inputs(100, 1))
    st, keep = dev_step(ops, [(100, 0, 0, pages_for(100))])
    state, out = torch.zeros(1, 8, 4, device=DEV), torch.empty(100, 8, device=DEV)
    with pytest.raises(ops.SeqError, match="step-size projection"):
        ops.selective_scan(u, dbc, None, gate, st, S.desc, state, out)
    with pytest.raises(ops.SeqError, match="work area"):
        ops.selective_scan(u, dbc, torch.zeros(100, 8, device=DEV), gate, st, S.desc, state, out)
    big = Scan(ops, 2, 300, 2)
    with pytest.raises(ops.SeqError, match="state size"):
        ops.selective_scan(u[:, :2].contiguous(), torch.zeros(100, 602, device=DEV), torch.zeros(100, 2, device=DEV), gate, st, big.desc, torch.zeros(1, 2, 300, device=DEV),
                           torch.empty(100, 2, device=DEV))


# ---- silu on a range of projected columns --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,dtype", [(1, torch.float32), (5, torch.bfloat16), (20, torch.float32), (20, torch.bfloat16), (70, torch.float32), (150, torch.bfloat16)])
@pytest.mark.parametrize("lo,hi", [(0, 0), (0, 130), (77, 201), (201, 300)])
def test_linear_with_silu_columns(ops, M, dtype, lo, hi):
    N, K = 300, 72
    x, w = rnd(M, K, seed=1).to(dtype), bf(rnd(N, K, seed=2, scale=K ** -0.5))
    y = torch.empty(M, N, device=DEV)
    ops.linear(x.to(DEV), w.to(DEV), y, silu=(lo, hi))
    ref = x.double() @ w.double().T
    ref[:, lo:hi] = O.silu(ref[:, lo:hi])
    close(y, ref, 1e-5)


# ---- router ----------------------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,groups,keep", [(8, 3, 4, 2), (6, 2, 3, 1), (12, 6, 2, 1), (9, 1, 9, 4), (64, 8, 8, 3), (5, 5, None, None), (7, 2, 7, 7)])
@pytest.mark.parametrize("T", [3, 40])
def test_router_groups_by_their_best_and_scores_as_weights(ops, E, top, groups, keep, T):
    scale, K = 1.7, 40
    x, w = rnd(T, K, seed=3), bf(rnd(E, K, seed=4, scale=3 * K ** -0.5))
    z = x.double() @ w.double().T
    r = {"experts": E, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups, "keep": keep}
    d = ops.route_desc(E, groups or 1, keep or 1, top, ops.ROUTE_SOFTMAX, group_best=1, renorm=False, scale=scale)
    ids, wts, zd = torch.empty(T * top, dtype=torch.int32, device=DEV), torch.empty(T * top, device=DEV), torch.empty(T, E, device=DEV)
    cnt = torch.full((E,), 99, dtype=torch.int32, device=DEV)
    ops.linear(x.to(DEV), w.to(DEV), zd)
    ops.moe_route_rule(zd, d, ids, wts, cnt)
    ref = [O.route(z[t], r) for t in range(T)]

    def check():
        for t in range(T):
            assert ids[t * top:(t + 1) * top].tolist() == ref[t][0]
            close(wts[t * top:(t + 1) * top], torch.tensor(ref[t][1]), 1e-5)
    check()
    assert torch.bincount(ids.cpu().long(), minlength=E).tolist() == cnt.tolist()
    if T <= 8:
        ids.fill_(-1), wts.zero_()
        ops.moe_router_rule(x.to(DEV), w.to(DEV), d, zd, ids, wts)
        check()


def test_router_group_score_is_the_largest_not_the_sum(ops):
    """group 0 holds the best expert and a bad one, group 1 two good ones: the largest counts, so group 0 is kept"""
    z = torch.tensor([[3.0, -5.0, 2.5, 2.5]])
    for best, want in ((1, [0, 1]), (2, [2, 3])):
        d = ops.route_desc(4, 2, 1, 2, ops.ROUTE_SOFTMAX, group_best=best, renorm=best == 2)
        ids, wts = torch.empty(2, dtype=torch.int32, device=DEV), torch.empty(2, device=DEV)
        ops.moe_route_rule(z.to(DEV), d, ids, wts, None)
        assert ids.tolist() == want
        close(wts, torch.softmax(z[0].double(), 0)[want] if best == 1 else torch.tensor([0.5, 0.5]), 1e-6)
    ids, wts = torch.empty(3, dtype=torch.int32, device=DEV), torch.empty(3, device=DEV)
    with pytest.raises(ops.SeqError, match="groups must divide"):
        ops.moe_route_rule(z.to(DEV), ops.route_desc(4, 2, 1, 3, ops.ROUTE_SOFTMAX, group_best=1), ids, wts, None)
    with pytest.raises(ops.SeqError, match="group's score"):
        ops.moe_route_rule(z.to(DEV), ops.route_desc(4, 2, 1, 2, ops.ROUTE_SOFTMAX, group_best=3), ids, wts, None)


# ---- residual of parallel layers ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W", [33, 48, 256, 1000, 1027, 4096, 8192])
@pytest.mark.parametrize("form", ["branches", "deferred", "plain", "experts", "sorted"])
def test_parallel_close(ops, W, form):
    T, eps, m = 9, 1e-3, 0.37
    x, y1, y2, y3 = (rnd(T, W, seed=i, scale=s) for i, s in ((1, 1.0), (2, 3.0), (3, 0.2), (4, 1.0)))
    w1, w2, fin, vec = (1 + 0.3 * rnd(W, seed=10 + i) for i in range(4))
    d = lambda t: t.to(DEV).contiguous()
    kw, mix, ff = {}, y1.double(), torch.zeros(T, W, dtype=F64)
    if form in ("branches", "experts", "sorted"):
        mix = 0.5 * O.rms_norm(y1.double(), eps, w1.double()) + 0.25 * O.rms_norm(y2.double(), eps, w2.double())
        kw.update(w_b1=d(w1), y2=d(y2), w_b2=d(w2), s1=0.5, s2=0.25)
    if form == "deferred":
        ss = rnd(T, 7, seed=5).abs()
        mix = y1.double() / torch.sqrt(ss.double().sum(1, keepdim=True) / 50 + eps)
        kw.update(sumsq=d(ss), sumsq_count=50)
    if form in ("branches", "deferred"):
        ff = y3.double()
        kw["y3"] = d(y3)
    if form in ("experts", "sorted"):
        top = 3
        ys, wts = rnd(T * top, W, seed=6), rnd(T * top, seed=7).abs()
        perm = torch.randperm(T * top, generator=torch.Generator().manual_seed(8)) if form == "sorted" else torch.arange(T * top)
        for t in range(T):
            for j in range(top):
                ff[t] += wts[t * top + j].double() * ys[perm[t * top + j]].double()
        kw.update(ys=d(ys), wts=d(wts), top=top, slot_of=d(perm.to(torch.int32)) if form == "sorted" else None)
    n = x.double() + m * (mix + ff)
    xo, ao = torch.empty(T, W, device=DEV), torch.empty(T, W, device=DEV)
    xd = d(x)
    ops.parallel_close(xd, d(y1), m, eps, x_out=xo, a_out=ao, fin_w=d(fin), **kw)
    close(xo, n, 3e-6)
    close(ao, O.rms_norm(n, eps, fin.double()), 5e-6)
    assert torch.equal(xd.cpu(), x)
    # a row added in front of a pass; in place; activation type; the final norm of some rows
    ab = torch.empty(T, W, device=DEV, dtype=torch.bfloat16)
    ops.parallel_close(xd, d(y1), m, eps, x_out=xd, a_out=ab, fin_w=d(fin), add_vec=d(vec), **kw)
    close(xd, n + vec.double(), 3e-6)
    close(ab.float(), O.rms_norm(n + vec.double(), eps, fin.double()), 8e-3)
    rows = torch.tensor([7, 2], dtype=torch.int32, device=DEV)
    a2 = torch.empty(2, W, device=DEV)
    ops.parallel_close(d(x), d(y1), m, eps, a_out=a2, fin_w=d(fin), rows=rows, **kw)
    close(a2, O.rms_norm(n, eps, fin.double())[[7, 2]], 5e-6)
    xo.zero_()
    ops.parallel_close(d(x), d(y1), m, eps, x_out=xo, **kw)
    close(xo, n, 3e-6)


@pytest.mark.parametrize("W", [6, 33, 64, 1024, 2052, 8192, 8200])
def test_embedding_without_positions(ops, W):
    T = 5
    table, ids = bf(rnd(20, W, seed=1)), torch.tensor([3, 19, 0, 3, 7], dtype=torch.int32)
    vec, fin = rnd(W, seed=2), 1 + 0.2 * rnd(W, seed=3)
    st, keep = dev_step(ops, [(T, 0, 0, [0])])
    x, x0, a = torch.empty(T, W, device=DEV), torch.empty(T, W, device=DEV), torch.empty(T, W, device=DEV)
    ops.embed_pos(table.to(DEV), ids.to(DEV), st, 1.5, None, x, 1e-4, x0=x0, add_vec=vec.to(DEV), fin_w=fin.to(DEV), a=a)
    e = table.double()[ids.long()] * 1.5
    close(x0, e, 1e-6)
    close(x, e + vec.double(), 1e-6)
    close(a, O.rms_norm(e + vec.double(), 1e-4, fin.double()), 2e-6)
    ab = torch.empty(T, W, device=DEV, dtype=torch.bfloat16)
    ops.embed_pos(table.to(DEV), ids.to(DEV), st, 1.0, None, x, 1e-4, a=ab)
    assert torch.equal(x.cpu(), table.float()[ids.long()]) and torch.equal(ab.cpu(), table[ids.long()])


# ---- windowed attention with biases ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,D,V,window", [(4, 2, 12, 20, 19), (6, 1, 24, 48, 33), (3, 3, 7, 5, 16), (2, 1, 40, 72, 1), (2, 2, 64, 32, 0)])
def test_windowed_attention_edges(ops, H, G, D, V, window):
    """every position has a key that answers one later query alone, placed just inside or just outside that query's window; scattered pages, portions
    and single tokens"""
    T, scale, bs = 120, 0.5, 16
    width = H * D + G * D + G * V
    x = rnd(T, width, seed=60) * 0.3
    bias = rnd(width, seed=61) * 0.3
    # the last tokens' queries point at one key each: the oldest visible one and the one before it
    edge = {100: 100 - window + 1, 101: 101 - window, 119: 119 - window + 1, 118: 118 - window} if window > 1 else {}
    for i, j in edge.items():
        u = rnd(D, seed=100 + i)
        for h in range(H):
            x[i, h * D:(h + 1) * D] = 2.0 * u - bias[h * D:(h + 1) * D]
        for g in range(G):
            x[j, H * D + g * D:H * D + (g + 1) * D] = 3.0 * u - bias[H * D + g * D:H * D + (g + 1) * D]
    b = (x + bias).double()
    q, k, v = b[:, :H * D].reshape(T, H, D), b[:, H * D:(H + G) * D].reshape(T, G, D), b[:, (H + G) * D:].reshape(T, G, V)
    ref = O.windowed_attention(q, k, v, scale, window).reshape(T, H * V)
    if edge:      # one window wider or narrower would show
        for other in (window - 1, window + 1):
            d = (O.windowed_attention(q, k, v, scale, other).reshape(T, H * V) - ref).abs().amax(1) / ref.abs().max()
            assert max(d[i].item() for i in edge) > 1e-2
    bd = bias.to(DEV)
    desc = ops.attn_desc(H, G, D, V, scale, gated=False, window=window, in_bias=bd)
    kp, vp = torch.full((12, bs, G, D), 9.0, device=DEV), torch.full((12, bs, G, V), 1e3, device=DEV)      # what earlier owners left
    pages = [7, 2, 11, 0, 5, 9, 3, 1]
    scratch = torch.empty(max([1] + [ops.attn_scratch_floats(t, 1, H, G, V, 128) for t in range(1, T + 1)]), device=DEV)
    lo = 0
    for n in [50, 2, 15, 1, 1, 30, 1, 1, 1, 2, 14, 1, 1]:
        st, keep = dev_step(ops, [(n, lo, 0, pages[:-(-(lo + n) // bs)])], bs)
        p, out = x[lo:lo + n].to(DEV).contiguous(), torch.empty(n, H * V, device=DEV)
        ops.attn_prep_ex(p, st, desc, kp, vp)
        ops.attn_ex(p, st, desc, kp, vp, out, scratch)
        close(out, ref[lo:lo + n], 2e-5)
        lo += n
    assert lo == T and ops.error_flags() == 0
