"""The operators the Vodelix design added to libb200seq, each alone, against the plain float64 restatement in tests/vodelix_oracle.py:
the delta rule in its single-token and chunked forms (portions, reused slots, extreme decays, keys that repeat, a far memory), the
sinusoidal embedding, the norm on both sides of a sublayer with its additions, the token-dependent addition in both forms, exact gelu
and tanh on every projection path, the choice weighted over the chosen logits, attention with a constant one in the denominator."""
import numpy as np
import pytest
import torch

import vodelix_oracle as O

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


# ---- delta rule --------------------------------------------------------------------------------------------------------------------------
class Delta:
    """one layer's weights and its reference from a projection row r | k | v | gate | removal logits | low rank"""

    def __init__(self, ops, H, D, V, rank, seed=0, w0_mean=-1.0, a_mean=0.0, eps=1e-5, unit_eps=1e-6):
        self.H, self.D, self.V, self.rank, self.eps, self.unit_eps = H, D, V, rank, eps, unit_eps
        self.w2 = bf(rnd(H * D, rank, seed=seed, scale=rank ** -0.5))
        self.w0, self.a_b, self.nw = rnd(H * D, seed=seed + 1) + w0_mean, rnd(H * D, seed=seed + 2) * 0.5 + a_mean, 1 + 0.2 * rnd(H * V, seed=seed + 3)
        self.dev = [t.to(DEV).contiguous() for t in (self.w2, self.w0, self.a_b, self.nw)]
        self.scale = float(np.exp(-0.5))
        self.desc = ops.delta_desc(H, D, V, rank, *self.dev, self.scale, unit_eps, eps)
        self.ops = ops

    def rows(self, T, seed):
        return rnd(T, self.desc.width, seed=seed)

    def ref(self, proj):
        H, D, V, d = self.H, self.D, self.V, self.desc
        x = proj.double()
        cut = lambda c, n: x[:, c:c + n]
        hd = lambda t, n: t.reshape(-1, H, n)
        dec = hd(O.delta_decay(torch.tanh(cut(d.w_col, self.rank)) @ self.w2.double().T, self.w0.double()), D)
        rem = hd(torch.sigmoid(cut(d.a_col, H * D) + self.a_b.double()), D)
        r, k, v = hd(cut(d.r_col, H * D), D), hd(cut(d.k_col, H * D), D), hd(cut(d.v_col, H * V), V)
        o, S = zip(*[O.delta_scan(r[:, h], k[:, h], v[:, h], dec[:, h], rem[:, h], unit_eps=self.unit_eps) for h in range(H)])
        out = O.rms(torch.stack(o, 1), self.eps).reshape(-1, H * V) * self.nw.double() * torch.sigmoid(cut(d.g_col, H * V))
        return out, torch.stack(S)

    def run(self, entries, proj, state, dtype=torch.float32):
        st, keep = dev_step(self.ops, entries)
        p = proj.to(DEV).contiguous()
        T = p.shape[0]
        out = torch.empty(T, self.H * self.V, device=DEV, dtype=dtype)
        wz, scratch = None, None
        if st.T != st.B:
            low, wz = torch.empty(T, self.rank, device=DEV), torch.empty(T, self.H * self.D, device=DEV)
            self.ops.act(p[:, self.desc.w_col:], self.ops.ACT_TANH, low)
            self.ops.linear(low, self.dev[0], wz)
            scratch = torch.empty(self.ops.delta_scratch_floats(T, st.B, self.H, self.D, self.V), device=DEV)
            scratch.fill_(float("nan"))      # nothing of an earlier step may be read
        self.ops.delta(p, st, self.desc, wz, state, out, scratch)
        return out


@pytest.mark.parametrize("H,D,V,rank", [(2, 64, 64, 16), (3, 5, 5, 3), (2, 16, 24, 8), (1, 80, 72, 9), (2, 128, 128, 32), (1, 200, 70, 20), (5, 33, 7, 1), (1, 1, 3, 2)])
def test_delta_over_portions_and_single_tokens(ops, H, D, V, rank):
    """two sequences share the steps, their slots hold another sequence's leftovers; portions around the chunk size, of one and of two tokens"""
    L = Delta(ops, H, D, V, rank, seed=10)
    n = {"a": 171, "b": 74}
    X = {k: L.rows(v, 20 + i) for i, (k, v) in enumerate(n.items())}
    ref = {k: L.ref(X[k]) for k in n}
    state = torch.full((3, H, D, V), 7.0, device=DEV)
    slot = {"a": 2, "b": 0}
    plan = [[("a", 33), ("b", 2)], [("b", 1), ("a", 1)], [("a", 2), ("b", 31)], [("b", 32), ("a", 1)], [("a", 64)], [("a", 1), ("b", 1)], [("a", 1)], [("b", 7), ("a", 68)]]
    fed = {"a": 0, "b": 0}
    for step in plan:
        out = L.run([(k, fed[s], slot[s], pages_for(fed[s] + k)) for s, k in step], torch.cat([X[s][fed[s]:fed[s] + k] for s, k in step]), state)
        o = 0
        for s, k in step:
            close(out[o:o + k], ref[s][0][fed[s]:fed[s] + k], 3e-5)
            fed[s] += k
            o += k
    assert fed == n
    for s in n:
        close(state[slot[s]], ref[s][1], 1e-5)
    assert (state[1] == 7.0).all() and ops.error_flags() == 0


@pytest.mark.parametrize("w0,a", [(9.0, 0.0), (9.0, 6.0), (-14.0, 6.0), (-14.0, -6.0), (0.0, 9.0)])
def test_delta_at_the_ends_of_decay_and_removal(ops, w0, a):
    """decays at their smallest (a chunk's product falls to 1e-9) and next to one, removal rates next to zero and to one"""
    L = Delta(ops, 2, 48, 40, 6, seed=30, w0_mean=w0, a_mean=a)
    x = L.rows(150, 31)
    state = torch.zeros(1, 2, 48, 40, device=DEV)
    ref, S = L.ref(x)
    out = L.run([(131, 0, 0, pages_for(131))], x[:131], state)
    close(out, ref[:131], 3e-5)
    for i in range(131, 150):
        close(L.run([(1, i, 0, pages_for(i + 1))], x[i:i + 1], state), ref[i:i + 1], 3e-5)
    close(state[0], S, 2e-5)


def test_delta_with_keys_that_repeat(ops):
    """the same key in every token (the removed row is then the last value): the triangular system is as coupled as it gets"""
    L = Delta(ops, 1, 32, 32, 4, seed=40, w0_mean=-9.0, a_mean=5.0)
    x = L.rows(100, 41)
    c = L.desc.k_col
    x[:, c:c + 32] = x[:1, c:c + 32] + 0.02 * x[:, c:c + 32]
    ref, S = L.ref(x)
    state = torch.zeros(1, 1, 32, 32, device=DEV)
    close(L.run([(100, 0, 0, pages_for(100))], x, state), ref, 1e-4)
    close(state[0], S, 5e-5)


@pytest.mark.parametrize("cut", [[700], [64, 2, 33, 400, 201], [699, 1]])
def test_delta_far_memory(ops, cut):
    """one key of its own, 700 tokens back, under decays next to one: the last token's query reads that value and nothing else, so a state
    that was lost, decayed twice or taken from another chunk shows"""
    H, D, V = 1, 32, 16
    L = Delta(ops, H, D, V, 4, seed=50, w0_mean=-16.0, a_mean=-4.0)
    T = 700
    x = L.rows(T, 51) * 0.3
    d = L.desc
    x[:, d.k_col] = 0.0                       # channel 0 belongs to the first token alone
    x[0, d.k_col:d.k_col + D] = 0.0
    x[0, d.k_col] = 6.0
    x[0, d.v_col:d.v_col + V] = torch.linspace(-3, 3, V)
    x[T - 1, d.r_col:d.r_col + D] = 0.0
    x[T - 1, d.r_col] = 5.0
    ref, _ = L.ref(x)
    want = torch.linspace(-3, 3, V, dtype=F64)
    assert torch.nn.functional.cosine_similarity(ref[-1] / L.nw.double() / torch.sigmoid(x[-1, d.g_col:d.g_col + V].double()), want, 0) > 0.999
    state = torch.full((2, H, D, V), 3.0, device=DEV)
    lo = 0
    for n in cut:
        out = L.run([(n, lo, 1, pages_for(lo + n))], x[lo:lo + n], state)
        close(out, ref[lo:lo + n], 5e-5)
        lo += n


def test_delta_many_entries_and_activation_type(ops):
    L = Delta(ops, 4, 24, 24, 5, seed=60)
    B = 9
    X = [L.rows(3 + b, 61 + b) for b in range(B)]
    state = torch.full((B, 4, 24, 24), 2.0, device=DEV)
    out = L.run([(3 + b - 1, 0, B - 1 - b, pages_for(3 + b)) for b in range(B)], torch.cat([x[:-1] for x in X]), state)
    last = L.run([(1, 2 + b, B - 1 - b, pages_for(3 + b)) for b in range(B)], torch.cat([x[-1:] for x in X]), state, torch.bfloat16)
    o = 0
    for b in range(B):
        ref, S = L.ref(X[b])
        close(out[o:o + 2 + b], ref[:-1], 3e-5)
        close(last[b:b + 1].float(), ref[-1:], 6e-3)
        close(state[B - 1 - b], S, 1e-5)
        o += 2 + b


def test_delta_rejects_what_it_cannot_hold(ops):
    L = Delta(ops, 1, 8, 8, 2, seed=70)
    st, keep = dev_step(ops, [(4, 0, 0, [0])])
    x, out, state = L.rows(4, 71).to(DEV), torch.empty(4, 8, device=DEV), torch.zeros(1, 1, 8, 8, device=DEV)
    with pytest.raises(ops.SeqError, match="work area"):
        ops.delta(x, st, L.desc, torch.zeros(4, 8, device=DEV), state, out, None)
    with pytest.raises(ops.SeqError, match="low-rank"):
        ops.delta(x, st, L.desc, None, state, out, torch.zeros(100000, device=DEV))
    L.desc.decay_scale = 3.0
    with pytest.raises(ops.SeqError, match="decay scale"):
        ops.delta(x, st, L.desc, torch.zeros(4, 8, device=DEV), state, out, torch.zeros(100000, device=DEV))


# ---- embedding -----------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W", [44, 33, 1026])
def test_sinusoidal_embedding(ops, W):
    table = bf(rnd(17, W, seed=80))
    ids = torch.tensor([3, 16, 0, 5, 5, 9], dtype=torch.int32)
    st, keep = dev_step(ops, [(4, 0, 0, [0]), (1, 40, 1, pages_for(41)), (1, 3001, 2, pages_for(3002))])
    pos = [0, 1, 2, 3, 40, 3001]
    ref = torch.stack([table.double()[int(i)] + O.sinusoid(p, W) for i, p in zip(ids, pos)])
    add, w = rnd(W, seed=81), 1 + 0.2 * rnd(W, seed=82)
    x, x0, a = (torch.empty(6, W, device=DEV) for _ in range(3))
    f = ops.position_frequencies(W, 10000.0).to(DEV)
    ops.embed_pos(table.to(DEV), ids.to(DEV), st, 1.0, f, x, 1e-3, x0=x0, add_vec=add.to(DEV), fin_w=w.to(DEV), a=a)
    close(x0, ref, 3e-7)
    close(x, ref + add.double(), 3e-7)
    close(a, O.rms(ref + add.double(), 1e-3) * w.double(), 2e-6)
    ab = torch.empty(6, W, device=DEV, dtype=torch.bfloat16)
    ops.embed_pos(table.to(DEV), ids.to(DEV), st, 1.5, f, x, 1e-3, a=ab)
    close(x, ref + 0.5 * table.double()[ids.long()], 3e-7)
    assert torch.equal(ab, x.to(torch.bfloat16))


# ---- norms on both sides ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W", [44, 33, 512, 1024, 4100, 8192, 9000])
@pytest.mark.parametrize("R", [3, 90])
def test_sandwich_norm(ops, W, R):
    eps = 1e-2
    x, y, ar = rnd(R, W, seed=90), rnd(R, W, seed=91, scale=0.1), rnd(R, W, seed=92)
    w, fw, av = 1 + 0.3 * rnd(W, seed=93), 1 + 0.3 * rnd(W, seed=94), rnd(W, seed=95)
    d = lambda t: t.to(DEV)
    base = x.double() + O.rms(y.double(), eps) * w.double()
    out, a = torch.empty(R, W, device=DEV), torch.empty(R, W, device=DEV, dtype=torch.bfloat16)
    ops.sandwich_norm(d(x), eps, y=d(y), w=d(w), x_out=out, a_out=a, fin_w=d(fw))
    close(out, base, 1e-6)
    close(a.float(), O.rms(base, eps) * fw.double(), 6e-3)
    full = base + ar.double() + av.double()
    xi = d(x)
    a32 = torch.empty(R, W, device=DEV)
    ops.sandwich_norm(xi, eps, y=d(y), w=d(w), add_row=d(ar), add_vec=d(av), x_out=xi, a_out=a32, fin_w=d(fw))       # in place
    close(xi, full, 1e-6)
    close(a32, O.rms(full, eps) * fw.double(), 2e-6)
    rows = torch.tensor([2, 0], dtype=torch.int32)
    g = torch.empty(2, W, device=DEV)
    ops.sandwich_norm(d(x), eps, y=d(y), w=d(w), a_out=g, fin_w=d(fw), rows=d(rows))
    close(g, (O.rms(base, eps) * fw.double())[rows.long()], 2e-6)
    ops.sandwich_norm(d(x), eps, add_vec=d(av), a_out=a32)                                                           # no result, no norm behind
    close(a32, x.double() + av.double(), 1e-6)


@pytest.mark.parametrize("W,dim,layer", [(44, 5, 2), (40, 8, 0), (1024, 16, 1), (96, 24, 3)])
def test_token_dependent_addition_in_both_forms(ops, W, dim, layer):
    eps, T, n = 1e-3, 5, 4
    P = {"side.embed": bf(rnd(13, n * dim, seed=100)), f"l{layer}.side.gate": bf(rnd(dim, W, seed=101, scale=1.5 * W ** -0.5)),
         f"l{layer}.side.proj": bf(rnd(W, dim, seed=102, scale=dim ** -0.5)), f"l{layer}.side.norm": 1 + 0.2 * rnd(W, seed=103)}
    toks = [12, 0, 7, 7, 3]
    ids = torch.tensor(toks, dtype=torch.int32, device=DEV)
    x, y, w, ar, av, fw = rnd(T, W, seed=104), rnd(T, W, seed=105), 1 + 0.2 * rnd(W, seed=106), rnd(T, W, seed=107), rnd(W, seed=108), 1 + 0.2 * rnd(W, seed=109)
    n1 = x.double() + O.rms(y.double(), eps) * w.double()
    ref = O.token_side(n1, toks, {k: v.double() for k, v in P.items()}, layer, dim, eps) + ar.double() + av.double()
    d = {k: v.to(DEV).contiguous() for k, v in P.items()}
    gate, proj, table, sw = d[f"l{layer}.side.gate"], d[f"l{layer}.side.proj"], d["side.embed"], d[f"l{layer}.side.norm"]
    dv = lambda t: t.to(DEV)
    x_out, a = torch.empty(T, W, device=DEV), torch.empty(T, W, device=DEV)
    ops.side_close(dv(x), dv(y), dv(w), eps, gate, proj, table, layer * dim, ids, sw, add_row=dv(ar), add_vec=dv(av), x_out=x_out, a_out=a, fin_w=dv(fw))
    close(x_out, ref, 3e-6)
    close(a, O.rms(ref, eps) * fw.double(), 5e-6)
    rows = torch.tensor([4, 1], dtype=torch.int32, device=DEV)
    g = torch.empty(2, W, device=DEV)
    ops.side_close(dv(x), dv(y), dv(w), eps, gate, proj, table, layer * dim, ids, sw, add_row=dv(ar), add_vec=dv(av), rows=rows, a_out=g, fin_w=dv(fw))
    close(g, (O.rms(ref, eps) * fw.double())[[4, 1]], 5e-6)
    z, sg, y2 = torch.empty(T, dim, device=DEV), torch.empty(T, dim, device=DEV), torch.empty(T, W, device=DEV)
    n1d = n1.float().to(DEV)
    ops.linear(n1d, gate, z)
    ops.token_gate(z, table, layer * dim, ids, sg)
    ops.linear(sg, proj, y2)
    ops.sandwich_norm(n1d, eps, y=y2, w=sw, add_row=dv(ar), add_vec=dv(av), x_out=x_out)
    close(x_out, ref, 3e-6)


# ---- activations and router ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind,ref", [("gelu_erf", O.gelu_erf), ("tanh", torch.tanh), ("relu2", O.relu_squared)])
def test_plain_activations_on_every_projection_path(ops, kind, ref):
    K, N = 64, 48
    w = bf(rnd(N, K, seed=110, scale=2 * K ** -0.5))
    for T, dt in ((1, torch.float32), (6, torch.bfloat16), (70, torch.bfloat16)):
        x = rnd(T, K, seed=111).to(dt)
        out = torch.empty(T, N, device=DEV)
        ops.linear_act(x.to(DEV), w.to(DEV), ops.ACT_KINDS[kind], out)
        close(out, ref(x.double() @ w.double().T), 2e-5 if dt == torch.float32 else 1e-4)
    z = rnd(9, N + 4, seed=112, scale=2.0)
    out = torch.empty(9, N, device=DEV)
    ops.act(z.to(DEV)[:, :N], ops.ACT_KINDS[kind], out)
    close(out, ref(z[:, :N].double()), 1e-6)
    # experts: per-pair rows, exact tiles, tensor-core tiles
    E = 3
    we = bf(rnd(E, N, K, seed=113, scale=2 * K ** -0.5))
    for T, dt in ((4, torch.float32), (80, torch.float32), (80, torch.bfloat16)):
        x = rnd(T, K, seed=114).to(dt)
        ids = torch.randint(0, E, (T,), generator=torch.Generator().manual_seed(115)).to(torch.int32)
        want = ref(torch.stack([x[t].double() @ we[int(ids[t])].double().T for t in range(T)]))
        out = torch.empty(T, N, device=DEV)
        xd, idd = x.to(DEV), ids.to(DEV)
        if T <= 8:
            ops.moe_linear(xd, 1, we.to(DEV), idd, None, None, T, ops.ACT_KINDS[kind], out)
            close(out, want, 2e-5)
            continue
        cnt = torch.bincount(ids.long(), minlength=E).to(torch.int32).to(DEV)
        offs, order, slot = torch.zeros(E + 1, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV)
        ops.moe_sort(idd, T, E, cnt, offs, order, slot)
        if dt == torch.bfloat16:
            xs = torch.empty(T, K, device=DEV, dtype=dt)
            ops.moe_gather(xd, 1, order, T, xs)
            ops.moe_linear(xs, 0, we.to(DEV), idd, order, offs, T, ops.ACT_KINDS[kind], out)
        else:
            ops.moe_linear(xd, 1, we.to(DEV), idd, order, offs, T, ops.ACT_KINDS[kind], out)
        close(out[slot.long()], want, 1e-4)


@pytest.mark.parametrize("E,top", [(5, 2), (40, 7), (3, 3), (9, 1)])
@pytest.mark.parametrize("spread", [1.0, 80.0])
def test_choice_weighted_over_the_chosen_logits(ops, E, top, spread):
    """spread 80: a soft-max over ALL logits would leave most of them zero and the order among those unknown"""
    T, K = 7, 32
    x, w = rnd(T, K, seed=120), bf(rnd(E, K, seed=121, scale=spread * K ** -0.5))
    z = x @ w.float().T
    ids, wts = torch.empty(T * top, dtype=torch.int32, device=DEV), torch.empty(T * top, device=DEV)
    for fused in (False, True):
        if fused:
            zz = torch.empty(T, E, device=DEV)
            ops.moe_router_ex(x.to(DEV), w.to(DEV), E, 1, 1, top, ops.ROUTE_TOP_SOFTMAX, None, zz, ids, wts)
        else:
            ops.moe_route_ex(z.to(DEV), E, 1, 1, top, ops.ROUTE_TOP_SOFTMAX, None, ids, wts, None)
        for t in range(T):
            i, c = O.route(z[t].double(), top)
            assert ids[t * top:(t + 1) * top].tolist() == i
            assert (wts[t * top:(t + 1) * top].cpu().double() - c).abs().max() < 1e-4 * (1 if spread == 1.0 else 10)


# ---- attention with a constant one in the denominator ---------------------------------------------------------------------------------------------
def attention_setup(ops, H, G, D, V, scale, T, seed):
    x = rnd(T, H * D + G * D + G * V, seed=seed)
    nq, nk = 1 + 0.3 * rnd(H * D, seed=seed + 1), 1 + 0.3 * rnd(G * D, seed=seed + 2)
    dev = dict(q=nq.to(DEV), k=nk.to(DEV), s=torch.zeros(H, device=DEV))
    desc = ops.attn_desc(H, G, D, V, scale, gated=False, qk_eps=1e-4, sink=dev["s"], q_norm_w=dev["q"], k_norm_w=dev["k"], norm_full=True)
    return x, nq, nk, desc, dev


def attention_ref(x, nq, nk, H, G, D, V, scale):
    T = x.shape[0]
    q = (O.rms(x[:, :H * D].double(), 1e-4) * nq.double()).reshape(T, H, D)
    k = (O.rms(x[:, H * D:(H + G) * D].double(), 1e-4) * nk.double()).reshape(T, G, D)
    return O.attend_with_unit_sink(q, k, x[:, (H + G) * D:].double().reshape(T, G, V), scale).reshape(T, H * V)


def attention_run(ops, desc, entries, x, kp, vp, H, V):
    st, keep = dev_step(ops, entries)
    p = x.to(DEV).contiguous()
    out = torch.empty(p.shape[0], H * V, device=DEV)
    n = ops.attn_scratch_floats(st.T, st.B, H, desc.G, V, st.max_blocks * st.block_size)
    scratch = torch.empty(max(n, 1), device=DEV)
    ops.attn_prep_ex(p, st, desc, kp, vp)
    ops.attn_ex(p, st, desc, kp, vp, out, scratch)
    return out


@pytest.mark.parametrize("H,G,D,V,scale", [(4, 1, 24, 32, 0.2), (6, 3, 10, 6, 0.5), (2, 2, 80, 64, 0.1), (3, 1, 7, 5, 0.3)])
def test_attention_over_shuffled_pages(ops, H, G, D, V, scale):
    T = 100
    x, nq, nk, desc, keep = attention_setup(ops, H, G, D, V, scale, T, 130)
    ref = attention_ref(x, nq, nk, H, G, D, V, scale)
    bt = torch.randperm(9, generator=torch.Generator().manual_seed(1)).tolist()
    kp, vp = torch.full((9, 16, G, D), 9.0, device=DEV), torch.full((9, 16, G, V), 9.0, device=DEV)
    lo = 0
    for n in (1, 2, 15, 47, 1, 30, 1, 1, 1, 1):      # portions across page borders and single tokens
        close(attention_run(ops, desc, [(n, lo, 0, bt)], x[lo:lo + n], kp, vp, H, V), ref[lo:lo + n], 2e-5)
        lo += n
    assert lo == T and ops.error_flags() == 0


@pytest.mark.parametrize("far", [0, 15, 16, 63, 64, 511])
def test_a_far_key_among_hundreds_and_the_one_in_the_denominator(ops, far):
    """one key stands out for the last token's query (score about 9, all others below zero): its value must come through, times e / (1 + e + rest);
    decoded alone (split keys) and inside a portion"""
    H, G, D, V, scale, T = 2, 1, 16, 8, 0.5, 600
    x, nq, nk, desc, keep = attention_setup(ops, H, G, D, V, scale, T, 140)
    nq.fill_(1.0), nk.fill_(1.0), keep["q"].fill_(1.0), keep["k"].fill_(1.0)
    q, k = x[:, :H * D].reshape(T, H, D), x[:, H * D:H * D + D]
    k[:] = 0.0
    k[:, 1:] = rnd(T, D - 1, seed=143)
    k[:, 0] = -1.0
    k[far] = 0.0
    k[far, 0] = 3.0
    q[T - 1] = 0.0
    q[T - 1, :, 0] = 2.0
    x[:, :H * D], x[:, H * D:H * D + D] = q.reshape(T, H * D), k
    ref = attention_ref(x, nq, nk, H, G, D, V, scale)
    v = x[far, H * D + D:].double()
    assert torch.nn.functional.cosine_similarity(ref[-1, :V], v, 0) > 0.97
    for cut in ([T - 1, 1], [T - 40, 40]):
        kp, vp = torch.zeros(38, 16, G, D, device=DEV), torch.zeros(38, 16, G, V, device=DEV)
        lo = 0
        for n in cut:
            out = attention_run(ops, desc, [(n, lo, 0, pages_for(T))], x[lo:lo + n], kp, vp, H, V)
            lo += n
        close(out[-1:], ref[-1:], 2e-5)


def test_the_one_dominates_when_all_scores_are_low(ops):
    """scores far below zero: without the added one the weights would sum to one, with it the result is nearly nothing"""
    H, G, D, V, T = 1, 1, 8, 4, 40
    x, nq, nk, desc, keep = attention_setup(ops, H, G, D, V, 3.0, T, 150)
    x[:, :D] = 1.0 + 0.01 * x[:, :D]
    x[:, D:2 * D] = -1.0 + 0.01 * x[:, D:2 * D]
    ref = attention_ref(x, nq, nk, H, G, D, V, 3.0)
    assert ref.abs().max() < 1e-4
    kp, vp = torch.zeros(3, 16, G, D, device=DEV), torch.zeros(3, 16, G, V, device=DEV)
    close(attention_run(ops, desc, [(39, 0, 0, pages_for(T))], x[:39], kp, vp, H, V), ref[:39], 1e-4)
    close(attention_run(ops, desc, [(1, 39, 0, pages_for(T))], x[39:], kp, vp, H, V), ref[39:], 1e-4)
