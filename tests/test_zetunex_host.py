"""Host side of the Zetunex design (no GPU): config.json -> generic specs, the order in which looped layers run, rejected configurations,
and the restatement the GPU tests compare with."""
import copy
import math

import pytest
import torch

import zetunex_oracle as O
from blazr_b200 import registry, zetunex
from blazr_b200.layered import AttentionSpec, DenseFfSpec, MoeFfSpec, RetentionSpec, ScanSpec, TwoBranchSpec, loop_runs


def cfg():
    moe = {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 6, "top": 3, "scale": 1.3, "groups": {"count": 3, "keep": 2}}}
    two = {"left": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3, "mask": {"size": 5}}, "right": {"inner": 20, "state": 6, "conv": 3, "dt_rank": 4}}
    return {"architecture": "Zetunex", "vocab": 61, "width": 40, "norm": {"eps": 1e-4}, "residual_mult": 0.6, "loop": {"start": 1, "stop": 3, "times": 3},
            "layers": [{"type": "lightning", "mixer": {"heads": 3, "dim": 10, "vdim": 7, "decay": [0.5, 0.9, 1.0]}, "mlp": {"kind": "dense", "ff": 56}},
                       {"type": "parallel", "mixer": two, "mlp": moe},
                       {"type": "lightning", "mixer": {"heads": 1, "dim": 4, "vdim": 9, "decay": [0.7]}, "mlp": None},
                       {"type": "parallel", "mixer": copy.deepcopy(two), "mlp": None}]}


def test_registered_and_mapped_onto_generic_specs():
    assert registry.LAYERED["Zetunex"] is zetunex.parse_config
    c = zetunex.parse_config(cfg())
    assert (c.layout, c.vocab, c.width, c.tied_head, c.eps, c.residual_mult, c.embed_scale, c.streams) == ("parallel", 61, 40, True, 1e-4, 0.6, 1.0, 1)
    assert [(l.kind, l.tensors, l.weights_of, l.enter) for l in c.layers] == [
        ("retention", 0, None, None), ("two_branch", 1, None, (False, 0)), ("retention", 2, None, None), ("two_branch", 1, 1, (False, 1)), ("retention", 2, 2, None),
        ("two_branch", 1, 1, (False, 2)), ("retention", 2, 2, None), ("two_branch", 3, None, None)]
    r = c.layers[0].mixer
    assert isinstance(r, RetentionSpec) and (r.heads, r.dim, r.vdim, r.decay) == (3, 10, 7, [0.5, 0.9, 1.0])
    assert (r.key_scale, r.qkv_silu, r.norm, r.gate, r.rot) == (1.0, True, "joint", "sigmoid", None)
    d = c.layers[0].ff
    assert isinstance(d, DenseFfSpec) and (d.ff, d.act, d.limit, d.alpha, d.up_shift) == (56, "swish_clamp", math.inf, 1.0, 0.0)
    m = c.layers[1].mixer
    assert isinstance(m, TwoBranchSpec) and (m.left_scale, m.right_scale, m.branch_norm) == (0.5, 0.5, True)
    a = m.left
    assert isinstance(a, AttentionSpec) and (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window) == (4, 2, 8, 12, 0.3, 5)
    assert a.bias and not a.out_bias and not a.gated and a.rot is None and a.qk_norm == "none" and not a.qk_unit_norm and not a.sink and not a.unit_sink and a.chunk == 0
    assert m.right == ScanSpec(inner=20, state=6, conv=3, dt_rank=4)
    f = c.layers[1].ff
    assert isinstance(f, MoeFfSpec) and (f.router, f.experts, f.top, f.ff, f.groups, f.keep, f.group_best, f.renorm, f.route_scale) == ("softmax", 6, 3, 12, 3, 2, 1, False, 1.3)
    assert (f.act, f.limit, f.alpha, f.up_shift, f.shared_ff, f.identity, f.correction) == ("swish_clamp", math.inf, 1.0, 0.0, 0, 0, False)
    assert c.layers[2].ff is None


@pytest.mark.parametrize("n,loop", [(4, (1, 3, 3)), (3, (0, 3, 2)), (5, (4, 5, 4)), (2, (0, 1, 1)), (3, None)])
def test_order_of_looped_layers(n, loop):
    runs = loop_runs(n, *(loop or (0, 0, 0)))
    ref = O.layer_order({"layers": [None] * n, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None})
    assert [(i, t if first else None) for i, t, first in runs] == ref


def test_optional_parts_may_be_absent():
    c = cfg()
    del c["loop"], c["layers"][1]["mlp"]["router"]["groups"], c["layers"][3]["mixer"]["left"]["mask"]
    p = zetunex.parse_config(c)
    assert len(p.layers) == 4 and all(l.enter is None and l.weights_of is None for l in p.layers) and p.layers[1].ff.groups == 1 and p.layers[3].mixer.left.window == 0
    c["loop"] = c["layers"][1]["mlp"]["router"]["groups"] = None
    assert len(zetunex.parse_config(c).layers) == 4


@pytest.mark.parametrize("edit,msg", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=2), "one value in"),
    (lambda c: c["layers"][0]["mixer"]["decay"].__setitem__(0, 1.5), "one value in"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "lacks 'vdim'"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "lacks 'scale'"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=-1), "must not be negative"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "lacks 'right'"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(conv=9), "convolution taps"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(state=0), "state must be positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=1), "router.groups"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "unknown feed-forward kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("times"), "lacks 'times'"),
    (lambda c: c.pop("residual_mult"), "lacks 'residual_mult'"),
    (lambda c: c.pop("norm"), "lacks 'norm'"),
])
def test_rejected_configurations(edit, msg):
    c = copy.deepcopy(cfg())
    edit(c)
    with pytest.raises(zetunex.ConfigError, match=msg):
        zetunex.parse_config(c)


def test_checkpoint_round_trip(tmp_path):
    from blazr_b200.safetensors_loader import load_checkpoint
    c = cfg()
    P = O.random_weights(c, seed=3)
    O.write_checkpoint(str(tmp_path), c, P)
    back, st = load_checkpoint(str(tmp_path))
    assert back == c and set(st.names()) == set(P) and all(torch.equal(st.tensor(n), P[n]) for n in P)


def test_restatement_is_causal_and_depends_on_every_earlier_token():
    c = cfg()
    P = O.random_weights(c, seed=1)
    t = torch.randint(0, 61, (12,), generator=torch.Generator().manual_seed(2)).tolist()
    a = O.forward(c, P, t)
    changed = list(t)
    changed[5] = (t[5] + 1) % 61
    b = O.forward(c, P, changed)
    assert torch.equal(a[:5], b[:5])
    assert ((a - b).abs().amax(-1)[5:] > 1e-6).all()


def test_restatement_against_other_forms():
    """the recurrences and masks written another way: decayed scores, unrolled products of decays, a masked soft-max over all keys"""
    g = torch.Generator().manual_seed(3)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    T = 9
    q, k, v, dec = r(T, 2, 5), r(T, 2, 5), r(T, 2, 4), [0.6, 0.95]
    got = O.decayed_linear_attention(q, k, v, dec)
    for h in range(2):
        for t in range(T):
            ref = sum(dec[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(got[t, h], ref)
    x, dt, A, B, C, D = r(T, 3), r(T, 3).abs(), -r(3, 4).abs(), r(T, 4), r(T, 4), r(3)
    y = O.selective_scan(x, dt, A, B, C, D)
    for t in range(T):
        for c in range(3):
            ref = D[c] * x[t, c]
            for j in range(t + 1):
                ref = ref + (torch.exp(A[c] * dt[j + 1:t + 1, c].sum()) * B[j] * C[t]).sum() * dt[j, c] * x[j, c]
            assert torch.allclose(y[t, c], ref)
    q, k, v = r(T, 4, 5), r(T, 2, 5), r(T, 2, 3)
    got = O.windowed_attention(q, k, v, 0.7, 4)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    mask = (j <= i) & (i - j < 4)
    for h in range(4):
        s = (q[:, h] @ k[:, h // 2].T * 0.7).masked_fill(~mask, float("-inf"))
        assert torch.allclose(got[:, h], torch.softmax(s, 1) @ v[:, h // 2])
    conv = O.causal_conv(r(T, 3), r(3, 4), r(3))
    assert conv.shape == (T, 3)


def test_restatement_of_the_choice():
    r = {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 1}}
    z = torch.tensor([1.0, -9.0, 0.9, 0.9, 0.0, 0.0], dtype=torch.float64)
    e, w = O.route(z, r)
    s = torch.softmax(z, 0)
    assert e == [0, 1] and w == pytest.approx([2 * s[0].item(), 2 * s[1].item()])
    assert O.route(z, {**r, "groups": None})[0] == [0, 2]
