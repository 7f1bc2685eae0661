"""Host side of the Vodelix design (no GPU): config.json -> generic specs, the order in which looped layers run, position frequencies,
rejected configurations, and the restatement the GPU tests compare with."""
import copy
import math

import numpy as np
import pytest
import torch

import vodelix_oracle as O
from blazr_b200 import registry, seqops, vodelix
from blazr_b200.layered import AttentionSpec, DeltaSpec, DenseFfSpec, MoeFfSpec


def cfg():
    moe = {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 20}}
    return {"architecture": "Vodelix", "vocab": 61, "width": 40, "norm": {"eps": 1e-4}, "token_side": {"dim": 6}, "loop": {"start": 1, "stop": 3, "times": 3},
            "layers": [{"type": "general_delta", "mixer": {"heads": 3, "dim": 10}, "mlp": {"kind": "dense", "ff": 56}},
                       {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3}, "mlp": moe},
                       {"type": "general_delta", "mixer": {"heads": 2, "dim": 7}, "mlp": None},
                       {"type": "attention", "mixer": {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 5, "scale": 0.5}, "mlp": None}]}


def test_registered_and_mapped_onto_generic_specs():
    assert registry.LAYERED["Vodelix"] is vodelix.parse_config
    c = vodelix.parse_config(cfg())
    assert (c.layout, c.vocab, c.width, c.tied_head, c.eps, c.norm_shift, c.position_base, c.token_side, c.embed_scale) == ("sandwich", 61, 40, True, 1e-4, 1.0, 10000.0, 6, 1.0)
    assert [(l.kind, l.tensors, l.weights_of, l.enter) for l in c.layers] == [
        ("delta", 0, None, None), ("attention", 1, None, (False, 0)), ("delta", 2, None, None), ("attention", 1, 1, (True, 1)), ("delta", 2, 2, None),
        ("attention", 1, 1, (True, 2)), ("delta", 2, 2, None), ("attention", 3, None, None)]
    d, a = c.layers[0], c.layers[1]
    assert isinstance(d.mixer, DeltaSpec) and (d.mixer.heads, d.mixer.dim, d.mixer.vdim, d.mixer.unit_eps) == (3, 10, 10, 1e-6)
    assert math.isclose(d.mixer.decay_scale, math.exp(-0.5)) and isinstance(d.ff, DenseFfSpec) and (d.ff.act, d.ff.ff) == ("relu2", 56)
    m = a.mixer
    assert isinstance(m, AttentionSpec) and (m.heads, m.kv_heads, m.dim, m.vdim, m.scale) == (4, 2, 8, 12, 0.3)
    assert m.unit_sink and not m.sink and m.rot is None and m.qk_norm == "full" and not m.gated and not m.bias and m.window == 0 and m.chunk == 0
    f = a.ff
    assert isinstance(f, MoeFfSpec) and (f.router, f.experts, f.top, f.ff, f.act, f.shared_ff, f.shared_gate, f.correction, f.identity) == ("top_softmax", 5, 2, 12, "gelu_erf", 20, False, False, 0)
    assert c.layers[2].ff is None


@pytest.mark.parametrize("n,loop", [(4, {"start": 1, "stop": 3, "times": 3}), (3, {"start": 0, "stop": 3, "times": 2}), (5, {"start": 4, "stop": 5, "times": 4}), (2, {"start": 0, "stop": 1, "times": 1}), (3, None)])
def test_order_of_looped_layers(n, loop):
    runs = vodelix.layer_runs(n, loop)
    ref = O.layer_runs({"layers": [None] * n, "loop": loop})
    assert [(i, t) for i, t, _ in runs] == ref
    assert [first for _, _, first in runs] == [t is not None and i == loop["start"] for i, t in ref]


def test_optional_parts_may_be_absent():
    c = cfg()
    del c["loop"], c["token_side"], c["layers"][1]["mlp"]["shared"]
    p = vodelix.parse_config(c)
    assert len(p.layers) == 4 and p.token_side == 0 and all(l.enter is None and l.weights_of is None for l in p.layers) and p.layers[1].ff.shared_ff == 0
    c["loop"] = c["token_side"] = None
    assert len(vodelix.parse_config(c).layers) == 4


@pytest.mark.parametrize("edit,msg", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "lacks 'scale'"),
    (lambda c: c["layers"][0]["mixer"].update(dim=0), "dim must be positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "router.top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "unknown feed-forward kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("times"), "lacks 'times'"),
    (lambda c: c["token_side"].pop("dim"), "lacks 'dim'"),
    (lambda c: c.pop("norm"), "lacks 'norm'"),
])
def test_rejected_configurations(edit, msg):
    c = copy.deepcopy(cfg())
    edit(c)
    with pytest.raises(vodelix.ConfigError, match=msg):
        vodelix.parse_config(c)


@pytest.mark.parametrize("W", [8, 33, 300])
def test_position_frequencies_in_two_parts(W):
    f = seqops.position_frequencies(W, 10000.0).double().numpy()
    want = 10000.0 ** (-2.0 * np.arange((W + 1) // 2) / W)
    assert f.shape == (2, (W + 1) // 2)
    np.testing.assert_allclose(f[0] + f[1], want, rtol=1e-13)
    np.testing.assert_allclose(f[0], want, rtol=1e-7)


def test_restatement_is_causal_and_depends_on_every_earlier_token():
    c = cfg()
    P = O.random_model(c, seed=1)
    t = torch.randint(0, 61, (12,), generator=torch.Generator().manual_seed(2)).tolist()
    a = O.forward(c, P, t)
    changed = list(t)
    changed[5] = (t[5] + 1) % 61
    b = O.forward(c, P, changed)
    assert torch.equal(a[:5], b[:5])
    assert ((a - b).abs().amax(-1)[5:] > 1e-6).all()


def test_restatement_against_the_textbook_forms():
    """the masked sums written another way: soft-max with one more key of score zero and value zero; the delta rule as a product of transition matrices"""
    g = torch.Generator().manual_seed(3)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v = r(6, 1, 5), r(6, 1, 5), r(6, 1, 4)
    got = O.attend_with_unit_sink(q, k, v, 0.7)
    for i in range(6):
        s = torch.cat([torch.zeros(1, dtype=torch.float64), (k[:i + 1, 0] @ q[i, 0]) * 0.7])
        assert torch.allclose(got[i, 0], torch.softmax(s, 0)[1:] @ v[:i + 1, 0])
    D = 4
    rr, kk, vv, w, a = r(5, D), r(5, D), r(5, 3), torch.rand(5, D, generator=g, dtype=torch.float64), torch.rand(5, D, generator=g, dtype=torch.float64)
    out, S = O.delta_scan(rr, kk, vv, w, a)
    M = torch.zeros(D, 3, dtype=torch.float64)
    for t in range(5):
        u = kk[t] / torch.sqrt((kk[t] ** 2).sum() + 1e-6)
        M = (torch.diag(w[t]) - torch.outer(a[t] * u, u)) @ M + torch.outer(kk[t], vv[t])
        assert torch.allclose(out[t], M.T @ rr[t])
    assert torch.allclose(S, M)
