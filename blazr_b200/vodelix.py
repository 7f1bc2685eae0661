"""Vodelix: a decoder-only design whose sublayers are normed on both sides (x <- x + norm(f(norm(x))), RMS norms with weights stored around
zero).  Its mixers are soft-max attention without positions in the scores (one weighted RMS norm over the whole query and key projections, a
constant one in the soft-max denominator) or a delta rule with a decay and a removal rate per key channel.  The feed-forward is dense
(squared relu) or a mixture of exact-gelu experts weighted by the soft-max over the chosen router logits, with a shared expert.  Positions
enter as a sinusoid added to the embedding; every layer adds a gated, projected row of a per-token table; a span of layers may run several
times with the same weights, each pass with a cache or state of its own.

This module only reads the design's config.json and maps it onto the generic specs of blazr_b200/layered.py (layout "sandwich"); the
mechanisms and their kernels are shared with any other layer-list design:

    config key                              -> spec
    vocab, width                            -> LayeredConfig.vocab / width (one residual stream, output projection = embedding table)
    norm.eps                                -> eps of every RMS norm (layer, q / k, head, token addition); LayeredConfig.norm_shift = 1
    token_side.dim                          -> LayeredConfig.token_side (0: none)
    loop.start / stop / times               -> the span's layers are listed `times` times; a repeated run names its layer's tensors (LayerSpec.tensors),
                                               borrows the weights of the first run (weights_of) and keeps a cache / state of its own; the first
                                               layer of each pass carries LayerSpec.enter = (pass > 0: the embedding output is added, row of loop.step)
    layers[i].type = "attention"            -> AttentionSpec(qk_norm "full", unit_sink, no rotation)
    layers[i].type = "general_delta"        -> DeltaSpec(heads, dim, vdim = dim, decay_scale exp(-1/2), unit_eps 1e-6); the rank of the low-rank decay
                                               branch is the shape of mix.w1
    layers[i].mlp = null                    -> no feed-forward sublayer
    layers[i].mlp.kind = "dense"            -> DenseFfSpec(ff, act "relu2")
    layers[i].mlp.kind = "moe"              -> MoeFfSpec(router "top_softmax", router.experts / top, expert.ff, act "gelu_erf", shared.ff without a token gate)

Tensor names: embed, final.norm, loop.step, side.embed, l<i>.{norm1,norm1b,norm2,norm2b}, attention l<i>.mix.{q,k,v,o,q.norm,k.norm}, delta rule
l<i>.mix.{r,k,v,g,a,a.b,w1,w2,w0,norm,o}, l<i>.mlp.{up,down}, l<i>.mlp.router, l<i>.mlp.e<j>.{up,down}, l<i>.mlp.shared.{up,down},
l<i>.side.{gate,proj,norm}.
"""
from __future__ import annotations

import math

from .layered import AttentionSpec, DeltaSpec, DenseFfSpec, LayeredConfig, LayerSpec, MoeFfSpec, loop_runs

ARCHITECTURE = "Vodelix"
POSITION_BASE = 10000.0
DECAY_SCALE = math.exp(-0.5)
KEY_UNIT_EPS = 1e-6
DENSE_ACT = "relu2"
EXPERT_ACT = "gelu_erf"


class ConfigError(ValueError):
    pass


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise ConfigError(f"config: {where} lacks '{key}'")
    return d[key]


def _size(d, key: str, where: str) -> int:
    n = int(_need(d, key, where))
    if n < 1:
        raise ConfigError(f"config: {where}: {key} must be positive")
    return n


def _mixer(kind: str, m: dict, where: str):
    """(spec kind, spec)"""
    if kind == "attention":
        spec = AttentionSpec(heads=_size(m, "heads", where), kv_heads=_size(m, "kv_heads", where), dim=_size(m, "dim", where), vdim=_size(m, "vdim", where),
                             scale=float(_need(m, "scale", where)), qk_unit_norm=False, gated=False, qk_norm="full", unit_sink=True)
        if spec.heads % spec.kv_heads:
            raise ConfigError(f"config: {where}: heads is not a multiple of kv_heads")
        return "attention", spec
    if kind == "general_delta":
        dim = _size(m, "dim", where)
        return "delta", DeltaSpec(heads=_size(m, "heads", where), dim=dim, vdim=dim, decay_scale=DECAY_SCALE, unit_eps=KEY_UNIT_EPS)
    raise ConfigError(f"config: {where}: unknown layer type '{kind}'")


def _feed_forward(mlp, where: str):
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        return DenseFfSpec(ff=_size(mlp, "ff", where), act=DENSE_ACT)
    if kind == "moe":
        r, ex, shared = _need(mlp, "router", where), _need(mlp, "expert", where), mlp.get("shared")
        spec = MoeFfSpec(experts=_size(r, "experts", where + ".router"), top=_size(r, "top", where + ".router"), ff=_size(ex, "ff", where + ".expert"), act=EXPERT_ACT,
                         router="top_softmax", shared_ff=_size(shared, "ff", where + ".shared") if shared is not None else 0, shared_gate=False)
        if spec.top > spec.experts:
            raise ConfigError(f"config: {where}: router.top must lie between 1 and router.experts")
        return spec
    raise ConfigError(f"config: {where}: unknown feed-forward kind '{kind}'")


def layer_runs(n: int, loop) -> list:
    """(layer, pass or None outside the loop, first layer of its pass) in the order they run"""
    if loop is None:
        return loop_runs(n)
    start, stop, times = (int(_need(loop, k, "loop")) for k in ("start", "stop", "times"))
    if not (0 <= start < stop <= n) or times < 1:
        raise ConfigError("config: loop: 0 <= start < stop <= number of layers, times >= 1")
    return loop_runs(n, start, stop, times)


def parse_config(cfg: dict) -> LayeredConfig:
    side = cfg.get("token_side")
    out = LayeredConfig(name=ARCHITECTURE, vocab=_size(cfg, "vocab", "top level"), width=_size(cfg, "width", "top level"), streams=1, norm_groups=1,
                        eps=float(_need(_need(cfg, "norm", "top level"), "eps", "norm")), canon_taps=0, embed_scale=1.0, layout="sandwich", tied_head=True,
                        depth_average=False, norm_shift=1.0, position_base=POSITION_BASE, token_side=_size(side, "dim", "token_side") if side is not None else 0)
    layers = []
    for i, lay in enumerate(_need(cfg, "layers", "top level")):
        where = f"layers[{i}]"
        kind, spec = _mixer(_need(lay, "type", where), _need(lay, "mixer", where), where + ".mixer")
        layers.append((kind, spec, _feed_forward(lay.get("mlp"), where + ".mlp")))
    first = {}
    for i, t, enters in layer_runs(len(layers), cfg.get("loop")):
        kind, spec, ff = layers[i]
        out.layers.append(LayerSpec(kind, spec, ff, weights_of=first.get(i), tensors=i, enter=(t > 0, t) if enters else None))
        first.setdefault(i, len(out.layers) - 1)
    return out
