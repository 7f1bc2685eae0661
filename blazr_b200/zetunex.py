"""Zetunex: a decoder-only design of parallel layers: one RMS norm per layer, whose output both the mixer and the feed-forward read,
x <- x + m (mixer(h) + ff(h)).  Its mixers are a linear attention with one fixed decay per head (silu on q, k and v, one norm over all heads, a
sigmoid gate) or two branches side by side: a windowed attention without positions, with biases on q, k and v, beside a selective scan; half the
sum of the two results, each normed over the model width.  The feed-forward is dense (silu-gated) or a mixture of silu-gated experts, chosen by
soft-max scores inside the best groups of experts (a group counts by its largest score) and weighted by those scores as they are, times a constant.
A span of layers may run several times with the same weights, each pass with a cache or state of its own and a learned row added in front of it.

This module only reads the design's config.json and maps it onto the generic specs of blazr_b200/layered.py (layout "parallel"); the mechanisms
and their kernels are shared with any other layer-list design:

    config key                              -> spec
    vocab, width                            -> LayeredConfig.vocab / width (one residual stream, output projection = embedding table)
    norm.eps                                -> eps of every RMS norm (layer, branch, heads)
    residual_mult                           -> LayeredConfig.residual_mult
    loop.start / stop / times               -> the span's layers are listed `times` times; a repeated run names its layer's tensors (LayerSpec.tensors),
                                               borrows the weights of the first run (weights_of) and keeps a cache / state of its own; the first
                                               layer of each pass carries LayerSpec.enter = (False, row of loop.step)
    layers[i].type = "lightning"            -> RetentionSpec(heads, dim, vdim, decay, key_scale 1, qkv_silu, norm "joint", gate "sigmoid")
    layers[i].type = "parallel"             -> TwoBranchSpec(left = AttentionSpec(biases on q / k / v, window = mask.size, no rotation),
                                               right = ScanSpec(inner, state, conv, dt_rank), scales 1/2, branch_norm)
    layers[i].mlp = null                    -> no feed-forward
    layers[i].mlp.kind = "dense"            -> DenseFfSpec(ff, silu gate: "swish_clamp" without a limit, alpha 1, up_shift 0)
    layers[i].mlp.kind = "moe"              -> MoeFfSpec(router "softmax", group_best 1, renorm False, route_scale = router.scale, router.experts / top /
                                               groups.(count, keep), expert.ff, the same silu gate)

Tensor names: embed, final.norm, loop.step, l<i>.norm1, linear attention l<i>.mix.{q,k,v,g,o,norm}, two-branch l<i>.mix.left.{q,k,v}(.b), left.o, left.out
and l<i>.mix.right.{in,conv,conv.b,x,dt,dt.b,A_log,D,o,out}, l<i>.mlp.{gate,up,down}, l<i>.mlp.router, l<i>.mlp.e<j>.{gate,up,down}.
"""
from __future__ import annotations

import math

from .layered import AttentionSpec, DenseFfSpec, LayeredConfig, LayerSpec, MoeFfSpec, RetentionSpec, ScanSpec, TwoBranchSpec, loop_runs

ARCHITECTURE = "Zetunex"
SILU_GATE = dict(act="swish_clamp", limit=math.inf, alpha=1.0, up_shift=0.0)


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


def _lightning(m: dict, where: str) -> RetentionSpec:
    spec = RetentionSpec(heads=_size(m, "heads", where), dim=_size(m, "dim", where), vdim=_size(m, "vdim", where), decay=[float(d) for d in _need(m, "decay", where)],
                         key_scale=1.0, qkv_silu=True, norm="joint", gate="sigmoid")
    if len(spec.decay) != spec.heads or any(not 0.0 < d <= 1.0 for d in spec.decay):
        raise ConfigError(f"config: {where}: decay lists one value in (0, 1] per head")
    return spec


def _two_branch(m: dict, where: str) -> TwoBranchSpec:
    a, r = _need(m, "left", where), _need(m, "right", where)
    wl, wr = where + ".left", where + ".right"
    left = AttentionSpec(heads=_size(a, "heads", wl), kv_heads=_size(a, "kv_heads", wl), dim=_size(a, "dim", wl), vdim=_size(a, "vdim", wl), scale=float(_need(a, "scale", wl)),
                         window=int((a.get("mask") or {}).get("size", 0)), qk_unit_norm=False, gated=False, bias=True)
    if left.heads % left.kv_heads:
        raise ConfigError(f"config: {wl}: heads is not a multiple of kv_heads")
    if left.window < 0:
        raise ConfigError(f"config: {wl}: mask.size must not be negative")
    right = ScanSpec(inner=_size(r, "inner", wr), state=_size(r, "state", wr), conv=_size(r, "conv", wr), dt_rank=_size(r, "dt_rank", wr))
    if right.conv > 8:
        raise ConfigError(f"config: {wr}: 1 to 8 convolution taps")
    return TwoBranchSpec(left, right, left_scale=0.5, right_scale=0.5, branch_norm=True)


def _feed_forward(mlp, where: str):
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        return DenseFfSpec(ff=_size(mlp, "ff", where), **SILU_GATE)
    if kind == "moe":
        r, ex = _need(mlp, "router", where), _need(mlp, "expert", where)
        g = r.get("groups")
        spec = MoeFfSpec(experts=_size(r, "experts", where + ".router"), top=_size(r, "top", where + ".router"), ff=_size(ex, "ff", where + ".expert"),
                         groups=_size(g, "count", where + ".router.groups") if g else 1, keep=_size(g, "keep", where + ".router.groups") if g else 1,
                         router="softmax", group_best=1, renorm=False, route_scale=float(r.get("scale", 1.0)), **SILU_GATE)
        if spec.top > spec.experts:
            raise ConfigError(f"config: {where}: router.top must lie between 1 and router.experts")
        if spec.experts % spec.groups or spec.keep > spec.groups or spec.keep * (spec.experts // spec.groups) < spec.top:
            raise ConfigError(f"config: {where}: router.groups does not fit experts / top")
        return spec
    raise ConfigError(f"config: {where}: unknown feed-forward kind '{kind}'")


def parse_config(cfg: dict) -> LayeredConfig:
    out = LayeredConfig(name=ARCHITECTURE, vocab=_size(cfg, "vocab", "top level"), width=_size(cfg, "width", "top level"), streams=1, norm_groups=1,
                        eps=float(_need(_need(cfg, "norm", "top level"), "eps", "norm")), canon_taps=0, embed_scale=1.0, layout="parallel", tied_head=True,
                        depth_average=False, residual_mult=float(_need(cfg, "residual_mult", "top level")))
    layers = []
    for i, lay in enumerate(_need(cfg, "layers", "top level")):
        where = f"layers[{i}]"
        kind, m = _need(lay, "type", where), _need(lay, "mixer", where)
        if kind == "lightning":
            spec = ("retention", _lightning(m, where + ".mixer"))
        elif kind == "parallel":
            spec = ("two_branch", _two_branch(m, where + ".mixer"))
        else:
            raise ConfigError(f"config: {where}: unknown layer type '{kind}'")
        layers.append(spec + (_feed_forward(lay.get("mlp"), where + ".mlp"),))
    n, loop = len(layers), cfg.get("loop")
    start = stop = times = 0
    if loop is not None:
        start, stop, times = (int(_need(loop, k, "loop")) for k in ("start", "stop", "times"))
        if not (0 <= start < stop <= n) or times < 1:
            raise ConfigError("config: loop: 0 <= start < stop <= number of layers, times >= 1")
    first = {}
    for i, t, enters in loop_runs(n, start, stop, times):
        kind, spec, ff = layers[i]
        out.layers.append(LayerSpec(kind, spec, ff, weights_of=first.get(i), tensors=i, enter=(False, t) if enters else None))
        first.setdefault(i, len(out.layers) - 1)
    return out
