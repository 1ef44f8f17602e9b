"""The Dufizen decoder as data: which parts each layer has and which checkpoint tensors fill which parameter.

The design: a token embedding; layers in an order that config.json lists, each a pre-norm block whose norms are root-mean-square
norms with weights stored around zero (the factor is 1 + w) and whose sublayers' results take a learned factor per column,
followed by a token input read from a side table; a span of layers may run several times in a row with the same weights and a
cache entry per pass, each pass entered through a product of the stream beside the embedding output plus a vector of the pass;
a final norm of the same kind and the output product with the embedding table.  Two kinds of mixer:

    'gla'               gated linear attention: a key-value recurrence with a decay per head and key channel,
                        sigmoid(z)^(1/tau), a normed and gated read-out
    'latent_attention'  softmax attention whose keys and values are expanded from a normed latent of `kv_rank` numbers per token,
                        with `rot_dim` rotated query/key dimensions (the key's shared by all heads, half-split pairs), a given
                        score scale, a sliding window, a learned sink per head and a sigmoid gate per head

The feed-forward is a mixture of experts of two products with the square of ReLU between them, chosen by the softmax over all
experts plus a correction among the best groups of experts and weighted by that softmax as it is, with an optional shared
expert; a layer may have none.

config.json keys: architecture, vocab, width, norm.eps, token_side.dim, loop {start, stop, times}, layers [{type, mixer {...},
mlp {kind, expert.ff, router {experts, top, groups {count, keep}}, shared.ff} | null}].  Tensor names: embed, final.norm, loop.in,
loop.step, side.embed, l<i>.norm1, l<i>.norm2, l<i>.ls1, l<i>.ls2, l<i>.side.{gate, proj, norm}, l<i>.mix.*, l<i>.mlp.{router,
correction, e<j>.{up, down}, shared.{up, down}}.
"""
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..config.args import ConfigError
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..weights.plan import Recipe, Source, WeightPlan
from .lasezen import _int, _num
from .tapupel import _obj, _stack, _unstack

KINDS = ("gla", "latent_attention")
DEFAULT_DECAY_RANK = 16              # of random weights; a checkpoint's tensors say it themselves
Shapes = Optional[Dict[str, Tuple[int, ...]]]


@dataclass(frozen=True)
class MlpArgs:
    ff: int                          # hidden size of one expert
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0               # 0: no shared expert


@dataclass(frozen=True)
class LayerArgs:
    kind: str
    mixer: Dict[str, Any]            # the layer's sizes and constants, checked
    mlp: Optional[MlpArgs] = None    # None: the layer has no feed-forward


@dataclass(frozen=True)
class DufizenArgs:
    vocab: int
    width: int
    norm_eps: float
    side_dim: int                    # columns of the side table per layer; 0: no token inputs
    layers: Tuple[LayerArgs, ...]
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    source: Dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, number of the pass if the run is a pass's first one) in running order."""
        start, stop, times = self.loop or (0, 0, 0)
        n = len(self.layers)
        out = [(i, None) for i in range(start)]
        for t in range(times):
            out += [(i, t if i == start else None) for i in range(start, stop)]
        return out + [(i, None) for i in range(stop, n)]

    def to_json(self) -> Dict[str, Any]:
        return dict(self.source)


def _mixer(kind: Any, m: Any, where: str) -> Dict[str, Any]:
    if kind not in KINDS:
        raise ConfigError(f"config.json: {where}'type' is {kind!r}; this design has {', '.join(KINDS)}")
    if not isinstance(m, dict):
        raise ConfigError(f"config.json: {where}'mixer' must be an object")
    w = where + "mixer."
    if kind == "gla":
        out = {k: _int(m, k, w) for k in ("heads", "dim", "vdim")}
        out["tau"] = _num(m, "tau", w)
        if not out["tau"] > 0:
            raise ConfigError(f"config.json: {w}tau must be positive")
        return out
    out = {k: _int(m, k, w) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    out["scale"] = _num(m, "scale", w)
    rot = _obj(m, "rot", w)
    dims, out["rot_base"] = _int(rot, "dims", w + "rot."), _num(rot, "base", w + "rot.")
    if dims != out["rot_dim"] or dims % 2:
        raise ConfigError(f"config.json: {w}rot.dims = {dims} must be even and equal rot_dim = {out['rot_dim']}")
    if not out["rot_base"] > 0:
        raise ConfigError(f"config.json: {w}rot.base must be positive")
    out["window"] = None if m.get("mask") is None else _int(_obj(m, "mask", w), "size", w + "mask.")
    return out


def _mlp(mlp: Any, where: str) -> Optional[MlpArgs]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}'mlp' must be null or an object of kind 'moe'")
    w = where + "mlp."
    expert, router = _obj(mlp, "expert", w), _obj(mlp, "router", w)
    wr = w + "router."
    count = keep = 1
    if router.get("groups") is not None:
        g = _obj(router, "groups", wr)
        count, keep = _int(g, "count", wr + "groups."), _int(g, "keep", wr + "groups.")
    out = MlpArgs(_int(expert, "ff", w + "expert."), experts=_int(router, "experts", wr), top=_int(router, "top", wr), groups=count, keep=keep,
                  shared_ff=0 if mlp.get("shared") is None else _int(_obj(mlp, "shared", w), "ff", w + "shared."))
    if out.experts % count or keep > count:
        raise ConfigError(f"config.json: {wr}groups: {keep} of {count} groups of {out.experts} experts")
    if out.top > keep * (out.experts // count):
        raise ConfigError(f"config.json: {wr}top = {out.top} of the {keep * (out.experts // count)} experts of {keep} groups")
    return out


def parse(cfg: Dict[str, Any]) -> DufizenArgs:
    if not isinstance(cfg, dict):
        raise ConfigError("config.json must hold one JSON object")
    layers = cfg.get("layers")
    if not isinstance(layers, list) or not layers:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    parsed = []
    for i, L in enumerate(layers):
        where = f"layers[{i}]."
        if not isinstance(L, dict):
            raise ConfigError(f"config.json: layers[{i}] must be an object")
        parsed.append(LayerArgs(L.get("type"), _mixer(L.get("type"), L.get("mixer"), where), _mlp(L.get("mlp"), where)))
    eps = _num(_obj(cfg, "norm", ""), "eps", "norm.")
    if eps < 0:
        raise ConfigError("config.json: norm.eps must not be negative")
    loop = None
    if cfg.get("loop") is not None:
        lp = _obj(cfg, "loop", "")
        loop = (_int(lp, "start", "loop.", 0), _int(lp, "stop", "loop."), _int(lp, "times", "loop."))
        if not loop[0] < loop[1] <= len(parsed):
            raise ConfigError(f"config.json: loop spans layers {loop[0]}..{loop[1] - 1} of {len(parsed)}")
    side = 0 if cfg.get("token_side") is None else _int(_obj(cfg, "token_side", ""), "dim", "token_side.")
    return DufizenArgs(vocab=_int(cfg, "vocab", ""), width=_int(cfg, "width", ""), norm_eps=eps, side_dim=side, layers=tuple(parsed),
                       loop=loop, source=dict(cfg))


def decay_rank(a: DufizenArgs, layer: int, shapes: Shapes) -> int:
    """The rank of a 'gla' layer's decay projection, which config.json does not name: the first dimension of the checkpoint's
    l<i>.mix.a1.  Without a checkpoint (random weights) `mixer.low_rank` if config.json has it, else a fixed number."""
    name = f"l{layer}.mix.a1"
    if shapes is not None and name in shapes:
        return int(shapes[name][0])
    r = a.source.get("layers", [{}] * (layer + 1))[layer].get("mixer", {}).get("low_rank")
    return r if isinstance(r, int) and r > 0 else DEFAULT_DECAY_RANK


def build_spec(a: DufizenArgs, shapes: Shapes = None) -> ModelSpec:
    D, eps = a.width, a.norm_eps
    norm = PartSpec("rmsnorm", dict(dim=D, eps=eps, one_plus=True))
    layers = []
    for i, L in enumerate(a.layers):
        m, position = L.mixer, None
        if L.kind == "gla":
            mixer = PartSpec("gla", dict(dim=D, n_head=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"], decay_rank=decay_rank(a, i, shapes),
                                         tau=m["tau"], eps=eps))
        else:
            position = PartSpec("rope", dict(head_dim=m["rot_dim"], base=m["rot_base"], pairing="half", freq_dtype="float64"))
            mixer = PartSpec("latent_attention", dict(dim=D, n_head=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
                                                      rank=m["kv_rank"], scale=m["scale"], eps=eps, window=m["window"], sink=True,
                                                      head_gate=True))
        parts = dict(mixer=mixer, mixer_norm=norm)
        if L.mlp is not None:
            parts.update(ffn_norm=norm, feed_forward=PartSpec("moe", dict(
                dim=D, hidden=L.mlp.ff, n_experts=L.mlp.experts, top=L.mlp.top, score="softmax", correction=True, activation="relu2",
                groups=(L.mlp.groups, L.mlp.keep), shared_hidden=L.mlp.shared_ff)))
        if a.side_dim:
            parts["token_input"] = PartSpec("gated_side", dict(dim=D, side_dim=a.side_dim, offset=i * a.side_dim, eps=eps))
        layers.append(LayerSpec(block="prenorm", parts=parts, position=position, block_params=dict(layer_scale=True)))
    schedule = [ScheduleEntry(layer=i, cache=r, junction=None if t is None else 0, turn=t or 0) for r, (i, t) in enumerate(a.runs())]
    # launches in turn: with kernels allowed to start under their predecessor another design of experts and attention stopped
    # making progress in some long prompt steps, and the pair of kernels behind that is not known
    spec = ModelSpec(architecture="dufizen", dim=D, vocab_size=a.vocab, layers=layers, schedule=schedule, final_norm=norm, tie_embeddings=True,
                     junctions=[] if a.loop is None else [PartSpec("pass_entry", dict(dim=D, passes=a.loop[2]))],
                     token_table=a.side_dim * len(a.layers), launch_overlap=False)
    spec.validate()
    return spec


def weight_plan(a: DufizenArgs, shapes: Shapes = None) -> WeightPlan:
    D, V = a.width, a.vocab
    r = [Recipe("embed.weight", [Source("embed", (V, D), "embedding")]), Recipe("final_norm.weight", [Source("final.norm", (D,), "bias")])]
    if a.loop is not None:
        r += [Recipe("junctions.0.weight", [Source("loop.in", (D, 2 * D))]), Recipe("junctions.0.step", [Source("loop.step", (a.loop[2], D))])]
    if a.side_dim:
        r.append(Recipe("token_table.weight", [Source("side.embed", (V, a.side_dim * len(a.layers)), "embedding")]))
    for i, L in enumerate(a.layers):
        s, t, m = f"l{i}.", f"layers.{i}.", L.mixer
        x, y = s + "mix.", t + "mixer."
        r += [Recipe(t + "mixer_norm.weight", [Source(s + "norm1", (D,), "bias")]), Recipe(t + "mixer_scale.weight", [Source(s + "ls1", (D,), "norm")])]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if L.kind == "gla":
            rank = decay_rank(a, i, shapes)
            r += [Recipe(y + "wq", [Source(x + "q", (H * d, D))]), Recipe(y + "wk", [Source(x + "k", (H * d, D))]),
                  Recipe(y + "wv", [Source(x + "v", (H * dv, D))]), Recipe(y + "wg", [Source(x + "g", (H * dv, D))]),
                  Recipe(y + "wa1", [Source(x + "a1", (rank, D))]), Recipe(y + "wa2", [Source(x + "a2", (H * d, rank))]),
                  Recipe(y + "a2_bias", [Source(x + "a2.b", (H * d,), "unit")]), Recipe(y + "norm", [Source(x + "norm", (dv,), "norm")]),
                  Recipe(y + "wo", [Source(x + "o", (D, H * dv))])]
        else:
            rot, R = m["rot_dim"], m["kv_rank"]
            r += [Recipe(y + "wq", [Source(x + "q", (H * (d + rot), D))]), Recipe(y + "wdkv", [Source(x + "dkv", (R + rot, D))]),
                  Recipe(y + "latent_norm", [Source(x + "dkv.norm", (R,), "norm")]),
                  Recipe(y + "wuk", [Source(x + "uk", (H * d, R))]), Recipe(y + "wuv", [Source(x + "uv", (H * dv, R))]),
                  Recipe(y + "sink", [Source(x + "sink", (H,), "unit")]), Recipe(y + "wg", [Source(x + "g", (H, D))]),
                  Recipe(y + "wo", [Source(x + "o", (D, H * dv))])]
        if L.mlp is not None:
            x, y = s + "mlp.", t + "feed_forward."
            E, F, Fs = L.mlp.experts, L.mlp.ff, L.mlp.shared_ff
            r += [Recipe(t + "ffn_norm.weight", [Source(s + "norm2", (D,), "bias")]), Recipe(t + "ffn_scale.weight", [Source(s + "ls2", (D,), "norm")]),
                  Recipe(y + "router", [Source(x + "router", (E, D))]), Recipe(y + "correction", [Source(x + "correction", (E,), "bias")])]
            for name, shape in (("up", (F, D)), ("down", (D, F))):
                r.append(Recipe(y + name, [Source(f"{x}e{e}.{name}", shape) for e in range(E)], _stack, _unstack))
            if Fs:
                r += [Recipe(y + "shared_up", [Source(x + "shared.up", (Fs, D))]), Recipe(y + "shared_down", [Source(x + "shared.down", (D, Fs))])]
        if a.side_dim:
            y = t + "token_input."
            r += [Recipe(y + "gate", [Source(s + "side.gate", (a.side_dim, D))]), Recipe(y + "proj", [Source(s + "side.proj", (D, a.side_dim))]),
                  Recipe(y + "norm", [Source(s + "side.norm", (D,), "norm")])]
    return WeightPlan(recipes=r, aliases={"head.weight": "embed.weight"})


DUFIZEN = register_architecture(Architecture(
    name="dufizen", aliases=("Dufizen",), parse=parse, build_spec=build_spec, weight_plan=weight_plan, shapes_from_checkpoint=True,
))
