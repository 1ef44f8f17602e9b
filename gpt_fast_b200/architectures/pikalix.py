"""The Pikalix decoder as data: which parts each layer has and which checkpoint tensors fill which parameter.

The design: a token embedding that passes a norm; several residual streams per token, all equal to it at the start, that every
sublayer reads as a weighted sum and writes back through a mixing matrix (`parts.streams`); pre-norm layers in an order that
config.json lists; the sum of the streams through a final norm and an output matrix of its own.  One kind of mixer:

    'attention'  grouped-query attention with biases on q, k and v, q and k normed over the whole projection ahead of an
                 interleaved rotation of each head's first dimensions, a sliding window, a given score scale and one added to the
                 softmax denominator.  A layer with 'kv_from' has queries only and reads the keys and values that another
                 layer cached.

The feed-forward of a layer is dense (the tanh form of GELU between two products), a mixture of SwiGLU experts (sigmoid scores
whose weights are taken as they are, a correction that counts for the choice only, the choice among the groups whose two best
choice scores have the largest sum, optionally a shared expert), or there is none.

config.json keys: architecture, vocab, width, streams, norm.eps, layers [{type, mixer {heads, kv_heads, dim, vdim, scale, mask.size,
rot {base, dims}, kv_from}, mlp {kind: 'dense', ff} | {kind: 'moe', expert.ff, router {experts, top, groups {count, keep}},
shared.ff} | null}].  Tensor names: embed, embed.norm, final.norm, head, l<i>.norm1, l<i>.norm2, l<i>.hc{1,2}.{in, out, mix},
l<i>.mix.{q, k, v, q.b, k.b, v.b, q.norm, k.norm, o}, l<i>.mlp.{up, down} or l<i>.mlp.{router, correction, e<j>.{gate, up, down},
shared.{gate, up, down}}.
"""
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple, Union

from ..config.args import ConfigError
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..weights.plan import Recipe, Source, WeightPlan
from .lasezen import _int, _num
from .tapupel import _obj, _stack, _unstack

GROUP_TERMS = 2                      # choice scores that make up a group's score
SINK = 0.0                           # the score of the sink: exp(0) joins every softmax denominator


@dataclass(frozen=True)
class MixerArgs:
    heads: int
    kv_heads: int
    dim: int                         # per-head query/key size
    vdim: int                        # per-head value size
    scale: float
    window: Optional[int] = None
    rot_base: float = 0.0
    rot_dims: int = 0                # 0: no rotation
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class DenseArgs:
    ff: int


@dataclass(frozen=True)
class MoeArgs:
    ff: int                          # hidden size of one expert
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0               # 0: no shared expert


@dataclass(frozen=True)
class LayerArgs:
    mixer: MixerArgs
    mlp: Union[DenseArgs, MoeArgs, None] = None


@dataclass(frozen=True)
class PikalixArgs:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[LayerArgs, ...]
    source: Dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    def to_json(self) -> Dict[str, Any]:
        return dict(self.source)


def _mixer(kind: Any, m: Any, where: str) -> MixerArgs:
    if kind != "attention":
        raise ConfigError(f"config.json: {where}'type' is {kind!r}; this design has 'attention'")
    if not isinstance(m, dict):
        raise ConfigError(f"config.json: {where}'mixer' must be an object")
    w = where + "mixer."
    sizes = {k: _int(m, k, w) for k in ("heads", "kv_heads", "dim", "vdim")}
    if sizes["heads"] % sizes["kv_heads"]:
        raise ConfigError(f"config.json: {w}{sizes['heads']} heads do not divide into {sizes['kv_heads']} kv_heads")
    base, dims = 0.0, 0
    if m.get("rot") is not None:
        rot = _obj(m, "rot", w)
        dims, base = _int(rot, "dims", w + "rot.", 0), _num(rot, "base", w + "rot.")
        if dims % 2 or dims > sizes["dim"]:
            raise ConfigError(f"config.json: {w}rot.dims = {dims} must be even and at most dim = {sizes['dim']}")
        if not base > 0:
            raise ConfigError(f"config.json: {w}rot.base must be positive")
    window = None if m.get("mask") is None else _int(_obj(m, "mask", w), "size", w + "mask.")
    return MixerArgs(scale=_num(m, "scale", w), window=window, rot_base=base, rot_dims=dims,
                     kv_from=None if m.get("kv_from") is None else _int(m, "kv_from", w, 0), **sizes)


def _mlp(mlp: Any, where: str) -> Union[DenseArgs, MoeArgs, None]:
    if mlp is None:
        return None
    w = where + "mlp."
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind == "dense":
        return DenseArgs(_int(mlp, "ff", w))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}'mlp' must be null or an object of kind 'dense' or 'moe'")
    expert, router = _obj(mlp, "expert", w), _obj(mlp, "router", w)
    wr = w + "router."
    count = keep = 1
    if router.get("groups") is not None:
        g = _obj(router, "groups", wr)
        count, keep = _int(g, "count", wr + "groups."), _int(g, "keep", wr + "groups.")
    out = MoeArgs(_int(expert, "ff", w + "expert."), experts=_int(router, "experts", wr), top=_int(router, "top", wr), groups=count, keep=keep,
                  shared_ff=0 if mlp.get("shared") is None else _int(_obj(mlp, "shared", w), "ff", w + "shared."))
    if out.experts % count or keep > count:
        raise ConfigError(f"config.json: {wr}groups: {keep} of {count} groups of {out.experts} experts")
    if out.top > keep * (out.experts // count):
        raise ConfigError(f"config.json: {wr}top = {out.top} of the {keep * (out.experts // count)} experts of {keep} groups")
    return out


def parse(cfg: Dict[str, Any]) -> PikalixArgs:
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
        parsed.append(LayerArgs(_mixer(L.get("type"), L.get("mixer"), where), _mlp(L.get("mlp"), where)))
    for i, L in enumerate(parsed):
        j = L.mixer.kv_from
        if j is None:
            continue
        where = f"layers[{i}].mixer."
        if j >= i or parsed[j].mixer.kv_from is not None:
            raise ConfigError(f"config.json: {where}kv_from = {j} must name an earlier layer with keys and values of its own")
        for k in ("kv_heads", "dim", "vdim"):
            if getattr(parsed[j].mixer, k) != getattr(L.mixer, k):
                raise ConfigError(f"config.json: {where}{k} differs from layer {j}'s, whose keys and values it reads")
    eps = _num(_obj(cfg, "norm", ""), "eps", "norm.")
    if eps < 0:
        raise ConfigError("config.json: norm.eps must not be negative")
    return PikalixArgs(vocab=_int(cfg, "vocab", ""), width=_int(cfg, "width", ""), streams=_int(cfg, "streams", ""), norm_eps=eps,
                       layers=tuple(parsed), source=dict(cfg))


def _attention(a: PikalixArgs, m: MixerArgs) -> PartSpec:
    return PartSpec("attention", dict(dim=a.width, n_head=m.heads, n_kv=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, window=m.window,
                                      scale=m.scale, bias=True, qk_norm_eps=a.norm_eps, qk_norm_whole=True, sink_value=SINK,
                                      shared_kv=m.kv_from is not None))


def _feed_forward(a: PikalixArgs, f: Union[DenseArgs, MoeArgs]) -> PartSpec:
    if isinstance(f, DenseArgs):
        return PartSpec("dense", dict(dim=a.width, hidden=f.ff, activation="gelu_tanh"))
    return PartSpec("moe", dict(dim=a.width, hidden=f.ff, n_experts=f.experts, top=f.top, score="sigmoid_plain", correction=True,
                                groups=(f.groups, f.keep, GROUP_TERMS), shared_hidden=f.shared_ff))


def build_spec(a: PikalixArgs) -> ModelSpec:
    norm = PartSpec("rmsnorm", dict(dim=a.width, eps=a.norm_eps))
    layers = []
    for L in a.layers:
        m = L.mixer
        parts = dict(mixer=_attention(a, m), mixer_norm=norm)
        if L.mlp is not None:
            parts.update(ffn_norm=norm, feed_forward=_feed_forward(a, L.mlp))
        position = PartSpec("rope", dict(head_dim=m.rot_dims, base=m.rot_base, pairing="interleaved", freq_dtype="float64")) if m.rot_dims else None
        layers.append(LayerSpec(block="streams", parts=parts, position=position, block_params=dict(streams=a.streams)))
    schedule = [ScheduleEntry(layer=i, cache=i, kv_from=L.mixer.kv_from) for i, L in enumerate(a.layers)]
    # launches in turn: with kernels allowed to start under their predecessor another design of experts and attention stopped
    # making progress in some long prompt steps, and the pair of kernels behind that is not known
    spec = ModelSpec(architecture="pikalix", dim=a.width, vocab_size=a.vocab, layers=layers, schedule=schedule, final_norm=norm,
                     embedding=PartSpec("normed", dict(dim=a.width, eps=a.norm_eps)), streams=a.streams, launch_overlap=False)
    spec.validate()
    return spec


def weight_plan(a: PikalixArgs) -> WeightPlan:
    D, V, n = a.width, a.vocab, a.streams
    r = [Recipe("embed.weight", [Source("embed", (V, D), "embedding")]), Recipe("head.weight", [Source("head", (V, D))]),
         Recipe("embedding.weight", [Source("embed.norm", (D,), "norm")]), Recipe("final_norm.weight", [Source("final.norm", (D,), "norm")])]
    ignored = []
    for i, L in enumerate(a.layers):
        s, t, m = f"l{i}.", f"layers.{i}.", L.mixer

        def around(number: int, role: str):
            c, y = f"{s}hc{number}.", f"{t}{role}_streams."
            return [Recipe(f"{t}{role}_norm.weight", [Source(f"{s}norm{number}", (D,), "norm")]),
                    Recipe(y + "enter", [Source(c + "in", (n,), "share")]), Recipe(y + "leave", [Source(c + "out", (n,), "norm")]),
                    Recipe(y + "mix", [Source(c + "mix", (n, n), "identity")])]
        r += around(1, "mixer")
        x, y = s + "mix.", t + "mixer."
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        r += [Recipe(y + "wq", [Source(x + "q", (H * d, D))]), Recipe(y + "bq", [Source(x + "q.b", (H * d,), "bias")]),
              Recipe(y + "q_norm", [Source(x + "q.norm", (H * d,), "norm")]), Recipe(y + "wo", [Source(x + "o", (D, H * dv))])]
        if m.kv_from is None:
            r += [Recipe(y + "wk", [Source(x + "k", (G * d, D))]), Recipe(y + "bk", [Source(x + "k.b", (G * d,), "bias")]),
                  Recipe(y + "k_norm", [Source(x + "k.norm", (G * d,), "norm")]),
                  Recipe(y + "wv", [Source(x + "v", (G * dv, D))]), Recipe(y + "bv", [Source(x + "v.b", (G * dv,), "bias")])]
        x, y = s + "mlp.", t + "feed_forward."
        if L.mlp is None:
            ignored.append(rf"l{i}\.(norm2|hc2\..*)")          # constants of a sublayer the layer does not have
            continue
        r += around(2, "ffn")
        F = L.mlp.ff
        if isinstance(L.mlp, DenseArgs):
            r += [Recipe(y + "up", [Source(x + "up", (F, D))]), Recipe(y + "down", [Source(x + "down", (D, F))])]
            continue
        E, Fs = L.mlp.experts, L.mlp.shared_ff
        r += [Recipe(y + "router", [Source(x + "router", (E, D))]), Recipe(y + "correction", [Source(x + "correction", (E,), "bias")])]
        for name, shape in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F))):
            r.append(Recipe(y + name, [Source(f"{x}e{e}.{name}", shape) for e in range(E)], _stack, _unstack))
        if Fs:
            r += [Recipe(y + f"shared_{name}", [Source(f"{x}shared.{name}", shape)])
                  for name, shape in (("gate", (Fs, D)), ("up", (Fs, D)), ("down", (D, Fs)))]
    return WeightPlan(recipes=r, ignored=tuple(ignored))


PIKALIX = register_architecture(Architecture(
    name="pikalix", aliases=("Pikalix",), parse=parse, build_spec=build_spec, weight_plan=weight_plan,
))
