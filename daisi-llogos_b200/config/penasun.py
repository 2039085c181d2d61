"""Typed configuration of the Penasun decoder and its model builder.

Penasun's config.json is nested and names its architecture under ``architecture``:

    {"architecture": "Penasun", "vocab": V, "width": D, "norm": {"eps": e},
     "layers": [{"type": "mamba2",
                 "mixer": {"heads": H, "vdim": P, "state": N, "groups": G, "conv": K, "norm_groups": n}, "mlp": ...},
                {"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": dq, "vdim": dv, "scale": s, "diff": d,
                           "q_temp": {"coef": c, "every": E} | null},
                 "mlp": {"kind": "moe",
                         "router": {"experts": E, "top": k, "identity": i, "scale": r, "groups": {"count": g, "keep": m} | null},
                         "expert": {"ff": F, "limit": l}} | null}, ...]}

Every layer names its own kind of mixer and its own sizes.  What the design fixes and no file says stands below as constants:
pre-norm sublayers with RMS norms (parts/block.py); "mamba2" is a state-space recurrence with a scalar decay per head
(parts/state_space.py); "attention" is differential attention without rotation, with biases on all four projections and queries
that grow with the logarithm of their position (parts/attention.py, parts/position.py); the mixture's router takes a softmax over
all experts, chooses by corrected scores within the best groups (a group is judged by its one largest corrected score) and
weighs with the plain scores as they are, and its last choices are identity experts; experts are gated in a clamped form
(parts/moe.py); the output head is the embedding table.  Tensor names: ``embed``, ``l<i>.norm{1,2}``,
``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``, ``l<i>.mix.{q,k,v,o}`` (+ ``.b``), ``l<i>.mix.{lq1,lk1,lq2,lk2}``,
``l<i>.mlp.{router,correction}``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``final.norm``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .dense import ConfigError, _need
from .fipavik import _float
from .karitar import _obj, _positive
from .memilorn import ClampedExpert, _expert, _gate, _positive_float

NAME = "Penasun"

# what the design fixes (the constants of a clamped expert are Memilorn's: config/memilorn.py)
MAPS = 2                            # softmax maps per head, whose outputs' difference is taken
ROUTER_SCORE = "softmax_all"        # scores are a softmax over all experts; the chosen ones' weights are not divided by their sum
GROUP_SCORE_TOP = 1                 # a group of experts is judged by its largest choice score
MIXER_KINDS = ("mamba2", "attention")


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class QueryTemp:
    coef: float
    every: float


@dataclass(frozen=True)
class DifferentialAttention:
    heads: int
    kv_heads: int
    dim: int              # elements of one map of a query or key head
    vdim: int
    scale: float
    diff: float
    q_temp: Optional[QueryTemp]


@dataclass(frozen=True)
class PenasunMoe:
    experts: int          # with matrices
    identity: int         # without
    top: int
    scale: float
    groups: int           # 0: no groups
    keep_groups: int
    expert: ClampedExpert


@dataclass(frozen=True)
class PenasunLayer:
    type: str             # one of MIXER_KINDS
    mixer: Union[StateSpaceMixer, DifferentialAttention]
    mlp: Optional[PenasunMoe]


@dataclass(frozen=True)
class PenasunConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[PenasunLayer, ...]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "PenasunConfig":
        vocab = _positive(d, "vocab")
        width = _positive(d, "width")
        eps = _positive_float(_obj(d, "norm"), "eps", "norm.")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError("config.json: missing key 'layers' (a non-empty list of layers)")
        layers = tuple(_layer(i, raw) for i, raw in enumerate(raw_layers))
        return cls(architecture=str(d.get("architecture", NAME)), vocab=vocab, width=width, norm_eps=eps, layers=layers)


def _whole(d: Mapping[str, Any], key: str, where: str, default: int) -> int:
    """A number of things that may be none (a missing key or null: ``default``)."""
    if d.get(key) is None:
        return default
    v = _need(d, key, int)
    if v < 0:
        raise ConfigError(f"config.json: {where}{key} must not be negative, got {v}")
    return v


def _mlp(raw: Any, where: str) -> Optional[PenasunMoe]:
    if raw is None:
        return None
    if not isinstance(raw, Mapping):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    if raw.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}kind = {raw.get('kind')!r} is not supported (known: 'moe')")
    router, rw = _obj(raw, "router"), where + "router."
    experts, top = _positive(router, "experts", rw), _positive(router, "top", rw)
    identity = _whole(router, "identity", rw, 0)
    routed = experts + identity
    if top > routed:
        raise ConfigError(f"config.json: {rw}top {top} exceeds the {routed} experts and identity experts")
    scale = 1.0 if router.get("scale") is None else _positive_float(router, "scale", rw)
    count = keep = 0
    if router.get("groups") is not None:
        groups = _obj(router, "groups")
        count, keep = _positive(groups, "count", rw + "groups."), _positive(groups, "keep", rw + "groups.")
        if routed % count or keep > count:
            raise ConfigError(f"config.json: {rw}groups: {routed} experts and identity experts in {count} groups of which {keep} are kept")
        if top > keep * (routed // count):
            raise ConfigError(f"config.json: {rw}top {top} exceeds the experts of {keep} groups")
    return PenasunMoe(experts, identity, top, scale, count, keep, _expert(_obj(raw, "expert"), where + "expert."))


def _layer(i: int, raw: Any) -> PenasunLayer:
    where = f"layers[{i}]."
    if not isinstance(raw, Mapping):
        raise ConfigError(f"config.json: layers[{i}] must be an object")
    kind = raw.get("type")
    if kind not in MIXER_KINDS:
        raise ConfigError(f"config.json: {where}type = {kind!r} is not supported (known: {', '.join(map(repr, MIXER_KINDS))})")
    if not isinstance(raw.get("mixer"), Mapping):
        raise ConfigError(f"config.json: {where}mixer must be an object")
    m, mw = raw["mixer"], where + "mixer."
    heads, vdim = _positive(m, "heads", mw), _positive(m, "vdim", mw)
    if kind == "mamba2":
        mixer = StateSpaceMixer(heads, vdim, _positive(m, "state", mw), _positive(m, "groups", mw), _positive(m, "conv", mw),
                                _positive(m, "norm_groups", mw))
        if heads % mixer.groups:
            raise ConfigError(f"config.json: {mw}heads {heads} is not a multiple of {mw}groups {mixer.groups}")
        if heads * vdim % mixer.norm_groups:
            raise ConfigError(f"config.json: {mw}heads * {mw}vdim = {heads * vdim} is not a multiple of {mw}norm_groups {mixer.norm_groups}")
    else:
        kv_heads = _positive(m, "kv_heads", mw)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {mw}heads {heads} is not a multiple of {mw}kv_heads {kv_heads}")
        temp = None
        if m.get("q_temp") is not None:
            qt = _obj(m, "q_temp")
            temp = QueryTemp(_float(qt, "coef", mw + "q_temp."), _positive_float(qt, "every", mw + "q_temp."))
        mixer = DifferentialAttention(heads, kv_heads, _positive(m, "dim", mw), vdim, _positive_float(m, "scale", mw),
                                      _float(m, "diff", mw), temp)
    return PenasunLayer(kind, mixer, _mlp(raw.get("mlp"), where + "mlp."))


def _temperature(encodings: Dict[str, PartSpec], temp: Optional[QueryTemp]) -> Optional[str]:
    """The name of the query factors for ``temp`` (layers with the same constants share them)."""
    if temp is None:
        return None
    name = f"q_temp{temp.coef!r}/{temp.every!r}"
    encodings.setdefault(name, PartSpec("query_temperature", {"coef": temp.coef, "every": temp.every}))
    return name


def penasun_spec(cfg: PenasunConfig) -> ModelSpec:
    """Parts and run order of a Penasun model (see the module's text for what the design fixes)."""
    encodings: Dict[str, PartSpec] = {}

    def norm(name: str, prefix: str = "") -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "tensor_names": {"weight": name}}, prefix)

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        if layer.type == "mamba2":
            mixer = PartSpec("state_space", {
                "hidden_size": cfg.width, "num_heads": m.heads, "value_dim": m.vdim, "state_size": m.state, "groups": m.groups,
                "conv_taps": m.conv, "norm_groups": m.norm_groups, "norm_eps": cfg.norm_eps,
                "tensor_names": {"in_proj.weight": "in", "conv.weight": "conv", "conv.bias": "conv.b", "norm.weight": "norm",
                                 "o_proj.weight": "o"}}, p + "mix.")
        else:
            names = {f"{x}_proj.{kind}": x + suffix for x in "qkvo" for kind, suffix in (("weight", ""), ("bias", ".b"))}
            mixer = PartSpec("attention", {
                "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "maps": MAPS, "diff": m.diff, "diff_eps": cfg.norm_eps, "qkv_bias": True, "out_bias": True, "qk_norm": False,
                "window": 0, "softmax_scale": m.scale, "position": None, "q_scale": _temperature(encodings, m.q_temp),
                "tensor_names": names}, p + "mix.")
        parts = {"norm1": norm("norm1", p), "mixer": mixer}
        ml = layer.mlp
        if ml is not None:
            parts["norm2"] = norm("norm2", p)
            parts["ffn"] = PartSpec("moe", {
                "hidden_size": cfg.width, "num_experts": ml.experts, "identity": ml.identity, "top": ml.top,
                "expert_size": ml.expert.ff, "router_bias": False, "score": ROUTER_SCORE, "correction": True, "normalize": False,
                "groups": ml.groups, "keep_groups": ml.keep_groups, "group_score_top": GROUP_SCORE_TOP, "weight_scale": ml.scale,
                **_gate(ml.expert),
                "tensor_names": {"router.weight": "router", "experts.*.gate_proj.weight": "e*.gate",
                                 "experts.*.up_proj.weight": "e*.up", "experts.*.down_proj.weight": "e*.down"},
            }, p + "mlp.")
        layers.append(LayerSpec("prenorm", parts))
    spec = ModelSpec(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=None,                       # the query factors are made for as many positions as the cache holds
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width,
                                               "tensor_names": {"weight": "embed"}}, ""),
        encodings=encodings,
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": "embed"}, ""),
        # a layer without a feed-forward has no use for the norm ahead of it
        ignorable_tensors=tuple(rf"l{i}\.norm2" for i, layer in enumerate(cfg.layers) if layer.mlp is None),
    )
    spec.validate()
    return spec
