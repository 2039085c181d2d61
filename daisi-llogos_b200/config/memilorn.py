"""Typed configuration of the Memilorn decoder and its model builder.

Memilorn's config.json is nested and names its architecture under ``architecture``:

    {"architecture": "Memilorn", "vocab": V, "width": D, "norm": {"eps": e},
     "layers": [{"type": "mlstm", "mixer": {"heads": H, "dim": dq, "vdim": dv, "gate_cap": c}, "mlp": ...},
                {"type": "latent_attention", "mixer": {"heads": H, "dim": dq, "vdim": dv, "kv_rank": L, "scale": s}, "mlp": ...},
                {"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": dq, "vdim": dv, "scale": s, "softcap": c | null,
                           "rot": {"base": b, "dims": R} | null},
                 "mlp": {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F, "limit": l},
                         "shared": {"ff": Fs, "limit": ls} | null} | null}, ...],
     "loop": {"start": a, "stop": b, "times": n} | null}

Every layer names its own kind of mixer and its own sizes.  ``loop`` runs layers a .. b-1 n times in a row with the same
weights, every pass with a cache or state of its own and, from the second on, with the embedding's output added to the
residual ahead of its first layer (``ScheduleEntry.add_embedding``).  What the design fixes and no file says stands below as
constants: pre-norm sublayers with layer norms without a bias and a learned scale per element on what they add
(parts/block.py: ``layer_scale``); "mlstm" is a matrix memory with exponential gates (parts/matrix_memory.py);
"latent_attention" keeps one latent vector per position and no rotated part (parts/latent_attention.py); "attention" is
grouped-query attention with neighbouring elements rotated, capped scores that are mixed over the heads and a learned sink
per head (parts/attention.py); both attentions gate every head with one number; the mixture's router takes sigmoids as they
are, on the experts' inputs, and its experts are gated in a clamped form (parts/moe.py); the output head is the embedding
table.  Tensor names: ``embed``, ``l<i>.norm{1,2}``, ``l<i>.ls{1,2}``, ``l<i>.mix.{q,k,v,g,o}``, ``l<i>.mix.{i,f}`` (+ ``.b``),
``l<i>.mix.norm``, ``l<i>.mix.{dkv,uk,uv}``, ``l<i>.mix.dkv.norm``, ``l<i>.mix.{talk,sink}``, ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down}``, ``final.norm``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .dense import ConfigError, _need
from .fipavik import Rotation, _float, _rotation
from .karitar import _obj, _positive

NAME = "Memilorn"

# what the design fixes
ROTATION_PAIRING = "adjacent"       # element 2i turns with element 2i + 1
ROUTER_SCORE = "sigmoid"            # the chosen experts' weights are their scores, not divided by their sum
WEIGHT_ON = "input"                 # the weight multiplies the expert's input
EXPERT_GATE_ALPHA = 1.702           # an expert's gate passes g sigmoid(1.702 g) ...
EXPERT_UP_OFFSET = 1.0              # ... and multiplies the up value plus one, both clamped by the config's limit
MIXER_KINDS = ("mlstm", "latent_attention", "attention")


@dataclass(frozen=True)
class MemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float


@dataclass(frozen=True)
class TalkingAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float        # 0: none
    rot: Optional[Rotation]


@dataclass(frozen=True)
class ClampedExpert:
    ff: int
    limit: Optional[float]


@dataclass(frozen=True)
class MemilornMoe:
    experts: int
    top: int
    expert: ClampedExpert
    shared: Optional[ClampedExpert]


@dataclass(frozen=True)
class MemilornLayer:
    type: str             # one of MIXER_KINDS
    mixer: Union[MemoryMixer, LatentMixer, TalkingAttention]
    mlp: Optional[MemilornMoe]


@dataclass(frozen=True)
class MemilornConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[MemilornLayer, ...]
    loop: Optional[Tuple[int, int, int]]       # (start, stop, times)

    def run_order(self) -> Tuple[Tuple[int, bool], ...]:
        """``(layer, whether the embedding's output is added ahead of it)`` in the order the layers run."""
        start, stop, times = self.loop or (0, 0, 1)
        order = [(i, False) for i in range(start)]
        for turn in range(times):
            order += [(i, turn > 0 and i == start) for i in range(start, stop)]
        return tuple(order + [(i, False) for i in range(stop, len(self.layers))])

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MemilornConfig":
        vocab = _positive(d, "vocab")
        width = _positive(d, "width")
        eps = _positive_float(_obj(d, "norm"), "eps", "norm.")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError("config.json: missing key 'layers' (a non-empty list of layers)")
        layers = tuple(_layer(i, raw) for i, raw in enumerate(raw_layers))
        loop = None
        if d.get("loop") is not None:
            lo = _obj(d, "loop")
            start, stop, times = _need(lo, "start", int), _need(lo, "stop", int), _need(lo, "times", int)
            if not (0 <= start <= stop <= len(layers)) or times < 1:
                raise ConfigError(f"config.json: loop start {start}, stop {stop}, times {times} does not fit "
                                  f"{len(layers)} layers (0 <= start <= stop <= layers, times >= 1)")
            loop = (start, stop, times)
        return cls(architecture=str(d.get("architecture", NAME)), vocab=vocab, width=width, norm_eps=eps, layers=layers, loop=loop)


def _positive_float(d: Mapping[str, Any], key: str, where: str) -> float:
    v = _float(d, key, where)
    if not v > 0:
        raise ConfigError(f"config.json: {where}{key} must be positive, got {v}")
    return v


def _expert(d: Mapping[str, Any], where: str) -> ClampedExpert:
    return ClampedExpert(_positive(d, "ff", where), None if d.get("limit") is None else _positive_float(d, "limit", where))


def _mlp(raw: Any, where: str) -> Optional[MemilornMoe]:
    if raw is None:
        return None
    if not isinstance(raw, Mapping):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    if raw.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}kind = {raw.get('kind')!r} is not supported (known: 'moe')")
    router = _obj(raw, "router")
    experts, top = _positive(router, "experts", where + "router."), _positive(router, "top", where + "router.")
    if top > experts:
        raise ConfigError(f"config.json: {where}router.top {top} exceeds {where}router.experts {experts}")
    shared = None
    if raw.get("shared") is not None:
        shared = _expert(_obj(raw, "shared"), where + "shared.")
    return MemilornMoe(experts, top, _expert(_obj(raw, "expert"), where + "expert."), shared)


def _layer(i: int, raw: Any) -> MemilornLayer:
    where = f"layers[{i}]."
    if not isinstance(raw, Mapping):
        raise ConfigError(f"config.json: layers[{i}] must be an object")
    kind = raw.get("type")
    if kind not in MIXER_KINDS:
        raise ConfigError(f"config.json: {where}type = {kind!r} is not supported (known: {', '.join(map(repr, MIXER_KINDS))})")
    if not isinstance(raw.get("mixer"), Mapping):
        raise ConfigError(f"config.json: {where}mixer must be an object")
    m, mw = raw["mixer"], where + "mixer."
    heads, dim, vdim = _positive(m, "heads", mw), _positive(m, "dim", mw), _positive(m, "vdim", mw)
    if kind == "mlstm":
        mixer = MemoryMixer(heads, dim, vdim, _positive_float(m, "gate_cap", mw))
    elif kind == "latent_attention":
        mixer = LatentMixer(heads, dim, vdim, _positive(m, "kv_rank", mw), _positive_float(m, "scale", mw))
    else:
        kv_heads = _positive(m, "kv_heads", mw)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {mw}heads {heads} is not a multiple of {mw}kv_heads {kv_heads}")
        cap = 0.0 if m.get("softcap") is None else _positive_float(m, "softcap", mw)
        mixer = TalkingAttention(heads, kv_heads, dim, vdim, _positive_float(m, "scale", mw), cap, _rotation(m, mw, dim, "dim"))
    return MemilornLayer(kind, mixer, _mlp(raw.get("mlp"), where + "mlp."))


def _encoding(encodings: Dict[str, PartSpec], rot: Optional[Rotation]) -> Optional[str]:
    """The name of the rotary tables for ``rot`` (layers with the same constants share them)."""
    if rot is None:
        return None
    name = f"rot{rot.dims}@{rot.base!r}"
    if name not in encodings:
        encodings[name] = PartSpec("rotary", {"head_dim": rot.dims, "rotary_dim": rot.dims, "theta": rot.base,
                                              "scaling": None, "pairing": ROTATION_PAIRING})
    return name


_GATED = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}


def _gate(e: ClampedExpert) -> Dict[str, Any]:
    return {"activation": "clamped", "gate_alpha": EXPERT_GATE_ALPHA, "up_offset": EXPERT_UP_OFFSET, "limit": e.limit}


def memilorn_spec(cfg: MemilornConfig) -> ModelSpec:
    """Parts and run order of a Memilorn model (see the module's text for what the design fixes)."""
    norm = {"size": cfg.width, "eps": cfg.norm_eps, "bias": False}
    encodings: Dict[str, PartSpec] = {}
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        common = {"hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim}
        if layer.type == "mlstm":
            mixer = PartSpec("matrix_memory", dict(common, **{
                "gate_cap": m.gate_cap, "norm_eps": cfg.norm_eps,
                "tensor_names": {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "g_proj.weight": "g",
                                 "i_gate.weight": "i", "f_gate.weight": "f", "i_gate.bias": "i.b", "f_gate.bias": "f.b",
                                 "norm.weight": "norm", "o_proj.weight": "o"}}), p + "mix.")
        elif layer.type == "latent_attention":
            mixer = PartSpec("latent_attention", dict(common, **{
                "rot_dim": 0, "kv_rank": m.kv_rank, "norm_eps": cfg.norm_eps, "softmax_scale": m.scale, "head_gate": True,
                "tensor_names": {"q_proj.weight": "q", "kv_down_proj.weight": "dkv", "kv_norm.weight": "dkv.norm",
                                 "k_up_proj.weight": "uk", "v_up_proj.weight": "uv", "gate_proj.weight": "g",
                                 "o_proj.weight": "o"}}), p + "mix.")
        else:
            mixer = PartSpec("attention", dict(common, **{
                "num_kv_heads": m.kv_heads, "qkv_bias": False, "qk_norm": False, "window": 0, "softmax_scale": m.scale,
                "softcap": m.softcap, "head_mix": True, "sink": "learned", "head_gate": True,
                "position": _encoding(encodings, m.rot),
                "tensor_names": {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
                                 "gate_proj.weight": "g", "head_mix.weight": "talk"}}), p + "mix.")

        def scale(name):
            return PartSpec("layer_scale", {"size": cfg.width, "tensor_names": {"weight": name}}, p)

        parts = {"norm1": PartSpec("layernorm", dict(norm, tensor_names={"weight": "norm1"}), p), "mixer": mixer,
                 "scale1": scale("ls1")}
        ml = layer.mlp
        if ml is not None:
            parts["norm2"] = PartSpec("layernorm", dict(norm, tensor_names={"weight": "norm2"}), p)
            parts["ffn"] = PartSpec("moe", {
                "hidden_size": cfg.width, "num_experts": ml.experts, "top": ml.top, "expert_size": ml.expert.ff,
                "router_bias": False, "score": ROUTER_SCORE, "normalize": False, "weight_on": WEIGHT_ON, **_gate(ml.expert),
                "shared_size": ml.shared.ff if ml.shared else 0, "shared_params": _gate(ml.shared) if ml.shared else None,
                "shared_prefix": "shared.", "shared_names": dict(_GATED),
                "tensor_names": {"router.weight": "router", "experts.*.gate_proj.weight": "e*.gate",
                                 "experts.*.up_proj.weight": "e*.up", "experts.*.down_proj.weight": "e*.down"},
            }, p + "mlp.")
            parts["scale2"] = scale("ls2")
        layers.append(LayerSpec("prenorm", parts))
    spec = ModelSpec(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=None,                       # the rotation has no limit of its own: the cache's size is the limit
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width,
                                               "tensor_names": {"weight": "embed"}}, ""),
        encodings=encodings,
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i, add_embedding=again) for i, again in cfg.run_order()),
        final_norm=PartSpec("layernorm", dict(norm, tensor_names={"weight": "final.norm"}), ""),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": "embed"}, ""),
    )
    spec.validate()
    return spec
