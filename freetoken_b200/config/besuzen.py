"""Typed configuration of the Besuzen decoder, read from ``config.json``.

Both sublayers of a Besuzen layer read the same residual row, each through a layer norm of its own (weight, no
bias), and join it together; the embedded row is scaled, and so are the logits::

    x_0 = embed[token] * c_e;   x <- x + (mixer(ln1(x)) + ff(ln2(x)));   logits = c_l * head ln(x)

* mixer ``attention``: grouped-query attention with biased q, k and v, interleaved rotary positions on the first
  ``rot.dims`` dimensions of a head, a sigmoid gate per output value, and values blended with those of the first
  layer that says ``v_mix``: ``v <- (1 - l) v + l v_first`` (the blended values are what is cached);
* mixer ``parallel``: ``left_scale * left + right_scale * right`` of the same input; left: attention without
  positions, biased q, k and v, a sigmoid gate per head; right: time mixing - projections that read mixes of the
  token's and the previous token's input, a state that decays per key channel, a bonus for the current token.
  The width of the middle of the decay's two-step projection is the one size config.json does not state: it is
  read from the checkpoint's tensor shapes (:func:`sizes_from_tensors`), or given as ``mixer.right.low_rank`` for a
  model without a checkpoint;
* feed-forward ``dense``: gated with tanh-GELU; ``moe``: experts ``silu(W_gate h) (W_up h)`` chosen by
  ``softmax(router)`` inside the ``groups.keep`` best of ``groups.count`` groups of neighbours (a group's value: its
  largest score), weighted by the scores, normalised; a shared expert, if there is one, is added times one
  sigmoid gate per token; ``null``: the layer has the mixer only.

config.json keys: ``architecture`` (``"Besuzen"``), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``logit_scale`` and ``layers[i]`` with ``type``, ``mixer`` (attention: ``heads, kv_heads, dim, vdim, scale, v_mix,
rot.{base, dims}``; parallel: ``left.{heads, kv_heads, dim, vdim, scale}``, ``right.{heads, dim}``, ``left_scale``,
``right_scale``) and ``mlp`` (dense: ``kind, ff``; moe: ``kind, expert.ff, router.{experts, top, groups.{count, keep}},
shared.ff``).  Tensors: ``embed``, ``final.norm``, ``head`` and ``l<i>.{norm1, norm2, mix.*, mlp.*}``.  The reference has no
model of this design; the module follows the shape of python/freetoken/models/minimax_m3/args.py:135-254.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .model_plan import ConfigError, LayerSpec, ModelPlan, PartSpec, RunEntry

ARCHITECTURE = "Besuzen"
MIXER_TYPES = ("attention", "parallel")
MLP_KINDS = ("dense", "moe")
# the design has no position table and no longest sequence of its own
NO_POSITION_LIMIT = 1 << 30


@dataclass(frozen=True)
class BesuzenAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float = 1.0
    rot_dims: int = 0            # 0: no rotation
    v_mix: bool = False


@dataclass(frozen=True)
class BesuzenTimeMixing:
    heads: int
    dim: int
    low_rank: int


@dataclass(frozen=True)
class BesuzenParallel:
    left: BesuzenAttention
    right: BesuzenTimeMixing
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class BesuzenMLP:
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0           # 0: no shared expert


@dataclass(frozen=True)
class BesuzenLayer:
    type: str
    mixer: Any
    mlp: Optional[BesuzenMLP]


def _need(d: Any, key: str, where: str) -> Any:
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key '{where}{key}' is missing")
    return d[key]


def _positive(where: str, **values: int) -> None:
    for name, v in values.items():
        if v <= 0:
            raise ConfigError(f"config.json: '{where}{name}' must be positive")


def _number(d: Mapping[str, Any], key: str, default: float) -> float:
    return default if d.get(key) is None else float(d[key])


def _read_attention(m: Any, where: str, rotates: bool) -> BesuzenAttention:
    heads, dim = int(_need(m, "heads", where)), int(_need(m, "dim", where))
    base, dims = 1.0, 0
    if rotates:
        rot = _need(m, "rot", where)
        base, dims = float(_need(rot, "base", where + "rot.")), int(_need(rot, "dims", where + "rot."))
        if dims < 0 or dims % 2 or dims > dim:
            raise ConfigError(f"config.json: '{where}rot.dims' = {dims} must be even and at most dim = {dim}")
        if dims and base <= 0:
            raise ConfigError(f"config.json: '{where}rot.base' must be positive")
    a = BesuzenAttention(heads=heads, kv_heads=int(m.get("kv_heads") or heads), dim=dim, vdim=int(m.get("vdim") or dim),
                         scale=float(_need(m, "scale", where)), rot_base=base, rot_dims=dims,
                         v_mix=bool(m.get("v_mix", False)) if rotates else False)
    _positive(where, heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim)
    if a.heads % a.kv_heads:
        raise ConfigError(f"config.json: '{where}kv_heads' = {a.kv_heads} does not divide heads = {a.heads}")
    if max(a.dim, a.vdim) > 1024:
        raise ConfigError(f"config.json: '{where}dim' and vdim above 1024 are not supported")
    return a


def _read_time_mixing(m: Any, where: str) -> BesuzenTimeMixing:
    r = BesuzenTimeMixing(heads=int(_need(m, "heads", where)), dim=int(_need(m, "dim", where)),
                          low_rank=int(m.get("low_rank") or 0))
    _positive(where, heads=r.heads, dim=r.dim)
    if r.dim > 256:
        raise ConfigError(f"config.json: '{where}dim' above 256 is not supported")
    if r.low_rank <= 0:
        raise ConfigError(f"config.json: '{where}low_rank' is neither given nor known from the checkpoint's tensor "
                          f"shapes (the width of the middle of the decay's two-step projection)")
    return r


def _read_mixer(kind: str, m: Any, where: str) -> Any:
    if kind == "attention":
        return _read_attention(m, where, rotates=True)
    return BesuzenParallel(_read_attention(_need(m, "left", where), where + "left.", rotates=False),
                           _read_time_mixing(_need(m, "right", where), where + "right."),
                           _number(m, "left_scale", 1.0), _number(m, "right_scale", 1.0))


def _read_mlp(mlp: Any, where: str) -> Optional[BesuzenMLP]:
    if not mlp:
        return None
    kind = str(mlp.get("kind", "dense"))
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: '{where}kind' = {kind!r} is not one of {list(MLP_KINDS)}")
    if kind == "dense":
        out = BesuzenMLP("dense", int(_need(mlp, "ff", where)))
        _positive(where, ff=out.ff)
        return out
    expert, router, shared = _need(mlp, "expert", where), _need(mlp, "router", where), mlp.get("shared")
    groups = router.get("groups") or {}
    count = int(groups.get("count", 1))
    out = BesuzenMLP("moe", int(_need(expert, "ff", where + "expert.")),
                     experts=int(_need(router, "experts", where + "router.")),
                     top=int(_need(router, "top", where + "router.")), groups=count,
                     keep=int(groups.get("keep", count)),
                     shared_ff=int(_need(shared, "ff", where + "shared.")) if shared else 0)
    _positive(where, ff=out.ff, experts=out.experts, top=out.top, groups=out.groups, keep=out.keep)
    if shared:
        _positive(where + "shared.", ff=out.shared_ff)
    if out.top > out.experts:
        raise ConfigError(f"config.json: '{where}router.top' = {out.top} exceeds experts = {out.experts}")
    if out.experts % out.groups or out.keep > out.groups or out.groups > 256:
        raise ConfigError(f"config.json: '{where}router.groups' = {out.groups} (keep {out.keep}) must divide "
                          f"experts = {out.experts}, keep at most count, count at most 256")
    if out.keep * (out.experts // out.groups) < out.top:
        raise ConfigError(f"config.json: '{where}router.top' = {out.top} experts do not fit into "
                          f"{out.keep} groups of {out.experts // out.groups}")
    return out


@dataclass(frozen=True)
class BesuzenConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[BesuzenLayer, ...]
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "BesuzenConfig":
        listed = _need(raw, "layers", "")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[BesuzenLayer] = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]."
            kind = str(_need(entry, "type", where))
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: '{where}type' = {kind!r} is not one of {list(MIXER_TYPES)}")
            layers.append(BesuzenLayer(kind, _read_mixer(kind, _need(entry, "mixer", where), where + "mixer."),
                                       _read_mlp(entry.get("mlp"), where + "mlp.")))
        blending = [(i, layer.mixer) for i, layer in enumerate(layers) if layer.type == "attention" and layer.mixer.v_mix]
        for i, m in blending[1:]:
            first = blending[0][1]
            if (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                raise ConfigError(f"config.json: 'layers[{i}].mixer' blends its values ({m.kv_heads} x {m.vdim}) with those "
                                  f"of layer {blending[0][0]} ({first.kv_heads} x {first.vdim})")
        cfg = cls(vocab=int(_need(raw, "vocab", "")), width=int(_need(raw, "width", "")),
                  norm_eps=float(_need(_need(raw, "norm", ""), "eps", "norm.")),
                  embedding_scale=_number(raw.get("embedding") or {}, "scale", 1.0),
                  logit_scale=_number(raw, "logit_scale", 1.0), layers=tuple(layers), raw=dict(raw))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if cfg.norm_eps < 0:
            raise ConfigError("config.json: 'norm.eps' must not be negative")
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

def sizes_from_tensors(raw: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Dict[str, Any]:
    """``raw`` with the size that only the checkpoint states filled in: the width of the middle of a time
    mixer's decay projection is the number of rows of ``l<i>.mix.right.w1``."""
    out = dict(raw)
    layers = []
    for i, entry in enumerate(raw.get("layers") or []):
        if isinstance(entry, Mapping) and entry.get("type") == "parallel" and isinstance(entry.get("mixer"), Mapping):
            right, shape = entry["mixer"].get("right"), shapes.get(f"l{i}.mix.right.w1")
            if shape and isinstance(right, Mapping) and not right.get("low_rank"):
                entry = {**entry, "mixer": {**entry["mixer"], "right": {**right, "low_rank": int(shape[0])}}}
        layers.append(entry)
    out["layers"] = layers
    return out


def _attention_spec(cfg: BesuzenConfig, a: BesuzenAttention, scope: str, gate: str, value_mix: Optional[str]) -> PartSpec:
    position = PartSpec("none", {})
    if a.rot_dims:
        position = PartSpec("rotary_interleaved", {"head_dim": a.dim, "rotary_dim": a.rot_dims, "theta": a.rot_base,
                                                   "max_position": NO_POSITION_LIMIT, "exact_angles": True})
    return PartSpec("paged_attention", {
        "hidden_size": cfg.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim,
        "value_dim": a.vdim, "sm_scale": a.scale, "qk_norm": "none", "sliding_window": None, "bias": True,
        "o_bias": False, "gate": gate, "value_mix": value_mix, "fill_heads": True, "position": position, "scope": scope,
        "checkpoint_names": {"qkv": "qkvg", "q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "q_norm": "q.norm",
                             "k_norm": "k.norm", "qkv_bias": "qkv.b", "q_bias": "q.b", "k_bias": "k.b",
                             "v_bias": "v.b", "value_mix": "vmix"}})


def _mixer_spec(cfg: BesuzenConfig, layer: BesuzenLayer, value_mix: Optional[str]) -> PartSpec:
    m = layer.mixer
    if layer.type == "attention":
        return _attention_spec(cfg, m, "mix", "element", value_mix)
    left = _attention_spec(cfg, m.left, "mix.left", "head", None)
    right = PartSpec("time_mixing", {
        "hidden_size": cfg.width, "heads": m.right.heads, "key_dim": m.right.dim, "head_dim": m.right.dim,
        "low_rank": m.right.low_rank, "norm_eps": cfg.norm_eps, "scope": "mix.right",
        "names": {"mu_r": "mu.r", "mu_k": "mu.k", "mu_v": "mu.v", "mu_g": "mu.g", "mu_w": "mu.w", "mu": "mu",
                  "r": "r", "k": "k", "v": "v", "gate": "g", "rkvg": "rkvg", "decay_down": "w1", "decay_up": "w2",
                  "w0": "w0", "u": "u", "norm": "norm", "o": "o"}})
    return PartSpec("mixer_sum", {"hidden_size": cfg.width, "members": (left, right),
                                  "scales": (m.left_scale, m.right_scale)})


def _glu_spec(cfg: BesuzenConfig, ff: int, activation: str, scope: str) -> PartSpec:
    return PartSpec("dense_mlp", {"hidden_size": cfg.width, "intermediate_size": ff, "activation": activation,
                                  "gated": True, "scope": scope,
                                  "names": {"gate": "gate", "up": "up", "down": "down", "gate_up": "gate_up"}})


def _mlp_spec(cfg: BesuzenConfig, mlp: BesuzenMLP) -> PartSpec:
    if mlp.kind == "dense":
        return _glu_spec(cfg, mlp.ff, "gelu_tanh", "mlp")
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "intermediate_size": mlp.ff, "num_experts": mlp.experts, "top_k": mlp.top,
        "scoring": "softmax", "use_bias": False, "renormalize": True, "scale": 1.0,
        "groups": mlp.groups, "keep_groups": mlp.keep, "group_top": 1,
        "shared": _glu_spec(cfg, mlp.shared_ff, "silu", "mlp.shared") if mlp.shared_ff else None,
        "shared_gate": bool(mlp.shared_ff), "activation": "silu", "scope": "mlp",
        "checkpoint_names": {"router": "router", "bias": "router.bias", "shared_gate": "shared.sg",
                             "router_gate": "router_sg", "gate_up": "experts.gate_up", "down": "experts.down",
                             "gate": "e{e}.gate", "up": "e{e}.up", "down_each": "e{e}.down"}})


def build_plan(cfg: BesuzenConfig) -> ModelPlan:
    W = cfg.width

    def norm(tensor: str, **more: Any) -> PartSpec:
        return PartSpec("layer_norm", {"size": W, "eps": cfg.norm_eps, "tensor": tensor, **more})

    layers: List[LayerSpec] = []
    source_seen = False
    for i, layer in enumerate(cfg.layers):
        value_mix = None
        if layer.type == "attention" and layer.mixer.v_mix:
            value_mix, source_seen = ("blend" if source_seen else "source"), True
        ffn = _mlp_spec(cfg, layer.mlp) if layer.mlp is not None else None
        layers.append(LayerSpec(
            prefix=f"l{i}", block=PartSpec("parallel_norms", {}), mixer=_mixer_spec(cfg, layer, value_mix),
            feed_forward=ffn, mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2") if ffn is not None else None))
    plan = ModelPlan(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "prefix": "",
                                               "tensor": "embed", "scale": cfg.embedding_scale}),
        layers=tuple(layers), schedule=tuple(RunEntry(i) for i in range(len(layers))),
        # the factor on the logits rides in the last norm: no pass over the logits
        final_norm=norm("final.norm", factor=cfg.logit_scale, prefix=""),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": W, "prefix": "", "tensor": "head",
                                  "tied_to": None}),
        max_position=NO_POSITION_LIMIT)
    plan.validate()
    return plan
