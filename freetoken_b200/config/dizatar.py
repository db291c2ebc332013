"""Typed configuration of the Dizatar decoder, read from ``config.json``.

Every sublayer of a Dizatar layer is normed on both sides, scaled element by element and by one
constant before it joins the residual stream ``x`` (``rms(v) = v / sqrt(mean(v^2) + eps) * w``)::

    x <- x + m ls1 rms_1b(mixer(rms_1(x)));   x <- x + m ls2 rms_2b(ff(rms_2(x)))

* mixer ``latent_attention``: queries straight from the input, keys and values made from a normed latent
  of ``kv_rank`` values plus ``rot_dim`` rotated key values shared by the heads (halves ``(i, i + rot_dim/2)``),
  causal softmax over all keys, no gate;
* feed-forward ``moe`` (or null: the layer has the mixer only): experts ``silu(W_gate h) (W_up h)`` chosen by
  ``softmax(router) + correction``, weighted by the uncorrected scores, normalised; the last
  ``router.identity`` outputs of the router hand the input back; a shared expert is added;
* layers ``start .. stop-1`` of ``loop`` run ``times`` times in a row with the same weights, every pass with a
  cache of its own, and before each pass ``x <- W [x ; x0]`` with the embedded row ``x0``;
* ``logits = cap tanh(head rms(x) / cap)``.

config.json keys: ``architecture`` (``"Dizatar"``), ``vocab``, ``width``, ``norm.eps``, ``residual_mult``,
``logit_softcap``, ``loop.{start, stop, times}`` (absent: no layer runs twice and no such matrix exists) and
``layers[i]`` with ``type``, ``mixer`` (``heads, dim, rot_dim, vdim, kv_rank, scale, rot.{base, dims}``) and ``mlp``
(``kind``, ``expert.ff``, ``router.{experts, top, identity}``, ``shared.ff``).  Tensors: ``embed``, ``loop.in``,
``final.norm``, ``head`` and ``l<i>.{norm1, norm1b, ls1, norm2, norm2b, ls2, mix.*, mlp.*}``.  The reference has no
model of this design; the module follows the shape of python/freetoken/models/minimax_m3/args.py:135-254.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .model_plan import ConfigError, LayerSpec, ModelPlan, PartSpec, RunEntry

ARCHITECTURE = "Dizatar"
MIXER_TYPES = ("latent_attention",)
MLP_KINDS = ("moe",)
# the design has no position table and no longest sequence of its own
NO_POSITION_LIMIT = 1 << 30


@dataclass(frozen=True)
class DizatarMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclass(frozen=True)
class DizatarMLP:
    ff: int
    experts: int
    top: int
    identity: int
    shared_ff: int               # 0: no shared expert


@dataclass(frozen=True)
class DizatarLayer:
    type: str
    mixer: DizatarMixer
    mlp: Optional[DizatarMLP]


def _need(d: Any, key: str, where: str) -> Any:
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key '{where}{key}' is missing")
    return d[key]


def _positive(where: str, **values: int) -> None:
    for name, v in values.items():
        if v <= 0:
            raise ConfigError(f"config.json: '{where}{name}' must be positive")


def _read_mixer(m: Any, where: str) -> DizatarMixer:
    rot_dim = int(m.get("rot_dim") or 0)
    base = 1.0
    if rot_dim:
        rot = _need(m, "rot", where)
        base = float(_need(rot, "base", where + "rot."))
        dims = int(rot.get("dims") or rot_dim)
        if dims != rot_dim or dims % 2:
            raise ConfigError(f"config.json: '{where}rot.dims' = {dims} must equal rot_dim = {rot_dim} and be even")
        if base <= 0:
            raise ConfigError(f"config.json: '{where}rot.base' must be positive")
    heads, dim = int(_need(m, "heads", where)), int(_need(m, "dim", where))
    a = DizatarMixer(heads=heads, dim=dim, rot_dim=rot_dim, vdim=int(m.get("vdim") or dim),
                     kv_rank=int(_need(m, "kv_rank", where)), scale=float(_need(m, "scale", where)), rot_base=base)
    _positive(where, heads=a.heads, dim=a.dim, vdim=a.vdim, kv_rank=a.kv_rank)
    if rot_dim < 0:
        raise ConfigError(f"config.json: '{where}rot_dim' must not be negative")
    if a.kv_rank + a.rot_dim > 1024:
        raise ConfigError(f"config.json: '{where}kv_rank' + rot_dim above 1024 is not supported")
    return a


def _read_mlp(mlp: Any, where: str) -> Optional[DizatarMLP]:
    if not mlp:
        return None
    kind = str(mlp.get("kind", "moe"))
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: '{where}kind' = {kind!r} is not one of {list(MLP_KINDS)}")
    expert, router = _need(mlp, "expert", where), _need(mlp, "router", where)
    shared = mlp.get("shared")
    out = DizatarMLP(ff=int(_need(expert, "ff", where + "expert.")),
                     experts=int(_need(router, "experts", where + "router.")),
                     top=int(_need(router, "top", where + "router.")), identity=int(router.get("identity") or 0),
                     shared_ff=int(_need(shared, "ff", where + "shared.")) if shared else 0)
    _positive(where, ff=out.ff, experts=out.experts, top=out.top)
    if out.identity < 0 or out.shared_ff < 0 or (shared and not out.shared_ff):
        raise ConfigError(f"config.json: '{where}' router.identity must not be negative, shared.ff must be positive")
    if out.top > out.experts + out.identity:
        raise ConfigError(f"config.json: '{where}router.top' = {out.top} exceeds the router's "
                          f"{out.experts + out.identity} outputs")
    return out


@dataclass(frozen=True)
class DizatarConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: float         # 0: the logits are not capped
    layers: Tuple[DizatarLayer, ...]
    loop: Optional[Tuple[int, int, int]]     # start, stop, times
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "DizatarConfig":
        listed = _need(raw, "layers", "")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[DizatarLayer] = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]."
            kind = str(_need(entry, "type", where))
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: '{where}type' = {kind!r} is not one of {list(MIXER_TYPES)}")
            layers.append(DizatarLayer(kind, _read_mixer(_need(entry, "mixer", where), where + "mixer."),
                                       _read_mlp(entry.get("mlp"), where + "mlp.")))
        loop = None
        if raw.get("loop"):
            loop = tuple(int(_need(raw["loop"], key, "loop.")) for key in ("start", "stop", "times"))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"config.json: 'loop' {loop[0]}..{loop[1]} x {loop[2]} does not fit "
                                  f"{len(layers)} layers")
        mult = raw.get("residual_mult")
        cfg = cls(vocab=int(_need(raw, "vocab", "")), width=int(_need(raw, "width", "")),
                  norm_eps=float(_need(_need(raw, "norm", ""), "eps", "norm.")),
                  residual_mult=1.0 if mult is None else float(mult),
                  logit_softcap=float(raw.get("logit_softcap") or 0.0), layers=tuple(layers), loop=loop,
                  raw=dict(raw))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if cfg.norm_eps < 0 or cfg.logit_softcap < 0:
            raise ConfigError("config.json: 'norm.eps' and 'logit_softcap' must not be negative")
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    def schedule(self) -> Tuple[RunEntry, ...]:
        """Layers in the order they run: the looped span ``times`` times in a row, its first layer
        behind the map of the stream each time."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(RunEntry(i) for i in range(n))
        start, stop, times = self.loop
        span = [RunEntry(i, stream_map=0 if i == start else None) for i in range(start, stop)]
        return tuple([RunEntry(i) for i in range(start)] + span * times + [RunEntry(i) for i in range(stop, n)])


def _mixer_spec(cfg: DizatarConfig, m: DizatarMixer) -> PartSpec:
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "qk_dim": m.dim, "v_dim": m.vdim, "rank": m.kv_rank,
        "sm_scale": m.scale, "norm_eps": cfg.norm_eps, "output_gate": False, "rot_dim": m.rot_dim, "scope": "mix",
        "position": PartSpec("rotary_neox", {"head_dim": max(m.rot_dim, 2), "rotary_dim": m.rot_dim,
                                             "theta": m.rot_base, "max_position": NO_POSITION_LIMIT,
                                             "exact_angles": True}),
        "names": {"q": "q", "down": "dkv", "latent_norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "o": "o",
                  "in": "q_dkv"}})


def _mlp_spec(cfg: DizatarConfig, mlp: DizatarMLP) -> PartSpec:
    shared = None
    if mlp.shared_ff:
        shared = PartSpec("dense_mlp", {"hidden_size": cfg.width, "intermediate_size": mlp.shared_ff,
                                        "activation": "silu", "gated": True, "scope": "mlp.shared",
                                        "names": {"gate": "gate", "up": "up", "down": "down", "gate_up": "gate_up"}})
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "intermediate_size": mlp.ff, "num_experts": mlp.experts, "top_k": mlp.top,
        "identity": mlp.identity, "shared": shared, "scoring": "softmax", "use_bias": True, "renormalize": True,
        "scale": 1.0, "activation": "silu", "scope": "mlp",
        "checkpoint_names": {"router": "router", "bias": "correction", "gate_up": "experts.gate_up",
                             "down": "experts.down", "gate": "e{e}.gate", "up": "e{e}.up",
                             "down_each": "e{e}.down"}})


def build_plan(cfg: DizatarConfig) -> ModelPlan:
    W = cfg.width

    def norm(tensor: str, scale: Optional[str] = None) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": cfg.norm_eps, "plus_one": False, "tensor": tensor,
                                    "scale_tensor": scale})

    layers: List[LayerSpec] = []
    for i, layer in enumerate(cfg.layers):
        ffn = _mlp_spec(cfg, layer.mlp) if layer.mlp is not None else None
        norms = {"mixer_out": norm("norm1b", "ls1")}
        if ffn is not None:
            norms["feed_forward_out"] = norm("norm2b", "ls2")
        layers.append(LayerSpec(
            prefix=f"l{i}", block=PartSpec("sandwich", {"residual_mult": cfg.residual_mult}),
            mixer=_mixer_spec(cfg, layer.mixer), feed_forward=ffn, mixer_norm=norm("norm1"),
            feed_forward_norm=norm("norm2") if ffn is not None else None, norms=norms))
    plan = ModelPlan(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "prefix": "",
                                               "tensor": "embed"}),
        layers=tuple(layers), schedule=cfg.schedule(),
        final_norm=PartSpec("rmsnorm", {**norm("final.norm").params, "prefix": ""}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": W, "prefix": "", "tensor": "head",
                                  "tied_to": None, "softcap": cfg.logit_softcap}),
        stream_maps=() if cfg.loop is None else (PartSpec("embedding_mix", {"hidden_size": W, "prefix": "",
                                                                            "tensor": "loop.in"}),),
        max_position=NO_POSITION_LIMIT)
    plan.validate()
    return plan
