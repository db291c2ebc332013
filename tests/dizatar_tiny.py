"""Tiny Dizatar configurations, random weights for them, and helpers of the tests.

The configurations differ from each other in every size and constant: widths, head counts (odd ones, one,
more than 16), unrotated, rotated and value sizes in every order, latents narrower and wider than the heads,
cached rows no kernel but the generic one takes, rows of the tensor-core kernels' own and of the paged
kernels' sizes, rows of more than 512 values; loops over the first layer, the middle, everything, none and
a single pass; experts with and without a shared one, none to many that hand their input back, one to all
chosen; layers without feed-forward; with and without a cap and a residual factor.
"""

from __future__ import annotations

import copy
from typing import Dict, List, Optional

import torch

import plain_dizatar as plain
from fazinex_tiny import make_engine, position_errors, tokens, write_model  # noqa: F401  (re-exported)
from tonapel_tiny import compare  # noqa: F401  (re-exported)


def layer(heads, dim, rot_dim, vdim, kv_rank, mlp=None, base=10000.0, scale=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
             "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}
    if not rot_dim:
        del mixer["rot"]
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def moe(experts, top, ff, identity=0, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, layers, eps=1e-6, mult: Optional[float] = None, cap: Optional[float] = None, loop=None):
    out = {"architecture": "Dizatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if mult is not None:
        out["residual_mult"] = mult
    if cap is not None:
        out["logit_softcap"] = cap
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# awkward sizes: nothing a multiple of 8 (the generic kernels everywhere), pages of 4
DZ_A: Dict = model(150, 42, [
    layer(3, 7, 6, 5, 11, moe(5, 3, 18, identity=2, shared=30), base=100.0),
    layer(2, 10, 2, 13, 9, None, base=700.0),
    layer(5, 4, 4, 6, 21, moe(4, 1, 22, identity=1), scale=0.6),
    layer(1, 9, 8, 3, 14, moe(3, 2, 10, shared=14)),
], eps=1e-5, mult=0.55, cap=2.0, loop=(1, 3, 2))

# rows of the own tensor-core kernels (88, 160 and 264 values), pages of 64: 5, 20 and 2 heads; the span at
# the end loops
DZ_B: Dict = model(320, 128, [
    layer(5, 24, 8, 40, 80, moe(8, 3, 64, identity=3, shared=96)),
    layer(20, 40, 32, 24, 128, moe(6, 2, 48, identity=1, shared=40), base=5000.0),
    layer(2, 72, 64, 112, 200, moe(4, 4, 32, identity=2)),
], eps=2e-6, mult=0.8, cap=3.0, loop=(1, 3, 3))

# one pass of everything, no cap, no factor; rows of 64 and 128 values (the paged kernels), nothing rotated,
# one expert beside three that hand the input back, all of them chosen
DZ_C: Dict = model(97, 72, [
    layer(4, 16, 16, 24, 48, moe(1, 4, 24, identity=3, shared=16)),
    layer(3, 32, 32, 8, 96, moe(2, 1, 40, identity=6)),
    layer(6, 8, 0, 16, 40, moe(6, 2, 16, shared=8)),
], eps=1e-4, loop=(0, 3, 1))

# no loop at all; a cached row of 544 values
DZ_D: Dict = model(110, 64, [
    layer(2, 16, 24, 32, 520, moe(3, 1, 24, shared=32), base=50.0),
    layer(17, 8, 8, 8, 16, None),
], mult=1.3, cap=1.0)

DZ = {"A": DZ_A, "B": DZ_B, "C": DZ_C, "D": DZ_D}
PAGE = {"A": 4, "B": 64, "C": 64, "D": 16}
SEEDS = {"A": 71, "B": 72, "C": 73, "D": 74}


def random_state(config: Dict, seed: int) -> Dict[str, torch.Tensor]:
    """Every tensor of a model of ``config`` by name, drawn so that activations stay of order one and
    rounded to bfloat16 (what the file holds), as float64."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in plain.expected_tensors(config).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        std, mean = (shape[-1] ** -0.5 if len(shape) > 1 else 1.0), 0.0
        if len(shape) == 1 and leaf != "mlp.correction":
            std, mean = 0.25, 1.0
        elif leaf == "mlp.correction":
            std = 0.1
        elif leaf == "embed":
            std = 1.0
        elif leaf == "mlp.router":
            std = 2.0 * shape[-1] ** -0.5
        t = torch.randn(*shape, generator=g, dtype=torch.float64) * std + mean
        out[name] = t.to(torch.bfloat16).double()
    return out


def write(folder: str, config: Dict, state: Dict[str, torch.Tensor]) -> str:
    return write_model(folder, config, {k: v.to(torch.bfloat16) for k, v in state.items()})


def write_tiny(folder: str, which: str) -> str:
    return write(folder, DZ[which], random_state(DZ[which], SEEDS[which]))


def one_layer(spec: Dict, vocab=90, width=48, **kw) -> Dict:
    return model(vocab, width, [copy.deepcopy(spec)], **kw)


def routed_runs(config: Dict) -> List[int]:
    """The layer runs that route, in order."""
    return [run for run, (i, _) in enumerate(plain.run_order(config)) if config["layers"][i]["mlp"]]


# Largest allowed error of a position's logits (see fazinex_tiny.position_errors).  float32: summation
# orders differ.  bfloat16: every stored activation is rounded to 8 bits; a lost key, a wrong expert, a
# forgotten map of the stream or a layer scale that is left out gives 0.2 and more.
TOL = {"float32": 5e-5, "bfloat16": 6e-2}
