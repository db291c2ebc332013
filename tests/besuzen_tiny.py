"""Tiny Besuzen configurations, random weights for them, and helpers of the tests.

The configurations differ from each other in every size and constant: widths, head counts (one, equal and
unequal query and key/value heads), key sizes below, equal to and above value sizes, rotation of none, a part
and all of a head, layers with and without value mixing (none, one, several, another layer between them), time
mixers with other heads than the attention beside them, middles of the decay projection of any width, groups
of experts of one, two and more of which one, some or all are kept, with and without a shared expert, layers
without feed-forward, scales above, below and equal to 1, every layer order.
"""

from __future__ import annotations

import copy
from typing import Dict, List

import torch

import plain_besuzen as plain
from fazinex_tiny import make_engine, position_errors, tokens, write_model  # noqa: F401  (re-exported)


def attention(heads, kv_heads, dim, vdim, rot_dims, base=10000.0, v_mix=True, scale=None, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                           "scale": scale or dim ** -0.5, "v_mix": v_mix,
                                           "rot": {"base": base, "dims": rot_dims}}, "mlp": mlp}


def parallel(left, right, left_scale=0.7, right_scale=0.9, mlp=None, scale=None):
    """``left``: (heads, kv_heads, dim, vdim); ``right``: (heads, dim, low_rank)."""
    heads, kv_heads, dim, vdim = left
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5},
                      "right": {"heads": right[0], "dim": right[1], "low_rank": right[2]},
                      "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, count, keep, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff},
           "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, layers, embedding_scale=1.0, logit_scale=1.0):
    return {"architecture": "Besuzen", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embedding_scale}, "logit_scale": logit_scale, "layers": layers}


# awkward sizes, nothing a multiple of 8; a layer without value mixing between two that mix; layers without
# feed-forward; no shared expert in one routed layer, no groups in another
BZ_A: Dict = model(150, 44, 1e-5, [
    parallel((3, 1, 10, 6), (2, 9, 5), 1.3, 0.4, moe(6, 2, 20, 3, 2, shared=14)),
    attention(4, 2, 12, 10, 6, base=100.0, mlp=dense(30)),
    attention(2, 2, 6, 14, 6, base=300.0, v_mix=False),
    attention(6, 2, 22, 10, 4, base=50.0, scale=0.3, mlp=moe(4, 3, 24, 1, 1)),
    parallel((2, 2, 5, 9), (3, 20, 1), 0.5, 1.1),
], embedding_scale=1.7, logit_scale=0.6)

# sizes the tensor-core attention kernels take, some filled up to them (40 and 56 to 64, 80 to 128), pages of 64
BZ_B: Dict = model(320, 128, 2e-6, [
    attention(8, 2, 64, 64, 32, base=5000.0, mlp=moe(8, 2, 64, 4, 2, shared=96)),
    parallel((4, 2, 64, 80), (4, 32, 16), 0.6, 0.8, dense(256)),
    attention(6, 2, 56, 64, 40, base=500000.0, mlp=moe(6, 1, 48, 6, 3, shared=64)),
    attention(2, 2, 32, 64, 16, v_mix=False, base=30000.0),
    parallel((6, 6, 32, 32), (2, 64, 24), 1.0, 1.0, moe(16, 4, 32, 2, 1)),
    attention(8, 2, 40, 64, 24, base=1000.0, mlp=dense(192)),
], embedding_scale=0.8, logit_scale=1.5)

# one value-mixing layer alone; one head; one expert of one; a width that is no multiple of 4 (no 16-byte
# pieces anywhere along a row of the residual); nothing rotates in one layer
BZ_C: Dict = model(97, 70, 1e-4, [
    parallel((1, 1, 33, 9), (1, 33, 3), 0.9, 0.9, moe(1, 1, 30, 1, 1, shared=20)),
    attention(6, 3, 8, 12, 8, base=1000.0, mlp=moe(8, 4, 16, 2, 2)),
    parallel((6, 2, 7, 7), (5, 8, 11), 2.0, 0.25, dense(100)),
    attention(1, 1, 40, 36, 0, v_mix=False, mlp=moe(9, 2, 12, 9, 4, shared=33)),
])

BZ = {"A": BZ_A, "B": BZ_B, "C": BZ_C}
PAGE = {"A": 4, "B": 64, "C": 12}
SEEDS = {"A": 81, "B": 82, "C": 83}


def random_state(config: Dict, seed: int, slow_decay: bool = False) -> Dict[str, torch.Tensor]:
    """Every tensor of a model of ``config`` by name, drawn so that activations stay of order one and
    rounded to bfloat16 (what the file holds), as float64.  ``slow_decay``: states that forget slowly, so
    that a token far back still counts."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in plain.expected_tensors(config).items():
        leaf = name.rsplit(".", 1)[-1]
        std, mean = (shape[-1] ** -0.5 if len(shape) > 1 else 1.0), 0.0
        if leaf in ("norm1", "norm2", "norm"):
            std, mean = 0.2, 1.0
        elif leaf == "b":
            std = 0.3
        elif leaf == "vmix":
            std, mean = 0.1, 0.45
        elif ".mu." in name:
            std, mean = 0.3, 0.5
        elif leaf == "w0":
            std, mean = 1.0, -7.0 if slow_decay else -1.0
        elif leaf == "w2":
            std = 0.5 * shape[-1] ** -0.5
        elif leaf == "u":
            std, mean = 0.5, 0.3
        elif leaf == "embed":
            std = 1.0
        elif leaf in ("router", "sg"):
            std = 2.0 * shape[-1] ** -0.5
        t = torch.randn(tuple(shape), generator=g, dtype=torch.float64) * std + mean
        out[name] = t.to(torch.bfloat16).double()
    return out


def file_config(config: Dict) -> Dict:
    """``config`` as a checkpoint's config.json states it: without the size that only tensor shapes give."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        if layer["type"] == "parallel":
            layer["mixer"]["right"].pop("low_rank", None)
    return out


def as_file(state: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    return {k: v.to(torch.bfloat16) for k, v in state.items()}


def write(folder: str, config: Dict, state: Dict[str, torch.Tensor]) -> str:
    return write_model(folder, file_config(config), as_file(state))


def write_tiny(folder: str, which: str) -> str:
    return write(folder, BZ[which], random_state(BZ[which], SEEDS[which]))


def several(layers, vocab=90, width=48, eps=1e-6, embedding_scale=1.2, logit_scale=0.8) -> Dict:
    return model(vocab, width, eps, copy.deepcopy(layers), embedding_scale, logit_scale)


def routed_layers(config: Dict) -> List[int]:
    return [i for i, l in enumerate(config["layers"]) if l["mlp"] and l["mlp"]["kind"] == "moe"]


# Largest allowed error of a position's logits (see fazinex_tiny.position_errors).  float32: summation
# orders differ, and recurrences carry their rounding along.  bfloat16: every stored activation is
# rounded to 8 bits; a lost state, a lost key, a shift from the wrong row or values that were not mixed give
# 0.2 and more.
TOL = {"float32": 5e-5, "bfloat16": 6e-2}


def rounding_noise(config: Dict, state, toks: List[int], want: torch.Tensor, expert_ids=None, draws: int = 3) -> torch.Tensor:
    """How far rounding alone moves each position: the largest error of the plain model over a few runs in
    which everything a 16-bit engine stores is off by up to half a unit in the last place.  A head of the time mixer
    divides its read-out by its root mean square; where the read-out nearly vanishes (a first token whose r, u and k
    are nearly orthogonal) its direction hangs on such a rounding."""
    worst = torch.zeros(len(toks), dtype=torch.float64)
    for draw in range(draws):
        g = torch.Generator().manual_seed(1000 + draw)
        store = lambda v: v * (1.0 + (2.0 * torch.rand(v.shape, generator=g, dtype=torch.float64) - 1.0) * 2.0 ** -8)
        got = plain.forward(config, state, toks, expert_ids=expert_ids, store=store)
        worst = torch.maximum(worst, position_errors(got, want))
    return worst


def compare(got: Dict[str, torch.Tensor], want: Dict[str, torch.Tensor], tol: float, what: str, noise=None,
            mostly: float = 0.9) -> None:
    """Every position of every request within ``tol``; in bfloat16 (``noise`` given: :func:`rounding_noise` by
    request) within the larger of ``tol`` and four times what rounding alone does there, where one position in fifty
    of a request (at least one) may lie between that and twice that.  The share ``mostly`` of the positions must be bound by ``tol``."""
    bound = total = 0
    for rid, w in want.items():
        g = got[rid]
        assert not torch.isnan(g).any(), f"{what}: request {rid} has positions without logits (or NaN)"
        err = position_errors(g, w)
        limit = torch.full_like(err, tol) if noise is None else (4.0 * noise[rid]).clamp(min=tol)
        bound, total = bound + int((limit == tol).sum()), total + len(err)
        over = err > limit
        allowed = max(1, len(w) // 50) if tol > 1e-3 else 0
        if int(over.sum()) > allowed or (err > 2 * limit).any():
            pos = int(over.nonzero()[0])
            raise AssertionError(f"{what}: request {rid}: first wrong position {pos} of {len(w)} (error "
                                 f"{float(err[pos]):.3e}, limit {float(limit[pos]):.3e}, worst {float(err.max()):.3e}, "
                                 f"{int(over.sum())} positions over their limit)")
    assert bound >= mostly * total, f"{what}: only {bound} of {total} positions are bound by {tol:.1e}"
