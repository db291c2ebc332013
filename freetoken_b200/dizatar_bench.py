"""Dizatar beside the Nirelix decoder at equal size: step throughput and kernel rooflines.

    python bench.py --design dizatar [--sizes w2048,w4096] [--steps K] [--warmup W]

For every size a four-layer Dizatar model whose middle two layers run twice (six layer runs, two maps of
the stream; latent attention over rows of 512 + 64 values, experts of which a quarter hand their input
back, a shared expert; random weights) and the engine's closest other model - a Nirelix decoder of six
latent-attention layers with the same head counts, head sizes, latent and experts, one residual stream
and a window longer than the context - run the same workload through ``Engine.step`` (the method of
:mod:`.design_bench`): one prompt of ``--prefill-tokens`` tokens, and decode steps at batch 8 and 1 on
contexts of ``--context`` tokens built by real prefill.

The second part times the design's own kernels beside the like kernel of the engine's other models, each
replayed from a CUDA graph over inputs rotated so that no repetition finds them in L2, as a fraction of
the measured peak: attention over latent rows (a decode batch, absorbed) beside the kernel for rows of
128 values and beside the generic kernel; prompt attention over made keys and values (expanded) beside
the paged tcgen05 kernel; the output norm that adds a routed feed-forward's rows, handed-back inputs and
shared row beside the plain one and beside ``rmsnorm``; the map of the stream; the latent store and the
gather.  One JSON line.
"""

from __future__ import annotations

import json
import time
from typing import Any, Callable, Dict, List

from .design_bench import _timed, measure_model

SIZES: Dict[str, Dict[str, int]] = {
    "w2048": dict(width=2048, heads=16, dim=128, rot=64, vdim=128, kv_rank=512, ff=1408, shared=2816, experts=12,
                  identity=4, top=3, vocab=32768),
    "w4096": dict(width=4096, heads=32, dim=128, rot=64, vdim=128, kv_rank=512, ff=2816, shared=5632, experts=12,
                  identity=4, top=3, vocab=32768),
}


def dizatar_config(s: Dict[str, int]) -> Dict[str, Any]:
    mixer = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["vdim"], "kv_rank": s["kv_rank"],
             "scale": (s["dim"] + s["rot"]) ** -0.5, "rot": {"base": 5e4, "dims": s["rot"]}}
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "shared": {"ff": s["shared"]},
           "router": {"experts": s["experts"], "top": s["top"], "identity": s["identity"]}}
    return {"architecture": "Dizatar", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "residual_mult": 0.5, "logit_softcap": 25.0, "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "latent_attention", "mixer": mixer, "mlp": mlp} for _ in range(4)]}


def nirelix_latent_config(s: Dict[str, int]) -> Dict[str, Any]:
    """Six layers, one stream; experts sized so that a token uses as many feed-forward weights as there."""
    mixer = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["vdim"], "q_rank": s["width"] // 2,
             "kv_rank": s["kv_rank"], "scale": (s["dim"] + s["rot"]) ** -0.5, "mask": {"size": 1 << 20},
             "rot": {"base": 5e4, "dims": s["rot"]}}
    used = s["top"] * s["experts"] / (s["experts"] + s["identity"]) * s["ff"] + s["shared"]
    ff = int(used / s["top"]) // 64 * 64
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": s["experts"], "top": s["top"], "scale": 1.0}}
    return {"architecture": "Nirelix", "vocab": s["vocab"], "width": s["width"], "streams": 1, "norm": {"eps": 1e-6},
            "layers": [{"type": "latent_attention", "mixer": mixer, "mlp": mlp} for _ in range(6)]}


def kernel_pairs(s: Dict[str, int], peaks: Dict[str, Any], reps: int = 10) -> Dict[str, Any]:
    import torch

    from .csrc import ops
    from .parts import linear
    from .parts.base import Workspace
    from .parts.position import rotary_table

    dev, bf = "cuda:0", torch.bfloat16
    hbm, tflops = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    W, H, P, R, rot, dq, dv = s["width"], s["heads"], 64, s["kv_rank"], s["rot"], s["dim"], s["vdim"]
    d = R + rot
    out: Dict[str, Any] = {}
    ints = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)

    def rotate(make: Callable[[], Any], nbytes: int, most: int = 16) -> List[Any]:
        return [make() for _ in range(min(most, max(2, -(-(256 << 20) // max(1, nbytes)))))]

    def run(name: str, launch: Callable[[int], None], sets: int, nbytes: float = 0.0, flops: float = 0.0) -> None:
        for i in range(min(sets, 3)):
            launch(i)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for i in range(sets):
                launch(i)
        graph.replay()
        ms = _timed(graph.replay, reps) / sets
        row: Dict[str, Any] = {"us": round(ms * 1e3, 2)}
        if nbytes:
            row["gbs"] = round(nbytes / (ms / 1e3) / 1e9, 1)
            row["frac_of_measured_copy_peak"] = round(nbytes / (ms / 1e3) / hbm, 3)
        if flops:
            row["tflops"] = round(flops / (ms / 1e3) / 1e12, 1)
            row["frac_of_measured_bf16_peak"] = round(flops / (ms / 1e3) / tflops, 3)
        out[name] = row

    # ---- decode attention over latent rows -------------------------------------------------------
    ws = Workspace(dev)
    for B, ctx in ((64, 2048), (8, 2048), (1, 2048), (4, 32768)):
        per_req = ctx // P
        n_pages = B * per_req
        pos, seg = ints([ctx - 1] * B), torch.arange(B, dtype=torch.int32, device=dev)
        table = torch.arange(1, n_pages + 1, dtype=torch.int32, device=dev).view(B, per_req)
        q_start = torch.arange(B + 1, dtype=torch.int32, device=dev)
        rt = ops.latent_row_tile(H, d, R)
        flat = [(i, r) for i in range(B) for r in range(0, H, rt)]
        fs, fr = ints([a for a, _ in flat]), ints([b for _, b in flat])
        planes = rotate(lambda: torch.randn(n_pages + 1, 1, P, d, device=dev, dtype=bf), n_pages * P * d * 2, most=4)
        q = torch.randn(B, H, d, device=dev, dtype=bf)
        o = torch.empty(B, H, R, device=dev, dtype=bf)
        run(f"attn_latent (absorbed, rows of {R} + {rot}), {B} x {ctx} keys",
            lambda i: ops.attn_latent(q, o, planes[i], fs, fr, q_start, pos, table, H, R, d ** -0.5, None, ctx, ws),
            len(planes), nbytes=B * ctx * d * 2)
        if B == 64:
            both = [p.unsqueeze(0).expand(2, *p.shape) for p in planes]
            og = torch.empty(B, H * d, device=dev, dtype=bf)
            run(f"generic kernel over the same rows, {B} x {ctx} keys",
                lambda i: ops.attn_paged_simt(q.view(B, H * d), og, both[i], pos, seg, table, H, 1, d, d ** -0.5, None),
                len(planes), nbytes=B * ctx * d * 2)
            small = rotate(lambda: torch.randn(n_pages + 1, 1, P, 128, device=dev, dtype=bf), n_pages * P * 256, most=8)
            both = [p.unsqueeze(0).expand(2, *p.shape) for p in small]
            qs, os_ = torch.randn(B, H * 128, device=dev, dtype=bf), torch.empty(B, H * 128, device=dev, dtype=bf)
            run(f"attn_decode over latent rows of 128, {B} x {ctx} keys",
                lambda i: ops.attn_decode(qs, os_, both[i], None, B, pos, seg, table, H, 1, 128, 128 ** -0.5, None, ctx, ws),
                len(small), nbytes=B * ctx * 128 * 2)
            del small, both
        del planes

    # ---- prompt attention: one portion -----------------------------------------------------------
    for T in (2048, 8192):
        tiles = list(range(0, T, 128))
        ts, tq, tr = ints([0] * len(tiles)), ints(tiles), ints([0] * len(tiles))
        qst, p0, kl = ints([0, T]), ints([0]), ints([T])
        width = H * (dq + rot) + d
        q = torch.randn(T, width, device=dev, dtype=bf)[:, :H * (dq + rot)]
        rows = torch.randn(T, d, device=dev, dtype=bf)
        made = torch.randn(T, H * (dq + dv), device=dev, dtype=bf)
        y = torch.empty(T, H * dv, device=dev, dtype=bf)
        pairs = T * (T + 1) / 2
        run(f"attn_prefill_mha (expanded, {dq} + {rot} -> {dv}), {T:,} tokens",
            lambda i: ops.attn_prefill_mha(q, made[:, :H * dq].unflatten(1, (H, dq)), rows[:, R:],
                                           made[:, H * dq:].unflatten(1, (H, dv)), y, ts, tq, tr, qst, p0, H, dq, rot,
                                           dv, (dq + rot) ** -0.5), 1, flops=2.0 * H * pairs * (dq + rot + dv))
        table = torch.arange(1, T // P + 1, dtype=torch.int32, device=dev).view(1, -1)
        cache = torch.randn(2, T // P + 1, H, P, 128, device=dev, dtype=bf)
        t64 = ints(list(range(0, T, 64)))
        q2, o2 = torch.randn(T, H * 128, device=dev, dtype=bf), torch.empty(T, H * 128, device=dev, dtype=bf)
        run(f"attn_prefill_tc (paged, a key head per head of 128), {T:,} tokens",
            lambda i: ops.attn_prefill_tc(q2, o2, cache, torch.zeros_like(t64), t64, qst, p0, table, H, H, 128,
                                          128 ** -0.5), 1, flops=2.0 * H * pairs * 256)
        pages = torch.randn(T // P + 1, 1, P, d, device=dev, dtype=bf)
        g = list(range(0, T, 64))
        gs, gk = ints([0] * len(g)), ints(g)
        run(f"latent_gather, {T:,} rows", lambda i: ops.latent_gather(pages, rows, gs, gk, gk, kl, p0, table), 1,
            nbytes=2 * T * d * 2)
        ops.check_tc_status(dev)
        del cache, q, made, y, q2, o2, pages

    # ---- rows: output norms, the stream's map, the latent store ----------------------------------
    k, E = s["top"], s["experts"]
    for T in (8192, 64):
        label = "8,192 tokens" if T == 8192 else "decode batch of 64"
        parts = rotate(lambda: torch.randn(T, k, W, device=dev, dtype=bf), T * W * (2 * k + 14), most=6)
        plain = [p[:, 0].contiguous() for p in parts]
        ids = torch.randint(0, E + s["identity"], (T, k), device=dev, dtype=torch.int32)
        wts = torch.rand(T, k, device=dev)
        extra = torch.randn(T, W, device=dev, dtype=bf)
        h = torch.randn(T, W, device=dev, dtype=bf)
        res = torch.zeros(T, W, device=dev)
        w1 = torch.ones(W, device=dev)
        nout = torch.empty(T, W, device=dev, dtype=bf)
        written = float((ids < E).sum()) / T
        back = float((ids >= E).any(1).sum()) / T
        run(f"norm_add + next norm over routed, handed-back and shared rows, {label}",
            lambda i: ops.norm_add(ops.RoutedRows(parts[i], ids, wts, E, h, extra), res, w1, 1e-6, False, 0.5,
                                   next_weight=w1, next_eps=1e-6, next_out=nout), len(parts),
            nbytes=T * W * (2 * written + 2 * back + 2 + 8 + 2))
        run(f"norm_add + next norm of one branch row, {label}",
            lambda i: ops.norm_add(plain[i], res, w1, 1e-6, False, 0.5, next_weight=w1, next_eps=1e-6, next_out=nout),
            len(parts), nbytes=T * W * (2 + 8 + 2))
        run(f"rmsnorm (residual add + norm of one row), {label}",
            lambda i: ops.rmsnorm(plain[i], res, w1, nout, 1e-6, False), len(parts), nbytes=T * W * (2 + 8 + 2))
        pair = torch.empty(T, 2 * W, device=dev, dtype=bf)
        run(f"cast_rows (the stream's copy for its map), {label}", lambda i: ops.cast_rows(res, pair[:, :W]), 1,
            nbytes=T * W * 6)
        mats = rotate(lambda: torch.randn(W, 2 * W, device=dev, dtype=bf), 2 * W * W * 2, most=8)
        run(f"embedding_mix product, {label}", lambda i: linear.linear(pair, mats[i], res), len(mats),
            nbytes=0.0 if T > 64 else (2 * W * W + T * 2 * W) * 2 + T * W * 4,
            flops=4.0 * T * W * W if T > 64 else 0.0)
        outb = torch.empty(T, W, device=dev, dtype=bf)
        run(f"linear product of the same size, bfloat16 result, {label}", lambda i: linear.linear(pair, mats[i], outb),
            len(mats), nbytes=0.0 if T > 64 else (2 * W * W + T * 2 * W) * 2 + T * W * 2,
            flops=4.0 * T * W * W if T > 64 else 0.0)
        del parts, plain, mats
        pos = torch.arange(T, dtype=torch.int32, device=dev)
        seg = torch.zeros(T, dtype=torch.int32, device=dev)
        table = torch.arange(1, -(-T // P) + 1, dtype=torch.int32, device=dev).view(1, -1)
        downs = rotate(lambda: torch.randn(T, H * (dq + rot) + d, device=dev, dtype=bf), T * (H * (dq + rot) + d) * 2, most=8)
        pages = torch.zeros(-(-T // P) + 1, 1, P, d, device=dev, dtype=bf)
        nw = torch.ones(R, device=dev)
        cs = rotary_table(rot, 5e4, dev, T, exact_angles=True)
        run(f"latent_store (norm, rotation, cache row, query tails in place), {label}",
            lambda i: ops.latent_store(downs[i][:, H * (dq + rot):], downs[i][:, :H * (dq + rot)], None, pages, nw, cs,
                                       pos, seg, table, heads=H, q_dim=dq, rank=R, rot=rot, interleaved=False, eps=1e-6,
                                       turn_q=True), len(downs), nbytes=T * (d * 4 + H * rot * 4))
        qkv = rotate(lambda: torch.randn(T, (H + 2 * 4) * 128, device=dev, dtype=bf), T * (H + 8) * 256, most=8)
        kv = torch.zeros(2, -(-T // P) + 1, 4, P, 128, device=dev, dtype=bf)
        qo = torch.empty(T, H * 128, device=dev, dtype=bf)
        qn = torch.ones(128, device=dev)
        cs2 = rotary_table(64, 5e4, dev, T, exact_angles=True)
        run(f"qk_rope_store (per-head norm, rotary, keys and values to pages), {label}",
            lambda i: ops.qk_rope_store(qkv[i], qo, kv, qn, qn, cs2, pos, seg, table, H, 4, 128, 64, 2, True, False,
                                        1e-6), len(qkv), nbytes=2 * T * (H + 8) * 256)
        del downs, qkv
    return out


def main(a) -> int:
    import torch

    from .benchmark import ClockSampler, load_peaks

    peaks = load_peaks()
    names = [n for n in a.sizes.split(",") if n.strip()]
    for n in names:
        if n not in SIZES:
            print(f"unknown size '{n}' (known: {', '.join(SIZES)})")
            return 2
    t0 = time.time()
    sizes: Dict[str, Any] = {}
    with ClockSampler() as clocks:
        for n in names:
            s = SIZES[n]
            sizes[n] = {"shape": s, "dizatar": measure_model(dizatar_config(s), a),
                        "nirelix_equal_size": measure_model(nirelix_latent_config(s), a)}
        kernels = kernel_pairs(SIZES[names[0]], peaks)
    torch.cuda.synchronize()
    line = {"bench": "design", "design": "Dizatar", "beside": "Nirelix decoder of latent-attention layers at equal size",
            "dtype": "bf16", "data": "synthetic: random weights, uniform random token ids",
            "layers": "4, the middle two twice: 6 layer runs (beside: 6 layers)",
            "context": a.context, "steps": a.steps, "warmup": max(3, a.warmup), "sizes": sizes,
            "kernels_at": names[0], "kernels": kernels,
            "peaks": {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "source": peaks["source"]},
            "clocks": clocks.summary(), "wall_s": round(time.time() - t0, 1)}
    print(json.dumps(line))
    return 0
