"""Besuzen beside the Tonapel decoder at equal size: step throughput and kernel rooflines.

    python bench.py --design besuzen [--sizes w2048,w4096] [--steps K] [--warmup W]

For every size a four-layer Besuzen model (attention + experts, parallel + dense, parallel + experts, attention +
dense; random weights) and the engine's closest other model - a Tonapel decoder of the same width, layer count,
head counts, head sizes, window longer than the context, feed-forwards and vocabulary, whose parallel layers also
run attention beside a recurrence - run the same workload through ``Engine.step`` (the method of
:mod:`.design_bench`): one prompt of ``--prefill-tokens`` tokens, and decode steps at batch 8 and 1 on contexts
of ``--context`` tokens built by real prefill.

The second part times the design's own kernels beside the like kernel of the engine's other models, each
replayed from a CUDA graph over inputs rotated so that no repetition finds them in L2, as a fraction of the
measured peak: the time mixer's scan beside the scan of the state space and of the delta rule with a decay per
key channel (which also carries one); the token shift beside the short convolution; two layer norms behind a
joined branch beside ``norm_add`` and ``rmsnorm``; rotation by pairs with blended values beside rotation by
halves; the four projections of the time mixer in one launch beside one product of the same bytes; selection
inside groups.  One JSON line.
"""

from __future__ import annotations

import json
import time
from typing import Any, Callable, Dict, List

from .design_bench import LAYERS, _timed, measure_model
from .tonapel_bench import tonapel_config

SIZES: Dict[str, Dict[str, int]] = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, vdim=128, tm_heads=32, tm_dim=64, low_rank=64, ff=8192,
                  experts=8, top=2, groups=4, keep=2, vocab=32768),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, tm_heads=64, tm_dim=64, low_rank=128, ff=14336,
                  experts=8, top=2, groups=4, keep=2, vocab=32768),
}


def besuzen_config(s: Dict[str, int]) -> Dict[str, Any]:
    d = s["dim"]
    heads = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": d, "vdim": s["vdim"], "scale": d ** -0.5}
    att = {**heads, "rot": {"base": 1e4, "dims": d // 2}, "v_mix": True}
    par = {"left": heads, "right": {"heads": s["tm_heads"], "dim": s["tm_dim"], "low_rank": s["low_rank"]},
           "left_scale": 0.7, "right_scale": 0.7}
    inter = max(128, (s["ff"] // 3) // 128 * 128)           # a token uses about as much as the dense one holds
    dense = {"kind": "dense", "ff": s["ff"] * 2 // 3 // 128 * 128}
    moe = {"kind": "moe", "expert": {"ff": inter}, "shared": {"ff": inter},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["keep"]}}}
    return {"architecture": "Besuzen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "embedding": {"scale": 0.7}, "logit_scale": 0.7,
            "layers": [{"type": "attention", "mixer": att, "mlp": moe}, {"type": "parallel", "mixer": par, "mlp": dense},
                       {"type": "parallel", "mixer": par, "mlp": moe}, {"type": "attention", "mixer": att, "mlp": dense}]}


def like_config(s: Dict[str, int], room: int) -> Dict[str, Any]:
    """The Tonapel decoder of equal size: its recurrences have as many values of state a head as the time mixer
    has channels times heads."""
    return tonapel_config({**s, "window": room, "ssd_heads": s["tm_heads"], "ssd_dim": s["tm_dim"], "state": 128,
                           "delta_heads": s["heads"]})


def kernel_pairs(s: Dict[str, int], peaks: Dict[str, Any], reps: int = 10) -> Dict[str, Any]:
    import torch

    from .csrc import ops
    from .parts.position import rotary_table

    dev, bf = "cuda:0", torch.bfloat16
    hbm = peaks["hbm_gbs"] * 1e9
    W, P = s["width"], 64
    out: Dict[str, Any] = {}
    ints = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)

    def rotate(make: Callable[[], Any], nbytes: int, most: int = 16) -> List[Any]:
        return [make() for _ in range(min(most, max(2, -(-(256 << 20) // max(1, nbytes)))))]

    def run(name: str, launch: Callable[[int], None], sets: int, nbytes: float) -> None:
        for i in range(min(sets, 3)):
            launch(i)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for i in range(sets):
                launch(i)
        graph.replay()
        ms = _timed(graph.replay, reps) / sets
        out[name] = {"us": round(ms * 1e3, 2), "gbs": round(nbytes / (ms / 1e3) / 1e9, 1),
                     "frac_of_measured_copy_peak": round(nbytes / (ms / 1e3) / hbm, 3)}

    def meta(lens):
        q = [0]
        for n in lens:
            q.append(q[-1] + n)
        seg = torch.cat([torch.full((n,), i, dtype=torch.int32) for i, n in enumerate(lens)]).to(dev)
        return seg, torch.arange(len(lens), dtype=torch.int32, device=dev), ints(q)

    H, D = s["tm_heads"], s["tm_dim"]
    inner = H * D
    for label, lens in (("one prompt portion of 8,192 tokens", [8192]), ("decode batch of 64", [1] * 64)):
        T, S = sum(lens), len(lens)
        seg, slot, q = meta(lens)
        y = torch.empty(T, inner, device=dev)
        # ---- scans with as many heads, each of 64 values; all read their states and write them back ----
        state_b = inner * D * 4
        rkv = rotate(lambda: torch.randn(3, T, inner, device=dev, dtype=bf), T * inner * 6 + S * state_b)
        states = [torch.zeros(S, inner * D, device=dev) for _ in rkv]
        decay, w0, u = torch.randn(T, inner, device=dev), torch.zeros(inner, device=dev), torch.ones(inner, device=dev)
        run(f"time_mixing_scan ({H} heads of {D} x {D}), {label}",
            lambda i: ops.time_mixing_scan(rkv[i][0], rkv[i][1], rkv[i][2], decay, w0, u, states[i], y, slot, q, H, D, D),
            len(rkv), nbytes=T * inner * (6 + 4 + 4) + 2 * S * state_b)
        qkv = [r.view(T, 3 * inner) for r in rkv]
        beta, a_log = torch.randn(T, H, device=dev, dtype=bf), torch.zeros(H, device=dev)
        run(f"channel_delta_scan ({H} heads of {D} x {D}), {label}",
            lambda i: ops.channel_delta_scan(qkv[i], beta, decay, w0, a_log, states[i], y, slot, q, H, H, D, D, 1e-6,
                                             D ** -0.5), len(qkv), nbytes=T * inner * (6 + 4 + 4) + 2 * S * state_b)
        del rkv, qkv, states
        ys = rotate(lambda: torch.randn(T, inner, device=dev), T * inner * 8, most=8)
        gate, gout = torch.randn(T, inner, device=dev, dtype=bf), torch.empty(T, inner, device=dev, dtype=bf)
        for name, groups in ((f"a norm per head of {D}", H), ("one norm a row", 1)):
            run(f"gated_norm ({name}), {label}",
                lambda i, g=groups: ops.gated_norm(ys[i], gate, u, gout, g, 1e-6, False), len(ys),
                nbytes=T * inner * (4 + 2 + 2))
        del ys
        N = 128
        C = inner + 2 * N
        xs = rotate(lambda: torch.randn(T, C, device=dev, dtype=bf) * 0.5, T * C * 2 + S * inner * N * 4)
        states = [torch.zeros(S, inner * N, device=dev) for _ in xs]
        dt, small = torch.randn(T, H, device=dev, dtype=bf), torch.zeros(H, device=dev)
        run(f"ssd_scan ({H} heads of {N} x {D}), {label}",
            lambda i: ops.ssd_scan(xs[i], dt, small, small, small, states[i], y, slot, q, H, D, N, 1), len(xs),
            nbytes=T * C * 2 + T * inner * 4 + 2 * S * inner * N * 4)
        del xs, states
        # ---- the token shift beside the short convolution -------------------------------------------
        xs = rotate(lambda: torch.randn(T, W, device=dev, dtype=bf), T * W * 12, most=8)
        mixed = [torch.empty(5, T, W, device=dev, dtype=bf) for _ in xs]
        mu = torch.rand(5, W, device=dev)
        last = [torch.zeros(S, W, device=dev) for _ in xs]
        run(f"token_shift (5 mixes), {label}", lambda i: ops.token_shift(xs[i], mu, mixed[i], last[i], seg, slot, q),
            len(xs), nbytes=6 * T * W * 2 + 2 * S * W * 4)
        cw, cb = torch.randn(W, 4, device=dev), torch.zeros(W, device=dev)
        cs_ = [torch.zeros(S, 3 * W, device=dev) for _ in xs]
        run(f"conv_silu (4 taps), {label}",
            lambda i: ops.conv_silu(xs[i], mixed[i][0], cw, cb, cs_[i], seg, slot, q), len(xs),
            nbytes=2 * T * W * 2 + 2 * S * 3 * W * 4)
        del mixed
        # ---- norms ------------------------------------------------------------------------------------
        k = s["top"]
        parts = rotate(lambda: torch.randn(T, k, W, device=dev, dtype=bf), T * W * (2 * k + 14), most=6)
        beside = [torch.randn(T, 2, W, device=dev, dtype=bf) for _ in parts]
        extra, gate = torch.randn(T, W, device=dev, dtype=bf), torch.rand(T, device=dev)
        sc, w1 = torch.ones(2, device=dev), torch.ones(W, device=dev)
        res = torch.zeros(T, W, device=dev)
        n1, n2 = torch.empty(T, W, device=dev, dtype=bf), torch.empty(T, W, device=dev, dtype=bf)
        run(f"join_layer_norm (two norms behind {k} routed rows, a gated shared row, two scaled mixers' rows), {label}",
            lambda i: ops.join_layer_norm(ops.RoutedRows(parts[i], extra=extra, extra_gate=gate, beside=beside[i],
                                                         beside_scale=sc), res, w1, 1e-6, n1, None, w1, 1e-6, n2),
            len(parts), nbytes=T * W * (2 * k + 2 + 4 + 8 + 4))
        run(f"join_layer_norm (two norms behind two rows), {label}",
            lambda i: ops.join_layer_norm(ops.RoutedRows(extra, beside=xs[i % len(xs)]), res, w1, 1e-6, n1, None, w1, 1e-6,
                                          n2), len(xs), nbytes=T * W * (4 + 8 + 4))
        plain = [p[:, 0].contiguous() for p in parts]
        run(f"norm_add + next norm of one branch row, {label}",
            lambda i: ops.norm_add(plain[i], res, w1, 1e-6, False, 0.5, next_weight=w1, next_eps=1e-6, next_out=n1),
            len(plain), nbytes=T * W * (2 + 8 + 2))
        run(f"rmsnorm (residual add + norm), {label}",
            lambda i: ops.rmsnorm(plain[i], res, w1, n1, 1e-6, False), len(plain), nbytes=T * W * (2 + 8 + 2))
        del parts, beside, plain, xs
        # ---- projection rows -> queries + cache -------------------------------------------------------
        hq, G, d = s["heads"], s["kv_heads"], s["dim"]
        width = (hq + 2 * G) * d
        npages = max(1, T // P) if S == 1 else S
        pos = torch.arange(T, dtype=torch.int32, device=dev) if S == 1 else torch.zeros(T, dtype=torch.int32, device=dev)
        table = torch.arange(1, npages + 1, dtype=torch.int32, device=dev).view(S, -1)
        srcs = rotate(lambda: torch.randn(T, width, device=dev, dtype=bf), 2 * T * width * 2, most=8)
        first, lam = torch.randn(T, G * d, device=dev, dtype=bf), torch.tensor(0.4, device=dev)
        q_out = torch.empty(T, hq * d, device=dev, dtype=bf)
        pages = torch.zeros(2, npages + 1, G, P, d, device=dev, dtype=bf)
        cs = rotary_table(d // 2, 1e4, dev, 8192, exact_angles=True)
        for name, pairs, blend in (("by pairs, values blended", True, True), ("by halves", False, False)):
            run(f"qk_rope_store ({name}), {label}",
                lambda i, p=pairs, b=blend: ops.qk_rope_store(
                    srcs[i], q_out, pages, None, None, cs, pos, seg, table, hq, G, d, d // 2, 0, False, p, 1e-6,
                    value_first=first if b else None, value_lambda=lam if b else None), len(srcs),
                nbytes=2 * T * width * 2 + (T * G * d * 2 if blend else 0))
        del srcs, pages
        # ---- selection ---------------------------------------------------------------------------------
        E = 64
        logits = [torch.randn(T, E + 1, device=dev) for _ in range(4)]
        plain = [x[:, :E].contiguous() for x in logits]
        ids, wts, tail = torch.empty(T, 4, dtype=torch.int32, device=dev), torch.empty(T, 4, device=dev), torch.empty(T, device=dev)
        run(f"router_select (64 experts, 8 groups by their largest, a gate), {label}",
            lambda i: ops.router_select(logits[i], None, ids, wts, 4, True, True, 1.0, 1, 8, 4, 1, tail), 4,
            nbytes=T * (E * 4 + 4 * 8))
        run(f"router_select (64 experts, 8 groups by their two largest), {label}",
            lambda i: ops.router_select(plain[i], None, ids, wts, 4, True, True, 1.0, 1, 8, 4), 4, nbytes=T * (E * 4 + 4 * 8))
        run(f"router_select (64 experts, no groups), {label}",
            lambda i: ops.router_select(plain[i], None, ids, wts, 4, True, True, 1.0), 4, nbytes=T * (E * 4 + 4 * 8))

    # ---- decode products: four projections in one launch, beside one product of the same bytes; gated pair -----
    for B in (8, 1):
        per = ops.pass_rows(B)
        sets = rotate(lambda: torch.randn(4, inner, W, device=dev, dtype=bf), 4 * inner * W * 2, most=6)
        x4, y4 = torch.randn(4 * B, W, device=dev, dtype=bf), torch.empty(4 * B, inner, device=dev, dtype=bf)
        run(f"skinny_gemm, four matrices against rows of their own, batch {B}",
            lambda i: ops.skinny_gemm(x4, sets[i], y4, group_rows=B, rows_per_pass=per), len(sets), nbytes=4 * inner * W * 2)
        y1 = torch.empty(B, 4 * inner, device=dev, dtype=bf)
        run(f"skinny_gemm, one matrix of the same bytes, batch {B}",
            lambda i: ops.skinny_gemm(x4[:B], sets[i].view(4 * inner, W), y1, rows_per_pass=per), len(sets),
            nbytes=4 * inner * W * 2)
        I = 2 * inner
        mid = torch.empty(B, I, device=dev, dtype=bf)
        run(f"skinny_gemm, gated pair in the epilogue, batch {B}",
            lambda i: ops.skinny_gemm(x4[:B], sets[i].view(2 * I, W), mid, glu=True, act="gelu_tanh", rows_per_pass=per),
            len(sets), nbytes=4 * inner * W * 2)
        del sets
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
            room = a.context + a.steps + a.warmup + 512
            sizes[n] = {"shape": s, "besuzen": measure_model(besuzen_config(s), a),
                        "tonapel_equal_size": measure_model(like_config(s, room), a)}
        kernels = kernel_pairs(SIZES[names[0]], peaks)
    torch.cuda.synchronize()
    line = {"bench": "design", "design": "Besuzen", "beside": "Tonapel decoder at equal size",
            "dtype": "bf16", "data": "synthetic: random weights, uniform random token ids", "layers": LAYERS,
            "context": a.context, "steps": a.steps, "warmup": max(3, a.warmup), "sizes": sizes,
            "kernels_at": names[0], "kernels": kernels,
            "peaks": {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "source": peaks["source"]},
            "clocks": clocks.summary(), "wall_s": round(time.time() - t0, 1)}
    print(json.dumps(line))
    return 0
