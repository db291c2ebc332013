"""Besuzen in the engine against the plain implementation: every new kernel alone, every mechanism alone in a
model of one or two layers, whole prompts against decoding, portions down to two tokens, mixed batches with
pages and state slots used again, a far key and a far token behind the state made decisive on purpose, the
first tokens, long decoding, three configurations that differ in every size, greedy generation through the
scheduler, the trace replay tool."""

import pytest
import torch

import besuzen_tiny as bz
import plain_besuzen as plain
import replay_driver as rd

pytestmark = pytest.mark.gpu

LENGTHS = {"A": [1, 2, 9, 37, 70], "B": [3, 150, 66, 200, 21], "C": [2, 35, 77, 5]}
CUTS = {"whole": rd.whole, "decode_tail": rd.decode_tail, "portions": rd.portions, "mixed": rd.mixed}
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def requests_of(which):
    vocab = bz.BZ[which]["vocab"]
    return {f"r{i}": bz.tokens(40 * i + ord(which), n, vocab) for i, n in enumerate(LENGTHS[which])}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {which: bz.write_tiny(str(tmp_path_factory.mktemp(f"bz{which}")), which) for which in bz.BZ}


_PLAIN = {}


def expected_for(config, state, reqs, dtype, routing=None):
    """``(logits, noise)`` of the plain model by request; in bfloat16 with the experts the engine chose (two correct
    implementations may choose differently where two router scores lie within rounding) and with what rounding
    alone does at every position, in float32 without (None)."""
    want, noise = {}, {}
    routed = bz.routed_layers(config)
    for rid, toks in reqs.items():
        ids = dict(zip(routed, routing[rid])) if dtype == "bfloat16" and routing else None
        key = (id(config), id(state), dtype, tuple(toks), None if ids is None else
               tuple(tuple(int(e) for row in ids[i] for e in sorted(row)) for i in routed))
        if key not in _PLAIN:
            logits = plain.forward(config, state, toks, expert_ids=ids)
            moved = bz.rounding_noise(config, state, toks, logits, ids) if dtype == "bfloat16" else None
            # config and state stay referenced by the value: their ids stay theirs
            _PLAIN[key] = (logits, moved, config, state)
        want[rid], noise[rid] = _PLAIN[key][:2]
    return want, noise if dtype == "bfloat16" else None


_STATES = {}


def state_of(which):
    if which not in _STATES:
        _STATES[which] = bz.random_state(bz.BZ[which], bz.SEEDS[which])
    return _STATES[which]


def run_engine(engine, reqs, schedule, routing=None):
    """Drive ``engine.step`` through a schedule; logits of every position of every request.  With ``routing`` (a
    dict) the experts the engine chose are left there: ``routing[request][j]`` is ``[positions, top]`` of the j-th
    routed layer."""
    from freetoken_b200.engine import StepEntry
    out = {rid: torch.full((len(t), engine.vocab_size), float("nan")) for rid, t in reqs.items()}
    for entries, ended in schedule:
        batch = [StepEntry(rid, reqs[rid][first:first + n], list(range(n))) for rid, first, n in entries]
        probe = {"router_ids": []} if routing is not None else None
        logits = engine.step(batch, probe=probe).float().cpu()
        row = 0
        for rid, first, n in entries:
            out[rid][first:first + n] = logits[row:row + n]
            if routing is not None:
                if rid not in routing:
                    routing[rid] = [torch.full((len(reqs[rid]), x.shape[1]), -1, dtype=torch.long)
                                    for x in probe["router_ids"]]
                for j, x in enumerate(probe["router_ids"]):
                    routing[rid][j][first:first + n] = x[row:row + n].cpu().long()
            row += n
        for rid in ended:
            engine.end_request(rid)
    engine.cache.check_integrity()
    return out


def run_and_compare(folder, config, state, reqs, schedule, dtype, page, what, tol=None):
    engine = bz.make_engine(folder, dtype, page, rd.peak_tokens(schedule, page), poison=True)
    routing = {} if bz.routed_layers(config) else None
    got = run_engine(engine, reqs, schedule, routing)
    want, noise = expected_for(config, state, reqs, dtype, routing)
    bz.compare(got, want, tol or bz.TOL[dtype], f"{what} [{dtype}]", noise)
    assert engine.cache.free_pages() == engine.cache.total_pages()
    return got


def close(got, want, dtype, what=""):
    tol = 2e-5 if dtype == "float32" else 2e-2
    g, w = got.double().cpu(), want.double()
    assert torch.allclose(g, w, atol=tol * max(1.0, float(w.abs().max())), rtol=tol), (what, float((g - w).abs().max()))


# ------------------------------------------------------------------ kernels, each alone
def segments(lens, slots):
    q = [0]
    for n in lens:
        q.append(q[-1] + n)
    seg = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).int().cuda()
    return seg, torch.tensor(slots, dtype=torch.int32).cuda(), torch.tensor(q, dtype=torch.int32).cuda()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H", [44, 70, 512, 1100, 3000, 8192, 9000])
def test_join_layer_norm(dtype, H):
    """Routed rows, a gated shared row and another sublayer's scaled rows join the residual; two norms of the
    new row (one with a bias), rows of every width class; without a branch the residual stays."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(H)
    T, k, m = 3, 3, 2
    dt = DTYPES[dtype]
    x = torch.randn(T, H) + 2.0                                     # a mean to take off
    rows, extra, beside = torch.randn(T, k, H).to(dt), torch.randn(T, H).to(dt), torch.randn(T, m, H).to(dt)
    gate, scale = torch.rand(T), torch.tensor([0.3, -1.2])
    w1, w2, b2 = torch.randn(H), torch.randn(H), torch.randn(H)
    d = lambda t: t.double()
    cu = lambda t: t.cuda().contiguous()
    residual, out, out2 = cu(x.clone()), torch.empty(T, H, dtype=dt, device="cuda"), torch.empty(T, H, dtype=dt, device="cuda")
    branch = ops.RoutedRows(cu(rows), extra=cu(extra), extra_gate=cu(gate), beside=cu(beside), beside_scale=cu(scale))
    ops.join_layer_norm(branch, residual, cu(w1), 1e-5, out, None, cu(w2), 1e-2, out2, cu(b2))
    other = (d(scale)[None, :, None] * d(beside)).sum(1)
    new = d(x) + d(rows).sum(1) + d(gate)[:, None] * d(extra) + other
    close(residual, new, "float32", "residual")
    close(out, plain.layer_norm(new, d(w1), 1e-5), dtype, "first norm")
    close(out2, plain.layer_norm(new, d(w2), 1e-2) + d(b2), dtype, "second norm")
    before = residual.clone()
    ops.join_layer_norm(None, residual, cu(w1), 1e-5, out)
    assert torch.equal(before, residual)
    close(out, plain.layer_norm(d(before.cpu()), d(w1), 1e-5), dtype, "no branch")
    ops.join_layer_norm(ops.RoutedRows(cu(beside), scale=cu(scale)), residual, cu(w1), 1e-5, out)
    close(residual, d(before.cpu()) + other, "float32", "scaled rows alone")
    # one plain row beside a plain row, and the same sum as a row of its own
    ops.join_layer_norm(ops.RoutedRows(cu(extra), beside=cu(rows[:, 0])), residual, cu(w1), 1e-5, out)
    close(residual, d(before.cpu()) + other + d(extra) + d(rows[:, 0]), "float32", "two plain rows")
    total = torch.empty(T, H, dtype=dt, device="cuda")
    ops.branch_sum(branch, total)
    close(total, new - d(x), dtype, "branch_sum")


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("W,M", [(40, 5), (7, 3), (1040, 5), (516, 1)])
def test_token_shift_in_segments(dtype, W, M):
    """Two requests cut into segments of one and more tokens: every mix sees the token before, across
    segments through the slot; slots of others stay; many tokens take the kernel that walks four."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(W)
    dt = DTYPES[dtype]
    n = 2300
    x = {r: torch.randn(n, W).to(dt) for r in "ab"}
    mu = torch.rand(M, W)
    state = torch.zeros(4, W + 4, device="cuda")
    state[:, W:] = 5.0
    at, got = {"a": 0, "b": 0}, {"a": [], "b": []}
    for step, cut in enumerate([(1, 2), (1, 1), (5, 4), (1100, 1030), (3, 1), (1190, 1262)]):
        order = ("a", "b") if step % 2 == 0 else ("b", "a")
        lens = [cut[0] if r == "a" else cut[1] for r in order]
        rows = torch.cat([x[r][at[r]:at[r] + m] for r, m in zip(order, lens)]).cuda()
        seg, slot, q = segments(lens, [2 if r == "a" else 0 for r in order])
        out = torch.empty(M, rows.shape[0], W, dtype=dt, device="cuda")
        ops.token_shift(rows, mu.cuda(), out, state[:, :W], seg, slot, q)
        first = 0
        for r, m in zip(order, lens):
            got[r].append(out[:, first:first + m].cpu())
            first += m
            at[r] += m
    for r in "ab":
        assert at[r] == n
        have = torch.cat(got[r], 1)
        for m in range(M):
            close(have[m], plain.shifted_mix(x[r].double(), mu[m].double()), dtype, f"mix {m}")
    assert float(state[1, :W].abs().max()) == 0 and bool((state[:, W:] == 5.0).all())
    assert torch.equal(state[2, :W].cpu(), x["a"][-1].float())


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H,D,P", [(2, 12, 12), (3, 9, 20), (1, 64, 64), (2, 100, 17), (1, 200, 33), (2, 32, 16), (1, 256, 5)])
def test_time_mixing_scan_in_segments(dtype, H, D, P):
    """Segments below, at and above a chunk, of two requests side by side; sizes that fill lanes and sizes
    that do not; decays from nothing kept to everything kept."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(D + P)
    dt = DTYPES[dtype]
    n = 50
    kd = H * D
    w0, u = torch.randn(kd) * 2 - 1, torch.randn(kd)
    data = {}
    for r in "ab":
        rk = [torch.randn(n, kd).to(dt) for _ in range(2)]
        data[r] = (*rk, torch.randn(n, H * P).to(dt), torch.randn(n, kd) * 2)
    want = {}
    for name, (r_, k_, v_, a_) in data.items():
        v3 = lambda t, s: t.double().view(n, H, s)
        w = torch.exp(-torch.exp(a_.double() + w0.double())).view(n, H, D)
        S = torch.zeros(H, D, P, dtype=torch.float64)
        out = torch.zeros(n, H, P, dtype=torch.float64)
        for t in range(n):
            kv = torch.einsum("hd,hp->hdp", v3(k_, D)[t], v3(v_, P)[t])
            out[t] = torch.einsum("hdp,hd->hp", S + u.double().view(H, D, 1) * kv, v3(r_, D)[t])
            S = w[t][:, :, None] * S + kv
        want[name] = out.reshape(n, H * P)
    width = max(kd, H * P)
    state = torch.zeros(4, H * D * P + 3, device="cuda")
    state[:, H * D * P:] = 7.0
    at, got = {"a": 0, "b": 0}, {"a": [], "b": []}
    for step, cut in enumerate([(1, 7), (8, 1), (9, 16), (1, 1), (15, 8), (16, 17)]):
        order = ("a", "b") if step % 2 == 0 else ("b", "a")
        lens = [cut[0] if r == "a" else cut[1] for r in order]
        T = sum(lens)
        parts = [torch.cat([data[r][j][at[r]:at[r] + m] for r, m in zip(order, lens)]) for j in range(4)]
        rkv = torch.zeros(3, T, width, dtype=dt, device="cuda")               # one row stride, wider than a row
        for j in range(3):
            rkv[j, :, :parts[j].shape[1]] = parts[j].cuda()
        seg, slot, q = segments(lens, [2 if r == "a" else 0 for r in order])
        o = torch.empty(T, H * P, device="cuda")
        ops.time_mixing_scan(rkv[0, :, :kd], rkv[1, :, :kd], rkv[2, :, :H * P], parts[3].cuda(), w0.cuda(), u.cuda(),
                             state[:, :H * D * P], o, slot, q, H, P, D)
        o = o.cpu()
        for r, m in zip(order, lens):
            got[r].append(o[:m])
            o = o[m:]
            at[r] += m
    for r in "ab":
        assert at[r] == n
        g, scale = torch.cat(got[r]).double(), float(want[r].abs().max())
        assert float((g - want[r]).abs().max()) < 3e-5 * scale, r
    assert float(state[1, :H * D * P].abs().max()) == 0 and bool((state[:, H * D * P:] == 7.0).all())


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H,G,d,rot,d_first", [(4, 2, 64, 32, 64), (3, 1, 20, 6, 14), (2, 2, 48, 48, 64), (4, 4, 32, 8, 48), (2, 1, 128, 0, 128)])
def test_pairs_and_blended_values_on_the_way_to_the_pages(dtype, H, G, d, rot, d_first):
    """Interleaved rotation of a part of every head and values blended with another layer's rows, whose heads
    are filled up to another size; few tokens and many (other kernels); without a blend values pass unchanged."""
    from freetoken_b200.csrc import ops
    from freetoken_b200.parts.position import rotary_table
    torch.manual_seed(d + rot)
    dt = DTYPES[dtype]
    page, lam = 8, 0.3
    for T in (3, 600):
        pos = torch.arange(5, 5 + T).int()
        seg = torch.zeros(T).int()
        npages = (T + 5) // page + 1
        table = torch.randperm(npages).add(1).int().view(1, -1)
        qkv = torch.randn(T, (H + 2 * G) * d + 8).to(dt)
        first = torch.randn(T, G * d_first + 16).to(dt)
        qw = (H + 2 * G) * d
        cs = rotary_table(rot, 900.0, "cuda", 1024, exact_angles=True) if rot else None
        pages = torch.zeros(2, npages + 1, G, page, d, dtype=dt, device="cuda")
        q = torch.empty(T, H * d, dtype=dt, device="cuda")
        for blend in (True, False):
            ops.qk_rope_store(qkv.cuda()[:, :qw], q, pages, None, None, cs, pos.cuda(), seg.cuda(), table.cuda(), H, G, d,
                              rot, 0, False, True, 1e-6,
                              value_first=first.cuda()[:, 8:8 + G * d_first] if blend else None,
                              value_lambda=torch.tensor(lam).cuda() if blend else None)
            full = torch.zeros(T + 5, qw, dtype=torch.float64)
            full[5:] = qkv[:, :qw].double()
            turned = plain.rotate_pairs(full[:, :(H + G) * d].reshape(T + 5, H + G, d), 900.0, rot)[5:] if rot \
                else full[5:, :(H + G) * d].reshape(T, H + G, d)
            v = full[5:, (H + G) * d:].reshape(T, G, d)
            if blend:
                f = torch.zeros(T, G, d, dtype=torch.float64)
                both = min(d, d_first)
                f[..., :both] = first[:, 8:8 + G * d_first].double().view(T, G, d_first)[..., :both]
                v = (1 - lam) * v + lam * f
            close(q, turned[:, :H].reshape(T, -1), dtype, "q")
            held = pages.cpu()[:, table[0, pos.long() // page].long(), :, pos.long() % page]      # [T, 2, G, d]
            held = held if held.shape[0] == T else held.transpose(0, 1)
            close(held[:, 0], turned[:, H:], dtype, "k")
            close(held[:, 1], v, dtype, "v")


@pytest.mark.parametrize("E,top,count,keep", [(8, 3, 4, 3), (6, 2, 3, 1), (12, 4, 1, 1), (9, 2, 9, 4), (64, 6, 8, 2), (5, 5, 5, 5)])
@pytest.mark.parametrize("terms", [1, 3])
def test_router_groups_by_their_largest_score_and_a_gate_behind_the_logits(E, top, count, keep, terms):
    from freetoken_b200.csrc import ops
    torch.manual_seed(E)
    router = {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}
    for T in (5, 70):
        pieces = torch.randn(T, terms, E + 1)
        sums = pieces.double().sum(1)
        want = [plain.choose_experts(row[:E], router) for row in sums]
        ids = torch.empty(T, top, dtype=torch.int32, device="cuda")
        weights, gate = torch.empty(T, top, device="cuda"), torch.empty(T, device="cuda")
        logits = pieces.reshape(T, -1).cuda()
        ops.router_select(logits, None, ids, weights, top, True, True, 1.0, terms, count, keep, 1, gate)
        for t in range(T):
            chosen = sorted(zip(ids[t].tolist(), weights[t].tolist()))
            expect = sorted(zip(want[t][0], want[t][1].tolist()))
            assert [e for e, _ in chosen] == [e for e, _ in expect]
            assert all(abs(a - b) < 1e-5 for (_, a), (_, b) in zip(chosen, expect))
        assert torch.allclose(gate.cpu().double(), torch.sigmoid(sums[:, E]), atol=1e-6)
        if ops.route_small_takes(T, E, top):
            R = T * top
            bufs = [torch.empty(m, dtype=torch.int32, device="cuda") for m in (E, E + 1, R, R, E + 1)]
            ids2, w2 = torch.empty_like(ids), torch.empty_like(weights)
            gate2 = torch.empty_like(gate)
            ops.route_small(logits, None, ids2, w2, *bufs, top, True, True, 1.0, terms, count, keep, group_top=1, tail=gate2)
            assert torch.equal(ids2, ids) and torch.equal(w2, weights) and torch.equal(gate2, gate)


@pytest.mark.parametrize("T", [1, 5, 20, 32])
def test_few_rows_bias_tanh_groups_of_rows_and_the_gated_pair(T):
    """The weight-streaming kernel's options, each against a float64 product."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(T)
    K, N, G = 264, 50, 4
    bf = torch.bfloat16
    x, w, bias = torch.randn(G, T, K).to(bf), (torch.randn(G, N, K) * K ** -0.5).to(bf), torch.randn(N)
    per = ops.pass_rows(T)
    y = torch.einsum("gtk,gnk->gtn", x.double(), w.double())
    out = torch.empty(G, T, N, dtype=bf, device="cuda")
    ops.skinny_gemm(x.cuda().view(G * T, K), w.cuda(), out.view(G * T, N), group_rows=T, rows_per_pass=per)
    close(out, y, "bfloat16", "groups")
    one = torch.empty(T, N, device="cuda")
    ops.skinny_gemm(x[0].cuda(), w[0].cuda(), one, rows_per_pass=per, bias=bias.cuda())
    close(one, y[0] + bias.double(), "float32", "bias")
    ops.skinny_gemm(x[0].cuda(), w[0].cuda(), one, rows_per_pass=per, unary="tanh")
    close(one, torch.tanh(y[0]), "float32", "tanh")
    mid = torch.empty(T, N // 2, dtype=bf, device="cuda")
    for act, fn in (("gelu_tanh", plain.gelu_tanh), ("silu", plain.silu)):
        ops.skinny_gemm(x[0].cuda(), w[0].cuda(), mid, rows_per_pass=per, glu=True, act=act)
        close(mid, fn(y[0][:, :N // 2]) * y[0][:, N // 2:], "bfloat16", act)


# ------------------------------------------------------------------- mechanisms, each alone
ATT = bz.attention(2, 1, 8, 8, 4)
ALONE = {
    "attention": bz.several([bz.attention(3, 1, 12, 10, 8)]),
    "attention_all_dimensions_turn_one_head": bz.several([bz.attention(1, 1, 20, 28, 20, base=77.0)]),
    "attention_nothing_turns_no_mixing": bz.several([bz.attention(4, 4, 6, 9, 0, v_mix=False, scale=0.9)]),
    "values_blended_across_layers": bz.several([bz.attention(2, 2, 8, 6, 4), bz.attention(4, 2, 10, 6, 10),
                                                bz.attention(2, 2, 4, 6, 2)]),
    "blended_from_a_later_layer_on": bz.several([bz.attention(2, 1, 8, 8, 4, v_mix=False), bz.attention(2, 2, 16, 12, 8),
                                                 bz.parallel((1, 1, 4, 4), (1, 4, 2)), bz.attention(2, 2, 8, 12, 8)]),
    "parallel": bz.several([bz.parallel((4, 2, 12, 7), (3, 10, 6), 0.6, 1.4)]),
    "parallel_left_only": bz.several([bz.parallel((3, 3, 8, 20), (1, 8, 2), 1.0, 0.0)]),
    "parallel_right_only": bz.several([bz.parallel((1, 1, 4, 4), (4, 24, 9), 0.0, 1.0)]),
    "time_mixing_one_wide_head": bz.several([bz.parallel((1, 1, 4, 4), (1, 150, 3), 0.2, 1.0)]),
    "dense_feed_forward": bz.several([{**ATT, "mlp": bz.dense(40)}]),
    "routed_with_shared_gate": bz.several([{**ATT, "mlp": bz.moe(8, 3, 16, 4, 2, shared=24)}]),
    "routed_without_shared_top_one": bz.several([{**ATT, "mlp": bz.moe(4, 1, 16, 1, 1)}]),
    "routed_every_group_kept": bz.several([{**ATT, "mlp": bz.moe(6, 4, 16, 3, 3, shared=8)}]),
    "two_norms_large_eps": bz.several([{**ATT, "mlp": bz.dense(24)}], eps=0.3),
    "scales": bz.several([ATT], embedding_scale=0.05, logit_scale=7.0),
}


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("what", list(ALONE))
def test_one_mechanism_alone(tmp_path, what, dtype):
    config = ALONE[what]
    state = bz.random_state(config, 31)
    folder = bz.write(str(tmp_path / "m"), config, state)
    reqs = {"a": bz.tokens(1, 41, 90), "b": bz.tokens(2, 3, 90), "c": bz.tokens(3, 1, 90)}
    for cut in ("whole", "portions", "decode_tail"):
        run_and_compare(folder, config, state, reqs, CUTS[cut](reqs), dtype, 8, f"{what}, {cut}")


# --------------------------------------------------------------- whole models, every cut
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("which", list(bz.BZ))
@pytest.mark.parametrize("cut", list(CUTS))
def test_cut_matches_plain(models, which, dtype, cut):
    """Exactly as many pages as the schedule's peak needs and (mixed) four slots for five requests: pages and
    state slots are used again; free pages hold NaN."""
    reqs = requests_of(which)
    run_and_compare(models[which], bz.BZ[which], state_of(which), reqs, CUTS[cut](reqs), dtype, bz.PAGE[which],
                    f"{which} {cut}")


@pytest.mark.parametrize("which", list(bz.BZ))
def test_float32_cuts_agree_bitwise(models, which):
    """In float32 the logits at a position depend neither on the cut nor on the batch: every token runs the
    same operations in the same order whatever else the step holds."""
    reqs = requests_of(which)
    results = {}
    for cut, fn in CUTS.items():
        schedule = fn(reqs)
        engine = bz.make_engine(models[which], "float32", bz.PAGE[which], rd.peak_tokens(schedule, bz.PAGE[which]))
        results[cut] = run_engine(engine, reqs, schedule)
    for cut in ("decode_tail", "portions", "mixed"):
        for rid in reqs:
            assert torch.equal(results[cut][rid], results["whole"][rid]), (cut, rid)


def test_tensor_core_attention_takes_the_filled_heads(models, monkeypatch):
    """Configuration B in bfloat16 (heads of 32, and of 40 to 80 filled up to 64 and 128): decoded tokens take
    the split-KV tensor-core kernel, prompt portions the tiled one, none the generic kernel."""
    from freetoken_b200.csrc import ops
    calls = {"prefill": 0, "decode": 0}
    real_p, real_d = ops.attn_prefill, ops.attn_decode
    monkeypatch.setattr(ops, "attn_prefill", lambda *a, **k: (calls.__setitem__("prefill", 1), real_p(*a, **k))[1])
    monkeypatch.setattr(ops, "attn_decode", lambda *a, **k: (calls.__setitem__("decode", 1), real_d(*a, **k))[1])
    monkeypatch.setattr(ops, "attn_paged_simt", lambda *a, **k: pytest.fail("the generic kernel ran"))
    reqs = requests_of("B")
    run_and_compare(models["B"], bz.BZ["B"], state_of("B"), reqs, rd.mixed(reqs), "bfloat16", 64, "B mixed, fast kernels")
    assert calls == {"prefill": 1, "decode": 1}


# --------------------------------------------------------------------- a far key that decides
def sharpen(config, state, asker, stand_in, lead, scope):
    """Choose a target token and rewrite the query projection of the first layer so that token ``asker``'s query
    is, in every head, a multiple of the target's key in the dimensions that do not turn and zero in those that do,
    with a score ``lead`` above every other token's: ``asker`` puts nearly all its weight on the target, whatever
    the distance.  Returns the target."""
    m = config["layers"][0]["mixer"]
    a = m if scope == "l0.mix." else m["left"]
    H, G, D = a["heads"], a["kv_heads"], a["dim"]
    turned = a["rot"]["dims"] if "rot" in a else 0
    h = plain.layer_norm(state["embed"] * config["embedding"]["scale"], state["l0.norm1"], config["norm"]["eps"])
    k = (h @ state[scope + "k"].T + state[scope + "k.b"]).view(-1, G, D)
    still = k.clone()
    still[:, :, :turned] = 0
    dots = torch.einsum("tgd,jgd->tjg", still, still)
    own = torch.diagonal(dots).T.clone()                             # [tokens, G]
    dots[torch.arange(len(h)), torch.arange(len(h))] = float("-inf")
    margin = own - dots.amax(1)
    usable = margin.amin(1)
    usable[[asker, stand_in]] = float("-inf")
    target = int(usable.argmax())
    assert float(usable[target]) > 0
    want = (lead / (margin[target] * a["scale"]))[:, None] * still[target]
    want = want.repeat_interleave(H // G, 0).reshape(-1) - state[scope + "q.b"]
    q, ha = state[scope + "q"], h[asker]
    q = q + ((want - q @ ha)[:, None] * ha[None, :]) / ha.dot(ha)
    state[scope + "q"] = q.to(torch.bfloat16).double()
    return target


FAR = {
    "attention": (lambda d, v: bz.attention(4, 2, d, v, d // 4 * 2, base=500.0), "l0.mix."),
    "parallel": (lambda d, v: bz.parallel((4, 2, d, v), (2, 8, 4), 1.0, 0.1), "l0.mix.left."),
}


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("kind", list(FAR))
@pytest.mark.parametrize("dim,vdim,page", [(20, 12, 8), (32, 32, 16), (40, 64, 64), (128, 64, 64)])
def test_a_far_key_decides(tmp_path, kind, dim, vdim, page, dtype):
    """The asking token finds its target at the very first position and right before, on and right after page
    borders, hundreds of keys back, from inside a prompt portion and as a decoded token."""
    make, scope = FAR[kind]
    config = bz.several([make(dim, vdim)], vocab=120, width=64)
    state = bz.random_state(config, 41)
    asker, stand_in = 7, 13
    target = sharpen(config, state, asker, stand_in, 12.0, scope)
    n = 330
    reqs = {}
    for place in (0, page - 1, page, page + 1, n - 45):
        toks = [t if t not in (asker, target) else stand_in for t in bz.tokens(60 + place, n, 120)]
        toks[place] = target
        for at in (n - 40, n - 1):
            toks[at] = asker
        reqs[f"p{place}"] = toks
    want, noise = expected_for(config, state, reqs, dtype)
    blind = [t if t != target else stand_in for t in reqs["p0"]]
    assert float(bz.position_errors(plain.forward(config, state, blind)[-1:], want["p0"][-1:])) > 0.2
    folder = bz.write(str(tmp_path / "m"), config, state)
    tol = bz.TOL[dtype] * (1 if dtype == "float32" else 2)      # a sharp softmax: rounding of scores counts more
    for cut in ("whole", "decode_tail", "mixed"):
        schedule = CUTS[cut](reqs)
        engine = bz.make_engine(folder, dtype, page, rd.peak_tokens(schedule, page), poison=True)
        bz.compare(run_engine(engine, reqs, schedule), want, tol, f"far key, {kind}, {cut} [{dtype}]", noise)


# ------------------------------------------------------- a token far back, through the state
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_a_far_token_reaches_through_the_state(tmp_path, dtype):
    """A state that forgets slowly, and only one token that writes much into it: it stands once, 250 to 300
    positions back - right before, on and right after a page border, and first of all - and reaches the last
    tokens only through the state carried from step to step (the attention beside it is scaled away).  Another
    token in its place changes their logits wholly."""
    vocab = 24
    config = bz.several([bz.parallel((1, 1, 8, 8), (3, 24, 6), 0.0, 1.5)], vocab=vocab, width=48)
    state = bz.random_state(config, 51, slow_decay=True)
    p, target, stand_in = "l0.mix.right.", 5, 6
    state[p + "w0"] = (state[p + "w0"] - 2.0).to(torch.bfloat16).double()
    state[p + "mu.v"] *= 0                        # values of the token alone, so that one matrix serves every token
    h = plain.layer_norm(state["embed"] * config["embedding"]["scale"], state["l0.norm1"], config["norm"]["eps"])
    y = 0.02 * (h @ state[p + "v"].T)             # everybody's values shrink ...
    y[target] = 4.0 * (h[target] @ state[p + "v"].T)       # ... but the target's grow
    state[p + "v"] = torch.linalg.lstsq(h, y).solution.T.contiguous().to(torch.bfloat16).double()
    page, n = 16, 300
    reqs = {}
    for place in (15, 16, 17, 0, 49):
        toks = [t if t != target else stand_in for t in bz.tokens(70 + place, n, vocab)]
        toks[place] = target
        reqs[f"t{place}"] = toks
    want, noise = expected_for(config, state, reqs, dtype)
    other = list(reqs["t16"])
    other[16] = stand_in
    assert float(bz.position_errors(plain.forward(config, state, other)[-1:], want["t16"][-1:])) > 0.3
    folder = bz.write(str(tmp_path / "m"), config, state)
    # the shrunk values are small differences of large products of a rounded input (whatever computes them)
    tol = bz.TOL[dtype] * (2 if dtype == "bfloat16" else 1)
    for cut in ("decode_tail", "portions", "mixed"):
        schedule = CUTS[cut](reqs)
        engine = bz.make_engine(folder, dtype, page, rd.peak_tokens(schedule, page), poison=True)
        bz.compare(run_engine(engine, reqs, schedule), want, tol, f"far token, {cut} [{dtype}]", noise, mostly=0.8)


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_the_previous_token_crosses_every_cut(tmp_path, dtype):
    """Mixes of one: the time mixer sees the previous token only, and a decay that keeps nothing: a shift from
    the wrong row, a stale slot or a slot that is not cleared changes the logits wholly."""
    config = bz.several([bz.parallel((1, 1, 8, 8), (2, 12, 3), 0.0, 1.0)])
    state = bz.random_state(config, 52)
    for name in "rkvgw":
        state[f"l0.mix.right.mu.{name}"] = torch.ones_like(state[f"l0.mix.right.mu.{name}"])
    state["l0.mix.right.w0"] = torch.full_like(state["l0.mix.right.w0"], 4.0)
    folder = bz.write(str(tmp_path / "m"), config, state)
    reqs = {f"r{i}": bz.tokens(90 + i, n, 90) for i, n in enumerate((1, 2, 17, 30, 9, 4))}
    for cut in CUTS:
        run_and_compare(folder, config, state, reqs, CUTS[cut](reqs), dtype, 8, f"previous token, {cut}")


# ------------------------------------------------- long prompts at sizes between tiny and real
LONG = bz.model(640, 256, 1e-5, [
    bz.attention(8, 2, 64, 64, 32, base=1e5, mlp=bz.dense(512)),
    bz.parallel((4, 4, 64, 112), (4, 64, 24), 0.9, 0.6, bz.moe(16, 4, 64, 4, 2, shared=128)),
    bz.attention(6, 2, 56, 64, 40, base=2e6, mlp=bz.moe(8, 2, 96, 2, 1)),
], embedding_scale=0.9, logit_scale=0.7)


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_long_prompts(tmp_path, dtype):
    """Prompts of up to 1,200 tokens (the kernels for many rows: batched products, the scan over dozens of
    chunks, the shift that walks four tokens), whole and in a mixed batch whose decoded tokens read hundreds of
    keys, states that forget slowly."""
    state = bz.random_state(LONG, 7, slow_decay=True)
    folder = bz.write(str(tmp_path / "m"), LONG, state)
    reqs = {f"r{i}": bz.tokens(11 * i + 3, n, LONG["vocab"]) for i, n in enumerate([1200, 500, 64, 65, 129])}
    for cut in ("whole", "mixed"):
        run_and_compare(folder, LONG, state, reqs, CUTS[cut](reqs), dtype, 64, f"long {cut}")


# --------------------------------------------------------- first tokens, long decoding
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_first_tokens_and_long_decoding(models, dtype):
    """A request that starts with a single token and is decoded one token at a time for 200 steps, beside a
    second request that joins later two tokens a step; against the whole sequences."""
    config, state = bz.BZ["A"], state_of("A")
    reqs = {"a": bz.tokens(5, 201, config["vocab"]), "b": bz.tokens(6, 120, config["vocab"])}
    schedule = []
    for i in range(201):
        entries = [("a", i, 1)]
        j = i - 60
        if 0 <= j < 60:
            entries.append(("b", 2 * j, 2))
        schedule.append((entries, ["a"] if i == 200 else []))
    schedule[-1] = (schedule[-1][0], ["a", "b"])
    run_and_compare(models["A"], config, state, reqs, schedule, dtype, 4, "long decoding")


# ------------------------------------------------------------------------ generation
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("which", ["A", "B"])
def test_greedy_generation_through_the_scheduler(models, which, dtype):
    """``LLM.generate`` (scheduler, overlapped steps, graph replay of decode steps in bfloat16): every generated
    token is the plain model's own greedy choice for the sequence so far, unless its two best logits - or two
    router scores somewhere in the sequence - lie within rounding of each other."""
    from freetoken_b200 import LLM, SamplingParams
    config, state = bz.BZ[which], state_of(which)
    llm = LLM(models[which], dtype, page_size=bz.PAGE[which], num_token_override=1024, max_running_req=3,
              max_extend_tokens=24)
    prompts = [bz.tokens(70 + i, n, config["vocab"]) for i, n in enumerate((3, 30, 11, 1, 47))]
    out = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    tie = 1e-4 if dtype == "float32" else 8e-2
    route_tie = 2e-2
    ties = 0
    for prompt, result in zip(prompts, out):
        seq = list(prompt)
        assert len(result["token_ids"]) == 12
        for token in result["token_ids"]:
            margins = []
            logits = plain.forward(config, state, seq, margins=margins)[-1]
            if token != int(logits.argmax()):
                margin = min((float(m.min()) for m in margins), default=float("inf"))
                near = float(logits.max() - logits[token]) < tie or (dtype == "bfloat16" and margin < route_tie)
                assert near, (dtype, len(seq), token, int(logits.argmax()), float(logits.max() - logits[token]), margin)
                ties += 1
                if margin < route_tie:
                    break            # another expert somewhere in the sequence: what follows is another sequence
            seq.append(int(token))
    assert ties == 0 if dtype == "float32" else ties <= 4
    if dtype == "bfloat16":
        assert llm.engine.graph_replays > 0


# -------------------------------------------------------------------- the replay tool
def test_trace_replay_tool(models, tmp_path):
    """``bin/trace_run`` on a Besuzen folder (whose config.json does not state the middle of the decay's
    projection): a mixed schedule with exactly the pages its peak needs."""
    which = "C"
    reqs = requests_of(which)
    schedule = rd.mixed(reqs)
    page = bz.PAGE[which]
    got = rd.run_trace_tool(models[which], "float32", reqs, schedule, str(tmp_path / "out"),
                            rd.peak_tokens(schedule, page), page, bz.BZ[which]["vocab"])
    bz.compare(got, expected_for(bz.BZ[which], state_of(which), reqs, "float32")[0], bz.TOL["float32"], "trace_run, mixed")
