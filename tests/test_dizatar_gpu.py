"""Dizatar in the engine against the plain implementation: every new kernel alone, every mechanism alone
in a one-layer model, whole prompts against decoding, portions down to two tokens, mixed batches with pages
used again, both forms of the latent attention in one batch, far keys made decisive on purpose, the first
tokens, long decoding, configurations that differ in every size, greedy generation through the scheduler,
the trace replay tool."""

import copy

import pytest
import torch

import dizatar_tiny as dz
import plain_dizatar as plain
import replay_driver as rd

pytestmark = pytest.mark.gpu

LENGTHS = {"A": [1, 2, 9, 37, 70], "B": [3, 150, 66, 260, 21], "C": [2, 75, 129, 5], "D": [40, 1, 97]}
CUTS = {"whole": rd.whole, "decode_tail": rd.decode_tail, "portions": rd.portions, "mixed": rd.mixed,
        # portions on either side of the length from which a context's keys and values are made
        "mixed_long": lambda reqs: rd.mixed(reqs, sizes=(64, 2, 100, 63, 17, 130))}
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def requests_of(which):
    vocab = dz.DZ[which]["vocab"]
    return {f"r{i}": dz.tokens(40 * i + ord(which), n, vocab) for i, n in enumerate(LENGTHS[which])}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {which: dz.write_tiny(str(tmp_path_factory.mktemp(f"dz{which}")), which) for which in dz.DZ}


def run_engine(engine, reqs, schedule, routing=None):
    """Drive ``engine.step`` through a schedule; logits of every position of every request.  With
    ``routing`` (a dict) the experts the engine chose are left there: ``routing[request][j]`` is
    ``[positions, top]`` of the j-th routed layer run."""
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
    engine.check_status()
    engine.cache.check_integrity()
    return out


def expected_for(config, state, reqs, dtype, routing=None):
    """The plain model's logits; in bfloat16 with the experts the engine chose (two correct
    implementations may choose differently where two choice scores lie within rounding)."""
    runs = dz.routed_runs(config)
    return {rid: plain.forward(config, state, toks, expert_ids=dict(zip(runs, routing[rid]))
                               if dtype == "bfloat16" and routing else None) for rid, toks in reqs.items()}


def run_and_compare(folder, config, state, reqs, schedule, dtype, page, what, tol=None):
    engine = dz.make_engine(folder, dtype, page, rd.peak_tokens(schedule, page), poison=True)
    routing = {} if dz.routed_runs(config) else None
    got = run_engine(engine, reqs, schedule, routing)
    dz.compare(got, expected_for(config, state, reqs, dtype, routing), tol or dz.TOL[dtype], f"{what} [{dtype}]")
    assert engine.cache.free_pages() == engine.cache.total_pages()
    return got


def close(got, want, dtype, what=""):
    tol = 2e-5 if dtype == "float32" else 2e-2
    g, w = got.double().cpu(), want.double()
    assert torch.allclose(g, w, atol=tol * max(1.0, float(w.abs().max())), rtol=tol), (what, float((g - w).abs().max()))


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------ kernels, each alone
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("T,k,H", [(3, 1, 40), (5, 3, 64), (2, 6, 1030), (9, 2, 2048), (1, 8, 4096), (4, 5, 45), (2, 33, 256)])
def test_rows_of_a_routed_feed_forward(dtype, T, k, H):
    """Routed rows, handed-back inputs (their slots' rows hold NaN: never read) and one shared row: the sum,
    the norm that adds it into the residual with the next norm and a copy behind it, the plain join; the next
    norm's output may lie where the handed-back input lies."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(T * 10 + k)
    dt = DTYPES[dtype]
    E = 4
    ids = torch.randint(0, E + 3, (T, k))
    ids[0, 0] = E                                          # at least one slot hands back, and one row has no expert at all
    if T > 1:
        ids[1] = E + 1
    w = torch.rand(T, k)
    rows = torch.randn(T, k, H).to(dt)
    h, extra, x = torch.randn(T, H).to(dt), torch.randn(T, H).to(dt), torch.randn(T, H)
    back = (w.double() * (ids >= E)).sum(1)
    masked = rows.double() * (ids < E)[:, :, None]
    garbage = rows.clone()
    garbage[ids >= E] = float("nan")
    w1, w2 = torch.randn(H), torch.randn(H)
    for with_ids, with_extra in ((True, True), (True, False), (False, True)):
        z = (masked if with_ids else rows.double()).sum(1) + (back[:, None] * h.double() if with_ids else 0) \
            + (extra.double() if with_extra else 0)
        branch = ops.RoutedRows((garbage if with_ids else rows).cuda(), ids.int().cuda() if with_ids else None,
                                w.cuda() if with_ids else None, E, h.cuda() if with_ids else None,
                                extra.cuda() if with_extra else None)
        out = torch.empty(T, H, dtype=dt, device="cuda")
        ops.branch_sum(branch, out)
        close(out, z, dtype, "branch_sum")
        res = x.cuda().clone()
        wide = torch.zeros(T, 2 * H + 8, dtype=dt, device="cuda")
        nxt = branch.source if with_ids else torch.empty(T, H, dtype=dt, device="cuda")
        ops.norm_add(branch, res, w1.cuda(), 1e-5, False, 0.7, next_weight=w2.cuda(), next_eps=1e-4, next_out=nxt,
                     copy_out=wide[:, 4:4 + H])
        new = x.double() + 0.7 * plain.rms(z, 1e-5) * w1.double()
        close(res, new, "float32" if dtype == "float32" else dtype, "residual")
        close(nxt, plain.rms(new, 1e-4) * w2.double(), dtype, "next norm")
        close(wide[:, 4:4 + H], new, dtype, "copy")
        assert float(wide[:, :4].abs().max()) == 0 and float(wide[:, 4 + H:].abs().max()) == 0
        if with_ids:
            branch.source = h.cuda()
        res = x.cuda().clone()
        ops.cast_rows(res, wide[:, :H], branch)
        close(res, x.double() + z, dtype, "join")
        close(wide[:, :H], x.double() + z, dtype, "join's copy")
    res = x.cuda().clone()
    ops.cast_rows(res, wide[:, H:2 * H])
    assert torch.equal(res, x.cuda()) and torch.equal(wide[:, H:2 * H], x.cuda().to(dt))


@pytest.mark.parametrize("E,identity,top,T", [(8, 2, 2, 5), (1, 3, 4, 3), (5, 20, 3, 70), (40, 24, 6, 700), (6, 1, 1, 8)])
def test_routes_of_identity_experts_lie_behind_all_others(E, identity, top, T):
    """Softmax over all outputs, chosen by score plus correction, weighted by the score alone; the sort
    places the identity experts' routes last and keeps them out of the list of busy experts - one launch for
    few tokens, two or three for many."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(E)
    n = E + identity
    logits, bias = torch.randn(T, n) * 2, torch.randn(n) * 0.2
    w = {"r.router": torch.eye(n, dtype=torch.float64), "r.correction": bias.double()}
    want_ids, s = plain.choose_experts(logits.double(), w, "r.", {"top": top})
    ids = torch.empty(T, top, dtype=torch.int32, device="cuda")
    wts = torch.empty(T, top, device="cuda")
    ops.router_select(logits.cuda(), bias.cuda(), ids, wts, top, True, True, 1.0)
    assert torch.equal(ids.cpu().long(), want_ids)
    picked = s.gather(1, want_ids)
    assert torch.allclose(wts.cpu().double(), picked / picked.sum(1, keepdim=True), atol=1e-6)
    R = T * top
    flat = want_ids.view(-1)
    order = torch.sort(flat, stable=True).indices
    counts = torch.bincount(flat, minlength=n)
    busy = [e for e in range(E) if counts[e] > 0]

    def check(bufs, what):
        c, off, sr, st, act = (b.cpu().long() for b in bufs)
        assert torch.equal(c, counts) and torch.equal(off, torch.cat([torch.zeros(1, dtype=torch.long), counts.cumsum(0)])), what
        assert torch.equal(sr, order) and torch.equal(st, order // top), what
        assert int(act[E]) == len(busy) and act[:len(busy)].tolist() == busy, what

    def bufs():
        return [torch.full((m,), -7, dtype=torch.int32, device="cuda") for m in (n, n + 1, R, R, E + 1)]
    for scratch in (None, torch.empty(ops.moe_sort_scratch(R, n), dtype=torch.int32, device="cuda")):
        b = bufs()
        ops.moe_sort(ids.view(-1), *b, n, top, scratch, busy_of=E)
        check(b, f"moe_sort, scratch {scratch is not None}")
    if ops.route_small_takes(T, n, top):
        b = bufs()
        ids2, w2 = torch.empty_like(ids), torch.empty_like(wts)
        ops.route_small(logits.cuda(), bias.cuda(), ids2, w2, *b, top, True, True, 1.0, busy_of=E)
        assert torch.equal(ids2, ids) and torch.equal(w2, wts)
        check(b, "route_small")


def test_gated_rows_in_pieces_and_turned_queries_in_place():
    from freetoken_b200.csrc import ops
    from freetoken_b200.parts.position import rotary_table
    torch.manual_seed(4)
    for I in (64, 88, 45):
        gu = (2 * torch.randn(7, 2 * I)).to(torch.bfloat16)
        mid = torch.empty(7, I, dtype=torch.bfloat16, device="cuda")
        ops.glu_rows(gu.cuda(), mid, "silu")
        g = gu.double()
        close(mid, plain.silu(g[:, :I]) * g[:, I:], "bfloat16", f"silu pair of {I}")
    for dt in (torch.float32, torch.bfloat16):
        heads, dq, rank, rot, page, T = 3, 5, 12, 6, 4, 9
        z = torch.randn(T, heads * (dq + rot) + rank + rot).to(dt)
        zc = z.cuda()
        pages = torch.zeros(4, 1, page, rank + rot, dtype=dt, device="cuda")
        q_abs = torch.zeros(T, heads, rank + rot, dtype=dt, device="cuda")
        w = torch.randn(rank)
        cut = heads * (dq + rot)
        ops.latent_store(zc[:, cut:], zc[:, :cut], q_abs, pages, w.cuda(), rotary_table(rot, 30.0, "cuda", 16, exact_angles=True),
                         ints(list(range(2, 2 + T))), ints([0] * T), ints([[1, 3, 2]]), heads=heads, q_dim=dq, rank=rank,
                         rot=rot, interleaved=False, eps=1e-5, turn_q=True)
        d = str(dt).split(".")[1]
        q = z[:, :cut].double().view(T, heads, dq + rot)
        turned = plain.rotate_halves(q[..., dq:], 30.0, rot, first=2)
        close(q_abs[:, :, rank:], turned, d, "query tails")
        close(zc[:, :cut].reshape(T, heads, dq + rot)[..., dq:], turned, d, "query tails in place")
        assert torch.equal(zc[:, :cut].reshape(T, heads, dq + rot)[..., :dq].cpu(), z[:, :cut].view(T, heads, dq + rot)[..., :dq])
        assert torch.equal(zc[:, cut:].cpu(), z[:, cut:])
        for t in range(T):
            p = t + 2
            row = pages[[1, 3, 2][p // page], 0, p % page].double().cpu()
            close(row[:rank], plain.rms(z[t, cut:cut + rank].double(), 1e-5) * w.double(), d, "latent")
            close(row[rank:], plain.rotate_halves(z[t, cut + rank:].double().view(1, 1, rot), 30.0, rot, first=p)[0, 0], d, "key part")


def paged_rows(segs, page, d):
    """Random cached rows of segments ``(pos0, n)`` in shuffled pages; everything else in the cache is NaN."""
    counts = [-(-(p + n) // page) for p, n in segs]
    order = (torch.randperm(sum(counts)) + 1).tolist()
    table = torch.zeros(len(segs), max(counts), dtype=torch.int32)
    pages = torch.full((sum(counts) + 1, 1, page, d), float("nan"), dtype=torch.bfloat16)
    rows = []
    for i, (p, n) in enumerate(segs):
        r = torch.randn(p + n, d).to(torch.bfloat16)
        rows.append(r)
        for j in range(counts[i]):
            table[i, j] = order.pop()
            part = r[j * page:(j + 1) * page]
            pages[table[i, j], 0, :len(part)] = part
    starts = [0]
    for _, n in segs:
        starts.append(starts[-1] + n)
    return pages.cuda(), table.cuda(), rows, ints(starts), ints([p for p, _ in segs]), ints([p + n for p, n in segs])


ROWS = [(104, 88, 7, 64), (576, 512, 16, 64), (576, 512, 33, 16), (40, 24, 3, 4), (24, 24, 20, 8), (1024, 1000, 5, 64),
        (264, 256, 16, 32), (120, 56, 1, 12), (160, 152, 20, 64), (576, 568, 20, 64), (320, 264, 2, 16), (256, 200, 18, 64)]


@pytest.mark.parametrize("d,rank,H,page", ROWS)
def test_absorbed_attention_over_rows_of_any_width(d, rank, H, page):
    """Single tokens and short portions together, one split and many, windows, pages of any size; rows past a
    request's end, or before its window, are never read (they hold NaN)."""
    from freetoken_b200.csrc import ops
    from freetoken_b200.parts.base import Workspace
    torch.manual_seed(d + H)
    ws = Workspace("cuda")
    for segs in ([(0, 1)], [(5, 1), (130, 1), (64, 2)], [(1300, 1), (63, 1), (62, 5)], [(0, 40), (300, 17), (31, 1)]):
        for window in (None, 33):
            pages, table, rows, starts, pos0, _ = paged_rows(segs, page, d)
            T = int(starts[-1])
            q = (torch.randn(T, H, d) * 0.5).to(torch.bfloat16)
            rt = ops.latent_row_tile(H, d, rank)
            flat = [(i, r) for i, (_, n) in enumerate(segs) for r in range(0, n * H, rt)]
            out = torch.full((T, H, rank), float("nan"), dtype=torch.bfloat16, device="cuda")
            ops.attn_latent(q.cuda(), out, pages, ints([a for a, _ in flat]), ints([b for _, b in flat]), starts, pos0,
                            table, H, rank, d ** -0.5, window, max(p + n for p, n in segs), ws)
            t = 0
            for i, (p, n) in enumerate(segs):
                for a in range(n):
                    keys = rows[i][max(0, p + a - window + 1) if window else 0:p + a + 1].double()
                    want = torch.softmax(q[t].double() @ keys.T * d ** -0.5, -1) @ keys[:, :rank]
                    close(out[t], want, "bfloat16", (segs, window, i, a))
                    t += 1
    ops.check_tc_status("cuda:0")


@pytest.mark.parametrize("dk,rot,dv,H,page,rank", [(56, 24, 40, 5, 64, 104), (128, 64, 128, 3, 64, 512), (24, 8, 8, 3, 4, 24),
                                                   (72, 0, 120, 2, 8, 40), (192, 64, 128, 4, 64, 256), (8, 40, 64, 5, 16, 16),
                                                   (16, 104, 72, 1, 12, 8)])
def test_expanded_attention_over_gathered_rows(dk, rot, dv, H, page, rank):
    """The context's cached rows gathered, keys and values made from them, prompts of several requests with
    contexts before them; key tiles that end inside another request's rows; windows."""
    from freetoken_b200.csrc import ops
    torch.manual_seed(dk + rot)
    d = rank + rot
    for segs in ([(0, 64)], [(0, 128), (0, 129)], [(37, 200), (130, 64), (64, 77)], [(700, 90)], [(0, 400), (3, 65)]):
        for window in (None, 50):
            pages, table, rows, starts, pos0, kv_len = paged_rows(segs, page, d)
            T = int(starts[-1])
            q = (torch.randn(T, H * (dk + rot) + 8) * 0.5).to(torch.bfloat16)
            up = (torch.randn(H * (dk + dv), rank) * rank ** -0.5).to(torch.bfloat16)
            tiles, blocks, at = [], [], 0
            for i, (p, n) in enumerate(segs):
                base = max(0, p - window + 1) // 64 * 64 if window else 0
                context = -(-(p + n - base) // 64) * 64
                tiles += [(i, q0, at - base) for q0 in range(0, n, 128)]
                blocks += [(i, base + k, at + k) for k in range(0, context, 64)]
                at += context
            flat = torch.full((at, d), float("nan"), dtype=torch.bfloat16, device="cuda")
            ops.latent_gather(pages, flat, *(ints([b[c] for b in blocks]) for c in range(3)), kv_len, pos0, table, window)
            assert not torch.isnan(flat).any()
            made = flat[:, :rank] @ up.cuda().t()
            out = torch.full((T, H * dv), float("nan"), dtype=torch.bfloat16, device="cuda")
            ops.attn_prefill_mha(q.cuda()[:, :H * (dk + rot)], made[:, :H * dk].unflatten(1, (H, dk)),
                                 flat[:, rank:] if rot else None, made[:, H * dk:].unflatten(1, (H, dv)), out,
                                 *(ints([t[c] for t in tiles]) for c in range(3)), starts, pos0, H, dk, rot, dv,
                                 (dk + rot) ** -0.5, window)
            t = 0
            for i, (p, n) in enumerate(segs):
                latent = rows[i].double()
                kv = (latent[:, :rank] @ up.double().T).to(torch.bfloat16).double()
                k, v = kv[:, :H * dk].view(-1, H, dk), kv[:, H * dk:].view(-1, H, dv)
                qd = q[t:t + n, :H * (dk + rot)].double().view(n, H, dk + rot)
                s = torch.einsum("ihd,jhd->hij", qd[..., :dk], k) + torch.einsum("ihd,jd->hij", qd[..., dk:], latent[:, rank:])
                a, b = torch.arange(p, p + n)[:, None], torch.arange(p + n)[None]
                hidden = (b > a) | ((a - b >= window) if window else (b > a))
                s = (s * (dk + rot) ** -0.5).masked_fill(hidden[None], float("-inf"))
                want = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v).reshape(n, H * dv)
                close(out[t:t + n], want, "bfloat16", (segs, window, i))
                t += n
    ops.check_tc_status("cuda:0")


def test_expanded_attention_repeats_bitwise_on_a_full_grid():
    from freetoken_b200.csrc import ops
    torch.manual_seed(1)
    T, H, dk, rot, dv = 1500, 16, 128, 64, 128
    q = torch.randn(T, H * (dk + rot), device="cuda", dtype=torch.bfloat16)
    rows = torch.randn(1536, rot, device="cuda", dtype=torch.bfloat16)
    made = torch.randn(1536, H * (dk + dv), device="cuda", dtype=torch.bfloat16)
    tiles = list(range(0, T, 128))
    first = None
    for _ in range(20):
        out = torch.empty(T, H * dv, device="cuda", dtype=torch.bfloat16)
        ops.attn_prefill_mha(q, made[:, :H * dk].unflatten(1, (H, dk)), rows, made[:, H * dk:].unflatten(1, (H, dv)), out,
                             ints([0] * len(tiles)), ints(tiles), ints([0] * len(tiles)), ints([0, T]), ints([0]), H, dk,
                             rot, dv, (dk + rot) ** -0.5)
        first = out if first is None else first
        assert torch.equal(out, first)
    ops.check_tc_status("cuda:0")


# ------------------------------------------------------------------- mechanisms, each alone
PLAIN = dz.layer(3, 8, 6, 10, 14)
ALONE = {
    "latent_attention": dz.one_layer(PLAIN),
    "one_head_narrow_latent": dz.one_layer(dz.layer(1, 12, 4, 20, 3, base=50.0)),
    "two_rotated_dimensions": dz.one_layer(dz.layer(2, 6, 2, 4, 9, base=3.0, scale=0.9)),
    "nothing_rotated": dz.one_layer(dz.layer(4, 8, 0, 16, 24)),
    "rows_wider_than_512": dz.one_layer(dz.layer(2, 8, 8, 16, 520)),
    "more_than_16_heads": dz.one_layer(dz.layer(18, 8, 8, 8, 32)),
    "latent_of_one_block_on_the_own_kernels": dz.one_layer(dz.layer(3, 16, 16, 24, 24)),
    "residual_factor": dz.one_layer(PLAIN, mult=0.3),
    "cap": dz.one_layer(PLAIN, cap=0.4),
    "experts": dz.one_layer(dz.layer(1, 4, 2, 4, 6, dz.moe(6, 2, 24))),
    "experts_that_hand_back": dz.one_layer(dz.layer(1, 4, 2, 4, 6, dz.moe(4, 3, 24, identity=4))),
    "a_shared_expert": dz.one_layer(dz.layer(1, 4, 2, 4, 6, dz.moe(5, 1, 16, shared=40))),
    "everything_chosen": dz.one_layer(dz.layer(1, 4, 2, 4, 6, dz.moe(2, 5, 16, identity=3, shared=8))),
    "loop_of_one_pass": dz.model(90, 48, [copy.deepcopy(PLAIN), dz.layer(2, 4, 4, 4, 8)], loop=(1, 2, 1)),
    "loop_over_the_first_layer": dz.model(90, 48, [copy.deepcopy(PLAIN), dz.layer(2, 4, 4, 4, 8)], loop=(0, 1, 4), mult=0.7),
    "loop_over_everything": dz.model(90, 48, [copy.deepcopy(PLAIN), dz.layer(2, 4, 4, 4, 8)], loop=(0, 2, 2)),
}


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("what", list(ALONE))
def test_one_mechanism_alone(tmp_path, what, dtype):
    config = ALONE[what]
    state = dz.random_state(config, 31)
    folder = dz.write(str(tmp_path / "m"), config, state)
    reqs = {"a": dz.tokens(1, 81, 90), "b": dz.tokens(2, 3, 90), "c": dz.tokens(3, 1, 90)}
    for cut in ("whole", "portions", "decode_tail"):
        run_and_compare(folder, config, state, reqs, CUTS[cut](reqs), dtype, 8, f"{what}, {cut}")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_a_correction_only_chooses(tmp_path, dtype):
    """Corrections that force an identity expert, or an expert the scores would never take, onto every
    token: the choice follows them, the weight is the score's share."""
    config = dz.one_layer(dz.layer(1, 4, 2, 4, 6, dz.moe(4, 2, 24, identity=2, shared=8)))
    for forced in ([0, 0, 0, 0, 30, 0], [0, 0, 30, 0, 0, 25], [0, 0, 0, 0, 30, 31]):
        state = dz.random_state(config, 33)
        state["l0.mlp.correction"] = torch.tensor(forced, dtype=torch.float64)
        folder = dz.write(str(tmp_path / "m"), config, state)
        reqs = {"a": dz.tokens(4, 40, 90), "b": dz.tokens(5, 2, 90)}
        run_and_compare(folder, config, state, reqs, rd.decode_tail(reqs), dtype, 8, f"correction {forced}")


# --------------------------------------------------------------- whole models, every cut
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("which", list(dz.DZ))
@pytest.mark.parametrize("cut", list(CUTS))
def test_cut_matches_plain(models, which, dtype, cut):
    """Exactly as many pages as the schedule's peak needs and (mixed) four slots for five requests: pages
    are used again; free pages hold NaN."""
    reqs = requests_of(which)
    state = dz.random_state(dz.DZ[which], dz.SEEDS[which])
    run_and_compare(models[which], dz.DZ[which], state, reqs, CUTS[cut](reqs), dtype, dz.PAGE[which], f"{which} {cut}")


@pytest.mark.parametrize("which", list(dz.DZ))
def test_float32_cuts_agree_bitwise(models, which):
    """In float32 the logits at a position depend neither on the cut nor on the batch: every token runs the
    same operations in the same order whatever else the step holds."""
    reqs = requests_of(which)
    results = {}
    for cut, fn in CUTS.items():
        schedule = fn(reqs)
        engine = dz.make_engine(models[which], "float32", dz.PAGE[which], rd.peak_tokens(schedule, dz.PAGE[which]))
        results[cut] = run_engine(engine, reqs, schedule)
    for cut in CUTS:
        for rid in reqs:
            assert torch.equal(results[cut][rid], results["whole"][rid]), (cut, rid)


def test_both_forms_run(models, monkeypatch):
    from freetoken_b200.csrc import ops
    calls = {}

    def count(name):
        real = getattr(ops, name)
        monkeypatch.setattr(ops, name, lambda *a, **k: (calls.__setitem__(name, calls.get(name, 0) + 1), real(*a, **k))[1])
    for name in ("attn_latent", "attn_prefill_mha", "latent_gather", "attn_paged_simt"):
        count(name)
    reqs = requests_of("B")
    state = dz.random_state(dz.DZ["B"], dz.SEEDS["B"])
    run_and_compare(models["B"], dz.DZ["B"], state, reqs, CUTS["mixed_long"](reqs), "bfloat16", 64, "B mixed, both forms")
    assert min(calls[n] for n in ("attn_latent", "attn_prefill_mha", "latent_gather")) > 0 and "attn_paged_simt" not in calls


# --------------------------------------------- other arrangements of the same parts
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("kind", ["prenorm", "parallel"])
def test_routed_rows_and_stream_maps_in_other_blocks(tmp_path, kind, dtype):
    """A design of the test's own: the same mixer, experts that hand back, shared expert and map of the stream
    around pre-norm or parallel blocks."""
    import dataclasses

    from freetoken_b200.config.dizatar import DizatarConfig, build_plan
    from freetoken_b200.config.model_plan import PartSpec
    from freetoken_b200.registry import Architecture, register_architecture

    def plan_of(cfg):
        plan = build_plan(cfg)
        layers = []
        for spec in plan.layers:
            spec = dataclasses.replace(spec, block=PartSpec(kind, {}), norms={})
            layers.append(spec if kind == "prenorm" else dataclasses.replace(spec, feed_forward_norm=None))
        return dataclasses.replace(plan, layers=tuple(layers))
    name = f"ToyRouted{kind}"
    register_architecture(Architecture(name, DizatarConfig.from_dict, plan_of, lambda cfg: cfg.to_dict()))
    config = dz.model(90, 48, [dz.layer(2, 8, 4, 12, 10, dz.moe(4, 2, 16, identity=2, shared=24)),
                               dz.layer(3, 8, 8, 8, 24, dz.moe(3, 2, 16, shared=8))], loop=(0, 2, 2), cap=2.0)
    state = dz.random_state(config, 35)
    drop = ("norm1b", "norm2b", "ls1", "ls2") + (("norm2",) if kind == "parallel" else ())
    state = {k: v for k, v in state.items() if k.split(".")[-1] not in drop}
    folder = dz.write(str(tmp_path / "m"), {**config, "architecture": name}, state)
    reqs = {"a": dz.tokens(1, 75, 90), "b": dz.tokens(2, 9, 90)}
    eps = config["norm"]["eps"]

    def forward(toks, chosen):
        x0 = state["embed"][torch.tensor(toks)]
        x = x0
        for run, (i, starts) in enumerate(plain.run_order(config)):
            layer, p = config["layers"][i], f"l{i}."
            if starts:
                x = torch.cat([x, x0], -1) @ state["loop.in"].T
            h = plain.rms(x, eps) * state[p + "norm1"]
            a = plain.latent_attention(h, state, p + "mix.", layer["mixer"], eps)
            if kind == "prenorm":
                x = x + a
                h = plain.rms(x, eps) * state[p + "norm2"]
                a = 0
            x = x + a + plain.routed_ff(h, state, p + "mlp.", layer["mlp"], None if chosen is None else chosen[run])
        out = plain.rms(x, eps) * state["final.norm"] @ state["head"].T
        return 2.0 * torch.tanh(out / 2.0)
    for cut in ("whole", "mixed_long"):
        schedule = CUTS[cut](reqs)
        engine = dz.make_engine(folder, dtype, 8, rd.peak_tokens(schedule, 8), poison=True)
        routing = {}
        got = run_engine(engine, reqs, schedule, routing)
        want = {r: forward(t, routing[r] if dtype == "bfloat16" else None) for r, t in reqs.items()}
        dz.compare(got, want, dz.TOL[dtype], f"{kind}, {cut} [{dtype}]")


# ------------------------------------------------------------ a far key, decisive on purpose
def sharpen(config, state, asker, target, beta):
    """Rewrite the first layer's query matrix so that token ``asker``'s unrotated query is ``beta`` times token
    ``target``'s unrotated key in every head and its rotated part is zero: wherever ``target`` stands, ``asker``
    puts nearly all its weight there."""
    m, eps = config["layers"][0]["mixer"], config["norm"]["eps"]
    H, D, R = m["heads"], m["dim"], m["rot_dim"]
    x = state["embed"][[asker, target]]
    if config.get("loop"):
        x = torch.cat([x, x], -1) @ state["loop.in"].T          # (the loop starts at layer 0: its first pass)
    h = plain.rms(x, eps) * state["l0.norm1"]
    c = plain.rms((state["l0.mix.dkv"] @ h[1])[:m["kv_rank"]], eps) * state["l0.mix.dkv.norm"]
    k = (state["l0.mix.uk"] @ c).view(H, D)
    want = torch.cat([beta * k, torch.zeros(H, R, dtype=torch.float64)], dim=1).reshape(-1)
    q = state["l0.mix.q"]
    q = q - (q @ h[0])[:, None] * h[0][None, :] / h[0].dot(h[0]) + want[:, None] * h[0][None, :] / h[0].dot(h[0])
    state["l0.mix.q"] = q.to(torch.bfloat16).double()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("heads,dim,rot,rank,page,loop", [(2, 16, 8, 20, 8, None), (3, 32, 24, 88, 64, (0, 1, 2)), (17, 24, 8, 40, 16, None),
                                                          (2, 24, 24, 520, 64, None), (2, 40, 32, 96, 64, (0, 1, 1))])
def test_a_far_key_decides(tmp_path, heads, dim, rot, rank, page, loop, dtype):
    """The target stands once, first of all and right before, on and right after a page's or tile's border, up
    to 600 positions back among hundreds of keys, and is asked for from inside a prompt portion and by the
    last decoded token (rows of 28 values: the generic kernel; 112, 48 and 544: both forms of the own kernels;
    128: the paged kernels).  Another token in its place changes the answer wholly."""
    config = dz.one_layer(dz.layer(heads, dim, rot, 16, rank, scale=0.25), vocab=120, width=64, loop=loop)
    state = dz.random_state(config, 41)
    asker, target = 7, 11
    sharpen(config, state, asker, target, beta=160.0 / dim)
    n = 620
    reqs = {}
    for place in (0, 63, 64, 65, 127, 300):
        toks = [t if t not in (asker, target) else 13 for t in dz.tokens(60 + place, n, 120)]
        toks[place] = target
        toks[n - 45] = toks[n - 1] = asker
        reqs[f"t{place}"] = toks
    want = {rid: plain.forward(config, state, t) for rid, t in reqs.items()}
    blind = [t if t != target else 13 for t in reqs["t64"]]
    off = dz.position_errors(plain.forward(config, state, blind), want["t64"])
    tol = dz.TOL[dtype] * (1 if dtype == "float32" else 2)      # a sharp softmax: rounding of scores counts more
    assert float(off[-1]) > 3 * tol and float(off[-45]) > 3 * tol
    folder = dz.write(str(tmp_path / "m"), config, state)
    for cut in ("whole", "decode_tail", "portions", "mixed_long"):
        schedule = CUTS[cut](reqs)
        engine = dz.make_engine(folder, dtype, page, rd.peak_tokens(schedule, page), poison=True)
        dz.compare(run_engine(engine, reqs, schedule), want, tol, f"far key, {cut} [{dtype}]")
        assert engine.cache.free_pages() == engine.cache.total_pages()


# ------------------------------------------------- long prompts at sizes between tiny and real
LONG = dz.model(640, 256, [
    dz.layer(4, 64, 32, 96, 192, dz.moe(12, 3, 128, identity=4, shared=192), base=40000.0),
    dz.layer(8, 32, 16, 64, 80, dz.moe(6, 2, 96, identity=1, shared=128), base=1e6),
    dz.layer(20, 16, 16, 16, 256),
], eps=1e-5, mult=0.6, cap=4.0, loop=(0, 2, 2))


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_long_prompts(tmp_path, dtype):
    """Prompts of up to 1,500 tokens (two dozen pages of 64), whole and in mixed batches whose decoded tokens
    read hundreds of keys and whose portions take both forms."""
    state = dz.random_state(LONG, 7)
    folder = dz.write(str(tmp_path / "m"), LONG, state)
    reqs = {f"r{i}": dz.tokens(11 * i + 3, n, LONG["vocab"]) for i, n in enumerate([1500, 500, 64, 65, 129])}
    for cut in ("whole", "mixed_long"):
        run_and_compare(folder, LONG, state, reqs, CUTS[cut](reqs), dtype, 64, f"long {cut}")


# --------------------------------------------------------- first tokens, long decoding
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("which", ["A", "B"])
def test_first_tokens_and_long_decoding(models, which, dtype):
    """A request that starts with a single token and is decoded one token at a time for 200 steps, beside a
    second one that joins later two tokens a step; against the whole sequences."""
    from freetoken_b200.engine import StepEntry
    config, page = dz.DZ[which], dz.PAGE[which]
    state = dz.random_state(config, dz.SEEDS[which])
    a, b = dz.tokens(5, 201, config["vocab"]), dz.tokens(6, 120, config["vocab"])
    engine = dz.make_engine(models[which], dtype, page, 2 * 256)
    reqs = {"a": a, "b": b}
    schedule = []
    for i in range(len(a)):
        entries, j = [("a", i, 1)], i - 60
        if 0 <= j < len(b) // 2:
            entries.append(("b", 2 * j, 2))
        schedule.append((entries, []))
    routing = {}
    got = run_engine(engine, reqs, schedule, routing)
    dz.compare(got, expected_for(config, state, reqs, dtype, routing), dz.TOL[dtype], f"long decoding [{dtype}]")


@pytest.mark.parametrize("which", ["B", "C", "D"])
def test_decode_steps_replayed_from_a_graph_equal_eager_ones(models, which):
    """The same tokens with and without graph replay of decode steps: the same bits."""
    from freetoken_b200.engine import Engine, EngineArgs, StepEntry
    config = dz.DZ[which]
    toks = {r: dz.tokens(90 + i, 170, config["vocab"]) for i, r in enumerate("xyz")}
    outs = []
    for most in (64, 0):
        engine = Engine.from_folder(models[which], EngineArgs(dtype="bfloat16", page_size=dz.PAGE[which], max_tokens=3 * 256,
                                                              cuda_graph_max_bs=most))
        rows = []
        engine.step([StepEntry(r, t[:100], []) for r, t in toks.items()])
        for i in range(100, 170):
            rows.append(engine.step([StepEntry(r, [t[i]], [0]) for r, t in toks.items()]).clone())
        engine.check_status()
        assert (engine.graph_replays > 40) == (most > 0)
        outs.append(torch.stack(rows))
    assert torch.equal(outs[0], outs[1])


# ------------------------------------------------------------------------ generation
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("which", ["A", "B", "C"])
def test_greedy_generation_through_the_scheduler(models, which, dtype):
    """``LLM.generate`` (scheduler, overlapped steps, graph replay of decode steps in bfloat16): every
    generated token is the plain model's own greedy choice for the sequence so far, unless its two best
    logits - or two choice scores of a router somewhere in the sequence - lie within rounding of each other."""
    from freetoken_b200 import LLM, SamplingParams
    config = dz.DZ[which]
    state = dz.random_state(config, dz.SEEDS[which])
    llm = LLM(models[which], dtype, page_size=dz.PAGE[which], num_token_override=1024, max_running_req=3,
              max_extend_tokens=80)
    prompts = [dz.tokens(70 + i, n, config["vocab"]) for i, n in enumerate((3, 90, 11, 1, 67))]
    out = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True))
    tie = 1e-4 if dtype == "float32" else 8e-2
    route_tie = 2e-2
    ties = 0
    for prompt, result in zip(prompts, out):
        seq = list(prompt)
        assert len(result["token_ids"]) == 10
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
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_trace_replay_tool(models, tmp_path, dtype):
    """``bin/trace_run`` on a Dizatar folder: a mixed schedule with exactly the pages its peak needs."""
    which = "D"
    reqs = requests_of(which)
    state = dz.random_state(dz.DZ[which], dz.SEEDS[which])
    schedule = rd.mixed(reqs)
    page = dz.PAGE[which]
    got = rd.run_trace_tool(models[which], dtype, reqs, schedule, str(tmp_path / "out"),
                            rd.peak_tokens(schedule, page), page, dz.DZ[which]["vocab"])
    dz.compare(got, expected_for(dz.DZ[which], state, reqs, "float32"), dz.TOL[dtype] * (1 if dtype == "float32" else 4),
               "trace_run, mixed")
