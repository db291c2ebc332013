"""A plain, slow implementation of the Dizatar decoder: one function per mechanism.

Everything is a loop or a dense tensor expression over one whole sequence in the working
precision of the weights handed in (the tests use float64); there is no cache, no state object
and no batching, and nothing here is shared with the engine's code.  ``cfg`` is the config.json
dictionary, ``w`` a dictionary of tensors by checkpoint name.

* block: every sublayer's output is RMS-normed, scaled element by element and by a constant before it
  joins the residual stream: ``x <- x + m * ls * rms_b(sub(rms_a(x)))``.
* ``latent_attention``: keys and values made from a normed latent, one rotated key part shared by the heads.
* ``routed_ff``: softmax-scored experts, some of which hand their input back, beside a shared expert.
* loop: a span of layers runs several times; before each pass the stream and the embedded row go
  through one matrix.
"""

import math

import torch


# ------------------------------------------------------------------ small functions
def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def silu(v):
    return v * torch.sigmoid(v)


def rotate_halves(v, base, dims, first=0):
    """``v`` ``[T, heads, dim]``: dimension i of the first ``dims`` turns with i + dims/2."""
    if dims == 0:
        return v
    i = torch.arange(dims // 2, dtype=torch.float64)
    a = torch.arange(first, first + v.shape[0], dtype=torch.float64)[:, None] * base ** (-2.0 * i / dims)[None, :]
    cos, sin = a.cos().to(v.dtype)[:, None, :], a.sin().to(v.dtype)[:, None, :]
    half = dims // 2
    x, y = v[..., :half], v[..., half:dims]
    return torch.cat([x * cos - y * sin, y * cos + x * sin, v[..., dims:]], dim=-1)


# ------------------------------------------------------------------------- mixer
def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, D, R, V, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    base = m["rot"]["base"] if R else 1.0
    k_rot = rotate_halves(down[:, rank:].reshape(T, 1, R), base, R)
    q_rot = rotate_halves(q[..., D:], base, R)
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :D], k)
              + torch.einsum("ihr,jr->hij", q_rot, k_rot[:, 0])) * m["scale"]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    scores = scores.masked_fill((j > i)[None], float("-inf"))
    out = torch.einsum("hij,jhd->ihd", torch.softmax(scores, dim=-1), v).reshape(T, H * V)
    return out @ w[p + "o"].T


# ------------------------------------------------------------------- feed-forward
def glu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose_experts(h, w, p, router, margins=None):
    """``(ids [T, top], scores [T, experts + identity])``.  ``margins`` (a list) receives, per token, by
    how much the last chosen expert's choice score beat the first one left out."""
    top = router["top"]
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    choice = s + w[p + "correction"]
    ids = choice.topk(top, dim=-1).indices
    if margins is not None:
        gap = torch.full((h.shape[0],), math.inf, dtype=h.dtype)
        if top < choice.shape[-1]:
            best = choice.topk(top + 1, dim=-1).values
            gap = best[:, top - 1] - best[:, top]
        margins.append(gap)
    return ids, s


def routed_ff(h, w, p, mlp, ids=None, margins=None):
    """``ids`` (``[T, top]``) overrides the choice; the weights are always those of the scores."""
    router = mlp["router"]
    own, s = choose_experts(h, w, p, router, margins)
    ids = own if ids is None else ids
    picked = s.gather(1, ids)
    weights = picked / (picked.sum(-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for slot in range(ids.shape[1]):
            e = int(ids[t, slot])
            y = h[t] if e >= router["experts"] else glu(h[t], w, f"{p}e{e}.")
            out[t] = out[t] + weights[t, slot] * y
    if mlp.get("shared"):
        out = out + glu(h, w, p + "shared.")
    return out


# --------------------------------------------------------------------------- model
def run_order(cfg):
    """``[(layer, starts a pass)]`` in the order of the run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)]
            + [(i, False) for i in range(b, n)])


def forward(cfg, w, tokens, expert_ids=None, trace=None, margins=None):
    """Logits ``[T, vocab]`` of one sequence.  ``expert_ids``: ``{run: ids [T, top]}`` to use instead of
    the plain choice, ``run`` counting the layer runs; ``trace``: a list that receives the residual
    after every run; ``margins``: a list that receives every routed run's choice margins."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    for run, (i, starts_pass) in enumerate(run_order(cfg)):
        layer, p = cfg["layers"][i], f"l{i}."
        if starts_pass:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T
        y = latent_attention(rms(x, eps) * w[p + "norm1"], w, p + "mix.", layer["mixer"], eps)
        x = x + m * w[p + "ls1"] * (rms(y, eps) * w[p + "norm1b"])
        if layer.get("mlp"):
            ids = None if expert_ids is None else expert_ids.get(run)
            y = routed_ff(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", layer["mlp"], ids, margins)
            x = x + m * w[p + "ls2"] * (rms(y, eps) * w[p + "norm2b"])
        if trace is not None:
            trace.append(x)
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def expected_tensors(cfg):
    """``{name: shape}`` of a checkpoint of ``cfg``."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    if cfg.get("loop"):
        out["loop.in"] = (W, 2 * W)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        for q in (1, 2) if mlp else (1,):
            out.update({f"{p}norm{q}": (W,), f"{p}norm{q}b": (W,), f"{p}ls{q}": (W,)})
        H, D, R, V, rank, x = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], p + "mix."
        out.update({x + "q": (H * (D + R), W), x + "dkv": (rank + R, W), x + "dkv.norm": (rank,),
                    x + "uk": (H * D, rank), x + "uv": (H * V, rank), x + "o": (W, H * V)})
        if not mlp:
            continue
        f, r = p + "mlp.", mlp["router"]
        outputs = r["experts"] + (r.get("identity") or 0)
        out.update({f + "router": (outputs, W), f + "correction": (outputs,)})
        experts = [(f"{f}e{e}.", mlp["expert"]["ff"]) for e in range(r["experts"])]
        if mlp.get("shared"):
            experts.append((f + "shared.", mlp["shared"]["ff"]))
        for e, ff in experts:
            out.update({e + "gate": (ff, W), e + "up": (ff, W), e + "down": (W, ff)})
    return out
