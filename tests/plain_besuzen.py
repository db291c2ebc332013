"""A plain, slow implementation of the Besuzen decoder: one function per mechanism.

Everything is a loop or a dense tensor expression over a whole sequence in the working precision of the
weights handed in (the tests use float64); there is no cache, no state object and no batching, and nothing
here is shared with the engine's code.  ``x`` is the residual stream ``[T, W]``, ``h`` a sublayer's input,
``W[name]`` the weights by their checkpoint names, ``c`` a mixer's or feed-forward's entry of config.json.

* layer:  ``x += mixer(ln1(x)) + ff(ln2(x))``, both norms of the same ``x``.
* ``attention``: biased projections, interleaved rotation, values mixed with the first such layer's, a gate
  per value.
* ``parallel``: ``a * gated_attention(h) + b * time_mixing(h)``.
* feed-forward: gated dense (tanh-GELU), or routed experts inside the best groups plus a gated shared expert.
"""

import math

import torch


def layer_norm(v, w, eps):
    d = v - v.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def silu(v):
    return v * torch.sigmoid(v)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(v, base, dims):
    """``v`` ``[T, heads, dim]`` at positions 0..T-1: of the first ``dims`` dimensions of each head, 2i and
    2i + 1 turn together by the angle p * base^(-2i/dims)."""
    T = v.shape[0]
    out = v.clone()
    for i in range(dims // 2):
        angle = torch.arange(T, dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
        cos, sin = angle.cos().to(v.dtype)[:, None], angle.sin().to(v.dtype)[:, None]
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = a * cos - b * sin
        out[..., 2 * i + 1] = b * cos + a * sin
    return out


def causal_softmax(q, k, v, scale):
    """``q`` ``[T, H, D]``, ``k`` ``[T, G, D]``, ``v`` ``[T, G, DV]`` -> ``[T, H, DV]``."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[2])
    seen = torch.ones(T, T, dtype=torch.bool).tril()
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * scale
        out[:, head] = torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ v[:, g]
    return out


def biased_qkv(h, p, W, c):
    T = h.shape[0]
    H, G, D, DV = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    return ((h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, D), (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, D),
            (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, DV))


def mixed_values(v, first, lam):
    """Values of a layer blended with those of the first layer that blends (``first`` None: this is it)."""
    return v if first is None else (1.0 - lam) * v + lam * first


def attention(h, p, W, c, first):
    """Returns ``(y, values)``; ``first`` holds the first value-mixing layer's values."""
    T = h.shape[0]
    q, k, v = biased_qkv(h, p, W, c)
    q = rotate_pairs(q, c["rot"]["base"], c["rot"]["dims"])
    k = rotate_pairs(k, c["rot"]["base"], c["rot"]["dims"])
    if c.get("v_mix"):
        v = mixed_values(v, first, W[p + "vmix"])
    o = causal_softmax(q, k, v, c["scale"]).reshape(T, -1)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T, v


def head_gated_attention(h, p, W, c):
    """No rotation; every head's output times one sigmoid gate."""
    T = h.shape[0]
    q, k, v = biased_qkv(h, p, W, c)
    o = causal_softmax(q, k, v, c["scale"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ W[p + "o"].T


def shifted_mix(h, mu):
    """``h_t + (h_{t-1} - h_t) mu`` with zeros before the sequence."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    return h + (before - h) * mu


def time_mixing_scan(r, k, v, w, u):
    """``r, k, w`` ``[T, H, D]``, ``v`` ``[T, H, D]``, ``u`` ``[H, D]``: per head ``o = (S + diag(u) k v^T)^T r``,
    then ``S <- diag(w) S + k v^T``."""
    T, H, D = k.shape
    out = torch.zeros_like(v)
    for head in range(H):
        S = v.new_zeros(D, v.shape[2])
        for t in range(T):
            kv = k[t, head][:, None] * v[t, head][None, :]
            out[t, head] = (S + u[head][:, None] * kv).T @ r[t, head]
            S = w[t, head][:, None] * S + kv
    return out


def time_mixing(h, p, W, c, eps, store=lambda v: v):
    T = h.shape[0]
    H, D = c["heads"], c["dim"]
    r, k, v, g = (store(store(shifted_mix(h, W[p + "mu." + n])) @ W[p + n].T) for n in "rkvg")
    low = torch.tanh(store(shifted_mix(h, W[p + "mu.w"])) @ W[p + "w1"].T)
    w = torch.exp(-torch.exp(low @ W[p + "w2"].T + W[p + "w0"]))
    o = time_mixing_scan(r.view(T, H, D), k.view(T, H, D), v.view(T, H, D), w.view(T, H, D), W[p + "u"])
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
    return (o.reshape(T, -1) * W[p + "norm"] * silu(g)) @ W[p + "o"].T


def glu(h, p, W, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose_experts(z, router, ids=None):
    """``(ids, weights, margin)`` of one token from its router logits ``z``: the best groups by their largest
    score, the best experts inside them; ``margin``: how far (in score) the choice is from another one.
    With ``ids`` those experts are taken instead."""
    s = torch.softmax(z, -1)
    E, top = router["experts"], router["top"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    count, keep = groups["count"], groups["keep"]
    per = E // count
    value = [float(s[g * per:(g + 1) * per].max()) for g in range(count)]
    order = sorted(range(count), key=lambda g: (-value[g], g))
    allowed = [e for g in sorted(order[:keep]) for e in range(g * per, (g + 1) * per)]
    ranked = sorted(allowed, key=lambda e: (-float(s[e]), e))
    margin = float("inf")
    if len(ranked) > top:
        margin = float(s[ranked[top - 1]] - s[ranked[top]])
    if keep < count:
        margin = min(margin, value[order[keep - 1]] - value[order[keep]])
    chosen = ranked[:top] if ids is None else [int(e) for e in ids]
    w = s[chosen]
    return chosen, w / (w.sum() + 1e-20), margin


def routed(h, p, W, c, ids=None, margins=None):
    z = h @ W[p + "router"].T
    out = torch.zeros_like(h)
    found = []
    for t in range(h.shape[0]):
        chosen, w, margin = choose_experts(z[t], c["router"], None if ids is None else ids[t])
        found.append(margin)
        for e, we in zip(chosen, w):
            out[t] += we * glu(h[t:t + 1], f"{p}e{e}.", W, silu)[0]
    if margins is not None:
        margins.append(torch.tensor(found))
    if c.get("shared"):
        out = out + torch.sigmoid(h @ W[p + "shared.sg"].T) * glu(h, p + "shared.", W, silu)
    return out


def forward(config, W, tokens, expert_ids=None, margins=None, layers_out=None, store=lambda v: v):
    """Logits ``[T, vocab]``.  ``store`` is applied to what an engine with 16-bit activations stores (the sublayers'
    inputs and outputs, a time mixer's mixes and projections): with a function that perturbs its argument by as
    much as such a rounding, the result shows how far rounding alone moves each position.  ``expert_ids``: ``{layer: [T, top]}``, experts to take instead of the chosen ones;
    ``margins`` (a list) takes every routed layer's margins ``[T]``, ``layers_out`` (a list) the residual stream
    after every layer."""
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"]
    first = None
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = store(layer_norm(x, W[p + "norm1"], eps))
        if layer["type"] == "attention":
            y, v = attention(h, p + "mix.", W, m, first)
            if m.get("v_mix") and first is None:
                first = v
        else:
            y = (m["left_scale"] * head_gated_attention(h, p + "mix.left.", W, m["left"])
                 + m["right_scale"] * time_mixing(h, p + "mix.right.", W, m["right"], eps, store))
        y = store(y)
        if mlp:
            g = store(layer_norm(x, W[p + "norm2"], eps))
            if mlp["kind"] == "dense":
                y = y + glu(g, p + "mlp.", W, gelu_tanh)
            else:
                y = y + routed(g, p + "mlp.", W, mlp, (expert_ids or {}).get(i), margins)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T * config["logit_scale"]


def expected_tensors(config):
    """Name -> shape of every tensor of a model of ``config`` (``mixer.right.low_rank`` filled in)."""
    width = config["width"]
    out = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}

    def linear(name, rows, cols, bias=False):
        out[name] = (rows, cols)
        if bias:
            out[name + ".b"] = (rows,)

    def gated(p, ff):
        linear(p + "gate", ff, width)
        linear(p + "up", ff, width)
        linear(p + "down", width, ff)

    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        out[p + "norm1"] = (width,)
        scopes = [("mix.", m)] if layer["type"] == "attention" else [("mix.left.", m["left"])]
        for scope, a in scopes:
            linear(p + scope + "q", a["heads"] * a["dim"], width, True)
            linear(p + scope + "k", a["kv_heads"] * a["dim"], width, True)
            linear(p + scope + "v", a["kv_heads"] * a["vdim"], width, True)
            linear(p + scope + "g", a["heads"] * (a["vdim"] if scope == "mix." else 1), width)
            linear(p + scope + "o", width, a["heads"] * a["vdim"])
        if layer["type"] == "attention":
            if m.get("v_mix"):
                out[p + "mix.vmix"] = ()
        else:
            r = p + "mix.right."
            n = m["right"]["heads"] * m["right"]["dim"]
            for name in "rkvgw":
                out[r + "mu." + name] = (width,)
            for name in "rkvg":
                linear(r + name, n, width)
            linear(r + "w1", m["right"]["low_rank"], width)
            linear(r + "w2", n, m["right"]["low_rank"])
            out[r + "w0"] = out[r + "norm"] = (n,)
            out[r + "u"] = (m["right"]["heads"], m["right"]["dim"])
            linear(r + "o", width, n)
        if mlp:
            out[p + "norm2"] = (width,)
            if mlp["kind"] == "dense":
                gated(p + "mlp.", mlp["ff"])
            else:
                linear(p + "mlp.router", mlp["router"]["experts"], width)
                for e in range(mlp["router"]["experts"]):
                    gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
                if mlp.get("shared"):
                    gated(p + "mlp.shared.", mlp["shared"]["ff"])
                    linear(p + "mlp.shared.sg", 1, width)
    return out
