"""A plain, slow restatement of the Bolinex design: whole sequences, no cache, no batching, one function per mechanism,
float64 by default.  It reads a configuration (the config.json dictionary) and the checkpoint's tensors by their
checkpoint names and shares no code with the library.

    start            x_p = embed[token_p] + pos[p]
    norm             (x - mean x) / sqrt(mean((x - mean x)^2) + eps) * w + b
    layer            h = norm1(x); x = x + mixer(h) + mlp(h); then the token side: e = the layer's dim values of the token's
                     row of side.embed, y = Wproj (gelu(Wgate x) * e), x = x + y / sqrt(mean(y^2) + eps) * w_side
    attention        q, k, v = Wq h, Wk h, Wv h; s = q.k * scale, then cap * tanh(s / cap), then
                     s - r1_h ln(1 + r2_h (i - j)); key j counts for query i when 0 <= i - j < mask.size; softmax;
                     out = Wo (heads * sigmoid(Wg h))
    value mixing     v = (1 - a) v + a v0 where the layer says v_mix, v0 being the values of the first such layer
    dense            Wdown relu(Wup h)^2
    experts          s = sigmoid(Wr h); choice scores c = s + correction; the experts in groups.count equal groups, a
                     group's score the sum of its two largest c; only the groups.keep best groups' experts count; the
                     ``top`` largest c among them; weights s as they are; expert: Wdown (silu(Wgate h) * Wup h); the
                     weighted sum, plus a shared expert of the same form
    output           logits = head norm_final(x)
"""
import math

import torch


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scores(q, k, scale, cap, r1, r2):
    """q [n, H, D], k [n, H, D] -> [H, n, n]: capped, then with the distance taken off (entries with j > i are not used)."""
    n = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    if r1 is not None:
        away = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(min=0).to(q.dtype)
        s = s - r1[:, None, None] * torch.log(1 + r2[:, None, None] * away[None])
    return s


def visible(n, size):
    """[n, n] bool: may query i (row) see key j (column); size 0: all earlier keys."""
    away = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (away >= 0) & (away < size) if size else away >= 0


def mix_values(v, v0, a):
    return (1 - a) * v + a * v0


def attention(h, w, p, m, first_values=None):
    """Returns (output, the values as they are cached [n, G * V])."""
    n = h.shape[0]
    H, D = int(m["heads"]), int(m["dim"])
    G, V = int(m.get("kv_heads", H)), int(m.get("vdim", D))
    q = (h @ w[p + "q"].T).reshape(n, H, D)
    k = (h @ w[p + "k"].T).reshape(n, G, D)
    v = h @ w[p + "v"].T
    if m.get("v_mix") and first_values is not None:
        v = mix_values(v, first_values, w[p + "vmix"])
    per = H // G
    s = scores(q, k.repeat_interleave(per, dim=1), float(m["scale"]), float(m.get("softcap") or 0), w[p + "r1"], w[p + "r2"])
    s = s.masked_fill(~visible(n, int((m.get("mask") or {}).get("size", 0)))[None], float("-inf"))
    pr = torch.softmax(s, dim=-1)
    o = torch.einsum("hij,jhv->ihv", pr, v.reshape(n, G, V).repeat_interleave(per, dim=1)).reshape(n, H * V)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, v


def dense_mlp(h, w, p):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def gated_unit(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(choice, top, count, keep):
    """The experts of one token: indices of the ``top`` largest choice scores among the ``keep`` best of ``count`` groups."""
    c = choice.tolist()
    size = len(c) // count
    group = [sum(sorted(c[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(count)]
    kept = sorted(range(count), key=lambda g: (-group[g], g))[:keep]
    allowed = [e for e in range(len(c)) if e // size in kept]
    return sorted(allowed, key=lambda e: (-c[e], e))[:top]


def route(h, w, p, mlp):
    """(chosen experts, a list of lists; all scores [n, experts])."""
    r = mlp["router"]
    s = sigmoid(h @ w[p + "router"].T)
    g = r.get("groups") or {"count": 1, "keep": 1}
    c = s + w[p + "correction"][None]
    return [choose(row, int(r["top"]), int(g["count"]), int(g["keep"])) for row in c], s


def experts_mlp(h, w, p, mlp):
    chosen, s = route(h, w, p, mlp)
    out = torch.zeros_like(h)
    for t, mine in enumerate(chosen):
        for e in mine:
            out[t] = out[t] + s[t, e] * gated_unit(h[t:t + 1], w, p + f"e{e}.")[0]
    if mlp.get("shared"):
        out = out + gated_unit(h, w, p + "shared.")
    return out


def token_side(x, w, p, ids, i, dim, eps):
    """What a layer adds for the tokens themselves."""
    e = w["side.embed"][ids][:, i * dim:(i + 1) * dim]
    y = (gelu(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms(y, eps) * w[p + "side.norm"]


def forward(config, weights, tokens, dtype=torch.float64, streams=None, normed=None):
    """Logits [n, vocab] of one sequence.  ``streams`` / ``normed``: lists that receive the stream after every layer and
    every layer's normed input."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][ids] + w["pos"][:len(ids)]
    v0 = None
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        if normed is not None:
            normed.append(h.clone())
        y, v = attention(h, w, p + "mix.", m, v0)
        if m.get("v_mix") and v0 is None:
            v0 = v
        mlp = layer.get("mlp")
        if mlp is not None:
            y = y + (dense_mlp(h, w, p + "mlp.") if mlp["kind"] == "dense" else experts_mlp(h, w, p + "mlp.", mlp))
        x = x + y
        if config.get("token_side"):
            x = x + token_side(x, w, p, ids, i, int(config["token_side"]["dim"]), eps)
        if streams is not None:
            streams.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
