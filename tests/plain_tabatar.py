"""A plain, slow restatement of the Tabatar design: whole sequences, no cache, no batching, one function per mechanism,
float64 by default.  It reads a configuration (the config.json dictionary) and the checkpoint's tensors by their
checkpoint names and shares no code with the library.

    start            every one of the ``streams`` copies: X_s = embed[token] * embedding.scale
    sublayer q       u = sum_s in_s X_s;  y = f(rms(u) * w);  X_t <- sum_s mix[s, t] X_s + out_t y   (q = 1: the mixer,
                     q = 2: the feed-forward, where there is one)
    order            layers start .. stop - 1 run ``times`` times in a row, each time from an empty past of their own
    attention        q, k normed per head over dim with a weight each, then the first rot.dims values turned in halves
                     (i with i + dims / 2), frequencies stretched below a wavelength; s = q.k * scale; key j counts for
                     query i when 0 <= i - j < mask.size; softmax; out = Wo (heads * sigmoid(Wg h))
    gla              a = sigmoid(Wa2 (Wa1 h) + b)^(1 / tau) per head and key channel;  S = diag(a) S + k v^T;
                     o = S^T q / sqrt(dim); each head / its root mean square * norm; out = Wo (o * silu(Wg h))
    dense            Wdown gelu(Wup h)
    experts          z = Wr h + b; the ``top`` largest z; weights softmax over those alone; expert: Wdown (silu(Wgate h) * Wup h);
                     the weighted sum, plus a shared expert of the same form times sigmoid(Wsg h)
    output           z = head rms_final(sum_s X_s) * logit_scale;  cap * tanh(z / cap)
"""
import math

import torch


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def mixed_in(X, w_in):
    """What a sublayer reads: X [streams, n, d] -> [n, d]."""
    out = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        out = out + w_in[s] * X[s]
    return out


def mixed_on(X, mix, w_out, y):
    """The streams after a sublayer, all from the old ones; mix[s, t] leads from s to t."""
    new = []
    for t in range(X.shape[0]):
        x = w_out[t] * y
        for s in range(X.shape[0]):
            x = x + mix[s, t] * X[s]
        new.append(x)
    return torch.stack(new)


def frequencies(rot):
    dims, sc = int(rot["dims"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims)
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def turned(x, rot, first=0):
    """x [n, heads, dim], positions first, first + 1, ..."""
    dims = int((rot or {}).get("dims", 0))
    if not dims:
        return x
    a = torch.arange(first, first + x.shape[0], dtype=torch.float64)[:, None] * frequencies(rot)[None]
    c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
    u, v = x[..., : dims // 2], x[..., dims // 2: dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(n, size):
    """[n, n] bool: may query i (row) see key j (column); size 0: all earlier keys."""
    away = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (away >= 0) & (away < size) if size else away >= 0


def attention(h, m, eps, w, p, first=0):
    n = h.shape[0]
    H, D = int(m["heads"]), int(m["dim"])
    G, V = int(m.get("kv_heads", H)), int(m.get("vdim", D))
    q = turned(rms((h @ w[p + "q"].T).reshape(n, H, D), eps) * w[p + "q.norm"], m.get("rot"), first)
    k = turned(rms((h @ w[p + "k"].T).reshape(n, G, D), eps) * w[p + "k.norm"], m.get("rot"), first)
    v = (h @ w[p + "v"].T).reshape(n, G, V)
    per = H // G
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(per, dim=1)) * float(m["scale"])
    s = s.masked_fill(~visible(n, int((m.get("mask") or {}).get("size", 0)))[None], float("-inf"))
    o = torch.einsum("hij,jhv->ihv", torch.softmax(s, dim=-1), v.repeat_interleave(per, dim=1)).reshape(n, H * V)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def decays(h, m, w, p):
    """[n, heads, dim]"""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return sigmoid(z).reshape(h.shape[0], int(m["heads"]), int(m["dim"])) ** (1.0 / float(m["tau"]))


def gla(h, m, eps, w, p):
    n, H, D = h.shape[0], int(m["heads"]), int(m["dim"])
    V = int(m.get("vdim", D))
    q = (h @ w[p + "q"].T).reshape(n, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).reshape(n, H, D)
    v = (h @ w[p + "v"].T).reshape(n, H, V)
    a = decays(h, m, w, p)
    S = torch.zeros(H, D, V, dtype=h.dtype)
    o = []
    for t in range(n):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o.append((S * q[t][:, :, None]).sum(1))
    o = rms(torch.stack(o), eps) * w[p + "norm"]
    return (o.reshape(n, H * V) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense_mlp(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def gated_unit(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top):
    """A list of (experts, weights) per token."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = []
    for row in z:
        mine = sorted(range(len(row)), key=lambda e: (-float(row[e]), e))[:top]
        e = torch.exp(row[mine] - row[mine].max())
        out.append((mine, e / e.sum()))
    return out


def experts_mlp(h, mlp, w, p):
    out = torch.zeros_like(h)
    for t, (mine, weight) in enumerate(route(h, w, p, int(mlp["router"]["top"]))):
        for e, x in zip(mine, weight):
            out[t] = out[t] + x * gated_unit(h[t:t + 1], w, p + f"e{e}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * gated_unit(h, w, p + "shared.")
    return out


def order(config):
    """The layers in the order in which they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def logits(config, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [n, vocab] of one sequence.  ``layers_out``: a list that receives the sum of the streams after every layer run."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(config.get("embedding", {}).get("scale", 1.0))
    plain = not any(".hc1." in k for k in w)  # one stream, to which sublayers add
    X = torch.stack([x] * int(config.get("streams") or 1))
    for i in order(config):
        layer, p = config["layers"][i], f"l{i}."
        for q in (1, 2):
            if q == 2 and layer.get("mlp") is None:
                continue
            u = X[0] if plain else mixed_in(X, w[p + f"hc{q}.in"])
            h = rms(u, eps) * w[p + f"norm{q}"]
            if q == 1:
                y = (attention if layer["type"] == "attention" else gla)(h, layer["mixer"], eps, w, p + "mix.")
            elif layer["mlp"]["kind"] == "dense":
                y = dense_mlp(h, w, p + "mlp.")
            else:
                y = experts_mlp(h, layer["mlp"], w, p + "mlp.")
            X = X + y if plain else mixed_on(X, w[p + f"hc{q}.mix"], w[p + f"hc{q}.out"], y)
        if layers_out is not None:
            layers_out.append(X.sum(0))
    z = (rms(X.sum(0), eps) * w["final.norm"]) @ w["head"].T * float(config.get("logit_scale") or 1.0)
    cap = float(config.get("logit_softcap") or 0.0)
    return cap * torch.tanh(z / cap) if cap else z
