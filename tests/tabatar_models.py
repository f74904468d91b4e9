"""Small Tabatar configurations and random weights for the tests, written from scratch here (checkpoint names and
config.json keys as a user's folder has them).  The configurations differ from one another in everything a configuration
can say: the order of the layers and their feed-forwards (dense, experts with and without a shared one, none), the loop
(none, one layer, all layers, twice, three times), the number of streams (one with weights of its own, two, three, four,
five), widths, heads and groups of heads, key and value sizes (equal, wider, narrower, no multiples of 8 or 4), rotated part
(all, some, none; scaled frequencies or not), windows (one key, inside a cache block, over its edge, larger than a decode
split, none), roots of the decays, ranks, experts and how many a token takes (one, all), scales and caps (none among them)."""
import json
import os
import random

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def rotation(dims, base, factor=None, low=1.0, high=4.0, original=64):
    out = {"base": base, "dims": dims}
    if factor is not None:
        out["scaling"] = {"factor": factor, "high": high, "low": low, "original": original}
    return out


def attention(heads, kv_heads, dim, vdim, scale, window, rot, mlp):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = rot
    return {"type": "attention", "mixer": m, "mlp": mlp}


def gla(heads, dim, vdim, tau, mlp):
    return {"type": "gla", "mixer": {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim}, "mlp": mlp}


def config(vocab, width, streams, layers, loop=None, eps=1e-5, embedding=1.0, logit_scale=1.0, cap=None):
    out = {"architecture": "Tabatar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
           "embedding": {"scale": embedding}, "layers": layers, "logit_scale": logit_scale}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if cap:
        out["logit_softcap"] = cap
    return out


# rank of the decays' low-rank product, by configuration (config.json does not say it)
RANKS = {"p": 8, "q": 5, "r": 3, "s": 16, "t": 4, "u": 12}

CONFIGS = {
    # three streams; one key/value head, values wider than keys, half of a head turned by scaled frequencies, a window over a
    # cache block's edge; the middle layers three times; a layer without feed-forward; experts without a shared one
    "p": config(97, 48, 3, [attention(4, 1, 16, 24, 0.4, 70, rotation(8, 500.0, 4.0), moe(5, 2, 20)),
                            gla(3, 12, 20, 4.0, dense(40)),
                            attention(4, 1, 16, 24, 0.4, 70, rotation(8, 500.0, 4.0), None),
                            gla(3, 12, 20, 4.0, moe(6, 3, 28, 36))], loop=(1, 3, 3), eps=1e-4, embedding=6.9, logit_scale=0.4, cap=8.0),
    # two streams; as many key/value heads as heads, values narrower, everything turned, a window of more than a decode split
    # and none; memories whose values are much wider than their keys; every expert taken; no loop, no cap
    "q": config(130, 64, 2, [gla(2, 16, 72, 16.0, moe(4, 4, 24, 16)),
                             attention(2, 2, 32, 16, 0.25, 300, rotation(32, 10000.0), dense(36)),
                             attention(2, 2, 32, 16, 0.25, 0, rotation(32, 10000.0), moe(3, 1, 24, 40))], embedding=8.0, logit_scale=2.0),
    # five streams (the general kernel), no size a multiple of 8 or of 4, no rotation, windows of one key and of seven, the whole
    # stack twice, decays to the first power
    "r": config(75, 38, 5, [attention(3, 1, 10, 6, 0.5, 7, None, moe(5, 2, 9, 7)), gla(3, 5, 7, 1.0, dense(22)),
                            attention(3, 3, 5, 7, 0.5, 1, rotation(2, 50.0), dense(13)), gla(2, 9, 3, 2.5, None)],
                loop=(0, 4, 2), eps=1e-6, embedding=3.0, cap=5.0),
    # heads and memories of 128 and 64 (the tensor-core attention kernels, four warps of channels), four streams, sixteen experts
    "s": config(101, 64, 4, [attention(8, 2, 128, 128, 0.09, 150, rotation(128, 500000.0, 8.0, 1.0, 4.0, 256), dense(72)),
                             gla(2, 128, 128, 16.0, moe(16, 4, 16, 24)),
                             gla(4, 64, 32, 8.0, dense(64)),
                             attention(4, 4, 64, 64, 0.125, 64, rotation(64, 10000.0), moe(16, 4, 16, 24))], loop=(1, 2, 2), eps=1e-6,
                embedding=8.0, logit_scale=0.6, cap=14.0),
    # one stream, with weights of its own; one layer, passed through four times
    "t": config(60, 40, 1, [gla(1, 40, 16, 3.0, moe(8, 3, 16, 8))], loop=(0, 1, 4), embedding=2.0, cap=30.0),
    # memories with key sizes over a warp of channels and its edges, two streams
    "u": config(83, 56, 2, [gla(2, 33, 17, 16.0, dense(24)), gla(1, 200, 40, 5.0, None), attention(5, 1, 8, 48, 0.4, 33, rotation(4, 100.0), dense(24))],
                embedding=4.0, logit_scale=0.7, cap=12.0),
}


def random_config(seed):
    """A configuration drawn from a seed: two to five layers with sizes from small lists."""
    r = random.Random(seed)
    dim, kv, window = r.choice([16, 32, 64, 128, 48]), r.choice([1, 2, 3]), r.choice([0, 1, 17, 64, 65, 110, 200])
    gdim, gheads = r.choice([16, 24, 32, 64, 100]), r.choice([1, 2, 4])

    def mlp():
        kind = r.choice(["dense", "moe", "moe", None])
        if kind == "dense":
            return dense(r.choice([48, 100, 360]))
        if kind == "moe":
            n = r.choice([2, 5, 8, 12])
            return moe(n, r.randint(1, n), r.choice([32, 88, 40]), r.choice([0, 24, 64]))
        return None

    layers = []
    for _ in range(r.choice([2, 3, 4, 5])):
        if r.random() < 0.5:
            rot = r.choice([None, rotation(r.choice([dim, dim // 2]), r.choice([100.0, 10000.0]), r.choice([None, 4.0]))])
            layers.append(attention(kv * r.choice([1, 2, 4]), kv, dim, r.choice([dim, 32, 64]), r.choice([dim ** -0.5, 0.2]), window, rot, mlp()))
        else:
            layers.append(gla(gheads, gdim, r.choice([gdim, 32, 64]), r.choice([1.0, 6.0, 16.0]), mlp()))
    n = len(layers)
    a = r.randint(0, n - 1)
    loop = r.choice([None, (a, r.randint(a + 1, n), r.choice([1, 2, 3]))])
    return config(r.choice([77, 200, 450, 513]), r.choice([64, 96, 192, 320]), r.choice([1, 2, 3, 4, 6]), layers, loop,
                  eps=r.choice([1e-5, 1e-6]), embedding=r.choice([1.0, 9.0]), logit_scale=r.choice([1.0, 0.45]), cap=r.choice([None, 11.0]))


def tensors(cfg, seed, rank=8, std=0.08, wide=4.0):
    """Matrices ~ N(0, std), the projections that decide (queries, keys, gates, routers) ``wide`` times wider (a tiny model
    with N(0, 0.02) has near-uniform attention rows in which a dropped key hardly shows), norm weights around one, mixing
    weights of every sign, decays' biases from strong to hardly any decay, all rounded to bfloat16 as a checkpoint stores them."""
    g = torch.Generator().manual_seed(seed)
    out = {}

    def mat(name, *shape, s=std):
        out[name] = (torch.randn(*shape, generator=g) * s).to(torch.bfloat16)

    def around(name, shape, centre, spread):
        out[name] = (centre + spread * (2 * torch.rand(shape, generator=g) - 1)).to(torch.bfloat16)

    def gated(p, ff):
        mat(p + ".gate", ff, d, s=2 * std), mat(p + ".up", ff, d, s=2 * std), mat(p + ".down", d, ff)

    d, S = cfg["width"], cfg["streams"]
    mat("embed", cfg["vocab"], d, s=0.5)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        h, k, v = m["heads"], m["dim"], m["vdim"]
        kv = m.get("kv_heads", h)
        for q in (1, 2) if mlp is not None else (1,):
            around(p + f"norm{q}", d, 1.0, 0.4)
            around(p + f"hc{q}.in", S, 1.0 / S, 0.5), around(p + f"hc{q}.out", S, 0.7, 0.6)
            out[p + f"hc{q}.mix"] = (0.85 * torch.eye(S) + 0.25 * (2 * torch.rand(S, S, generator=g) - 1)).to(torch.bfloat16)
        mat(p + "mix.q", h * k, d, s=wide * std), mat(p + "mix.k", kv * k, d, s=wide * std)
        mat(p + "mix.v", kv * v, d, s=2 * std), mat(p + "mix.g", h * v, d, s=wide * std), mat(p + "mix.o", d, h * v)
        if layer["type"] == "attention":
            around(p + "mix.q.norm", k, 1.2, 0.6), around(p + "mix.k.norm", k, 1.2, 0.6)
        else:
            around(p + "mix.norm", v, 1.0, 0.5)
            mat(p + "mix.a1", rank, d, s=2 * std), mat(p + "mix.a2", h * k, rank, s=wide * std)
            around(p + "mix.a2.b", h * k, 2.0, 4.0)
        if mlp is not None and mlp["kind"] == "dense":
            mat(p + "mlp.up", mlp["ff"], d, s=2 * std), mat(p + "mlp.down", d, mlp["ff"])
        elif mlp is not None:
            n = mlp["router"]["experts"]
            for j in range(n):
                gated(p + f"mlp.e{j}", mlp["expert"]["ff"])
            mat(p + "mlp.router", n, d, s=wide * std), around(p + "mlp.router.b", n, 0.0, 2.0)
            if mlp.get("shared"):
                gated(p + "mlp.shared", mlp["shared"]["ff"]), mat(p + "mlp.shared.sg", 1, d, s=2 * std)
    around("final.norm", d, 1.0, 0.4)
    mat("head", cfg["vocab"], d, s=2 * std)
    return out


def write_folder(path, cfg, weights):
    from fms_b200.weights.safetensors_io import write_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as fh:
        json.dump(cfg, fh, indent=1)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.contiguous() for k, v in weights.items()}, {})
    return path


def prompt(cfg, length, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (length,), generator=g).tolist()
