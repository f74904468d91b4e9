"""Small Bolinex configurations and random weights for the tests, written from scratch here (checkpoint names and
config.json keys as a user's folder has them).  The configurations differ from one another in everything a configuration
can say: the order of the layers and their feed-forwards (dense, experts, none), widths, heads and groups of heads (one,
some, as many as heads), key and value sizes (equal, wider, narrower, no multiples of 8), windows (one key, inside a cache
block, over its edge, larger than a decode split, different from layer to layer), caps, which layers mix their values (all,
none, all but the first, layers of other heads than the first), experts (2 to 16 in 1 to as many groups as experts), top,
the shared expert, the values at the side (none, few, no multiple of 8), the number of learned positions."""
import json
import os
import random

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared, count, keep):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "top": top},
            "shared": {"ff": shared}}


def attention(heads, kv_heads, dim, vdim, scale, cap, window, v_mix, mlp):
    return {"type": "attention", "mlp": mlp, "mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": window},
                                                       "scale": scale, "softcap": cap, "v_mix": v_mix, "vdim": vdim}}


def config(vocab, width, side, positions, layers, eps=1e-5):
    out = {"architecture": "Bolinex", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps}, "layers": layers}
    if side:
        out["token_side"] = {"dim": side}
    return out


CONFIGS = {
    # one key/value head; values narrower than keys; a window inside one cache block and one over its edge; the first layer
    # mixes no values and the second is the first that does; nine experts in three groups of which one stays; a layer
    # without feed-forward
    "p": config(97, 48, 6, 640, [attention(4, 1, 24, 8, 0.3, 5.0, 20, False, moe(9, 2, 20, 28, 3, 1)),
                                 attention(4, 1, 24, 8, 0.3, 5.0, 90, True, dense(40)),
                                 attention(4, 1, 24, 8, 0.2, 8.0, 90, True, None),
                                 attention(2, 1, 16, 8, 0.3, 5.0, 20, True, moe(9, 2, 20, 28, 3, 1))], eps=1e-4),
    # as many key/value heads as heads; values wider than keys; a window longer than a decode split; every layer mixes;
    # every expert taken, all groups kept
    "q": config(130, 64, 16, 700, [attention(2, 2, 16, 40, 0.3, 50.0, 300, True, dense(36)),
                                   attention(2, 2, 16, 40, 0.3, 50.0, 300, True, moe(4, 4, 24, 16, 2, 2)),
                                   attention(2, 2, 16, 40, 0.3, 50.0, 300, True, moe(6, 2, 24, 40, 1, 1))]),
    # no size a multiple of 8 (or of 4); groups of one expert; windows of one key and of seven; nobody mixes values
    "r": config(75, 36, 5, 600, [attention(3, 1, 10, 6, 0.5, 2.0, 7, False, moe(5, 2, 9, 7, 5, 3)),
                                 attention(6, 3, 6, 10, 0.5, 3.0, 1, False, dense(22)),
                                 attention(3, 3, 5, 7, 0.5, 2.0, 65, False, moe(2, 1, 9, 11, 1, 1))], eps=1e-6),
    # heads of 128 and of 64 (the tensor-core attention kernels in bfloat16, queries read where the projection left them);
    # the second layer mixes the values of a layer with other heads; sixteen experts in four groups of which two stay; the
    # last layer's heads differ in size
    "s": config(101, 64, 24, 1024, [attention(8, 2, 128, 128, 0.09, 30.0, 150, True, moe(16, 4, 16, 24, 4, 2)),
                                    attention(4, 4, 64, 64, 0.125, 20.0, 210, True, dense(72)),
                                    attention(8, 2, 128, 64, 0.09, 30.0, 64, False, moe(16, 4, 16, 24, 4, 2))]),
    # no side at all, more value columns in the projection than anything else, two groups, a single layer that says v_mix
    "t": config(60, 40, 0, 320, [attention(5, 1, 8, 48, 0.4, 10.0, 33, False, dense(24)),
                                 attention(5, 5, 8, 16, 0.4, 10.0, 64, True, moe(8, 3, 16, 8, 2, 1))]),
}


def random_config(seed):
    """A configuration drawn from a seed: two to five layers with sizes from small lists."""
    r = random.Random(seed)
    kv, dim = r.choice([1, 2, 3, 4]), r.choice([16, 32, 64, 128, 48, 80])
    vdim = r.choice([dim, 32, 64, 128])

    def mlp():
        kind = r.choice(["dense", "moe", "moe", None])
        if kind == "dense":
            return dense(r.choice([48, 100, 360]))
        if kind == "moe":
            count = r.choice([1, 2, 4])
            size = r.choice([2, 3, 5])
            keep = r.randint(1, count)
            return moe(count * size, r.randint(1, keep * size), r.choice([32, 88, 40]), r.choice([24, 64, 90]), count, keep)
        return None

    layers = []
    for _ in range(r.choice([2, 3, 4, 5])):
        per = r.choice([1, 2, 4])
        layers.append(attention(kv * per, kv, dim, vdim, r.choice([dim ** -0.5, 0.125]), r.choice([5.0, 25.0, 60.0]),
                                r.choice([1, 17, 64, 65, 110, 200, 1000]), r.choice([True, True, False]), mlp()))
    return config(r.choice([77, 200, 450, 513]), r.choice([64, 96, 192, 320]), r.choice([4, 8, 32, 20]), r.choice([200, 333]), layers,
                  eps=r.choice([1e-5, 1e-6]))


def tensors(cfg, seed, std=0.08):
    """Matrices ~ N(0, std) with the projections of queries, keys and gates four times wider (a tiny model with
    N(0, 0.02) has near-uniform attention rows in which a dropped key hardly shows), norm weights around one with biases
    around zero, distances' numbers of either order of size, all rounded to bfloat16 as a checkpoint stores them."""
    g = torch.Generator().manual_seed(seed)
    out = {}

    def mat(name, *shape, s=std):
        out[name] = (torch.randn(*shape, generator=g) * s).to(torch.bfloat16)

    def around(name, n, centre, spread):
        out[name] = (centre + spread * (2 * torch.rand(n, generator=g) - 1)).to(torch.bfloat16)

    def gated(p, ff):
        mat(p + ".gate", ff, d, s=3 * std), mat(p + ".up", ff, d, s=3 * std), mat(p + ".down", d, ff)

    d, side = cfg["width"], int((cfg.get("token_side") or {}).get("dim", 0))
    mat("embed", cfg["vocab"], d, s=1.0), mat("pos", cfg["max_positions"], d, s=0.7)
    if side:
        mat("side.embed", cfg["vocab"], side * len(cfg["layers"]), s=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h, kv, k, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        around(p + "norm1", d, 1.0, 0.4), around(p + "norm1.b", d, 0.0, 0.4)
        mat(p + "mix.q", h * k, d, s=4 * std), mat(p + "mix.k", kv * k, d, s=4 * std), mat(p + "mix.v", kv * v, d, s=4 * std)
        mat(p + "mix.g", h * v, d, s=4 * std), mat(p + "mix.o", d, h * v)
        around(p + "mix.r1", h, 1.3, 1.2), around(p + "mix.r2", h, 0.5, 0.45)
        if m["v_mix"]:
            out[p + "mix.vmix"] = torch.tensor(0.2 + 0.5 * float(torch.rand(1, generator=g))).to(torch.bfloat16)
        mlp = layer["mlp"]
        if mlp is not None and mlp["kind"] == "dense":
            mat(p + "mlp.up", mlp["ff"], d, s=3 * std), mat(p + "mlp.down", d, mlp["ff"])
        elif mlp is not None:
            n = mlp["router"]["experts"]
            for j in range(n):
                gated(p + f"mlp.e{j}", mlp["expert"]["ff"])
            gated(p + "mlp.shared", mlp["shared"]["ff"])
            # corrections that make every choice score negative
            mat(p + "mlp.router", n, d, s=6 * std), around(p + "mlp.correction", n, -1.6, 0.5)
        if side:
            mat(p + "side.gate", side, d, s=2 * std), mat(p + "side.proj", d, side, s=4 * std), around(p + "side.norm", d, 0.5, 0.3)
    around("final.norm", d, 1.0, 0.4), around("final.norm.b", d, 0.0, 0.4)
    mat("head", cfg["vocab"], d)
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
