"""The Tabatar design on the GPU against its plain restatement (tests/plain_tabatar.py): every mechanism alone (the streams,
attention, the memory chunk by chunk and token by token, the choice of experts, the ungated feed-forward, the capped logits),
then whole models of several shapes through the engine: prompts, token-by-token decoding (graphs included), prompts cut into
portions, unequal batches, slots and blocks that are used again, long decoding, greedy generation, the trace program and the
command line."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tabatar as pt
import tabatar_models as tm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}


def _weights(which, mild):
    """Sharp weights for the float32 comparisons (peaked attention rows, saturated gates, strong decays), mild ones for
    bfloat16, where 16-bit rounding of large scores would itself move the softmax by several percent."""
    i = list(tm.CONFIGS).index(which)
    return tm.tensors(tm.CONFIGS[which], seed=31 + i, rank=tm.RANKS[which], std=0.04, wide=1.5) if mild else \
        tm.tensors(tm.CONFIGS[which], seed=11 + i, rank=tm.RANKS[which])


def K(which, dtype):
    return which + ("_mild" if dtype == "bf16" else "")


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("tabatar")
    out = {}
    for which, cfg in tm.CONFIGS.items():
        for mild in (False, True):
            name = which + ("_mild" if mild else "")
            out[name] = tm.write_folder(str(root / name), cfg, _weights(which, mild))
    return out


class Oracle:
    def __init__(self, cfg, weights):
        self.cfg, self.weights, self._memo = cfg, weights, {}

    def logits(self, ids):
        key = tuple(ids)
        if key not in self._memo:
            self._memo[key] = pt.logits(self.cfg, self.weights, ids)
        return self._memo[key]

    def moved_by_rounding(self, ids):
        """Per position, how far 32-bit arithmetic moves the plain implementation's own logits."""
        key = ("moved",) + tuple(ids)
        if key not in self._memo:
            single = pt.logits(self.cfg, self.weights, ids, dtype=torch.float32).double()
            self._memo[key] = (single - self.logits(ids)).abs().max(-1).values
        return self._memo[key]


@pytest.fixture(scope="module")
def oracles():
    return {which + ("_mild" if mild else ""): Oracle(cfg, _weights(which, mild))
            for which, cfg in tm.CONFIGS.items() for mild in (False, True)}


_models = {}


def model_of(folders, which, dtype):
    from fms_b200.models import get_model

    key = (which, dtype)
    if key not in _models:
        _models[key] = get_model("hf_pretrained", model_path=folders[K(which, dtype)], device_type="cuda", data_type=dtype)
    return _models[key]


def close(got, want, dtype, loose=1.0, keep=None):
    want = want.to(torch.float64)
    got = got.detach().cpu().to(torch.float64)
    assert got.shape == want.shape and torch.isfinite(got).all()
    if keep is not None:
        got, want = got[keep], want[keep]
    top = want.abs().max().item() if want.numel() else 1.0
    if dtype == "fp32":
        torch.testing.assert_close(got, want, atol=3e-5 * loose * max(1.0, top), rtol=1e-4 * loose)
    else:
        torch.testing.assert_close(got, want, atol=0.03 * loose * top, rtol=0.03 * loose)


def close_logits(got, oracle, ids, dtype, rows=None):
    """float32: as sharp as for a mechanism alone; where that fails, a position is allowed four times what 32-bit rounding does
    to the plain implementation itself there (a normed read-out that nearly cancels brings its rounding back at full
    size in any 32-bit implementation).  bfloat16: by rows, the root mean square of the difference over the vocabulary against
    the logits' spread; a choice of experts that 16-bit rounding of the layers before decides otherwise moves a row by
    more, so one row in twelve may lie beyond the bound, none beyond six times it."""
    want = oracle.logits(ids)
    want = want if rows is None else want[rows]
    if dtype == "fp32":
        try:
            close(got, want, dtype)
        except AssertionError:
            moved = oracle.moved_by_rounding(ids)
            moved = moved if rows is None else moved[rows]
            diff = (got.detach().cpu().double() - want.double()).abs()
            bound = 3e-5 * max(1.0, want.abs().max().item()) + 1e-4 * want.abs() + 4.0 * moved[:, None]
            assert got.shape == want.shape and bool((diff <= bound).all()), f"{int((diff > bound).sum())} values differ, by up to {diff.max():.3g}"
        return
    got = got.detach().cpu().double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    diff = got - want
    e = (diff - diff.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / oracle.logits(ids).std()
    assert int((e > 0.06).sum()) <= max(1, len(e) // 12) and float(e.max()) < 0.36 and float(e.median()) < 0.03, \
        f"{int((e > 0.06).sum())} of {len(e)} rows, median {e.median():.3g}, worst {e.max():.3g}"


def part_with(part, tensors, dtype):
    for q, owner, local, decl in part.named_decls():
        owner.set_tensor(local, tensors[q].to(device="cuda", dtype=dtype).contiguous())
    part.finalize(torch.device("cuda"), dtype)
    return part


def step_through(mixer, x, cuts, dtype, lanes=1, room=1280):
    """Runs x [n, dim] through a mixer as ``lanes`` equal sequences side by side, each cut into steps of the given sizes;
    returns the first sequence's rows (the others must equal them)."""
    from fms_b200.cache import Cache
    from fms_b200.engine.batch import Batch

    cache = Cache([mixer.cache_request()], max_tokens=room * lanes, max_positions=room, dtype=dtype, device="cuda")
    slots = cache.begin(lanes)
    out, at = [], 0
    for n in cuts:
        before = cache.prepare(slots, [n] * lanes)
        batch = Batch.from_lists(slots, before, [[0] * n] * lanes, [[]] * lanes, "cuda")
        piece = x[at:at + n].contiguous()
        y = mixer.forward(piece.repeat(lanes, 1) if lanes > 1 else piece, batch, cache.layer_view(0), True)
        for lane in range(1, lanes):
            assert torch.equal(y[:n], y[lane * n:(lane + 1) * n])
        out.append(y[:n])
        cache.commit(slots, [n] * lanes)
        at += n
    assert at == x.shape[0]
    from fms_b200.kernels import ops
    ops.check_error_flag("cuda")
    return torch.cat(out)


def pad_rows(t, rows):
    return torch.cat([t, torch.zeros(rows - t.shape[0], t.shape[1], dtype=t.dtype)]) if rows > t.shape[0] else t


# ---- mechanisms alone ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("dim", [5, 36, 256, 1000, 4096, 5000])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 9])
def test_streams_alone(dtype, dim, streams):
    """From the embedding's rows through three sublayers and the last sum: what a sublayer reads, what becomes of every
    stream (all from the old ones), the rows gathered for the head; more rows than multiprocessors and few."""
    from fms_b200.config import NormSpec
    from fms_b200.parts import build_norm
    from fms_b200.parts.streams import HyperConnection, StreamMix, StreamSet

    dt = DTYPES[dtype]
    for n in (7, 300):
        g = torch.Generator().manual_seed(dim + streams)
        start = torch.randn(n, dim, generator=g) * 2
        norm = part_with(build_norm(NormSpec("rmsnorm", dim, 1e-2)), {"weight": (0.5 + torch.rand(dim, generator=g)).bfloat16()}, dt)
        gain = norm.tensor("weight").double().cpu()
        hcs, outs = [], []
        for _ in range(3):
            w = {"in": torch.randn(streams, generator=g), "out": torch.randn(streams, generator=g), "mix": torch.randn(streams, streams, generator=g) * streams ** -0.5}
            w = {k: v.bfloat16() for k, v in w.items()}
            hcs.append((part_with(HyperConnection(streams), w, dt), {k: v.double() for k, v in w.items()}))
            outs.append(torch.randn(n, dim, generator=g).to(dt))
        X = torch.stack([start.double()] * streams)
        have, pending = StreamSet(start.cuda(), streams), None
        for (hc, w), y in zip(hcs, outs):
            h = norm.apply_mixed(have, pending, hc.w_in, dt)
            close(h, pt.rms(pt.mixed_in(X, w["in"]), 1e-2) * gain, dtype)
            X = pt.mixed_on(X, w["mix"], w["out"], y.double())
            pending = StreamMix(y.cuda(), hc)
        before = have.rows.clone()
        rows = torch.tensor([n - 1, 0, 2], dtype=torch.int32).cuda()
        last = pt.rms(X.sum(0), 1e-2) * gain
        close(norm.apply(have, pending, dt, rows=rows), last[[n - 1, 0, 2]], dtype)
        assert torch.equal(have.rows, before)  # with rows the streams stay as they are
        close(norm.apply(have, pending, dt), last, dtype)
        close(have.rows.transpose(0, 1), X, "fp32")


def attention_tensors(g, dim_in, m, std=0.3):
    h, kv, k, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mk = lambda *s, sd=std: (torch.randn(*s, generator=g) * sd).to(torch.bfloat16)
    gain = lambda: (0.4 + 2.0 * torch.rand(k, generator=g)).to(torch.bfloat16)
    return {"q": mk(h * k, dim_in), "k": mk(kv * k, dim_in), "v": mk(kv * v, dim_in), "q.norm": gain(), "k.norm": gain(),
            "g": mk(h * v, dim_in), "o": mk(dim_in, h * v)}


def mixer_of(layer, dim_in, w, eps, dt, rank=0):
    """The framework's mixer as a model of this design builds it."""
    from fms_b200.models.tabatar import Tabatar, TabatarConfig
    from fms_b200.parts import build_mixer
    from fms_b200.parts.linear_attention import GatedLinearAttention

    layer = json.loads(json.dumps(layer))
    if layer["type"] == "gla":
        layer["mixer"]["rank"] = rank
    spec = Tabatar(TabatarConfig(width=dim_in, norm_eps=eps, layers=[layer]))._mixer_spec(layer)
    if layer["type"] == "attention":
        return part_with(build_mixer(spec), {"in_proj.weight": torch.cat([w[n] for n in "qkvg"]), "q_norm": w["q.norm"],
                                             "k_norm": w["k.norm"], "dense.weight": w["o"]}, dt)
    m = layer["mixer"]
    rows = GatedLinearAttention.fused_rows(m["heads"], m["dim"], m["vdim"], rank)
    return part_with(build_mixer(spec), {"in_proj.weight": pad_rows(torch.cat([w[n] for n in ("q", "k", "v", "g", "a1")]), rows),
                                         "norm": w["norm"], "dense.weight": w["o"], "decay_out.weight": w["a2"],
                                         "decay_out.bias": w["a2.b"]}, dt)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("shape", [(4, 2, 16, 16, 70, 16, None), (6, 1, 24, 40, 0, 8, 3.0), (2, 2, 10, 6, 65, 10, None), (3, 3, 64, 64, 200, 64, 4.0),
                                   (8, 2, 128, 128, 300, 128, 8.0), (5, 5, 6, 20, 1, 0, None), (2, 1, 250, 100, 64, 100, None),
                                   (4, 1, 32, 32, 0, 32, 2.0), (2, 1, 256, 256, 129, 256, None)])
def test_attention_alone(dtype, shape):
    heads, kv, dim, vdim, window, rot, factor = shape
    layer = tm.attention(heads, kv, dim, vdim, (0.25 if dtype == "bf16" else 0.6) * 3 / dim, window,
                         tm.rotation(rot, 300.0, factor, 1.0, 4.0, 32) if rot else None, None)
    dt, dim_in, n = DTYPES[dtype], 40, 700
    g = torch.Generator().manual_seed(sum(int(x or 0) for x in shape))
    w = attention_tensors(g, dim_in, layer["mixer"])
    mixer = mixer_of(layer, dim_in, w, 1e-5, dt)
    x = torch.randn(n, dim_in, generator=g).to(dt)
    want = pt.attention(x.double(), layer["mixer"], 1e-5, {k: v.double() for k, v in w.items()}, "")
    # whole; portions whose edges fall on and beside the cache's blocks of 64; the last rows one by one (the decode kernels,
    # over the edges of their splits of 256 keys)
    for cuts in ([n], [63, 1, 1, 63, 2, 128, 442], [600] + [1] * 100, [250] + [1] * 12 + [438]):
        close(step_through(mixer, x.cuda(), cuts, dt), want, dtype)
    close(step_through(mixer, x[:260].cuda(), [257, 2, 1], dt, lanes=3), want[:260], dtype)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("dim", [16, 64, 128])
def test_one_key_just_inside_and_just_outside_a_window(dtype, dim):
    """Inputs made so that a fault shows: the query of every ninth row is ONE earlier row's key (without rotation), so that its
    score stands out among more than a hundred, for rows whose marked key is the last one the window keeps and for rows
    whose marked key is the first it has dropped; in prompts, in portions, and when decoding."""
    window, n, heads = 130, 560, 2
    layer = tm.attention(heads, 1, dim, dim, 9.0 / dim, window, None, None)
    m, dt = layer["mixer"], DTYPES[dtype]
    g = torch.Generator().manual_seed(78 + dim)
    # the input's first half makes queries and its second keys and values, through the same matrix
    a = (torch.randn(dim, 24, generator=g) * 0.3).bfloat16()
    zero = torch.zeros_like(a)
    w = attention_tensors(g, 48, m)
    w.update({"q": torch.cat([torch.cat([a, zero], 1)] * heads), "k": torch.cat([zero, a], 1), "q.norm": torch.ones(dim).bfloat16(),
              "k.norm": torch.ones(dim).bfloat16()})
    x = torch.randn(n, 48, generator=g)
    inside, outside = [], []
    for t in range(140, n, 9):
        back = window - 1 if (t // 9) % 2 else window
        x[t, :24] = x[t - back, 24:]
        (inside if back == window - 1 else outside).append(t)
    x = x.to(dt)
    d = {k: v.double() for k, v in w.items()}
    run = lambda size: pt.attention(x.double(), dict(m, mask={"size": size}), 1e-6, d, "")
    want = run(window)
    # the oracle itself says that the edge matters: one position more or less and the marked rows come out otherwise
    assert (want[outside] - run(window + 1)[outside]).abs().max() > 0.2 * want.abs().max()
    assert (want[inside] - run(window - 1)[inside]).abs().max() > 0.2 * want.abs().max()
    mixer = mixer_of(layer, 48, w, 1e-6, dt)
    for cuts in ([n], [129, 1, 1, 129, 2, 128, 170], [135] + [1] * 425, [2] * 280):
        close(step_through(mixer, x.cuda(), cuts, dt), want, dtype)


def test_a_key_far_back_and_the_first_tokens():
    """Every seventh row asks for ONE row 290 and more positions back through rotated queries and keys: its score is the
    largest by far only if both were turned by their own positions; and sequences of one and two tokens."""
    dim, n = 32, 600
    layer = tm.attention(2, 1, dim, dim, 0.4, 0, tm.rotation(4, 100000.0, 8.0, 1.0, 4.0, 64), None)
    g = torch.Generator().manual_seed(5)
    a = (torch.randn(dim, 24, generator=g) * 0.3).bfloat16()
    zero = torch.zeros_like(a)
    w = attention_tensors(g, 48, layer["mixer"])
    w.update({"q": torch.cat([torch.cat([a, zero], 1)] * 2), "k": torch.cat([zero, a], 1)})
    x = torch.randn(n, 48, generator=g)
    for t in range(300, n, 7):
        x[t, :24] = x[t - 290 - (t % 10), 24:]
    d = {k: v.double() for k, v in w.items()}
    want = pt.attention(x.double(), layer["mixer"], 1e-6, d, "")
    near = pt.attention(x.double()[200:], layer["mixer"], 1e-6, d, "", first=200)
    assert (want[300:] - near[100:]).abs().max() > 0.2 * want.abs().max()
    mixer = mixer_of(layer, 48, w, 1e-6, torch.float32)
    for cuts in ([n], [520] + [1] * 80, [2] * 300):
        close(step_through(mixer, x.cuda(), cuts, torch.float32), want, "fp32")
    for t in (0, 1):
        close(step_through(mixer, x[:t + 1].cuda(), [t + 1], torch.float32), want[:t + 1], "fp32")


def gla_tensors(g, dim_in, m, rank, centre=2.0, spread=4.0, std=0.3):
    h, k, v = m["heads"], m["dim"], m["vdim"]
    mk = lambda *s, sd=std: (torch.randn(*s, generator=g) * sd).to(torch.bfloat16)
    return {"q": mk(h * k, dim_in), "k": mk(h * k, dim_in), "v": mk(h * v, dim_in), "g": mk(h * v, dim_in), "o": mk(dim_in, h * v),
            "norm": (0.5 + torch.rand(v, generator=g)).to(torch.bfloat16), "a1": mk(rank, dim_in), "a2": mk(h * k, rank),
            "a2.b": (centre + spread * (2 * torch.rand(h * k, generator=g) - 1)).to(torch.bfloat16)}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("shape", [(2, 24, 56, 5), (3, 12, 20, 16), (1, 40, 8, 3), (5, 6, 7, 8), (2, 96, 40, 16), (2, 128, 64, 24), (1, 256, 24, 1),
                                   (4, 64, 128, 16), (1, 33, 33, 12), (2, 32, 16, 4), (1, 128, 200, 40)])
def test_gated_linear_attention_alone(dtype, shape):
    """Decays of every kind: hardly any, around a half, and ones so strong that a product over a chunk is far below the smallest
    number (tau 1 with logits of -60: what a form that divides by them would turn into infinities)."""
    heads, dim, vdim, rank = shape
    dt, dim_in, n = DTYPES[dtype], 40, 331
    for tau, centre, spread in ((16.0, 2.0, 4.0), (1.0, -10.0, 50.0), (4.0, 9.0, 3.0)):
        layer = tm.gla(heads, dim, vdim, tau, None)
        g = torch.Generator().manual_seed(sum(shape) + int(tau))
        w = gla_tensors(g, dim_in, layer["mixer"], rank, centre, spread)
        mixer = mixer_of(layer, dim_in, w, 1e-4, dt, rank)
        x = torch.randn(n, dim_in, generator=g).to(dt)
        want = pt.gla(x.double(), layer["mixer"], 1e-4, {k: v.double() for k, v in w.items()}, "")
        # whole (in chunks of tokens); portions that run in chunks beside ones that run token by token, with edges on and beside
        # both kinds' runs of sixteen; a prompt and then row by row
        for cuts in ([n], [1, 2, 15, 16, 17, 1, 33, 246], [32, 47, 48, 49, 31, 124], [250] + [1] * 81):
            close(step_through(mixer, x.cuda(), cuts, dt), want, dtype, loose=2.0)
    close(step_through(mixer, x.cuda(), [2, 329], dt, lanes=3), want, dtype, loose=2.0)
    close(step_through(mixer, x[:60].cuda(), [2] * 30, dt), want[:60], dtype, loose=2.0)


def test_the_memory_keeps_the_first_tokens_for_a_thousand_steps():
    """Decays so near to one that what the first tokens wrote is still read 1,100 tokens later (the oracle without the first
    200 tokens gives another result), in a prompt, in portions and token by token."""
    dim_in, n = 24, 1100
    g = torch.Generator().manual_seed(9)
    x = torch.randn(n, dim_in, generator=g)
    x[:200] *= 3.0
    layer = tm.gla(3, 16, 24, 16.0, None)
    w = gla_tensors(g, dim_in, layer["mixer"], 4, centre=7.0, spread=0.5)
    w["a2"] = w["a2"] * 0.1
    d = {k: v.double() for k, v in w.items()}
    want = pt.gla(x.double(), layer["mixer"], 1e-5, d, "")
    late = pt.gla(x.double()[200:], layer["mixer"], 1e-5, d, "")
    assert (want[1000:] - late[800:]).abs().max() > 0.1 * want[1000:].abs().max()
    mixer = mixer_of(layer, dim_in, w, 1e-5, torch.float32, 4)
    for cuts in ([n], [1000] + [1] * 100, [7] * 100 + [400]):
        close(step_through(mixer, x.cuda(), cuts, torch.float32), want, "fp32", loose=3.0)


def test_the_memory_of_unequal_sequences_in_one_step():
    """Sequences of 1, 16, 17, 33 and 70 rows side by side, twice in a row: every one equals itself alone, and a slot that no
    sequence of the step holds stays as it was."""
    from fms_b200.cache import Cache
    from fms_b200.engine.batch import Batch

    layer = tm.gla(2, 32, 40, 8.0, None)
    g = torch.Generator().manual_seed(3)
    w = gla_tensors(g, 24, layer["mixer"], 6)
    mixer = mixer_of(layer, 24, w, 1e-5, torch.float32, 6)
    lengths = [1, 16, 17, 33, 70]
    cache = Cache([mixer.cache_request()], max_tokens=1280, max_positions=1280, dtype=torch.float32, device="cuda", max_slots=6)
    slots = cache.begin(6)
    cache.layer_view(0).state[slots[5]].fill_(7.0)
    xs = [torch.randn(2 * n, 24, generator=g) for n in lengths]
    got = [[] for _ in xs]
    for part in range(2):
        before = cache.prepare(slots[:5], lengths)
        batch = Batch.from_lists(slots[:5], before, [[0] * n for n in lengths], [[]] * 5, "cuda")
        y = mixer.forward(torch.cat([x[part * n:(part + 1) * n] for x, n in zip(xs, lengths)]).cuda(), batch, cache.layer_view(0), True)
        cache.commit(slots[:5], lengths)
        for i, piece in enumerate(torch.split(y, lengths)):
            got[i].append(piece)
    for x, rows in zip(xs, got):
        close(torch.cat(rows), pt.gla(x.double(), layer["mixer"], 1e-5, {k: v.double() for k, v in w.items()}, ""), "fp32", loose=2.0)
    assert bool((cache.layer_view(0).state[slots[5]] == 7.0).all())


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("shape", [(40, 5, 2, 12, 0, 1), (64, 8, 3, 24, 40, 1), (64, 8, 8, 24, 16, 8), (36, 6, 1, 10, 7, 9), (64, 16, 4, 32, 24, 40),
                                   (128, 12, 3, 48, 64, 70), (64, 7, 2, 40, 24, 300)])
def test_experts_alone(dtype, shape):
    """Routing by logits with a bias of their own size, weights from the chosen alone (one expert: weight one), a shared unit
    with its gate; few rows (the router's product in the routing kernel) and many (the library's)."""
    from fms_b200.config import FeedForwardSpec
    from fms_b200.parts import build_feed_forward
    from fms_b200.parts.experts import RoutedExperts

    dim, experts, top, ff, shared, rows = shape
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(sum(shape))
    mk = lambda *s, sd=0.2: (torch.randn(*s, generator=g) * sd).bfloat16()
    w = {"router": mk(experts, dim, sd=0.3), "router.b": torch.randn(experts, generator=g).bfloat16(), "shared.sg": mk(1, dim)}
    for e, f in [(f"e{j}", ff) for j in range(experts)] + ([("shared", shared)] if shared else []):
        w.update({e + ".gate": mk(f, dim), e + ".up": mk(f, dim), e + ".down": mk(dim, f)})
    x = torch.randn(rows, dim, generator=g).to(dt)
    mlp = tm.moe(experts, top, ff, shared)
    spec = FeedForwardSpec("routed_experts", dim=dim, hidden=ff, options=(
        ("experts", experts), ("top", top), ("scoring", "softmax_chosen"), ("router_bias", True), ("unit", "silu"),
        ("shared", FeedForwardSpec("glu", dim=dim, hidden=shared) if shared else None), ("shared_gate", bool(shared))))
    router = torch.cat([w["router"]] + ([w["shared.sg"]] if shared else []))
    tensors = {"router.weight": pad_rows(router, RoutedExperts.router_rows(experts, bool(shared))), "router_bias": w["router.b"],
               "gate_up": torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)]),
               "down": torch.stack([w[f"e{e}.down"] for e in range(experts)])}
    if shared:
        tensors.update({"shared.wg1_fused.weight": torch.cat([w["shared.gate"], w["shared.up"]]), "shared.w2.weight": w["shared.down"]})
    part = part_with(build_feed_forward(spec), tensors, dt)
    d = {k: v.double() for k, v in w.items()}
    want = pt.experts_mlp(x.double(), mlp, d, "")
    z = (x.double() @ d["router"].T + d["router.b"]).sort(-1, descending=True).values
    keep = (z[:, top - 1] - z[:, top] > 1e-3) if top < experts else torch.ones(rows, dtype=torch.bool)  # no close call
    close(part.forward(x.cuda()), want, dtype, loose=2, keep=keep)
    # the weights are those of the chosen: with a softmax over all of them the result would be another
    if 1 < top < experts and rows >= 8:
        p = torch.softmax(x.double() @ d["router"].T + d["router.b"], -1).topk(top).values.sum(-1)
        assert float((1 - p).abs().max()) > 0.05
    if keep[0]:  # a row's result does not depend on the other rows of the step
        close(part.forward(x[:1].cuda()), want[:1], dtype, loose=2)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("act", ["gelu-tanh", "silu", "relu", "gelu", "relu_squared"])
def test_ungated_feed_forward_alone(dtype, act):
    """Every number of rows for which another kernel makes the first product: 1 and 8 (weight-streaming), 9 and 300 (the library's
    and the activation after it), 512 (tcgen05, the activation in its epilogue)."""
    from fms_b200.config import FeedForwardSpec
    from fms_b200.parts import build_feed_forward

    dt = DTYPES[dtype]
    acts = {"gelu-tanh": pt.gelu, "silu": pt.silu, "relu": torch.relu, "relu_squared": lambda x: torch.relu(x) ** 2,
            "gelu": lambda x: 0.5 * x * (1 + torch.erf(x / math.sqrt(2)))}
    for dim, hidden in ((64, 200), (36, 22), (72, 328)):
        g = torch.Generator().manual_seed(dim)
        up, down = ((torch.randn(a, b, generator=g) * 0.2).bfloat16() for a, b in ((hidden, dim), (dim, hidden)))
        part = part_with(build_feed_forward(FeedForwardSpec("mlp", dim=dim, hidden=hidden, activation=act)), {"w1.weight": up, "w2.weight": down}, dt)
        for rows in (1, 8, 9, 300, 512):
            x = torch.randn(rows, dim, generator=g).to(dt)
            close(part.forward(x.cuda()), acts[act](x.double() @ up.double().T) @ down.double().T, dtype, loose=1.5)
    from fms_b200.kernels import ops
    ops.check_error_flag("cuda")


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("scale,cap", [(0.5, 3.0), (2.0, 0.0), (1.0, 50.0)])
def test_capped_logits_alone(dtype, scale, cap):
    from fms_b200.kernels import ops

    for rows, vocab, dim in ((1, 77, 40), (8, 20000, 64), (13, 331, 36), (70, 130, 64)):
        g = torch.Generator().manual_seed(rows)
        x, w = torch.randn(rows, dim, generator=g).to(DTYPES[dtype]), (torch.randn(vocab, dim, generator=g)).to(DTYPES[dtype])
        z = x.double() @ w.double().T * scale
        got = ops.capped_logits(x.cuda(), w.cuda(), scale, cap)
        assert got.dtype == torch.float32
        close(got, cap * torch.tanh(z / cap) if cap else z, "fp32", loose=3)


# ---- whole models -------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("which", list(tm.CONFIGS))
def test_whole_prompts_alone(folders, oracles, which, dtype):
    model = model_of(folders, which, dtype)
    engine = model.new_engine(max_tokens=1024, sampling=False)
    for i, n in enumerate((1, 2, 63, 64, 65, 300)):
        ids = tm.prompt(tm.CONFIGS[which], n, i)
        (slot,) = engine.begin(1)
        got = engine.step([slot], [ids], [list(range(n))])
        engine.release([slot])
        close_logits(got, oracles[K(which, dtype)], ids, dtype)
    engine.check()
    assert engine.cache.slots.n_held == 0 and all(g.pool.n_held == 0 for g in engine.cache.groups if hasattr(g, "pool"))


@pytest.mark.parametrize("which", ["p", "r", "t"])
def test_the_sum_of_the_streams_after_every_run(folders, which):
    """The streams after each run of a layer, float32, against the oracle's, further runs of a loop included.  The engine keeps
    a layer's last output pending for the kernel that mixes it in; here it is mixed in with the checkpoint's own weights."""
    cfg, weights = tm.CONFIGS[which], _weights(which, False)
    model = model_of(folders, which, "fp32")
    ids = tm.prompt(cfg, 90, 7)
    want, got = [], []
    pt.logits(cfg, weights, ids, layers_out=want)
    blocks = list({id(b): b for b in model.decoder.blocks}.values())
    originals = {id(b): b.forward for b in blocks}
    runs = iter(pt.order(cfg))

    def recording(block):
        def forward(residual, pending, batch, view, writes_cache, dtype):
            i = next(runs)
            out = originals[id(block)](residual, pending, batch, view, writes_cache, dtype)
            q = 2 if cfg["layers"][i]["mlp"] is not None else 1
            X = residual.rows.double().cpu().transpose(0, 1) if residual.rows is not None else torch.stack([residual.start.double().cpu()] * cfg["streams"])
            w = [weights[f"l{i}.hc{q}.{n}"].double() for n in ("mix", "out")]
            got.append(pt.mixed_on(X, w[0], w[1], out.delta.double().cpu()).sum(0))
            return out
        return forward

    try:
        for b in blocks:
            b.forward = recording(b)
        engine = model.new_engine(max_tokens=256, sampling=False)
        (slot,) = engine.begin(1)
        engine.step([slot], [ids], [[0]])
        engine.release([slot])
    finally:
        for b in blocks:
            del b.forward
    assert len(got) == len(want) == len(pt.order(cfg))
    for have, ref in zip(got, want):
        close(have, ref, "fp32", loose=3.0)


@pytest.mark.parametrize("which,dtype", [("p", "fp32"), ("q", "fp32"), ("r", "bf16"), ("s", "fp32"), ("t", "fp32"), ("u", "bf16")])
def test_token_by_token_from_the_first_token(folders, oracles, which, dtype):
    """Decode steps from a sequence's very first token (the first plain, the second captured, the rest replayed), over the edge
    of a cache block, twice in the same slot."""
    engine = model_of(folders, which, dtype).new_engine(max_tokens=256, sampling=False)
    for rep in range(2):
        ids = tm.prompt(tm.CONFIGS[which], 70, 20 + rep)
        (slot,) = engine.begin(1)
        got = torch.cat([engine.step([slot], [[t]], [[0]]) for t in ids])
        engine.release([slot])
        close_logits(got, oracles[K(which, dtype)], ids, dtype)
    assert engine.graphs_captured >= 1
    engine.check()


@pytest.mark.parametrize("which,dtype", [("p", "fp32"), ("q", "bf16"), ("r", "fp32"), ("s", "bf16"), ("q", "fp32"), ("u", "fp32")])
def test_prompt_then_long_decoding_over_split_edges(folders, oracles, which, dtype):
    """A prompt of 250 tokens, then 290 one by one: the decode kernels go from one split of 256 keys to three, windows pass over
    decoded tokens, the memories carry their states for 290 steps."""
    engine = model_of(folders, which, dtype).new_engine(max_tokens=1024, sampling=False)
    ids = tm.prompt(tm.CONFIGS[which], 540, 31)
    (slot,) = engine.begin(1)
    got = [engine.step([slot], [ids[:250]], [list(range(250))])]
    got += [engine.step([slot], [[t]], [[0]]) for t in ids[250:]]
    engine.release([slot])
    close_logits(torch.cat(got), oracles[K(which, dtype)], ids, dtype)
    engine.check()


@pytest.mark.parametrize("which,dtype", [(w, "fp32") for w in tm.CONFIGS] + [("p", "bf16"), ("s", "bf16")])
def test_prompts_cut_into_portions(folders, oracles, which, dtype):
    engine = model_of(folders, which, dtype).new_engine(max_tokens=1024, sampling=False)
    ids = tm.prompt(tm.CONFIGS[which], 420, 41)
    for cuts in ([2, 3, 59, 1, 64, 65, 6, 220], [193, 2, 225], [1, 1, 2, 416], [2] * 40 + [340]):
        (slot,) = engine.begin(1)
        got, at = [], 0
        for n in cuts:
            got.append(engine.step([slot], [ids[at:at + n]], [list(range(n))]))
            at += n
        engine.release([slot])
        close_logits(torch.cat(got), oracles[K(which, dtype)], ids, dtype)
    engine.check()


@pytest.mark.parametrize("which,dtype", [(w, "fp32") for w in tm.CONFIGS] + [("q", "bf16"), ("s", "bf16")])
def test_unequal_batches_freed_slots_and_poisoned_blocks(folders, oracles, which, dtype):
    """Requests of unequal lengths start together and go on one token at a time while the shorter ones end; then everything
    the cache holds is filled with NaN and new requests take the freed slots and blocks.  Every request against the oracle,
    alone."""
    cfg = tm.CONFIGS[which]
    engine = model_of(folders, which, dtype).new_engine(max_tokens=64 * 12, max_slots=5, sampling=False)
    for round_ in range(2):
        lengths, extra = ((1, 70, 5, 131, 64), (3, 9, 0, 12, 12)) if round_ == 0 else ((210, 2, 33), (5, 5, 1))
        full = [tm.prompt(cfg, n + e, 50 + 10 * round_ + i) for i, (n, e) in enumerate(zip(lengths, extra))]
        slots = engine.begin(len(lengths))
        got = [[] for _ in lengths]
        first = engine.step(slots, [f[:n] for f, n in zip(full, lengths)], [list(range(n)) for n in lengths])
        for i, piece in enumerate(torch.split(first, list(lengths))):
            got[i].append(piece)
        for t in range(max(extra)):
            live = [i for i in range(len(lengths)) if t < extra[i]]
            out = engine.step([slots[i] for i in live], [[full[i][lengths[i] + t]] for i in live])
            for i, row in zip(live, out):
                got[i].append(row[None])
            engine.release([slots[i] for i in live if t + 1 == extra[i]])
        engine.release([slots[i] for i in range(len(lengths)) if extra[i] == 0])
        for i, f in enumerate(full):
            close_logits(torch.cat(got[i]), oracles[K(which, dtype)], f, dtype)
        assert engine.cache.slots.n_held == 0
        for g in engine.cache.groups:
            g.storage.fill_(float("nan") if g.storage.is_floating_point() else 12345)
    engine.check()


def test_many_sequences_in_one_decode_step_fill_rows_and_graphs(folders, oracles):
    """Eleven sequences decode together (filled up to twelve rows with rows in the spare slot), then nine of them."""
    which, cfg = "p", tm.CONFIGS["p"]
    engine = model_of(folders, which, "fp32").new_engine(max_tokens=64 * 24, sampling=False)
    full = [tm.prompt(cfg, 3 + 5 * i + 6, 70 + i) for i in range(11)]
    slots = engine.begin(11)
    engine.step(slots, [f[:-6] for f in full], [[] for _ in full])
    got = [[] for _ in full]
    for t in range(6):
        live = list(range(11)) if t < 3 else list(range(2, 11))
        out = engine.step([slots[i] for i in live], [[full[i][len(full[i]) - 6 + t]] for i in live])
        for i, row in zip(live, out):
            got[i].append(row[None])
    engine.release(slots)
    for i, f in enumerate(full):
        rows = list(range(len(f) - 6, len(f) - 6 + len(got[i])))
        close_logits(torch.cat(got[i]), oracles[which], f, "fp32", rows=rows)
    engine.check()


@pytest.mark.parametrize("seed", range(8))
def test_drawn_configurations(seed, tmp_path):
    """Configurations drawn from seeds (any layers in any order under any loop), float32: a prompt whole, and two unequal
    requests decoding together."""
    from fms_b200.models import get_model

    cfg = tm.random_config(seed)
    oracle = Oracle(cfg, tm.tensors(cfg, seed, 8, std=0.05, wide=2.0))
    model = get_model("hf_pretrained", model_path=tm.write_folder(str(tmp_path / "m"), cfg, oracle.weights), device_type="cuda", data_type="fp32")
    engine = model.new_engine(max_tokens=1024, max_slots=4, sampling=False)
    a, b = tm.prompt(cfg, 150, seed), tm.prompt(cfg, 40, seed + 1)
    (slot,) = engine.begin(1)
    close_logits(engine.step([slot], [a], [list(range(150))]), oracle, a, "fp32")
    engine.release([slot])
    slots = engine.begin(2)
    first = engine.step(slots, [a[:135], b[:25]], [list(range(135)), list(range(25))])
    ga, gb = [first[:135]], [first[135:]]
    for t in range(15):
        out = engine.step(slots, [[a[135 + t]], [b[25 + t]]])
        ga.append(out[:1]), gb.append(out[1:])
    engine.release(slots)
    close_logits(torch.cat(ga), oracle, a, "fp32"), close_logits(torch.cat(gb), oracle, b, "fp32")
    engine.check()


def test_greedy_generation_through_generate(folders, oracles):
    from fms_b200.utils.generation import generate

    which, cfg = "q", tm.CONFIGS["q"]
    prompts = [tm.prompt(cfg, n, 80 + i) for i, n in enumerate((5, 1, 40))]
    out = generate(model_of(folders, which, "fp32"), [torch.tensor(p) for p in prompts], max_new_tokens=10, do_sample=False)
    for p, o in zip(prompts, out):
        o = o.tolist()
        assert o[: len(p)] == p and len(o) == len(p) + 10
        for k in range(len(p), len(o)):  # every new token is the oracle's choice given what came before
            row = oracles[which].logits(o[:k])[-1]
            best = row.topk(2).values
            if best[0] - best[1] > 1e-3:
                assert o[k] == int(row.argmax())


def test_trace_program_replays_a_batch(folders, oracles, tmp_path):
    """Two requests whose shorter one ends first, in bfloat16 and float32, and a step in which nothing is wanted."""
    which, cfg = "p", tm.CONFIGS["p"]
    a, b = tm.prompt(cfg, 70, 90), tm.prompt(cfg, 9, 91)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:7], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[66]], "want": []}, {"id": "b", "tokens": [b[7]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[67]], "want": [0]}, {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [a[68]], "want": [0]}], "end": ["a"]}]
    for name, dtype in (("float32", "fp32"), ("bfloat16", "bf16")):
        out = tmp_path / name
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders[K(which, dtype)], "--dtype", name,
                               "--out", str(out), "--max-tokens", "79"],
                              input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        assert not os.path.exists(str(out / "1.f32"))
        read = lambda i: torch.from_numpy(np.fromfile(str(out / f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]))
        oracle = oracles[K(which, dtype)]
        close_logits(read(0)[:2], oracle, a, dtype, rows=[0, 65]), close_logits(read(0)[2:], oracle, b, dtype, rows=[4])
        close_logits(read(2)[:1], oracle, a, dtype, rows=[67]), close_logits(read(2)[1:], oracle, b, dtype, rows=[8])
        close_logits(read(3), oracle, a, dtype, rows=[68])


def test_command_line_and_sampling(folders, oracles):
    """The command line finds the design through config.json: greedy tokens equal the oracle's choices; with sampling
    (temperature, top-k) every token is among the oracle's k best given what came before."""
    from fms_b200.utils.generation import generate

    which, cfg = "s", tm.CONFIGS["s"]
    prompts = [tm.prompt(cfg, n, 95 + i) for i, n in enumerate((4, 9))]
    args = [sys.executable, os.path.join(ROOT, "bin", "fms_inference"), "--architecture", "hf_pretrained", "--model_path", folders[which],
            "--default_dtype", "fp32", "--batch_input", "--max_new_tokens", "6", "--deterministic"]
    for p in prompts:
        args += ["--prompt_ids", ",".join(str(t) for t in p)]
    proc = subprocess.run(args, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [[int(x) for x in l.split(",")] for l in proc.stdout.splitlines() if l.strip()]
    assert len(lines) == 2
    for p, o in zip(prompts, lines):
        assert o[: len(p)] == p and len(o) == len(p) + 6
        for k in range(len(p), len(o)):
            row = oracles[which].logits(o[:k])[-1]
            best = row.topk(2).values
            if best[0] - best[1] > 1e-3:
                assert o[k] == int(row.argmax())
    out = generate(model_of(folders, which, "fp32"), [torch.tensor(p) for p in prompts], max_new_tokens=8, do_sample=True,
                   temperature=0.8, top_k=3, seed=5)
    for p, o in zip(prompts, out):
        o = o.tolist()
        for k in range(len(p), len(o)):
            row = oracles[which].logits(o[:k])[-1]
            kth = row.topk(4).values
            assert row[o[k]] >= kth[2] - 1e-4 or kth[2] - kth[3] < 1e-3
