"""Tabatar on the CPU: configuration, registry, checkpoint adapter, the loop's entries in the cache, the one error for a
checkpoint that does not fit; and the plain restatement by hand (streams mixed from the old ones, stretched frequencies, a
window's edge, decays, the softmax over the chosen, the order of runs)."""
import json
import math

import pytest
import torch

import plain_tabatar as pt
import tabatar_models as tm


def test_config_json_registry_adapter_and_the_loop(tmp_path):
    from fms_b200 import models
    from fms_b200.cache.requests import KVRequest, StateRequest
    from fms_b200.models import get_model
    from fms_b200.models.tabatar import Tabatar

    assert "tabatar" in models.list_models() and "tiny" in models.list_variants("tabatar")
    cfg = tm.CONFIGS["p"]
    raw = tm.tensors(cfg, 1, tm.RANKS["p"])
    model = get_model("hf_pretrained", model_path=tm.write_folder(str(tmp_path / "p"), cfg, raw), device_type="cpu", data_type="fp32")
    assert isinstance(model, Tabatar)
    spec = model.decoder_spec()
    assert all(b.arrangement == "hyper_connected" for b in spec.layers)
    assert (spec.streams, spec.embedding_scale, spec.logit_scale, spec.logit_softcap) == (3, 6.9, 0.4, 8.0)
    # layers 1 and 2 three times: the runs in order, each with an entry of its own and the first run's weights
    assert [c.layer for c in spec.schedule] == [0, 1, 2, 4, 5, 6, 7, 3]
    assert [b.weights_of for b in spec.layers] == [None] * 4 + [1, 2, 1, 2]
    assert model.decoder.blocks[4] is model.decoder.blocks[1] and model.decoder.blocks[7] is model.decoder.blocks[2]
    r = model.decoder.cache_requests()
    assert len(r) == 8 and r[0] == KVRequest(1, 32, 70) and r[6] == StateRequest((3, 20, 12), torch.float32, "state_matrix")
    assert [b.mixer.kind for b in spec.layers[:4]] == ["sink_attention", "gla", "sink_attention", "gla"]
    assert [None if b.feed_forward is None else b.feed_forward.kind for b in spec.layers[:4]] == ["routed_experts", "mlp", None, "routed_experts"]
    sd = model.state_dict()
    f = {k: v.float() for k, v in raw.items()}
    assert torch.equal(sd["layers.0.mix.in_proj.weight"], torch.cat([f["l0.mix." + n] for n in "qkvg"]))
    fused = sd["layers.1.mix.in_proj.weight"]  # [q; k; v; g; a1], zeros up to a multiple of 8
    want = torch.cat([f["l1.mix." + n] for n in ("q", "k", "v", "g", "a1")])
    assert fused.shape[0] % 8 == 0 and torch.equal(fused[:want.shape[0]], want) and not fused[want.shape[0]:].any()
    assert torch.equal(sd["layers.1.mix.decay_out.weight"], f["l1.mix.a2"]) and torch.equal(sd["layers.1.mix.decay_out.bias"], f["l1.mix.a2.b"])
    # experts without a shared one: the router as it is; with one: its gate's row behind the experts', then zeros
    assert torch.equal(sd["layers.0.mlp.router.weight"], f["l0.mlp.router"])
    router = sd["layers.3.mlp.router.weight"]
    assert router.shape == (8, 48) and torch.equal(router[:7], torch.cat([f["l3.mlp.router"], f["l3.mlp.shared.sg"]])) and not router[7].any()
    assert torch.equal(sd["layers.3.mlp.gate_up"][4], torch.cat([f["l3.mlp.e4.gate"], f["l3.mlp.e4.up"]]))
    assert torch.equal(sd["layers.3.mlp.shared.wg1_fused.weight"], torch.cat([f["l3.mlp.shared.gate"], f["l3.mlp.shared.up"]]))
    assert torch.equal(sd["layers.1.mlp.w1.weight"], f["l1.mlp.up"]) and torch.equal(sd["layers.1.mlp.w2.weight"], f["l1.mlp.down"])
    hc = model.decoder.blocks[3].feed_forward_connection
    assert torch.equal(hc.on, torch.cat([f["l3.hc2.mix"].reshape(-1), f["l3.hc2.out"]])) and torch.equal(hc.w_in, f["l3.hc2.in"])
    again = Tabatar.config_from_json(json.loads(json.dumps(model.config_json())))
    assert again == model.config


def test_what_config_json_leaves_out(tmp_path):
    from fms_b200.models import get_model

    cfg = tm.CONFIGS["q"]
    raw = tm.tensors(cfg, 3, tm.RANKS["q"])
    lean = json.loads(json.dumps(cfg))
    del lean["embedding"], lean["logit_scale"], lean["streams"]
    lean["loop"] = None
    del lean["layers"][0]["mlp"]["expert"], lean["layers"][0]["mlp"]["router"]["experts"], lean["layers"][0]["mlp"]["shared"]["ff"]
    del lean["layers"][1]["mlp"]["ff"], lean["layers"][1]["mixer"]["kv_heads"]
    model = get_model("hf_pretrained", model_path=tm.write_folder(str(tmp_path / "q"), lean, raw), device_type="cpu", data_type="bf16")
    spec = model.decoder_spec()
    assert (spec.streams, spec.embedding_scale, spec.logit_scale, spec.logit_softcap) == (2, 1.0, 1.0, 0.0)
    assert model.decoder.blocks[0].mixer.rank == 5 and [c.layer for c in spec.schedule] == [0, 1, 2]
    assert [b.mixer.window for b in spec.layers] == [0, 300, 0]
    # one stream and no weights that mix it: sublayers add to it
    bare = json.loads(json.dumps(cfg))
    bare["streams"] = 1
    raw = {k: v for k, v in raw.items() if ".hc" not in k}
    model = get_model("hf_pretrained", model_path=tm.write_folder(str(tmp_path / "b"), bare, raw), device_type="cpu", data_type="bf16")
    assert all(b.arrangement == "pre_norm" for b in model.decoder_spec().layers) and model.decoder.spec.streams == 0


def test_a_checkpoint_that_does_not_fit_is_refused_with_one_error(tmp_path):
    from fms_b200.models import get_model
    from fms_b200.weights import WeightError

    cfg = tm.CONFIGS["s"]
    weights = tm.tensors(cfg, 2, tm.RANKS["s"])
    del weights["l0.mix.g"], weights["l1.mlp.e2.down"], weights["l2.mix.a2.b"], weights["l3.hc2.mix"], weights["l1.mlp.router.b"]
    weights["l1.hc1.in"] = weights["l1.hc1.in"][:-1]
    weights["stray"] = torch.zeros(3, dtype=torch.bfloat16)
    with pytest.raises(WeightError) as e:
        get_model("hf_pretrained", model_path=tm.write_folder(str(tmp_path / "s"), cfg, weights), device_type="cpu", data_type="fp32")
    for name in ("layers.0.mix.in_proj.weight", "layers.1.mlp.down", "layers.2.mix.decay_out.bias", "layers.3.hc2.mix", "layers.1.mlp.router_bias"):
        assert name in e.value.missing
    assert "stray" in e.value.unexpected and any(n == "layers.1.hc1.in" for n, _, _ in e.value.wrong_shapes)


def test_config_json_of_another_design_or_with_unknown_parts_is_refused():
    from fms_b200.models.tabatar import Tabatar

    with pytest.raises(ValueError):
        Tabatar.config_from_json({"architecture": "Other"})
    for change, what in ((lambda c: c["layers"][0].update(type="convolution"), "convolution"), (lambda c: c.pop("norm"), "norm"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse"), (lambda c: c["loop"].update(stop=9), "loop")):
        bad = json.loads(json.dumps(tm.CONFIGS["p"]))
        change(bad)
        with pytest.raises(ValueError, match=what):
            Tabatar.config_from_json(bad)


def test_random_weights_of_a_registered_variant():
    from fms_b200.models import get_model

    model = get_model("tabatar", "tiny", device_type="cpu", data_type="bf16")
    assert [c.layer for c in model.decoder.spec.schedule] == [0, 1, 2, 4, 5, 3] and model.decoder.spec.streams == 3
    assert model.cache_bytes_per_token() == 3 * 2 * 2 * 32 * 2  # three runs of attention layers


def test_plain_streams_are_mixed_from_the_old_ones():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=torch.float64)
    mix = torch.tensor([[2.0, 3.0], [5.0, 7.0]], dtype=torch.float64)  # [from, to]
    y = torch.tensor([[100.0, 0.0]], dtype=torch.float64)
    new = pt.mixed_on(X, mix, torch.tensor([1.0, -1.0], dtype=torch.float64), y)
    assert new[0].tolist() == [[2 * 1 + 5 * 10 + 100.0, 2 * 2 + 5 * 20.0]] and new[1].tolist() == [[3 * 1 + 7 * 10 - 100.0, 3 * 2 + 7 * 20.0]]
    assert pt.mixed_in(X, torch.tensor([0.5, -1.0], dtype=torch.float64)).tolist() == [[-9.5, -19.0]]


def test_plain_frequencies_window_and_order():
    rot = tm.rotation(8, 10.0, 4.0, 1.0, 4.0, 40)  # wavelengths 6.3, 11.2, 19.9, 35.3: kept below 10, stretched above 40
    f = pt.frequencies(rot)
    plain = [10.0 ** (-i / 4) for i in range(4)]
    assert f[0] == plain[0]
    s = (40 / (2 * math.pi / plain[2]) - 1.0) / 3.0
    assert abs(float(f[2]) - ((1 - s) * plain[2] / 4 + s * plain[2])) < 1e-15
    assert float(pt.frequencies(tm.rotation(8, 10.0, 4.0, 1.0, 4.0, 10))[3]) == plain[3] / 4
    x = torch.arange(6, dtype=torch.float64).reshape(1, 1, 6)  # position 3, the pair (0, 2) of four turned values; 4 and 5 pass
    t = pt.turned(x, tm.rotation(4, 7.0), first=3)
    assert abs(float(t[0, 0, 0]) - (0 * math.cos(3) - 2 * math.sin(3))) < 1e-12 and abs(float(t[0, 0, 2]) - (2 * math.cos(3))) < 1e-12
    assert t[0, 0, 4:].tolist() == [4.0, 5.0]
    ok = pt.visible(6, 3)
    assert ok[4].tolist() == [False, False, True, True, True, False] and pt.visible(3, 0)[2].all()
    assert pt.order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3]
    assert pt.order({"layers": [0] * 2}) == [0, 1]


def test_plain_decays_and_memory():
    m = {"heads": 1, "dim": 2, "vdim": 1, "tau": 2.0}
    e = torch.eye(2, dtype=torch.float64)
    w = {"a1": e, "a2": e, "a2.b": torch.tensor([0.0, 1.0], dtype=torch.float64), "q": e * math.sqrt(2.0), "k": e,
         "v": torch.tensor([[1.0, 1.0]], dtype=torch.float64), "g": torch.tensor([[0.0, 0.0]], dtype=torch.float64),
         "norm": torch.ones(1, dtype=torch.float64), "o": torch.ones(2, 1, dtype=torch.float64)}
    h = torch.tensor([[1.0, 0.0], [0.0, 2.0]], dtype=torch.float64)
    a = pt.decays(h, m, w, "")
    assert abs(float(a[1, 0, 0]) - math.sqrt(0.5)) < 1e-12 and abs(float(a[1, 0, 1]) - (1 / (1 + math.exp(-3.0))) ** 0.5) < 1e-12
    w["g"] = torch.tensor([[1.0, 1.0]], dtype=torch.float64)
    out = pt.gla(h, m, 3.0, w, "")  # S after token 0: [1, 0]; after token 1: [a, 2 * 2]; o = (q . S): 1 * 1, then 2 * 4
    silu = lambda x: x / (1 + math.exp(-x))
    assert abs(float(out[0, 0]) - 1 / math.sqrt(1 + 3.0) * silu(1.0)) < 1e-12
    assert abs(float(out[1, 0]) - 8 / math.sqrt(64 + 3.0) * silu(2.0)) < 1e-12


def test_plain_weights_are_the_softmax_over_the_chosen():
    w = {"router": torch.tensor([[1.0], [2.0], [0.0], [3.0]], dtype=torch.float64), "router.b": torch.tensor([0.0, 0.0, 9.0, -9.0], dtype=torch.float64)}
    (mine, weight), = pt.route(torch.tensor([[1.0]], dtype=torch.float64), w, "", 2)
    assert mine == [2, 1]  # by logit with the bias in it: 1, 2, 9, -6
    assert abs(float(weight[1]) - 1 / (1 + math.exp(7.0))) < 1e-12 and abs(float(weight.sum()) - 1) < 1e-12
