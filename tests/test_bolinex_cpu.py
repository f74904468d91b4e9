"""Bolinex on the CPU: configuration, registry, checkpoint adapter, the cache's entries, the one error for a checkpoint
that does not fit; and the plain restatement by hand (a window's edge, the cap and the distance, mixed values, the choice
among groups, the token side)."""
import json
import math

import pytest
import torch

import bolinex_models as bm
import plain_bolinex as pb


def test_config_json_round_trip_registry_and_joint_tensors(tmp_path):
    from fms_b200 import models
    from fms_b200.cache.requests import KVRequest
    from fms_b200.models import get_model
    from fms_b200.models.bolinex import Bolinex

    assert "bolinex" in models.list_models() and "tiny" in models.list_variants("bolinex")
    cfg = bm.CONFIGS["p"]
    raw = bm.tensors(cfg, 1)
    folder = bm.write_folder(str(tmp_path / "p"), cfg, raw)
    model = get_model("hf_pretrained", model_path=folder, device_type="cpu", data_type="fp32")  # found by "architecture"
    assert isinstance(model, Bolinex)
    spec = model.decoder_spec()
    assert all(b.arrangement == "parallel_joint" and b.mixer.kind == "sink_attention" for b in spec.layers)
    assert [None if b.feed_forward is None else b.feed_forward.kind for b in spec.layers] == \
        ["routed_experts", "projected_unit", None, "routed_experts"]
    assert [dict(b.mixer.options)["v_mix"] for b in spec.layers] == ["", "first", "mixed", "mixed"]
    assert [b.mixer.window for b in spec.layers] == [20, 90, 90, 20]
    assert spec.final_norm.kind == "layernorm" and spec.embedding.kind == "table_and_positions" and spec.max_positions == 640
    sd = model.state_dict()
    f = {k: v.float() for k, v in raw.items()}
    # [q; k; v; g; shared gate; shared up] and [o | shared down]; with a dense feed-forward [q; k; v; g; up] and [o | down]
    assert torch.equal(sd["layers.0.in_proj.weight"], torch.cat([f["l0.mix." + n] for n in "qkvg"]
                                                               + [f["l0.mlp.shared.gate"], f["l0.mlp.shared.up"]]))
    assert torch.equal(sd["layers.0.out_proj.weight"], torch.cat([f["l0.mix.o"], f["l0.mlp.shared.down"]], 1))
    assert torch.equal(sd["layers.1.in_proj.weight"], torch.cat([f["l1.mix." + n] for n in "qkvg"] + [f["l1.mlp.up"]]))
    assert torch.equal(sd["layers.1.out_proj.weight"], torch.cat([f["l1.mix.o"], f["l1.mlp.down"]], 1))
    assert torch.equal(sd["layers.2.out_proj.weight"], f["l2.mix.o"]) and sd["layers.2.in_proj.weight"].shape == (96 + 24 + 8 + 32, 48)
    assert torch.equal(sd["layers.3.mlp.gate_up"][7], torch.cat([f["l3.mlp.e7.gate"], f["l3.mlp.e7.up"]]))
    assert torch.equal(sd["layers.2.side.table"], f["side.embed"][:, 12:18]) and sd["layers.1.mix.vmix"].shape == ()
    assert torch.equal(sd["embedding.positions"], f["pos"]) and torch.equal(sd["final_norm.bias"], f["final.norm.b"])
    requests = model.decoder.cache_requests()
    assert requests[0] == KVRequest(1, 32, 20) and requests[1] == KVRequest(1, 32, 90) and requests[3] == KVRequest(1, 16, 20)
    assert json.loads(json.dumps(model.config_json())) == cfg


def test_without_a_side_and_with_sizes_left_out(tmp_path):
    from fms_b200.models import get_model

    cfg = bm.CONFIGS["t"]
    assert "token_side" not in cfg
    lean = json.loads(json.dumps(cfg))
    del lean["layers"][0]["mlp"]["ff"], lean["layers"][1]["mlp"]["expert"], lean["layers"][1]["mlp"]["shared"]["ff"]
    del lean["layers"][1]["mlp"]["router"]["experts"]
    folder = bm.write_folder(str(tmp_path / "t"), lean, bm.tensors(cfg, 3))
    model = get_model("hf_pretrained", model_path=folder, device_type="cpu", data_type="bf16")
    assert model.config_json() == cfg and model.decoder.blocks[0].token_side is None
    assert "layers.1.mix.vmix" in model.state_dict() and "layers.0.mix.vmix" not in model.state_dict()


def test_a_checkpoint_that_does_not_fit_is_refused_with_one_error(tmp_path):
    from fms_b200.models import get_model
    from fms_b200.weights import WeightError

    cfg = bm.CONFIGS["q"]
    weights = bm.tensors(cfg, 2)
    del weights["l0.mix.g"], weights["l1.mlp.e2.down"], weights["l2.mix.vmix"], weights["final.norm.b"]
    weights["l1.mix.r2"] = weights["l1.mix.r2"][:-1]
    weights["stray"] = torch.zeros(3, dtype=torch.bfloat16)
    folder = bm.write_folder(str(tmp_path / "q"), cfg, weights)
    with pytest.raises(WeightError) as e:
        get_model("hf_pretrained", model_path=folder, device_type="cpu", data_type="fp32")
    for name in ("layers.0.in_proj.weight", "layers.1.mlp.down", "layers.2.mix.vmix", "final_norm.bias"):
        assert name in e.value.missing
    assert "stray" in e.value.unexpected and any(n == "layers.1.mix.r2" for n, _, _ in e.value.wrong_shapes)
    # the number of the first layer that mixes is not used, and may be absent
    weights = bm.tensors(cfg, 2)
    del weights["l0.mix.vmix"]
    get_model("hf_pretrained", model_path=bm.write_folder(str(tmp_path / "q2"), cfg, weights), device_type="cpu", data_type="fp32")


def test_config_json_of_another_design_or_with_unknown_parts_is_refused():
    from fms_b200.models.bolinex import Bolinex

    with pytest.raises(ValueError):
        Bolinex.config_from_json({"architecture": "Other"})
    for change, what in ((lambda c: c["layers"][0].update(type="convolution"), "convolution"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse"), (lambda c: c.pop("max_positions"), "max_positions")):
        bad = json.loads(json.dumps(bm.CONFIGS["r"]))
        change(bad)
        with pytest.raises(ValueError, match=what):
            Bolinex.config_from_json(bad)
    bad = json.loads(json.dumps(bm.CONFIGS["r"]))
    bad["layers"][0]["mlp"]["router"]["top"] = 4  # three groups of one expert stay
    from fms_b200.engine.decoder import Decoder
    with pytest.raises(ValueError, match="top 4"):
        Decoder(Bolinex(Bolinex.config_from_json(bad)).decoder_spec(), torch.float32)


def test_random_weights_of_a_registered_variant():
    from fms_b200.models import get_model

    model = get_model("bolinex", "tiny", device_type="cpu", data_type="bf16")
    assert model.decoder.blocks[1].feed_forward.groups == 4 and model.decoder.blocks[0].mixer.v_mix == "first"
    assert model.cache_bytes_per_token() == 4 * 2 * 2 * 32 * 2


def test_plain_window_cap_distance_and_mixing():
    ok = pb.visible(6, 3)
    assert ok[4].tolist() == [False, False, True, True, True, False] and ok[0].tolist() == [True] + [False] * 5
    assert pb.visible(4, 1).tolist() == torch.eye(4).bool().tolist()
    q, k = torch.tensor([[[1.0]], [[2.0]]], dtype=torch.float64), torch.tensor([[[3.0]], [[-4.0]]], dtype=torch.float64)
    s = pb.scores(q, k, 0.5, 2.0, torch.tensor([1.5], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64))
    assert abs(float(s[0, 1, 0]) - (2 * math.tanh(3.0 / 2) - 1.5 * math.log(1.5))) < 1e-12  # distance 1
    assert abs(float(s[0, 1, 1]) - 2 * math.tanh(-4.0 / 2)) < 1e-12  # distance 0: nothing is taken off
    assert torch.equal(pb.mix_values(torch.tensor([4.0]), torch.tensor([8.0]), torch.tensor(0.25)), torch.tensor([5.0]))


def test_plain_choice_among_groups():
    # groups (0, 1, 2) and (3, 4, 5): the best single expert lies in the group whose two best are worse together
    c = torch.tensor([-0.1, -2.0, -3.0, -0.9, -1.0, -1.5])
    assert pb.choose(c, 2, 2, 1) == [3, 4]  # -1.9 beats -2.1
    assert pb.choose(c, 2, 2, 2) == [0, 3]
    assert pb.choose(c, 3, 2, 1) == [3, 4, 5]  # experts outside of the group are out, however negative the last one is
    assert pb.choose(c, 2, 6, 2) == [0, 3] and pb.choose(c, 1, 1, 1) == [0]
    # the weights are the scores, without the correction and without a division by their sum
    h = torch.tensor([[1.0]], dtype=torch.float64)
    w = {"router": torch.tensor([[2.0], [1.0]], dtype=torch.float64), "correction": torch.tensor([-5.0, 0.0], dtype=torch.float64)}
    for e in ("e0.", "e1."):
        w[e + "gate"] = w[e + "up"] = w[e + "down"] = torch.tensor([[1.0]], dtype=torch.float64)
    got = pb.experts_mlp(h, w, "", {"router": {"top": 1, "groups": {"count": 1, "keep": 1}}})
    sig = 1 / (1 + math.exp(-1.0))
    assert abs(float(got) - sig * sig) < 1e-12  # expert 1: its score sigmoid(1) times silu(1) * 1


def test_plain_token_side_takes_its_own_layers_columns():
    w = {"side.embed": torch.arange(12, dtype=torch.float64).reshape(2, 6), "l1.side.gate": torch.ones(2, 3, dtype=torch.float64),
         "l1.side.proj": torch.eye(3, 2, dtype=torch.float64), "l1.side.norm": torch.tensor([1.0, 2.0, 3.0], dtype=torch.float64)}
    x = torch.tensor([[1.0, 2.0, -1.0]], dtype=torch.float64)
    g = pb.gelu(torch.tensor(2.0, dtype=torch.float64))
    y = torch.stack([g * 8, g * 9, 0 * g])  # token 1's values 2 and 3 of its row 6..11
    want = y / torch.sqrt((y * y).mean() + 1e-5) * torch.tensor([1.0, 2.0, 3.0])
    torch.testing.assert_close(pb.token_side(x, w, "l1.", torch.tensor([1]), 1, 2, 1e-5)[0], want)
