"""Mimolix on the CPU: reading config.json, the order of runs, the weight plan, random weights, and the plain
implementation's own consistency."""
import copy
import json

import pytest
import torch

import mimolix_configs as mc
import plain_mimolix as px
from geneinfer_b200.config import ConfigError, MimolixConfig, parse_config
from geneinfer_b200.weights import load_model_folder

CASES = {"a": mc.MIM_A, "b": mc.MIM_B, "c": mc.MIM_C, "d": mc.MIM_D}


@pytest.mark.parametrize("case", sorted(CASES))
def test_configuration_round_trip_and_translation(case):
    arch, cfg = parse_config(CASES[case])
    assert arch.name == "Mimolix" and isinstance(cfg, MimolixConfig)
    assert parse_config(json.loads(json.dumps(cfg.to_json())))[1] == cfg
    spec = cfg.model_spec()
    spec.validate()
    n = len(CASES[case]["layers"])
    order = px.layer_runs(CASES[case])
    assert [(e.layer, e.stream_input) for e in spec.schedule] == order
    # every run has a cache of its own: the first pass the layer's, later passes a layer that owns no weights
    caches = [e.layer if e.cache_of is None else e.cache_of for e in spec.schedule]
    assert len(set(caches)) == len(caches) and len(spec.layers) == len(order)
    for e in spec.schedule:
        if e.cache_of is not None:
            assert e.cache_of >= n and spec.shared_layers[e.cache_of] == e.layer
    assert (spec.stream_input is None) == ("loop" not in CASES[case]) and spec.embedding_scale == CASES[case].get("embedding", {}).get("scale", 1.0)
    assert all(l.block == "parallel" and l.block_params["residual_mult"] == CASES[case].get("residual_mult", 1.0) for l in spec.layers)


def test_every_constant_is_read_from_the_file():
    spec = parse_config(mc.MIM_A)[1].model_spec()
    att = spec.layers[0].mixer.params
    assert (att["num_heads"], att["num_kv_heads"], att["head_dim"], att["value_dim"], att["scale"], att["maps"]) == (4, 2, 16, 24, 0.3, 2)
    assert att["map_weight"] == 0.4 and att["map_factor"] == 0.6 and att["query_temperature"] == (0.5, 7.0) and att["qk_norm_eps"] == 1e-5
    assert spec.layers[2].mixer.params["query_temperature"] is None
    d = spec.layers[1].mixer.params
    assert (d["num_heads"], d["num_key_heads"], d["key_dim"], d["value_dim"], d["conv_taps"], d["norm_eps"]) == (6, 2, 16, 40, 3, 1e-5)
    f = spec.layers[0].feed_forward.params
    assert (f["intermediate_size"], f["experts"], f["top"], f["router_scale"], f["shared"]["intermediate_size"]) == (40, 5, 2, 1.5, 56)
    assert f["scores"] == "softmax" and f["renormalise"] and not f["gated"] and f["activation"] == "relu2"
    assert spec.layers[1].feed_forward.params["shared"] is None and spec.layers[2].feed_forward.params["router_scale"] == 1.0
    assert spec.layers[3].feed_forward is None


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="lightning"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=8), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c.update(loop={"start": 2, "stop": 2, "times": 2}), "loop"),
    (lambda c: c.update(loop={"start": 0, "stop": 9, "times": 2}), "loop"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_bad_configurations_are_refused(change, message):
    cfg = copy.deepcopy(mc.MIM_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        parse_config(cfg)


def test_random_weights_folder_loads_by_name(tmp_path):
    folder = mc.make_model_dir(mc.MIM_A, 5, str(tmp_path / "m"))
    _, cfg, params = load_model_folder(folder)
    assert params["layers.0.mixer.w_qkv"].shape == (2 * 4 * 16 + 2 * 2 * 16 + 2 * 24, 96) and params["layers.0.mixer.w_o"].shape == (96, 4 * 24)
    assert params["layers.0.mixer.q_norm"].shape == (16,) and params["layers.0.mixer.lq1"].shape == (16,)
    assert params["layers.1.mixer.w_in"].shape == (2 * 2 * 16 + 2 * 6 * 40 + 2 * 6, 96)
    assert params["layers.1.mixer.conv"].shape == (2 * 2 * 16 + 6 * 40, 3) and params["layers.3.mixer.conv"].shape[1] == 1
    assert params["layers.0.feed_forward.w_up"].shape == (5, 40, 96) and params["layers.0.feed_forward.w_down"].shape == (5, 96, 40)
    assert params["layers.0.feed_forward.shared.w_up"].shape == (56, 96) and "layers.1.feed_forward.shared.w_up" not in params
    assert params["stream_input.weight"].shape == (96, 192) and params["final_norm.bias"].shape == (96,)
    assert not any(k.startswith(("layers.3.feed_forward", "layers.4.")) for k in params)
    assert "stream_input.weight" not in load_model_folder(mc.make_model_dir(mc.MIM_C, 5, str(tmp_path / "c")))[2]


def test_plain_model_is_causal_and_its_passes_read_the_embedding(tmp_path):
    folder = mc.make_model_dir(mc.MIM_A, 8, str(tmp_path / "m"))
    w, raw = px.load(folder)
    toks = list(range(40, 75))
    after = []
    full = px.forward(w, raw, toks, layers_out=after)
    assert torch.allclose(px.forward(w, raw, toks[:20]), full[:20], rtol=0, atol=1e-9)
    assert [i for i, _ in px.layer_runs(raw)] == [0, 1, 2, 1, 2, 1, 2, 3] and len(after) == 8
    assert [s for _, s in px.layer_runs(raw)] == [False, True, False, True, False, True, False, False]
    w2 = dict(w)
    w2["loop.in"] = torch.cat([w["loop.in"][:, :96], torch.zeros(96, 96)], dim=1)
    assert float((px.forward(w2, raw, toks) - full).abs().max()) > 1e-3


def test_plain_delta_rule_recalls_what_was_written_and_overwrites_it():
    """With no fading and full steps, a key reads back exactly what was last written under it."""
    g = torch.Generator().manual_seed(1)
    T, d, dv = 6, 4, 3
    keys = torch.eye(d, dtype=torch.float64)[[0, 1, 2, 1, 3, 0]].view(T, 1, d)
    v = torch.randn(T, 1, dv, generator=g, dtype=torch.float64)
    o, S = px.delta_rule(keys, keys, v, torch.ones(T, 1, dtype=torch.float64), torch.ones(T, 1, dtype=torch.float64))
    assert torch.allclose(o, v)
    assert torch.allclose(S[0], torch.stack([v[5, 0], v[3, 0], v[2, 0], v[4, 0]]))
