"""Kidarax on the CPU: reading config.json, the order of runs, the weight plan, random weights, and the plain
implementation's own consistency."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import kidarax_configs as kc
import plain_kidarax as pk
from geneinfer_b200.config import ConfigError, KidaraxConfig, parse_config
from geneinfer_b200.weights import load_model_folder

CASES = {"a": kc.KID_A, "b": kc.KID_B, "c": kc.KID_C, "d": kc.KID_D}


@pytest.mark.parametrize("case", sorted(CASES))
def test_configuration_round_trip_and_translation(case):
    arch, cfg = parse_config(CASES[case])
    assert arch.name == "Kidarax" and isinstance(cfg, KidaraxConfig)
    assert parse_config(json.loads(json.dumps(cfg.to_json())))[1] == cfg
    spec = cfg.model_spec()
    spec.validate()
    n = len(CASES[case]["layers"])
    order = pk.layer_runs(CASES[case])
    assert [(e.layer, e.stream_input) for e in spec.schedule] == order
    # every run has a cache of its own: the first pass the layer's, later passes a layer that owns no weights
    caches = [e.layer if e.cache_of is None else e.cache_of for e in spec.schedule]
    assert len(set(caches)) == len(caches) and len(spec.layers) == len(order)
    for e in spec.schedule:
        if e.cache_of is not None:
            assert e.cache_of >= n and spec.shared_layers[e.cache_of] == e.layer
    assert (spec.stream_input is None) == ("loop" not in CASES[case]) and spec.tie_word_embeddings
    assert (spec.logit_transform.params["factor"] if spec.logit_transform else 1.0) == CASES[case].get("logit_scale", 1.0)
    for l, raw in zip(spec.layers, CASES[case]["layers"]):
        assert l.block == "sandwich" and l.mixer_norm.kind == "dynamic_tanh" and ("feed_forward_out_norm" in l.extra) == bool(raw["mlp"])


def test_a_loop_of_one_pass_adds_nothing():
    spec = parse_config(dict(kc.KID_A, loop={"start": 0, "stop": 3, "times": 1}))[1].model_spec()
    assert spec.stream_input is None and len(spec.schedule) == 4 and not any(e.stream_input for e in spec.schedule)


def test_every_constant_is_read_from_the_file():
    spec = parse_config(kc.KID_A)[1].model_spec()
    att = spec.layers[0].mixer.params
    assert (att["num_heads"], att["num_kv_heads"], att["head_dim"], att["value_dim"], att["scale"]) == (6, 2, 24, 40, 0.21)
    assert att["bias"] and att["output_gate"] and att["position"].params == {
        "head_dim": 24, "rotary_dim": 16, "theta": 10000.0, "pairing": "half_split", "linear_scaling": {"factor": 2.5}}
    r = spec.layers[1].mixer.params
    assert (r["num_heads"], r["key_dim"], r["value_dim"], r["decay"], r["norm_eps"], r["query_scale"]) == (3, 16, 40, [0.9, 0.97, 0.999], 1e-5, 0.25)
    assert r["norm_per_head"] and not r["norm_weights"] and r["gate"] == "silu" and r["activation"] == "none"
    l = spec.layers[2].mixer.params
    assert (l["num_heads"], l["head_dim"], l["rotary_dim"], l["value_dim"], l["kv_rank"], l["scale"], l["q_rank"]) == (5, 12, 8, 20, 24, 0.25, None)
    assert l["position"].params["ramp_scaling"] == {"factor": 4.0, "original": 64.0, "fast": 16.0, "slow": 1.5} and l["head_gate"]
    f = spec.layers[0].feed_forward.params
    assert (f["intermediate_size"], f["experts"], f["top"], f["shared"]["intermediate_size"]) == (40, 5, 2, 56)
    assert f["scores"] == "sigmoid" and f["weigh_input"] and f["shared_gate"] and f["activation"] == "silu"
    assert spec.layers[1].feed_forward.params == {"hidden_size": 96, "intermediate_size": 136, "activation": "relu2"}
    assert spec.layers[2].feed_forward.params["shared"] is None and not spec.layers[2].feed_forward.params["shared_gate"]
    assert spec.layers[3].feed_forward is None


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="lightning"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=15), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 0}), "positive"),
    (lambda c: c["layers"][1]["mixer"]["decay"].append(0.5), "decay"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=8), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="table"), "kind"),
    (lambda c: c["layers"][2]["mlp"].pop("expert"), "expert"),
    (lambda c: c.update(loop={"start": 2, "stop": 2, "times": 2}), "loop"),
    (lambda c: c.update(loop={"start": 0, "stop": 9, "times": 2}), "loop"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_bad_configurations_are_refused(change, message):
    cfg = copy.deepcopy(kc.KID_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        parse_config(cfg)


def test_random_weights_folder_loads_by_name(tmp_path):
    folder = kc.make_model_dir(kc.KID_A, 5, str(tmp_path / "m"))
    _, cfg, params = load_model_folder(folder)
    assert params["layers.0.mixer.w_qkv"].shape == (6 * 24 + 2 * 24 + 2 * 40 + 6 * 40, 96) and params["layers.0.mixer.b_qkv"].shape == (272,)
    assert params["layers.0.mixer.w_o"].shape == (96, 6 * 40)
    assert params["layers.1.mixer.w_in"].shape == (2 * 3 * 16 + 2 * 3 * 40, 96) and params["layers.1.feed_forward.w_up"].shape == (136, 96)
    assert params["layers.2.mixer.w_down"].shape == (5 * 20 + 24 + 8 + 5, 96) and params["layers.2.mixer.sink"].shape == (5,)
    assert params["layers.0.feed_forward.w_gate_up"].shape == (5, 80, 96) and params["layers.0.feed_forward.shared_gate"].shape == (1, 96)
    assert "layers.2.feed_forward.shared_gate" not in params
    for n in ("mixer_norm", "mixer_out_norm", "feed_forward_norm", "feed_forward_out_norm"):
        assert params[f"layers.0.{n}.weight"].shape == (96,) and params[f"layers.0.{n}.alpha"].shape == ()
    assert params["final_norm.alpha"].shape == () and params["head.weight"] is params["embedding.weight"]
    assert not any(k.startswith(("layers.3.feed_forward", "layers.4.")) for k in params)


def test_plain_model_is_causal_and_its_further_passes_read_the_embedding(tmp_path):
    folder = kc.make_model_dir(kc.KID_A, 8, str(tmp_path / "m"))
    w, raw = pk.load(folder)
    toks = list(range(40, 75))
    after = []
    full = pk.forward(w, raw, toks, layers_out=after)
    assert torch.allclose(pk.forward(w, raw, toks[:20]), full[:20], rtol=0, atol=1e-9)
    assert [i for i, _ in pk.layer_runs(raw)] == [0, 1, 2, 1, 2, 1, 2, 3] and len(after) == 8
    assert [s for _, s in pk.layer_runs(raw)] == [False, False, False, True, False, True, False, False]


def test_plain_retention_is_a_sum_over_the_past():
    g = torch.Generator().manual_seed(1)
    T, H, d, dv = 7, 2, 5, 3
    q, k = torch.randn(T, H, d, generator=g, dtype=torch.float64), torch.randn(T, H, d, generator=g, dtype=torch.float64)
    v = torch.randn(T, H, dv, generator=g, dtype=torch.float64)
    o, S = pk.retention(q, k, v, [0.5, 0.9])
    for h, fade in enumerate((0.5, 0.9)):
        want = sum(fade ** (T - 1 - j) * float(q[T - 1, h] @ k[j, h]) * v[j, h] for j in range(T))
        assert torch.allclose(o[T - 1, h], want)
    more, _ = pk.retention(q[4:], k[4:], v[4:], [0.5, 0.9], pk.retention(q[:4], k[:4], v[:4], [0.5, 0.9])[1])
    assert torch.allclose(more, o[4:])


def test_frequencies_of_the_scaled_rotations():
    """The part's frequencies against the plain ones, and the plain ones against their ends: fast pairs keep theirs, slow pairs
    are stretched by the factor."""
    from geneinfer_b200.parts import POSITION_ENCODINGS, BuildContext
    build = BuildContext(torch.device("cpu"), torch.float32, 64)
    for layer in kc.KID_A["layers"] + kc.KID_B["layers"] + kc.KID_C["layers"] + kc.KID_D["layers"]:
        if layer["type"] == "retention":
            continue
        m = layer["mixer"]
        cfg = parse_config(kc.model(32, 50, 1e-5, [layer]))[1]
        spec = cfg.model_spec().layers[0].mixer.params["position"]
        part = POSITION_ENCODINGS[spec.kind](dict(spec.params), {}, build)
        f, mult = pk.pair_frequencies(m["rot"])
        assert np.allclose(part.freq.numpy(), f, rtol=1e-6) and part.amplitude == pytest.approx(mult) and not part.interleaved
    f, mult = pk.pair_frequencies({"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
    assert f[0] == 1.0 and f[31] == pytest.approx(10000.0 ** (-62 / 64) / 8) and mult == pytest.approx(0.1 * math.log(8) + 1)
