"""Kidarax on the GPU against the plain implementation in plain_kidarax.py: each kernel and each mechanism alone, then whole
models through the step engine under different cuts of the same requests (whole prompts, token-by-token decoding,
portions down to two tokens, mixed batches on reused pages and state slots), keys made to stand out far back and at page
borders, values that a state must keep, sinks that outweigh the keys, the first tokens of a sequence, and greedy
generation through the engine's own entry point and scheduler."""
import copy
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kidarax_configs as kc
import plain_kidarax as pk
import tiny_configs as tc
import trace_tools as tt
from test_gpu_fovezen import StateCtx
from test_gpu_nipadra import _run_mixer

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
F = torch.float64
EPS = 1e-5


def _build(dtype, max_position=4096):
    from geneinfer_b200.parts import BuildContext
    return BuildContext(DEV, dtype, max_position)


def _bf(t):
    return t.to(torch.bfloat16).float()


def _rnd(dtype):
    return pk.ident if dtype is torch.float32 else pk.bf16


def _close(got, want, dtype, what, f32=2e-5, b16=2e-2):
    err = float((got.double() - want.double()).abs().max() / max(1.0, float(want.abs().max())))
    assert err < (f32 if dtype is torch.float32 else b16), f"{what}: {err}"


def _mat(rows, cols, g, std=0.3):
    return _bf(torch.randn(rows, cols, generator=g) * std)


# ------------------------------------------------------------------------------------------ kernels alone
def _norm(D, g, alpha):
    return {"n": 1 + 0.3 * torch.randn(D, generator=g), "n.b": torch.randn(D, generator=g), "n.alpha": torch.tensor(alpha)}


def _consts(w):
    return float(w["n.alpha"]), w["n"].to(DEV), w["n.b"].to(DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [200, 7, 1026, 4500])
def test_dynamic_tanh_kernel(dtype, D):
    """Small and saturating arguments, gathered rows, widths with and without 16-byte pieces."""
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(D)
    x = torch.randn(9, D, generator=g) * torch.tensor([1e-4, 1.0, 30.0] * 3)[:, None]
    w = _norm(D, g, 0.7)
    want = pk.tanh_norm(w, "n", x.double())
    out = torch.full((9, D), float("nan"), dtype=dtype, device=DEV)
    kernels.dynamic_tanh(x.to(DEV), *_consts(w), out)
    _close(out.cpu().float(), want, dtype, "norm", f32=1e-6, b16=1e-2)
    rows = torch.tensor([8, 0, 3, 3], dtype=torch.int32)
    some = torch.full((4, D), float("nan"), dtype=dtype, device=DEV)
    kernels.dynamic_tanh(x.to(DEV), *_consts(w), some, rows=rows.to(DEV))
    assert torch.equal(some, out[rows.long().to(DEV)])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [200, 7, 4500])
@pytest.mark.parametrize("more", [False, True])
def test_end_of_a_sublayer_with_norms_before_and_after(dtype, D, more):
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(D + 1)
    T = 5
    x, y, z = (torch.randn(T, D, generator=g) for _ in range(3))
    a, b = _norm(D, g, 1.3), _norm(D, g, 0.4)
    want = x.double() + pk.tanh_norm(a, "n", y.double()) + (z.double() if more else 0.0)
    xd, yd = x.to(DEV).clone(), y.to(DEV).clone()
    xn = torch.full((T, D), float("nan"), dtype=dtype, device=DEV)
    kernels.add_dynamic_tanh(yd, _consts(a), xd, z.to(DEV) if more else None, _consts(b), xn, clear_y=True)
    _close(xd.cpu(), want, torch.float32, "stream", f32=1e-6)
    _close(xn.cpu().float(), pk.tanh_norm(b, "n", want), dtype, "next input", f32=2e-6, b16=1e-2)
    assert not yd.any()
    alone = torch.empty_like(xn)
    kernels.dynamic_tanh(xd, *_consts(b), alone)
    assert torch.equal(alone, xn)                      # the same arithmetic in either kernel
    # the sum alone, y kept
    x2, y2 = x.to(DEV).clone(), y.to(DEV).clone()
    kernels.add_dynamic_tanh(y2, _consts(a), x2, z.to(DEV) if more else None)
    assert torch.equal(x2, xd) and torch.equal(y2.cpu(), y)
    kernels.add_stream(x2, z.to(DEV))
    assert torch.equal(x2, xd + z.to(DEV))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, hd, vd, dims", [(4, 2, 16, 24, 16), (2, 2, 10, 7, 6), (6, 1, 40, 96, 20), (2, 1, 128, 64, 128), (3, 3, 250, 33, 2)])
def test_biases_and_rotation_before_the_store(dtype, H, G, hd, vd, dims):
    """Biases on queries, keys and values (none on the columns behind), the first ``dims`` dimensions rotated in halves, positions
    far from zero."""
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(H * 7 + hd)
    T, page, first = 11, 4, 1000 * 4
    n = H * hd + G * hd + G * vd
    proj = torch.randn(T, n + 5, generator=g)
    bias = torch.cat([torch.randn(n, generator=g) * 3, torch.zeros(5)])
    rot = {"base": 500.0, "dims": dims, "scaling": {"factor": 2.5}}
    f, _ = pk.pair_frequencies(rot)
    tables = torch.zeros(1, 1003, dtype=torch.int32)
    tables[0, 1000:] = torch.tensor([2, 0, 1])
    q = torch.full((T, H * hd), float("nan"), dtype=dtype, device=DEV)
    kcache, vcache = (torch.full((3, G, page, w), float("nan"), dtype=dtype, device=DEV) for w in (hd, vd))
    kernels.norm_rope_store(proj.to(DEV), 0, H * hd, (H + G) * hd, None, None, 0.0, torch.tensor(f, dtype=torch.float32, device=DEV), False,
                            torch.arange(first, first + T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV),
                            tables.to(DEV), q, kcache, vcache, H, G, hd, page, value_dim=vd, bias=bias.to(DEV))
    full = (proj + bias).double()
    _close(q.cpu().float().view(T, H, hd), pk.rotate(full[:, :H * hd].view(T, H, hd), rot, first), dtype, "queries", f32=2e-6, b16=1e-2)
    order = [2, 0, 1]
    keys = torch.stack([kcache[order[t // page], :, t % page].cpu().float() for t in range(T)])
    vals = torch.stack([vcache[order[t // page], :, t % page].cpu().float() for t in range(T)])
    _close(keys, pk.rotate(full[:, H * hd:(H + G) * hd].view(T, G, hd), rot, first), dtype, "keys in their pages", f32=2e-6, b16=1e-2)
    _close(vals, full[:, (H + G) * hd:n].view(T, G, vd), dtype, "values in their pages", f32=1e-6, b16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E, top, D", [(5, 2, 40), (40, 7, 96), (3, 3, 17), (1, 1, 24), (300, 12, 64)])
def test_sigmoid_routing_with_the_gate_of_a_shared_expert(dtype, E, top, D):
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(E)
    T = 21
    x, w, sg = torch.randn(T, D, generator=g).to(dtype), torch.randn(E, D, generator=g) * 0.3, torch.randn(D, generator=g) * 0.3
    tm = kernels.grouped_tile_rows()
    tiles = kernels.route_tiles(T, top, E)
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    srt, grp, cnt = (torch.empty(n, dtype=torch.int32, device=DEV) for n in (tiles * tm, tiles, 1))
    gate = torch.full((T,), float("nan"), device=DEV)
    kernels.route(x.to(DEV), w.to(DEV), None, top, ids, wts, srt, grp, cnt, gate_w=sg.to(DEV), gate_out=gate)
    want_ids, want_w = pk.route({"router": w}, "", top, x.double(), pk.ident)
    assert torch.equal(ids.cpu().long().sort(1).values, want_ids.sort(1).values)
    got = torch.zeros(T, E, dtype=F).scatter_(1, ids.cpu().long(), wts.cpu().double())
    _close(got, torch.zeros(T, E, dtype=F).scatter_(1, want_ids, want_w), torch.float32, "weights", f32=5e-6)
    _close(gate.cpu(), torch.sigmoid(x.double() @ sg.double()), torch.float32, "gate", f32=5e-6)


def _experts(D, f, g, p=""):
    w = {p + "router": _mat(f["router"]["experts"], D, g)}
    for part, ff in [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
        for n, shape in (("gate", (ff, D)), ("up", (ff, D)), ("down", (D, ff))):
            w[f"{p}{part}.{n}"] = _mat(*shape, g, 0.2)
    if f.get("shared"):
        w[p + "shared.sg"] = _mat(1, D, g)
    return w


def _experts_part(D, f, w, dtype, p=""):
    from geneinfer_b200.parts import FEED_FORWARDS
    E = f["router"]["experts"]
    cat = lambda q: torch.cat([w[q + ".gate"], w[q + ".up"]])
    weights = {"router": w[p + "router"], "w_gate_up": torch.stack([cat(f"{p}e{e}") for e in range(E)]),
               "w_down": torch.stack([w[f"{p}e{e}.down"] for e in range(E)])}
    shared = None
    if f.get("shared"):
        weights["shared.w_gate_up"], weights["shared.w_down"], weights["shared_gate"] = cat(p + "shared"), w[p + "shared.down"], w[p + "shared.sg"]
        shared = {"hidden_size": D, "intermediate_size": f["shared"]["ff"]}
    return FEED_FORWARDS["routed_experts"]({"hidden_size": D, "intermediate_size": f["expert"]["ff"], "experts": E, "top": f["router"]["top"],
                                            "weigh_input": True, "shared": shared, "shared_gate": shared is not None}, weights, _build(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 6, 150])
@pytest.mark.parametrize("D, f", [(64, kc.moe(40, 5, 2, 56)), (72, kc.moe(24, 7, 3)), (100, kc.moe(30, 3, 1, 20)), (96, kc.moe(96, 4, 4, 64)),
                                  (48, kc.moe(20, 33, 6, 12)), (128, kc.moe(64, 5, 2, 200))])
def test_experts_whose_weights_scale_their_inputs(dtype, T, D, f):
    """Few pairs (tiles on the CUDA cores) and many (the tensor cores, where the sizes allow it), with and without a gated shared
    expert. A weight on the output instead gives something else."""
    g = torch.Generator().manual_seed(D + T)
    w = _experts(D, f, g)
    h = _bf(torch.randn(T, D, generator=g))
    y = torch.randn(T, D, generator=g)
    w["router"] = w["router"] * 0.3                       # weights around one half
    yd = y.to(DEV).clone()
    _experts_part(D, f, w, dtype).forward(StateCtx(dtype, 1), h.to(DEV).to(dtype), yd)
    want = pk.experts(w, "", f, h.double(), _rnd(dtype))
    _close(yd.cpu() - y, want, dtype, f"experts, {T} tokens", b16=2e-2)
    ids, s = pk.route(w, "", f["router"]["top"], h.double(), pk.ident)
    other = torch.stack([sum(s[t, c] * pk.gated_mlp(w, f"e{ids[t, c]}.", h[t:t + 1].double(), pk.ident)[0] for c in range(ids.shape[1])) for t in range(T)])
    if f.get("shared"):
        other = other + torch.sigmoid(h.double() @ w["shared.sg"].double().T) * pk.gated_mlp(w, "shared.", h.double(), pk.ident)
    assert float((other - want).abs().max()) > 0.1 * float(want.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 40, 200])
@pytest.mark.parametrize("D, ff", [(64, 136), (100, 44), (96, 30)])
def test_squared_relu_feed_forward(dtype, T, D, ff):
    from geneinfer_b200.parts import FEED_FORWARDS
    g = torch.Generator().manual_seed(ff)
    w = {"up": _mat(ff, D, g), "down": _mat(D, ff, g)}
    part = FEED_FORWARDS["mlp"]({"hidden_size": D, "intermediate_size": ff, "activation": "relu2"}, {"w_up": w["up"], "w_down": w["down"]}, _build(dtype))
    h = _bf(torch.randn(T, D, generator=g))
    y = torch.zeros(T, D, device=DEV)
    part.forward(StateCtx(dtype, 1), h.to(DEV).to(dtype), y)
    _close(y.cpu(), pk.squared_relu_mlp(w, "", h.double(), _rnd(dtype)), dtype, "feed-forward", b16=2e-2)


# ------------------------------------------------------------------------------------------ mixers alone
CUTS = {"whole": [[40, 2, 19]], "token by token": [[1, 1, 1]] * 2 + [[1, 0, 1]] * 17 + [[1, 0, 0]] * 21,
        "portions": [[2, 1, 3], [5, 1, 2], [2, 0, 14], [31, 0, 0]], "tail decoded": [[30, 2, 10]] + [[1, 0, 1]] * 9 + [[1, 0, 0]]}

ROT = {"base": 300.0, "dims": 16, "scaling": {"factor": 2.0}}
ATT = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.5, "rot": ROT}
ATT_FORMS = [ATT, dict(ATT, heads=3, kv_heads=3, dim=10, vdim=14, rot=dict(ROT, dims=6, scaling=None)), dict(ATT, heads=6, kv_heads=1, dim=24, vdim=64),
             # keys as wide as the values: the sizes of the tensor-core kernels, and others
             dict(ATT, heads=4, kv_heads=4, dim=32, vdim=32), dict(ATT, heads=8, kv_heads=2, dim=64, vdim=64, scale=0.2, rot=dict(ROT, dims=64)),
             dict(ATT, heads=2, kv_heads=1, dim=128, vdim=128, scale=0.1, rot=dict(ROT, dims=32)), dict(ATT, heads=12, kv_heads=1, dim=64, vdim=64, scale=0.1),
             dict(ATT, heads=4, kv_heads=1, dim=48, vdim=48), dict(ATT, heads=2, kv_heads=2, dim=200, vdim=200, scale=0.1),
             # the row-form kernel's tensor-core sizes: values in whole 64s, keys in whole 16s
             dict(ATT, heads=20, kv_heads=1, dim=80, vdim=64, scale=0.2), dict(ATT, heads=8, kv_heads=1, dim=64, vdim=192, scale=0.2),
             dict(ATT, heads=6, kv_heads=2, dim=32, vdim=128), dict(ATT, heads=2, kv_heads=1, dim=128, vdim=320, scale=0.1)]


def _att_weights(D, m, g, p="p."):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {p + "g": _mat(H * dv, D, g), p + "o": _mat(D, H * dv, g)}
    for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
        w[p + n], w[p + n + ".b"] = _mat(rows, D, g), torch.randn(rows, generator=g) * 0.5
    return w


def _position(rot, size):
    """The PartSpec of a rotation as the configuration translates it."""
    from geneinfer_b200.config.kidarax import Rotation
    s = rot.get("scaling")
    ramp = (s["original"], s["fast"], s["slow"]) if s and "original" in s else None
    return Rotation(rot["base"], rot["dims"], s["factor"] if s else None, ramp).spec(size)


def _att_part(D, m, w, dtype, p="p."):
    from geneinfer_b200.parts import MIXERS
    return MIXERS["attention"](
        {"hidden_size": D, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
         "scale": m["scale"], "window": None, "position": _position(m["rot"], m["dim"]), "bias": True, "output_gate": True},
        {"w_qkv": torch.cat([w[p + n] for n in ("q", "k", "v", "g")]), "b_qkv": torch.cat([w[p + n + ".b"] for n in ("q", "k", "v")]),
         "w_o": w[p + "o"]}, _build(dtype))


def _pages(part, dtype, n, max_len=256, page_size=8):
    need = part.cache_need()
    return StateCtx(dtype, n, Hkv=need.num_kv_heads, hd=need.head_dim, vd=need.value_width, page_size=page_size, max_len=max_len)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", ATT_FORMS)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_attention_with_biases_and_a_gate_per_value(dtype, m, cut):
    D = 40
    g = torch.Generator().manual_seed(9)
    w = _att_weights(D, m, g)
    part = _att_part(D, m, w, dtype)
    inputs = [_bf(torch.randn(n, D, generator=g)) for n in (40, 2, 19)]
    want = [pk.attention_mixer(w, "p.", m, x.double(), EPS, _rnd(dtype)) for x in inputs]
    got = _run_mixer(part, _pages(part, dtype, 3), inputs, CUTS[cut], dtype, D)
    for r in range(3):
        _close(got[r], want[r], dtype, f"attention, request {r}, {cut}", b16=3e-2)


def test_attention_on_pages_that_the_tma_kernels_cannot_tile():
    D, m = 40, dict(ATT, heads=4, kv_heads=2, dim=64, vdim=64, scale=0.2)
    g = torch.Generator().manual_seed(10)
    w = _att_weights(D, m, g)
    for dtype in DTYPES:
        part = _att_part(D, m, w, dtype)
        inputs = [_bf(torch.randn(n, D, generator=g)) for n in (40, 2, 19)]
        want = [pk.attention_mixer(w, "p.", m, x.double(), EPS, _rnd(dtype)) for x in inputs]
        got = _run_mixer(part, _pages(part, dtype, 3, max_len=240, page_size=12), inputs, CUTS["portions"], dtype, D)
        for r in range(3):
            _close(got[r], want[r], dtype, f"pages of 12, request {r}", b16=3e-2)


YARN = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}
LAT = {"heads": 5, "dim": 12, "rot_dim": 8, "vdim": 20, "kv_rank": 24, "scale": 0.3, "rot": {"base": 1000.0, "dims": 8, "scaling": YARN}}


def _lat(**kw):
    m = dict(LAT, **kw)
    m["rot"] = dict(LAT["rot"], dims=m["rot_dim"], **({"scaling": kw["scaling"]} if "scaling" in kw else {}))
    m.pop("scaling", None)
    return m


LAT_FORMS = [LAT, _lat(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=18, scaling=None), _lat(heads=2, dim=16, rot_dim=2, vdim=40, kv_rank=40),
             # latents of the tensor-core form: few heads, sixteen, more than sixteen; a latent in whole 64s
             _lat(heads=8, dim=32, rot_dim=16, vdim=48, kv_rank=64, scale=0.15), _lat(heads=16, dim=24, rot_dim=32, vdim=64, kv_rank=128, scale=0.15),
             _lat(heads=20, dim=48, rot_dim=64, vdim=32, kv_rank=192, scale=0.1), _lat(heads=4, dim=64, rot_dim=32, vdim=128, kv_rank=512, scale=0.1)]


def _lat_weights(D, m, g, p="p."):
    H, d, r, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    return {p + "q": _mat(H * (d + r), D, g), p + "dkv": _mat(kr + r, D, g), p + "dkv.norm": 1 + 0.3 * torch.randn(kr, generator=g),
            p + "uk": _mat(H * d, kr, g, kr ** -0.5), p + "uv": _mat(H * dv, kr, g, kr ** -0.5), p + "g": _mat(H, D, g), p + "o": _mat(D, H * dv, g),
            p + "sink": torch.randn(H, generator=g)}


def _lat_part(D, m, w, dtype, p="p."):
    from geneinfer_b200.parts import MIXERS
    return MIXERS["latent_attention"](
        {"hidden_size": D, "num_heads": m["heads"], "head_dim": m["dim"], "rotary_dim": m["rot_dim"], "value_dim": m["vdim"], "q_rank": None,
         "kv_rank": m["kv_rank"], "scale": m["scale"], "window": None, "norm_eps": EPS, "position": _position(m["rot"], m["rot_dim"]),
         "sink": "learned", "head_gate": True},
        {"w_down": torch.cat([w[p + n] for n in ("q", "dkv", "g")]), "kv_latent_norm": w[p + "dkv.norm"], "w_uk": w[p + "uk"],
         "w_uv": w[p + "uv"], "w_o": w[p + "o"], "sink": w[p + "sink"]}, _build(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", LAT_FORMS)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_latent_attention_with_a_gate_per_head(dtype, m, cut):
    D = 40
    g = torch.Generator().manual_seed(19)
    w = _lat_weights(D, m, g)
    part = _lat_part(D, m, w, dtype)
    inputs = [_bf(torch.randn(n, D, generator=g)) for n in (40, 2, 19)]
    want = [pk.latent_attention_mixer(w, "p.", m, x.double(), EPS, _rnd(dtype)) for x in inputs]
    got = _run_mixer(part, _pages(part, dtype, 3), inputs, CUTS[cut], dtype, D)
    for r in range(3):
        _close(got[r], want[r], dtype, f"latent attention, request {r}, {cut}", b16=3e-2)


@pytest.mark.parametrize("m", [LAT, _lat(heads=16, dim=24, rot_dim=32, vdim=64, kv_rank=128, scale=0.15)])
def test_a_sink_that_outweighs_the_keys_of_the_first_tokens(m):
    """Large sinks: left out, scaled, or counted twice, the first rows would change by far more than the bound."""
    D = 40
    g = torch.Generator().manual_seed(23)
    w = _lat_weights(D, m, g)
    w["p.sink"] = torch.linspace(1.0, 5.0, m["heads"])
    x = _bf(torch.randn(9, D, generator=g))
    want = pk.latent_attention_mixer(w, "p.", m, x.double(), EPS, pk.ident)
    for change in (lambda s: s - 50.0, lambda s: s * m["scale"], lambda s: s + 0.6931):
        other = pk.latent_attention_mixer(dict(w, **{"p.sink": change(w["p.sink"])}), "p.", m, x.double(), EPS, pk.ident)
        assert float((other[:3] - want[:3]).abs().max()) > 0.02 * float(want.abs().max())
    for cuts in ([[9]], [[1]] * 9, [[2], [2], [5]]):
        part = _lat_part(D, m, w, torch.float32)
        got = _run_mixer(part, _pages(part, torch.float32, 1), [x], cuts, torch.float32, D)
        _close(got[0], want, torch.float32, f"sinks, {len(cuts)} steps")


def _sharp(kind, m, D, n, key, query, g):
    """Weights and inputs with one score that stands out: the query at ``query`` answers the key at ``key`` in the unrotated part."""
    w = (_att_weights if kind == "attention" else _lat_weights)(D, m, g)
    x = _bf(torch.randn(n, D, generator=g) * 0.3)
    x[:, 0] = x[:, 1] = 0.0
    w["p.q"] = w["p.q"] * 0.02
    w["p.q"][:, 1] = 0.0
    H, d = m["heads"], m["dim"]
    if kind == "attention":
        at = d - 1                                       # a dimension behind the rotated ones
        w["p.k"], w["p.k.b"], w["p.q.b"] = w["p.k"] * 0.02, w["p.k.b"] * 0.0, w["p.q.b"] * 0.0
        w["p.k"][:, 0] = 0.0
        w["p.q"].view(H, d, D)[:, at, 1] = 6.0
        w["p.k"].view(m["kv_heads"], d, D)[:, at, 0] = 6.0
    else:
        w["p.dkv"][:, 0] = 0.0
        w["p.dkv"][:4, 0] = 40.0                         # the latent of the marked token points where no other does
        w["p.uk"] = w["p.uk"] * 0.05
        w["p.uk"].view(H, d, -1)[:, 0, :4] = 2.0
        w["p.q"].view(H, d + m["rot_dim"], D)[:, 0, 1] = 3.0
    x[key, 0] = 3.0
    x[query, 1] = 3.0
    return w, x


SHARP = [("attention", dict(ATT, heads=4, kv_heads=2, dim=24, vdim=40, scale=0.3)),
         ("attention", dict(ATT, heads=4, kv_heads=2, dim=64, vdim=64, scale=0.2)),
         ("attention", dict(ATT, heads=4, kv_heads=1, dim=32, vdim=64, scale=0.3)),
         ("latent", LAT), ("latent", _lat(heads=16, dim=24, rot_dim=32, vdim=48, kv_rank=128, scale=0.3))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("back", [0, 1, 15, 16, 17, 255, 256, 650])
@pytest.mark.parametrize("form", range(len(SHARP)))
def test_one_key_among_hundreds(dtype, back, form):
    """The last query answers one key far back, at a page border, at the border of a decode chunk or its own, as the end of a prompt
    and decoded."""
    D, n = 24, 700
    kind, m = SHARP[form]
    g = torch.Generator().manual_seed(15)
    w, x = _sharp(kind, m, D, n, n - 1 - back, n - 1, g)
    mixer = pk.attention_mixer if kind == "attention" else pk.latent_attention_mixer
    want = mixer(w, "p.", m, x.double(), EPS, _rnd(dtype))
    moved = x.clone()
    moved[n - 1 - back, 0] = 0.0
    assert float((mixer(w, "p.", m, moved.double(), EPS, _rnd(dtype))[-1] - want[-1]).abs().max()) > 0.1 * float(want[-1].abs().max())
    part = (_att_part if kind == "attention" else _lat_part)(D, m, w, dtype)
    for cuts in ([[n - 30]] + [[1]] * 30, [[300], [398], [2]]):
        got = _run_mixer(part, _pages(part, dtype, 1, max_len=704, page_size=16), [x], cuts, dtype, D)
        _close(got[0][-1], want[-1], dtype, f"key {back} back among {n}, {len(cuts)} steps", b16=4e-2)


@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_rotations_tell_positions_apart(kind):
    """Only the rotated dimensions carry a score, at positions far from zero: a frequency, an amplitude or a pairing that is wrong
    changes the rows."""
    D, n = 24, 300
    g = torch.Generator().manual_seed(29)
    if kind == "attention":
        m = dict(ATT, heads=3, kv_heads=3, dim=16, vdim=16, scale=1.0, rot={"base": 40.0, "dims": 12, "scaling": {"factor": 3.0}})
        w, mixer, build = _att_weights(D, m, g), pk.attention_mixer, _att_part
    else:
        m = _lat(heads=3, dim=4, rot_dim=12, scale=1.0)
        w, mixer, build = _lat_weights(D, m, g), pk.latent_attention_mixer, _lat_part
        w["p.uk"] = w["p.uk"] * 0.0
    x = _bf(torch.randn(n, D, generator=g))
    want = mixer(w, "p.", m, x.double(), EPS, pk.ident)
    plain = dict(m, rot=dict(m["rot"], scaling=None))
    assert float((mixer(w, "p.", plain, x.double(), EPS, pk.ident)[n // 2:] - want[n // 2:]).abs().max()) > 0.05 * float(want.abs().max())
    for cuts in ([[n]], [[n - 20]] + [[1]] * 20):
        part = build(D, m, w, torch.float32)
        got = _run_mixer(part, _pages(part, torch.float32, 1, max_len=304), [x], cuts, torch.float32, D)
        _close(got[0], want, torch.float32, f"rotation, {len(cuts)} steps", f32=4e-5)


RET = {"heads": 3, "dim": 16, "vdim": 40, "decay": [0.9, 0.97, 0.999]}
RET_FORMS = [RET, {"heads": 2, "dim": 64, "vdim": 64, "decay": [0.5, 0.9995]}, {"heads": 4, "dim": 7, "vdim": 9, "decay": [1.0, 0.99, 0.2, 0.0]},
             {"heads": 1, "dim": 200, "vdim": 33, "decay": [0.98]}, {"heads": 2, "dim": 128, "vdim": 128, "decay": [0.95, 0.999]}]


def _ret_weights(D, m, g, p="p."):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    return {p + "q": _mat(H * d, D, g), p + "k": _mat(H * d, D, g), p + "v": _mat(H * dv, D, g), p + "g": _mat(H * dv, D, g), p + "o": _mat(D, H * dv, g)}


def _ret_part(D, m, w, dtype, p="p."):
    from geneinfer_b200.parts import MIXERS
    return MIXERS["linear_attention"](
        {"hidden_size": D, "num_heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"], "decay": m["decay"], "norm_eps": EPS,
         "activation": "none", "query_scale": m["dim"] ** -0.5, "norm_per_head": True, "norm_weights": False, "gate": "silu"},
        {"w_in": torch.cat([w[p + n] for n in ("q", "k", "v", "g")]), "w_o": w[p + "o"]}, _build(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", RET_FORMS)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_retention_mixer(dtype, m, cut):
    D = 48
    g = torch.Generator().manual_seed(4)
    w = _ret_weights(D, m, g)
    part = _ret_part(D, m, w, dtype)
    assert part.state_need().shape == (m["heads"] * m["dim"] * m["vdim"],) and part.cache_need() is None
    inputs = [_bf(torch.randn(n, D, generator=g)) for n in (40, 2, 19)]
    want = [pk.retention_mixer(w, "p.", m, x.double(), EPS, _rnd(dtype)) for x in inputs]
    got = _run_mixer(part, StateCtx(dtype, 3, state_floats=part.state_need().shape[0]), inputs, CUTS[cut], dtype, D)
    for r in range(3):
        _close(got[r], want[r], dtype, f"retention, request {r}, {cut}", f32=4e-5, b16=3e-2)


@pytest.mark.parametrize("cuts", [[[700]], [[300], [398], [2]], [[129], [1], [570]], [[690]] + [[1]] * 10])
def test_retention_keeps_one_token_among_hundreds(cuts):
    """Token 3 is written under a key that the last token alone reads: a head that hardly fades still has it, through the parts
    that a long portion is cut into and from step to step."""
    D, n = 16, 700
    m = {"heads": 2, "dim": 8, "vdim": 12, "decay": [0.9999, 0.9]}
    g = torch.Generator().manual_seed(31)
    w = _ret_weights(D, m, g)
    x = _bf(torch.randn(n, D, generator=g) * 0.05)
    x[:, 0] = x[:, 1] = 0.0
    w["p.q"], w["p.k"] = w["p.q"] * 0.05, w["p.k"] * 0.05
    w["p.q"].view(2, 8, D)[:, 5, 1], w["p.k"].view(2, 8, D)[:, 5, 0] = 9.0, 9.0
    x[3, 0], x[n - 1, 1] = 2.0, 2.0
    want = pk.retention_mixer(w, "p.", m, x.double(), EPS, pk.ident)
    gone = x.clone()
    gone[3] = 0.0
    assert float((pk.retention_mixer(w, "p.", m, gone.double(), EPS, pk.ident)[-1] - want[-1]).abs().max()) > 0.1 * float(want[-1].abs().max())
    part = _ret_part(D, m, w, torch.float32)
    got = _run_mixer(part, StateCtx(torch.float32, 1, state_floats=part.state_need().shape[0], max_len=704), [x], cuts, torch.float32, D)
    _close(got[0][-1], want[-1], torch.float32, "the kept token", f32=1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_in_one_batch_equal_each_alone(dtype):
    """Three unequal requests batched against each alone, on scattered pages and other state slots: the same bits."""
    D = 40
    g = torch.Generator().manual_seed(17)
    parts = [_att_part(D, m, _att_weights(D, m, g), dtype) for m in (ATT_FORMS[0], ATT_FORMS[4], ATT_FORMS[10])]
    parts += [_lat_part(D, m, _lat_weights(D, m, g), dtype) for m in (LAT_FORMS[0], LAT_FORMS[4])] + [_ret_part(D, RET, _ret_weights(D, RET, g), dtype)]
    for part in parts:
        ctx_of = (lambda n: StateCtx(dtype, n, state_floats=part.state_need().shape[0])) if part.state_need() else (lambda n: _pages(part, dtype, n))
        inputs = [_bf(torch.randn(n, D, generator=g)) for n in (33, 5, 12)]
        together = _run_mixer(part, ctx_of(3), inputs, [[20, 1, 3], [1, 1, 2], [12, 3, 7]], dtype, D)
        for r in range(3):
            alone = _run_mixer(part, ctx_of(1), [inputs[r]], [[[20, 1, 3][r]], [[1, 1, 2][r]], [[12, 3, 7][r]]], dtype, D)
            _close(alone[0], together[r], dtype, f"request {r} in a batch", f32=1e-5, b16=1e-2)


# ------------------------------------------------------------------------------------------ the arrangement alone
@pytest.mark.parametrize("kind", ["dynamic_tanh", "rmsnorm"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_sandwich_blocks_in_a_row(kind, dtype):
    """Two layers of squared-ReLU feed-forwards around retention mixers, the second without a feed-forward, run twice with the
    embedding's output added in between: norms of either kind."""
    from geneinfer_b200.config import LayerSpec, PartSpec
    from geneinfer_b200.parts import BLOCKS, STREAM_INPUTS, LayerRun
    D, T = 48, 21
    g = torch.Generator().manual_seed(3)
    norm_spec = PartSpec(kind, {"size": D, "eps": EPS})

    def norm_weights(alpha):
        w = {"weight": 1 + 0.2 * torch.randn(D, generator=g), "bias": 0.1 * torch.randn(D, generator=g), "alpha": torch.tensor(alpha)}
        return w

    def apply(w, v):
        if kind == "rmsnorm":
            return pk.unit_rms(v, EPS) * w["weight"].double()
        return pk.tanh_norm({"n": w["weight"], "n.b": w["bias"], "n.alpha": w["alpha"]}, "n", v)

    blocks, plain = [], []
    for i in range(2):
        w, ff = _ret_weights(D, RET, g), {"up": _mat(56, D, g), "down": _mat(D, 56, g)}
        norms = {n: norm_weights(0.3 + 0.2 * j) for j, n in enumerate(("mixer_norm", "mixer_out_norm", "feed_forward_norm", "feed_forward_out_norm"))}
        spec = LayerSpec(mixer=PartSpec("linear_attention", {
            "hidden_size": D, "num_heads": 3, "key_dim": 16, "value_dim": 40, "decay": RET["decay"], "norm_eps": EPS, "activation": "none",
            "query_scale": 0.25, "norm_per_head": True, "norm_weights": False, "gate": "silu"}),
            feed_forward=PartSpec("mlp", {"hidden_size": D, "intermediate_size": 56, "activation": "relu2"}) if i == 0 else None,
            mixer_norm=norm_spec, feed_forward_norm=norm_spec if i == 0 else None, block="sandwich",
            extra={"mixer_out_norm": norm_spec, **({"feed_forward_out_norm": norm_spec} if i == 0 else {})})
        weights = {f"{n}.{k}": v for n, ws in norms.items() for k, v in ws.items()}
        weights.update({"mixer.w_in": torch.cat([w["p." + n] for n in ("q", "k", "v", "g")]), "mixer.w_o": w["p.o"],
                        "feed_forward.w_up": ff["up"], "feed_forward.w_down": ff["down"]})
        blocks.append(BLOCKS["sandwich"](spec, weights, _build(dtype)))
        plain.append((w, ff if i == 0 else None, norms))
    add = STREAM_INPUTS["embedding_add"]({"hidden_size": D}, {}, _build(dtype))
    runs = [LayerRun(0, 0, True), LayerRun(1, 1, True), LayerRun(0, 2, True, True), LayerRun(1, 3, True)]
    for run, after in zip(runs, runs[1:]):
        blocks[run.layer].followed_in_run(run, blocks[after.layer], add if after.stream_input else None)
    x = torch.randn(T, D, generator=g)
    want = x.double()
    for run in runs:
        w, ff, norms = plain[run.layer]
        want = want + x.double() if run.stream_input else want
        want = want + apply(norms["mixer_out_norm"], pk.retention_mixer(w, "p.", RET, apply(norms["mixer_norm"], want), EPS, _rnd(dtype)))
        if ff is not None:
            want = want + apply(norms["feed_forward_out_norm"], pk.squared_relu_mlp(ff, "", apply(norms["feed_forward_norm"], want), _rnd(dtype)))

    class Ctx(StateCtx):
        tapping = False

        def state(self, layer):
            return states[layer]

        def scratch(self, name, shape, dtype, capacity=None):
            return buffers.setdefault((name, tuple(shape), dtype), super().scratch(name, shape, dtype, capacity))

        def recorded(self, owner, key, launch):
            launch()

    for tapping in (False, True):
        buffers = {}
        states = [torch.zeros(2, 3 * 16 * 40, device=DEV) for _ in runs]
        ctx = Ctx(dtype, 1, state_floats=1)
        ctx.tapping = tapping
        ctx.begin([T])
        xd = x.to(DEV).clone()
        add.begin(ctx, xd)
        for run in runs:
            if run.stream_input:
                add.forward(ctx, xd)
            blocks[run.layer].forward(ctx, run, xd)
        _close(xd.cpu(), want, dtype, f"two passes over two layers, {kind}, listening {tapping}", f32=5e-5, b16=4e-2)


# ------------------------------------------------------------------------------------------ whole models
_TMP = {}
LENGTHS = {"a": [1, 2, 3, 75, 20, 120, 47, 30], "b": [150, 4, 64, 1, 180], "c": [90, 2, 33, 1, 140, 17], "d": [1, 2, 100, 30, 7]}
CONFIGS = {"a": kc.KID_A, "b": kc.KID_B, "c": kc.KID_C, "d": kc.KID_D}


def _all_chosen(config):
    """The same model with every expert chosen. With experts left out, rounding may turn a close choice over, in an engine as in
    the plain model with rounded operands; comparisons in bfloat16 that are to hold at every position use this form."""
    config = copy.deepcopy(config)
    for layer in config["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return config


def _config(case):
    return _all_chosen(CONFIGS[case[0]]) if case.endswith("all") else CONFIGS[case]


def _model_dir(case, tmp_path_factory):
    if case not in _TMP:
        _TMP[case] = kc.make_model_dir(_config(case), 20 + ord(case[0]), str(tmp_path_factory.mktemp("kidarax_" + case)))
    return _TMP[case]


def _case(case, dtype):
    return case if dtype == "float32" else case + "_all"


def _requests(case):
    return {f"r{i}": tc.random_tokens(n, CONFIGS[case[0]]["vocab"], 400 + i) for i, n in enumerate(LENGTHS[case[0]])}


_PLAIN = {}


def _plain(case, folder, rounded=False, single=False):
    key = (case, rounded, single)
    if key not in _PLAIN:
        w, cfg = pk.load(folder)
        _PLAIN[key] = {rid: pk.forward(w, cfg, toks, torch.float32 if single else F, pk.bf16 if rounded else pk.ident).double().numpy()
                       for rid, toks in _requests(case).items()}
    return _PLAIN[key]


def _bound(exact, other, floor, times=3.0):
    """``times`` the distance between the plain model in two precisions, and at least ``floor``."""
    return max(floor, times * max(tt.rel_err(other[r], exact[r]) for r in exact))


def _tolerance(case, folder, dtype):
    """bfloat16: three times the distance between the exact plain model and the plain model with bfloat16 operands of the matrix
    products. 32-bit: 3e-5, or eight times the distance between the plain model in float64 and in float32 where that is more."""
    if dtype == "float32":
        return _bound(_plain(case, folder), _plain(case, folder, single=True), 3e-5, 8.0)
    return _bound(_plain(case, folder), _plain(case, folder, True), 0.0)


def _engine(folder, dtype, n_pages, max_requests=4, page_size=16, max_step_tokens=512):
    from geneinfer_b200.engine.loading import load_model
    from geneinfer_b200.engine.step import StepEngine
    model = load_model(folder, dtype=dtype, max_position=512)
    return StepEngine(model, page_size=page_size, n_pages=n_pages, max_requests=max_requests, max_step_tokens=max_step_tokens,
                      debug_checks=True)


def _all_free(engine):
    return engine.cache.slots.free_count == engine.max_requests and all(g.pool.free_count == g.pool.n_pages for g in engine.cache.groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["a", "b", "c", "d"])
def test_whole_prompts_decoding_portions_and_mixed_batches_agree_with_the_plain_model(case, dtype, tmp_path_factory):
    case = _case(case, dtype)
    folder = _model_dir(case, tmp_path_factory)
    reqs, plain, tol = _requests(case), _plain(case, folder), _tolerance(case, folder, dtype)
    traces = {"whole": tt.trace_whole(reqs), "decode": tt.trace_tail_decode(reqs, tail=40), "portions": tt.trace_portions(reqs),
              "mixed": tt.trace_mixed(reqs, seed=3, tail=12), "mixed2": tt.trace_mixed(reqs, seed=8, max_live=3, tail=30)}
    results = {}
    for name, steps in traces.items():
        # the pool holds what the trace's live requests need, no more: pages and state slots are used again
        n_pages = tt.max_tokens_of(steps, reqs, 16) // 16
        engine = _engine(folder, dtype, n_pages)
        got = tt.run_in_process(engine, steps)
        engine.check_status()
        tt.compare(got, plain, tol, f"Kidarax {case} {dtype} {name}")
        engine.cache.check_invariants()
        assert _all_free(engine)
        results[name] = got
    if dtype == "float32":       # the same position under different cuts: equal but for rounding
        for name in ("decode", "portions", "mixed"):
            for key, row in results[name].items():
                ref = results["whole"][key]
                assert float(np.abs(row - ref).max()) < tol * max(1.0, float(np.abs(ref).max())), (name, key)


@pytest.mark.parametrize("case", ["a", "b", "c"])
def test_chosen_experts_in_bfloat16(case, tmp_path_factory):
    """With experts left out, a close choice may turn over by rounding: nearly all positions lie within the bound that holds
    where every expert is chosen, and the typical one well inside it."""
    folder, folder_all = _model_dir(case, tmp_path_factory), _model_dir(case + "_all", tmp_path_factory)
    reqs, plain, tol = _requests(case), _plain(case, folder), _tolerance(case + "_all", folder_all, "bfloat16")
    for steps in (tt.trace_whole(reqs), tt.trace_mixed(reqs, seed=3, tail=12)):
        engine = _engine(folder, "bfloat16", tt.max_tokens_of(steps, reqs, 16) // 16)
        got = tt.run_in_process(engine, steps)
        engine.check_status()
        errs = np.array([tt.rel_err(row, plain[rid][pos]) for (rid, pos), row in got.items()])
        assert np.isfinite(errs).all() and np.median(errs) < tol and (errs > 2 * tol).mean() < 0.35, (np.median(errs), (errs > 2 * tol).mean(), tol)


def test_the_stream_after_every_layer_run(tmp_path_factory):
    """After each run of a layer (a looped layer counts every time), for a prompt fed whole and in portions."""
    folder = _model_dir("a", tmp_path_factory)
    w, cfg = pk.load(folder)
    toks = tc.random_tokens(45, 211, 6)
    after = []
    pk.forward(w, cfg, toks, layers_out=after)
    for sizes in ((45,), (7, 30, 2, 6)):
        engine = _engine(folder, "float32", n_pages=8)
        seen = []

        def tap(tag, layer, tensor, ctx):
            if tag == "ffn_out":
                seen.append((layer, tensor.detach().float().cpu()))
        engine.tap = tap
        tt.run_in_process(engine, tt.trace_portions({"r": toks}, sizes=sizes))
        runs = len(after)
        assert [l for l, _ in seen[:runs]] == [i for i, _ in pk.layer_runs(cfg)]
        for i in range(runs):
            got = torch.cat([t for _, t in seen[i::runs]])
            assert float((got.double() - after[i]).abs().max()) < 3e-5 * float(after[i].abs().max()), f"run {i}, portions {sizes}"


def test_listening_to_the_stream_does_not_change_the_logits(tmp_path_factory):
    folder = _model_dir("a", tmp_path_factory)
    steps = tt.trace_portions({"r": tc.random_tokens(45, 211, 6)}, sizes=(7, 30, 2, 6))
    got = []
    for listen in (False, True):
        engine = _engine(folder, "float32", n_pages=8)
        if listen:
            engine.tap = lambda *a: None
        got.append(tt.run_in_process(engine, steps))
    for key, row in got[0].items():
        assert float(np.abs(row - got[1][key]).max()) < 1e-5 * max(1.0, float(np.abs(row).max())), key


def test_passes_keep_caches_and_states_of_their_own_and_share_weights(tmp_path_factory):
    engine = _engine(_model_dir("a", tmp_path_factory), "float32", n_pages=8)
    runs = engine.model.runs
    assert [r.layer for r in runs] == [0, 1, 2, 1, 2, 1, 2, 3] and len({r.cache_layer for r in runs}) == 8
    assert [r.stream_input for r in runs] == [False, False, False, True, False, True, False, False]
    assert engine.model.layers[4] is engine.model.layers[1] and engine.model.layers[7] is engine.model.layers[2]
    assert sorted(engine.layer_state) == [1, 3, 4, 6] and sorted(engine.layer_pages) == [0, 2, 5, 7]
    assert len({t.data_ptr() for t in engine.layer_state.values()}) == 4


def test_long_decoding_under_graphs(tmp_path_factory):
    """170 tokens decoded one by one after a 12-token prompt, over page borders; CUDA graphs replay the steps."""
    toks = tc.random_tokens(182, 211, 77)
    for dtype in ("float32", "bfloat16"):
        case = _case("a", dtype)
        folder = _model_dir(case, tmp_path_factory)
        w, cfg = pk.load(folder)
        want = {"r": pk.forward(w, cfg, toks).numpy()}
        tol = _tolerance(case, folder, dtype) if dtype == "float32" else _bound(want, {"r": pk.forward(w, cfg, toks, rnd=pk.bf16).numpy()}, 0.0)
        engine = _engine(folder, dtype, n_pages=12)
        got = tt.run_in_process(engine, tt.trace_tail_decode({"r": toks}, tail=170))
        tt.compare(got, want, tol, f"long decoding {dtype}")
        assert engine.graph_replays > 100 and _all_free(engine)


def test_state_slots_start_from_zero_when_they_are_used_again(tmp_path_factory):
    folder = _model_dir("c", tmp_path_factory)
    reqs = _requests("c")
    engine = _engine(folder, "float32", n_pages=10, max_requests=1)
    plain = _plain("c", folder)
    for rid in ("r0", "r4", "r2", "r0"):
        got = tt.run_in_process(engine, tt.trace_portions({rid: reqs[rid]}, sizes=(9, 2, 40)))
        tt.compare(got, plain, _tolerance("c", folder, "float32"), f"request {rid} on the one slot")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine_and_its_scheduler(dtype, tmp_path_factory):
    from geneinfer_b200 import Engine
    folder = _model_dir(_case("b", dtype), tmp_path_factory)
    w, cfg = pk.load(folder)
    prompts = [tc.random_tokens(n, 300, 900 + n) for n in (5, 40, 1, 18, 9)]
    engine = Engine(folder, dtype=dtype, max_seq_len=256, max_running=3, kv_pages=60, step_tokens=32, prefill_chunk=16)
    got = engine.generate(prompts, max_new_tokens=10, temperature=0.0)
    for prompt, gen in zip(prompts, got):
        assert len(gen) == 10
        tokens = list(prompt)
        for k, t in enumerate(gen):
            logits = pk.forward(w, cfg, tokens)[-1].numpy()
            best = int(np.argmax(logits))
            if t != best:                 # only a near-tie may differ
                assert float(logits[best] - logits[t]) < (1e-4 if dtype == "float32" else 2e-2) * float(np.abs(logits).max()), (k, t, best)
            tokens.append(t)
    assert engine.stats.max_running_seen == 3 and engine.steps.cache.slots.free_count == 3


def test_generation_with_preemption_gives_the_same_tokens(tmp_path_factory):
    """A pool too small for all running requests: the scheduler gives up and recomputes some, states included."""
    from geneinfer_b200 import Engine
    folder = _model_dir("b", tmp_path_factory)
    prompts = [tc.random_tokens(n, 300, 40 + n) for n in (50, 44, 61)]
    plenty = Engine(folder, dtype="float32", max_seq_len=128, max_running=3, kv_pages=40).generate(prompts, max_new_tokens=40, temperature=0.0)
    engine = Engine(folder, dtype="float32", max_seq_len=128, max_running=3, kv_pages=14)
    assert engine.generate(prompts, max_new_tokens=40, temperature=0.0) == plenty
    assert engine.stats.preemptions > 0


@pytest.mark.parametrize("page_size", [8, 12, 64])
def test_other_page_sizes(page_size, tmp_path_factory):
    from geneinfer_b200.engine.loading import load_model
    from geneinfer_b200.engine.step import StepEngine
    for dtype in ("float32", "bfloat16"):
        case = _case("b", dtype)
        folder = _model_dir(case, tmp_path_factory)
        reqs = {k: v for k, v in list(_requests(case).items())[:3]}
        steps = tt.trace_mixed(reqs, seed=2, tail=20)
        model = load_model(folder, dtype=dtype, max_position=384)
        engine = StepEngine(model, page_size=page_size, n_pages=tt.max_tokens_of(steps, reqs, 64) // page_size + 8, max_requests=4,
                            max_step_tokens=512, debug_checks=True)
        got = tt.run_in_process(engine, steps)
        engine.check_status()
        tt.compare(got, _plain(case, folder), _tolerance(case, folder, dtype), f"page size {page_size} {dtype}")


def test_trace_replay_tool_and_command_line(tmp_path, tmp_path_factory):
    folder = _model_dir("d", tmp_path_factory)
    reqs = {k: v for k, v in list(_requests("d").items())[1:5]}
    steps = tt.trace_mixed(reqs, seed=5, max_live=2, tail=6)
    got = tt.run_trace_tool(folder, "float32", steps, tt.max_tokens_of(steps, reqs), str(tmp_path / "out"), 77)
    tt.compare(got, _plain("d", folder), _tolerance("d", folder, "float32"), "trace replay")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "gi_generate"), "--model", folder, "--prompt-ids", "5 9 2 70",
                        "--steps", "12", "--temperature", "0", "--no-echo", "--dtype", "fp32", "--max-seq-len", "64"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    out = [int(t) for t in p.stdout.split()]
    w, cfg = pk.load(folder)
    tokens = [5, 9, 2, 70]
    for t in out[:4]:
        logits = pk.forward(w, cfg, tokens)[-1].numpy()
        assert t == int(np.argmax(logits)) or float(logits.max() - logits[t]) < 1e-4
        tokens.append(t)
    assert len(out) == 9


def _random_config(seed):
    """A configuration drawn from a seed: sizes, layer order, loop and constants all differ from case to case."""
    import random
    r = random.Random(seed)
    width = r.choice([64, 72, 96, 160, 176, 320, 90])
    layers = []
    for _ in range(r.randint(1, 5)):
        mlp = None
        if r.random() < 0.8:
            experts = r.randint(1, 12)
            mlp = kc.dense(r.choice([50, 96, 260])) if r.random() < 0.3 else \
                kc.moe(r.choice([16, 40, 64, 100]), experts, r.randint(1, experts), r.choice([None, 24, 80, 136]))
        kind = r.choice(["retention", "attention", "latent"])
        if kind == "retention":
            heads = r.randint(1, 6)
            layers.append(kc.retention(heads, r.choice([8, 16, 32, 44, 64, 130]), r.choice([8, 20, 32, 64, 100]),
                                       [r.choice([0.5, 0.9, 0.99, 0.999, 0.9999]) for _ in range(heads)], mlp))
        elif kind == "attention":
            kv, dim = r.choice([1, 2, 3]), r.choice([8, 16, 20, 32, 48, 64, 128])
            layers.append(kc.attention(kv * r.choice([1, 2, 4, 8]), kv, dim, r.choice([dim, 16, 48, 64, 96]), r.choice([0.08, 0.125, 0.4]),
                                       r.choice([100.0, 10000.0, 500000.0]), r.choice([2, dim // 4 * 2, dim]), r.choice([None, 2.0, 7.5]), mlp))
        else:
            layers.append(kc.latent(r.choice([1, 3, 8, 16, 18]), r.choice([8, 20, 32, 64]), r.choice([2, 8, 16, 32]), r.choice([8, 24, 64, 72]),
                                    r.choice([16, 36, 64, 128, 192]), r.choice([0.08, 0.15, 0.3]), r.choice([100.0, 10000.0, 500000.0]),
                                    r.choice([None, (4.0, 64, 32.0, 1.0), (16.0, 4096, 16.0, 0.7), (2.0, 17, 3.0, 2.9)]), mlp))
    n = len(layers)
    loop = None
    if r.random() < 0.7:
        start = r.randint(0, n - 1)
        loop = (start, r.randint(start + 1, n), r.randint(1, 3))
    return kc.model(width, r.randint(50, 600), r.choice([1e-6, 1e-5, 1e-3]), layers, logit_scale=r.choice([None, 0.5, 3.0]), loop=loop)


@pytest.mark.parametrize("seed", range(int(os.environ.get("GENEINFER_TEST_SEEDS", "12"))))
def test_random_configurations_under_a_mixed_trace(seed, tmp_path):
    for dtype in ("float32", "bfloat16"):
        config = _random_config(seed)
        if dtype == "bfloat16":
            config = _all_chosen(config)
        folder = kc.make_model_dir(config, 100 + seed, str(tmp_path / dtype))
        w, cfg = pk.load(folder)
        reqs = {f"r{i}": tc.random_tokens(n, config["vocab"], 700 + 10 * seed + i) for i, n in enumerate([130, 3, 61, 1, 200, 18])}
        exact = {rid: pk.forward(w, cfg, toks).numpy() for rid, toks in reqs.items()}
        other = {rid: pk.forward(w, cfg, toks, *((torch.float32,) if dtype == "float32" else (F, pk.bf16))).double().numpy() for rid, toks in reqs.items()}
        tol = _bound(exact, other, 3e-5, 8.0) if dtype == "float32" else _bound(exact, other, 0.0, 4.0)
        steps = tt.trace_mixed(reqs, seed=seed, tail=10)
        engine = _engine(folder, dtype, tt.max_tokens_of(steps, reqs, 16) // 16)
        got = tt.run_in_process(engine, steps)
        engine.check_status()
        tt.compare(got, exact, tol, f"random configuration {seed} {dtype}: {config}")
        assert _all_free(engine)
