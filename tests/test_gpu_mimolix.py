"""Mimolix on the GPU against the plain implementation in plain_mimolix.py: each kernel and each mechanism alone, then
whole models through the step engine under different cuts of the same requests (whole prompts, token-by-token decoding,
portions down to two tokens, mixed batches on reused pages and state slots), keys made to stand out far back, at page
borders and in one score map only, writes that a state must keep or replace, the first tokens of a sequence, and greedy
generation through the engine's own entry point and scheduler."""
import copy
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import mimolix_configs as mc
import plain_mimolix as px
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


def _close(got, want, dtype, what, f32=2e-5, b16=2e-2):
    err = float((got.double() - want.double()).abs().max() / max(1.0, float(want.abs().max())))
    assert err < (f32 if dtype is torch.float32 else b16), f"{what}: {err}"


def _mat(rows, cols, g, std=0.3):
    return _bf(torch.randn(rows, cols, generator=g) * std)


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [200, 7, 1026, 4500])
def test_layer_norm_kernel(dtype, D):
    """A mean far from zero (a variance taken from sums of squares would lose it), gathered rows, odd widths, more than a
    block keeps in registers."""
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(D)
    x = torch.randn(9, D, generator=g) * 2 + torch.tensor([0.0, 50.0, -300.0] * 3)[:, None]
    w, b = 1 + 0.3 * torch.randn(D, generator=g), torch.randn(D, generator=g)
    want = px.layer_norm(x.double(), w, b, EPS)
    out = torch.full((9, D), float("nan"), dtype=dtype, device=DEV)
    kernels.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), out, EPS)
    _close(out.cpu().float(), want, dtype, "layer norm", f32=3e-5, b16=1e-2)
    rows = torch.tensor([8, 0, 3, 3], dtype=torch.int32)
    some = torch.full((4, D), float("nan"), dtype=dtype, device=DEV)
    kernels.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), some, EPS, rows=rows.to(DEV))
    assert torch.equal(some, out[rows.long().to(DEV)])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [200, 7, 4500])
def test_end_of_a_layer_with_a_layer_norm_or_a_hand_over(dtype, D):
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(D + 1)
    T, m = 5, 0.37
    x, y, start = torch.randn(T, D, generator=g) + 3, torch.randn(T, D, generator=g), torch.randn(T, D, generator=g)
    w, b = torch.randn(D, generator=g), torch.randn(D, generator=g)
    fresh = x.double() + m * y.double()
    xd, yd = x.to(DEV).clone(), y.to(DEV).clone()
    xn = torch.full((T, D), float("nan"), dtype=dtype, device=DEV)
    kernels.depth_mix(xd, yd, m, next_weight=w.to(DEV), next_bias=b.to(DEV), eps=EPS, xn_out=xn)
    _close(xd.cpu(), fresh, torch.float32, "stream", f32=1e-6)
    _close(xn.cpu().float(), px.layer_norm(fresh, w, b, EPS), dtype, "next layer's input", f32=5e-6, b16=1e-2)
    assert not yd.any()
    alone = torch.empty_like(xn)
    kernels.layer_norm(xd, w.to(DEV), b.to(DEV), alone, EPS)
    assert torch.equal(alone, xn)                      # the same arithmetic in either kernel
    # the stream handed over to a product, which adds to ``start``
    xd, yd = x.to(DEV).clone(), y.to(DEV).clone()
    kernels.depth_mix(xd, yd, m, handover=start.to(DEV), xn_out=xn)
    assert torch.equal(xd.cpu(), start) and not yd.any()
    _close(xn.cpu().float(), fresh, dtype, "stream as the product reads it", f32=1e-6, b16=1e-2)
    xd = x.to(DEV).clone()
    kernels.take_stream(xd, start.to(DEV), xn)
    assert torch.equal(xd.cpu(), start) and torch.equal(xn.cpu(), x.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("more", [0, 5])
@pytest.mark.parametrize("H, G, dim, vd, temp", [(4, 2, 16, 24, (0.5, 3)), (2, 2, 7, 10, None), (6, 1, 40, 96, (0.3, 1)), (2, 1, 128, 64, (-0.1, 2.5))])
def test_maps_norm_and_store(dtype, H, G, dim, vd, temp, more):
    """``more``: how much wider the rows of queries and keys (values: twice that) are than what they hold."""
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(H * 7 + dim)
    T, page = 11, 4
    ld = 2 * (H + G) * dim + G * vd + 3
    proj = torch.randn(T, ld, generator=g) * 2
    qw, kw = torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    tables = torch.tensor([[2, 0, 1]], dtype=torch.int32)
    w, wv = 2 * dim + more, vd + 2 * more
    q = torch.full((T, 2 * H * w), float("nan"), dtype=dtype, device=DEV)
    kc, vc = (torch.full((3, G, page, n), float("nan"), dtype=dtype, device=DEV) for n in (w, wv))
    kernels.maps_norm_store(proj.to(DEV), 3, 3 + 2 * H * dim, 3 + 2 * (H + G) * dim, qw.to(DEV), kw.to(DEV), EPS, temp,
                            torch.arange(T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV), tables.to(DEV), q,
                            kc, vc, H, G, dim, vd, page)
    pq = px.unit_rms(proj[:, 3:3 + 2 * H * dim].double().view(T, H, 2, dim), EPS) * qw
    pk = px.unit_rms(proj[:, 3 + 2 * H * dim:3 + 2 * (H + G) * dim].double().view(T, G, 2, dim), EPS) * kw
    if temp:
        pq = pq * px.query_temperature(T, *temp, F)[:, None, None, None]
    rows = torch.zeros(T, H, 2, w, dtype=F)
    rows[:, :, 0, :dim], rows[:, :, 1, dim:2 * dim] = pq[:, :, 0], pq[:, :, 1]
    _close(q.cpu().float().view(T, H, 2, w), rows, dtype, "query rows", f32=5e-6, b16=1e-2)
    order = [2, 0, 1]
    keys = torch.stack([kc[order[t // page], :, t % page].cpu().float() for t in range(T)])
    vals = torch.stack([vc[order[t // page], :, t % page].cpu().float() for t in range(T)])
    pad = torch.nn.functional.pad
    _close(keys, pad(pk.reshape(T, G, 2 * dim), (0, more)), dtype, "keys in their pages", f32=5e-6, b16=1e-2)
    _close(vals, pad(proj[:, 3 + 2 * (H + G) * dim:].view(T, G, vd), (0, 2 * more)), dtype, "values in their pages", f32=1e-7, b16=1e-2)


@pytest.mark.parametrize("out_dtype", DTYPES)
@pytest.mark.parametrize("in_dtype", DTYPES)
@pytest.mark.parametrize("H, vd", [(3, 24), (1, 7), (5, 128), (2, 500)])
def test_maps_combine(in_dtype, out_dtype, H, vd):
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(vd)
    a = torch.randn(6, H, 2, vd + 3, generator=g).to(in_dtype)           # rows wider than what they hold
    out = torch.full((6, H * vd), float("nan"), dtype=out_dtype, device=DEV)
    kernels.maps_combine(a.view(6, -1).to(DEV), out, 0.83, 1e-3, 0.4, H)
    want = px.difference_of_maps(a[:, :, 0, :vd].double(), a[:, :, 1, :vd].double(), 0.83, 0.6, 1e-3)
    _close(out.cpu().float(), want.reshape(6, -1), out_dtype, "difference of the maps", f32=3e-6, b16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E, top, D", [(5, 2, 40), (40, 7, 96), (3, 3, 17), (1, 1, 24), (300, 12, 64)])
def test_softmax_routing_with_renormalised_weights(dtype, E, top, D):
    from geneinfer_b200.ops import kernels
    g = torch.Generator().manual_seed(E)
    T = 21
    x, w = torch.randn(T, D, generator=g).to(dtype), torch.randn(E, D, generator=g) * 0.6
    tm = kernels.grouped_tile_rows()
    tiles = kernels.route_tiles(T, top, E)
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    srt, grp, cnt = (torch.empty(n, dtype=torch.int32, device=DEV) for n in (tiles * tm, tiles, 1))
    kernels.route(x.to(DEV), w.to(DEV), None, top, ids, wts, srt, grp, cnt, scores="softmax", renormalise=True, factor=1.7)
    want_ids, want_w = px.route({"router": w}, "", {"top": top, "scale": 1.7}, x.double(), F, px.ident)
    assert torch.equal(ids.cpu().long().sort(1).values, want_ids.sort(1).values)
    got = torch.zeros(T, E, dtype=F).scatter_(1, ids.cpu().long(), wts.cpu().double())
    _close(got, torch.zeros(T, E, dtype=F).scatter_(1, want_ids, want_w), torch.float32, "weights", f32=5e-6)


@pytest.mark.parametrize("M", [1, 9, 40, 100, 130, 300])
@pytest.mark.parametrize("N, K", [(96, 64), (300, 200), (72, 1024), (20, 40), (513, 72)])
def test_product_with_the_squared_relu_in_its_epilogue(M, N, K):
    from geneinfer_b200.ops import kernels
    from geneinfer_b200.ops.linear import Linear
    g = torch.Generator().manual_seed(M + N)
    a, w = _bf(torch.randn(M, K, generator=g)), _mat(N, K, g, K ** -0.5)
    lin = Linear(w, torch.bfloat16, DEV)
    out = torch.full((M, N), float("nan"), dtype=torch.bfloat16, device=DEV)
    kernels.gemm_tc(a.to(DEV).bfloat16(), lin.weight, out, w_tiles=lin.weight_tiles, act="relu2")
    want = torch.relu(a.double() @ w.double().T) ** 2
    _close(out.cpu().float(), want, torch.bfloat16, f"{M} x {N} x {K}", b16=1e-2)
    assert kernels.gemm_tc_status(DEV) == 0


def _experts(D, f, g, p=""):
    w = {p + "router": _mat(f["router"]["experts"], D, g)}
    for e in range(f["router"]["experts"]):
        w[f"{p}e{e}.up"], w[f"{p}e{e}.down"] = _mat(f["expert"]["ff"], D, g, 0.2), _mat(D, f["expert"]["ff"], g, 0.2)
    if f.get("shared"):
        w[p + "shared.up"], w[p + "shared.down"] = _mat(f["shared"]["ff"], D, g, 0.2), _mat(D, f["shared"]["ff"], g, 0.2)
    return w


def _experts_part(D, f, w, dtype, p=""):
    from geneinfer_b200.parts import FEED_FORWARDS
    E = f["router"]["experts"]
    weights = {"router": w[p + "router"], "w_up": torch.stack([w[f"{p}e{e}.up"] for e in range(E)]),
               "w_down": torch.stack([w[f"{p}e{e}.down"] for e in range(E)])}
    shared = None
    if f.get("shared"):
        weights["shared.w_up"], weights["shared.w_down"] = w[p + "shared.up"], w[p + "shared.down"]
        shared = {"hidden_size": D, "intermediate_size": f["shared"]["ff"], "activation": "relu2"}
    return FEED_FORWARDS["routed_experts"]({"hidden_size": D, "intermediate_size": f["expert"]["ff"], "experts": E, "top": f["router"]["top"],
                                            "gated": False, "activation": "relu2", "scores": "softmax", "renormalise": True,
                                            "router_scale": f["router"].get("scale", 1.0), "shared": shared}, weights, _build(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 6, 150])
@pytest.mark.parametrize("D, f", [(64, mc.moe(40, 5, 2, 1.5, 56)), (72, mc.moe(24, 7, 3, 0.8)), (100, mc.moe(30, 3, 1, None, 20)),
                                  (96, mc.moe(96, 4, 4, 2.0, 64)), (48, mc.moe(20, 33, 6, 1.0, 12))])
def test_squared_relu_experts(dtype, T, D, f):
    """Few pairs (tiles on the CUDA cores) and many (the tensor cores, where the sizes allow it), with and without a shared expert."""
    g = torch.Generator().manual_seed(D + T)
    w = _experts(D, f, g)
    h = _bf(torch.randn(T, D, generator=g))
    part = _experts_part(D, f, w, dtype)
    ctx = StateCtx(dtype, 1)
    y = torch.randn(T, D, generator=g)
    yd = y.to(DEV).clone()
    part.forward(ctx, h.to(DEV).to(dtype), yd)
    want = px.feed_forward(w, "", f, h.double(), F, px.ident if dtype is torch.float32 else px.bf16)
    _close(yd.cpu() - y, want, dtype, f"experts, {T} tokens", b16=2e-2)


# ------------------------------------------------------------------------------------------ the recurrence alone
def _delta_inputs(n, H, G, dk, dv, g, pad=0):
    C = 2 * G * dk + H * dv
    return torch.randn(n, C + 2 * H + pad, generator=g)


def _plain_delta(rows, conv, a_log, dt_bias, H, G, dk, dv, q_scale):
    T, C = rows.shape[0], conv.shape[0]
    x = px.silu(px.short_conv(rows[:, :C].double(), conv))
    share = torch.arange(H) // (H // G)
    q = px.unit_vector(x[:, :G * dk].reshape(T, G, dk))[:, share] * q_scale
    k = px.unit_vector(x[:, G * dk:2 * G * dk].reshape(T, G, dk))[:, share]
    beta = torch.sigmoid(rows[:, C:C + H].double())
    decay = torch.exp(-torch.exp(a_log.double()) * px.softplus(rows[:, C + H:C + 2 * H].double() + dt_bias.double()))
    return px.delta_rule(q, k, x[:, 2 * G * dk:].reshape(T, H, dv), beta, decay)


def _run_delta(seqs, cuts, conv, a_log, dt_bias, H, G, dk, dv, q_scale, slots, blocks=None, lead=5):
    """Feeds the rows of ``seqs`` through the kernel under ``cuts``; returns outputs and the whole state tensor."""
    from geneinfer_b200.ops import kernels
    C, taps = conv.shape
    floats = lead + H * dk * dv
    floats += -floats % 4
    state = torch.zeros(max(slots) + 2, floats + (taps - 1) * C, device=DEV)
    at, got = [0] * len(seqs), [[] for _ in seqs]
    for lengths in cuts:
        live = [r for r, n in enumerate(lengths) if n]
        rows = torch.cat([seqs[r][at[r]:at[r] + lengths[r]] for r in live]).to(DEV)
        T = rows.shape[0]
        starts = np.cumsum([0] + [lengths[r] for r in live])
        row_req = torch.cat([torch.full((lengths[r],), i) for i, r in enumerate(live)]).int().to(DEV)
        i32 = lambda v: torch.tensor([int(x) for x in v], dtype=torch.int32, device=DEV)
        out = torch.full((T, H * dv), float("nan"), device=DEV)
        qkv, gates = torch.full((T, C), float("nan"), device=DEV), torch.full((T, 2 * H), float("nan"), device=DEV)
        in_blocks = kernels.gated_delta_in_blocks(T, len(live)) if blocks is None else blocks
        coefs = torch.full((T, H, kernels.gated_delta_coefs()), float("nan"), device=DEV) if in_blocks else None
        kernels.gated_delta(rows, 0, C, C + H, conv.to(DEV), a_log.to(DEV), dt_bias.to(DEV), q_scale, state, lead, floats, row_req,
                            i32(starts[:-1]), i32([lengths[r] for r in live]), i32([slots[r] for r in live]), qkv, gates, out, H, G, dk, dv,
                            coefs)
        for i, r in enumerate(live):
            got[r].append(out[starts[i]:starts[i + 1]].cpu())
            at[r] += lengths[r]
    return [torch.cat(o) for o in got], state.cpu()


@pytest.mark.parametrize("H, G, dk, dv, taps", [(4, 2, 16, 24, 3), (3, 3, 40, 33, 1), (6, 1, 64, 64, 4), (2, 2, 100, 20, 5), (2, 1, 128, 96, 2),
                                                (1, 1, 200, 72, 4), (2, 2, 7, 5, 17), (8, 4, 96, 128, 4)])
def test_gated_delta_kernel(H, G, dk, dv, taps):
    """Outputs, the state and the convolution's inputs left in the slots, against the plain recurrence, token by token and in
    blocks of eight (whose last one may not be whole); token by token the same bits whichever way the requests are cut."""
    g = torch.Generator().manual_seed(H * 100 + dk)
    conv = torch.randn(2 * G * dk + H * dv, taps, generator=g) * 0.6
    a_log, dt_bias = torch.rand(H, generator=g) * 2 - 1, torch.randn(H, generator=g) - 2
    lens = [90, 2, 37]
    seqs = [_delta_inputs(n, H, G, dk, dv, g, pad=1) for n in lens]
    args = (conv, a_log, dt_bias, H, G, dk, dv, dk ** -0.5)
    want = [_plain_delta(s, *args) for s in seqs]
    slots = [3, 0, 1]
    base = None
    ragged = [[1, 1, 1], [40, 1, 2], [2, 0, 1], [47, 0, 33]]
    for cuts, blocks in (([[90, 2, 37]], True), ([[90, 2, 37]], False), (ragged, True), (ragged, False), (ragged, None),
                         ([[2, 0, 0], [0, 2, 3]] + [[1, 0, 1]] * 34 + [[54, 0, 0]], None)):
        got, state = _run_delta(seqs, cuts, *args, slots, blocks)
        for r in range(3):
            _close(got[r], want[r][0].reshape(lens[r], H * dv), torch.float32, f"outputs of request {r}, {len(cuts)} steps", f32=1e-5)
            _close(state[slots[r], 5:5 + H * dk * dv], want[r][1].reshape(-1), torch.float32, f"state of request {r}", f32=1e-5)
            if taps > 1:
                kept = torch.zeros(taps - 1, conv.shape[0])
                tail = seqs[r][-(taps - 1):, :conv.shape[0]]
                kept[taps - 1 - tail.shape[0]:] = tail
                assert torch.equal(state[slots[r], -(taps - 1) * conv.shape[0]:].view(taps - 1, -1), kept)
        assert not state[:, :5].any() and not state[2].any() and not state[4].any()
        if blocks is False:
            base = base or (got, state)
            assert all(torch.equal(a, b) for a, b in zip(got, base[0])) and torch.equal(state, base[1])


def test_gated_delta_remembers_replaces_and_forgets():
    """Written by hand: token 3 writes a value under a key that token 250 reads back from a head that does not fade; token 120
    writes another value under the same key in a second sequence and replaces it; a fading head has lost it."""
    H, G, dk, dv, n = 2, 2, 16, 16, 251
    g = torch.Generator().manual_seed(3)
    C = 2 * G * dk + H * dv
    conv = torch.zeros(C, 2)
    conv[:, 1] = 1.0
    rows = torch.zeros(n, C + 2 * H)
    rows[:, C:C + H] = -30.0                                    # beta = 0: nothing is written ...
    rows[:, C + H:] = torch.tensor([-30.0, 0.0])               # head 0 keeps, head 1 fades
    rows[:, :2 * G * dk] = torch.randn(n, 2 * G * dk, generator=g) * 0.1
    key = torch.full((dk,), -40.0)
    key[5] = 6.0
    val = torch.randn(H * dv, generator=g) + 3

    def write(r, t, v):
        r[t, G * dk:2 * G * dk] = key.repeat(G)
        r[t, 2 * G * dk:C] = v
        r[t, C:C + H] = 30.0                                   # ... but where a step is 1
    write(rows, 3, val)
    rows[n - 1, :G * dk] = key.repeat(G)
    other = rows.clone()
    write(other, 120, -val)
    args = (conv, torch.zeros(H), torch.zeros(H), H, G, dk, dv, 1.0)
    for cuts in ([[n, n]], [[200, 1]] + [[1, 1]] * 51 + [[0, 199]], [[3, 2], [2, 119], [129, 3], [117, 127]]):
        got, _ = _run_delta([rows, other], cuts, *args, [1, 0])
        last = [o[-1].view(H, dv) for o in got]
        assert torch.allclose(last[0][0], px.silu(val[:dv]), rtol=1e-4, atol=1e-4)
        assert torch.allclose(last[1][0], px.silu(-val[:dv]), rtol=1e-4, atol=1e-4)
        assert float(last[0][1].abs().max()) < 1e-6
        for o, r in zip(got, (rows, other)):
            _close(o, _plain_delta(r, *args)[0].reshape(n, H * dv), torch.float32, "by hand", f32=1e-5)


# ------------------------------------------------------------------------------------------ mixers alone
CUTS = {"whole": [[40, 2, 19]], "token by token": [[1, 1, 1]] * 2 + [[1, 0, 1]] * 17 + [[1, 0, 0]] * 21,
        "portions": [[2, 1, 3], [5, 1, 2], [2, 0, 14], [31, 0, 0]], "tail decoded": [[30, 2, 10]] + [[1, 0, 1]] * 9 + [[1, 0, 0]]}

MAPS = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.5, "diff": 0.4, "q_temp": {"coef": 0.6, "every": 7}}
MAPS_FORMS = [MAPS, dict(MAPS, heads=3, kv_heads=3, dim=10, vdim=14, q_temp=None), dict(MAPS, heads=6, kv_heads=1, dim=24, vdim=64),
              # two maps as wide as the values at the sizes of the tensor-core kernels: 32, 64 and 128 wide rows
              dict(MAPS, heads=4, kv_heads=2, dim=16, vdim=32), dict(MAPS, heads=4, kv_heads=2, dim=32, vdim=64, diff=0.7),
              dict(MAPS, heads=2, kv_heads=1, dim=64, vdim=128, scale=0.2), dict(MAPS, heads=16, kv_heads=1, dim=32, vdim=64),
              # the row-form kernel's sizes: values in whole 64s, rows of two maps in whole 16s
              dict(MAPS, heads=20, kv_heads=2, dim=40, vdim=64), dict(MAPS, heads=8, kv_heads=1, dim=64, vdim=192),
              # widened with zeros in bfloat16: keys to the values' width, values to the keys', both; too narrow to be widened
              dict(MAPS, heads=4, kv_heads=2, dim=20, vdim=64), dict(MAPS, heads=4, kv_heads=4, dim=64, vdim=40),
              dict(MAPS, heads=6, kv_heads=3, dim=36, vdim=80), dict(MAPS, heads=3, kv_heads=1, dim=34, vdim=20),
              dict(MAPS, heads=2, kv_heads=2, dim=136, vdim=200)]


def _maps_weights(D, m, g, p="p."):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {p + "q": _mat(2 * H * d, D, g), p + "k": _mat(2 * G * d, D, g), p + "v": _mat(G * dv, D, g), p + "o": _mat(D, H * dv, g),
         p + "q.norm": 1 + 0.3 * torch.randn(d, generator=g), p + "k.norm": 1 + 0.3 * torch.randn(d, generator=g)}
    w.update({p + n: torch.randn(d, generator=g) * 0.2 for n in ("lq1", "lk1", "lq2", "lk2")})
    return w


def _maps_part(D, m, w, dtype, p="p.", eps=EPS):
    from geneinfer_b200.config import PartSpec
    from geneinfer_b200.parts import MIXERS
    weights = {"w_qkv": torch.cat([w[p + "q"], w[p + "k"], w[p + "v"]]), "w_o": w[p + "o"], "q_norm": w[p + "q.norm"], "k_norm": w[p + "k.norm"]}
    weights.update({n: w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")})
    temp = m.get("q_temp")
    return MIXERS["attention"]({"hidden_size": D, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                                "value_dim": m["vdim"], "scale": m["scale"], "window": None, "position": PartSpec("none", {}), "qk_norm_eps": eps,
                                "maps": 2, "map_weight": m["diff"], "map_factor": 1 - m["diff"],
                                "query_temperature": (temp["coef"], temp["every"]) if temp else None}, weights, _build(dtype))


def _maps_ctx(part, dtype, n, max_len=256, page_size=8):
    need = part.cache_need()
    return StateCtx(dtype, n, Hkv=need.num_kv_heads, hd=need.head_dim, vd=need.value_width, page_size=page_size, max_len=max_len)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", MAPS_FORMS)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_attention_with_two_score_maps(dtype, m, cut):
    D = 40
    g = torch.Generator().manual_seed(9)
    w = _maps_weights(D, m, g)
    part = _maps_part(D, m, w, dtype)
    need = part.cache_need()
    width = next((w for w in (16, 32, 64, 128) if w >= max(2 * m["dim"], m["vdim"])), 0)
    fast = dtype is torch.bfloat16 and width > 0 and width <= 2 * m["dim"] + m["vdim"] and 2 * m["heads"] // m["kv_heads"] <= 16
    assert part.fast == fast and part.row_form != fast
    assert (need.num_kv_heads, need.head_dim, need.value_width) == (m["kv_heads"], *((width, width) if fast else (2 * m["dim"], m["vdim"])))
    inputs = [_bf(torch.randn(n, D, generator=g)) for n in (40, 2, 19)]
    rnd = px.ident if dtype is torch.float32 else px.bf16
    want = [px.attention_mixer(w, "p.", m, x.double(), EPS, F, rnd) for x in inputs]
    got = _run_mixer(part, _maps_ctx(part, dtype, 3), inputs, CUTS[cut], dtype, D)
    for r in range(3):
        _close(got[r], want[r], dtype, f"two maps, request {r}, {cut}", b16=3e-2)


def _sharp_maps(m, D, n, key, query, which, g):
    """Weights and inputs with one score that stands out: map ``which`` of the query at ``query`` answers the key at ``key``."""
    w = _maps_weights(D, m, g)
    x = _bf(torch.randn(n, D, generator=g) * 0.3)
    x[:, 0] = x[:, 1] = 0.0
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    w["p.q"], w["p.k"] = w["p.q"] * 0.02, w["p.k"] * 0.02
    w["p.q"][:, 1] = 0.0
    w["p.k"][:, 0] = 0.0
    w["p.q"].view(H, 2, d, D)[:, which, 2, 1] = 8.0
    w["p.k"].view(G, 2, d, D)[:, which, 2, 0] = 8.0
    w["p.q.norm"], w["p.k.norm"] = torch.full((d,), 2.0), torch.full((d,), 2.0)
    x[key, 0] = 3.0
    x[query, 1] = 3.0
    return w, x


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("back", [0, 1, 15, 16, 17, 255, 256, 650])
@pytest.mark.parametrize("form", [0, 1, 2])
def test_one_key_among_hundreds_in_one_map(dtype, which, back, form):
    """The last query answers one key, in one map only, far back, at a page border, at the border of a decode chunk or its own,
    as the end of a prompt and decoded."""
    D, n = 24, 700
    m = [dict(MAPS, heads=2, kv_heads=1, scale=1.0, q_temp=None), dict(MAPS, heads=4, kv_heads=2, dim=32, vdim=64, scale=0.7, q_temp=None),
         dict(MAPS, heads=4, kv_heads=1, dim=24, vdim=64, scale=0.8, q_temp=None)][form]
    g = torch.Generator().manual_seed(15)
    w, x = _sharp_maps(m, D, n, n - 1 - back, n - 1, which, g)
    rnd = px.ident if dtype is torch.float32 else px.bf16
    want = px.attention_mixer(w, "p.", m, x.double(), EPS, F, rnd)
    moved = x.clone()
    moved[n - 1 - back, 0] = 0.0
    assert float((px.attention_mixer(w, "p.", m, moved.double(), EPS, F, rnd)[-1] - want[-1]).abs().max()) > 0.1 * float(want[-1].abs().max())
    part = _maps_part(D, m, w, dtype)
    for cuts in ([[n - 30]] + [[1]] * 30, [[300], [398], [2]]):
        got = _run_mixer(part, _maps_ctx(part, dtype, 1, max_len=704, page_size=16), [x], cuts, dtype, D)
        _close(got[0][-1], want[-1], dtype, f"key {back} back among {n}, map {which}, {len(cuts)} steps", b16=4e-2)


def test_query_temperature_steps_at_block_ends():
    """A large factor per block: one position off at a block's end changes the row."""
    D, n = 32, 40
    m = dict(MAPS, q_temp={"coef": 2.5, "every": 8})
    g = torch.Generator().manual_seed(21)
    w = _maps_weights(D, m, g)
    x = _bf(torch.randn(n, D, generator=g))
    want = px.attention_mixer(w, "p.", m, x.double(), EPS, F, px.ident)
    assert px.query_temperature(17, 2.5, 8, F).tolist() == [1.0] * 7 + [1 + 2.5 * math.log(2)] * 8 + [1 + 2.5 * math.log(3)] * 2
    part = _maps_part(D, m, w, torch.float32)
    for cuts in ([[n]], [[7], [1], [1], [6], [2], [23]], [[1]] * n):
        got = _run_mixer(part, _maps_ctx(part, torch.float32, 1), [x], cuts, torch.float32, D)
        _close(got[0], want, torch.float32, f"temperature, {len(cuts)} steps")


DELTA = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 40, "conv": 3}


def _delta_weights(D, m, g, p="p."):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {p + "b": _mat(H, D, g), p + "a": _mat(H, D, g), p + "g": _mat(H * dv, D, g), p + "o": _mat(D, H * dv, g),
         p + "A_log": torch.rand(H, generator=g) * 2 - 1, p + "dt_bias": torch.randn(H, generator=g) - 2,
         p + "norm": 1 + 0.2 * torch.randn(dv, generator=g)}
    for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
        w[p + n], w[p + n + ".conv"] = _mat(rows, D, g), torch.randn(rows, m["conv"], generator=g) * 0.6
    return w


def _delta_part(D, m, w, dtype, p="p."):
    from geneinfer_b200.parts import MIXERS
    return MIXERS["gated_delta"](
        {"hidden_size": D, "num_heads": m["heads"], "num_key_heads": m["kv_heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
         "conv_taps": m["conv"], "norm_eps": EPS},
        {"w_in": torch.cat([w[p + n] for n in ("q", "k", "v", "g", "b", "a")]), "conv": torch.cat([w[p + n + ".conv"] for n in ("q", "k", "v")]),
         "a_log": w[p + "A_log"], "dt_bias": w[p + "dt_bias"], "norm": w[p + "norm"], "w_o": w[p + "o"]}, _build(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [DELTA, dict(DELTA, heads=3, kv_heads=1, dim=64, vdim=64, conv=4), dict(DELTA, heads=3, kv_heads=3, dim=20, vdim=9, conv=1),
                               dict(DELTA, heads=2, kv_heads=2, dim=128, vdim=128, conv=5)])
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_gated_delta_mixer(dtype, m, cut):
    D = 48
    g = torch.Generator().manual_seed(4)
    w = _delta_weights(D, m, g)
    part = _delta_part(D, m, w, dtype)
    C = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]
    assert part.state_need().shape == (m["heads"] * m["dim"] * m["vdim"] + (m["conv"] - 1) * C,) and part.cache_need() is None
    inputs = [_bf(torch.randn(n, D, generator=g)) for n in (40, 2, 19)]
    rnd = px.ident if dtype is torch.float32 else px.bf16
    want = [px.delta_mixer(w, "p.", m, x.double(), EPS, F, rnd) for x in inputs]
    got = _run_mixer(part, StateCtx(dtype, 3, state_floats=part.state_need().shape[0]), inputs, CUTS[cut], dtype, D)
    for r in range(3):
        _close(got[r], want[r], dtype, f"delta mixer, request {r}, {cut}", f32=4e-5, b16=3e-2)


@pytest.mark.parametrize("cuts", [[[1], [1], [1], [1], [5]], [[2], [2], [5]], [[9]], [[3], [1], [5]]])
def test_the_first_tokens_see_zeros_before_the_sequence_through_the_convolution(cuts):
    D, m = 24, dict(DELTA, conv=5)
    g = torch.Generator().manual_seed(13)
    w = _delta_weights(D, m, g)
    x = _bf(torch.randn(9, D, generator=g))
    want = px.delta_mixer(w, "p.", m, x.double(), EPS, F, px.ident)
    part = _delta_part(D, m, w, torch.float32)
    got = _run_mixer(part, StateCtx(torch.float32, 1, state_floats=part.state_need().shape[0]), [x], cuts, torch.float32, D)
    _close(got[0], want, torch.float32, f"first tokens, cuts {cuts}", f32=4e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_in_one_batch_equal_each_alone(dtype):
    """Three unequal requests batched against each alone, on scattered pages and other state slots: the same bits (the
    recurrence may run in blocks of tokens in one and token by token in the other: equal but for rounding)."""
    D = 40
    g = torch.Generator().manual_seed(17)
    fast = dict(MAPS, dim=32, vdim=64)
    fast_part, maps_part = (_maps_part(D, m, _maps_weights(D, m, g), dtype) for m in (fast, MAPS))
    delta_part = _delta_part(D, DELTA, _delta_weights(D, DELTA, g), dtype)
    for part, ctx_of in ((maps_part, lambda n: _maps_ctx(maps_part, dtype, n)), (fast_part, lambda n: _maps_ctx(fast_part, dtype, n)),
                         (delta_part, lambda n: StateCtx(dtype, n, state_floats=delta_part.state_need().shape[0]))):
        inputs = [_bf(torch.randn(n, D, generator=g)) for n in (33, 5, 12)]
        together = _run_mixer(part, ctx_of(3), inputs, [[20, 1, 3], [1, 1, 2], [12, 3, 7]], dtype, D)
        for r in range(3):
            alone = _run_mixer(part, ctx_of(1), [inputs[r]], [[[20, 1, 3][r]], [[1, 1, 2][r]], [[12, 3, 7][r]]], dtype, D)
            if part is delta_part:
                _close(alone[0], together[r], dtype, f"request {r} in a batch", f32=1e-5, b16=1e-2)
            else:
                assert torch.equal(alone[0], together[r]), f"request {r} depends on its batch"


# ------------------------------------------------------------------------------------------ whole models
_TMP = {}
LENGTHS = {"a": [1, 2, 3, 75, 20, 120, 47, 30], "b": [150, 4, 64, 1, 180], "c": [90, 2, 33, 1, 140, 17], "d": [1, 2, 100, 30, 7]}
CONFIGS = {"a": mc.MIM_A, "b": mc.MIM_B, "c": mc.MIM_C, "d": mc.MIM_D}


def _all_chosen(config):
    """The same model with every expert chosen. With experts left out, rounding may turn a close choice over, in an engine as in
    the plain model with rounded operands; comparisons in bfloat16 that are to hold at every position use this form."""
    config = copy.deepcopy(config)
    for layer in config["layers"]:
        if layer["mlp"]:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return config


def _config(case):
    return _all_chosen(CONFIGS[case[0]]) if case.endswith("all") else CONFIGS[case]


def _model_dir(case, tmp_path_factory):
    if case not in _TMP:
        _TMP[case] = mc.make_model_dir(_config(case), 20 + ord(case[0]), str(tmp_path_factory.mktemp("mimolix_" + case)))
    return _TMP[case]


def _case(case, dtype):
    return case if dtype == "float32" else case + "_all"


def _requests(case):
    return {f"r{i}": tc.random_tokens(n, CONFIGS[case[0]]["vocab"], 400 + i) for i, n in enumerate(LENGTHS[case[0]])}


_PLAIN = {}


def _plain(case, folder, rounded=False, single=False):
    key = (case, rounded, single)
    if key not in _PLAIN:
        w, cfg = px.load(folder)
        _PLAIN[key] = {rid: px.forward(w, cfg, toks, torch.float32 if single else F, px.bf16 if rounded else px.ident).double().numpy()
                       for rid, toks in _requests(case).items()}
    return _PLAIN[key]


def _bound(exact, other, floor, times=3.0):
    """``times`` the distance between the plain model in two precisions, and at least ``floor``."""
    return max(floor, times * max(tt.rel_err(other[r], exact[r]) for r in exact))


def _tolerance(case, folder, dtype):
    """bfloat16: three times the distance between the exact plain model and the plain model with bfloat16 operands of the matrix
    products. 32-bit: 3e-5, or eight times the distance between the plain model in float64 and in float32 where that is more
    (norms that follow a nearly cancelling difference of maps or read-out raise a position's rounding in any implementation)."""
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
        tt.compare(got, plain, tol, f"Mimolix {case} {dtype} {name}")
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
    w, cfg = px.load(folder)
    toks = tc.random_tokens(45, 211, 6)
    after = []
    px.forward(w, cfg, toks, layers_out=after)
    for sizes in ((45,), (7, 30, 2, 6)):
        engine = _engine(folder, "float32", n_pages=8)
        seen = []

        def tap(tag, layer, tensor, ctx):
            if tag == "ffn_out":
                seen.append((layer, tensor.detach().float().cpu()))
        engine.tap = tap
        tt.run_in_process(engine, tt.trace_portions({"r": toks}, sizes=sizes))
        runs = len(after)
        assert [l for l, _ in seen[:runs]] == [i for i, _ in px.layer_runs(cfg)]
        for i in range(runs):
            got = torch.cat([t for _, t in seen[i::runs]])
            assert float((got.double() - after[i]).abs().max()) < 3e-5 * float(after[i].abs().max()), f"run {i}, portions {sizes}"


def test_passes_keep_caches_and_states_of_their_own_and_share_weights(tmp_path_factory):
    engine = _engine(_model_dir("a", tmp_path_factory), "float32", n_pages=8)
    runs = engine.model.runs
    assert [r.layer for r in runs] == [0, 1, 2, 1, 2, 1, 2, 3] and len({r.cache_layer for r in runs}) == 8
    assert [r.stream_input for r in runs] == [False, True, False, True, False, True, False, False]
    assert engine.model.layers[4] is engine.model.layers[1] and engine.model.layers[7] is engine.model.layers[2]
    assert sorted(engine.layer_state) == [1, 3, 4, 6] and sorted(engine.layer_pages) == [0, 2, 5, 7]
    assert len({t.data_ptr() for t in engine.layer_state.values()}) == 4


def test_long_decoding_under_graphs(tmp_path_factory):
    """170 tokens decoded one by one after a 12-token prompt, over page borders; CUDA graphs replay the steps."""
    toks = tc.random_tokens(182, 211, 77)
    for dtype in ("float32", "bfloat16"):
        case = _case("a", dtype)
        folder = _model_dir(case, tmp_path_factory)
        w, cfg = px.load(folder)
        want = {"r": px.forward(w, cfg, toks).numpy()}
        engine = _engine(folder, dtype, n_pages=12)
        got = tt.run_in_process(engine, tt.trace_tail_decode({"r": toks}, tail=170))
        tt.compare(got, want, _tolerance(case, folder, dtype), f"long decoding {dtype}")
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
    w, cfg = px.load(folder)
    prompts = [tc.random_tokens(n, 300, 900 + n) for n in (5, 40, 1, 18, 9)]
    engine = Engine(folder, dtype=dtype, max_seq_len=256, max_running=3, kv_pages=60, step_tokens=32, prefill_chunk=16)
    got = engine.generate(prompts, max_new_tokens=10, temperature=0.0)
    for prompt, gen in zip(prompts, got):
        assert len(gen) == 10
        tokens = list(prompt)
        for k, t in enumerate(gen):
            logits = px.forward(w, cfg, tokens)[-1].numpy()
            best = int(np.argmax(logits))
            if t != best:                 # only a near-tie may differ
                assert float(logits[best] - logits[t]) < (1e-4 if dtype == "float32" else 8e-2), (k, t, best)
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
    w, cfg = px.load(folder)
    tokens = [5, 9, 2, 70]
    for t in out[:4]:
        logits = px.forward(w, cfg, tokens)[-1].numpy()
        assert t == int(np.argmax(logits)) or float(logits.max() - logits[t]) < 1e-4
        tokens.append(t)
    assert len(out) == 9


def _random_config(seed):
    """A configuration drawn from a seed: sizes, layer order, loop and constants all differ from case to case."""
    import random
    r = random.Random(seed)
    width = r.choice([64, 72, 96, 160, 176, 256, 320, 90])
    layers = []
    for _ in range(r.randint(1, 5)):
        mlp = None
        if r.random() < 0.8:
            experts = r.randint(1, 12)
            mlp = mc.moe(r.choice([16, 40, 64, 100]), experts, r.randint(1, experts), r.choice([None, 0.7, 2.0]), r.choice([None, 24, 80, 136]))
        kv = r.choice([1, 2, 3])
        if r.random() < 0.5:
            dim = r.choice([8, 16, 20, 32, 48, 64])
            layers.append(mc.attention(kv * r.choice([1, 2, 4]), kv, dim, r.choice([2 * dim, 16, 48, 64, 96]), r.choice([0.08, 0.125, 0.4]),
                                       r.choice([0.1, 0.5, 0.8]), temp=r.choice([None, (0.4, 16), (0.2, 50), (1.0, 3)]), mlp=mlp))
        else:
            layers.append(mc.delta(kv * r.choice([1, 2, 3]), kv, r.choice([8, 16, 32, 44, 64, 96, 130]), r.choice([8, 20, 32, 64, 100]),
                                   r.choice([1, 2, 3, 4]), mlp=mlp))
    n = len(layers)
    loop = None
    if r.random() < 0.7:
        start = r.randint(0, n - 1)
        loop = (start, r.randint(start + 1, n), r.randint(1, 3))
    return mc.model(width, r.randint(50, 600), r.choice([1e-6, 1e-5, 1e-3]), layers, scale=r.choice([None, 0.5, 3.0]),
                    mult=r.choice([None, 0.3, 0.7]), loop=loop)


@pytest.mark.parametrize("seed", range(int(os.environ.get("GENEINFER_TEST_SEEDS", "12"))))
def test_random_configurations_under_a_mixed_trace(seed, tmp_path):
    for dtype in ("float32", "bfloat16"):
        config = _random_config(seed)
        if dtype == "bfloat16":
            config = _all_chosen(config)
        folder = mc.make_model_dir(config, 100 + seed, str(tmp_path / dtype))
        w, cfg = px.load(folder)
        reqs = {f"r{i}": tc.random_tokens(n, config["vocab"], 700 + 10 * seed + i) for i, n in enumerate([130, 3, 61, 1, 200, 18])}
        exact = {rid: px.forward(w, cfg, toks).numpy() for rid, toks in reqs.items()}
        other = {rid: px.forward(w, cfg, toks, *((torch.float32,) if dtype == "float32" else (F, px.bf16))).double().numpy() for rid, toks in reqs.items()}
        tol = _bound(exact, other, 3e-5, 8.0) if dtype == "float32" else _bound(exact, other, 0.0)
        steps = tt.trace_mixed(reqs, seed=seed, tail=10)
        engine = _engine(folder, dtype, tt.max_tokens_of(steps, reqs, 16) // 16)
        got = tt.run_in_process(engine, steps)
        engine.check_status()
        tt.compare(got, exact, tol, f"random configuration {seed} {dtype}: {config}")
        assert _all_free(engine)
