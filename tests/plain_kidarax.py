"""A plain, slow implementation of the Kidarax design: whole sequences, no cache, no batching, one function per
mechanism, on the CPU. It is the oracle of the Kidarax tests and shares no code with the engine (its own reading of
config.json, its own loops over tokens).

Notation. The stream x starts as x0 = E[token]; ahead of every pass over the layers of ``loop`` but the first, x0 is added
to it. A layer does x <- x + N1'(mixer(N1(x))) and, with a feed-forward, x <- x + N2'(ff(N2(x))); every N is
tanh(alpha x) w + b with one number alpha per norm. The logits are the embedding table's product with N(x), times a factor.

Every function takes ``dt`` (float64 for an oracle without rounding of its own, float32 otherwise) and ``rnd``,
applied where a bfloat16 engine stores an operand of a matrix product in 16 bits.
"""
from __future__ import annotations

import json
import math
from typing import Dict, List, Optional

import torch

import plain_model as pm


def ident(t):
    return t


def bf16(t):
    return t.to(torch.bfloat16).to(t.dtype)


def load(model_dir: str):
    with open(f"{model_dir}/config.json") as f:
        cfg = json.load(f)
    return pm.read_safetensors_f32(f"{model_dir}/model.safetensors"), cfg


# ------------------------------------------------------------------------------------ small pieces
def tanh_norm(W, name, x):
    dt = x.dtype
    return torch.tanh(W[name + ".alpha"].to(dt) * x) * W[name].to(dt) + W[name + ".b"].to(dt)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def linear(w, h, rnd):
    """W h for every row of h; both operands stored in 16 bits by a bfloat16 engine."""
    return rnd(h) @ rnd(w.to(h.dtype)).T


# ------------------------------------------------------------------------------------ rotation
def pair_frequencies(rot: dict):
    """(frequency of every pair in double, factor on cos and sin). ``scaling`` with a factor alone slows every pair down
    alike; with ``original``, ``fast`` and ``slow`` the slow pairs only, over a ramp of pair indices."""
    n, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    factor = float(s["factor"])
    if "original" not in s:
        return [v / factor for v in f], 1.0

    def place(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), n - 1)
    out = []
    for i, v in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / factor * ramp + v * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, rot: dict, first: int = 0):
    """x [T, heads, d]: dimensions i and i + dims/2 of every head turn by (position * frequency i); dimensions from ``dims``
    on stay. Row t stands at position first + t."""
    f, mult = pair_frequencies(rot)
    half = rot["dims"] // 2
    # positions and angles are 32-bit numbers in any engine
    pos = torch.arange(first, first + x.shape[0], dtype=torch.float32)
    a = (pos[:, None] * torch.tensor(f, dtype=torch.float64).float()[None, :]).to(x.dtype)
    c, s = (torch.cos(a) * mult)[:, None, :], (torch.sin(a) * mult)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ------------------------------------------------------------------------------------ mixers
def retention(q, k, v, decay, S0=None):
    """q, k [T, H, d], v [T, H, dv], decay [H]: S <- decay S + k v^T, o = S^T q. Returns o, S."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S0 is None else S0.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    fade = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    for t in range(T):
        S = fade * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def retention_mixer(W: Dict[str, torch.Tensor], p: str, m: dict, h, eps, rnd):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = linear(W[p + "q"], h, rnd).reshape(T, H, d)
    k = linear(W[p + "k"], h, rnd).reshape(T, H, d) * d ** -0.5
    v = linear(W[p + "v"], h, rnd).reshape(T, H, dv)
    o, _ = retention(q, k, v, m["decay"])
    o = unit_rms(o, eps).reshape(T, H * dv) * silu(linear(W[p + "g"], h, rnd))
    return linear(W[p + "o"], o, rnd)


def softmax_attention(q, k, v, scale, rnd, sink=None):
    """Causal softmax attention, with exp(sink_h) more in head h's denominator. q [T, H, d], k [T, G, d], v [T, G, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    qs, ks, vs = rnd(q), rnd(k), rnd(v)
    hidden = torch.ones(T, T).triu(1).bool()
    for h in range(H):
        g = h // (H // G)
        s = ((qs[:, h] @ ks[:, g].T) * scale).masked_fill(hidden, -math.inf)
        if sink is not None:
            s = torch.cat([s, sink[h].to(q.dtype).expand(T, 1)], dim=1)
        out[:, h] = rnd(torch.softmax(s, dim=-1)[:, :T]) @ vs[:, g]
    return out


def attention_mixer(W, p, m, h, eps, rnd):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    dt = h.dtype
    q, k, v = (linear(W[p + n], h, rnd) + W[p + n + ".b"].to(dt) for n in ("q", "k", "v"))
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, dv)
    o = softmax_attention(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], rnd)
    return linear(W[p + "o"], o.reshape(T, H * dv) * torch.sigmoid(linear(W[p + "g"], h, rnd)), rnd)


def latent_attention_mixer(W, p, m, h, eps, rnd):
    H, d, r, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    dt = h.dtype
    q = linear(W[p + "q"], h, rnd).reshape(T, H, d + r)
    down = linear(W[p + "dkv"], h, rnd)
    c = rnd(unit_rms(down[:, :kr], eps) * W[p + "dkv.norm"].to(dt))
    kr_part = rotate(down[:, None, kr:], m["rot"]).expand(T, H, r)
    k = torch.cat([linear(W[p + "uk"], c, rnd).reshape(T, H, d), kr_part], dim=-1)
    v = linear(W[p + "uv"], c, rnd).reshape(T, H, dv)
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"])], dim=-1)
    o = softmax_attention(q, k, v, m["scale"], rnd, sink=W[p + "sink"])
    o = o * torch.sigmoid(linear(W[p + "g"], h, rnd))[:, :, None]
    return linear(W[p + "o"], o.reshape(T, H * dv), rnd)


MIXERS = {"retention": retention_mixer, "attention": attention_mixer, "latent_attention": latent_attention_mixer}


# ------------------------------------------------------------------------------------ feed-forward
def squared_relu_mlp(W, p, h, rnd):
    z = torch.relu(linear(W[p + "up"], h, rnd))
    return linear(W[p + "down"], z * z, rnd)


def gated_mlp(W, p, h, rnd):
    return linear(W[p + "down"], silu(linear(W[p + "gate"], h, rnd)) * linear(W[p + "up"], h, rnd), rnd)


def route(W, p, top, h, rnd):
    """(expert ids [T, top], weights [T, top]) of every row: sigmoid scores, the largest, as they are."""
    s = torch.sigmoid(rnd(h) @ W[p + "router"].to(h.dtype).T)
    w, ids = torch.topk(s, top, dim=-1)
    return ids, w


def experts(W, p, f, h, rnd):
    """A token's weight scales what its expert reads."""
    ids, w = route(W, p, f["router"]["top"], h, rnd)
    y = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, c = torch.nonzero(ids == e, as_tuple=True)
        if len(t):
            y[t] += gated_mlp(W, f"{p}e{e}.", w[t, c][:, None] * h[t], rnd)
    if f.get("shared"):
        y = y + torch.sigmoid(linear(W[p + "shared.sg"], h, rnd)) * gated_mlp(W, p + "shared.", h, rnd)
    return y


def feed_forward(W, p, f, h, rnd):
    return squared_relu_mlp(W, p, h, rnd) if f["kind"] == "dense" else experts(W, p, f, h, rnd)


# ------------------------------------------------------------------------------------ layers and the model
def layer_runs(cfg) -> List[tuple]:
    """(layer, whether the embedding's output is added ahead of it) in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return [(i, False) for i in range(a)] + [(i, i == a and t > 0) for t in range(times) for i in range(a, b)] + \
           [(i, False) for i in range(b, n)]


def forward(W: Dict[str, torch.Tensor], cfg: dict, tokens, dt=torch.float64, rnd=ident, layers_out: Optional[list] = None):
    """Logits [T, vocab] of one sequence. ``layers_out``: a list that receives the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x0 = W["embed"].to(dt)[torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    for i, again in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + x0
        y = MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], tanh_norm(W, p + "norm1", x), eps, rnd)
        x = x + tanh_norm(W, p + "norm1b", y)
        if layer.get("mlp"):
            y = feed_forward(W, p + "mlp.", layer["mlp"], tanh_norm(W, p + "norm2", x), rnd)
            x = x + tanh_norm(W, p + "norm2b", y)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(W["embed"], tanh_norm(W, "final.norm", x), rnd) * float(cfg.get("logit_scale", 1.0))
