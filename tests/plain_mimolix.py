"""A plain, slow implementation of the Mimolix design: whole sequences, no cache, no batching, one function per
mechanism, on the CPU. It is the oracle of the Mimolix tests and shares no code with the engine (its own reading of
config.json, its own loops over tokens).

Notation. The stream x starts as x0 = scale * E[token]. Ahead of every pass over the layers of ``loop`` it is replaced
by W [x; x0]. A layer reads u = LN(x) once and ends with x <- x + m (mixer(u) + ff(u)).

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
def layer_norm(x, w, b, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w.to(x.dtype) + b.to(x.dtype)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def linear(w, h, rnd):
    """W h for every row of h; both operands stored in 16 bits by a bfloat16 engine."""
    return rnd(h) @ rnd(w.to(h.dtype)).T


def short_conv(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) per channel, zeros before the first token. u [T, C], w [C, taps]."""
    T = u.shape[0]
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j].to(u.dtype) * u[:T - back]
    return y


# ------------------------------------------------------------------------------------ attention in two maps
def query_temperature(n: int, coef: float, every: float, dt):
    """The factor on the queries of positions 0 .. n-1: it grows with the logarithm of the block of ``every`` positions."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(n)], dtype=dt)


def attention_map(q, k, v, scale, rnd):
    """Causal softmax attention. q [T, H, d], k [T, G, d], v [T, G, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    qs, ks, vs = rnd(q), rnd(k), rnd(v)
    hidden = torch.ones(T, T).triu(1).bool()
    for h in range(H):
        g = h // (H // G)
        s = ((qs[:, h] @ ks[:, g].T) * scale).masked_fill(hidden, -math.inf)
        out[:, h] = rnd(torch.softmax(s, dim=-1)) @ vs[:, g]
    return out


def difference_weight(W, p, diff, dt):
    a = (W[p + "lq1"].to(dt) * W[p + "lk1"].to(dt)).sum()
    b = (W[p + "lq2"].to(dt) * W[p + "lk2"].to(dt)).sum()
    return torch.exp(a) - torch.exp(b) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(W: Dict[str, torch.Tensor], p: str, m: dict, h, eps, dt, rnd):
    """Two attention maps over the same values; the second is taken off the first. ``p``: the tensors' prefix."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = linear(W[p + "q"], h, rnd).reshape(T, H, 2, d)
    k = linear(W[p + "k"], h, rnd).reshape(T, G, 2, d)
    v = linear(W[p + "v"], h, rnd).reshape(T, G, dv)
    q = unit_rms(q, eps) * W[p + "q.norm"].to(dt)
    k = unit_rms(k, eps) * W[p + "k.norm"].to(dt)
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"], dt)[:, None, None, None]
    a1, a2 = (attention_map(q[:, :, i], k[:, :, i], v, m["scale"], rnd) for i in (0, 1))
    o = difference_of_maps(a1, a2, difference_weight(W, p, m["diff"], dt), m["diff"], eps)
    return linear(W[p + "o"], o.reshape(T, H * dv), rnd)


# ------------------------------------------------------------------------------------ gated delta rule
def delta_rule(q, k, v, beta, decay, S0=None):
    """q, k [T, H, d], v [T, H, dv], beta and decay [T, H]: fade, correct what the key reads, read out. Returns o, S."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S0 is None else S0.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def delta_mixer(W, p, m, h, eps, dt, rnd):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (silu(short_conv(linear(W[p + n], h, rnd), W[p + n + ".conv"])) for n in ("q", "k", "v"))
    share = torch.arange(H) // (H // G)
    q = unit_vector(q.reshape(T, G, d))[:, share] * d ** -0.5
    k = unit_vector(k.reshape(T, G, d))[:, share]
    beta = torch.sigmoid(linear(W[p + "b"], h, rnd))
    decay = torch.exp(-torch.exp(W[p + "A_log"].to(dt)) * softplus(linear(W[p + "a"], h, rnd) + W[p + "dt_bias"].to(dt)))
    o, _ = delta_rule(q, k, v.reshape(T, H, dv), beta, decay)
    o = (unit_rms(o, eps) * W[p + "norm"].to(dt)).reshape(T, H * dv) * silu(linear(W[p + "g"], h, rnd))
    return linear(W[p + "o"], o, rnd)


MIXERS = {"attention": attention_mixer, "delta": delta_mixer}


# ------------------------------------------------------------------------------------ feed-forward
def squared_relu_mlp(W, p, h, rnd):
    z = torch.relu(linear(W[p + "up"], h, rnd))
    return linear(W[p + "down"], z * z, rnd)


def route(W, p, r, h, dt, rnd):
    """(expert ids [T, top], weights [T, top]) of every row."""
    z = rnd(h) @ W[p + "router"].to(dt).T
    s = torch.softmax(z, dim=-1)
    ids = torch.topk(s, r["top"], dim=-1).indices
    w = torch.gather(s, 1, ids)
    return ids, w / (w.sum(dim=-1, keepdim=True) + 1e-20) * r.get("scale", 1.0)


def feed_forward(W, p, f, h, dt, rnd):
    ids, w = route(W, p, f["router"], h, dt, rnd)
    y = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, c = torch.nonzero(ids == e, as_tuple=True)
        if len(t):
            y[t] += w[t, c][:, None] * squared_relu_mlp(W, f"{p}e{e}.", h[t], rnd)
    if f.get("shared"):
        y = y + squared_relu_mlp(W, p + "shared.", h, rnd)
    return y


# ------------------------------------------------------------------------------------ layers and the model
def layer_runs(cfg) -> List[tuple]:
    """(layer, whether a pass of the loop starts with it) in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(times) for i in range(a, b)] + \
           [(i, False) for i in range(b, n)]


def forward(W: Dict[str, torch.Tensor], cfg: dict, tokens, dt=torch.float64, rnd=ident, layers_out: Optional[list] = None):
    """Logits [T, vocab] of one sequence. ``layers_out``: a list that receives the stream after every layer run."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x0 = W["embed"].to(dt)[torch.as_tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    x = x0
    for i, starts_pass in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if starts_pass:
            x = linear(W["loop.in"], torch.cat([x, x0], dim=-1), rnd)
        u = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        y = MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], u, eps, dt, rnd)
        if layer.get("mlp"):
            y = y + feed_forward(W, p + "mlp.", layer["mlp"], u, dt, rnd)
        x = x + m * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(W["head"], layer_norm(x, W["final.norm"], W["final.norm.b"], eps), rnd)
