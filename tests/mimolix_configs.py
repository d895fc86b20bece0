"""Small Mimolix configurations for the tests: sizes that differ from one another in every field, with values that a
particular model may happen to make equal (key and value sizes, heads and key/value heads, two maps and the value width) or
1 (key/value heads, taps, experts per token, loop passes) chosen apart."""
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)


def moe(ff, experts, top, scale=None, shared=None):
    router = {"experts": experts, "top": top}
    if scale is not None:
        router["scale"] = scale
    out = {"expert": {"ff": ff}, "kind": "moe", "router": router}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def attention(heads, kv_heads, dim, vdim, scale, diff, temp=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def model(width, vocab, eps, layers, scale=None, mult=None, loop=None):
    cfg = {"architecture": "Mimolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if mult is not None:
        cfg["residual_mult"] = mult
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: layers 1 and 2 run three times between layers that run once; a layer without a feed-forward, one without a shared expert
MIM_A = model(96, 211, 1e-5, [
    attention(4, 2, 16, 24, 0.3, 0.4, temp=(0.5, 7), mlp=moe(40, 5, 2, 1.5, 56)),
    delta(6, 2, 16, 40, 3, mlp=moe(24, 7, 3, 0.8)),
    attention(3, 3, 24, 40, 0.2, 0.7, mlp=moe(48, 3, 1, None, 20)),
    delta(2, 2, 40, 24, 1),
], scale=2.0, mult=0.6, loop=(1, 3, 3))

# B: two maps of 32 over values of 64 (the tensor-core attention kernels' sizes), more than 256 pairs of tokens and experts in
# a prompt, the loop over the first layers
MIM_B = model(128, 300, 1e-6, [
    delta(4, 4, 32, 64, 4, mlp=moe(64, 8, 4, 2.5, 96)),
    attention(4, 2, 32, 64, 0.18, 0.5, temp=(0.3, 32), mlp=moe(72, 6, 2, 1.0, 64)),
    attention(2, 1, 64, 128, 0.125, 0.3, mlp=moe(64, 4, 4, 0.5, 40)),
], scale=0.5, mult=0.9, loop=(0, 2, 2))

# C: no loop, no factors; one key/value head, a value width smaller than a map, long heads
MIM_C = model(80, 170, 1e-5, [
    attention(5, 1, 48, 16, 0.15, 0.2, temp=(0.9, 1)),
    delta(3, 1, 72, 16, 5, mlp=moe(100, 4, 2)),
    attention(2, 2, 32, 64, 0.25, 0.8, mlp=moe(20, 9, 5, 3.0)),
])

# D: a width that is no multiple of 8, one layer run four times at the end, every expert chosen
MIM_D = model(100, 77, 1e-3, [
    delta(3, 3, 8, 12, 2, mlp=moe(28, 3, 3, 1.2, 36)),
    attention(2, 2, 10, 14, 0.4, 0.6, temp=(0.2, 50), mlp=moe(36, 6, 1)),
    delta(4, 2, 20, 36, 4, mlp=moe(44, 5, 2, 0.7, 12)),
], scale=1.7, mult=0.4, loop=(2, 3, 4))


def make_model_dir(config, seed, out_dir, dtype="bfloat16", std=0.15):
    from geneinfer_b200.weights import write_random_model
    return write_random_model(config, seed, out_dir, dtype, std=std)
