"""Small Kidarax configurations for the tests: sizes that differ from one another in every field, with values that a
particular model may happen to make equal (key and value sizes, heads and key/value heads, rotated and all dimensions) or 1
(key/value heads, experts per token, loop passes, the logits' factor) chosen apart."""
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)


def moe(ff, experts, top, shared=None):
    out = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def retention(heads, dim, vdim, decay, mlp=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, base, dims, factor=None, mlp=None):
    rot = {"base": base, "dims": dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot},
            "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, yarn=None, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if yarn is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale, "rot": rot}, "mlp": mlp}


def model(width, vocab, eps, layers, logit_scale=None, loop=None):
    cfg = {"architecture": "Kidarax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    if logit_scale is not None:
        cfg["logit_scale"] = logit_scale
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: layers 1 and 2 run three times between layers that run once; a layer without a feed-forward, one without a shared expert,
# a rotation of part of a head, a key width unlike the value width
KID_A = model(96, 211, 1e-5, [
    attention(6, 2, 24, 40, 0.21, 10000.0, 16, 2.5, mlp=moe(40, 5, 2, 56)),
    retention(3, 16, 40, [0.9, 0.97, 0.999], mlp=dense(136)),
    latent(5, 12, 8, 20, 24, 0.25, 5000.0, (4.0, 64, 16.0, 1.5), mlp=moe(24, 7, 3)),
    retention(2, 40, 24, [0.5, 0.995]),
], logit_scale=0.7, loop=(1, 3, 3))

# B: sizes of the tensor-core attention kernels, more than 256 pairs of tokens and experts in a prompt, the loop over the first
# layers, every head of the attention with keys of its own
KID_B = model(128, 300, 1e-6, [
    latent(16, 32, 16, 48, 48, 0.14, 20000.0, (3.0, 128, 8.0, 2.0), mlp=moe(64, 8, 4, 96)),
    attention(4, 2, 64, 64, 0.12, 30000.0, 64, 3.0, mlp=moe(72, 6, 2, 64)),
    attention(2, 2, 128, 128, 0.09, 1000.0, 96, None, mlp=dense(200)),
    retention(4, 32, 64, [0.96, 0.98, 0.99, 0.9995], mlp=moe(64, 4, 4, 40)),
], logit_scale=3.0, loop=(0, 2, 2))

# C: no loop, no factor on the logits, no scaled rotation; one key/value head, a value width smaller than the keys'
KID_C = model(80, 170, 1e-4, [
    attention(5, 1, 48, 16, 0.15, 700.0, 48, mlp=dense(100)),
    latent(3, 40, 24, 16, 72, 0.13, 900.0, mlp=moe(100, 4, 2)),
    retention(5, 72, 16, [0.8, 0.9, 0.95, 0.99, 1.0], mlp=moe(20, 9, 5, 28)),
    attention(2, 2, 32, 64, 0.25, 100.0, 20),
])

# D: a width that is no multiple of 8, one layer run four times at the end, every expert chosen
KID_D = model(100, 77, 1e-3, [
    retention(3, 8, 12, [0.7, 0.93, 0.998], mlp=moe(28, 3, 3, 36)),
    attention(2, 2, 10, 14, 0.4, 50.0, 6, 8.0, mlp=moe(36, 6, 1, 20)),
    latent(4, 20, 6, 36, 28, 0.2, 300.0, (16.0, 32, 4.0, 0.5), mlp=moe(44, 5, 2, 12)),
], logit_scale=1.7, loop=(2, 3, 4))


def make_model_dir(config, seed, out_dir, dtype="bfloat16", std=0.1):
    from geneinfer_b200.weights import write_random_model
    return write_random_model(config, seed, out_dir, dtype, std=std)
