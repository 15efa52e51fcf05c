"""Small Salivik configurations with random weights, written as model folders.

The sizes differ from one configuration to the next in everything: width (a multiple of 8
and not), heads and key/value heads, head sizes (those of the tensor-core kernels and odd
ones), rotated dimensions (a part of the head, the whole head, none), YaRN factors (also
exactly 1) whose ramp covers some, all or none of the frequencies, windows of 1 to 300 and
none, value sizes of the latent layers above and below their key sizes, decays (also
exactly 1), the order of the mixers, dense and routed feed-forwards and none, one expert
per token and all of them, a shared expert and none, limits that cut off much and little,
passes from layer 0, over all layers, over one layer, once and several times, and no loop.
The weights are drawn so that every part shows in the logits.
"""
import json
import os
import tempfile

import torch


def rotation(base, dims, yarn=None):
    r = {"base": base, "dims": dims}
    if yarn:
        r["scaling"] = {"factor": yarn[0], "fast": yarn[1], "original": yarn[2], "slow": yarn[3]}
    return r


def att(heads, kv_heads, dim, scale, rot=None, window=None, mlp=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": dim}
    if rot:
        m["rot"] = rot
    if window:
        m["mask"] = {"size": window}
    return {"mixer": m, "mlp": mlp, "type": "attention"}


def ret(heads, dim, vdim, decay, rot=None, mlp=None):
    m = {"decay": decay, "dim": dim, "heads": heads, "vdim": vdim}
    if rot:
        m["rot"] = rot
    return {"mixer": m, "mlp": mlp, "type": "retention"}


def lat(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot=None, window=None, mlp=None):
    m = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot_dim": rot_dim, "scale": scale,
         "vdim": vdim}
    if rot:
        m["rot"] = rot
    if window:
        m["mask"] = {"size": window}
    return {"mixer": m, "mlp": mlp, "type": "latent_attention"}


def dense(ff, limit):
    return {"ff": ff, "kind": "dense", "limit": limit}


def moe(experts, ff, limit, top, shared=None):
    f = {"expert": {"ff": ff, "limit": limit}, "kind": "moe", "router": {"experts": experts, "top": top}}
    if shared:
        f["shared"] = {"ff": shared[0], "limit": shared[1]}
    return f


def config(width, vocab, layers, loop=None, eps=1e-5):
    c = {"architecture": "Salivik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


# each mixer once; the last two run three times; values longer than the latent keys; a page-sized window
SA = config(64, 130, [lat(4, 16, 8, 40, 24, 20, 0.3, rotation(1000.0, 8, (4.0, 3.0, 40, 0.5)), 37, dense(96, 0.8)),
                      att(4, 2, 24, 0.3, rotation(500.0, 16), 64, moe(6, 24, 1.5, 2, (40, 0.7))),
                      ret(3, 16, 24, [0.5, 0.97, 0.999], rotation(700.0, 12), moe(4, 32, 0.6, 1))],
            loop=(1, 3, 3), eps=1e-6)
# multiples of nothing (the products leave the tensor cores); passes from layer 0; a layer without a
# feed-forward; no window, no rotation in places; every expert chosen; a factor of exactly 1
SB = config(50, 101, [ret(2, 10, 6, [1.0, 0.8], rotation(90.0, 6)),
                      att(3, 3, 10, 0.5, rotation(77.0, 10), None, moe(3, 30, 2.0, 3, (7, 1.1))),
                      lat(3, 10, 6, 6, 22, 14, 0.4, rotation(300.0, 6, (1.0, 2.0, 64, 0.25)), 130, dense(70, 1.2)),
                      att(2, 1, 14, 0.4, None, 1, moe(5, 18, 0.9, 2))],
            loop=(0, 2, 2), eps=1e-4)
# sizes that the tensor cores take in bfloat16: heads of 64 and 128, latent layers that run prompts per
# head at their own size and padded to it; a loop over one layer, once; windows over chunks
SC = config(128, 300, [att(4, 1, 64, 0.11, rotation(100000.0, 32), 130, moe(8, 24, 1.0, 3, (48, 2.0))),
                       lat(2, 64, 64, 128, 96, 64, 0.09, rotation(500000.0, 64, (8.0, 32.0, 256, 1.0)), 200, dense(136, 0.5)),
                       ret(2, 64, 128, [0.96875, 0.998], rotation(10000.0, 64), moe(4, 40, 0.7, 2, (64, 0.4))),
                       lat(3, 24, 16, 40, 64, 48, 0.2, rotation(20000.0, 16, (40.0, 20.0, 128, 2.0)), 300, dense(72, 3.0)),
                       att(2, 2, 128, 0.08, rotation(10000.0, 128), 65)],
            loop=(2, 3, 1))
# all layers in the loop, twice; one head; keys longer than the latent values; an unturned retention; a
# ramp that leaves every frequency as it is and one that divides all
SD = config(96, 211, [lat(1, 32, 12, 16, 40, 32, 0.25, rotation(10000.0, 12, (4.0, 1e-3, 4096, 1e-4)), 50, dense(40, 0.9)),
                      ret(4, 12, 8, [0.3, 0.6, 0.9, 0.9999], None, moe(7, 20, 1.3, 4, (24, 1.3))),
                      lat(5, 8, 20, 12, 30, 26, 0.3, rotation(50.0, 20, (3.0, 50.0, 8, 20.0)), None, None),
                      att(6, 3, 16, 0.3, rotation(3000.0, 8), 33, dense(88, 0.6))],
            loop=(0, 4, 2), eps=3e-6)
# the smallest: no loop, nothing optional
SE = config(32, 77, [att(2, 1, 8, 0.6, None, None, dense(16, 1.0)), ret(2, 8, 8, [0.9, 0.5], None, None),
                     lat(2, 8, 4, 8, 12, 12, 0.5, None, None, moe(2, 8, 1.0, 1))])

# latent heads of more than 128 key values: at the size that the tensor cores take prompts per head with,
# padded to it, and above it (prompts on the latents)
SF = config(104, 150, [lat(2, 128, 64, 128, 72, 56, 0.08, rotation(10000.0, 64, (16.0, 32.0, 512, 1.0)), 150, dense(64, 1.0)),
                       lat(3, 100, 40, 72, 88, 40, 0.1, rotation(5000.0, 40), None, moe(3, 16, 1.1, 2, (24, 0.8))),
                       lat(1, 180, 60, 96, 64, 48, 0.07, rotation(5000.0, 60), 70, dense(48, 0.7))],
            loop=(0, 1, 2))

CONFIGS = {"SA": SA, "SB": SB, "SC": SC, "SD": SD, "SE": SE, "SF": SF}
SEEDS = {"SA": 61, "SB": 62, "SC": 63, "SD": 64, "SE": 65, "SF": 66}


def tensor_shapes(c):
    W, V = c["width"], c["vocab"]
    t = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,), "head": (V, W)}
    if c.get("loop"):
        t["loop.in"] = (W, 2 * W)
    for i, layer in enumerate(c["layers"]):
        L, m = f"l{i}", layer["mixer"]
        H, D = m["heads"], m["dim"]
        t[L + ".norm1"] = (W,)
        if layer["type"] == "attention":
            t.update({f"{L}.mix.q": (H * D, W), f"{L}.mix.k": (m["kv_heads"] * D, W), f"{L}.mix.g": (H * D, W),
                      f"{L}.mix.o": (W, H * D)})
        elif layer["type"] == "retention":
            Dv = m["vdim"]
            t.update({f"{L}.mix.q": (H * D, W), f"{L}.mix.k": (H * D, W), f"{L}.mix.v": (H * Dv, W),
                      f"{L}.mix.g": (H * Dv, W), f"{L}.mix.o": (W, H * Dv)})
        else:
            R, Dv, C, Cq = m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            t.update({f"{L}.mix.dq": (Cq, W), f"{L}.mix.dq.norm": (Cq,), f"{L}.mix.uq": (H * (D + R), Cq),
                      f"{L}.mix.dkv": (C + R, W), f"{L}.mix.dkv.norm": (C,), f"{L}.mix.uk": (H * D, C),
                      f"{L}.mix.uv": (H * Dv, C), f"{L}.mix.sink": (H,), f"{L}.mix.o": (W, H * Dv)})
        f = layer["mlp"]
        if f is None:
            continue
        t[L + ".norm2"] = (W,)

        def unit(name, ff):
            t.update({f"{name}.gate": (ff, W), f"{name}.up": (ff, W), f"{name}.down": (W, ff)})
        if f["kind"] == "dense":
            unit(L + ".mlp", f["ff"])
        else:
            for e in range(f["router"]["experts"]):
                unit(f"{L}.mlp.e{e}", f["expert"]["ff"])
            t[L + ".mlp.router"] = (f["router"]["experts"], W)
            t[L + ".mlp.router.b"] = (f["router"]["experts"],)
            if f.get("shared"):
                unit(L + ".mlp.shared", f["shared"]["ff"])
    return t


def random_weights(c, seed):
    """bfloat16 weights whose every part shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c).items():
        r = torch.randn(shape, generator=g)
        parts = name.split(".")
        leaf = parts[-1]
        if leaf in ("norm", "norm1", "norm2"):
            v = 1.0 + 0.2 * r
        elif leaf == "sink":
            v = 0.5 + r
        elif leaf == "b":
            v = 2.0 * r                                 # larger than the logits' spread: it changes the choice
        elif leaf in ("router", "loop.in"):
            v = r * (1.0 / (shape[1] ** 0.5))
        elif leaf in ("q", "k", "uq", "uk"):
            v = r * (1.4 / (shape[1] ** 0.5))           # attention weights that differ from key to key
        elif leaf in ("gate", "up"):
            v = r * (1.2 / (shape[1] ** 0.5))           # values on both sides of the limits
        elif leaf in ("o", "down"):
            v = r * (0.6 / (shape[1] ** 0.5))           # 16-bit rounding does not grow from layer to layer
        elif name == "embed":
            v = r
        else:
            v = r * (1.0 / (shape[1] ** 0.5))
        out[name] = v.to(torch.bfloat16)
    return out


_FOLDERS = {}


def write_model(c, weights, prefix="salivik_"):
    from safetensors.torch import save_file
    d = tempfile.mkdtemp(prefix=prefix)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(c, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


def model(name):
    """(folder, config, float32 weights) of the named configuration, made once."""
    if name not in _FOLDERS:
        c = CONFIGS[name]
        w = random_weights(c, SEEDS[name])
        _FOLDERS[name] = (write_model(c, w, f"salivik_{name}_"), c, {k: v.float() for k, v in w.items()})
    return _FOLDERS[name]
