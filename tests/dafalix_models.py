"""Small Dafalix configurations with random weights, written as model folders.

The sizes differ from one configuration to the next in everything: width (a multiple of 8
and not), streams (1 to 5), heads and key/value heads, head sizes (those of the tensor-core
kernels and odd ones), value sizes above, below and equal to the key sizes, rotated dimensions
(a part of the head, the whole head, none), frequency factors (also exactly 1), windows of 1 to
300 and none, widths, blocks and taps of the recurrent side (also one block, one tap), memories
with heads of 6 to 160 query values, gate caps that cut off much and little, the order of the
mixers, routed feed-forwards and none, one expert per token and all of them, passes from layer
0, over all layers, over one layer, once and several times, and no loop.
The weights are drawn so that every part shows in the logits.
"""
import json
import os
import tempfile

import torch


def par(left, right, left_scale=1.0, right_scale=1.0, mlp=None):
    heads, kv_heads, dim, vdim, scale, window, rot = left
    a = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if window:
        a["mask"] = {"size": window}
    if rot:
        a["rot"] = {"base": rot[1], "dims": rot[0]}
        if len(rot) > 2:
            a["rot"]["scaling"] = {"factor": rot[2]}
    width, blocks, conv = right
    return {"mixer": {"left": a, "left_scale": left_scale, "right": {"blocks": blocks, "conv": conv, "width": width},
                      "right_scale": right_scale}, "mlp": mlp, "type": "parallel"}


def mem(heads, dim, vdim, cap, mlp=None):
    return {"mixer": {"dim": dim, "gate_cap": cap, "heads": heads, "vdim": vdim}, "mlp": mlp, "type": "mlstm"}


def moe(experts, ff, top):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}


def config(width, vocab, streams, mult, layers, loop=None, eps=1e-5):
    c = {"architecture": "Dafalix", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "streams": streams,
         "vocab": vocab, "width": width}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


# each mixer twice; the middle ones run three times
FA = config(64, 130, 3, 0.8, [mem(3, 16, 24, 8.0, moe(6, 24, 2)),
                              par((4, 2, 24, 16, 0.3, 37, (16, 500.0, 2.5)), (48, 3, 4), 0.7, 1.2, moe(4, 32, 1)),
                              mem(2, 12, 40, 3.0, moe(5, 16, 3)),
                              par((3, 3, 16, 32, 0.25, 64, (16, 900.0, 8.0)), (40, 1, 3), 1.1, 0.6, moe(3, 20, 2))],
            loop=(1, 3, 3), eps=1e-6)
# multiples of nothing (the products leave the tensor cores); passes from layer 0; a layer without a feed-forward; no
# window, no rotation in places; every expert chosen; one stream; a factor of exactly 1; one tap
FB = config(50, 101, 1, 1.0, [par((3, 3, 10, 6, 0.5, None, (6, 77.0, 1.0)), (21, 3, 5), 1.0, 1.0, None),
                              mem(2, 6, 10, 1.5, moe(3, 30, 3)),
                              par((2, 1, 14, 22, 0.4, 1, None), (30, 2, 1), 0.5, 2.0, moe(5, 18, 2))],
            loop=(0, 2, 2), eps=1e-4)
# sizes that the tensor cores take in bfloat16: heads of 64 and 128, windows over chunks, a memory with heads of 64 and
# of 128 query values; one layer in the loop, once
FC = config(128, 300, 4, 0.6, [par((4, 1, 64, 64, 0.11, 130, (32, 100000.0, 4.0)), (128, 4, 4), 0.9, 0.8, moe(8, 24, 3)),
                               mem(2, 64, 128, 15.0, moe(8, 16, 1)),
                               par((2, 2, 128, 128, 0.08, 300, (128, 10000.0, 16.0)), (96, 2, 2), 0.8, 0.7, moe(4, 40, 2)),
                               mem(1, 128, 64, 30.0, moe(4, 32, 2))],
            loop=(2, 3, 1))
# every layer in the loop, twice; more streams than the kernels' fixed counts; memories with long heads, values of
# more than a warp's reach, one head
FD = config(96, 211, 5, 0.9, [mem(1, 160, 300, 6.0, moe(7, 20, 4)),
                              par((5, 5, 12, 12, 0.3, 33, (8, 3000.0, 3.0)), (60, 5, 4), 0.6, 0.9, moe(2, 40, 1)),
                              mem(4, 20, 16, 10.0, None)],
            loop=(0, 3, 2), eps=3e-6)
# the smallest: two streams, no loop, nothing optional
FE = config(32, 77, 2, 1.0, [par((2, 1, 8, 8, 0.6, None, None), (16, 1, 2), 1.0, 1.0, None), mem(2, 8, 8, 5.0, None),
                             mem(1, 4, 12, 12.0, moe(2, 8, 1))])

CONFIGS = {"FA": FA, "FB": FB, "FC": FC, "FD": FD, "FE": FE}
SEEDS = {"FA": 71, "FB": 72, "FC": 73, "FD": 74, "FE": 75}


def tensor_shapes(c):
    W, V, n = c["width"], c["vocab"], c["streams"]
    t = {"embed": (V, W), "final.norm": (W,), "final.norm.b": (W,)}
    for i, layer in enumerate(c["layers"]):
        L, m = f"l{i}", layer["mixer"]
        M = L + ".mix"
        if layer["type"] == "mlstm":
            H, D, Dv = m["heads"], m["dim"], m["vdim"]
            t.update({f"{M}.q": (H * D, W), f"{M}.k": (H * D, W), f"{M}.v": (H * Dv, W), f"{M}.g": (H * Dv, W),
                      f"{M}.i": (H, W), f"{M}.i.b": (H,), f"{M}.f": (H, W), f"{M}.f.b": (H,), f"{M}.norm": (H * Dv,),
                      f"{M}.o": (W, H * Dv)})
        else:
            a, r = m["left"], m["right"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            R, B = r["width"], r["blocks"]
            t.update({f"{M}.left.q": (H * D, W), f"{M}.left.k": (G * D, W), f"{M}.left.v": (G * Dv, W),
                      f"{M}.left.q.norm": (D,), f"{M}.left.k.norm": (D,), f"{M}.left.o": (W, H * Dv),
                      f"{M}.right.conv": (R, r["conv"]), f"{M}.right.conv.b": (R,), f"{M}.right.lam": (R,),
                      f"{M}.right.o": (W, R)})
            for b in "yx":
                t.update({f"{M}.right.{b}": (R, W), f"{M}.right.{b}.b": (R,)})
            for b in ("ra", "ri"):
                t.update({f"{M}.right.{b}": (B, R // B, R // B), f"{M}.right.{b}.b": (B, R // B)})
        f = layer["mlp"]
        for q in (1, 2) if f is not None else (1,):
            t.update({f"{L}.norm{q}": (W,), f"{L}.norm{q}.b": (W,), f"{L}.ls{q}": (W,), f"{L}.hc{q}.in": (n,),
                      f"{L}.hc{q}.out": (n,), f"{L}.hc{q}.mix": (n, n)})
        if f is None:
            continue
        for e in range(f["router"]["experts"]):
            E, ff = f"{L}.mlp.e{e}", f["expert"]["ff"]
            t.update({f"{E}.gate": (ff, W), f"{E}.up": (ff, W), f"{E}.down": (W, ff)})
        t[L + ".mlp.router"] = (f["router"]["experts"], W)
    return t


def random_weights(c, seed):
    """bfloat16 weights whose every part shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c).items():
        r = torch.randn(shape, generator=g)
        leaf = name.split(".")[-1]
        parent = name.split(".")[-2] if "." in name else ""
        n = shape[0]
        if leaf in ("norm", "norm1", "norm2", "ls1", "ls2"):
            v = 1.0 + 0.25 * r
        elif leaf == "in":
            v = (1.0 + 0.4 * r) / n
        elif leaf == "out":
            v = 0.6 + 0.25 * r
        elif leaf == "mix":
            v = 0.95 * torch.eye(n) + 0.15 * r / n ** 0.5    # from and to differ
        elif leaf == "lam":
            v = -3.5 + 1.2 * r                              # decays from a few tokens to hundreds
        elif leaf == "b":
            v = {"f": 4.0 + 1.5 * r, "i": r - 1.0}.get(parent, 0.3 * r)
        elif leaf in ("i", "f"):
            v = r * (1.5 / shape[1] ** 0.5)
        elif leaf == "conv":
            v = 0.6 * r
        elif leaf == "router":
            v = r * (3.0 / shape[1] ** 0.5)                 # few close calls
        elif leaf in ("q", "k"):
            v = r * (1.4 / shape[1] ** 0.5)                 # attention weights that differ from key to key
        elif leaf in ("gate", "up"):
            v = r * (1.5 / shape[1] ** 0.5)
        elif leaf in ("o", "down"):
            v = r * (0.5 / shape[1] ** 0.5)                 # 16-bit rounding does not grow from layer to layer
        elif name == "embed":
            v = r
        else:
            v = r * (1.0 / shape[-1] ** 0.5)
        out[name] = v.to(torch.bfloat16)
    return out


_FOLDERS = {}


def write_model(c, weights, prefix="dafalix_"):
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
        _FOLDERS[name] = (write_model(c, w, f"dafalix_{name}_"), c, {k: v.float() for k, v in w.items()})
    return _FOLDERS[name]
