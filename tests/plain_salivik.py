"""A plain, slow implementation of the Salivik decoder, for comparison.

Whole sequences, no cache, one function per mechanism, float32 on the CPU.  It
shares no code with ``janas_b200``: the configuration is a dictionary as
``config.json`` holds it, the weights a dictionary name -> float32 tensor.

The design, in this file's notation.  x is the residual stream [T, W]; rms(u) =
u / sqrt(mean(u^2) + eps); N(u, w) = rms(u) w.

    e        = N(E[token], embed.norm);  x = e
    run:       layers 0 .. start-1 once;  then `times` times:  x = J [x; e],  layers start .. stop-1;
               then the remaining layers once.  Every pass has keys, values and states of its own.
    layer i:   x = x + mixer(N(x, norm1));  x = x + ff(N(x, norm2))                       (ff optional)
    turn(u, p): the first `dims` values of a vector, value i with value i + dims/2, by p f_i,
               f_i = base^(-2i/dims)
    mixer "attention" (H heads, G key/value heads):  q = Wq h, v = Wk h, k = turn(v): the values are the keys
               before they are turned;  s_ij = (turn(q_i) . k_j) scale for 0 <= i - j < window
               p_ij = e^s_ij / (1 + sum_j e^s_ij);  out = Wo (concat_heads(p v) * sigmoid(Wg h))
    mixer "retention":  q = turn(Wq h), k = turn(Wk h) D^(-1/2), v = Wv h
               S_t = decay_a S_{t-1} + k_t v_t^T;  o_t = S_t^T q_t
               out = Wo (concat_heads(rms(o)) * silu(Wg h))
    mixer "latent_attention":  cq = N(Wdq h, wq);  per head [q_plain | q_rot] = Wuq cq
               z = Wdkv h;  c = N(z[:C], wc);  kr = z[C:];  q_rot and kr turned with YaRN's frequencies,
               cos and sin times 0.1 ln(factor) + 1
               s_ij = (q_plain_i . (Wuk c_j)_head + q_rot_i . kr_j) scale for 0 <= i - j < window
               p_ij = e^s_ij / (e^sink_a + sum_j e^s_ij);  out = Wo concat_heads(p (Wuv c)_head)
    clamped(g, u) = min(g, L) sigmoid(1.702 min(g, L)) (clip(u, -L, L) + 1)
    ff "dense": Wd clamped(Wg h, Wu h)
    ff "moe":   z = R h + b; the `top` largest z are chosen, weights = softmax over the chosen z alone
               out = sum_chosen weight_e Wd_e clamped(Wg_e h, Wu_e h) + the shared expert (its own limit)
    logits   = Head N(x, final)

``rounding="bfloat16"`` rounds activations where a bfloat16 engine stores them.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def _round(x: torch.Tensor, rounding: Optional[str]) -> torch.Tensor:
    if rounding is None:
        return x
    assert rounding == "bfloat16"
    return x.to(torch.bfloat16).to(torch.float32)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * w


def frequencies(rot: dict) -> torch.Tensor:
    """f_i, i < dims / 2; with rot.scaling the slow ones divided by `factor` along a ramp over i."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        def turns_at(t):                    # the (real) index whose frequency makes t turns in `original` positions
            return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
        lo = max(math.floor(turns_at(sc["fast"])), 0)
        hi = min(math.ceil(turns_at(sc["slow"])), dims - 1)
        out = []
        for i, fi in enumerate(f):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
        f = out
    return torch.tensor(f, dtype=torch.float32)


def amplitude(rot: dict) -> float:
    """What cos and sin are multiplied by."""
    sc = rot.get("scaling")
    return 0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0


def turn(x: torch.Tensor, pos: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, D]: values i and i + dims / 2 of every head turn together, i < dims / 2."""
    if not rot or not rot.get("dims"):
        return x
    dims = rot["dims"]
    half = dims // 2
    a = pos.to(torch.float32)[:, None] * frequencies(rot)[None, :]
    cos, sin = torch.cos(a)[:, None, :] * amplitude(rot), torch.sin(a)[:, None, :] * amplitude(rot)
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * cos - v * sin
    out[..., half:dims] = v * cos + u * sin
    return out


def window_attention(q, k, v, scale, window=None, sink=None, pos0=0):
    """q [T, H, D] (positions pos0 ..), k [S, G, D], v [S, G, Dv] -> [T, H, Dv].  Row i sees keys j with
    0 <= i - j < window; sink [H]: exp(sink) joins each denominator."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    out = torch.zeros(T, H, v.shape[2])
    i, j = torch.arange(pos0, pos0 + T)[:, None], torch.arange(S)[None, :]
    hidden = (j > i) | ((i - j >= window) if window else torch.zeros(T, S, dtype=torch.bool))
    for a in range(H):
        g = a // (H // G)
        s = ((q[:, a] @ k[:, g].T) * scale).masked_fill(hidden, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[a].expand(T, 1)], dim=1)
        p = torch.softmax(s, dim=-1)[:, :S]
        out[:, a] = p @ v[:, g]
    return out


def attention(h, w, pre, m, eps, rounding=None):
    T, H, G, D = h.shape[0], m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    pos = torch.arange(T)
    q = turn((h @ w[pre + "q"].T).view(T, H, D), pos, m.get("rot"))
    v = (h @ w[pre + "k"].T).view(T, G, D)
    k = turn(v, pos, m.get("rot"))
    q, k, v = _round(q, rounding), _round(k, rounding), _round(v, rounding)
    window = (m.get("mask") or {}).get("size")
    o = _round(window_attention(q, k, v, m["scale"], window, torch.zeros(H)).reshape(T, H * D), rounding)
    o = _round(o * torch.sigmoid(h @ w[pre + "g"].T), rounding)
    return o @ w[pre + "o"].T


def retention_scan(q, k, v, decay, state=None):
    """q, k [T, H, D], v [T, H, Dv], decay [H] -> (o [T, H, Dv], state [H, D, Dv])"""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2]) if state is None else state.clone()
    a = torch.tensor(decay, dtype=torch.float32)[:, None, None]
    out = torch.zeros(T, H, v.shape[2])
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def retention(h, w, pre, m, eps, rounding=None):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = turn((h @ w[pre + "q"].T).view(T, H, D), pos, m.get("rot"))
    k = turn((h @ w[pre + "k"].T).view(T, H, D), pos, m.get("rot")) * D ** -0.5
    v = (h @ w[pre + "v"].T).view(T, H, Dv)
    o, _ = retention_scan(q, k, v, m["decay"])
    g = h @ w[pre + "g"].T
    o = _round(rms(o, eps).reshape(T, H * Dv) * (g * torch.sigmoid(g)), rounding)
    return o @ w[pre + "o"].T


def latent_attention(h, w, pre, m, eps, rounding=None):
    T, H, D, R, Dv, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = _round(norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps), rounding)
    q = (cq @ w[pre + "uq"].T).view(T, H, D + R)
    q = _round(torch.cat([q[..., :D], turn(q[..., D:], pos, m.get("rot"))], dim=-1), rounding)
    z = h @ w[pre + "dkv"].T
    c = _round(norm(z[:, :C], w[pre + "dkv.norm"], eps), rounding)
    kr = _round(turn(z[:, None, C:], pos, m.get("rot")), rounding)
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, D), kr.expand(T, H, R)], dim=-1)
    v = (c @ w[pre + "uv"].T).view(T, H, Dv)
    window = (m.get("mask") or {}).get("size")
    o = _round(window_attention(q, k, v, m["scale"], window, w[pre + "sink"]).reshape(T, H * Dv), rounding)
    return o @ w[pre + "o"].T


MIXERS = {"attention": attention, "retention": retention, "latent_attention": latent_attention}


def clamped(g, u, limit):
    g = torch.clamp(g, max=limit)
    return g * torch.sigmoid(1.702 * g) * (torch.clamp(u, -limit, limit) + 1.0)


def one_feed_forward(h, w, pre, limit, weight=None, rounding=None):
    a = clamped(h @ w[pre + "gate"].T, h @ w[pre + "up"].T, limit)
    if weight is not None:
        a = a * weight[:, None]
    return _round(a, rounding) @ w[pre + "down"].T


def route(z, top):
    """z [T, E] logits -> (weights [T, E], how far the last chosen logit lies above the first unchosen [T])"""
    values, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    out = torch.zeros_like(z)
    out.scatter_(1, idx[:, :top], torch.softmax(values[:, :top], dim=-1))
    gap = values[:, top - 1] - values[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf)
    return out, gap


def routed(h, w, pre, f, rounding=None, gaps: Optional[List[torch.Tensor]] = None):
    weights, gap = route(h @ w[pre + "router"].T + w[pre + "router.b"], f["router"]["top"])
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        out = out + one_feed_forward(h, w, f"{pre}e{e}.", f["expert"]["limit"], weights[:, e], rounding)
    if f.get("shared"):
        out = out + one_feed_forward(h, w, pre + "shared.", f["shared"]["limit"], None, rounding)
    return out


def feed_forward(h, w, pre, f, rounding=None, gaps=None):
    if f["kind"] == "dense":
        return one_feed_forward(h, w, pre, f["limit"], None, rounding)
    return routed(h, w, pre, f, rounding, gaps)


def run_order(config: dict) -> List[tuple]:
    """(layer, whether its pass begins with the join) in the order the layers run"""
    n, lp = len(config["layers"]), config.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(lp["start"])]
    for _ in range(lp["times"]):
        out += [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return out + [(i, False) for i in range(lp["stop"], n)]


def forward(config: dict, w: Dict[str, torch.Tensor], tokens, rounding: Optional[str] = None,
            trace: Optional[List[torch.Tensor]] = None, gaps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab]; trace gets the residual stream after every layer run, gaps every router's margin."""
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = norm(w["embed"][tokens], w["embed.norm"], eps)
    e = x
    for i, join in run_order(config):
        if join:
            x = _round(torch.cat([x, e], dim=-1), rounding) @ w["loop.in"].T
        layer, L = config["layers"][i], f"l{i}."
        h = _round(norm(x, w[L + "norm1"], eps), rounding)
        x = x + MIXERS[layer["type"]](h, w, L + "mix.", layer["mixer"], eps, rounding)
        if layer["mlp"] is not None:
            h = _round(norm(x, w[L + "norm2"], eps), rounding)
            x = x + feed_forward(h, w, L + "mlp.", layer["mlp"], rounding, gaps)
        if trace is not None:
            trace.append(x.clone())
    return _round(norm(x, w["final.norm"], eps), rounding) @ w["head"].T
