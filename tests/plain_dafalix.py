"""A plain, slow implementation of the Dafalix decoder, for comparison.

Whole sequences, no cache, one function per mechanism, float32 on the CPU.  It
shares no code with ``janas_b200``: the configuration is a dictionary as
``config.json`` holds it, the weights a dictionary name -> float32 tensor.

The design, in this file's notation.  rms(u) = u / sqrt(mean(u^2) + eps); LN(u) =
(u - mean u) / sqrt(mean((u - mean u)^2) + eps) * w + b.

    streams    X_1 .. X_n [T, W], all E[token] at the start
    run:       layers 0 .. start-1 once, layers start .. stop-1 `times` times, then the remaining layers; every
               pass has keys, values and states of its own
    sublayer q (1: mixer, 2: feed-forward, where there is one):
               y = ls_q * f(LN_q(sum_s in_q[s] X_s));   X_t <- sum_s mix_q[s, t] X_s + m out_q[t] y   (all t at once)
    mixer "parallel":  left_scale * attention(h) + right_scale * lru(h)
      attention (H heads, G key/value heads):  q, k, v = Wq h, Wk h, Wv h;  q, k <- rms per head times a weight, then
               value i of the first `dims` turns with value i + dims/2 by p base^(-2i/dims) / factor
               s_ij = (q_i . k_j) scale for 0 <= i - j < window;  softmax;  Wo concat_heads(p v)
      lru:     g = gelu_tanh(Wy h + by);  u = conv(Wx h + bx) + bc;  per block b of the channels
               r = sigmoid(Ra_b u_b + ra_b),  i = sigmoid(Ri_b u_b + ri_b)
               a = exp(-8 r softplus(lam));  S_t = a S_{t-1} + sqrt(1 - a^2) i u;  Wo (S g)
    mixer "mlstm":     q = Wq h D^(-1/2), k = Wk h, v = Wv h;  c(z) = cap tanh(z / cap)
               i = c(Wi h + bi), f = log sigmoid(c(Wf h + bf));  m_t = max(f + m_{t-1}, i), m_{-1} = 0
               S_t = e^(f + m_{t-1} - m_t) S_{t-1} + e^(i - m_t) k v^T, the same for n_t with k alone
               o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6);  Wo (concat_heads(rms(o)) w * sigmoid(Wg h))
    ff "moe":  s = sigmoid(R h); the `top` largest are chosen;  sum_chosen Wd_e (silu(Wg_e s_e h) * (Wu_e s_e h))
    logits   = E LN_final(sum_t X_t)

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


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------ streams
def read_streams(X: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """X [T, streams, W], w_in [streams] -> [T, W]"""
    u = torch.zeros(X.shape[0], X.shape[2])
    for s in range(X.shape[1]):
        u = u + w_in[s] * X[:, s]
    return u


def write_streams(X: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, w_out: torch.Tensor, m: float) -> torch.Tensor:
    """a row of mix per stream before, a column per stream after; the old streams alone are read"""
    out = torch.zeros_like(X)
    for t in range(X.shape[1]):
        for s in range(X.shape[1]):
            out[:, t] += mix[s, t] * X[:, s]
        out[:, t] += m * w_out[t] * y
    return out


# ---------------------------------------------------------------- attention
def turn(x: torch.Tensor, pos: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, D]: values i and i + dims / 2 of every head turn together, i < dims / 2."""
    if not rot or not rot.get("dims"):
        return x
    dims = rot["dims"]
    half = dims // 2
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) / factor for i in range(half)], dtype=torch.float32)
    a = pos.to(torch.float32)[:, None] * f[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out = x.clone()
    out[..., :half] = u * cos - v * sin
    out[..., half:dims] = v * cos + u * sin
    return out


def window_attention(q, k, v, scale, window=None, pos0=0):
    """q [T, H, D] (positions pos0 ..), k [S, G, D], v [S, G, Dv] -> [T, H, Dv].  Row i sees keys j with
    0 <= i - j < window."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    out = torch.zeros(T, H, v.shape[2])
    i, j = torch.arange(pos0, pos0 + T)[:, None], torch.arange(S)[None, :]
    hidden = (j > i) | ((i - j >= window) if window else torch.zeros(T, S, dtype=torch.bool))
    for a in range(H):
        g = a // (H // G)
        s = ((q[:, a] @ k[:, g].T) * scale).masked_fill(hidden, float("-inf"))
        out[:, a] = torch.softmax(s, dim=-1) @ v[:, g]
    return out


def attention(h, w, pre, m, eps, rounding=None):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rms((h @ w[pre + "q"].T).view(T, H, D), eps) * w[pre + "q.norm"]
    k = rms((h @ w[pre + "k"].T).view(T, G, D), eps) * w[pre + "k.norm"]
    v = (h @ w[pre + "v"].T).view(T, G, Dv)
    q, k = turn(q, pos, m.get("rot")), turn(k, pos, m.get("rot"))
    q, k, v = _round(q, rounding), _round(k, rounding), _round(v, rounding)
    window = (m.get("mask") or {}).get("size")
    o = _round(window_attention(q, k, v, m["scale"], window).reshape(T, H * Dv), rounding)
    return o @ w[pre + "o"].T


# ------------------------------------------------------- gated linear recurrence
def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor, before: Optional[torch.Tensor] = None):
    """u [T, C], w [C, taps] (its last column meets the newest input), b [C]; before [taps - 1, C]: the inputs
    ahead of u, zeros when absent"""
    T, taps = u.shape[0], w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, u.shape[1]) if before is None else before, u])
    out = b.expand(T, -1).clone()
    for j in range(taps):
        out = out + w[:, j] * full[j:j + T]
    return out


def block_linear(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C] in equal parts, each through its own matrix w[p] and bias b[p]"""
    parts = u.view(u.shape[0], w.shape[0], -1)
    return torch.stack([parts[:, p] @ w[p].T + b[p] for p in range(w.shape[0])], dim=1).reshape(u.shape)


def lru_scan(u, r, i, lam, state=None):
    """u, r, i [T, C] (r and i after their sigmoids), lam [C] -> (S [T, C], the state after the last token)"""
    S = torch.zeros(u.shape[1]) if state is None else state.clone()
    log_a = -8.0 * r * torch.log1p(torch.exp(lam))
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return out, S


def lru(h, w, pre, m, eps, rounding=None):
    g = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = causal_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    ur = _round(u, rounding)
    r = torch.sigmoid(block_linear(ur, w[pre + "ra"], w[pre + "ra.b"]))
    i = torch.sigmoid(block_linear(ur, w[pre + "ri"], w[pre + "ri.b"]))
    S, _ = lru_scan(u, r, i, w[pre + "lam"])
    return _round(S * g, rounding) @ w[pre + "o"].T


def parallel(h, w, pre, m, eps, rounding=None):
    return (m["left_scale"] * attention(h, w, pre + "left.", m["left"], eps, rounding) +
            m["right_scale"] * lru(h, w, pre + "right.", m["right"], eps, rounding))


# -------------------------------------------------------------------- mLSTM
def mlstm_gates(zi, zf, cap):
    """zi, zf [T, H]: the gates' sums, biases included -> (log input gate, log forget gate)"""
    i, f = cap * torch.tanh(zi / cap), cap * torch.tanh(zf / cap)
    return i, -torch.log1p(torch.exp(-f.abs())) + torch.clamp(f, max=0.0)


def mlstm_scan(q, k, v, i, f, state=None):
    """q (scaled), k [T, H, D], v [T, H, Dv], i, f [T, H] -> (o [T, H, Dv], (m [H], n [H, D], S [H, D, Dv]))"""
    T, H, D = q.shape
    if state is None:
        m, n, S = torch.zeros(H), torch.zeros(H, D), torch.zeros(H, D, v.shape[2])
    else:
        m, n, S = (t.clone() for t in state)
    out = torch.zeros(T, H, v.shape[2])
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(dim=1) / den[:, None]
    return out, (m, n, S)


def mlstm(h, w, pre, m, eps, rounding=None):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[pre + "k"].T).view(T, H, D)
    v = (h @ w[pre + "v"].T).view(T, H, Dv)
    i, f = mlstm_gates(h @ w[pre + "i"].T + w[pre + "i.b"], h @ w[pre + "f"].T + w[pre + "f.b"], m["gate_cap"])
    o, _ = mlstm_scan(q, k, v, i, f)
    o = rms(o, eps).reshape(T, H * Dv) * w[pre + "norm"] * torch.sigmoid(h @ w[pre + "g"].T)
    return _round(o, rounding) @ w[pre + "o"].T


MIXERS = {"parallel": parallel, "mlstm": mlstm}


# ------------------------------------------------------------- feed-forward
def expert(h, w, pre, rounding=None):
    g, u = h @ w[pre + "gate"].T, h @ w[pre + "up"].T
    return _round(g * torch.sigmoid(g) * u, rounding) @ w[pre + "down"].T


def route(z, top):
    """z [T, E] logits -> (weights [T, E], how far the last chosen logit lies above the first unchosen [T])"""
    s = torch.sigmoid(z)
    order = torch.sort(s, dim=-1, descending=True, stable=True).indices
    out = torch.zeros_like(z)
    out.scatter_(1, order[:, :top], torch.gather(s, 1, order[:, :top]))
    ranked = torch.gather(z, 1, order)
    gap = ranked[:, top - 1] - ranked[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf)
    return out, gap


def routed(h, w, pre, f, rounding=None, gaps: Optional[List[torch.Tensor]] = None):
    weights, gap = route(h @ w[pre + "router"].T, f["router"]["top"])
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        rows = torch.nonzero(weights[:, e])[:, 0]
        if len(rows):
            out[rows] += expert(weights[rows, e, None] * h[rows], w, f"{pre}e{e}.", rounding)
    return out


# -------------------------------------------------------------------- model
def run_order(config: dict) -> List[int]:
    n, lp = len(config["layers"]), config.get("loop")
    if not lp:
        return list(range(n))
    return (list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] +
            list(range(lp["stop"], n)))


def forward(config: dict, w: Dict[str, torch.Tensor], tokens, rounding: Optional[str] = None,
            trace: Optional[List[torch.Tensor]] = None, gaps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab]; trace gets the sum of the streams after every layer run, gaps every router's margin."""
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = x[:, None, :].expand(-1, config["streams"], -1).clone()

    def sublayer(q, L, f):
        nonlocal X
        hc = f"{L}hc{q}."
        u = read_streams(X, w[hc + "in"])
        h = _round(layer_norm(u, w[f"{L}norm{q}"], w[f"{L}norm{q}.b"], eps), rounding)
        X = write_streams(X, w[f"{L}ls{q}"] * f(h), w[hc + "mix"], w[hc + "out"], mult)

    for i in run_order(config):
        layer, L = config["layers"][i], f"l{i}."
        sublayer(1, L, lambda h: MIXERS[layer["type"]](h, w, L + "mix.", layer["mixer"], eps, rounding))
        if layer["mlp"] is not None:
            sublayer(2, L, lambda h: routed(h, w, L + "mlp.", layer["mlp"], rounding, gaps))
        if trace is not None:
            trace.append(X.sum(dim=1))
    h = _round(layer_norm(X.sum(dim=1), w["final.norm"], w["final.norm.b"], eps), rounding)
    return h @ w["embed"].T
