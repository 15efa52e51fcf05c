"""The Salivik design on the GPU: each mechanism's kernel alone against the plain
restatement, then whole models through the engine under every way of cutting the
work, and greedy generation through the library's own entry point."""
import copy

import numpy as np
import pytest
import torch

import plain_salivik as ps
from salivik_models import CONFIGS, model
from helpers import rel_err, run_trace, trace_batches, trace_tail, trace_whole

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64


def ops():
    from janas_b200.csrc import ops as o
    return o


def rnd(*shape, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed * 7919 + sum(shape) + len(shape))
    return torch.randn(*shape, generator=g) * scale


def bf(x):
    return x.to(torch.bfloat16).float()


def close(got, want, tol, what=""):
    err = (got - want).abs().max() / want.abs().max()
    assert err <= tol, f"{what} {err:.3e}"


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def row_arrays(rows):
    """rows: per sequence (first position, count) -> positions and sequences of all rows."""
    row_pos = torch.tensor([p for (p0, cnt) in rows for p in range(p0, p0 + cnt)], dtype=torch.int32)
    row_seq = torch.tensor([i for i, (p0, cnt) in enumerate(rows) for _ in range(cnt)], dtype=torch.int32)
    return row_pos, row_seq


def cuts(total, sizes):
    """(first, count) pieces of 0 .. total whose sizes cycle through ``sizes``."""
    out, at, j = [], 0, 0
    while at < total:
        n = min(sizes[j % len(sizes)], total - at)
        out.append((at, n))
        at, j = at + n, j + 1
    return out


class Paged:
    """Pages of several sequences that lie in no order."""

    def __init__(self, lens, seed):
        need = [(n + PAGE - 1) // PAGE for n in lens]
        self.lens = lens
        self.n_pages = sum(need) + 3
        perm = torch.randperm(self.n_pages, generator=torch.Generator().manual_seed(seed)).tolist()
        self.table = torch.full((len(lens), (max(need) + 7) // 8 * 8), -1, dtype=torch.int32)
        for i, n in enumerate(need):
            for j in range(n):
                self.table[i, j] = perm.pop()

    def fill(self, per_seq, dtype):
        """per_seq[i]: [len, heads, dim] -> a cache tensor [pages, heads, PAGE, dim]"""
        heads, dim = per_seq[0].shape[1:]
        c = torch.zeros(self.n_pages, heads, PAGE, dim)
        for i, n in enumerate(self.lens):
            for t in range(n):
                c[int(self.table[i, t // PAGE]), :, t % PAGE] = per_seq[i][t]
        return c.to(dtype).to(DEV)

    def read(self, cache, seq, pos):
        return cache[int(self.table[seq, pos // PAGE]), :, pos % PAGE]


def tables(rot, n_pos):
    """cos and sin as the library makes them, from the plain form's frequencies."""
    return ops().rope_table(ps.frequencies(rot).to(DEV), n_pos, ps.amplitude(rot))


# ------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("rot", [{"base": 1000.0, "dims": 10},
                                 {"base": 10000.0, "dims": 16,
                                  "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}},
                                 {"base": 500.0, "dims": 6, "scaling": {"factor": 1.0, "original": 64, "fast": 2.0, "slow": 0.5}}])
def test_rotation_table(rot):
    """The position part's own table (frequencies, ramp, amplitude) against the plain form's angles."""
    from janas_b200.config import PartSpec
    from janas_b200.parts import build_part
    params = {"rotary_dim": rot["dims"], "theta": rot["base"], "max_positions": 1 << 20}
    if "scaling" in rot:
        params["yarn"] = rot["scaling"]
    pos = build_part("position", PartSpec("rope_neox", params), torch.float32, DEV)
    pos.prepare(700)
    ang = torch.arange(700, dtype=torch.float32)[:, None] * ps.frequencies(rot)[None, :]
    # an angle's own rounding grows with the position
    for got, want in ((pos.cos, torch.cos(ang.double())), (pos.sin, torch.sin(ang.double()))):
        assert (got.cpu().double() - want * ps.amplitude(rot)).abs().max() <= 3e-4 * ps.amplitude(rot)
        assert (got.cpu().double()[:20] - want[:20] * ps.amplitude(rot)).abs().max() <= 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,W,S", [(1, 50, 0), (5, 64, 1), (130, 300, 3), (9, 2048, 2), (3, 37, 5)])
def test_join_of_two_streams(dtype, n, W, S):
    """The residual stream with what is still to be added, and the embedding output, side by side; the
    stream is left at zero."""
    x, e = rnd(n, W, seed=1), rnd(n, W, seed=2)
    delta = rnd(S, n, W, seed=3) if S else None
    xd = x.to(DEV).clone()
    got = ops().join_rows(xd, None if delta is None else delta.to(DEV), e.to(DEV), dtype).float().cpu()
    want = torch.cat([x + (delta.sum(0) if S else 0.0), e], dim=1)
    close(got, want, 1e-6 if dtype == torch.float32 else 5e-3)
    assert float(xd.abs().max()) == 0.0


@pytest.mark.parametrize("n,ff,S,limit", [(1, 70, 1, 0.8), (5, 1000, 2, 2.0), (40, 512, 1, 7.0), (300, 136, 1, 0.5)])
def test_clamped_unit(n, ff, S, limit):
    """Values far beyond the limits on both sides, on one side of the gate alone, through the
    element-wise kernel and the product's own epilogue."""
    z = rnd(S, n, 2 * ff, scale=2.0, seed=2)
    z[:, 0, :8] = torch.tensor([-40.0, 40.0, -9.0, 9.0, 0.0, 1e4, -1e4, 0.3])
    z[:, 0, ff:ff + 8] = torch.tensor([40.0, -40.0, 9.0, 9.0, -9.0, 1e4, -1e4, 0.0])
    want = ps.clamped(z.sum(0)[:, :ff], z.sum(0)[:, ff:], limit)
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
        got = ops().swiglu(z.to(DEV), dt, 1.702, limit, 1.0).float().cpu()
        close(got, want, tol)
    k = 96
    h, w = bf(rnd(n, k, seed=3)), bf(rnd(2 * ff, k, seed=4) / k ** 0.5) * 2.0
    got = ops().linear_swiglu(h.to(torch.bfloat16).to(DEV), w.to(torch.bfloat16).to(DEV), 1.702, limit, 1.0)
    assert got is not None and ops().gemm_tc_error() == 0
    p = h @ w.T
    close(got.float().cpu(), ps.clamped(p[:, :ff], p[:, ff:], limit), 6e-3)
    # the plain unit is what it was: SiLU(gate) * up
    close(ops().swiglu(z.to(DEV), torch.float32).cpu(), torch.nn.functional.silu(z.sum(0)[:, :ff]) * z.sum(0)[:, ff:], 2e-6)


@pytest.mark.parametrize("E,top,S", [(12, 2, 1), (5, 5, 2), (3, 1, 1), (64, 7, 3), (130, 4, 1)])
def test_router_with_a_softmax_over_the_chosen(E, top, S):
    n = 150
    P = rnd(S, n, E + 5, seed=E)
    bias = rnd(E, seed=1)
    got, _ = ops().moe_route(P.to(DEV), 5, E, None, 1, 1, top, E, 1.0, chosen_softmax=True, bias=bias.to(DEV))
    want, gap = ps.route(P.sum(0)[:, 5:] + bias, top)
    got = got.cpu()
    assert gap.min() > 1e-6
    assert torch.equal(got != 0, want != 0) and int((got != 0).sum(1).max()) == top
    assert (got - want).abs().max() <= 2e-6 and (got.sum(1) - 1).abs().max() <= 1e-6


def test_the_routers_bias_decides_and_weighs():
    """A bias changes the choice and is part of the weights (a correction changes the choice alone); the
    other logits do not enter the weights, however large they are all together."""
    z = torch.tensor([[2.0, 1.9, 1.8, 1.7, 0.0, 0.0]])
    bias = torch.tensor([0.0, 0.0, 0.0, 3.0, 2.5, 0.0])
    w, _ = ops().moe_route(z.to(DEV), 0, 6, None, 1, 1, 2, 6, 1.0, chosen_softmax=True, bias=bias.to(DEV))
    assert torch.nonzero(w[0]).flatten().tolist() == [3, 4]
    assert (w[0].cpu()[3:5] - torch.softmax(torch.tensor([4.7, 2.5]), 0)).abs().max() <= 1e-6
    w, _ = ops().moe_route(z.to(DEV), 0, 6, bias.to(DEV), 1, 1, 2, 6, 1.0, chosen_softmax=True)
    assert torch.nonzero(w[0]).flatten().tolist() == [3, 4]
    assert (w[0].cpu()[3:5] - torch.softmax(torch.tensor([1.7, 0.0]), 0)).abs().max() <= 1e-6
    # logits whose exponentials overflow
    w, _ = ops().moe_route((z + 300.0).to(DEV), 0, 6, None, 1, 1, 2, 6, 1.0, chosen_softmax=True)
    assert (w[0].cpu()[:2] - torch.softmax(torch.tensor([2.0, 1.9]), 0)).abs().max() <= 3e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,E,ff,sf,S", [(9, 5, 12, 20, 2), (70, 3, 7, 9, 1), (2, 8, 32, 0, 3), (1, 2, 5, 64, 1)])
def test_experts_and_a_shared_expert(dtype, n, E, ff, sf, S):
    """Clamped units with constants of their own for the experts and the shared expert; unchosen
    experts' sums are not used even where they are not numbers."""
    z = rnd(S, n, 2 * (E * ff + sf) + 3, scale=2.0, seed=1)
    w = torch.rand(n, E + 2, generator=torch.Generator().manual_seed(2)) + 0.1
    w[:, 1] = 0.0
    z[:, :, 2 * ff:4 * ff] = float("nan")
    got = ops().gated_weighted(z.to(DEV), w.to(DEV), E, ff, "silu", dtype, shared_ff=sf,
                               units=(1.702, 1.1, 1.0, 1.702, 0.6, 1.0)).float().cpu()
    full = z.sum(0)
    ex = full[:, :2 * E * ff].reshape(n, E, 2, ff)
    want = (ps.clamped(ex[:, :, 0], ex[:, :, 1], 1.1) * w[:, :E, None])
    want[:, 1] = 0.0
    sh = full[:, 2 * E * ff:2 * E * ff + 2 * sf]
    want = torch.cat([want.reshape(n, E * ff), ps.clamped(sh[:, :sf], sh[:, sf:], 0.6)], dim=1)
    close(got, want, 2e-6 if dtype == torch.float32 else 5e-3)


# ------------------------------------------------------------------- retention
@pytest.mark.parametrize("H,D,Dv,rot,S,col0,n", [(2, 16, 24, 12, 1, 0, 9), (3, 10, 6, 4, 2, 5, 70), (4, 64, 128, 64, 3, 8, 5),
                                                 (2, 24, 8, 0, 1, 0, 130), (1, 40, 40, 8, 2, 4, 3)])
def test_turned_and_scaled_heads(H, D, Dv, rot, S, col0, n):
    src = rnd(S, n, col0 + H * (2 * D + Dv) + 7, seed=3)
    pos = torch.randint(0, 500, (n,), generator=torch.Generator().manual_seed(4), dtype=torch.int32)
    spec = {"base": 800.0, "dims": rot} if rot else None
    cos, sin = tables(spec, 512) if rot else (None, None)
    got = ops().turn_heads(src.to(DEV), col0, H, D, Dv, cos, sin, pos.to(DEV), D ** -0.5).cpu()
    f = src.sum(0)[:, col0:]
    q = ps.turn(f[:, :H * D].reshape(n, H, D), pos, spec).reshape(n, -1)
    k = ps.turn(f[:, H * D:2 * H * D].reshape(n, H, D), pos, spec).reshape(n, -1) * D ** -0.5
    close(got, torch.cat([q, k, f[:, 2 * H * D:2 * H * D + H * Dv]], dim=1), 1e-4)
    # with the table itself the arithmetic is exact to rounding
    if rot:
        c, s = cos.cpu()[pos.long()][:, None], sin.cpu()[pos.long()][:, None]
        a = f[:, :H * D].reshape(n, H, D)
        u, v = a[..., :rot // 2], a[..., rot // 2:rot]
        want = torch.cat([u * c - v * s, v * c + u * s, a[..., rot:]], dim=-1).reshape(n, -1)
        close(got[:, :H * D], want, 1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,H,Dv,S", [(5, 4, 16, 1), (70, 3, 10, 2), (300, 2, 128, 3), (8, 20, 128, 5), (2, 5, 256, 1), (4, 1, 24, 1),
                                      (3, 2, 300, 2)])
def test_norm_per_head_and_silu_gate(dtype, n, H, Dv, S):
    y, g = rnd(n, H * Dv, scale=3.0, seed=1), rnd(S, n, H * Dv + 8, seed=2)
    gs = g.sum(0)[:, 4:4 + H * Dv]
    want = ps.rms(y.view(n, H, Dv), 1e-5).reshape(n, -1) * gs * torch.sigmoid(gs)
    for few in (False, True):
        got = ops().gated_part_norm(y.to(DEV), H, None, 1e-5, dtype, post=g.to(DEV), post_col0=4, few_rows=few,
                                    post_silu=True).float().cpu()
        close(got, want, 3e-6 if dtype == torch.float32 else 1e-2)


def run_retention(src, H, D, Dv, decay, rot, sizes, max_len=0):
    """src [T, H (2 D + Dv)] cut into portions, each through the rotation and the recurrence with the
    state the last one left."""
    T = src.shape[0]
    cos, sin = tables(rot, T)
    st = torch.zeros(3, H, D, Dv, device=DEV)
    outs = []
    for p0, cnt in cuts(T, sizes):
        row_pos, _ = row_arrays([(p0, cnt)])
        a = ops().turn_heads(src[None, p0:p0 + cnt].contiguous().to(DEV), 0, H, D, Dv, cos, sin, row_pos.to(DEV), D ** -0.5)
        outs.append(ops().matrix_state_scan(a, H, H, D, Dv, 2 * H * D, H * D, 0, st, i32([0] * cnt), i32([1]), 1,
                                            every_row_starts=cnt == 1, decay=torch.tensor(decay).to(DEV),
                                            max_len=cnt if max_len else 0).cpu())
    assert float(st[0].abs().max()) == 0.0 and float(st[2].abs().max()) == 0.0
    return torch.cat(outs), st[1].cpu()


@pytest.mark.parametrize("sizes,max_len", [([700], 0), ([700], 1), ([2], 0), ([64, 3, 61, 2, 130], 1), ([1], 0), ([300, 1, 1, 280], 1)])
def test_retention_state_over_portions(sizes, max_len):
    H, D, Dv, decay = 3, 12, 20, [0.5, 0.97, 1.0]
    rot = {"base": 600.0, "dims": 8}
    src = rnd(700, H * (2 * D + Dv), seed=5)
    got, st = run_retention(src, H, D, Dv, decay, rot, sizes, max_len)
    pos = torch.arange(700)
    q = ps.turn(src[:, :H * D].reshape(-1, H, D), pos, rot)
    k = ps.turn(src[:, H * D:2 * H * D].reshape(-1, H, D), pos, rot) * D ** -0.5
    want, ws = ps.retention_scan(q, k, src[:, 2 * H * D:].reshape(-1, H, Dv), decay)
    for a in range(H):
        close(got.view(-1, H, Dv)[:, a], want[:, a], 5e-4 if decay[a] == 1.0 else 1e-4, f"head {a}")
    close(st, ws, 5e-4)


def test_retention_keeps_and_loses_a_far_token():
    """One token's value is written 600 tokens before the query that asks for it (in values that do
    not turn): kept whole by a decay of 1, mostly by 0.999, lost by 0.9."""
    H, D, Dv, T = 3, 8, 4, 700
    src = torch.zeros(T, H * (2 * D + Dv))
    src[50, H * D + 7::D][:H] = 1.0
    for a in range(H):
        src[50, H * D + a * D + 7] = D ** 0.5
        src[650, a * D + 7] = 1.0
        src[50, 2 * H * D + a * Dv:2 * H * D + (a + 1) * Dv] = torch.tensor([1.0, 2.0, -3.0, 4.0])
    for sizes in ([T], [100, 2, 400], [1]):
        got, _ = run_retention(src, H, D, Dv, [1.0, 0.999, 0.9], {"base": 100.0, "dims": 4}, sizes, 1)
        got = got.view(T, H, Dv)
        v = torch.tensor([1.0, 2.0, -3.0, 4.0])
        assert (got[650, 0] - v).abs().max() <= 1e-5
        assert (got[650, 1] - v * 0.999 ** 600).abs().max() <= 1e-4
        assert got[650, 2].abs().max() <= 1e-20
        assert got[649].abs().max() == 0.0 and got[651].abs().max() == 0.0


# ------------------------------------------------------ windows, sinks, values that are keys
def run_attention(dtype, nh, nkv, hd, rot, lens, rows, window, sink, standout=(), seed=0, decode=False, mode="plain"):
    """The products' sums [q | k] of whole sequences go through the kernel that turns and appends (pages in
    no order; the values are the keys' sums), then the rows of ``rows`` ask.  standout: (sequence, key
    position, query position): that key is made to dominate that query's scores through its last value,
    which does not turn, and its other values are 5 (which the value shows and the turned key does not)."""
    P = Paged(lens, seed)
    scale = 0.25
    prods = [rnd(n, (nh + nkv) * hd, scale=0.5, seed=seed + 10 + i) for i, n in enumerate(lens)]
    for (si, kp, qp) in standout:
        k = prods[si][:, nh * hd:].view(-1, nkv, hd)
        q = prods[si][:, :nh * hd].view(-1, nh, hd)
        k[:, :, hd - 1] = 0.0
        k[kp, :, :hd - 1] = 5.0
        q[qp] = 0.0
        q[qp, :, hd - 1] = 12.0
        k[kp, :, hd - 1] = 8.0                              # a score of 24 where all others are 0
    spec = {"base": 300.0, "dims": rot} if rot else None
    cos, sin = tables(spec, max(lens)) if rot else (None, None)
    kc, vc = (torch.zeros(P.n_pages, nkv, PAGE, hd, dtype=dtype, device=DEV) for _ in range(2))
    want, qs = [], []
    tol_q = 2e-4 if dtype == torch.float32 else 1e-2
    for i, n in enumerate(lens):
        pos = torch.arange(n)
        q = ps.turn(prods[i][:, :nh * hd].reshape(n, nh, hd), pos, spec)
        v = prods[i][:, nh * hd:].reshape(n, nkv, hd)
        k = ps.turn(v, pos, spec)
        if dtype == torch.bfloat16:
            q, k, v = bf(q), bf(k), bf(v)
        p0, cnt = rows[i]
        want.append(ps.window_attention(q[p0:p0 + cnt], k[:p0 + cnt], v[:p0 + cnt], scale, window, sink, p0))
        row_pos, row_seq = row_arrays([(0, 0)] * i + [(0, n)])
        got_q = ops().qkv_prepare_append(prods[i][None].contiguous().to(DEV), None, None, None, 0.0, cos, sin,
                                         row_pos.to(DEV), row_seq.to(DEV), P.table.to(DEV), kc, vc, nh,
                                         values_from_keys=True)
        close(got_q.float().cpu(), q, tol_q, "q")
        kh, vh = kc.float().cpu(), vc.float().cpu()
        for p in range(0, n, 13):
            assert torch.equal(P.read(vh, i, p), prods[i][p, nh * hd:].reshape(nkv, hd).to(dtype).float())
            assert (P.read(kh, i, p) - k[p]).abs().max() <= tol_q * k.abs().max()
        qs.append(got_q[p0:p0 + cnt])
    row_pos, row_seq = row_arrays(rows)
    chunk = ops().attention_chunk()
    max_chunks = int(row_pos.max()) // chunk + 1
    if window:
        max_chunks = min(max_chunks, (window - 1) // chunk + 2)
    kw = {}
    if mode == "plain":
        kw["force_simt"] = True
    elif not decode:
        per = ops().attention_block_positions(nh, nkv)
        r0, at = [], 0
        for (p0, cnt) in rows:
            r0.append(at)
            at += cnt
        kw["blocks"] = ops().attention_blocks(r0, [p for p, _ in rows], [c for _, c in rows], per, torch.device(DEV))
    got = ops().attention(torch.cat(qs), kc, vc, row_pos.to(DEV), row_seq.to(DEV), P.table.to(DEV), window or 0, scale,
                          max_chunks, decode=decode, sink=sink.to(DEV), **kw).float().cpu()
    assert ops().attn_tc_error() == 0
    return got, torch.cat(want)


ATT_KERNELS = [(torch.float32, "plain", 4, 2, 24, 8), (torch.bfloat16, "plain", 6, 3, 48, 30), (torch.float32, "plain", 3, 3, 10, 0),
               (torch.bfloat16, "tc", 4, 1, 64, 32), (torch.bfloat16, "tc", 2, 2, 128, 64)]


@pytest.mark.parametrize("dtype,mode,nh,nkv,hd,rot", ATT_KERNELS)
@pytest.mark.parametrize("decode", [False, True])
def test_a_key_that_stands_out(dtype, mode, nh, nkv, hd, rot, decode):
    """Far back, at a page's first and last place and a chunk's border: the row that asks gets the key's
    value, which is the key before it was turned, almost alone; then the first tokens of a sequence."""
    tol = 5e-4 if dtype == torch.float32 else 2e-2
    sink = torch.zeros(nh)
    lens = [700, 70]
    for kp in (0, 63, 64, 127, 128, 383, 384, 640):
        rows = [(699, 1), (69, 1)] if decode else [(650, 50), (0, 70)]
        got, want = run_attention(dtype, nh, nkv, hd, rot, lens, rows, None, sink, [(0, kp, 699)], kp, decode, mode)
        close(got, want, tol, f"key {kp}")
        assert (got[-2 if decode else 49, :, :hd - 1] - 5.0).abs().max() < 0.1
    for n in (1, 2, 3):
        rows = [(n - 1, 1)] if decode else [(0, n)]
        got, want = run_attention(dtype, nh, nkv, hd, rot, [n], rows, 37, sink, (), n, decode, mode)
        close(got, want, tol, f"length {n}")


@pytest.mark.parametrize("dtype,mode,nh,nkv,hd,rot", ATT_KERNELS)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 37, 64, 128, 200])
def test_keys_just_inside_and_outside_a_window(dtype, mode, nh, nkv, hd, rot, decode, window):
    tol = 5e-4 if dtype == torch.float32 else 2e-2
    sink = torch.zeros(nh)
    for qp in (window - 1, window, 299, 450):
        for kp, inside in ((qp + 1 - window, True), (qp - window, False)):
            if kp < 0 or (window == 1 and not inside and kp == qp):
                continue
            rows = [(qp, 1)] if decode else [(max(0, qp - 20), min(21, qp + 1))]
            got, want = run_attention(dtype, nh, nkv, hd, rot, [451], rows, window, sink, [(0, kp, qp)], qp, decode, mode)
            if kp != qp:
                assert (float(got[-1, :, :hd - 1].mean()) > 4.5) == inside
            close(got, want, tol, f"window {window} query {qp} key {kp}")


@pytest.mark.parametrize("dtype,mode,nh,nkv,hd,rot", ATT_KERNELS)
@pytest.mark.parametrize("decode", [False, True])
def test_a_sink_takes_its_share(dtype, mode, nh, nkv, hd, rot, decode):
    """Sinks that outweigh every key, that nobody feels, and the one in the denominator (a sink of score 0)
    on a first token, which then keeps e^s / (1 + e^s) of its value."""
    tol = 5e-4 if dtype == torch.float32 else 2e-2
    sink = torch.linspace(-30.0, 12.0, nh)
    rows = [(299, 1), (69, 1)] if decode else [(260, 40), (0, 70)]
    got, want = run_attention(dtype, nh, nkv, hd, rot, [300, 70], rows, 50, sink, (), 3, decode, mode)
    close(got, want, tol)
    assert got[-1, nh - 1].abs().max() < 0.1 * got[-1, 0].abs().max()
    got, want = run_attention(dtype, nh, nkv, hd, rot, [1], [(0, 1)], 50, torch.zeros(nh), (), 5, decode, mode)
    close(got, want, tol)


# ------------------------------------------------------------ latent attention
@pytest.mark.parametrize("nh,nkv,window", [(2, 2, 0), (3, 1, 130), (4, 4, 64), (1, 1, 1), (8, 2, 200)])
def test_keys_of_192_and_values_of_128_on_the_tensor_cores(nh, nkv, window):
    """Prompt rows of unequal sequences, whole and from a later position on, with a sink; then one key made
    to stand out just inside and just outside the window, and far back without one."""
    hd, vd, scale = 192, 128, 0.05
    assert ops().lib().jb_attn_tc_prefill_ok(nh, nkv, hd, vd)
    sink = torch.linspace(-1.0, 2.0, nh)
    per = ops().attention_block_positions(nh, nkv, hd)
    assert per == 128 // (nh // nkv)

    def run(lens, rows, qs, ks, vs):
        P = Paged(lens, 11)
        want = torch.cat([ps.window_attention(qs[i], ks[i][:p0 + cnt], vs[i][:p0 + cnt], scale, window or None, sink, p0)
                          for i, (p0, cnt) in enumerate(rows)])
        row_pos, row_seq = row_arrays(rows)
        r0, at = [], 0
        for (_, cnt) in rows:
            r0.append(at)
            at += cnt
        blocks = ops().attention_blocks(r0, [p for p, _ in rows], [c for _, c in rows], per, torch.device(DEV))
        chunk = ops().attention_chunk()
        got = ops().attention(torch.cat(qs).to(torch.bfloat16).to(DEV), P.fill(ks, torch.bfloat16), P.fill(vs, torch.bfloat16),
                              row_pos.to(DEV), row_seq.to(DEV), P.table.to(DEV), window, scale,
                              int(row_pos.max()) // chunk + 1, blocks=blocks, sink=sink.to(DEV)).float().cpu()
        assert ops().attn_tc_error() == 0
        return got, want

    lens, rows = [1, 300, 131, 520], [(0, 1), (0, 300), (100, 31), (0, 520)]
    qs = [bf(rnd(cnt, nh, hd, seed=i)) for i, (_, cnt) in enumerate(rows)]
    ks = [bf(rnd(n, nkv, hd, seed=10 + i)) for i, n in enumerate(lens)]
    vs = [bf(rnd(n, nkv, vd, seed=20 + i)) for i, n in enumerate(lens)]
    got, want = run(lens, rows, qs, ks, vs)
    close(got, want, 2e-2)
    for qp in (max(window - 1, 0), window + 3, 383, 599):
        for kp, inside in ((max(0, qp + 1 - window) if window else 3, True), (qp - window, False)):
            if kp < 0 or kp > qp or (not window and not inside):
                continue
            rows = [(max(0, qp - 30), min(31, qp + 1))]
            q, k, v = bf(rnd(rows[0][1], nh, hd, seed=kp)), bf(rnd(600, nkv, hd, scale=0.3, seed=kp + 1)), bf(rnd(600, nkv, vd, seed=kp + 2))
            q[-1] = 0.0
            q[-1, :, 150] = 20.0                    # a place that only the keys' third part has
            k[:, :, 150] = 0.0
            k[kp, :, 150] = 24.0
            v[kp] = 5.0
            got, want = run([600], rows, [q], [k], [v])
            close(got, want, 2e-2, f"query {qp} key {kp}")
            assert (float(got[-1].mean()) > 4.5) == inside


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,R,dims,Dv,C,Cq,window,halves", [(4, 16, 8, 8, 24, 40, 24, 37, True), (3, 10, 6, 6, 6, 22, 14, 0, True),
                                                              (2, 64, 64, 64, 128, 96, 48, 130, True), (1, 24, 16, 12, 40, 64, 32, 64, True),
                                                              (2, 16, 8, 8, 16, 32, 16, 20, False)])
def test_latent_attention_steps(dtype, H, D, R, dims, Dv, C, Cq, window, halves):
    """The mixer's kernels in a row, from the products' sums to the heads' outputs, against the plain
    form that builds every head's keys and values: prompt rows of two sequences, then one more token
    of each from the cache."""
    eps, scale = 1e-5, 0.6 / (D + R) ** 0.5
    rot = {"base": 900.0, "dims": dims, "scaling": {"factor": 4.0, "original": 100, "fast": 5.0, "slow": 0.5}}
    lens = [150, 70]
    P = Paged([n + 1 for n in lens], 5)
    cos, sin = tables(rot, 256)
    wq, wc = 1 + rnd(Cq, scale=0.2, seed=1), 1 + rnd(C, scale=0.2, seed=2)
    w_uq, w_uk, w_uv = rnd(H * (D + R), Cq, seed=3) / Cq ** 0.5, rnd(H * D, C, seed=4) / C ** 0.5, rnd(H * Dv, C, seed=5) / C ** 0.5
    if dtype == torch.bfloat16:
        w_uq, w_uk, w_uv = bf(w_uq), bf(w_uk), bf(w_uv)
    sink = rnd(H, seed=6)
    sums = [rnd(3, n + 1, Cq + C + R, seed=20 + i) for i, n in enumerate(lens)]
    cache = torch.zeros(P.n_pages, 1, PAGE, C + R, dtype=dtype, device=DEV)
    w_ukT = ops().transpose_heads(w_uk.to(dtype).to(DEV), H)

    def rd(x):
        return bf(x) if dtype == torch.bfloat16 else x

    def turned(x, pos):
        if halves:
            return ps.turn(x, pos, rot)
        # neighbours (2i, 2i + 1): the halves' form on reordered values
        order = torch.cat([torch.arange(0, dims, 2), torch.arange(1, dims, 2), torch.arange(dims, x.shape[-1])])
        out = torch.empty_like(x)
        out[..., order] = ps.turn(x[..., order], pos, rot)
        return out

    def plain(i, p0, cnt):
        z = sums[i].sum(0)
        T = lens[i] + 1
        pos = torch.arange(T)
        cq = rd(ps.norm(z[:, :Cq], wq, eps))
        c = rd(ps.norm(z[:, Cq:Cq + C], wc, eps))
        kr = rd(turned(z[:, None, Cq + C:], pos))
        q = (cq @ w_uq.T).reshape(T, H, D + R)
        q = torch.cat([rd(q[..., :D]), rd(turned(q[..., D:], pos))], dim=-1)
        k = torch.cat([(c @ w_uk.T).view(T, H, D), kr.expand(T, H, R)], dim=-1)
        v = (c @ w_uv.T).view(T, H, Dv)
        return ps.window_attention(q[p0:p0 + cnt], k[:p0 + cnt], v[:p0 + cnt], scale, window or None, sink, p0), c, kr

    def run(rows, decode):
        row_pos, row_seq = row_arrays(rows)
        Pm = torch.cat([sums[i][:, p0:p0 + cnt] for i, (p0, cnt) in enumerate(rows)], dim=1).contiguous().to(DEV)
        cq = ops().latent_down(Pm, Cq, wq.to(DEV), C, wc.to(DEV), R, cos, sin, row_pos.to(DEV), row_seq.to(DEV),
                               P.table.to(DEV), cache, eps, halves=halves)
        Q = ops().linear(cq, w_uq.to(dtype).to(DEV), force_simt=True)
        q_lat = ops().latent_queries(Q, w_ukT, H, D, R, C, cos, sin, row_pos.to(DEV), dtype, halves=halves)
        chunk = ops().attention_chunk()
        chunks = int(row_pos.max()) // chunk + 1
        if window:
            chunks = min(chunks, (window - 1) // chunk + 2)
        o = ops().attention(q_lat, cache, None, row_pos.to(DEV), row_seq.to(DEV), P.table.to(DEV), window, scale,
                            chunks, decode=decode, value_dim=C, head_major=True, sink=sink.to(DEV))
        A = torch.stack([ops().linear(o[h], w_uv.to(dtype).to(DEV)[h * Dv:(h + 1) * Dv], force_simt=True)
                         for h in range(H)])
        return A.float().sum(1).cpu().transpose(0, 1)          # [rows, H, Dv]

    tol = 1e-4 if dtype == torch.float32 else 4e-2
    got = run([(0, lens[0]), (0, lens[1])], False)
    close(got, torch.cat([plain(i, 0, lens[i])[0] for i in range(2)]), tol, "prompt")
    _, c, kr = plain(1, 0, lens[1])
    row = P.read(cache.float().cpu(), 1, lens[1] - 1).reshape(-1)
    assert (row - torch.cat([c[lens[1] - 1], kr[lens[1] - 1, 0]])).abs().max() <= (1e-4 if dtype == torch.float32 else 2e-2) * row.abs().max()
    got = run([(lens[0], 1), (lens[1], 1)], True)
    close(got, torch.cat([plain(i, lens[i], 1)[0] for i in range(2)]), tol, "one more token")


@pytest.mark.parametrize("dtype,C,R,H", [(torch.float32, 40, 8, 3), (torch.bfloat16, 40, 8, 3), (torch.bfloat16, 96, 32, 5),
                                         (torch.bfloat16, 22, 6, 2), (torch.bfloat16, 64, 16, 20),
                                         (torch.bfloat16, 128, 64, 40)])
@pytest.mark.parametrize("window", [1, 64, 75, 200])
def test_a_latent_just_inside_and_outside_a_window(dtype, C, R, H, window):
    """A cached row at a window's edge dominates a query's scores: inside, the weighted sum is that row's
    latent part; outside, it does not show."""
    scale, n = 0.1, 600
    for qp in (window - 1, window, 383, 599):
        for kp, inside in ((qp + 1 - window, True), (qp - window, False)):
            if kp < 0:
                continue
            rows_k = rnd(n, 1, C + R, scale=0.3, seed=kp)
            q = rnd(1, H, C + R, seed=kp + 1)
            d = q[0, 0] / q[0, 0].norm()
            q[0, :] = d * 6.0
            rows_k[kp, 0] = d * (14.0 / scale / 6.0)
            if dtype == torch.bfloat16:
                rows_k, q = bf(rows_k), bf(q)
            sink = torch.linspace(-1.0, 2.0, H)
            want = ps.window_attention(q, rows_k[:qp + 1], rows_k[:qp + 1, :, :C], scale, window, sink, qp)
            P = Paged([n], kp)
            for decode in (False, True):
                got = ops().attention(q.to(dtype).to(DEV), P.fill([rows_k], dtype), None, i32([qp]), i32([0]),
                                      P.table.to(DEV), window, scale, (window - 1) // ops().attention_chunk() + 2,
                                      decode=decode, value_dim=C, sink=sink.to(DEV)).float().cpu()
                close(got, want, 2e-5 if dtype == torch.float32 else 2e-2, f"window {window} query {qp} key {kp}")
            near = (want[0, 0] - rows_k[kp, 0, :C]).abs().max() < 0.05 * rows_k[kp, 0].abs().max()
            assert bool(near) == inside


# ------------------------------------------------------------------ whole models
LENGTHS = {"SA": [1, 2, 9, 70, 131, 260], "SB": [1, 3, 64, 65, 200, 410], "SC": [2, 17, 128, 129, 300, 520],
           "SD": [1, 5, 33, 64, 190, 330], "SE": [1, 2, 4, 30, 66, 140], "SF": [1, 3, 40, 129, 257, 420]}
FP32_TOL = 5e-5
BF16_TOL = 5e-2
CLOSE_CALL = 5e-2
_ENGINES = {}
_PLAIN = {}


def requests(name):
    rng = np.random.default_rng(900 + len(name) + ord(name[1]))
    return [rng.integers(0, CONFIGS[name]["vocab"], size=n).tolist() for n in LENGTHS[name]]


def engine(name, dtype, max_tokens=2048):
    from janas_b200.engine import Engine
    key = (name, dtype, max_tokens)
    if key not in _ENGINES:
        _ENGINES[key] = Engine.open(model(name)[0], dtype=dtype, max_tokens=max_tokens)
    return _ENGINES[key]


def plain_logits(name, toks, rounding=None):
    """The plain model's logits, and for every position how close the closest choice of any of its
    routers was."""
    key = (name, tuple(toks), rounding)
    if key not in _PLAIN:
        _, c, w = model(name)
        gaps = []
        logits = ps.forward(c, w, list(toks), rounding, None, gaps).numpy()
        m = torch.stack(gaps).min(0).values.numpy() if gaps else np.full(len(toks), np.inf)
        _PLAIN[key] = (logits, m)
    return _PLAIN[key]


def check(name, dtype, got, reqs, ids):
    for rid, toks in zip(ids, reqs):
        have = np.stack([got[rid][p] for p in range(len(toks))])
        if dtype == "float32":
            e = rel_err(have, plain_logits(name, toks)[0])
            assert e <= FP32_TOL, f"{name} {rid} len {len(toks)}: {e:.3e}"
        else:
            # With 16-bit products two of a router's logits that are closer than their rounding can change
            # places; such a token takes another expert in either implementation, which is no fault, and
            # the tokens after it see other keys, values and states.  Every token before the first such
            # close call is held to the limit, of the ones from there on a tenth may be over it (the
            # float32 runs hold every token to theirs).
            want, gap = plain_logits(name, toks, "bfloat16")
            assert np.isfinite(have).all()
            err = np.abs(have - want).max(1) / np.abs(want).max()
            close_calls = np.nonzero(gap < CLOSE_CALL)[0]
            first = int(close_calls[0]) if len(close_calls) else len(toks)
            assert (err[:first] <= BF16_TOL).all(), \
                f"{name} {rid} len {len(toks)}: {err[:first].max():.3e} at {np.nonzero(err[:first] > BF16_TOL)[0].tolist()}"
            over = np.nonzero(err[first:] > BF16_TOL)[0] + first
            assert len(over) <= (len(toks) - first + 9) // 10, f"{name} {rid} len {len(toks)}: over at {over.tolist()}"
            assert np.median(err) <= BF16_TOL / 3 and (err <= 0.8).all(), f"{name} {rid}: {err.max():.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, dtype):
    reqs = requests(name)
    got = run_trace(engine(name, dtype), trace_whole(reqs))
    check(name, dtype, got, reqs, [f"r{i}" for i in range(len(reqs))])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_layer_by_layer(name):
    """The residual stream after every layer run (a repeated layer counts every time)."""
    from janas_b200.engine.engine import StepEntry
    toks = requests(name)[3]
    _, c, w = model(name)
    trace = []
    ps.forward(c, w, toks, None, trace)
    e = engine(name, "float32")
    s = e.new_sequence()
    got = e.step_trace([StepEntry(s, toks, [])])
    e.free_sequence(s)
    assert len(got) == len(trace) == len(ps.run_order(c))
    for i, (g, t) in enumerate(zip(got, trace)):
        err = np.abs(np.asarray(g).reshape(t.shape) - t.numpy()).max() / t.abs().max().item()
        assert err <= 2e-5, f"layer run {i}: {err:.3e}"


def test_every_part_shows():
    """The plain model with one mechanism changed or left out is far from the engine's logits: the
    comparison tells."""
    name = "SA"
    toks = requests(name)[4]
    _, c, w = model(name)
    have = np.stack([run_trace(engine(name, "float32"), trace_whole([toks]))["r0"][p] for p in range(len(toks))])
    assert rel_err(have, ps.forward(c, w, toks).numpy()) <= FP32_TOL

    def put(key_end, value):
        def f(d, ww):
            hit = [k for k in ww if k.endswith(key_end)]
            assert hit
            for k in hit:
                ww[k] = torch.full_like(ww[k], value)
        return f

    def join_of_one(which):
        def f(d, ww):
            ww["loop.in"] = ww["loop.in"].clone()
            ww["loop.in"][:, which * d["width"]:(which + 1) * d["width"]] = 0.0
        return f

    L = [lambda d, i=i: d["layers"][i]["mixer"] for i in range(3)]
    M = [lambda d, i=i: d["layers"][i]["mlp"] for i in range(3)]
    changes = [lambda d, ww: L[0](d)["rot"].pop("scaling"),
               lambda d, ww: L[0](d)["rot"]["scaling"].update(factor=2.0),
               lambda d, ww: L[0](d)["rot"]["scaling"].update(fast=1.0),
               lambda d, ww: L[0](d)["rot"]["scaling"].update(slow=0.1),
               lambda d, ww: L[0](d)["rot"]["scaling"].update(original=400),
               lambda d, ww: L[0](d)["mask"].update(size=38),
               lambda d, ww: L[0](d)["mask"].update(size=36),
               lambda d, ww: L[0](d).update(scale=0.25),
               lambda d, ww: L[1](d)["rot"].update(dims=12),
               lambda d, ww: L[1](d)["rot"].update(base=400.0),
               lambda d, ww: L[1](d)["mask"].update(size=65),
               lambda d, ww: L[1](d)["mask"].update(size=63),
               lambda d, ww: L[1](d).update(scale=0.25),
               lambda d, ww: L[2](d)["rot"].update(dims=16),
               lambda d, ww: L[2](d).update(decay=[0.5, 0.97, 0.99]),
               lambda d, ww: L[2](d).update(decay=[0.97, 0.5, 0.999]),
               lambda d, ww: M[0](d).update(limit=0.9),
               lambda d, ww: M[1](d)["expert"].update(limit=1.3),
               lambda d, ww: M[1](d)["shared"].update(limit=0.9),
               lambda d, ww: M[1](d).update(shared=None),
               lambda d, ww: M[1](d)["router"].update(top=1),
               lambda d, ww: M[2](d)["router"].update(top=2),
               lambda d, ww: M[2](d)["expert"].update(limit=0.7),
               lambda d, ww: d["loop"].update(times=2),
               lambda d, ww: d["loop"].update(stop=2),
               lambda d, ww: d["loop"].update(start=0),
               lambda d, ww: d["norm"].update(eps=1e-2),
               join_of_one(0), join_of_one(1), put("mix.sink", -30.0), put("l1.mix.g", 0.0), put("l2.mix.g", 0.1),
               put("router.b", 0.0), put("embed.norm", 1.0), put("final.norm", 1.0), put("norm1", 1.0), put("norm2", 1.0),
               put("dq.norm", 1.0), put("dkv.norm", 1.0)]
    for i, change in enumerate(changes):
        d, ww = copy.deepcopy(c), dict(w)
        change(d, ww)
        assert rel_err(have, ps.forward(d, ww, toks).numpy()) > 1e-3, f"change {i} does not show"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_then_token_by_token(name, dtype):
    reqs = requests(name)
    got = run_trace(engine(name, dtype), trace_tail(reqs, tail=140))     # over page, chunk and window borders
    check(name, dtype, got, reqs, [f"r{i}" for i in range(len(reqs))])


def trace_portions(reqs, sizes):
    """Each request alone, cut into portions whose sizes cycle through ``sizes``."""
    steps, k = [], 0
    for i, toks in enumerate(reqs):
        for (at, n) in cuts(len(toks), sizes[i % len(sizes):] + sizes[:i % len(sizes)]):
            steps.append({"step": k, "entries": [{"id": f"r{i}", "tokens": toks[at:at + n], "want": list(range(n))}],
                          "end": [f"r{i}"] if at + n == len(toks) else []})
            k += 1
    return steps


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions(name, dtype):
    """Portions of two tokens, of a page, over a chunk and over a window: keys, values and states pass from
    one portion to the next, in every pass over a layer of its own."""
    reqs = requests(name)
    for sizes in ([2], [64, 3, 61, 2, 130], [7, 1, 128]):
        sel = reqs if sizes != [2] else reqs[:4]
        got = run_trace(engine(name, dtype), trace_portions(sel, sizes))
        check(name, dtype, got, sel, [f"r{i}" for i in range(len(sel))])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_batches_of_unequal_requests(name, dtype):
    reqs = requests(name)
    # two batches one after the other in a cache that holds little more than one of them: slots (the
    # states) and pages are used again by other sequences
    b0 = [(reqs[5], len(reqs[5]) - 20), (reqs[0], 1), (reqs[3], len(reqs[3]) - 33), (reqs[2], 2)]
    b1 = [(reqs[4], len(reqs[4]) - 9), (reqs[1], 1), (reqs[3], 40)]
    for b in (b0, b1):
        for i, (t, p) in enumerate(b):
            b[i] = (t, max(1, min(p, len(t))))
    need = max(sum((len(t) + 63) // 64 * 64 for t, _ in b) for b in (b0, b1))
    e = engine(name, dtype, max_tokens=need)
    got = run_trace(e, trace_batches([b0, b1, b0]))
    for b, batch in enumerate([b0, b1, b0]):
        check(name, dtype, got, [t for t, _ in batch], [f"b{b}r{i}" for i in range(len(batch))])
    e.cache.check()
    # in 32-bit a request's logits are the same bits whatever runs beside it
    if dtype == "float32":
        alone = run_trace(e, trace_tail([b0[0][0]], tail=20))
        for p in range(len(b0[0][0])):
            assert np.array_equal(alone["r0"][p], got["b0r0"][p])


def test_every_pass_has_places_of_its_own():
    """The cache manager's view of a model whose layers run several times: a state per pass over a
    retention layer, a group per kind of attention with an entry per pass, windows that give pages back."""
    e = engine("SA", "bfloat16")
    d = e.cache._op("describe")
    m = [l["mixer"] for l in CONFIGS["SA"]["layers"]]
    assert d["state_bytes"] == [4 * m[2]["heads"] * m[2]["dim"] * m[2]["vdim"]] * 3
    groups = {(g["head_dim"], g["window"], g["values_in_keys"]): len(g["entries"]) for g in d["groups"]}
    assert groups == {(m[0]["kv_rank"] + m[0]["rot_dim"], 37, True): 1, (m[1]["dim"], 64, False): 3}


@pytest.mark.parametrize("name", ["SC", "SF"])
def test_prompts_per_head_against_prompts_on_the_latents(name):
    """In bfloat16 whole prompts may form keys and values per head (at their own size, or padded to the
    kernel's); on the latents, as every other step, the same prompts give the same logits."""
    from janas_b200.config import config_from_dict
    from janas_b200.engine import Engine
    _, c, w = model(name)
    e = engine(name, "bfloat16")
    d = config_from_dict(c).to_model_spec().to_json()
    n = 0
    for l in d["layers"]:
        if l["mixer"]["kind"] == "latent_attention":
            l["mixer"]["params"]["per_head_prompts"] = False
            n += 1
    assert n == {"SC": 2, "SF": 3}[name]
    from janas_b200.config import ModelSpec
    other = Engine.from_spec(ModelSpec.from_json(d), {k: v.to(torch.bfloat16).to(DEV) for k, v in w.items()}, dtype="bfloat16",
                             max_tokens=2048)
    reqs = requests(name)
    a, b = run_trace(e, trace_whole(reqs)), run_trace(other, trace_whole(reqs))
    for i, toks in enumerate(reqs):
        x, y = (np.stack([g[f"r{i}"][p] for p in range(len(toks))]) for g in (a, b))
        err = np.abs(x - y).max(1) / np.abs(y).max()
        assert np.median(err) <= 1.5e-2 and np.mean(err > BF16_TOL) <= 0.1, (i, err.max())
    check(name, "bfloat16", b, reqs, [f"r{i}" for i in range(len(reqs))])
    other.close()


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", ["SA", "SD"])
def test_greedy_generation_through_the_entry_point(name):
    import janas_b200
    folder, c, w = model(name)
    llm = janas_b200.open(folder, janas_b200.LLMParams(n_ctx=512, dtype="float32", max_batch=4, max_tokens=1024))
    prompts = [requests(name)[2], requests(name)[1], requests(name)[3][:50]]
    outs, _ = llm.generate_batch(prompts, [12, 5, 9])
    for p, o, n in zip(prompts, outs, [12, 5, 9]):
        seq = list(p)
        for _ in range(n):
            lg = ps.forward(c, w, seq)[-1]
            top = torch.topk(lg, 2).values
            nxt = int(lg.argmax())
            if (top[0] - top[1]) < 1e-4 * lg.abs().max():
                break                                   # a tie within rounding: stop comparing
            assert o[len(seq) - len(p)] == nxt
            seq.append(nxt)
    llm.close()


def test_long_decoding_with_captured_steps():
    """bfloat16 decode steps are captured and replayed: 300 tokens after a short prompt, against the
    plain model on the whole sequence."""
    name = "SC"
    rng = np.random.default_rng(78)
    toks = rng.integers(0, CONFIGS[name]["vocab"], size=340).tolist()
    got = run_trace(engine(name, "bfloat16"), trace_tail([toks], tail=300))
    check(name, "bfloat16", got, [toks], ["r0"])
