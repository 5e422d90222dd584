"""Migosun on the GPU: every mechanism alone and whole models against the plain oracle, in fp32 (sharp), bf16 and fp16."""
import json
import os
import subprocess

import pytest
import torch

import migosun_util as mu
from oracle import migosun_oracle as mo

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16, torch.float16]
EPS = {torch.float32: 2e-6, torch.bfloat16: 4e-3, torch.float16: 6e-4}  # relative error of one rounded result


def _ops():
    from gpt_fast.ops import CudaOps
    return CudaOps


@pytest.fixture(autouse=True)
def _check_waits_and_options():
    from gpt_fast import _C
    yield
    for name, value in ((b"window_tc", 1), (b"scan_columns", 0), (b"scan_warps", 0), (b"scan_lanes", 0)):
        _C.check(_C.lib.lri_set_option(name, value))
    torch.cuda.synchronize()
    _C.check(_C.lib.lri_gemm_status())


def _randn(g, *shape, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _rel(got, ref):
    got, ref = got.double().cpu(), ref.double().cpu()
    assert torch.isfinite(got).all()
    return ((got - ref).norm() / ref.norm()).item()


# ---- mechanisms alone ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,streams,dim", [(1, 1, 64), (3, 3, 101), (2, 4, 4096), (40, 2, 1032), (20, 6, 2048), (5, 8, 9000), (7, 11, 260),
                                              (300, 4, 1600)])
def test_streams(dtype, rows, streams, dim):
    """A join's new streams come from the old ones all at once; the next sublayer's input and the plain sum at the end."""
    g = torch.Generator().manual_seed(rows + dim)
    ops, eps, vocab = _ops(), 1e-3, 37
    x, y = _randn(g, rows, streams, dim), _randn(g, rows, dim, dtype=dtype)
    mix, out, w_in, norm = _randn(g, streams, streams, dtype=dtype), *(_randn(g, n, dtype=dtype) for n in (streams, streams, dim))
    want = torch.einsum("st,rsd->rtd", mix.double(), x.double()) + out.double()[None, :, None] * y.double()[:, None]
    for nxt in (w_in, None):
        u = torch.einsum("t,rtd->rd", w_in.double(), want) if nxt is not None else want.sum(1)
        got, normed = x.clone().cuda(), torch.empty(rows, dim, dtype=dtype, device="cuda")
        ops.join_streams(got, y.cuda(), mix.cuda(), out.cuda(), nxt.cuda() if nxt is not None else None, norm.cuda(), eps, normed, rows,
                         write=nxt is not None)
        assert _rel(got, want if nxt is not None else x) < 2e-6
        assert _rel(normed, mo.rms_norm(u, norm.double(), eps)) < EPS[dtype]
    table, idx = _randn(g, vocab, dim, dtype=dtype), torch.randint(0, vocab, (rows,), generator=g)
    for ids in (idx, idx.int()):
        got = torch.empty(rows, streams, dim, device="cuda")
        ops.embed_streams(table.cuda(), ids.cuda(), 0.3, got, w_in.cuda(), norm.cuda(), eps, normed)
        e = table.double()[idx] * 0.3
        assert _rel(got, e[:, None].expand(-1, streams, -1)) < 1e-6
        assert _rel(normed, mo.rms_norm(e * w_in.double().sum(), norm.double(), eps)) < EPS[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,I,K", [(1, 40, 64), (1, 33, 36), (5, 72, 256), (8, 51, 640), (16, 64, 128), (40, 136, 192), (64, 33, 72), (65, 72, 64),
                                   (130, 264, 320), (200, 37, 96), (90, 24, 20)])
def test_gateup_with_the_clamped_unit(dtype, M, I, K):
    """Inputs on both sides of the limit, gates far below zero (which is not clamped)."""
    g = torch.Generator().manual_seed(M + I)
    ops, glu = _ops(), (1.702, 0.9, 1.0)
    x, w1 = _randn(g, M, K, dtype=dtype), _randn(g, 2 * I, K, dtype=dtype, scale=1.5 * K ** -0.5)
    nb = ops.gateup_glu_workspace_bytes(dtype, M, I, K)
    ws = torch.empty(nb, dtype=torch.uint8, device="cuda") if nb else None
    h = torch.full((M, I), float("nan"), dtype=dtype, device="cuda")
    ops.gateup_glu(x.cuda(), w1.cuda(), h, M, glu, workspace=ws)
    u = x.double() @ w1.double().T
    assert _rel(h, mo.clamped_glu(u[:, I:], u[:, :I], glu[1])) < EPS[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("given_sums", [False, True])
@pytest.mark.parametrize("B,S,H,G,d,dv,rot,pos0", [(1, 5, 3, 1, 20, 12, 6, 0), (2, 7, 4, 2, 32, 40, 32, 11), (1, 300, 8, 8, 64, 16, 16, 900), (3, 1, 16, 2, 8, 8, 2, 5),
                                                   (1, 1, 32, 8, 128, 128, 64, 70), (1, 90, 6, 3, 48, 24, 20, 3), (2, 3, 5, 5, 9, 7, 0, 4)])
def test_norm_over_all_heads_rotation_and_cache(dtype, given_sums, B, S, H, G, d, dv, rot, pos0):
    """One norm over the whole projection (heads of very different size), partial rotation at far positions, cache rows."""
    from gpt_fast.mixers import rotate_half_table
    g = torch.Generator().manual_seed(S + d)
    ops, smax, base, eps = _ops(), pos0 + S + 3, 300.0, 1e-4
    q_off, k_off, v_off = 8, 8 + H * d, 8 + (H + G) * d
    ld = v_off + G * dv + (-(v_off + G * dv)) % 8
    proj = _randn(g, B * S, ld)
    proj[:, q_off:q_off + d] *= 30.0  # the first head decides the norm of the others
    qn, kn = _randn(g, H * d, dtype=dtype), _randn(g, G * d, dtype=dtype)
    kc, vc = (torch.zeros(B, G, smax, n, dtype=dtype, device="cuda") for n in (d, dv))
    q = torch.full((B * S, H, d), float("nan"), dtype=dtype, device="cuda")
    pos = torch.arange(pos0, pos0 + S)
    x = proj.double()
    sums, widths = None, (H * d, G * d)
    if given_sums:  # as if other ranks held as many heads again
        sums, widths = torch.empty(B * S, 2, device="cuda"), (2 * H * d, 2 * G * d)
        ops.row_squares(proj.cuda(), ld, q_off, H * d, k_off, G * d, sums, B * S)
        own = torch.stack([(x[:, q_off:k_off] ** 2).sum(-1), (x[:, k_off:v_off] ** 2).sum(-1)], -1)
        assert _rel(sums, own) < 1e-6
    ops.grouped_prepare(proj.cuda(), ld, (q_off, k_off, v_off), qn.cuda(), kn.cuda(), sums, widths, eps,
                        rotate_half_table(smax, max(rot, 2), base, "cpu").cuda(), rot, pos.cuda(), q, kc, vc, B, S, H)

    def normed(v, w, width):
        return v / torch.sqrt((v * v).sum(-1, keepdim=True) / width + eps) * w.double()

    for b in range(B):
        r = x[b * S:(b + 1) * S]
        for got, off, heads, w, width in ((q.view(B, S, H, d)[b], q_off, H, qn, widths[0]),
                                          (kc[b, :, pos0:pos0 + S].transpose(0, 1), k_off, G, kn, widths[1])):
            want = normed(r[:, off:off + heads * d], w, width).view(S, heads, d)
            want = mo.rotate_first_dims(want, pos, rot, base) if rot else want
            assert _rel(got, want) < EPS[dtype]
        assert _rel(vc[b, :, pos0:pos0 + S].transpose(0, 1), r[:, v_off:v_off + G * dv].view(S, G, dv)) < EPS[dtype]
    assert kc[:, :, :pos0].abs().sum() == 0 and kc[:, :, pos0 + S:].abs().sum() == 0


def _attention_ref(q, k, v, sink, qpos, window, chunk, scale):
    """q [S, H, d] at positions qpos, k and v [n, G, ..] at positions 0 .. n - 1"""
    H, G = q.shape[1], k.shape[1]
    group = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, group]) * scale
    dist = qpos[:, None] - torch.arange(k.shape[0])[None, :]
    ok = dist >= 0
    if window:
        ok &= dist < window
    if chunk:
        ok &= (qpos // chunk)[:, None] == (torch.arange(k.shape[0]) // chunk)[None, :]
    s = s.masked_fill(~ok, float("-inf"))
    p = mo.softmax_with_sink(s, sink) if sink is not None else torch.softmax(s, -1)
    return torch.einsum("hij,jhd->ihd", p, v[:, group])


def _plant(q, k, i, j, h, strength):
    """Makes key row j stand out for query i of head h: it is aligned with the query."""
    u = q[i, h].float()
    k[j, h // (q.shape[1] // k.shape[1])] = (u * strength / u.norm()).to(k.dtype)


@pytest.mark.parametrize("plain", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,H,G,d,dv,pos0,window,chunk,sink", [
    (300, 4, 2, 40, 48, 0, 0, 75, True), (130, 6, 1, 128, 128, 200, 0, 64, True), (257, 2, 2, 64, 64, 63, 0, 65, False), (200, 3, 3, 72, 24, 13, 0, 1000, True),
    (33, 2, 1, 8, 8, 0, 0, 1, True), (150, 4, 4, 96, 64, 90, 31, 0, True), (400, 2, 1, 64, 120, 7, 50, 96, False), (520, 2, 2, 32, 32, 0, 0, 0, True),
    (150, 2, 1, 20, 12, 40, 0, 31, True), (2, 4, 2, 32, 16, 95, 0, 96, True), (17, 8, 2, 104, 88, 5, 0, 7, True), (140, 2, 1, 160, 136, 60, 0, 50, True)])
def test_grouped_attention_prompt(plain, dtype, S, H, G, d, dv, pos0, window, chunk, sink):
    """Portions that start inside a chunk: the chunk's first position seen, the one before it not (planted keys on both
    sides), sinks that take most of the weight, caches with rows behind the newest one."""
    from gpt_fast import _C
    if plain and dtype == torch.float32:
        pytest.skip("fp32 always runs the plain kernel")
    _C.lib.lri_set_option(b"window_tc", 0 if plain else 1)
    g = torch.Generator().manual_seed(S + chunk + window)
    B, n, scale, factor = 2, pos0 + S, 1.3 * d ** -0.5, 0.8
    q, k, v = _randn(g, B, S, H, d, dtype=dtype), _randn(g, B, n, G, d, dtype=dtype), _randn(g, B, n, G, dv, dtype=dtype)
    for x, i in enumerate(range(0, S, 13)):
        p, h = pos0 + i, x % H
        first = max(0, p - window + 1 if window else 0, p // chunk * chunk if chunk else 0)
        j = first if x % 2 == 0 or first == 0 else first - 1
        _plant(q[1], k[1], i, j, h, 12.0)
    sk = (_randn(g, H) * 2 + 1).to(dtype) if sink else None
    smax, off, ld = n + 9, 16, 16 + H * dv + (8 if dv % 8 == 0 else 3)
    kc, vc = (torch.randn(B, G, smax, x, generator=g).to(dtype) for x in (d, dv))
    kc[:, :, :n], vc[:, :, :n] = k.transpose(1, 2), v.transpose(1, 2)
    out = torch.full((B * S, ld), float("nan"), dtype=dtype, device="cuda")
    pos = torch.arange(pos0, pos0 + S)
    _ops().grouped_attention(q.cuda(), kc.cuda(), vc.cuda(), sk.cuda() if sink else None, out.view(-1)[off:], ld, factor, pos.int().cuda(), window,
                             chunk, scale, B, S, H)
    assert torch.isnan(out[:, :off].float()).all() and torch.isnan(out[:, off + H * dv:].float()).all()
    for b in range(B):
        want = _attention_ref(q[b].double(), k[b].double(), v[b].double(), sk.double() if sink else None, pos, window, chunk, scale) * factor
        got = out.view(B, S, ld)[b, :, off:off + H * dv].reshape(S, H, dv)
        assert _rel(got, want) < EPS[dtype]
        worst = (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)
        assert worst.max() < 12 * EPS[dtype]


@pytest.mark.parametrize("plain", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,H,G,d,dv,smax,window,chunk,positions", [
    (1, 8, 2, 96, 64, 700, 0, 77, [0, 1, 63, 76, 77, 78, 153, 154, 155, 699]), (3, 4, 4, 64, 128, 200, 0, 64, [5, 63, 64, 65, 199]),
    (2, 6, 1, 40, 24, 500, 129, 0, [128, 129, 300]), (1, 2, 1, 20, 12, 90, 0, 17, [16, 17, 18, 80]), (2, 16, 2, 128, 128, 300, 0, 4096, [299]),
    (1, 3, 3, 16, 16, 70, 0, 1, [0, 1, 64, 69]), (1, 12, 1, 56, 8, 400, 100, 150, [99, 100, 149, 150, 310]), (40, 8, 8, 64, 64, 64, 0, 0, [63])])
def test_grouped_attention_single_token(plain, dtype, B, H, G, d, dv, smax, window, chunk, positions):
    from gpt_fast import _C
    if plain and dtype == torch.float32:
        pytest.skip("fp32 always runs the plain kernel")
    _C.lib.lri_set_option(b"window_tc", 0 if plain else 1)
    scale = d ** -0.5
    for pos in positions:
        g = torch.Generator().manual_seed(pos)
        q, kc, vc = _randn(g, B, H, d, dtype=dtype), _randn(g, B, G, smax, d, dtype=dtype), _randn(g, B, G, smax, dv, dtype=dtype)
        first = max(0, pos - window + 1 if window else 0, pos // chunk * chunk if chunk else 0)
        for b in range(B):  # a row just inside or just outside
            j = first if (pos + b) % 2 or first == 0 else first - 1
            u = q[b, H - 1].float()
            kc[b, G - 1, j] = (u * 12.0 / u.norm()).to(dtype)
        sink = (_randn(g, H) + 1).to(dtype)
        out = torch.full((B, H * dv + 8), float("nan"), dtype=dtype, device="cuda")
        _ops().grouped_attention(q.cuda(), kc.cuda(), vc.cuda(), sink.cuda(), out, H * dv + 8, 1.5, torch.tensor([pos]).cuda(), window, chunk, scale,
                                 B, 1, H)
        for b in range(B):
            want = 1.5 * _attention_ref(q[b].double()[None], kc[b].double().transpose(0, 1), vc[b].double().transpose(0, 1), sink.double(),
                                        torch.tensor([pos]), window, chunk, scale)
            assert _rel(out[b, : H * dv].view(1, H, dv), want) < EPS[dtype], (pos, b)


class _Delta:
    """Random inputs of the gated delta rule on a projection buffer, its parameters, and the oracle on them."""

    def __init__(self, dtype, B, n, H, G, C, E, taps, ra, rg, bias, seed=0):
        g = torch.Generator().manual_seed(seed + n + C)
        self.dtype, self.B, self.n, self.H, self.G, self.C, self.E, self.taps, self.eps = dtype, B, n, H, G, C, E, taps, 1e-4
        pad = [-r % 8 for r in (ra, rg)]
        widths = dict(q=G * C, k=G * C, v=H * E, a1=ra + pad[0], g1=rg + pad[1], b=H)
        self.offs, at = {}, 8
        for k, w in widths.items():
            self.offs[k], at = at, at + w
        self.ld = at + -at % 8
        self.proj = _randn(g, B, n, self.ld)
        self.convs = [_randn(g, w, taps, dtype=dtype) for w in (G * C, G * C, H * E)]
        self.a2 = torch.cat([_randn(g, H * C, ra, dtype=dtype, scale=ra ** -0.5), torch.zeros(H * C, pad[0], dtype=dtype)], 1)
        self.g2 = torch.cat([_randn(g, H * E, rg, dtype=dtype, scale=rg ** -0.5), torch.zeros(H * E, pad[1], dtype=dtype)], 1)
        self.a_log, self.dt_bias, self.norm = (_randn(g, H) - 1).to(dtype), (_randn(g, H * C) + bias).to(dtype), _randn(g, E, dtype=dtype)
        self.ring = torch.zeros(B, taps, 2 * G * C + H * E, device="cuda")
        self.state = torch.full((B, H, C, E), 7.0, device="cuda")  # a call at position 0 must not see it

    def low(self, name):
        x = self.proj[..., self.offs[name]:self.offs[name] + (self.a2 if name == "a1" else self.g2).shape[1]]
        return x.to(self.dtype).double()

    def oracle(self, b):
        p, o, H, G, C, E = self.proj[b].double(), self.offs, self.H, self.G, self.C, self.E
        q, k, v = (mo.silu(mo.short_conv(p[:, o[t]:o[t] + w.shape[0]], w.double())) for t, w in zip("qkv", self.convs))
        group = torch.arange(H) // (H // G)
        q = (mo.unit(q.view(-1, G, C)) * C ** -0.5)[:, group]
        k = mo.unit(k.view(-1, G, C))[:, group]
        z = (self.low("a1")[b] @ self.a2.double().T).view(-1, H, C)
        dec = mo.delta_decay(z, self.a_log.double(), self.dt_bias.double())
        out, st = mo.delta_recurrence(q, k, v.view(-1, H, E), dec, torch.sigmoid(p[:, o["b"]:o["b"] + H]))
        gate = torch.sigmoid(self.low("g1")[b] @ self.g2.double().T).view(-1, H, E)
        return out, st, mo.rms_norm(out, self.norm.double(), self.eps) * gate

    def blocks(self, s0, S):
        """Rows s0 .. s0 + S - 1 through the block form; raw results [B, S, H, E]."""
        ops, B, H, C, E = _ops(), self.B, self.H, self.C, self.E
        z = (self.low("a1")[:, s0:s0 + S] @ self.a2.double().T).float().reshape(B * S, H * C).contiguous().cuda()
        nb = B * ops.state_blocks(S)
        blocks = [torch.full((r, w), float("nan"), device="cuda") for r, w in ((4 * nb, H * C), (4 * nb, H * C), (4 * nb, H * C), (nb, H * C), (nb, H * 32))]
        v, o = torch.full((B * S, H * E), float("nan"), device="cuda"), torch.full((B * S, H, E), float("nan"), device="cuda")
        pos = torch.arange(s0, s0 + S).cuda()
        proj = self.proj[:, s0:s0 + S].reshape(B * S, self.ld).contiguous().cuda()
        ops.delta_blocks(proj, self.ld, [self.offs[k] for k in "qkvb"], [c.cuda() for c in self.convs], self.ring, z, self.a_log.cuda(),
                         self.dt_bias.cuda(), pos, blocks, v, B, S, H, self.G, C, E)
        ops.state_scan(blocks, True, v, H * E, self.state, pos, o, B, S)
        return o.view(B, S, H, E).double().cpu()

    def step(self, s):
        """Token s through the one-kernel form: normed and gated results times 0.7."""
        B, H, E = self.B, self.H, self.E
        ld = H * E + 24
        out = torch.full((B, ld), float("nan"), dtype=self.dtype, device="cuda")
        _ops().delta_step(self.proj[:, s].contiguous().cuda(), self.ld, [self.offs[k] for k in ("q", "k", "v", "a1", "g1", "b")],
                          [c.cuda() for c in self.convs], self.ring, self.a2.cuda(), self.g2.cuda(), self.a_log.cuda(), self.dt_bias.cuda(),
                          self.norm.cuda(), self.eps, 0.7, self.state, torch.tensor([s]).cuda(), out.view(-1)[8:], ld, B, self.G)
        assert torch.isnan(out[:, :8].float()).all() and torch.isnan(out[:, 8 + H * E:].float()).all()
        return out[:, 8:8 + H * E].double().cpu().view(B, H, E) / 0.7


DELTA_SIZES = [(1, 41, 2, 1, 12, 20, 4, 5, 9, -1.0), (2, 60, 4, 2, 64, 64, 3, 16, 8, -3.0), (1, 75, 2, 2, 128, 96, 4, 24, 16, 0.0), (1, 33, 3, 3, 48, 128, 1, 8, 8, 3.0),
               (2, 37, 2, 1, 9, 7, 2, 1, 1, -1.0), (1, 30, 1, 1, 200, 40, 7, 8, 70, -2.0), (1, 24, 1, 1, 32, 32, 4, 8, 8, 60.0),
               (1, 14, 2, 1, 256, 250, 4, 8, 8, -1.0), (30, 9, 4, 2, 52, 72, 3, 16, 8, -1.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", DELTA_SIZES + [(1, 26, 1, 1, 300, 24, 4, 8, 8, -1.0)], ids=str)
def test_gated_delta_in_portions(dtype, size):
    """The block form over portions of any cut (convolution inputs and state carried over), decays near 1 (bias -3) and
    vanishing (bias 60), against the recurrence token by token."""
    B, n = size[:2]
    for cuts in ([n], [1, 2, 3, 4, 5], [2], [7, 1, 16, 1]):
        c = _Delta(dtype, *size)
        got, at, i = [], 0, 0
        while at < n:
            k = min(cuts[min(i, len(cuts) - 1)], n - at)
            got.append(c.blocks(at, k))
            at, i = at + k, i + 1
        got = torch.cat(got, 1)
        for b in range(B):
            out, st, _ = c.oracle(b)
            assert _rel(got[b], out) < 3e-6 and _rel(c.state[b], st) < 3e-6, cuts


@pytest.mark.parametrize("columns,warps,lanes", [(1, 1, 8), (2, 2, 8), (4, 4, 8), (4, 1, 16), (1, 4, 16), (2, 1, 16)])
def test_state_scan_launch_shapes(columns, warps, lanes):
    from gpt_fast import _C
    for name, value in ((b"scan_columns", columns), (b"scan_warps", warps), (b"scan_lanes", lanes)):
        _C.check(_C.lib.lri_set_option(name, value))
    for size in (DELTA_SIZES[1], DELTA_SIZES[2], DELTA_SIZES[4]):
        c = _Delta(torch.float32, *size)
        got = c.blocks(0, size[1])
        for b in range(size[0]):
            assert _rel(got[b], c.oracle(b)[0]) < 3e-6 and _rel(c.state[b], c.oracle(b)[1]) < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", DELTA_SIZES, ids=str)
def test_gated_delta_steps(dtype, size):
    """The one-kernel step from position 0 on, and behind a portion through the block form."""
    B, n = size[:2]
    for start in (0, 6):
        c = _Delta(dtype, *size)
        if start:
            c.blocks(0, start)
        got = torch.stack([c.step(s) for s in range(start, n)], 1)
        for b in range(B):
            _, st, gated = c.oracle(b)
            assert _rel(got[b], gated[start:]) < max(EPS[dtype], 5e-6) and _rel(c.state[b], st) < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,n,H,C,E,rank,tau,bias", [(1, 41, 2, 12, 20, 5, 7.0, 0.0), (2, 50, 3, 64, 128, 16, 16.0, 2.0), (1, 66, 2, 128, 200, 24, 1.0, -8.0),
                                                     (1, 30, 1, 9, 7, 1, 4.0, 0.0), (1, 23, 1, 256, 256, 8, 16.0, 5.0), (1, 21, 2, 400, 300, 8, 2.0, 0.0)])
def test_gated_linear_attention(dtype, B, n, H, C, E, rank, tau, bias):
    """Block form in portions and the one-kernel step, with decays near 0 and near 1."""
    g, ops, eps = torch.Generator().manual_seed(n + C), _ops(), 1e-4
    pad = -rank % 8
    offs, at = {}, 8
    for k, w in dict(q=H * C, k=H * C, v=H * E, g=H * E, a1=rank + pad).items():
        offs[k], at = at, at + w
    ld = at + -at % 8
    proj = _randn(g, B, n, ld)
    a2 = torch.cat([_randn(g, H * C, rank, dtype=dtype, scale=rank ** -0.5), torch.zeros(H * C, pad, dtype=dtype)], 1)
    a2_bias, norm = (_randn(g, H * C) + bias).to(dtype), _randn(g, E, dtype=dtype)
    zs = (proj[..., offs["a1"]:offs["a1"] + rank + pad].to(dtype).double() @ a2.double().T).float()
    ref = []
    for b in range(B):
        p = proj[b].double()
        q, k, v = (p[:, offs[t]:offs[t] + H * w].view(n, H, w) for t, w in (("q", C), ("k", C), ("v", E)))
        dec = torch.exp(torch.nn.functional.logsigmoid(zs[b].double() + a2_bias.double()) / tau).view(n, H, C)
        out, st = mo.linear_attention_recurrence(q * C ** -0.5, k, v, dec)
        gated = mo.rms_norm(out, norm.double(), eps) * mo.silu(p[:, offs["g"]:offs["g"] + H * E]).view(n, H, E)
        ref.append((out, st, gated))

    def portion(state, s0, S):
        nb = B * ops.state_blocks(S)
        blocks = [torch.full((r, w), float("nan"), device="cuda") for r, w in ((4 * nb, H * C), (1, 1), (4 * nb, H * C), (nb, H * C), (nb, H * 32))]
        x = proj[:, s0:s0 + S].reshape(B * S, ld).contiguous().cuda()
        o, pos = torch.full((B * S, H, E), float("nan"), device="cuda"), torch.arange(s0, s0 + S).cuda()
        ops.gla_blocks(x, ld, (offs["q"], offs["k"]), zs[:, s0:s0 + S].reshape(B * S, -1).contiguous().cuda(), a2_bias.cuda(), tau, blocks, B, S, H, C)
        ops.state_scan(blocks, False, x.view(-1)[offs["v"]:], ld, state, pos, o, B, S)
        gated = torch.full((B * S, H * E), float("nan"), dtype=dtype, device="cuda")
        ops.head_norm_gate(o, norm.cuda(), eps, x.view(-1)[offs["g"]:], ld, "silu", 0.5, gated, H * E, B * S, H)
        return o.view(B, S, H, E).double().cpu(), gated.view(B, S, H, E).double().cpu() / 0.5

    for cuts in ([n], [1, 2, 3, 4, 5], [9, 2]):
        state = torch.full((B, H, C, E), 7.0, device="cuda")
        got, at, i = [], 0, 0
        while at < n:
            k = min(cuts[min(i, len(cuts) - 1)], n - at)
            got.append(portion(state, at, k))
            at, i = at + k, i + 1
        for b in range(B):
            assert _rel(torch.cat([x for x, _ in got], 1)[b], ref[b][0]) < 3e-6 and _rel(state[b], ref[b][1]) < 3e-6, cuts
            assert _rel(torch.cat([x for _, x in got], 1)[b], ref[b][2]) < max(EPS[dtype], 5e-6)
    if not ops.state_step_supports(C, E, rank + pad, 0):
        assert C > 256 or E > 256
        return
    state, out = torch.full((B, H, C, E), 7.0, device="cuda"), []
    for s in range(n):
        y = torch.full((B, H * E), float("nan"), dtype=dtype, device="cuda")
        ops.gla_step(proj[:, s].contiguous().cuda(), ld, [offs[k] for k in ("q", "k", "v", "a1", "g")], a2.cuda(), a2_bias.cuda(), tau, norm.cuda(), eps,
                     0.5, state, torch.tensor([s]).cuda(), y, H * E, B)
        out.append(y.double().cpu().view(B, H, E) / 0.5)
    for b in range(B):
        assert _rel(torch.stack(out, 1)[b], ref[b][2]) < max(EPS[dtype], 5e-6) and _rel(state[b], ref[b][1]) < 3e-6


# ---- whole models ------------------------------------------------------------------------------------------------
LIMIT = {torch.float32: (2e-5, 2e-4), torch.bfloat16: (2e-2, 6e-2), torch.float16: (4e-3, 2e-2)}  # median and largest error


def _close(got, ref, dtype, what=""):
    e = mu.row_err(got, ref).flatten()
    assert torch.isfinite(e).all() and e.median() < LIMIT[dtype][0] and e.max() < LIMIT[dtype][1], (what, e.median(), e.max())


_CACHE = {}


def _case(name, n=150, seed=1):
    if (name, n, seed) not in _CACHE:
        cfg, _ = mu.CONFIGS[name]
        w, toks = mu.weights(mu.CONFIGS[name], 8), None
        toks = mu.tokens(cfg, n, seed)
        _CACHE[name, n, seed] = (cfg, w, toks, mu.reference(cfg, w, toks))
    return _CACHE[name, n, seed]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(mu.CONFIGS))
@pytest.mark.parametrize("cuts", [[150], [1], [2], [100, 1], [3, 2, 64, 16, 17, 1], [65, 7]], ids=str)
def test_model_prompts_portions_and_single_tokens(name, dtype, cuts):
    cfg, w, toks, ref = _case(name)
    model = mu.build(cfg, w, dtype, "cuda", 1, 152)
    _close(mu.feed(model, toks[None], cuts)[0], ref, dtype, cuts)


@pytest.mark.parametrize("name", ["uneven", "tiles"])
def test_logits_do_not_depend_on_the_cuts(name):
    """fp32: the same position, however its tokens were fed, up to rounding (far below the distance to the oracle's limits)."""
    cfg, w, toks, _ = _case(name)
    model = mu.build(cfg, w, torch.float32, "cuda", 1, 152)
    whole = mu.feed(model, toks[None], [150])
    for cuts in ([1], [2], [49, 1, 2], [51, 3]):
        e = mu.row_err(mu.feed(model, toks[None], cuts), whole)
        assert e.median() < 5e-6 and e.max() < 2e-4, (cuts, e.max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["uneven", "tiles"])
def test_batches_and_reused_rows(name, dtype):
    """Rows of a batch do not see one another; a row that served a longer sequence serves another from position 0, with
    the old keys, states and convolution inputs still in memory."""
    cfg, w, toks, ref = _case(name)
    model = mu.build(cfg, w, dtype, "cuda", 3, 152)
    rows = torch.stack([toks[:90], mu.tokens(cfg, 90, 11), mu.tokens(cfg, 90, 12)])
    refs = torch.stack([mu.reference(cfg, w, r) for r in rows])
    _close(mu.feed(model, rows, [80, 1]), refs, dtype)
    other = mu.tokens(cfg, 60, 13)
    want = mu.reference(cfg, w, other)
    _close(mu.feed(model, other[None], [20, 1, 30])[0], want, dtype, "reused")
    _close(mu.feed(model, other[None, :5], [1])[0], want[:5], dtype, "first tokens, reused, one by one")
    _close(mu.feed(model, rows[:2], [33, 1, 40]), refs[:2], dtype, "two rows of three")
    if dtype == torch.float32:
        alone = mu.build(cfg, w, dtype, "cuda", 1, 152)
        assert mu.row_err(mu.feed(alone, rows[1:2], [80, 1]), mu.feed(model, rows, [80, 1])[1:2]).max() < 2e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_chunk_edge_reaches_the_logits(dtype):
    """Attention alone (the recurrence's output projection zero): the first token of the query's chunk changes its logits,
    the last token of the chunk before does not; in a prompt, decoded, and in a portion that begins at the edge."""
    chunk = 40
    case = mu.config(128, 90, 2, [(mu.side_by_side((4, 2, 32, 32, chunk, 16, 1e4, 0.3), (2, 2, 16, 16, 3, (8, 8))), None)])
    cfg, w = case[0], mu.weights(case, 5)
    w["l0.mix.right.o"].zero_()
    n, qpos = 130, 100
    for cuts in ([n], [qpos, 1], [80, 50], [79, 2, 49]):
        for j, seen in ((80, True), (79, False), (qpos - 1, True)):
            base = mu.tokens(cfg, n, 21)
            moved = base.clone()
            moved[j] = (moved[j] + 37) % 90
            model = mu.build(cfg, w, dtype, "cuda", 1, n)
            a, b = (mu.feed(model, t[None], cuts)[0, qpos] for t in (base, moved))
            if seen:
                assert (a - b).abs().max() > 1e-2, (cuts, j)
            else:
                assert torch.equal(a, b), (cuts, j)
            assert mu.row_err(b[None], mu.reference(cfg, w, moved)[qpos][None]).max() < LIMIT[dtype][1]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["parallel", "gla"])
def test_a_far_token_reaches_the_logits_through_the_state(kind, dtype):
    """One layer with slow decays: a token hundreds of positions back, many chunks and portions ago, still shows."""
    layer = mu.side_by_side((2, 1, 16, 16, 8, 8, 1e4, 0.3), (2, 2, 32, 32, 3, (8, 8))) if kind == "parallel" else mu.linear(2, 32, 32, 16.0, 8)
    case = mu.config(64, 60, 2, [(layer, None)])
    cfg, w = case[0], mu.weights(case, 5)
    if kind == "parallel":
        w["l0.mix.right.dt_bias"].fill_(-9.0)
        w["l0.mix.right.b"].mul_(0.05)
    else:
        w["l0.mix.a2.b"].fill_(9.0)
    base, n = mu.tokens(cfg, 420, 3), 420
    moved = base.clone()
    moved[7] = (moved[7] + 11) % 60
    ra, rb = mu.reference(cfg, w, base), mu.reference(cfg, w, moved)
    assert (ra[-1] - rb[-1]).abs().max() > 0.02
    for cuts in ([n], [400, 1], [3, 130, 2, 64]):
        model = mu.build(cfg, w, dtype, "cuda", 1, 424)
        a, b = mu.feed(model, base[None], cuts)[0], mu.feed(model, moved[None], cuts)[0]
        _close(a, ra, dtype, cuts)
        _close(b, rb, dtype, cuts)
        if dtype == torch.float32:
            assert _rel((a - b)[-1], (ra - rb)[-1]) < 1e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_greedy_decoding_through_the_device_loop(dtype):
    """DeviceLoop (captured steps, state put back after the warm-up) against the oracle fed the same tokens: every
    chosen token is the oracle's best, or within rounding of it."""
    from gpt_fast.generate import DeviceLoop
    cfg, w, toks, _ = _case("tiles")
    model = mu.build(cfg, w, dtype, "cuda", 2, 240)
    prompt = torch.stack([toks[:30], mu.tokens(cfg, 30, 31)])
    pos = torch.arange(30, dtype=torch.int32, device="cuda")
    new = 160
    histories = []
    for head, k in (("replicated", 8), ("vocab-parallel", 5)):
        first = model.prefill_last(prompt.cuda(), pos)[:, -1].float().argmax(-1, keepdim=True)
        loop = DeviceLoop(model, 2, steps_per_replay=k, head=head)
        loop.start(first, 30)
        histories.append(torch.cat([first.int(), loop.run(new)], dim=1).cpu())
    assert torch.equal(histories[0], histories[1])
    for b in range(2):
        seq = torch.cat([prompt[b], histories[0][b].long()])
        ref = mu.reference(cfg, w, seq[:-1])[29:]
        best = ref.max(-1).values
        chosen = ref.gather(1, seq[30:, None]).squeeze(1)
        slack = (3e-4 if dtype == torch.float32 else 0.25) * ref.std(-1)
        assert (best - chosen < slack).float().mean() > (0.999 if dtype == torch.float32 else 0.95)


def test_sampling_and_last_logits():
    cfg, w, toks, ref = _case("uneven")
    model = mu.build(cfg, w, torch.bfloat16, "cuda", 1, 152)
    pos = torch.arange(60, dtype=torch.int32, device="cuda")
    last = model.prefill_last(toks[None, :60].cuda(), pos)[0, 0].float().cpu()
    full = mu.build(cfg, w, torch.bfloat16, "cuda", 1, 152)(toks[None, :60].cuda(), pos)[0, -1].float().cpu()
    assert torch.allclose(last, full, atol=3e-2 * full.abs().max())
    state = [s.clone() for s in model.recurrent_state()]
    nxt, p = toks[None, 60:61].int().cuda(), torch.tensor([60], dtype=torch.int32, device="cuda")
    greedy = model.decode_greedy(nxt, p).clone()
    for s, s0 in zip(model.recurrent_state(), state):
        s.copy_(s0)
    gen = torch.Generator(device="cuda").manual_seed(1)
    assert torch.equal(greedy, model.decode_sample(nxt, p, temperature=0.7, top_k=1, generator=gen))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_checkpoint_folder_and_trace_replay(tmp_path, dtype):
    """bin/trace_run on a checkpoint folder: two requests one after the other, portions and single tokens."""
    import numpy as np
    cfg, w, toks, ref = _case("uneven")
    mu.save(cfg, w, tmp_path / "model")
    os.makedirs(tmp_path / "out")
    other = mu.tokens(cfg, 40, 77)
    ref2 = mu.reference(cfg, w, other)
    cuts, steps, want = [50, 1, 2, 60, 1, 36], [], []
    at = 0
    for k in cuts:
        steps.append({"entries": [{"id": "a", "tokens": toks[at:at + k].tolist(), "want": list(range(k))}], "end": ["a"] if at + k == 150 else []})
        want.append(ref[at:at + k])
        at += k
    steps.append({"entries": [{"id": "b", "tokens": other[:39].tolist(), "want": []}], "end": []})
    steps.append({"entries": [{"id": "b", "tokens": other[39:].tolist(), "want": [0]}], "end": ["b"]})
    want += [None, ref2[39:]]
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", str(dtype)[6:], "--out",
                        str(tmp_path / "out"), "--max-tokens", "150"], input=text, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    for i, ref_i in enumerate(want):
        path = tmp_path / "out" / f"{i}.f32"
        assert path.exists() == (ref_i is not None)
        if ref_i is not None:
            got = torch.from_numpy(np.fromfile(path, dtype="<f4")).view(-1, cfg["vocab"])
            assert got.shape == ref_i.shape and mu.row_err(got, ref_i).max() < LIMIT[dtype][1]
