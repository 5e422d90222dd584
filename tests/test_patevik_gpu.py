"""Patevik on the GPU: every mechanism alone and whole models against the plain oracle, in fp32 (sharp), bf16 and fp16."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import patevik_util as pu
from oracle import patevik_oracle as po

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16, torch.float16]
EPS = {torch.float32: 2e-6, torch.bfloat16: 4e-3, torch.float16: 6e-4}  # relative error of one rounded result


def _ops():
    from gpt_fast.ops import CudaOps
    return CudaOps


@pytest.fixture(autouse=True)
def _restore_options():
    from gpt_fast import _C
    yield
    for name in (b"window_tc", b"hgrn2_blocks"):
        _C.lib.lri_set_option(name, 1)
    _C.lib.lri_set_option(b"moe_stream_pairs", 10)
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
@pytest.mark.parametrize("M,N,K", [(1, 72, 64), (1, 101, 36), (5, 130, 256), (8, 104, 640), (13, 96, 128), (40, 264, 192), (64, 66, 72),
                                   (65, 136, 64), (200, 101, 96), (300, 520, 320), (130, 24, 20)])
def test_linear_f32(dtype, M, N, K):
    g = torch.Generator().manual_seed(M + N)
    x, w = _randn(g, M, K, dtype=dtype), _randn(g, N, K, dtype=dtype, scale=K ** -0.5)
    ops = _ops()
    nb = ops.linear_f32_workspace_bytes(M, N)
    ws = torch.empty(nb, dtype=torch.uint8, device="cuda") if nb else None
    y = torch.full((M, N), float("nan"), device="cuda")
    ops.linear_f32(x.cuda(), w.cuda(), y, M, workspace=ws)
    assert _rel(y, x.double() @ w.double().T) < 3e-6
    if dtype == torch.float32 or K % 8:
        z = torch.full((M, N), float("nan"), device="cuda", dtype=dtype)
        ops.linear(x.cuda(), w.cuda(), z, M)
        assert _rel(z, x.double() @ w.double().T) < EPS[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,dim", [(1, 64), (3, 101), (2, 4096), (5, 2600), (40, 96), (300, 1032), (20, 4096), (2, 9000)])
def test_gated_norm_add(dtype, rows, dim):
    g = torch.Generator().manual_seed(rows + dim)
    ops, eps = _ops(), 1e-3
    slots_n, y_rows = 3, 3 * rows + 5
    y, resid, gate = _randn(g, y_rows, dim, dtype=dtype), _randn(g, rows, dim), _randn(g, rows, dim + 12)
    bias, post, nxt = (_randn(g, dim, dtype=dtype) for _ in range(3))
    slots = torch.randint(0, y_rows, (rows, slots_n), generator=g).int()
    r, normed = resid.clone().cuda(), torch.empty(rows, dim, dtype=dtype, device="cuda")
    ops.gated_norm_add(r, y.cuda(), gate.cuda(), dim + 12, bias.cuda(), post.cuda(), eps, nxt.cuda(), normed, rows, slots_n,
                       slots.cuda(), y_rows)
    t = y.double()[slots.long()].sum(1) * torch.sigmoid(gate[:, :dim].double() + bias.double())
    want = resid.double() + po.rms_norm(t, post.double(), eps)
    assert _rel(r, want) < 2e-6
    assert _rel(normed, po.rms_norm(want, nxt.double(), eps)) < EPS[dtype]
    # consecutive slots without an index list, and the sum alone
    out = torch.empty(rows, dim, dtype=dtype, device="cuda")
    ops.sum_slots(y.cuda(), rows, 3, None, 3 * rows, out)
    assert _rel(out, y[: 3 * rows].double().view(rows, 3, dim).sum(1)) < EPS[dtype]
    # embedding
    idx = torch.randint(0, y_rows, (rows,), generator=g)
    for ids in (idx, idx.int()):
        ops.embed_norm(y.cuda(), ids.cuda(), r, nxt.cuda(), eps, normed)
        assert torch.equal(r.cpu(), y.float()[idx])
        assert _rel(normed, po.rms_norm(y.double()[idx], nxt.double(), eps)) < EPS[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,S,H,dn,dr,r,pos0", [(1, 5, 3, 20, 6, 36, 0), (2, 7, 4, 32, 16, 64, 11), (1, 300, 9, 64, 32, 72, 900), (3, 1, 17, 8, 2, 24, 5)])
def test_latent_prepare_rotation_and_cache(dtype, B, S, H, dn, dr, r, pos0):
    """Rotation by halves at far positions, latent norm, cache rows; then the visible rows come back in order."""
    from gpt_fast.mixers import rotate_half_table
    g = torch.Generator().manual_seed(S)
    ops, smax, base, eps = _ops(), pos0 + S + 3, 300.0, 1e-4
    q_off, kv_off = 16, 16 + H * (dn + dr)
    ld = kv_off + r + dr + (-(kv_off + r + dr)) % 8
    proj, norm = _randn(g, B * S, ld), _randn(g, r, dtype=dtype)
    cache = torch.zeros(B, smax, r + dr, dtype=dtype, device="cuda")
    q = torch.empty(B * S, H, dn + dr, dtype=dtype, device="cuda")
    pos = torch.arange(pos0, pos0 + S)
    table = rotate_half_table(smax, dr, base, "cpu").cuda()
    ops.latent_prepare(proj.cuda(), ld, q_off, kv_off, norm.cuda(), eps, table, pos.cuda(), q, (H * (dn + dr), dn + dr), q.view(-1)[dn:],
                       (H * (dn + dr), dn + dr), cache, B, S, H, dn, dr, r)
    x = proj.double().view(B, S, ld)
    for b in range(B):
        qr = x[b, :, q_off:kv_off].view(S, H, dn + dr)
        want = torch.cat([qr[..., :dn], po.rotate_half_pairs(qr[..., dn:], pos, base)], -1)
        assert _rel(q.view(B, S, H, -1)[b], want) < EPS[dtype]
        kv = x[b, :, kv_off:kv_off + r + dr]
        want = torch.cat([po.rms_norm(kv[:, :r], norm.double(), eps), po.rotate_half_pairs(kv[:, r:], pos, base)], -1)
        assert _rel(cache[b, pos0:pos0 + S], want) < EPS[dtype]
    assert cache[:, :pos0].abs().sum() == 0 and cache[:, pos0 + S:].abs().sum() == 0
    hist = 4
    lat = torch.empty(B, hist + S, r, dtype=dtype, device="cuda")
    rot = torch.empty(B, hist + S, dr, dtype=dtype, device="cuda")
    ops.latent_window(cache, r, dr, pos.cuda(), B, hist, hist + S, lat, rot)
    for j in range(hist + S):
        p = pos0 - hist + j
        row = cache[:, p] if p >= 0 else torch.zeros_like(cache[:, 0])
        assert torch.equal(torch.cat([lat[:, j], rot[:, j]], -1), row)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,H,n_in,n_out", [(1, 5, 36, 20), (1, 4, 128, 512), (3, 2, 64, 72), (9, 3, 520, 40)])
@pytest.mark.parametrize("transposed", [False, True])
def test_head_linear(dtype, M, H, n_in, n_out, transposed):
    g = torch.Generator().manual_seed(n_in)
    x = _randn(g, M, H, n_in + 8, dtype=dtype)
    w = _randn(g, H, *((n_in, n_out) if transposed else (n_out, n_in)), dtype=dtype, scale=n_in ** -0.5)
    y = torch.full((M, H, n_out + 16), float("nan"), dtype=dtype, device="cuda")
    _ops().head_linear(x.cuda(), (H * (n_in + 8), n_in + 8), w.cuda(), transposed, y, (H * (n_out + 16), n_out + 16), M, H, n_in, n_out)
    want = torch.einsum("mhi,hio->mho" if transposed else "mhi,hoi->mho", x[..., :n_in].double(), w.double())
    assert _rel(y[..., :n_out], want) < EPS[dtype]
    assert torch.isnan(y[..., n_out:].float()).all()


def _attention_ref(q, k, k2, v, qpos, kpos, window, scale):
    s = torch.einsum("ihd,jhd->hij", q[..., : k.shape[-1]], k) + torch.einsum("ihd,jd->hij", q[..., k.shape[-1]:], k2)
    d = qpos[:, None] - kpos[None, :]
    ok = (d >= 0) & (d < window) & (kpos >= 0)[None, :]
    return torch.einsum("hij,jhd->ihd", torch.softmax((s * scale).masked_fill(~ok, float("-inf")), -1), v)


def _plant(q, k, i, j, h, strength=14.0):
    """Makes key row j stand out for query i of head h (and only there): it is aligned with the query."""
    u = q[i, h, : k.shape[-1]].float()
    k[j, h] = (u * strength / u.norm()).to(k.dtype)


@pytest.mark.parametrize("plain", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,H,d1,d2,dv,history,pos0,window", [
    (300, 2, 40, 24, 48, 0, 0, 75), (130, 3, 128, 64, 128, 63, 200, 64), (257, 2, 64, 32, 64, 64, 64, 65), (200, 1, 72, 8, 24, 40, 13, 100),
    (520, 2, 96, 64, 128, 0, 0, 4096), (33, 2, 8, 8, 8, 0, 0, 1), (150, 2, 20, 6, 12, 30, 90, 31), (2, 3, 32, 16, 32, 20, 40, 21)])
def test_window_attention_prompt(plain, dtype, S, H, d1, d2, dv, history, pos0, window):
    """Prompt form: the window's edges with planted keys exactly inside and exactly outside, keys before the portion,
    keys that do not exist (before position 0)."""
    from gpt_fast import _C
    if plain and dtype == torch.float32:
        pytest.skip("fp32 always runs the plain kernel")
    _C.lib.lri_set_option(b"window_tc", 0 if plain else 1)
    g = torch.Generator().manual_seed(S + window)
    B, n = 2, history + S
    scale = 1.3 * (d1 + d2) ** -0.5
    q = _randn(g, B, S, H, d1 + d2, dtype=dtype)
    k, v, k2 = _randn(g, B, n, H, d1, dtype=dtype), _randn(g, B, n, H, dv, dtype=dtype), _randn(g, B, n, d2, dtype=dtype)
    for i in range(0, S, 17):  # key row of query i is history + i
        inside, outside = history + i - window + 1, history + i - window
        h = (i // 17) % H
        if i % 2 == 0 and inside >= 0:
            _plant(q[1], k[1], i, inside, h)
        elif outside >= 0:
            _plant(q[1], k[1], i, outside, h)
    kv = torch.cat([k.reshape(B, n, H * d1), v.reshape(B, n, H * dv)], -1).contiguous()
    ld = H * (d1 + dv)
    out = torch.full((B * S, H * dv), float("nan"), dtype=dtype, device="cuda")
    pos = torch.arange(pos0, pos0 + S)
    kvd = kv.cuda()
    _ops().window_attention(q.cuda(), (H * (d1 + d2), d1 + d2), kvd, (n * ld, ld, d1), k2.cuda(), (n * d2, d2), kvd.view(-1)[H * d1:],
                            (n * ld, ld, dv), out, pos.int().cuda(), history, n, window, scale, B, S, H, d1, d2, dv)
    for b in range(B):
        want = _attention_ref(q[b].double(), k[b].double(), k2[b].double(), v[b].double(), pos, torch.arange(n) + pos0 - history, window,
                              scale)
        got = out.view(B, S, H, dv)[b]
        assert _rel(got, want) < EPS[dtype]
        worst = (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)
        assert worst.max() < 12 * EPS[dtype]


@pytest.mark.parametrize("plain", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,H,r,dr,smax,window,positions", [
    (1, 5, 80, 32, 700, 77, [0, 1, 63, 64, 76, 77, 78, 127, 128, 500, 699]), (3, 5, 48, 16, 200, 64, [5, 63, 64, 199]),
    (2, 17, 256, 64, 500, 129, [128, 129, 300]), (1, 2, 36, 6, 90, 17, [16, 17, 80]), (2, 16, 512, 64, 300, 4096, [299]), (1, 3, 16, 16, 70, 1, [0, 64, 69])])
def test_window_attention_single_token(plain, dtype, B, H, r, dr, smax, window, positions):
    """Single-token form on cached rows, with a planted row just inside or just outside the window."""
    from gpt_fast import _C
    if plain and dtype == torch.float32:
        pytest.skip("fp32 always runs the plain kernel")
    _C.lib.lri_set_option(b"window_tc", 0 if plain else 1)
    ops, L, scale = _ops(), r + dr, 1.0 / (r + dr) ** 0.5
    nb = ops.window_attention_scratch_bytes(B, H, r, min(window, smax))
    scratch = torch.empty(max(nb, 16), dtype=torch.uint8, device="cuda")
    for pos in positions:
        g = torch.Generator().manual_seed(pos)
        q, cache = _randn(g, B, H, L, dtype=dtype), _randn(g, B, smax, L, dtype=dtype)
        edge = pos - window + (1 if pos % 2 else 0)
        if edge >= 0:
            u = q[0, 0].float()
            cache[0, edge] = (u * 12.0 / u.norm()).to(dtype)
        out = torch.full((B, H * r), float("nan"), dtype=dtype, device="cuda")
        c = cache.cuda()
        ops.window_attention(q.cuda(), (H * L, L), c, (smax * L, L, 0), c.view(-1)[r:], (smax * L, L), c, (smax * L, L, 0), out,
                             torch.tensor([pos]).cuda(), -1, smax, window, scale, B, 1, H, r, dr, r, scratch)
        for b in range(B):
            lat = cache[b].double()[:, None, :r].expand(smax, H, r)
            want = _attention_ref(q[b].double()[None], lat, cache[b].double()[:, r:], lat, torch.tensor([pos]), torch.arange(smax), window, scale)
            assert _rel(out[b].view(1, H, r), want) < EPS[dtype], (pos, b)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B,S,H,C,E,bias,spread", [
    (1, 1, 2, 12, 20, 0, 1), (2, 5, 3, 64, 64, 0, 1), (1, 16, 2, 32, 32, 0, 2), (1, 300, 3, 20, 48, 1, 2), (2, 131, 2, 128, 128, 3, 2),
    (1, 700, 1, 64, 96, 4, 1), (1, 90, 2, 96, 16, -30, 20), (3, 33, 2, 16, 160, 0, 1), (1, 40, 1, 300, 24, 0, 1)])
def test_hgrn2(dtype, B, S, H, C, E, bias, spread):
    """Token-by-token and block forms from zero and from a state, with gates near 0, near 1 and at their lower bound."""
    from gpt_fast import _C
    g = torch.Generator().manual_seed(S + C)
    ops, eps = _ops(), 1e-4
    q_off, f_off, v_off = 8, 8 + H * C, 8 + 2 * H * C
    ld = v_off + H * E + (-(v_off + H * E)) % 8
    proj = _randn(g, B * S, ld)
    proj[:, f_off:v_off] = proj[:, f_off:v_off] * spread + bias
    fb, norm = _randn(g, H * C, dtype=dtype), _randn(g, E, dtype=dtype)
    low = (torch.rand(H * C, generator=g) * (torch.rand(H * C, generator=g) > 0.4)).clamp(max=0.98).to(dtype)
    st0 = _randn(g, B, H, C, E)
    x = proj.double()
    q = torch.nn.functional.silu(x[:, q_off:f_off]).view(B, S, H, C)
    f = (low.double() + (1 - low.double()) * torch.sigmoid(x[:, f_off:v_off] + fb.double())).view(B, S, H, C)
    v = x[:, v_off:v_off + H * E].to(dtype).double().view(B, S, H, E)
    for pos0 in (0, 9):
        ref = [po.hgrn2_recurrence(q[b], f[b], v[b], st0[b].double() if pos0 else None) for b in range(B)]
        for blocks in (1, 0):
            _C.lib.lri_set_option(b"hgrn2_blocks", blocks)
            st, out = st0.clone().cuda(), torch.full((B * S, H * E), float("nan"), dtype=dtype, device="cuda")
            ws = torch.empty(ops.hgrn2_workspace_bytes(dtype, B, S, H, C, E), dtype=torch.uint8, device="cuda")
            ops.hgrn2(proj.cuda(), ld, q_off, f_off, v_off, fb.cuda(), low.cuda(), norm.cuda(), eps, st,
                      torch.arange(pos0, pos0 + S).cuda(), out, B, S, H, C, E, ws)
            for b in range(B):
                assert _rel(st[b], ref[b][1]) < 5e-6, (pos0, blocks)
                want = po.rms_norm(ref[b][0], norm.double(), eps).reshape(S, H * E)
                assert _rel(out.view(B, S, -1)[b], want) < max(EPS[dtype], 5e-6), (pos0, blocks)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,experts,top,dim,ff", [(1, 5, 2, 64, 40), (3, 1, 1, 72, 24), (20, 6, 6, 128, 72), (150, 4, 1, 64, 136), (300, 12, 3, 192, 64),
                                                     (40, 3, 2, 20, 12)])
def test_mixture_of_experts(dtype, rows, experts, top, dim, ff):
    """Routing, packing by expert and both projections; packed and pair-by-pair forms."""
    from gpt_fast import _C
    g = torch.Generator().manual_seed(rows + ff)
    ops, pairs, glu = _ops(), rows * top, (1.702, 0.8, 1.0)
    x = _randn(g, rows, dim, dtype=dtype)
    logits = _randn(g, rows, experts + 8)
    w1, w2 = _randn(g, experts, 2 * ff, dim, dtype=dtype, scale=2 * dim ** -0.5), _randn(g, experts, dim, ff, dtype=dtype, scale=ff ** -0.5)
    best = torch.topk(torch.sigmoid(logits[:, :experts].double()), top, dim=-1)
    want = torch.zeros(rows, dim, dtype=torch.float64)
    for t in range(rows):
        for k in range(top):
            u = w1[best.indices[t, k]].double() @ (best.values[t, k] * x[t].double())
            want[t] += w2[best.indices[t, k]].double() @ po.clamped_glu(u[ff:], u[:ff], glu[1])
    xd, w1d, w2d, ld = x.cuda(), w1.cuda(), w2.cuda(), experts + 8

    def ints(n):
        return torch.zeros(n, dtype=torch.int32, device="cuda")

    for stream_pairs in (0, 65535):
        _C.lib.lri_set_option(b"moe_stream_pairs", stream_pairs)
        ids, scores, slots, y_rows = ints(pairs), torch.empty(pairs, device="cuda"), None, pairs
        if ops.moe_packs(dtype, rows, top, dim, ff):
            tiles = ops.moe_max_tiles(rows, top, experts)
            counts, rank, first, tl = ints(experts), ints(pairs), ints(experts), ints(1 + tiles)
            packed = torch.zeros(128 * tiles, dim, dtype=dtype, device="cuda")
            scale, slots = torch.zeros(128 * tiles, device="cuda"), ints(pairs)
            h, y, y_rows = torch.empty(128 * tiles, ff, dtype=dtype, device="cuda"), torch.empty(128 * tiles, dim, dtype=dtype, device="cuda"), 128 * tiles
            for _ in range(2):  # the second call finds the counts as the first left them
                ops.moe_route(logits.cuda(), ld, experts, top, rows, ids, scores, counts, rank)
                ops.moe_pack(xd, rows, top, experts, ids, scores, rank, counts, first, tl, tiles, packed, scale, slots)
            assert counts.sum() == 0 and len(set(slots.tolist())) == pairs
            ops.moe_gateup(packed, w1d, h, None, None, pairs, top, glu, tiles=tl, row_scale=scale, max_tiles=tiles)
            ops.moe_down(h, w2d, y, None, pairs, tiles=tl, max_tiles=tiles)
        else:
            h, y = torch.empty(pairs, ff, dtype=dtype, device="cuda"), torch.empty(pairs, dim, dtype=dtype, device="cuda")
            ops.moe_route(logits.cuda(), ld, experts, top, rows, ids, scores)
            ops.moe_gateup(xd, w1d, h, ids, scores, pairs, top, glu)
            ops.moe_down(h, w2d, y, ids, pairs)
        assert torch.equal(ids.view(rows, top).cpu().long(), best.indices)
        assert _rel(scores.view(rows, top), best.values) < 1e-6
        out = torch.empty(rows, dim, dtype=dtype, device="cuda")
        ops.sum_slots(y, rows, top, slots, y_rows, out)
        assert _rel(out, want) < 2 * EPS[dtype]


def test_router_ties_take_the_lowest_expert():
    logits = torch.tensor([[1.0, 2.0, 2.0, 2.0], [0.0, 0.0, 0.0, 0.0]]).cuda()
    ids, scores = torch.zeros(4, dtype=torch.int32, device="cuda"), torch.empty(4, device="cuda")
    _ops().moe_route(logits, 4, 4, 2, 2, ids, scores)
    assert ids.tolist() == [1, 2, 0, 1]


# ---- whole models ------------------------------------------------------------------------------------------------
LIMIT = {torch.float32: (2e-5, 2e-4), torch.bfloat16: (2e-2, 6e-2), torch.float16: (4e-3, 2e-2)}  # median and largest error


def _close(got, ref, dtype, what=""):
    e = pu.row_err(got, ref).flatten()
    assert torch.isfinite(e).all() and e.median() < LIMIT[dtype][0] and e.max() < LIMIT[dtype][1], (what, e.median(), e.max())


_CACHE = {}


def _case(name, dtype, n=150, seed=1):
    """(config, weights, tokens, oracle logits).  In 16 bits a close router decision may go the other way, which no limit
    could tell from a fault: there every token uses all experts (the choice itself is tested in fp32 and alone)."""
    key = (name, dtype == torch.float32, n, seed)
    if key not in _CACHE:
        cfg = copy.deepcopy(pu.CONFIGS[name])
        for layer in cfg["layers"]:
            if layer["mlp"] and dtype != torch.float32:
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
        w = pu.weights(cfg, 7)
        toks = pu.tokens(cfg, n, seed)
        _CACHE[key] = (cfg, w, toks, pu.reference(cfg, w, toks))
    return _CACHE[key]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(pu.CONFIGS))
@pytest.mark.parametrize("cuts", [[150], [1], [2], [100, 1], [3, 2, 64, 16, 17, 1], [65, 7]], ids=str)
def test_model_prompts_portions_and_single_tokens(name, dtype, cuts):
    cfg, w, toks, ref = _case(name, dtype)
    model = pu.build(cfg, w, dtype, "cuda", 1, 152)
    _close(pu.feed(model, toks[None], cuts)[0], ref, dtype, cuts)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["uneven", "tiles"])
def test_batches_and_reused_rows(name, dtype):
    """Rows of a batch do not see one another; a row that served a longer sequence serves another from position 0."""
    cfg, w, toks, ref = _case(name, dtype)
    model = pu.build(cfg, w, dtype, "cuda", 3, 152)
    rows = torch.stack([toks[:90], pu.tokens(cfg, 90, 11), pu.tokens(cfg, 90, 12)])
    refs = torch.stack([pu.reference(cfg, w, r) for r in rows])
    _close(pu.feed(model, rows, [80, 1]), refs, dtype)
    other = pu.tokens(cfg, 60, 13)
    _close(pu.feed(model, other[None], [20, 1, 30])[0], pu.reference(cfg, w, other), dtype, "reused")
    _close(pu.feed(model, rows[:2], [33, 1, 40]), refs[:2], dtype, "two rows of three")
    if dtype == torch.float32:
        alone = pu.build(cfg, w, dtype, "cuda", 1, 152)
        assert (pu.feed(alone, rows[1:2], [80, 1]) - pu.feed(model, rows, [80, 1])[1:2]).abs().max() < 1e-4


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_window_edge_reaches_the_logits(dtype):
    """One attention layer with a strong key: moving the planted token across the window's edge changes the logits of
    the query by a lot when it is inside and not at all when it is outside; in a prompt and decoded."""
    window = 40
    cfg = pu.config(128, 90, [(pu.latent(2, 32, 16, 32, 48, window), None)])
    w = pu.weights(cfg, 5)
    n, qpos = 130, 120
    for decoded in (False, True):
        for gap, seen in ((window - 1, True), (window, False)):
            base = pu.tokens(cfg, n, 21)
            moved = base.clone()
            moved[qpos - gap] = (moved[qpos - gap] + 37) % 90
            model = pu.build(cfg, w, dtype, "cuda", 1, n)
            cuts = [qpos, 1] if decoded else [n]
            a, b = (pu.feed(model, t[None], cuts)[0, qpos] for t in (base, moved))
            if seen:
                assert (a - b).abs().max() > 1e-2, (decoded, gap)
            else:
                assert torch.equal(a, b), (decoded, gap)
            assert pu.row_err(b[None], pu.reference(cfg, w, moved)[qpos][None]).max() < LIMIT[dtype][1]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_greedy_decoding_through_the_device_loop(dtype):
    """DeviceLoop (captured steps, state put back after the warm-up) against the oracle fed the same tokens: every
    chosen token is the oracle's best, or within rounding of it."""
    from gpt_fast.generate import DeviceLoop
    cfg, w, toks, _ = _case("tiles", dtype)
    model = pu.build(cfg, w, dtype, "cuda", 2, 240)
    prompt = torch.stack([toks[:30], pu.tokens(cfg, 30, 31)])
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
        ref = pu.reference(cfg, w, seq[:-1])[29:]
        best = ref.max(-1).values
        chosen = ref.gather(1, seq[30:, None]).squeeze(1)
        slack = (3e-4 if dtype == torch.float32 else 0.25) * ref.std(-1)
        assert (best - chosen < slack).float().mean() > (0.999 if dtype == torch.float32 else 0.95)


def test_sampling_and_last_logits():
    cfg, w, toks, ref = _case("uneven", torch.bfloat16)
    model = pu.build(cfg, w, torch.bfloat16, "cuda", 1, 152)
    pos = torch.arange(60, dtype=torch.int32, device="cuda")
    last = model.prefill_last(toks[None, :60].cuda(), pos)[0, 0].float().cpu()
    full = pu.build(cfg, w, torch.bfloat16, "cuda", 1, 152)(toks[None, :60].cuda(), pos)[0, -1].float().cpu()
    assert torch.allclose(last, full, atol=3e-2 * full.abs().max())
    state = [s.clone() for s in model.recurrent_state()]
    nxt, p = toks[None, 60:61].int().cuda(), torch.tensor([60], dtype=torch.int32, device="cuda")
    greedy = model.decode_greedy(nxt, p).clone()
    for s, s0 in zip(model.recurrent_state(), state):
        s.copy_(s0)
    gen = torch.Generator(device="cuda").manual_seed(1)
    assert torch.equal(greedy, model.decode_sample(nxt, p, temperature=0.7, top_k=1, generator=gen))


def test_checkpoint_folder_and_trace_replay(tmp_path):
    """bin/trace_run on a checkpoint folder: two requests one after the other, portions and single tokens."""
    import numpy as np
    cfg, w, toks, ref = _case("uneven", torch.float32)
    pu.save(cfg, w, tmp_path / "model")
    os.makedirs(tmp_path / "out")
    other = pu.tokens(cfg, 40, 77)
    ref2 = pu.reference(cfg, w, other)
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
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out",
                        str(tmp_path / "out"), "--max-tokens", "150"], input=text, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    for i, ref_i in enumerate(want):
        path = tmp_path / "out" / f"{i}.f32"
        assert path.exists() == (ref_i is not None)
        if ref_i is not None:
            got = torch.from_numpy(np.fromfile(path, dtype="<f4")).view(-1, cfg["vocab"])
            assert got.shape == ref_i.shape and pu.row_err(got, ref_i).max() < LIMIT[torch.float32][1]


def test_trace_replay_refuses_types_without_kernels(tmp_path):
    json.dump(dict(num_hidden_layers=1, vocab_size=64, num_attention_heads=2, hidden_size=64, intermediate_size=128),
              open(tmp_path / "config.json", "w"))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "8"], input="", capture_output=True, text=True, timeout=300)
    assert r.returncode == 3
