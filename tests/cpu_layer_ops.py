"""CPU stand-in for the device ops of layer-list designs, from the oracle's functions.  TEST INFRASTRUCTURE: it lets the
engine's host code (order of steps, buffers, sharding, all-reduces) run on CPU ranks; the product never uses it."""
import torch

from oracle import migosun_oracle as mo
from oracle import patevik_oracle as po


def _rows(t, rows, cols):
    return t.view(-1)[: rows * cols].view(rows, cols)


class CpuLayerOps:
    name = "cpu-oracle-stand-in"
    linear_workspace_bytes = linear_f32_workspace_bytes = staticmethod(lambda *a: 0)
    hgrn2_workspace_bytes = window_attention_scratch_bytes = staticmethod(lambda *a: 0)
    moe_packs = staticmethod(lambda *a: False)
    moe_max_tiles = staticmethod(lambda *a: 1)

    @staticmethod
    def linear(x, w, out, rows, addend=None, workspace=None):
        _rows(out, rows, w.shape[0])[:] = _rows(x, rows, w.shape[1]) @ w.T

    linear_f32 = linear

    @staticmethod
    def embed_norm(table, idx, resid, weight, eps, normed):
        x = table[idx.reshape(-1).long()].float()
        resid[: x.shape[0]] = x
        normed[: x.shape[0]] = po.rms_norm(x, weight, eps)

    @staticmethod
    def _sum(y, rows, n_slots, slots, d):
        idx = slots[: rows * n_slots].long() if slots is not None else torch.arange(rows * n_slots)
        return y.view(-1, d)[idx].view(rows, n_slots, d).sum(1)

    @classmethod
    def sum_slots(cls, y, rows, n_slots, slots, y_rows, out):
        out[:rows] = cls._sum(y, rows, n_slots, slots, out.shape[-1])

    @classmethod
    def gated_norm_add(cls, resid, y, gate, gate_ld, bias, post, eps, nxt, normed, rows, n_slots=1, slots=None, y_rows=None):
        d = resid.shape[-1]
        t = cls._sum(y, rows, n_slots, slots, d) * torch.sigmoid(_rows(gate, rows, gate_ld)[:, :d] + bias)
        resid[:rows] += po.rms_norm(t, post, eps)
        normed[:rows] = po.rms_norm(resid[:rows], nxt, eps)

    @staticmethod
    def latent_prepare(proj, ld, q_off, kv_off, norm, eps, table, pos, qn, qn_pitch, qr, qr_pitch, cache, B, S, H, dn, dr, r):
        rows = B * S
        x = _rows(proj, rows, ld)
        p = pos.long().repeat(B)
        cs = table[p]

        def rot(v):  # [rows, ..., dr]
            c, s = cs[..., 0], cs[..., 1]
            while c.dim() < v.dim():
                c, s = c.unsqueeze(1), s.unsqueeze(1)
            a, b = v[..., : dr // 2], v[..., dr // 2:]
            return torch.cat([a * c - b * s, b * c + a * s], -1)

        q = x[:, q_off:q_off + H * (dn + dr)].view(rows, H, dn + dr)
        torch.as_strided(qn, (rows, H, dn), (*qn_pitch, 1), qn.storage_offset())[:] = q[..., :dn]
        torch.as_strided(qr, (rows, H, dr), (*qr_pitch, 1), qr.storage_offset())[:] = rot(q[..., dn:])
        kv = x[:, kv_off:kv_off + r + dr]
        lat = torch.cat([po.rms_norm(kv[:, :r], norm, eps), rot(kv[:, r:])], -1)
        cache[:B, pos.long()] = lat.view(B, S, -1)

    @staticmethod
    def latent_window(cache, r, dr, pos, B, history, rows, lat, k_rot):
        p = int(pos[0]) - history + torch.arange(rows)
        v = cache[:B, p.clamp(min=0)] * (p >= 0)[None, :, None]
        _rows(lat, B * rows, r)[:] = v[..., :r].reshape(B * rows, r)
        _rows(k_rot, B * rows, dr)[:] = v[..., r:].reshape(B * rows, dr)

    @staticmethod
    def head_linear(x, x_pitch, w, transposed, y, y_pitch, rows, H, n_in, n_out):
        xv = torch.as_strided(x, (rows, H, n_in), (*x_pitch, 1), x.storage_offset())
        yv = torch.as_strided(y, (rows, H, n_out), (*y_pitch, 1), y.storage_offset())
        m = w.reshape(H, n_in, n_out) if transposed else w.reshape(H, n_out, n_in).transpose(1, 2)
        yv[:] = torch.einsum("rhi,hio->rho", xv, m)

    @staticmethod
    def window_attention(q, q_pitch, k, k_pitch, k2, k2_pitch, v, v_pitch, out, pos, history, k_rows, window, scale, B, S, H,
                         d1, d2, dv, scratch=None):
        def view(t, n, pitch):
            return torch.as_strided(t, (B, k_rows, H, n), (pitch[0], pitch[1], pitch[2], 1), t.storage_offset())

        qv = torch.as_strided(q, (B, S, H, d1 + d2), (S * q_pitch[0], *q_pitch, 1), q.storage_offset())
        kv, vv = view(k, d1, k_pitch), view(v, dv, v_pitch)
        k2v = torch.as_strided(k2, (B, k_rows, d2), (*k2_pitch, 1), k2.storage_offset())
        score = torch.einsum("bihd,bjhd->bhij", qv[..., :d1], kv) + torch.einsum("bihd,bjd->bhij", qv[..., d1:], k2v)
        kp = torch.arange(k_rows) + (0 if history < 0 else int(pos[0]) - history)
        dist_ = pos.long()[:, None] - kp[None, :]
        ok = (dist_ >= 0) & (dist_ < window) & (kp >= 0)[None, :]
        p = torch.softmax((score * scale).masked_fill(~ok, float("-inf")), -1)
        _rows(out, B * S, H * dv)[:] = torch.einsum("bhij,bjhd->bihd", p, vv).reshape(B * S, H * dv)

    @staticmethod
    def hgrn2(proj, ld, q_off, f_off, v_off, f_bias, lower, norm, eps, state, pos, out, B, S, H, C, E, ws):
        x = _rows(proj, B * S, ld).view(B, S, ld)
        for b in range(B):
            q = x[b, :, q_off:q_off + H * C]
            q = (q * torch.sigmoid(q)).view(S, H, C)
            f = (lower + (1 - lower) * torch.sigmoid(x[b, :, f_off:f_off + H * C] + f_bias)).view(S, H, C)
            st = None if int(pos[0]) == 0 else state[b].clone()
            o, st = po.hgrn2_recurrence(q, f, x[b, :, v_off:v_off + H * E].reshape(S, H, E), st)
            state[b] = st
            _rows(out, B * S, H * E)[b * S:(b + 1) * S] = po.rms_norm(o, norm, eps).reshape(S, H * E)

    @staticmethod
    def moe_route(logits, ld, n, top, rows, ids, scores, counts=None, rank=None):
        z = torch.as_strided(logits, (rows, n), (ld, 1), logits.storage_offset())
        best = torch.topk(torch.sigmoid(z), top, dim=-1)
        ids[: rows * top] = best.indices.reshape(-1).int()
        scores[: rows * top] = best.values.reshape(-1)

    @staticmethod
    def moe_gateup(x, w1, hidden, ids, scores, pairs, top, glu, **kw):
        n, two_ff, d = w1.shape
        assert glu[0] == 1.702 and glu[2] == 1.0
        for i in range(pairs):
            u = w1[int(ids[i])] @ (scores[i] * x[i // top])
            hidden.view(-1)[i * two_ff // 2:(i + 1) * two_ff // 2] = po.clamped_glu(u[two_ff // 2:], u[: two_ff // 2], glu[1])

    @staticmethod
    def moe_down(hidden, w2, y, ids, pairs, **kw):
        n, d, ff = w2.shape
        for i in range(pairs):
            y.view(-1)[i * d:(i + 1) * d] = w2[int(ids[i])] @ hidden.view(-1)[i * ff:(i + 1) * ff]

    # ---- residual streams, grouped attention, matrix states, dense unit ----------------------------------------------
    gateup_glu_workspace_bytes = staticmethod(lambda *a: 0)
    state_blocks = staticmethod(lambda S: -(-S // 4))
    state_step_supports = staticmethod(lambda *a: False)

    @staticmethod
    def embed_streams(table, idx, scale, streams, in_next, weight, eps, normed):
        x = table[idx.reshape(-1).long()].float() * scale
        n = x.shape[0]
        streams[:n] = x[:, None]
        normed[:n] = mo.rms_norm(torch.einsum("s,rsd->rd", in_next, streams[:n]), weight, eps)

    @staticmethod
    def join_streams(streams, y, mix, out, in_next, weight, eps, normed, rows, write=True):
        new = torch.einsum("st,rsd->rtd", mix, streams[:rows]) + out[None, :, None] * y[:rows, None]
        if write:
            streams[:rows] = new
        normed[:rows] = mo.rms_norm(new.sum(1) if in_next is None else torch.einsum("s,rsd->rd", in_next, new), weight, eps)

    @staticmethod
    def gateup_glu(x, w1, h, rows, glu, workspace=None):
        assert glu[0] == 1.702 and glu[2] == 1.0
        u = _rows(x, rows, w1.shape[1]) @ w1.T
        ff = w1.shape[0] // 2
        _rows(h, rows, ff)[:] = mo.clamped_glu(u[:, ff:], u[:, :ff], glu[1])

    @staticmethod
    def row_squares(x, ld, off1, n1, off2, n2, sums, rows):
        v = _rows(x, rows, ld)
        sums[:rows, 0], sums[:rows, 1] = (v[:, off1:off1 + n1] ** 2).sum(-1), (v[:, off2:off2 + n2] ** 2).sum(-1)

    @staticmethod
    def grouped_prepare(proj, ld, offs, q_norm, k_norm, sums, widths, eps, table, rot_dims, pos, q, kc, vc, B, S, H):
        rows, (_, G, _, d), dv = B * S, kc.shape, vc.shape[3]
        x, cs = _rows(proj, rows, ld), table[pos.long().repeat(B)][:, None]

        def normed(off, heads, w, i):
            v = x[:, off:off + heads * d]
            total = sums[:rows, i:i + 1] if sums is not None else (v * v).sum(-1, keepdim=True)
            v = (v / torch.sqrt(total / widths[i] + eps) * w).view(rows, heads, d)
            a, b = v[..., : rot_dims // 2], v[..., rot_dims // 2:rot_dims]
            c, s = cs[..., : rot_dims // 2, 0], cs[..., : rot_dims // 2, 1]
            return torch.cat([a * c - b * s, b * c + a * s, v[..., rot_dims:]], -1)

        _rows(q, rows, H * d)[:] = normed(offs[0], H, q_norm, 0).reshape(rows, -1)
        kc[:B, :, pos.long()] = normed(offs[1], G, k_norm, 1).view(B, S, G, d).transpose(1, 2)
        vc[:B, :, pos.long()] = x[:, offs[2]:offs[2] + G * dv].view(B, S, G, dv).transpose(1, 2)

    @staticmethod
    def grouped_attention(q, kc, vc, sink, out, out_ld, factor, pos, window, chunk, scale, B, S, H):
        _, G, smax, d = kc.shape
        dv, group = vc.shape[3], torch.arange(H) // (H // G)
        i, j = pos.long()[:, None], torch.arange(smax)[None, :]
        ok = j <= i
        if window:
            ok &= i - j < window
        if chunk:
            ok &= i // chunk == j // chunk
        y = torch.as_strided(out, (B * S, H * dv), (out_ld, 1), out.storage_offset())
        for b in range(B):
            qb = _rows(q, B * S, H * d)[b * S:(b + 1) * S].view(S, H, d)
            score = (torch.einsum("ihd,hjd->hij", qb, kc[b][group]) * scale).masked_fill(~ok, float("-inf"))
            y[b * S:(b + 1) * S] = factor * torch.einsum("hij,hjd->ihd", mo.softmax_with_sink(score, sink), vc[b][group]).reshape(S, -1)

    @staticmethod
    def round_columns(x, ld, off, n, y, rows):
        _rows(y, rows, n)[:] = _rows(x, rows, ld)[:, off:off + n]

    # the block vectors carry q, k, decay and step size as they are
    @staticmethod
    def delta_blocks(proj, ld, offs, convs, ring, z, a_log, dt_bias, pos, blocks, v, B, S, H, G, C, E):
        qd, kd, ku, _, coef = blocks
        x, taps, p0 = _rows(proj, B * S, ld).view(B, S, ld), convs[0].shape[1], int(pos[0])
        group = torch.arange(H) // (H // G)
        for b in range(B):
            parts, at = [], 0
            for off, w in zip(offs, convs):
                n = w.shape[0]
                old = [ring[b, (p0 - j) % taps, at:at + n] if p0 - j >= 0 else torch.zeros(n) for j in range(taps - 1, 0, -1)]
                seq = torch.cat([torch.stack(old), x[b, :, off:off + n]]) if old else x[b, :, off:off + n]
                parts.append(mo.silu(mo.short_conv(seq, w))[taps - 1:])
                at += n
            for s in range(max(0, S - taps), S):
                ring[b, (p0 + s) % taps] = torch.cat([x[b, s, o:o + w.shape[0]] for o, w in zip(offs, convs)])
            r = slice(b * S, (b + 1) * S)
            _rows(qd, B * S, H * C)[r] = (mo.unit(parts[0].view(S, G, C)) * C ** -0.5)[:, group].reshape(S, -1)
            _rows(kd, B * S, H * C)[r] = mo.unit(parts[1].view(S, G, C))[:, group].reshape(S, -1)
            _rows(v, B * S, H * E)[r] = parts[2]
            _rows(ku, B * S, H * C)[r] = mo.delta_decay(_rows(z, B * S, H * C)[r].view(S, H, C), a_log, dt_bias).reshape(S, -1)
            _rows(coef, B * S, H)[r] = torch.sigmoid(x[b, :, offs[3]:offs[3] + H])

    @staticmethod
    def gla_blocks(proj, ld, offs, z, bias, tau, blocks, B, S, H, C):
        qd, _, ku, _, coef = blocks
        x, n = _rows(proj, B * S, ld), H * C
        _rows(qd, B * S, n)[:] = x[:, offs[0]:offs[0] + n] * C ** -0.5
        _rows(ku, B * S, n)[:] = torch.exp(torch.nn.functional.logsigmoid(_rows(z, B * S, n) + bias) / tau)
        CpuLayerOps._gla_k = x[:, offs[1]:offs[1] + n].clone()

    @staticmethod
    def state_scan(blocks, delta, v, v_row, state, pos, o, B, S):
        qd, kd, ku, _, coef = blocks
        _, H, C, E = state.shape
        vv = torch.as_strided(v, (B * S, H * E), (v_row, 1), v.storage_offset())
        for b in range(B):
            r = slice(b * S, (b + 1) * S)
            st = None if int(pos[0]) == 0 else state[b].clone()
            q, g = (_rows(t, B * S, H * C)[r].view(S, H, C) for t in (qd, ku))
            k = (_rows(kd, B * S, H * C) if delta else CpuLayerOps._gla_k)[r].view(S, H, C)
            if delta:
                out, st = mo.delta_recurrence(q, k, vv[r].view(S, H, E), g, _rows(coef, B * S, H)[r], st)
            else:
                out, st = mo.linear_attention_recurrence(q, k, vv[r].view(S, H, E), g, st)
            state[b] = st
            _rows(o, B * S, H * E)[r] = out.reshape(S, -1)

    @staticmethod
    def head_norm_gate(o, norm, eps, gate, gate_ld, activation, scale, out, out_ld, rows, H):
        E = norm.numel()
        g = torch.as_strided(gate, (rows, H * E), (gate_ld, 1), gate.storage_offset())
        act = torch.sigmoid(g) if activation == "sigmoid" else mo.silu(g)
        y = mo.rms_norm(_rows(o, rows, H * E).view(rows, H, E), norm, eps).reshape(rows, -1) * act * scale
        torch.as_strided(out, (rows, H * E), (out_ld, 1), out.storage_offset())[:] = y
