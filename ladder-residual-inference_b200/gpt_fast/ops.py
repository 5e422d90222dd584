"""The fused device operations of the decode/prefill step as Python callables over the C ABI.

`CudaOps` is the only implementation the package ships; it needs liblri_b200.so and CUDA
tensors and raises otherwise.  The engine takes the ops object as a parameter so that host-side
schedule logic can be exercised by tests with a stand-in.
"""
import ctypes

import torch

from . import _C


class CudaOps:
    name = "sm_100a"

    # ---- F1 and embedding -----------------------------------------------------------------
    @staticmethod
    def embedding(table, idx, out):
        _C.require_cuda(table, idx, out)
        if idx.dtype not in (torch.int32, torch.int64):
            idx = idx.to(torch.int64)
        idx = idx.contiguous()
        n = idx.numel()
        _C.check(_C.lib.lri_embedding(_C.dtype_code(table.dtype), table.data_ptr(), idx.data_ptr(),
                                      int(idx.dtype == torch.int64), out.data_ptr(), n, table.shape[1],
                                      table.shape[0], _C.stream_handle()))

    @staticmethod
    def add_rmsnorm(residual, add1, add2, weight, eps, residual_out, normed_out, rows, scale=1.0):
        _C.require_cuda(residual)
        dim = residual.shape[-1]
        _C.check(_C.lib.lri_add_rmsnorm(_C.dtype_code(residual.dtype), residual.data_ptr(), _C.ptr(add1), _C.ptr(add2),
                                        float(scale), _C.ptr(weight), float(eps), _C.ptr(residual_out),
                                        _C.ptr(normed_out), rows, dim, _C.stream_handle()))

    # ---- linear family -----------------------------------------------------------------------
    @staticmethod
    def linear(x, w, out, rows, addend=None, workspace=None):
        _C.require_cuda(x, w, out)
        n, k = w.shape
        ws_ptr, ws_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) if workspace is not None else (None, 0)
        _C.check(_C.lib.lri_linear(_C.dtype_code_any(x.dtype), x.data_ptr(), w.data_ptr(), _C.ptr(addend), out.data_ptr(),
                                   rows, n, k, ws_ptr, ws_bytes, _C.stream_handle()))

    @staticmethod
    def linear_workspace_bytes(rows, n):
        return _C.lib.lri_linear_workspace_bytes(rows, n)

    @staticmethod
    def qkv_workspace_bytes(rows, n_head, n_kv, head_dim):
        return _C.lib.lri_qkv_workspace_bytes(rows, n_head, n_kv, head_dim)

    @staticmethod
    def gateup_workspace_bytes(rows, inter):
        return _C.lib.lri_gateup_workspace_bytes(rows, inter)

    @staticmethod
    def qkv_rope_kvcache(x, wqkv, table, table_gathered, input_pos, q_out, k_cache, v_cache, B, S, n_head, n_kv,
                         head_dim, workspace):
        _C.require_cuda(x, wqkv, table, input_pos, q_out, k_cache, v_cache)
        assert input_pos.dtype in (torch.int32, torch.int64)
        k = wqkv.shape[1]
        smax = k_cache.shape[2]
        ws_ptr, ws_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) if workspace is not None else (None, 0)
        _C.check(_C.lib.lri_qkv_rope_kvcache(
            _C.dtype_code(x.dtype), x.data_ptr(), wqkv.data_ptr(), table.data_ptr(), input_pos.data_ptr(),
            int(input_pos.dtype == torch.int64), q_out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), B, S, k,
            n_head, n_kv, head_dim, smax, table.shape[0], int(table_gathered), ws_ptr, ws_bytes, _C.stream_handle()))

    @staticmethod
    def gateup_swiglu(x, w1, h, rows, workspace):
        _C.require_cuda(x, w1, h)
        two_i, k = w1.shape
        ws_ptr, ws_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) if workspace is not None else (None, 0)
        _C.check(_C.lib.lri_gateup_swiglu(_C.dtype_code(x.dtype), x.data_ptr(), w1.data_ptr(), h.data_ptr(), rows,
                                          two_i // 2, k, ws_ptr, ws_bytes, _C.stream_handle()))

    # ---- greedy head ---------------------------------------------------------------------------------
    @staticmethod
    def lm_head_argmax_scratch_bytes(rows=0, n=0):
        return _C.lib.lri_lm_head_argmax_scratch_bytes()

    @staticmethod
    def lm_head_argmax(x, w, index_offset, token_out, rows, scratch, comm_handle=None, logits_ws=None, workspace=None,
                       timeout_ms=2000):
        """token_out[m] = arg-max over the whole vocabulary of sequence m, where `w` holds this rank's rows
        starting at vocabulary index `index_offset` (w may have no rows)."""
        _C.require_cuda(x, token_out, scratch)
        assert token_out.dtype == torch.int32
        n = w.shape[0]
        k = w.shape[1] if w.dim() == 2 else x.shape[-1]
        lw_ptr, lw_bytes = (logits_ws.data_ptr(), logits_ws.numel() * logits_ws.element_size()) if logits_ws is not None else (None, 0)
        ws_ptr, ws_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) if workspace is not None else (None, 0)
        _C.check(_C.lib.lri_lm_head_argmax(comm_handle, _C.dtype_code(x.dtype), x.data_ptr(), w.data_ptr() if n else None,
                                           rows, n, k, index_offset, token_out.data_ptr(), scratch.data_ptr(),
                                           scratch.numel() * scratch.element_size(), lw_ptr, lw_bytes, ws_ptr, ws_bytes,
                                           timeout_ms, _C.stream_handle()))

    # ---- attention ---------------------------------------------------------------------------------
    @staticmethod
    def attn_decode_scratch_bytes(B, n_head, n_kv, head_dim, num_splits):
        return _C.lib.lri_attn_decode_scratch_bytes(B, n_head, n_kv, head_dim, num_splits)

    @staticmethod
    def attention(q, k_cache, v_cache, input_pos, out, B, S, n_head, n_kv, head_dim, scratch, num_splits):
        _C.require_cuda(q, k_cache, v_cache, input_pos, out)
        code = _C.dtype_code(q.dtype)
        smax = k_cache.shape[2]
        i64 = int(input_pos.dtype == torch.int64)
        if S == 1:
            _C.check(_C.lib.lri_attn_decode(code, q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                            input_pos.data_ptr(), i64, out.data_ptr(), B, n_head, n_kv, head_dim,
                                            smax, num_splits, scratch.data_ptr(),
                                            scratch.numel() * scratch.element_size(), _C.stream_handle()))
        else:
            _C.check(_C.lib.lri_attn_prefill(code, q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                             input_pos.data_ptr(), i64, out.data_ptr(), B, S, n_head, n_kv, head_dim,
                                             smax, _C.stream_handle()))


    # ---- layers with an fp32 residual stream ---------------------------------------------------------
    @staticmethod
    def linear_f32(x, w, out, rows, workspace=None):
        """out (fp32) = x w^T, unrounded."""
        _C.require_cuda(x, w, out)
        n, k = w.shape
        ws_ptr, ws_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) if workspace is not None else (None, 0)
        _C.check(_C.lib.lri_linear_f32(_C.dtype_code_any(x.dtype), x.data_ptr(), w.data_ptr(), out.data_ptr(), rows, n, k,
                                       ws_ptr, ws_bytes, _C.stream_handle()))

    @staticmethod
    def linear_f32_workspace_bytes(rows, n):
        return _C.lib.lri_linear_f32_workspace_bytes(rows, n)

    @staticmethod
    def embed_norm(table, idx, resid, weight, eps, normed):
        _C.require_cuda(table, idx, resid)
        if idx.dtype not in (torch.int32, torch.int64):
            idx = idx.to(torch.int64)
        idx = idx.contiguous()
        _C.check(_C.lib.lri_embed_norm(_C.dtype_code_any(table.dtype), table.data_ptr(), idx.data_ptr(),
                                       int(idx.dtype == torch.int64), table.shape[0], resid.data_ptr(), _C.ptr(weight),
                                       float(eps), _C.ptr(normed), idx.numel(), table.shape[1], _C.stream_handle()))

    @staticmethod
    def gated_norm_add(resid, y, gate, gate_ld, gate_bias, post_weight, eps, next_weight, normed, rows, n_slots=1,
                       slots=None, y_rows=None):
        """resid += post norm of the gated sum over slots of y; normed = norm of the new residual.  `gate` is a
        view that starts at the gate's first column of an fp32 buffer with row pitch gate_ld."""
        _C.require_cuda(resid, y)
        _C.check(_C.lib.lri_gated_norm_add(_C.dtype_code_any(y.dtype), resid.data_ptr(), y.data_ptr(), _C.ptr(slots), n_slots,
                                           y_rows if y_rows is not None else rows * n_slots, _C.ptr(gate), gate_ld,
                                           _C.ptr(gate_bias), _C.ptr(post_weight), float(eps), resid.data_ptr(),
                                           _C.ptr(next_weight), _C.ptr(normed), rows, resid.shape[-1], _C.stream_handle()))

    @staticmethod
    def sum_slots(y, rows, n_slots, slots, y_rows, out):
        """out[r] = sum of the rows slots[r, :] of y (slots None: rows r * n_slots ...), rounded once."""
        _C.require_cuda(y, out)
        _C.check(_C.lib.lri_gated_norm_add(_C.dtype_code_any(y.dtype), None, y.data_ptr(), _C.ptr(slots), n_slots, y_rows, None, 0,
                                           None, None, 0.0, None, None, out.data_ptr(), rows, out.shape[-1],
                                           _C.stream_handle()))

    # ---- latent attention ------------------------------------------------------------------------------
    @staticmethod
    def latent_prepare(proj, ld, q_off, kv_off, norm_weight, eps, table, input_pos, qn, qn_pitch, qr, qr_pitch, cache, B, S,
                       heads, dim, rot_dim, rank):
        """qn_pitch, qr_pitch: (row, head) element pitches of the unrotated and the rotated part of q."""
        _C.require_cuda(proj, norm_weight, table, input_pos, qn, qr, cache)
        _C.check(_C.lib.lri_latent_prepare(
            _C.dtype_code_any(cache.dtype), proj.data_ptr(), ld, q_off, kv_off, norm_weight.data_ptr(), float(eps),
            table.data_ptr(), table.shape[0], input_pos.data_ptr(), int(input_pos.dtype == torch.int64), qn.data_ptr(),
            qn_pitch[0], qn_pitch[1], qr.data_ptr(), qr_pitch[0], qr_pitch[1], cache.data_ptr(), cache.shape[1], B, S, heads,
            dim, rot_dim, rank, _C.stream_handle()))

    @staticmethod
    def latent_window(cache, rank, rot_dim, input_pos, B, history, rows, latent, k_rot):
        _C.require_cuda(cache, input_pos, latent, k_rot)
        _C.check(_C.lib.lri_latent_window(_C.dtype_code_any(cache.dtype), cache.data_ptr(), cache.shape[1], rank, rot_dim,
                                          input_pos.data_ptr(), int(input_pos.dtype == torch.int64), B, history, rows,
                                          latent.data_ptr(), k_rot.data_ptr(), _C.stream_handle()))

    @staticmethod
    def head_linear(x, x_pitch, w, transposed, y, y_pitch, rows, heads, n_in, n_out):
        """y[row, head] = W[head] x[row, head]; pitches are (row, head) in elements."""
        _C.require_cuda(x, w, y)
        _C.check(_C.lib.lri_head_linear(_C.dtype_code_any(w.dtype), x.data_ptr(), x_pitch[0], x_pitch[1], w.data_ptr(),
                                        int(transposed), y.data_ptr(), y_pitch[0], y_pitch[1], rows, heads, n_in, n_out,
                                        _C.stream_handle()))

    @staticmethod
    def window_attention(q, q_pitch, k, k_pitch, k2, k2_pitch, v, v_pitch, out, input_pos, history, k_rows, window, scale, B,
                         S, heads, d1, d2, dv, scratch=None):
        """q_pitch (row, head); k_pitch, v_pitch (batch, row, head); k2_pitch (batch, row), in elements."""
        _C.require_cuda(q, k, k2, v, out, input_pos)
        _C.check(_C.lib.lri_window_attention(
            _C.dtype_code_any(q.dtype), q.data_ptr(), *q_pitch, k.data_ptr(), *k_pitch, k2.data_ptr(), *k2_pitch,
            v.data_ptr(), *v_pitch, out.data_ptr(), input_pos.data_ptr(), int(input_pos.dtype == torch.int64), history,
            k_rows, window, float(scale), B, S, heads, d1, d2, dv, _C.ptr(scratch),
            scratch.numel() * scratch.element_size() if scratch is not None else 0, _C.stream_handle()))

    @staticmethod
    def window_attention_scratch_bytes(B, heads, dv, keys):
        return _C.lib.lri_window_attention_scratch_bytes(B, heads, dv, keys)

    # ---- recurrence ----------------------------------------------------------------------------------------
    @staticmethod
    def hgrn2_workspace_bytes(dtype, B, S, heads, dim, vdim):
        return _C.lib.lri_hgrn2_workspace_bytes(_C.dtype_code_any(dtype), B, S, heads, dim, vdim)

    @staticmethod
    def hgrn2(proj, ld, q_off, f_off, v_off, f_bias, lower, norm_weight, eps, state, input_pos, out, B, S, heads, dim, vdim,
              workspace):
        _C.require_cuda(proj, f_bias, lower, norm_weight, state, input_pos, out, workspace)
        _C.check(_C.lib.lri_hgrn2(
            _C.dtype_code_any(out.dtype), proj.data_ptr(), ld, q_off, f_off, v_off, f_bias.data_ptr(), lower.data_ptr(),
            norm_weight.data_ptr(), float(eps), state.data_ptr(), input_pos.data_ptr(), int(input_pos.dtype == torch.int64),
            out.data_ptr(), B, S, heads, dim, vdim, workspace.data_ptr(), workspace.numel() * workspace.element_size(),
            _C.stream_handle()))

    # ---- mixture of experts -----------------------------------------------------------------------------------
    @staticmethod
    def moe_packs(dtype, rows, top, dim, ff):
        return bool(_C.lib.lri_moe_packs(_C.dtype_code_any(dtype), rows, top, dim, ff))

    @staticmethod
    def moe_max_tiles(rows, top, experts):
        return _C.lib.lri_moe_max_tiles(rows, top, experts)

    @staticmethod
    def moe_route(logits, ld, experts, top, rows, ids, scores, counts=None, rank=None):
        _C.require_cuda(logits, ids, scores)
        _C.check(_C.lib.lri_moe_route(logits.data_ptr(), ld, experts, top, rows, ids.data_ptr(), scores.data_ptr(),
                                      _C.ptr(counts), _C.ptr(rank), _C.stream_handle()))

    @staticmethod
    def moe_pack(x, rows, top, experts, ids, scores, rank, counts, first_row, tiles, max_tiles, packed, row_scale, slots):
        _C.require_cuda(x, packed)
        _C.check(_C.lib.lri_moe_pack(_C.dtype_code(x.dtype), x.data_ptr(), rows, x.shape[-1], top, experts, ids.data_ptr(),
                                     scores.data_ptr(), rank.data_ptr(), counts.data_ptr(), first_row.data_ptr(),
                                     tiles.data_ptr(), max_tiles, packed.data_ptr(), row_scale.data_ptr(), slots.data_ptr(),
                                     _C.stream_handle()))

    @staticmethod
    def moe_gateup(x, w1, hidden, ids, scores, pairs, top, glu, tiles=None, row_scale=None, max_tiles=0):
        """w1 [experts, 2 ff, dim]; glu = (alpha, limit, offset); with `tiles` x and hidden are packed rows."""
        _C.require_cuda(x, w1, hidden)
        experts, two_ff, dim = w1.shape
        _C.check(_C.lib.lri_moe_gateup(_C.dtype_code_any(x.dtype), x.data_ptr(), w1.data_ptr(), hidden.data_ptr(), _C.ptr(ids),
                                       _C.ptr(scores), pairs, top, _C.ptr(tiles), _C.ptr(row_scale), max_tiles, experts,
                                       two_ff // 2, dim, *[float(g) for g in glu], _C.stream_handle()))

    @staticmethod
    def moe_down(hidden, w2, y, ids, pairs, tiles=None, max_tiles=0):
        _C.require_cuda(hidden, w2, y)
        experts, dim, ff = w2.shape
        _C.check(_C.lib.lri_moe_down(_C.dtype_code_any(hidden.dtype), hidden.data_ptr(), w2.data_ptr(), y.data_ptr(),
                                     _C.ptr(ids), pairs, _C.ptr(tiles), max_tiles, experts, dim, ff, _C.stream_handle()))

    # ---- residual held as several streams ------------------------------------------------------------------
    @staticmethod
    def embed_streams(table, idx, scale, streams, in_next, weight, eps, normed):
        """Every stream of `streams` [rows, n, dim] = scale * table row; normed = norm of their sum weighted by in_next."""
        _C.require_cuda(table, idx, streams, in_next, weight, normed)
        if idx.dtype not in (torch.int32, torch.int64):
            idx = idx.to(torch.int64)
        idx = idx.contiguous()
        _C.check(_C.lib.lri_embed_streams(_C.dtype_code_any(table.dtype), table.data_ptr(), idx.data_ptr(),
                                          int(idx.dtype == torch.int64), table.shape[0], float(scale), streams.data_ptr(),
                                          _C.ptr(in_next), weight.data_ptr(), float(eps), normed.data_ptr(), idx.numel(),
                                          streams.shape[1], table.shape[1], _C.stream_handle()))

    @staticmethod
    def join_streams(streams, y, mix, out, in_next, weight, eps, normed, rows, write=True):
        """streams [.., n, dim] <- mix of the old ones + out * y (write=False: not stored); normed = norm of the sum weighted
        by in_next (None: plain sum)."""
        _C.require_cuda(streams, y, mix, out, in_next, weight, normed)
        _C.check(_C.lib.lri_join_streams(_C.dtype_code_any(y.dtype), streams.data_ptr(), y.data_ptr(), mix.data_ptr(),
                                         out.data_ptr(), streams.data_ptr() if write else None, _C.ptr(in_next), weight.data_ptr(),
                                         float(eps), normed.data_ptr(), rows, streams.shape[1], streams.shape[2],
                                         _C.stream_handle()))

    # ---- gate/up with the clamped unit -----------------------------------------------------------------------
    @staticmethod
    def gateup_glu_workspace_bytes(dtype, rows, inter, k):
        return _C.lib.lri_gateup_glu_workspace_bytes(_C.dtype_code_any(dtype), rows, inter, k)

    @staticmethod
    def gateup_glu(x, w1, h, rows, glu, workspace=None):
        """w1 [2 ff, dim] = [up | gate]; glu = (alpha, limit, offset)."""
        _C.require_cuda(x, w1, h)
        two_i, k = w1.shape
        ws_ptr, ws_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) if workspace is not None else (None, 0)
        _C.check(_C.lib.lri_gateup_glu(_C.dtype_code_any(x.dtype), x.data_ptr(), w1.data_ptr(), h.data_ptr(), rows, two_i // 2, k,
                                       *[float(g) for g in glu], ws_ptr, ws_bytes, _C.stream_handle()))

    # ---- grouped attention on a cache ------------------------------------------------------------------------
    @staticmethod
    def row_squares(x, ld, off1, n1, off2, n2, sums, rows):
        _C.require_cuda(x, sums)
        _C.check(_C.lib.lri_row_squares(x.data_ptr(), ld, off1, n1, off2, n2, sums.data_ptr(), rows, _C.stream_handle()))

    @staticmethod
    def grouped_prepare(proj, ld, offs, q_norm, k_norm, sums, widths, eps, table, rot_dims, input_pos, q, k_cache, v_cache, B, S,
                        n_head):
        """offs: columns of q, k, v in proj; widths: elements that the norms of q and k run over; sums: their sums of
        squares where other ranks hold a part."""
        _C.require_cuda(proj, q_norm, k_norm, sums, table, input_pos, q, k_cache, v_cache)
        _, n_kv, smax, dim = k_cache.shape
        _C.check(_C.lib.lri_grouped_prepare(
            _C.dtype_code_any(k_cache.dtype), proj.data_ptr(), ld, *offs, q_norm.data_ptr(), k_norm.data_ptr(), _C.ptr(sums), *widths,
            float(eps), table.data_ptr(), table.shape[0], rot_dims, input_pos.data_ptr(), int(input_pos.dtype == torch.int64),
            q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), smax, B, S, n_head, n_kv, dim, v_cache.shape[3],
            _C.stream_handle()))

    @staticmethod
    def grouped_attention(q, k_cache, v_cache, sink, out, out_ld, out_scale, input_pos, window, chunk, scale, B, S, n_head):
        """window, chunk: 0 for none; sink: a logit per head or None; out starts at the first column to write."""
        _C.require_cuda(q, k_cache, v_cache, sink, out, input_pos)
        _, n_kv, smax, dim = k_cache.shape
        _C.check(_C.lib.lri_grouped_attention(
            _C.dtype_code_any(q.dtype), q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), _C.ptr(sink), out.data_ptr(), out_ld,
            float(out_scale), input_pos.data_ptr(), int(input_pos.dtype == torch.int64), smax, window, chunk, float(scale), B, S,
            n_head, n_kv, dim, v_cache.shape[3], _C.stream_handle()))

    # ---- matrix-state recurrences ------------------------------------------------------------------------------
    # blocks = (qd, kd, ku, decay, coef): vectors and coefficients of blocks of four tokens, fp32 (kd unused without the
    # delta rule)
    @staticmethod
    def state_blocks(S):
        return _C.lib.lri_state_blocks(S)

    @staticmethod
    def delta_blocks(proj, ld, offs, convs, ring, z, a_log, dt_bias, input_pos, blocks, v, B, S, heads, kv_heads, dim, vdim):
        """offs: columns of q, k, v, b; convs: [channels, taps] of q, k, v; z: the decays' projection."""
        _C.require_cuda(proj, *convs, ring, z, a_log, dt_bias, input_pos, *blocks, v)
        _C.check(_C.lib.lri_delta_blocks(
            _C.dtype_code_any(a_log.dtype), proj.data_ptr(), ld, *offs, *[c.data_ptr() for c in convs], convs[0].shape[1],
            ring.data_ptr(), z.data_ptr(), a_log.data_ptr(), dt_bias.data_ptr(), input_pos.data_ptr(),
            int(input_pos.dtype == torch.int64), *[x.data_ptr() for x in blocks], v.data_ptr(), B, S, heads, kv_heads, dim, vdim,
            _C.stream_handle()))

    @staticmethod
    def gla_blocks(proj, ld, offs, z, bias, tau, blocks, B, S, heads, dim):
        """offs: columns of q, k."""
        qd, _, ku, decay, coef = blocks
        _C.require_cuda(proj, z, bias, qd, ku, decay, coef)
        _C.check(_C.lib.lri_gla_blocks(_C.dtype_code_any(bias.dtype), proj.data_ptr(), ld, *offs, z.data_ptr(), bias.data_ptr(),
                                       float(tau), qd.data_ptr(), ku.data_ptr(), decay.data_ptr(), coef.data_ptr(), B, S, heads, dim,
                                       _C.stream_handle()))

    @staticmethod
    def state_scan(blocks, delta, v, v_row, state, input_pos, o, B, S):
        """v starts at its first column."""
        _C.require_cuda(*[x for x in blocks if x is not None], v, state, input_pos, o)
        qd, kd, ku, decay, coef = blocks
        _, heads, dim, vdim = state.shape
        _C.check(_C.lib.lri_state_scan(qd.data_ptr(), kd.data_ptr() if delta else None, ku.data_ptr(), decay.data_ptr(),
                                       coef.data_ptr(), v.data_ptr(), v_row, state.data_ptr(), input_pos.data_ptr(),
                                       int(input_pos.dtype == torch.int64), o.data_ptr(), B, S, heads, dim, vdim,
                                       _C.stream_handle()))

    @staticmethod
    def state_step_supports(dim, vdim, decay_rank, gate_rank):
        return bool(_C.lib.lri_state_step_supports(dim, vdim, decay_rank, gate_rank))

    @staticmethod
    def delta_step(proj, ld, offs, convs, ring, a2, g2, a_log, dt_bias, norm, eps, factor, state, input_pos, out, out_ld, B, kv_heads):
        """offs: columns of q, k, v, a1, g1, b; out starts at the first column to write."""
        _C.require_cuda(proj, *convs, ring, a2, g2, a_log, dt_bias, norm, state, input_pos, out)
        _, heads, dim, vdim = state.shape
        _C.check(_C.lib.lri_delta_step(
            _C.dtype_code_any(out.dtype), proj.data_ptr(), ld, *offs, *[c.data_ptr() for c in convs], convs[0].shape[1], ring.data_ptr(),
            a2.data_ptr(), a2.shape[1], g2.data_ptr(), g2.shape[1], a_log.data_ptr(), dt_bias.data_ptr(), norm.data_ptr(), float(eps),
            float(factor), state.data_ptr(), input_pos.data_ptr(), int(input_pos.dtype == torch.int64), out.data_ptr(), out_ld, B,
            heads, kv_heads, dim, vdim, _C.stream_handle()))

    @staticmethod
    def gla_step(proj, ld, offs, a2, bias, tau, norm, eps, factor, state, input_pos, out, out_ld, B):
        """offs: columns of q, k, v, a1, g."""
        _C.require_cuda(proj, a2, bias, norm, state, input_pos, out)
        _, heads, dim, vdim = state.shape
        _C.check(_C.lib.lri_gla_step(
            _C.dtype_code_any(out.dtype), proj.data_ptr(), ld, *offs, a2.data_ptr(), a2.shape[1], bias.data_ptr(), float(tau),
            norm.data_ptr(), float(eps), float(factor), state.data_ptr(), input_pos.data_ptr(), int(input_pos.dtype == torch.int64),
            out.data_ptr(), out_ld, B, heads, dim, vdim, _C.stream_handle()))

    @staticmethod
    def head_norm_gate(o, norm_weight, eps, gate, gate_ld, activation, scale, out, out_ld, rows, heads):
        """activation: "sigmoid" or "silu" of the gate; gate and out start at their first column."""
        _C.require_cuda(o, norm_weight, gate, out)
        act = {"sigmoid": _C.GATE_SIGMOID, "silu": _C.GATE_SILU}[activation]
        _C.check(_C.lib.lri_head_norm_gate(_C.dtype_code_any(out.dtype), o.data_ptr(), norm_weight.data_ptr(), float(eps),
                                           gate.data_ptr(), gate_ld, act, float(scale), out.data_ptr(), out_ld, rows, heads,
                                           norm_weight.numel(), _C.stream_handle()))

    @staticmethod
    def round_columns(x, ld, off, n, y, rows):
        _C.require_cuda(x, y)
        _C.check(_C.lib.lri_round_columns(_C.dtype_code_any(y.dtype), x.data_ptr(), ld, off, n, y.data_ptr(), rows, _C.stream_handle()))


def decode_splits(B, n_head, n_kv, smax, head_dim=128):
    """Number of sequence ranges for decode attention, fixed per cache geometry so that the launch
    grid never depends on the current position.  The rule lives in the library
    (lri_attn_decode_plan), next to the choice of the kernel it has to agree with."""
    n = ctypes.c_int(0)
    _C.check(_C.lib.lri_attn_decode_plan(B, n_head, n_kv, head_dim, smax, ctypes.byref(n)))
    return n.value
