"""Whole-model forward of designs given as a list of layers (token mixer + feed-forward) on preallocated buffers.

The heads (logits, last position, greedy, sampling), the tensor-parallel plumbing and the calling conventions are
`engine.Engine`'s; what differs is the body between embedding and final norm.  Every sublayer is

    h      = norm(residual)                           prepared by the step before it
    in     = in_proj(h)                               fp32, one projection per sublayer (none for a dense gated unit)
    y      = sublayer(in or h)
    join   the result enters the fp32 residual and the next sublayer's norm is taken, in one fused pass

and there are two kinds of residual: one stream with a gate and a post norm on the result (`GatedResidual`), or several
streams that a sublayer mixes (`StreamBranch`).

A forward reads positions from the device and can be captured in a CUDA graph.  A batch row's first position decides
whether a recurrence starts anew (0) or continues, so a row is reused by feeding position 0 again.
"""
import os

import torch
import torch.distributed as dist

from .engine import Engine
from .mixers import LatentAttention, StreamBranch, _offsets


class LayerEngine(Engine):
    def setup(self, max_batch, max_seq, device, dtype):
        cfg = self.cfg
        self.d, self.dtype = cfg.dim, dtype
        self.max_batch, self.max_seq = max_batch, max_seq
        rows = self.max_rows = max_batch * max_seq
        ops = self.ops

        def buf(n, cols, dt=dtype):
            return torch.empty(n, cols, dtype=dt, device=device)

        branches = self.branches = [br for b in self.model.layers for br in (b.mixer, b.mlp) if br is not None]
        subs = [m for br in branches for m in ((br.sublayer.left, br.sublayer.right) if br.sublayer.kind == "parallel" else (br.sublayer,))]
        mixers = [b.mixer.sublayer for b in self.model.layers]

        def of(kind):
            return [m for m in subs if m.kind == kind]

        def most(ms, f):
            return max((f(m) for m in ms), default=0)

        streams = getattr(cfg, "streams", None)
        self.resid = torch.empty(rows, self.d, dtype=torch.float32, device=device) if streams is None else \
            torch.empty(rows, streams, self.d, dtype=torch.float32, device=device)
        self.normed, self.part = buf(rows, self.d), buf(rows, self.d)
        in_rows = [br.in_proj.weight.shape[0] for br in branches if br.in_proj is not None]
        self.proj = buf(rows, max(in_rows, default=1), torch.float32)
        self.y = buf(rows, max(m.out_width for m in mixers))

        def workspace(size_fn, *ns):
            size = max((max(size_fn(rows, n), size_fn(min(rows, 64), n)) for n in ns), default=0)
            return torch.empty(size, dtype=torch.uint8, device=device) if size else None

        self.ws_in = workspace(ops.linear_f32_workspace_bytes, *in_rows)
        self.ws_out = workspace(ops.linear_workspace_bytes, self.d)

        latent, hgrn, moes, glus = of("latent_attention"), of("hgrn2"), of("moe"), of("glu")
        grouped, delta, gla = of("chunked_attention"), of("gated_delta"), of("gla")
        if latent or grouped:
            self.q = buf(rows, max(most(latent, lambda m: m.q_rows), most(grouped, lambda m: m.heads * m.dim)))
        if latent:
            self.q_latent = buf(max_batch, max(m.heads * (m.rank + m.rot_dim) for m in latent))
            self.o_latent = buf(max_batch, max(m.heads * m.rank for m in latent))
            # what a prompt portion sees (history + its own tokens) never exceeds the cache
            self.win_latent = buf(rows, max(m.rank for m in latent))
            self.win_rot = buf(rows, max(m.rot_dim for m in latent))
            self.win_kv = buf(rows, max(m.heads * (m.dim + m.vdim) for m in latent))
            # fewer sequences are cut into more splits: the largest batch is not the largest scratch
            size = max(ops.window_attention_scratch_bytes(b, m.heads, m.rank, min(m.window, max_seq))
                       for m in latent for b in range(1, max_batch + 1))
            self.attn_scratch = torch.empty(max(size, 16), dtype=torch.uint8, device=device)
            self.ws_expand = workspace(ops.linear_workspace_bytes, self.win_kv.shape[1])
        if grouped and self.comm.world > 1:
            self.qk_sums = buf(rows, 2, torch.float32)
        if hgrn:
            size = max(ops.hgrn2_workspace_bytes(dtype, b, max_seq, m.heads, m.dim, m.vdim)
                       for m in hgrn for b in range(1, max_batch + 1))
            self.ws_hgrn = torch.empty(max(size, 16), dtype=torch.uint8, device=device)
        if delta or gla:
            scans = delta + gla
            self.low = buf(rows, max(most(scans, lambda m: m.a2.shape[1]), most(delta, lambda m: m.g2.shape[1])))
            hc = most(scans, lambda m: m.heads * m.dim)
            self.scan_z, self.scan_o = buf(rows, hc, torch.float32), buf(rows, most(scans, lambda m: m.out_width), torch.float32)
            # every sequence's tokens are cut in blocks from the call's first on
            blocks = max(b * ops.state_blocks(max_seq) for b in (1, max_batch))
            vectors = buf(4 * blocks, hc, torch.float32), buf(4 * blocks if delta else 0, hc, torch.float32), buf(4 * blocks, hc, torch.float32)
            self.scan_blocks = vectors + (buf(blocks, hc, torch.float32), buf(blocks, 32 * most(scans, lambda m: m.heads), torch.float32))
            self.ws_low = workspace(ops.linear_f32_workspace_bytes, *[m.a2.shape[0] for m in scans], *[m.g2.shape[0] for m in delta])
        if delta:
            self.scan_v = buf(rows, most(delta, lambda m: m.out_width), torch.float32)
            self.scan_gate = buf(rows, most(delta, lambda m: m.out_width), torch.float32)
        if glus:
            self.glu_hidden = buf(rows, most(glus, lambda m: m.ff))
            self.ws_glu = workspace(lambda n, m: ops.gateup_glu_workspace_bytes(dtype, n, m.ff, self.d), *glus)
        if moes:
            def ints(n):
                return torch.zeros(n, dtype=torch.int32, device=device)

            pairs = rows * most(moes, lambda m: m.top)
            tiles = most(moes, lambda m: ops.moe_max_tiles(rows, m.top, m.experts))
            packed = any(ops.moe_packs(dtype, rows, m.top, self.d, m.ff) for m in moes)
            out_rows = max(pairs, 128 * tiles) if packed else pairs
            self.moe_ids, self.moe_rank, self.moe_slots = ints(pairs), ints(pairs), ints(pairs)
            self.moe_scores = torch.empty(pairs, dtype=torch.float32, device=device)
            self.moe_counts, self.moe_first = ints(most(moes, lambda m: m.experts)), ints(most(moes, lambda m: m.experts))
            self.moe_tiles = ints(1 + tiles)
            self.moe_hidden = buf(out_rows, most(moes, lambda m: m.ff))
            self.moe_out = buf(out_rows, self.d)
            if packed:
                self.moe_packed = buf(128 * tiles, self.d)
                self.moe_scale = torch.zeros(128 * tiles, dtype=torch.float32, device=device)
        self.side_stream = None
        if of("chunked_attention") and self.comm.world == 1 and self.resid.is_cuda and os.environ.get("LRI_SIDE_STREAM", "1") != "0":
            self.side_stream = torch.cuda.Stream()
            self._fork, self._join_event = torch.cuda.Event(), torch.cuda.Event()
        self._setup_head(max_batch, device, dtype)
        self.ready = True

    # ------------------------------------------------------------------------------------------
    # Mixers leave the rows that their output projection reads in self.y.
    def _latent_attention(self, m: LatentAttention, rows, B, S, pos, eps):
        ops, cache = self.ops, m.kv_cache.rows
        H, dn, dr, dv, r, ld = m.heads, m.dim, m.rot_dim, m.vdim, m.rank, self.ld
        q_off = self.off
        kv_off = q_off + m.q_rows
        smax, row_len = cache.shape[1], r + dr
        w_k, w_v = m.expand.weight[: H * dn], m.expand.weight[H * dn:]
        if S == 1:
            # scores and weighted sums on the cached latents: q^T W_uk, attention, W_uv o
            ql = self.q_latent.view(-1)[: B * H * row_len]
            ol = self.o_latent.view(-1)[: B * H * r]
            ops.latent_prepare(self.proj, ld, q_off, kv_off, m.latent_norm, eps, m.rope_table, pos, self.q, (H * dn, dn),
                               ql[r:], (H * row_len, row_len), cache, B, S, H, dn, dr, r)
            ops.head_linear(self.q, (H * dn, dn), w_k, True, ql, (H * row_len, row_len), B, H, dn, r)
            ops.window_attention(ql, (H * row_len, row_len), cache, (smax * row_len, row_len, 0), cache.view(-1)[r:],
                                 (smax * row_len, row_len), cache, (smax * row_len, row_len, 0), ol, pos, -1, smax,
                                 m.window, m.scale, B, 1, H, r, dr, r, self.attn_scratch)
            ops.head_linear(ol, (H * r, r), w_v, False, self.y, (H * dv, dv), B, H, r, dv)
            return
        # prompt portion: the visible latents are expanded to per-head keys and values
        history = min(m.window - 1, smax - S)
        n = history + S
        kv = self.win_kv.view(-1)[: B * n * H * (dn + dv)]
        ld_kv = H * (dn + dv)
        ops.latent_prepare(self.proj, ld, q_off, kv_off, m.latent_norm, eps, m.rope_table, pos, self.q,
                           (H * (dn + dr), dn + dr), self.q.view(-1)[dn:], (H * (dn + dr), dn + dr), cache, B, S, H, dn, dr, r)
        ops.latent_window(cache, r, dr, pos, B, history, n, self.win_latent, self.win_rot)
        ops.linear(self.win_latent, m.expand.weight, kv, B * n, workspace=self.ws_expand)
        ops.window_attention(self.q, (H * (dn + dr), dn + dr), kv, (n * ld_kv, ld_kv, dn), self.win_rot, (n * dr, dr),
                             kv[H * dn:], (n * ld_kv, ld_kv, dv), self.y, pos, history, n, m.window, m.scale, B, S, H, dn, dr, dv)

    def _hgrn2(self, m, rows, B, S, pos, eps):
        q_off = self.off
        f_off = q_off + m.heads * m.dim
        self.ops.hgrn2(self.proj, self.ld, q_off, f_off, f_off + m.heads * m.dim, m.f_bias, m.lower, m.norm, eps,
                       m.kv_cache.state, pos, self.y, B, S, m.heads, m.dim, m.vdim, self.ws_hgrn)

    def _low_rank(self, off, w, out, rows):
        """out (fp32) = w x, x the columns of the input projection from `off` on, in the storage type."""
        self.ops.round_columns(self.proj, self.ld, off, w.shape[1], self.low, rows)
        self.ops.linear_f32(self.low, w, out, rows, workspace=self.ws_low)

    def _gla(self, m, rows, B, S, pos, eps):
        ops, at, proj = self.ops, _offsets(m.parts(), self.off), self.proj.view(-1)
        if S == 1 and ops.state_step_supports(m.dim, m.vdim, m.a2.shape[1], 0):
            ops.gla_step(self.proj, self.ld, [at[k] for k in ("q", "k", "v", "a1", "g")], m.a2, m.a2_bias, m.tau, m.norm, eps, 1.0,
                         m.kv_cache.state, pos, self.y, m.out_width, B)
            return
        self._low_rank(at["a1"], m.a2, self.scan_z, rows)
        ops.gla_blocks(self.proj, self.ld, (at["q"], at["k"]), self.scan_z, m.a2_bias, m.tau, self.scan_blocks, B, S, m.heads, m.dim)
        ops.state_scan(self.scan_blocks, False, proj[at["v"]:], self.ld, m.kv_cache.state, pos, self.scan_o, B, S)
        ops.head_norm_gate(self.scan_o, m.norm, eps, proj[at["g"]:], self.ld, "silu", 1.0, self.y, m.out_width, rows, m.heads)

    def _grouped(self, m, at, y, y_ld, factor, rows, B, S, pos, eps):
        ops, sums = self.ops, None
        if self.comm.world > 1:  # the norms run over the heads of all ranks
            sums = self.qk_sums
            ops.row_squares(self.proj, self.ld, at["q"], m.heads * m.dim, at["k"], m.kv_heads * m.dim, sums, rows)
            dist.all_reduce(sums[:rows])
        kc, vc = m.kv_cache.k_cache, m.kv_cache.v_cache
        ops.grouped_prepare(self.proj, self.ld, (at["q"], at["k"], at["v"]), m.q_norm, m.k_norm, sums, m.norm_widths, eps,
                            m.rope_table, m.rot_dims, pos, self.q, kc, vc, B, S, m.heads)
        ops.grouped_attention(self.q, kc, vc, m.sink, y, y_ld, factor, pos, m.window, m.chunk, m.scale, B, S, m.heads)

    def _gated_delta(self, m, at, y, y_ld, factor, rows, B, S, pos, eps):
        ops, convs, ring = self.ops, (m.conv_q, m.conv_k, m.conv_v), m.conv_state.ring
        if S == 1 and ops.state_step_supports(m.dim, m.vdim, m.a2.shape[1], m.g2.shape[1]):
            ops.delta_step(self.proj, self.ld, [at[k] for k in ("q", "k", "v", "a1", "g1", "b")], convs, ring, m.a2, m.g2, m.a_log,
                           m.dt_bias, m.norm, eps, factor, m.kv_cache.state, pos, y, y_ld, B, m.kv_heads)
            return
        self._low_rank(at["a1"], m.a2, self.scan_z, rows)
        self._low_rank(at["g1"], m.g2, self.scan_gate, rows)
        v = m.out_width
        ops.delta_blocks(self.proj, self.ld, (at["q"], at["k"], at["v"], at["b"]), convs, ring, self.scan_z, m.a_log, m.dt_bias,
                         pos, self.scan_blocks, self.scan_v, B, S, m.heads, m.kv_heads, m.dim, m.vdim)
        ops.state_scan(self.scan_blocks, True, self.scan_v, v, m.kv_cache.state, pos, self.scan_o, B, S)
        ops.head_norm_gate(self.scan_o, m.norm, eps, self.scan_gate, v, "sigmoid", factor, y, y_ld, rows, m.heads)

    def _parallel(self, m, rows, B, S, pos, eps):
        """The sides read the same projections and write their own columns of y; on one GPU they run on two streams."""
        at, ld = _offsets(m.parts(), self.off), m.out_width
        y = self.y.view(-1)

        def offsets(side):
            return {k[len(side) + 1:]: v for k, v in at.items() if k.startswith(side + ".")}

        def left():
            self._grouped(m.left, offsets("left"), y, ld, m.scales[0], rows, B, S, pos, eps)

        def right():
            self._gated_delta(m.right, offsets("right"), y[m.left.out_width:], ld, m.scales[1], rows, B, S, pos, eps)

        if self.side_stream is None:
            left()
            right()
            return
        main, side = torch.cuda.current_stream(), self.side_stream
        self._fork.record(main)
        side.wait_event(self._fork)
        with torch.cuda.stream(side):
            left()
            self._join_event.record(side)
        right()
        main.wait_event(self._join_event)

    def _experts(self, m, rows):
        """Returns (result rows, slots, number of result rows): the row of each (token, choice) pair in self.moe_out."""
        ops, pairs = self.ops, rows * m.top
        logits = self.proj.view(-1)[self.off:]
        if not ops.moe_packs(self.dtype, rows, m.top, self.d, m.ff):
            ops.moe_route(logits, self.ld, m.experts, m.top, rows, self.moe_ids, self.moe_scores)
            ops.moe_gateup(self.normed, m.w1, self.moe_hidden, self.moe_ids, self.moe_scores, pairs, m.top, m.glu)
            ops.moe_down(self.moe_hidden, m.w2, self.moe_out, self.moe_ids, pairs)
            return None, pairs
        tiles = ops.moe_max_tiles(rows, m.top, m.experts)
        ops.moe_route(logits, self.ld, m.experts, m.top, rows, self.moe_ids, self.moe_scores, self.moe_counts, self.moe_rank)
        ops.moe_pack(self.normed, rows, m.top, m.experts, self.moe_ids, self.moe_scores, self.moe_rank, self.moe_counts,
                     self.moe_first, self.moe_tiles, tiles, self.moe_packed, self.moe_scale, self.moe_slots)
        ops.moe_gateup(self.moe_packed, m.w1, self.moe_hidden, None, None, pairs, m.top, m.glu, tiles=self.moe_tiles,
                       row_scale=self.moe_scale, max_tiles=tiles)
        ops.moe_down(self.moe_hidden, m.w2, self.moe_out, None, pairs, tiles=self.moe_tiles, max_tiles=tiles)
        return self.moe_slots, 128 * tiles

    def _start(self, idx, first):
        m, eps = self.model, self.cfg.norm_eps
        if isinstance(first, StreamBranch):
            self.ops.embed_streams(m.tok_embeddings.weight, idx, self.cfg.embed_scale, self.resid, first.w_in, first.pre_norm, eps,
                                   self.normed)
        else:
            self.ops.embed_norm(m.tok_embeddings.weight, idx, self.resid, first.pre_norm, eps, self.normed)

    def _join(self, branch, nxt, y, rows, n_slots=1, slots=None, y_rows=None):
        """The sublayer's result (the sum of y's slots) enters the residual; normed = norm for the next sublayer or the head."""
        ops, eps = self.ops, self.cfg.norm_eps
        weight = nxt.pre_norm if nxt is not None else self.model.norm.weight
        streams = isinstance(branch, StreamBranch)
        if (self.comm.world > 1 or streams) and (n_slots > 1 or slots is not None):
            ops.sum_slots(y, rows, n_slots, slots, y_rows, self.part)
            y, n_slots, slots, y_rows = self.part, 1, None, None
        if self.comm.world > 1:  # ranks hold partial sums of y
            self.comm.all_reduce(y, rows)
        if streams:
            ops.join_streams(self.resid, y, branch.w_mix, branch.w_out, nxt.w_in if nxt is not None else None, weight, eps,
                             self.normed, rows, write=nxt is not None)
        else:
            ops.gated_norm_add(self.resid, y, self.proj, self.ld, branch.gate_bias, branch.post_norm, eps, weight, self.normed, rows,
                               n_slots=n_slots, slots=slots, y_rows=y_rows)

    def _in_proj(self, branch, rows):
        self.off = branch.gate_rows
        if branch.in_proj is not None:
            self.ld = branch.in_proj.weight.shape[0]
            self.ops.linear_f32(self.normed, branch.in_proj.weight, self.proj, rows, workspace=self.ws_in)

    def _body(self, idx, rows, B, S, pos):
        eps, ops = self.cfg.norm_eps, self.ops
        run = {"latent_attention": self._latent_attention, "hgrn2": self._hgrn2, "gla": self._gla, "parallel": self._parallel}
        self._start(idx, self.branches[0])
        for i, branch in enumerate(self.branches):
            nxt = self.branches[i + 1] if i + 1 < len(self.branches) else None
            self._in_proj(branch, rows)
            sub = branch.sublayer
            if sub.kind == "moe":
                slots, y_rows = self._experts(sub, rows)
                self._join(branch, nxt, self.moe_out, rows, sub.top, slots, y_rows)
            elif sub.kind == "glu":
                ops.gateup_glu(self.normed, sub.w1, self.glu_hidden, rows, sub.glu, workspace=self.ws_glu)
                ops.linear(self.glu_hidden, sub.w2, self.part, rows, workspace=self.ws_out)
                self._join(branch, nxt, self.part, rows)
            else:
                run[sub.kind](sub, rows, B, S, pos, eps)
                ops.linear(self.y, sub.wo.weight, self.part, rows, workspace=self.ws_out)
                self._join(branch, nxt, self.part, rows)
