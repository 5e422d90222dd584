"""Whole-model forward of designs given as a list of layers (token mixer + feed-forward, each in a gated, doubly
normed residual branch) on preallocated buffers.

The heads (logits, last position, greedy, sampling), the tensor-parallel plumbing and the calling conventions are
`engine.Engine`'s; what differs is the body between embedding and final norm:

    h        = norm(x)                                             first one fused with the embedding
    gate|in  = in_proj(h)                                          fp32, one projection per sublayer
    y        = mixer(in)  or  experts(h, router logits in `in`)
    x, h     = x + post_norm(sigmoid(gate + bias) * y), next norm  one fused pass over the fp32 residual

A forward reads positions from the device and can be captured in a CUDA graph.  A batch row's first position decides
whether a recurrence starts anew (0) or continues, so a row is reused by feeding position 0 again.
"""
import torch

from .engine import Engine
from .mixers import LatentAttention


class LayerEngine(Engine):
    def setup(self, max_batch, max_seq, device, dtype):
        cfg = self.cfg
        self.d, self.dtype = cfg.dim, dtype
        self.max_batch, self.max_seq = max_batch, max_seq
        rows = self.max_rows = max_batch * max_seq
        ops = self.ops

        def buf(n, cols, dt=dtype):
            return torch.empty(n, cols, dtype=dt, device=device)

        mixers = [b.mixer.sublayer for b in self.model.layers]
        latent = [m for m in mixers if m.kind == "latent_attention"]
        hgrn = [m for m in mixers if m.kind == "hgrn2"]
        moes = [b.mlp.sublayer for b in self.model.layers if b.mlp is not None]
        branches = [b.mixer for b in self.model.layers] + [b.mlp for b in self.model.layers if b.mlp is not None]

        self.resid = buf(rows, self.d, torch.float32)
        self.normed, self.part = buf(rows, self.d), buf(rows, self.d)
        self.proj = buf(rows, max(br.in_proj.weight.shape[0] for br in branches), torch.float32)
        self.y = buf(rows, max(m.out_width for m in mixers))

        def workspace(size_fn, n):
            size = max(size_fn(rows, n), size_fn(min(rows, 64), n))
            return torch.empty(size, dtype=torch.uint8, device=device) if size else None

        self.ws_in = workspace(ops.linear_f32_workspace_bytes, self.proj.shape[1])
        self.ws_out = workspace(ops.linear_workspace_bytes, self.d)

        if latent:
            self.q = buf(rows, max(m.q_rows for m in latent))
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
        if hgrn:
            size = max(ops.hgrn2_workspace_bytes(dtype, b, max_seq, m.heads, m.dim, m.vdim)
                       for m in hgrn for b in range(1, max_batch + 1))
            self.ws_hgrn = torch.empty(max(size, 16), dtype=torch.uint8, device=device)
        if moes:
            def most(f):
                return max(f(m) for m in moes)

            def ints(n):
                return torch.zeros(n, dtype=torch.int32, device=device)

            pairs = rows * most(lambda m: m.top)
            tiles = most(lambda m: ops.moe_max_tiles(rows, m.top, m.experts))
            packed = any(ops.moe_packs(dtype, rows, m.top, self.d, m.ff) for m in moes)
            out_rows = max(pairs, 128 * tiles) if packed else pairs
            self.moe_ids, self.moe_rank, self.moe_slots = ints(pairs), ints(pairs), ints(pairs)
            self.moe_scores = torch.empty(pairs, dtype=torch.float32, device=device)
            self.moe_counts, self.moe_first = ints(most(lambda m: m.experts)), ints(most(lambda m: m.experts))
            self.moe_tiles = ints(1 + tiles)
            self.moe_hidden = buf(out_rows, most(lambda m: m.ff))
            self.moe_out = buf(out_rows, self.d)
            if packed:
                self.moe_packed = buf(128 * tiles, self.d)
                self.moe_scale = torch.zeros(128 * tiles, dtype=torch.float32, device=device)
        self._setup_head(max_batch, device, dtype)
        self.ready = True

    # ------------------------------------------------------------------------------------------
    def _latent_attention(self, m: LatentAttention, rows, B, S, pos, eps):
        ops, cache = self.ops, m.kv_cache.rows
        H, dn, dr, dv, r, ld = m.heads, m.dim, m.rot_dim, m.vdim, m.rank, self.ld
        q_off = self.d
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
        q_off = self.d
        f_off = q_off + m.heads * m.dim
        self.ops.hgrn2(self.proj, self.ld, q_off, f_off, f_off + m.heads * m.dim, m.f_bias, m.lower, m.norm, eps,
                       m.kv_cache.state, pos, self.y, B, S, m.heads, m.dim, m.vdim, self.ws_hgrn)

    def _experts(self, m, rows):
        """Returns (result rows, slots, number of result rows): the row of each (token, choice) pair in self.moe_out."""
        ops, pairs = self.ops, rows * m.top
        logits = self.proj.view(-1)[self.d:]
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

    def _join(self, branch, y, rows, next_norm, n_slots=1, slots=None, y_rows=None):
        """x += post_norm(gate * sum of y's slots); normed = norm of x for the next sublayer (or the head)."""
        if self.comm.world > 1:
            # ranks hold partial sums of y: add the slots, then the ranks
            if n_slots > 1 or slots is not None:
                self.ops.sum_slots(y, rows, n_slots, slots, y_rows, self.part)
                y, n_slots, slots, y_rows = self.part, 1, None, None
            self.comm.all_reduce(y, rows)
        self.ops.gated_norm_add(self.resid, y, self.proj, self.ld, branch.gate_bias, branch.post_norm, self.cfg.norm_eps,
                                next_norm, self.normed, rows, n_slots=n_slots, slots=slots, y_rows=y_rows)

    def _in_proj(self, branch, rows):
        self.ld = branch.in_proj.weight.shape[0]
        self.ops.linear_f32(self.normed, branch.in_proj.weight, self.proj, rows, workspace=self.ws_in)

    def _body(self, idx, rows, B, S, pos):
        m, eps, ops = self.model, self.cfg.norm_eps, self.ops
        norms = []  # the norm each sublayer's join prepares
        for block in m.layers:
            norms += [block.mixer.pre_norm] + ([block.mlp.pre_norm] if block.mlp is not None else [])
        norms.append(m.norm.weight)
        n = 0
        ops.embed_norm(m.tok_embeddings.weight, idx, self.resid, norms[0], eps, self.normed)
        for block in m.layers:
            n += 1
            mixer = block.mixer.sublayer
            self._in_proj(block.mixer, rows)
            (self._latent_attention if mixer.kind == "latent_attention" else self._hgrn2)(mixer, rows, B, S, pos, eps)
            ops.linear(self.y, mixer.wo.weight, self.part, rows, workspace=self.ws_out)
            self._join(block.mixer, self.part, rows, norms[n])
            if block.mlp is not None:
                n += 1
                self._in_proj(block.mlp, rows)
                moe = block.mlp.sublayer
                slots, y_rows = self._experts(moe, rows)
                self._join(block.mlp, self.moe_out, rows, norms[n], moe.top, slots, y_rows)
