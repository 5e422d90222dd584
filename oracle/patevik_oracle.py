"""Plain, slow PyTorch-on-CPU statement of the Patevik design, one function per mechanism.

Test infrastructure: it shares no code with the package, works on whole sequences with explicit
loops and masks, and keeps no cache.  Every function takes and returns tensors of one dtype (fp32 or
fp64); weights are a dict keyed by checkpoint tensor names, `cfg` is the checkpoint's config dict.

Notation: rows of a matrix are tokens; `E(x)` is the elementwise logistic function.
"""
import math

import torch


def rms_norm(x, weight, eps):
    """x_i / sqrt(mean_j x_j^2 + eps) * weight_i over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def rotate_half_pairs(x, positions, base):
    """Rotates the pairs (i, i + n/2) of the last dimension n by positions * base^(-2 i / n).
    x [tokens, ..., n]; angles are evaluated in fp64."""
    n = x.shape[-1]
    i = torch.arange(n // 2, dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * torch.exp(-(2.0 * i / n) * math.log(base))
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [n // 2]
    c, s = torch.cos(ang).to(x.dtype).view(shape), torch.sin(ang).to(x.dtype).view(shape)
    u, v = x[..., : n // 2], x[..., n // 2:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def window_mask(n, window):
    """[n, n] bool: query i sees key j when 0 <= i - j < window."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < window)


def latent_attention(h, w, mixer, eps, prefix=""):
    """Multi-head attention whose keys and values are linear images of one normed latent per token plus a
    rotated key part shared by the heads.  h [tokens, d] -> [tokens, d]."""
    H, dn, dr, dv, r = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    n = h.shape[0]
    pos = torch.arange(n)
    q = (h @ w[prefix + "q"].T).view(n, H, dn + dr)
    down = h @ w[prefix + "dkv"].T
    lat = rms_norm(down[:, :r], w[prefix + "dkv.norm"], eps)
    k_rot = rotate_half_pairs(down[:, r:], pos, mixer["rot"]["base"])
    q_rot = rotate_half_pairs(q[..., dn:], pos, mixer["rot"]["base"])
    k = (lat @ w[prefix + "uk"].T).view(n, H, dn)
    v = (lat @ w[prefix + "uv"].T).view(n, H, dv)
    score = torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    score = (score * mixer["scale"]).masked_fill(~window_mask(n, mixer["mask"]["size"]), float("-inf"))
    out = torch.einsum("hij,jhd->ihd", torch.softmax(score, dim=-1), v)
    return out.reshape(n, H * dv) @ w[prefix + "o"].T


def hgrn2_recurrence(q, f, v, state=None):
    """state[h, c, e] <- f[h, c] state[h, c, e] + (1 - f[h, c]) v[h, e];  out[h, e] = sum_c q[h, c] state[h, c, e].
    q, f [tokens, H, C], v [tokens, H, E] -> (out [tokens, H, E], last state)."""
    n, H, C = q.shape
    st = torch.zeros(H, C, v.shape[-1], dtype=q.dtype) if state is None else state
    out = []
    for t in range(n):
        st = f[t][:, :, None] * st + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hc,hce->he", q[t], st))
    return torch.stack(out), st


def hgrn2(h, w, mixer, eps, prefix=""):
    """Linear attention whose per-channel forget gate f (bounded below) also scales what is written."""
    H, C, E = mixer["heads"], mixer["dim"], mixer["vdim"]
    n = h.shape[0]
    q = h @ w[prefix + "q"].T
    q = q * torch.sigmoid(q)
    low = w[prefix + "lower"]
    f = low + (1 - low) * torch.sigmoid(h @ w[prefix + "f"].T + w[prefix + "f.b"])
    v = h @ w[prefix + "v"].T
    o, _ = hgrn2_recurrence(q.view(n, H, C), f.view(n, H, C), v.view(n, H, E))
    o = rms_norm(o, w[prefix + "norm"], eps)
    return o.reshape(n, H * E) @ w[prefix + "o"].T


def clamped_glu(gate, up, limit):
    """g = min(gate, limit), u = clamp(up, -limit, limit);  g E(1.702 g) (u + 1)."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def route(h, router, top):
    """Logistic router: the `top` largest scores of every token, unnormalised.  -> (indices, scores) [tokens, top]."""
    score = torch.sigmoid(h @ router.T)
    best = torch.topk(score, top, dim=-1)
    return best.indices, best.values


def moe(h, w, mlp, prefix=""):
    """Sum over a token's chosen experts of expert(score * h)."""
    idx, score = route(h, w[prefix + "router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(idx.shape[1]):
            p = f"{prefix}e{int(idx[t, k])}."
            x = score[t, k] * h[t]
            out[t] += w[p + "down"] @ clamped_glu(w[p + "gate"] @ x, w[p + "up"] @ x, mlp["expert"]["limit"])
    return out


def gated_postnorm_add(x, y, h, w_gate, b_gate, w_post, eps):
    """x + rms_norm(E(h w_gate^T + b) * y) with weight w_post: a sublayer's result enters the residual."""
    return x + rms_norm(torch.sigmoid(h @ w_gate.T + b_gate) * y, w_post, eps)


MIXERS = {"latent_attention": latent_attention, "hgrn2": hgrn2}


def forward(cfg, weights, tokens, dtype=torch.float32, layer_outputs=None):
    """Logits [tokens, vocab] of one sequence; `layer_outputs` (a list) receives the residual after each layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, w, layer["mixer"], eps, p + "mix.")
        x = gated_postnorm_add(x, y, h, w[p + "rg1"], w[p + "rg1.b"], w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            y = moe(h, w, layer["mlp"], p + "mlp.")
            x = gated_postnorm_add(x, y, h, w[p + "rg2"], w[p + "rg2.b"], w[p + "norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
