"""Plain, slow PyTorch-on-CPU statement of the Migosun design, one function per mechanism.

Test infrastructure: it shares no code with the package, works on whole sequences with explicit loops and masks, and keeps
no cache.  Every function takes and returns tensors of one dtype (fp32 or fp64); weights are a dict keyed by checkpoint
tensor names, `cfg` is the checkpoint's config dict.  Rows of a matrix are tokens.
"""
import math

import torch


def rms_norm(x, weight, eps):
    """x_i / sqrt(mean_j x_j^2 + eps) * weight_i over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def silu(x):
    return x * torch.sigmoid(x)


def unit(x):
    """x / sqrt(sum_j x_j^2 + 1e-6) over the last dimension."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def rotate_first_dims(x, positions, dims, base):
    """Rotates the pairs (i, i + dims/2) among the first `dims` of the last dimension by positions * base^(-2 i / dims).
    x [tokens, heads, n]; angles are evaluated in fp64."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * torch.exp(-(2.0 * i / dims) * math.log(base))
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def chunk_mask(n, size):
    """[n, n] bool: query i sees key j when j <= i and both lie in the same chunk of `size` positions."""
    i = torch.arange(n)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def softmax_with_sink(score, sink):
    """exp(score_j) / (sum_j exp(score_j) + exp(sink)): score [heads, i, j], sink [heads]."""
    s = sink[:, None, None].expand(score.shape[0], score.shape[1], 1)
    return torch.softmax(torch.cat([score, s], dim=-1), dim=-1)[..., :-1]


def chunked_attention(h, w, m, eps, prefix=""):
    """Grouped-query attention inside chunks; q and k normed over all their rows before rotation.  -> [tokens, H * vdim]"""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    pos = torch.arange(n)
    q = rms_norm(h @ w[prefix + "q"].T, w[prefix + "q.norm"], eps).view(n, H, d)
    k = rms_norm(h @ w[prefix + "k"].T, w[prefix + "k.norm"], eps).view(n, G, d)
    v = (h @ w[prefix + "v"].T).view(n, G, dv)
    q = rotate_first_dims(q, pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_first_dims(k, pos, m["rot"]["dims"], m["rot"]["base"])
    group = torch.arange(H) // (H // G)
    score = torch.einsum("ihd,jhd->hij", q, k[:, group]) * m["scale"]
    score = score.masked_fill(~chunk_mask(n, m["mask"]["size"]), float("-inf"))
    out = torch.einsum("hij,jhd->ihd", softmax_with_sink(score, w[prefix + "sink"]), v[:, group])
    return out.reshape(n, H * dv)


def short_conv(x, taps):
    """y_t[c] = sum_j taps[c, j] x_{t - (T - 1) + j}[c], zeros before the start; x [tokens, c], taps [c, T]."""
    T = taps.shape[1]
    padded = torch.cat([torch.zeros(T - 1, x.shape[1], dtype=x.dtype), x])
    return sum(taps[:, j] * padded[j:j + x.shape[0]] for j in range(T))


def delta_recurrence(q, k, v, g, beta, state=None):
    """S <- g * S (rows of S by key channel); u = beta (v - S^T k); S <- S + k u^T; o = S^T q.
    q, k, g [tokens, H, C], v [tokens, H, E], beta [tokens, H] -> (o [tokens, H, E], last state [H, C, E])."""
    st = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        st = g[t][:, :, None] * st
        u = beta[t][:, None] * (v[t] - torch.einsum("hce,hc->he", st, k[t]))
        st = st + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hce,hc->he", st, q[t]))
    return torch.stack(out), st


def delta_decay(z, A_log, dt_bias):
    """exp(-exp(A_log_h) softplus(z + dt_bias)); z [tokens, H, C], A_log [H], dt_bias [H * C]."""
    a = torch.nn.functional.softplus(z + dt_bias.view(1, *z.shape[1:]), threshold=1e9)
    return torch.exp(-torch.exp(A_log)[None, :, None] * a)


def gated_delta(h, w, m, eps, prefix=""):
    """Gated delta rule with a decay per key channel, short convolutions and a gated output norm.  -> [tokens, H * vdim]"""
    H, G, C, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q, k, v = (silu(short_conv(h @ w[prefix + t].T, w[prefix + t + ".conv"])) for t in ("q", "k", "v"))
    group = torch.arange(H) // (H // G)
    q = (unit(q.view(n, G, C)) * C ** -0.5)[:, group]
    k = unit(k.view(n, G, C))[:, group]
    beta = torch.sigmoid(h @ w[prefix + "b"].T)
    g = delta_decay(((h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T).view(n, H, C), w[prefix + "A_log"], w[prefix + "dt_bias"])
    o, _ = delta_recurrence(q, k, v.view(n, H, E), g, beta)
    o = rms_norm(o, w[prefix + "norm"], eps)
    return o.reshape(n, H * E) * torch.sigmoid((h @ w[prefix + "g1"].T) @ w[prefix + "g2"].T)


def parallel(h, w, m, eps, prefix=""):
    """Both mixers on the same input, their projected results weighted and added."""
    left = chunked_attention(h, w, m["left"], eps, prefix + "left.") @ w[prefix + "left.o"].T
    right = gated_delta(h, w, m["right"], eps, prefix + "right.") @ w[prefix + "right.o"].T
    return m["left_scale"] * left + m["right_scale"] * right


def linear_attention_recurrence(q, k, v, g, state=None):
    """S <- g * S + k v^T; o = S^T q.  Shapes as delta_recurrence."""
    st = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        st = g[t][:, :, None] * st + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hce,hc->he", st, q[t]))
    return torch.stack(out), st


def gla(h, w, m, eps, prefix=""):
    """Gated linear attention with a decay per key channel."""
    H, C, E = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = (h @ w[prefix + "q"].T * C ** -0.5).view(n, H, C)
    k, v = (h @ w[prefix + "k"].T).view(n, H, C), (h @ w[prefix + "v"].T).view(n, H, E)
    z = (h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "a2.b"]
    g = torch.exp(torch.nn.functional.logsigmoid(z) / m["tau"]).view(n, H, C)
    o, _ = linear_attention_recurrence(q, k, v, g)
    o = rms_norm(o, w[prefix + "norm"], eps).reshape(n, H * E)
    return (o * silu(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def clamped_glu(gate, up, limit):
    """g = min(gate, limit), u = clamp(up, -limit, limit);  g sigmoid(1.702 g) (u + 1)."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense_mlp(h, w, m, prefix=""):
    return clamped_glu(h @ w[prefix + "gate"].T, h @ w[prefix + "up"].T, m["limit"]) @ w[prefix + "down"].T


def join_streams(streams, w_in, w_mix, w_out, sublayer):
    """u = sum_s in[s] x_s; y = sublayer(u); x_t <- sum_s mix[s, t] x_s + out[t] y.  streams [s, tokens, d]"""
    y = sublayer(torch.einsum("s,snd->nd", w_in, streams))
    return torch.einsum("st,snd->tnd", w_mix, streams) + w_out[:, None, None] * y


MIXERS = {"parallel": parallel, "gla": gla}


def forward(cfg, weights, tokens, dtype=torch.float32, layer_outputs=None):
    """Logits [tokens, vocab] of one sequence; `layer_outputs` (a list) receives the sum of the streams after each layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = x[None].repeat(cfg["streams"], 1, 1)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."

        def hc(q):
            return (w[f"{p}hc{q}.{t}"] for t in ("in", "mix", "out"))

        x = join_streams(x, *hc(1), lambda u: MIXERS[layer["type"]](rms_norm(u, w[p + "norm1"], eps), w, layer["mixer"], eps, p + "mix."))
        if layer.get("mlp") is not None:
            x = join_streams(x, *hc(2), lambda u: dense_mlp(rms_norm(u, w[p + "norm2"], eps), w, layer["mlp"], p + "mlp."))
        if layer_outputs is not None:
            layer_outputs.append(x.sum(0))
    return rms_norm(x.sum(0), w["final.norm"], eps) @ w["embed"].T
