"""Every device op of one engine step, timed in isolation against its roofline (a measurement aid).

`record(engine, step)` runs `step()` once with the engine's ops wrapped and keeps the calls; `time_calls` groups
them by op and shape, captures all calls of a group (one per layer, each with its own weights) into a CUDA graph
and replays it, so that a call neither finds its weights in L2 nor waits for the host.  `cost` gives a call's
algorithmic bytes and FLOPs; its roofline time is the larger of bytes / memory bandwidth and FLOPs / tensor rate.
"""
import torch

# a call that is only valid right after another one is timed together with it
_JOINED = {"moe_pack": "moe_route"}
_HOST_ONLY = ("moe_packs", "moe_max_tiles", "state_step_supports", "state_blocks")


class _Recorder:
    def __init__(self, ops):
        self._ops, self.calls = ops, []

    def __getattr__(self, name):
        f = getattr(self._ops, name)
        if not callable(f) or name in _HOST_ONLY or name.endswith("_bytes"):
            return f

        def call(*a, **kw):
            if name in _JOINED and self.calls and self.calls[-1][-1][0] == _JOINED[name]:
                self.calls[-1].append((name, f, a, kw))
            else:
                self.calls.append([(name, f, a, kw)])
            return f(*a, **kw)

        return call


def record(engine, step):
    real, rec = engine.ops, _Recorder(engine.ops)
    engine.ops = rec
    try:
        with torch.no_grad():
            step()
        torch.cuda.synchronize()
    finally:
        engine.ops = real
    return rec.calls


def _visible(S, pos0, window, chunk=0):
    """Visible (query, key) pairs of S queries from position pos0 on."""
    return sum(min(pos0 + i + 1, window, (pos0 + i) % chunk + 1 if chunk else window) for i in range(S))


def cost(name, a, kw, pos0, experts_used):
    """(bytes, flops) of one call; 2-byte storage, fp32 projections and residual."""
    if name == "embed_norm":
        n, d = a[1].numel(), a[0].shape[1]
        return n * d * 8, 0
    if name == "embedding":
        return a[1].numel() * a[0].shape[1] * 4, 0
    if name == "add_rmsnorm":
        rows, d = a[7], a[0].shape[-1]
        return rows * d * 2 * (2 + (a[1] is not None) + (a[2] is not None) + (a[5] is not None)), 0
    if name in ("linear", "linear_f32"):
        (n, k), m = a[1].shape, a[3]
        return n * k * 2 + m * k * 2 + m * n * (4 if name == "linear_f32" else 2), 2 * m * n * k
    if name == "lm_head_argmax":
        (n, k), m = a[1].shape, a[4]
        return n * k * 2 + m * k * 2, 2 * m * n * k
    if name == "gated_norm_add":
        rows, d = a[9], a[0].shape[-1]
        return rows * d * (2 * kw.get("n_slots", 1) + 4 + 8 + 2), 0
    if name == "qkv_rope_kvcache":
        (n, k), m = a[1].shape, a[8] * a[9]
        return n * k * 2 + m * (k + n) * 2, 2 * m * n * k
    if name == "gateup_swiglu":
        (n, k), m = a[1].shape, a[3]
        return n * k * 2 + m * (k + n // 2) * 2, 2 * m * n * k
    if name == "attention":
        B, S, nh, nkv, hd = a[5:10]
        pairs = _visible(S, pos0, 1 << 60)
        return B * 2 * (2 * S * nh * hd + 2 * nkv * hd * (pos0 + S)), 4 * B * nh * hd * pairs
    if name == "latent_prepare":
        B, S, H, dn, dr, r = a[13:19]
        return B * S * (H * (dn + dr) + r + dr) * 6, 0
    if name == "latent_window":
        return a[4] * min(a[6], pos0 + a[6] - a[5]) * (a[1] + a[2]) * 4, 0
    if name == "head_linear":
        rows, H, n_in, n_out = a[6:10]
        return 2 * H * (n_in * n_out + rows * (n_in + n_out)), 2 * rows * H * n_in * n_out
    if name == "window_attention":
        window, (B, S, H, d1, d2, dv) = a[12], a[14:20]
        keys = min(pos0 + S, window + S - 1)
        shared = a[3][2] == 0
        per_key = (d1 + d2) if shared else H * (d1 + dv) + d2
        return 2 * B * (S * H * (d1 + d2 + dv) + keys * per_key), 2 * B * H * (d1 + d2 + dv) * _visible(S, pos0, window)
    if name == "hgrn2":
        B, S, H, C, E = a[12:17]
        return B * (S * H * ((2 * C + E) * 4 + E * 2) + 8 * H * C * E), 4 * B * S * H * C * E
    if name in ("embed_streams", "join_streams"):
        n, d = (a[1].numel(), a[0].shape[1]) if name == "embed_streams" else (a[8], a[0].shape[2])
        streams = (a[3] if name == "embed_streams" else a[0]).shape[1]
        moved = streams * 4 + 4 if name == "embed_streams" else streams * (8 if kw.get("write", True) else 4) + 4
        return n * d * moved, 0
    if name == "gateup_glu":
        (n, k), m = a[1].shape, a[3]
        return n * k * 2 + m * (k + n // 2) * 2, 2 * m * n * k
    if name == "grouped_prepare":
        B, S, H = a[14:17]
        (_, G, _, d), dv = a[12].shape, a[13].shape[3]
        return B * S * ((H + G) * d + G * dv) * 6, 0
    if name == "grouped_attention":
        window, chunk, (B, S, H) = a[8], a[9], a[11:14]
        (_, G, _, d), dv = a[1].shape, a[2].shape[3]
        first = max(0, pos0 - window + 1 if window else 0, pos0 // chunk * chunk if chunk else 0)
        pairs = _visible(S, pos0, window or 1 << 60, chunk)
        return 2 * B * (S * H * (d + dv) + (pos0 + S - first) * G * (d + dv)), 2 * B * H * (d + dv) * pairs
    if name == "delta_blocks":
        B, S, H, G, C, E = a[11:17]
        return 4 * B * S * ((2 * G * C + H * E) + H * C + 3 * H * C + H * C // 4 + H * E + 8 * H), 0
    if name == "gla_blocks":
        B, S, H, C = a[7:11]
        return 4 * B * S * (3 * H * C + 2 * H * C + H * C // 4 + 8 * H), 0
    if name == "state_scan":
        # the recurrence's own inputs (q, k, decay, v) and results, however the blocks carry them
        B, S = a[7:9]
        _, H, C, E = a[4].shape
        return 4 * B * (S * (3 * H * C + 2 * H * E) + 2 * H * C * E), (8 if a[1] else 6) * B * S * H * C * E
    if name in ("delta_step", "gla_step"):
        st, B, a2 = (a[12], a[16], a[5]) if name == "delta_step" else (a[9], a[13], a[3])
        _, H, C, E = st.shape
        low = a2.numel() + (a[6].numel() if name == "delta_step" else 0)
        return B * (8 * H * C * E + 4 * H * (2 * C + 2 * E)) + 2 * low, (8 if name == "delta_step" else 6) * B * H * C * E
    if name == "head_norm_gate":
        return a[9] * a[10] * a[1].numel() * 10, 0
    if name == "round_columns":
        return a[5] * a[3] * 6, 0
    if name == "moe_route":
        return a[4] * a[2] * 4, 0
    if name == "moe_pack":
        d = a[0].shape[-1]
        return a[1] * d * 2 * (1 + a[2]), 0
    if name == "moe_gateup":
        (_, n, k), pairs = a[1].shape, a[5]
        return experts_used(pairs) * n * k * 2 + pairs * (k + n // 2) * 2, 2 * pairs * n * k
    if name == "moe_down":
        (_, n, k), pairs = a[1].shape, a[4]
        return experts_used(pairs) * n * k * 2 + pairs * (k + n) * 2, 2 * pairs * n * k
    return 0, 0


def _key(call):
    def shape(x):
        if isinstance(x, (tuple, list)):
            return tuple(shape(y) for y in x)
        return tuple(x.shape) if torch.is_tensor(x) else x

    out = []
    for name, _, a, kw in call:
        out.append((name, tuple(shape(x) for x in a if not isinstance(x, float)),
                    tuple(sorted(k for k in kw))))
    return tuple(out)


def time_calls(calls, pos0, hbm_gbs, tflops, experts=None, min_us=20000.0):
    """[{op, calls, us, gbs, tflops, frac}] per group, in order of first use.  experts: number of experts of the
    model's layers (expected number of distinct ones used by `pairs` uniform choices)."""
    groups = {}
    for c in calls:
        groups.setdefault(_key(c), []).append(c)

    def used(pairs):
        return experts * (1 - (1 - 1 / experts) ** pairs) if experts else 1

    rows = []
    for group in groups.values():
        rounds = max(1, -(-16 // len(group)))

        def run():
            for _ in range(rounds):
                for call in group:
                    for _, f, a, kw in call:
                        f(*a, **kw)

        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side), torch.no_grad():
            run()
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph), torch.no_grad():
            run()

        def timed(reps):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            for _ in range(reps):
                graph.replay()
            e1.record()
            torch.cuda.synchronize()
            return e0.elapsed_time(e1) * 1e3

        timed(1)
        reps = max(3, min(50, int(min_us / max(timed(1), 1.0)) + 1))
        us = timed(reps) / (reps * rounds * len(group))
        nbytes = flops = 0
        for name, _, a, kw in group[0]:
            b, f = cost(name, a, kw, pos0, used)
            nbytes, flops = nbytes + b, flops + f
        ideal = max(nbytes / (hbm_gbs * 1e3), flops / (tflops * 1e6))
        rows.append({"op": "+".join(n for n, *_ in group[0]), "calls": len(group), "us": us, "bytes": nbytes, "flops": flops,
                     "gbs": nbytes / us / 1e3, "tflops": flops / us / 1e6, "frac": ideal / us,
                     "bound": "tensor" if flops / (tflops * 1e6) > nbytes / (hbm_gbs * 1e3) else "hbm"})
    return rows
