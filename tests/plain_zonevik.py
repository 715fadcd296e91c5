"""A plain, slow implementation of the Zonevik decoder in float64 on the CPU: one function a mechanism, whole sequences at
once, no cache.  It shares no code with the engine; the tests hold the engine to it.

``cfg`` is the dictionary of config.json, ``W`` a dictionary name -> float64 tensor; ``h`` is a sublayer's input ``[T, width]``;
linear weights are stored ``[out, in]`` and applied as ``h @ W.T``; positions count from 0.
"""
import math

import torch

F = torch.float64


def dynamic_tanh(x, W, name):
    """tanh(alpha x) * w + b element by element; no statistics."""
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def time_conv(h, w, b=None):
    """h [T, C], w [C, taps]: out_t = sum_j w[:, j] * h_(t - taps + 1 + j) (+ b), zeros before the start."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * h[:T - back]
    return out if b is None else out + b


def yarn_frequencies(dims, base, scaling):
    """The frequency of every pair and the factor that cos and sin are multiplied by; ``scaling`` None: plain rotary."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def place(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))

    lo = max(math.floor(place(float(scaling["fast"]))), 0)
    hi = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, rot):
    """x [T, heads, d]: the pairs (2i, 2i + 1) of every head's first ``dims`` elements turn by position * frequency_i."""
    if rot is None or not rot.get("dims"):
        return x
    freqs, mag = yarn_frequencies(int(rot["dims"]), rot["base"], rot.get("scaling"))
    out = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(F) * f
        c, s = mag * torch.cos(a)[:, None], mag * torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(i, j, size, keep_first):
    """Does the query at position i see the key at position j?  ``size`` None: every earlier key."""
    if j > i:
        return False
    return size is None or i - j < size or j < keep_first


def visibility(T, size, keep_first):
    """[query, key] of ``visible`` for a sequence of T tokens."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def softmax_attention(q, k, v, scale, size, keep_first, probs=None):
    """q [T, H, d], k [T, G, d], v [T, G, vd]; ``probs`` (a list) receives the weights [H, T, T]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = visibility(T, size, keep_first)
    out, kept = torch.zeros(T, H, v.shape[2], dtype=F), []
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * scale
        p = torch.softmax(torch.where(seen, s, torch.full_like(s, -math.inf)), dim=-1)
        out[:, hh] = p @ v[:, g]
        kept.append(p)
    if probs is not None:
        probs.append(torch.stack(kept))
    return out


def attention(h, W, p, m, gate, probs=None):
    """Grouped-query attention; biases where the checkpoint has them; ``gate``: the concatenated heads times sigmoid(W_g h)."""
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def project(n):
        y = h @ W[p + n].T
        return y + W[p + n + ".b"] if (p + n + ".b") in W else y

    pos = torch.arange(T)
    q = rotate_pairs(project("q").reshape(T, H, d), pos, m.get("rot"))
    k = rotate_pairs(project("k").reshape(T, G, d), pos, m.get("rot"))
    v = project("v").reshape(T, G, vd)
    mask = m.get("mask") or {}
    o = softmax_attention(q, k, v, float(m["scale"]), mask.get("size"), int(mask.get("keep_first") or 0), probs).reshape(T, H * vd)
    if gate:
        o = o * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def delta_state_walk(q, k, v, g, beta, S=None):
    """The gated delta rule, token by token: q, k [T, H, d], v [T, H, vd], g and beta [T, H].  Returns o [T, H, vd] and the last state."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta(h, W, p, m, eps):
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(time_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vector(q.reshape(T, G, d)) * d ** -0.5
    k = unit_vector(k.reshape(T, G, d))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o, _ = delta_state_walk(q, k, v.reshape(T, H, vd), g, beta)
    o = unit_rms(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).reshape(T, H, vd)
    return o.reshape(T, H * vd) @ W[p + "o"].T


def ssd_state_walk(B, C, x, dt, a_log, D, S=None):
    """The state-space dual scan, token by token: B, C [T, H, N] (each head's group's), x [T, H, vd], dt [T, H]."""
    T, H, N = B.shape
    S = torch.zeros(H, N, x.shape[2], dtype=F) if S is None else S.clone()
    out = torch.zeros(T, H, x.shape[2], dtype=F)
    for t in range(T):
        S = torch.exp(-torch.exp(a_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t]
    return out, S


def mamba2(h, W, p, m, eps):
    T, H, vd, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    proj = h @ W[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(time_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    dt = softplus(dt + W[p + "dt_bias"])
    rep = H // G
    B, C = (y.reshape(T, G, N).repeat_interleave(rep, dim=1) for y in (B, C))
    y, _ = ssd_state_walk(B, C, x.reshape(T, H, vd), dt, W[p + "A_log"], W[p + "D"])
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = unit_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * W[p + "norm"]
    return y @ W[p + "o"].T


def parallel(h, W, p, m, eps, probs=None):
    left = attention(h, W, p + "left.", m["left"], False, probs)
    right = mamba2(h, W, p + "right.", m["right"], eps)
    return 0.5 * (unit_rms(left, eps) * W[p + "left.out"] + unit_rms(right, eps) * W[p + "right.out"])


def route(h, r, W, p):
    """Per token: the chosen experts and their weights, the sigmoid scores as they are; a group counts by the sum of its two best."""
    s = torch.sigmoid(h @ W[p + "router"].T)
    choice, groups = s.clone(), r.get("groups")
    if groups:
        per = int(r["experts"]) // int(groups["count"])
        by_group = s.reshape(-1, int(groups["count"]), per)
        score = torch.topk(by_group, min(2, per), dim=-1).values.sum(-1)
        allowed = torch.zeros_like(score, dtype=torch.bool).scatter_(1, torch.topk(score, int(groups["keep"]), dim=-1).indices, True)
        choice = torch.where(allowed.repeat_interleave(per, dim=1), choice, torch.full_like(choice, -math.inf))
    idx = torch.topk(choice, int(r["top"]), dim=-1).indices
    return idx, torch.gather(s, 1, idx)


def mixture(h, W, p, mlp):
    idx, w = route(h, mlp["router"], W, p)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        y = (silu(h @ W[f"{p}e{e}.gate"].T) * (h @ W[f"{p}e{e}.up"].T)) @ W[f"{p}e{e}.down"].T
        out += (w * (idx == e)).sum(-1, keepdim=True) * y
    return out


def run_order(cfg):
    """(layer, does it open a pass of the loop) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    once = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + once * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


def layer(x, W, cfg, i, probs=None):
    L, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    h = dynamic_tanh(x, W, p + "norm1")
    if L["type"] == "attention":
        a = attention(h, W, p + "mix.", L["mixer"], True, probs)
    elif L["type"] == "delta":
        a = delta(h, W, p + "mix.", L["mixer"], eps)
    elif L["type"] == "parallel":
        a = parallel(h, W, p + "mix.", L["mixer"], eps, probs)
    else:
        raise ValueError(L["type"])
    x = x + dynamic_tanh(a, W, p + "norm1b")
    if L.get("mlp") is not None:
        x = x + dynamic_tanh(mixture(dynamic_tanh(x, W, p + "norm2"), W, p + "mlp.", L["mlp"]), W, p + "norm2b")
    return x


def forward(cfg, W, tokens, streams=None, probs=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) receives the stream after every layer run, ``probs`` the weights
    of every attention that ran."""
    x0 = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    x = x0
    for i, opens in run_order(cfg):
        if opens:
            x = torch.cat([x, x0], dim=-1) @ W["loop.in"].T
        x = layer(x, W, cfg, i, probs)
        if streams is not None:
            streams.append(x)
    return dynamic_tanh(x, W, "final.norm") @ W["embed"].T


# ---- what a checkpoint of a configuration holds, and seeded random ones ------------------------------------

def tensor_shapes(cfg):
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (V, W)}

    def norm(name):
        out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

    norm("final.norm")
    if cfg.get("loop"):
        out["loop.in"] = (W, 2 * W)
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        norm(p + "norm1"), norm(p + "norm1b")
        q = p + "mix."
        if L["type"] == "attention":
            H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * vd, W), q + "g": (H * vd, W), q + "o": (W, H * vd)})
        elif L["type"] == "delta":
            H, G, d, vd, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * vd)):
                out.update({q + n: (rows, W), q + n + ".conv": (rows, taps)})
            out.update({q + "b": (H, W), q + "a": (H, W), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (vd,), q + "g": (H * vd, W), q + "o": (W, H * vd)})
        else:
            lm, r = m["left"], m["right"]
            H, G, d, vd = lm["heads"], lm["kv_heads"], lm["dim"], lm["vdim"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * vd)):
                out.update({q + "left." + n: (rows, W), q + "left." + n + ".b": (rows,)})
            out[q + "left.o"] = (W, H * vd)
            H, vd, N, G, taps = r["heads"], r["vdim"], r["state"], r["groups"], r["conv"]
            ch = H * vd + 2 * G * N
            out.update({q + "right.in": (H * vd + ch + H, W), q + "right.conv": (ch, taps), q + "right.conv.b": (ch,), q + "right.dt_bias": (H,),
                        q + "right.A_log": (H,), q + "right.D": (H,), q + "right.norm": (H * vd,), q + "right.o": (W, H * vd),
                        q + "left.out": (W,), q + "right.out": (W,)})
        if mlp is None:
            continue
        norm(p + "norm2"), norm(p + "norm2b")
        out[p + "mlp.router"] = (mlp["router"]["experts"], W)
        ff = mlp["expert"]["ff"]
        for e in range(mlp["router"]["experts"]):
            out.update({f"{p}mlp.e{e}.gate": (ff, W), f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return out


def random_weights(cfg, seed, gain=1.0):
    """Seeded weights in bfloat16 (as a checkpoint stores them): matrices of a size that keeps activations of order one, norm
    weights around one, decays that forget over a few to a few hundred tokens."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = torch.randn(shape, generator=g)
        elif last == "alpha":
            t = 0.5 + 0.4 * torch.rand(shape, generator=g)
        elif last in ("norm1", "norm2", "norm1b", "norm2b", "norm", "out", "D"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif last == "b" and len(shape) == 1:
            t = 0.2 * torch.randn(shape, generator=g)
        elif last == "A_log":
            t = 0.5 * torch.randn(shape, generator=g)
        elif last == "dt_bias":
            t = -3.0 + 1.5 * torch.randn(shape, generator=g)
        elif last == "conv":
            t = 0.6 * torch.randn(shape, generator=g)
        elif last == "router":
            t = gain * 2.0 * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        else:
            t = gain * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def as_float64(W):
    return {k: v.to(F) for k, v in W.items()}
