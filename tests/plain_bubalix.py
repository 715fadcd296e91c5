"""A plain, slow implementation of the Bubalix decoder in float64 on the CPU: one function a mechanism, whole sequences at
once, no cache.  It shares no code with the engine; the tests hold the engine to it.

``cfg`` is the dictionary of config.json, ``W`` a dictionary name -> float64 tensor (integer tables stay integers); ``h`` is a
sublayer's input ``[T, width]``; linear weights are stored ``[out, in]`` and applied as ``h @ W.T``; positions count from 0.
"""
import math

import torch

F = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the gain's distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def time_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] * u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


# ---- rotation ----------------------------------------------------------------------------------------------

def stretched_frequencies(rot):
    """The frequency of every rotated pair and the factor on cos and sin."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def place(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(float(sc["fast"]))), 0)
    hi = min(math.ceil(place(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: element i of the first ``dims`` is paired with element i + dims / 2; the rest pass unchanged."""
    if not rot or not rot.get("dims"):
        return x
    f, mag = stretched_frequencies(rot)
    r = int(rot["dims"]) // 2
    a = positions.to(F)[:, None] * torch.tensor(f, dtype=F)[None]
    c, s = (mag * torch.cos(a))[:, None], (mag * torch.sin(a))[:, None]
    u, v = x[..., :r], x[..., r:2 * r]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * r:]], dim=-1)


# ---- scores and softmax --------------------------------------------------------------------------------------

def visible(i, j, size):
    """Does the query at position i see the key at position j?  ``size`` None: every earlier key."""
    return j <= i and (size is None or i - j < size)


def visibility(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def distance_slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def softmax_with_sink(s, seen, sink):
    """Weights of the visible scores s [T, T] under a softmax whose denominator also holds exp(sink) (None: no sink)."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, torch.as_tensor(float(sink), dtype=F))
    e = torch.exp(s - m)
    z = e.sum(-1, keepdim=True)
    return e / (z + torch.exp(float(sink) - m) if sink is not None else z)


def query_temperature(positions, t):
    """The factor on a query at each position."""
    return 1.0 + float(t["coef"]) * torch.log(torch.floor((positions.to(F) + 1.0) / float(t["every"])) + 1.0)


# ---- mixers ---------------------------------------------------------------------------------------------------

def latent_pair(h, W, p, m, eps, positions):
    """What a token leaves for later ones: its normed latent [T, kv_rank] and its rotated key part [T, rot_dim]."""
    y = h @ W[p + "dkv"].T
    r = int(m["kv_rank"])
    c = unit_rms(y[:, :r], eps) * W[p + "dkv.norm"]
    return c, rotate_halves(y[:, None, r:], positions, m.get("rot"))[:, 0]


def latent_attention(h, W, p, m, eps, probs=None):
    T, H, d, rd, vd = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ W[p + "q"].T).reshape(T, H, d + rd)
    qn, qr = q[..., :d], rotate_halves(q[..., d:], pos, m.get("rot"))
    c, kr = latent_pair(h, W, p, m, eps, pos)
    k = (c @ W[p + "uk"].T).reshape(T, H, d)
    v = (c @ W[p + "uv"].T).reshape(T, H, vd)
    seen, out, kept = visibility(T, None), torch.zeros(T, H, vd, dtype=F), []
    for hh in range(H):
        s = (qn[:, hh] @ k[:, hh].T + qr[:, hh] @ kr.T) * float(m["scale"])
        w = softmax_with_sink(s, seen, W[p + "sink"][hh])
        out[:, hh] = w @ v[:, hh]
        kept.append(w)
    if probs is not None:
        probs.append(torch.stack(kept))
    return (out.reshape(T, H * vd) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def attention(h, W, p, m, probs=None):
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k, v = (time_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in ("q", "k", "v"))
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, vd)
    if m.get("q_temp"):
        q = q * query_temperature(pos, m["q_temp"])[:, None, None]
    seen = visibility(T, (m.get("mask") or {}).get("size"))
    away = (pos[:, None] - pos[None, :]).to(F)
    out, kept = torch.zeros(T, H, vd, dtype=F), []
    for hh in range(H):
        g = hh // (H // G)
        s = capped((q[:, hh] @ k[:, g].T) * float(m["scale"]), m.get("softcap")) - distance_slope(hh, H) * away
        w = softmax_with_sink(s, seen, W[p + "sink"][hh])
        out[:, hh] = w @ v[:, g]
        kept.append(w)
    if probs is not None:
        probs.append(torch.stack(kept))
    out = out * torch.sigmoid(h @ W[p + "g"].T)[..., None]
    return out.reshape(T, H * vd) @ W[p + "o"].T


# ---- feed-forward, token input, layer ------------------------------------------------------------------------

def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def mixture(h, tokens, W, p, mlp):
    """The experts that the table names for a token, equally weighted, and the shared expert."""
    chosen = W[p + "table"].long()[tokens]
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        share = (chosen == e).to(F).sum(-1, keepdim=True) / float(mlp["router"]["top"])
        out += share * expert(h, W, f"{p}e{e}.")
    return out + expert(h, W, p + "shared.") if mlp.get("shared") else out


def token_input(x, tokens, W, p, i, dim, eps):
    """The layer's share of the token's side vector, gated by the stream, projected and normed."""
    e = W["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ W[p + "gate"].T) * e) @ W[p + "proj"].T
    return unit_rms(y, eps) * W[p + "norm"]


def layer(x, tokens, W, cfg, i, probs=None):
    L, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    h = centred_norm(x, W[p + "norm1"], eps)
    if L["type"] == "latent_attention":
        y = latent_attention(h, W, p + "mix.", L["mixer"], eps, probs)
    elif L["type"] == "attention":
        y = attention(h, W, p + "mix.", L["mixer"], probs)
    else:
        raise ValueError(L["type"])
    if L.get("mlp") is not None:
        y = y + mixture(h, tokens, W, p + "mlp.", L["mlp"])
    x = x + y
    if cfg.get("token_side"):
        x = x + token_input(x, tokens, W, p + "side.", i, int(cfg["token_side"]["dim"]), eps)
    return x


def forward(cfg, W, tokens, streams=None, probs=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) receives the stream after every layer, ``probs`` the weights of
    every attention that ran."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i in range(len(cfg["layers"])):
        x = layer(x, tokens, W, cfg, i, probs)
        if streams is not None:
            streams.append(x)
    return centred_norm(x, W["final.norm"], float(cfg["norm"]["eps"])) @ W["head"].T


# ---- what a checkpoint of a configuration holds, and seeded random ones ------------------------------------

def tensor_shapes(cfg):
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    side = int(cfg["token_side"]["dim"]) if cfg.get("token_side") else 0
    if side:
        out["side.embed"] = (V, side * len(cfg["layers"]))
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        q = p + "mix."
        H, vd = m["heads"], m["vdim"]
        out[p + "norm1"] = (W,)
        if L["type"] == "latent_attention":
            d, rd, r = m["dim"], m["rot_dim"], m["kv_rank"]
            out.update({q + "q": (H * (d + rd), W), q + "dkv": (r + rd, W), q + "dkv.norm": (r,), q + "uk": (H * d, r), q + "uv": (H * vd, r),
                        q + "g": (H * vd, W)})
        else:
            G, d, taps = m["kv_heads"], m["dim"], m["conv"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * vd)):
                out.update({q + n: (rows, W), q + n + ".conv": (rows, taps)})
            out[q + "g"] = (H, W)
        out.update({q + "sink": (H,), q + "o": (W, H * vd)})
        if mlp is not None:
            ff = mlp["expert"]["ff"]
            out[p + "mlp.table"] = (V, mlp["router"]["top"])
            parts = [(f"e{e}", ff) for e in range(mlp["router"]["experts"])] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else [])
            for n, size in parts:
                out.update({f"{p}mlp.{n}.gate": (size, W), f"{p}mlp.{n}.up": (size, W), f"{p}mlp.{n}.down": (W, size)})
        if side:
            out.update({p + "side.gate": (side, W), p + "side.proj": (W, side), p + "side.norm": (W,)})
    return out


def random_weights(cfg, seed, gain=1.0):
    """Seeded weights as a checkpoint stores them (bfloat16, tables int32): matrices of a size that keeps activations of order
    one, gains around one, sinks that take a visible share of a softmax."""
    g = torch.Generator().manual_seed(seed)
    experts = {f"l{i}.mlp.table": int(L["mlp"]["router"]["experts"]) for i, L in enumerate(cfg["layers"]) if L.get("mlp")}
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last == "table":
            out[name] = torch.rand(shape[0], experts[name], generator=g).argsort(1)[:, :shape[1]].to(torch.int32).contiguous()
            continue
        if name in ("embed", "side.embed"):
            t = torch.randn(shape, generator=g)
        elif name == "final.norm" or last == "norm1":
            t = 0.2 * torch.randn(shape, generator=g)
        elif last == "norm":
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif last == "sink":
            t = 1.0 + torch.randn(shape, generator=g)
        elif last == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        else:
            t = gain * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def as_float64(W):
    return {k: v if not v.is_floating_point() else v.to(F) for k, v in W.items()}
