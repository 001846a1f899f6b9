"""Plain, slow PyTorch statement of the hybrid designs (one function per mechanism, token by token where
there is a recurrence). It is the yardstick of the hybrid tests and shares no code with the package."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def causal_attention(q, k, v, scale):
    """q [T, H, dk]; k [T, G, dk]; v [T, G, dv]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), 1), float("-inf"))
        s = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (s / s.sum(-1, keepdim=True)) @ v[:, g]
    return out


def short_conv(x, w):
    """Causal per-channel convolution, last tap = current token. x [T, C], w [C, taps]."""
    T, C = x.shape
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta):
    """q, k, g [T, H, dk]; v [T, H, dv]; beta [T, H] -> [T, H, dv]."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def gla_recurrence(q, k, v, alpha):
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out


def gated_attention(h, W, p, c, eps):
    T = h.shape[0]
    H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_norm((h @ W[p + "q"].T).view(T, H, dk), W[p + "q.norm"], eps)
    k = rms_norm((h @ W[p + "k"].T).view(T, G, dk), W[p + "k.norm"], eps)
    v = (h @ W[p + "v"].T).view(T, G, dv)
    o = causal_attention(q, k, v, c["scale"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ W[p + "o"].T


def gated_delta(h, W, p, c, eps):
    T = h.shape[0]
    H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = silu(short_conv(h @ W[p + "q"].T, W[p + "q.conv"])).view(T, G, dk)
    k = silu(short_conv(h @ W[p + "k"].T, W[p + "k.conv"])).view(T, G, dk)
    v = silu(short_conv(h @ W[p + "v"].T, W[p + "v.conv"])).view(T, H, dv)
    q, k = unit(q) * dk ** -0.5, unit(k)
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]
    g = torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(z).view(T, H, dk))
    o = delta_recurrence(q, k, v, g, beta)
    gate = torch.sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T).view(T, H, dv)
    return (rms_norm(o, W[p + "norm"], eps) * gate).reshape(T, H * dv) @ W[p + "o"].T


def gla(h, W, p, c, eps):
    T = h.shape[0]
    H, dk, dv = c["heads"], c["dim"], c["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, dk) * dk ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, dk)
    v = (h @ W[p + "v"].T).view(T, H, dv)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = torch.sigmoid(z).pow(1.0 / c["tau"]).view(T, H, dk)
    o = rms_norm(gla_recurrence(q, k, v, alpha), W[p + "norm"], eps)
    return (o.reshape(T, H * dv) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(h, W, p, c, eps):
    a = rms_norm(gated_attention(h, W, p + "left.", c["left"], eps), W[p + "left.out"], eps)
    b = rms_norm(gated_delta(h, W, p + "right.", c["right"], eps), W[p + "right.out"], eps)
    return 0.5 * (a + b)


MIXERS = {"gla": gla, "parallel": parallel}


def dense_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ------------------------------------------------------------------ Lebedra
def rotate_pairs(x, pos, base):
    """Interleaved rotation: components 2i and 2i + 1 of x [T, ..., n] turn by pos * base^(-2i / n)."""
    n = x.shape[-1]
    out = x.clone()
    for i in range(n // 2):
        a = pos.to(torch.float64) * float(base) ** (-2.0 * i / n)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        shape = [-1] + [1] * (x.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def sink_attention(q, k, v, scale, sink):
    """Causal attention with one more term exp(sink[h]) in the denominator. q [T, H, dk]; k [T, H, dk]; v [T, H, dv]."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    future = torch.triu(torch.ones(T, T, dtype=torch.bool), 1)
    for h in range(H):
        s = ((q[:, h] @ k[:, h].T) * scale).masked_fill(future, float("-inf"))
        m = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink[h]))
        e = torch.exp(s - m)
        out[:, h] = (e @ v[:, h]) / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - m))
    return out


def latent_parts(h, W, p, c, eps, pos):
    """(queries [T, H, dim + rot], latent [T, rank], shared rotated key [T, rot])."""
    T, H, dn, dr, r = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    base = c["rot"]["base"]
    q = (h @ W[p + "q"].T).view(T, H, dn + dr)
    q = torch.cat([q[..., :dn], rotate_pairs(q[..., dn:], pos, base)], -1)
    kv = h @ W[p + "dkv"].T
    return q, rms_norm(kv[:, :r], W[p + "dkv.norm"], eps), rotate_pairs(kv[:, r:], pos, base)


def latent_attention(h, W, p, c, eps):
    T, H, dn, dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q, lat, kr = latent_parts(h, W, p, c, eps, torch.arange(T))
    k = torch.cat([(lat @ W[p + "uk"].T).view(T, H, dn), kr[:, None, :].expand(T, H, kr.shape[1])], -1)
    v = (lat @ W[p + "uv"].T).view(T, H, dv)
    return sink_attention(q, k, v, c["scale"], W[p + "sink"]).reshape(T, H * dv) @ W[p + "o"].T


def relu_ff(h, W, p):
    return (torch.clamp(h @ W[p + "gate"].T, min=0) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def clamped_expert(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T


def choose_experts(z, correction, r):
    """Router logits of one token -> list of (expert, weight)."""
    E, n, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
    s = torch.exp(z - z.max())
    s = s / s.sum()
    choice = (s + correction).tolist()
    size = E // n
    best = sorted(range(n), key=lambda g: -max(choice[g * size:(g + 1) * size]))[:keep]
    allowed = [e for e in range(E) if e // size in best]
    picked = sorted(allowed, key=lambda e: -choice[e])[: r["top"]]
    return [(e, s[e]) for e in picked]


def moe(h, W, p, c):
    z = h @ W[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in choose_experts(z[t], W[p + "correction"], c["router"]):
            out[t] += w * clamped_expert(h[t:t + 1], W, p + f"e{e}.", c["expert"]["limit"])[0]
    return out


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh((2 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def token_side(x, W, p, e, eps):
    return rms_norm((gelu_tanh(x @ W[p + "gate"].T) * e) @ W[p + "proj"].T, W[p + "norm"], eps)


def forward_lebedra(cfg, W, tokens, dtype=torch.float64, trace=None):
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, m, n = cfg["norm"]["eps"], cfg["residual_mult"], cfg["token_side"]["dim"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][tok]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * rms_norm(latent_attention(x, W, p + "mix.", L["mixer"], eps), W[p + "norm1"], eps)
        if L["mlp"] is not None:
            y = moe(x, W, p + "mlp.", L["mlp"]) if L["mlp"]["kind"] == "moe" else relu_ff(x, W, p + "mlp.")
            x = x + m * rms_norm(y, W[p + "norm2"], eps)
        x = x + m * token_side(x, W, p + "side.", W["side.embed"][tok][:, i * n:(i + 1) * n], eps)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


# ------------------------------------------------------------------ Dogozen
def rms_norm_around_zero(x, w, eps):
    return rms(x, eps) * (1 + w)


def frequencies(r):
    """Angle per position of every rotated pair, with the optional stretching of long wavelengths: pairs that turn
    fewer than ``low`` times within ``original`` positions are slowed by ``factor``, those that turn more than ``high``
    times are not, and those between are blended linearly in the number of turns."""
    out = []
    for i in range(r["dims"] // 2):
        f = float(r["base"]) ** (-2.0 * i / r["dims"])
        sc = r.get("scaling")
        if sc:
            turns = sc["original"] * f / (2 * torch.pi)
            if turns < sc["low"]:
                f = f / sc["factor"]
            elif turns <= sc["high"]:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_halves(x, pos, r):
    """Components i and i + dims / 2 of x [T, heads, n] turn together; those from ``dims`` on stay."""
    out, half = x.clone(), r["dims"] // 2
    for i, f in enumerate(frequencies(r)):
        a = pos.to(torch.float64) * f
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


def query_temperature(pos, c):
    return 1 + c["coef"] * torch.log(torch.floor((pos + 1).to(torch.float64) / c["every"]) + 1)


def window_sink_attention(q, k, v, scale, window=None, sink=None):
    """Query i sees keys j <= i, with ``window`` only those with i - j < window; with ``sink`` the denominator has one
    more term per query head. q [T, H, dk]; k [T, G, dk]; v [T, G, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            lo = 0 if window is None else max(0, i - window + 1)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            m = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - m)
            out[i, h] = (e @ v[lo:i + 1, g]) / (e.sum() + (0 if sink is None else torch.exp(sink[h] - m)))
    return out


def tempered_attention(h, W, p, c, eps, kv):
    """Attention with unit-rms queries and keys, query temperature and a gate per channel; ``kv`` (layer -> keys and
    values) receives the layer's own and gives those of a layer that shares them."""
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    pos = torch.arange(T)
    q = rms((h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, c["dim"]), eps)
    if c.get("q_temp"):
        q = q * query_temperature(pos, c["q_temp"]).to(q.dtype)[:, None, None]
    if c.get("kv_from") is None:
        k = rms((h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, c["dim"]), eps)
        v = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, c["vdim"])
        kv[p] = (k, v)
    else:
        k, v = kv[f"l{c['kv_from']}.mix."]
    o = window_sink_attention(q, k, v, c["scale"]).reshape(T, H * c["vdim"])
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def window_attention(h, W, p, c):
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    pos = torch.arange(T)
    q = rotate_halves((h @ W[p + "q"].T).view(T, H, c["dim"]), pos, c["rot"])
    k = rotate_halves((h @ W[p + "k"].T).view(T, G, c["dim"]), pos, c["rot"])
    v = (h @ W[p + "v"].T).view(T, G, c["vdim"])
    o = window_sink_attention(q, k, v, c["scale"], c["mask"]["size"], W[p + "sink"])
    return o.reshape(T, H * c["vdim"]) @ W[p + "o"].T


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, channels]; A [channels, n]; B, C [T, n]; D [channels] -> y [T, channels]."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba(h, W, p, c):
    n, r = c["state"], c["dt_rank"]
    xz = h @ W[p + "in"].T
    x, z = xz[:, : c["inner"]], xz[:, c["inner"]:]
    x = silu(short_conv(x, W[p + "conv"]) + W[p + "conv.b"])
    low = x @ W[p + "x"].T
    dt = softplus(low[:, :r] @ W[p + "dt"].T + W[p + "dt.b"])
    y = selective_scan(x, dt, -torch.exp(W[p + "A_log"]), low[:, r:r + n], low[:, r + n:], W[p + "D"])
    return (y * silu(z)) @ W[p + "o"].T


def scaled_parallel(h, W, p, c):
    return (c["left_scale"] * window_attention(h, W, p + "left.", c["left"])
            + c["right_scale"] * mamba(h, W, p + "right.", c["right"]))


def choose_by_sigmoid(z, r):
    """Router logits of one token -> list of (expert, weight): groups by the sum of their two best scores, weights
    normalised over the chosen experts."""
    s = torch.sigmoid(z)
    g = r.get("groups") or {"count": 1, "keep": 1}
    size = r["experts"] // g["count"]
    score = s.tolist()
    rank = lambda i: sum(sorted(score[i * size:(i + 1) * size])[-2:])
    best = sorted(range(g["count"]), key=lambda i: -rank(i))[: g["keep"]]
    allowed = [e for e in range(r["experts"]) if e // size in best]
    picked = sorted(allowed, key=lambda e: -score[e])[: r["top"]]
    total = sum(s[e] for e in picked) + 1e-20
    return [(e, s[e] / total * r["scale"]) for e in picked]


def sigmoid_moe(h, W, p, c):
    z = h @ W[p + "router"].T
    out = dense_ff(h, W, p + "shared.") if c.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in choose_by_sigmoid(z[t], c["router"]):
            out[t] += w * dense_ff(h[t:t + 1], W, p + f"e{e}.")[0]
    return out


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def forward_dogozen(cfg, W, tokens, dtype=torch.float64, trace=None):
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kv = {}
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm_around_zero(x, W[p + "norm1"], eps)
        y = (tempered_attention(h, W, p + "mix.", L["mixer"], eps, kv) if L["type"] == "attention"
             else scaled_parallel(h, W, p + "mix.", L["mixer"]))
        x = x + rms_norm_around_zero(y, W[p + "norm1b"], eps)
        if L["mlp"] is not None:
            h = rms_norm_around_zero(x, W[p + "norm2"], eps)
            y = sigmoid_moe(h, W, p + "mlp.", L["mlp"]) if L["mlp"]["kind"] == "moe" else dense_ff(h, W, p + "mlp.")
            x = x + rms_norm_around_zero(y, W[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x)
    return soft_cap(rms_norm_around_zero(x, W["final.norm"], eps) @ W["embed"].T, cfg["logit_softcap"])


# ------------------------------------------------------------------ Zigivik
def one_number_norm(x, g, eps):
    return rms(x, eps) * g


def input_conv(h, w):
    """What a mixer reads: h plus a causal convolution of it per channel."""
    return h + short_conv(h, w)


def yarn_frequencies(r):
    """(angle per position of every rotated pair, factor of cosines and sines). Pairs up to the one that turns ``fast``
    times within ``original`` positions keep their frequency, those from the one that turns ``slow`` times on are
    slowed by ``factor``, with a linear ramp over the pair's number between."""
    n, base, sc = r["dims"], float(r["base"]), r.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return f, 1.0
    pair = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair(sc["fast"])), 0), min(math.ceil(pair(sc["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / sc["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1


def turn_halves(x, pos, r):
    """Components i and i + dims / 2 of x [T, heads, n] turn together, with yarn_frequencies; the rest stays."""
    out, half = x.clone(), r["dims"] // 2
    freq, amp = yarn_frequencies(r)
    for i, f in enumerate(freq):
        a = pos.to(torch.float64) * f
        c, s = (amp * torch.cos(a)).to(x.dtype)[:, None], (amp * torch.sin(a)).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


def turn_pairs(x, pos, r):
    """Components 2i and 2i + 1 of the first ``dims`` of x [T, heads, n] turn together; the rest stays."""
    out = x.clone()
    out[..., : r["dims"]] = rotate_pairs(x[..., : r["dims"]], pos, r["base"])
    return out


def banded_attention(q, k, v, scale, window=None, plus_one=False):
    """Query i sees keys j <= i, with ``window`` only those with i - j < window; ``plus_one``: one is added to the
    denominator. q [T, H, dk]; k [T, G, dk]; v [T, G, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    i = torch.arange(T)
    hidden = i[None, :] > i[:, None]
    if window is not None:
        hidden = hidden | (i[:, None] - i[None, :] >= window)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(hidden, float("-inf"))
        m = s.max(-1, keepdim=True).values
        if plus_one:
            m = torch.clamp(m, min=0.0)
        e = torch.exp(s - m)
        out[:, h] = (e @ v[:, g]) / (e.sum(-1, keepdim=True) + (torch.exp(-m) if plus_one else 0.0))
    return out


def low_rank_queries(h, W, p, eps):
    return rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T


def window_latent_attention(h, W, p, c, eps, kept):
    """``kept`` (layer -> latent and rotated key part) receives the layer's own and gives those of a layer that shares
    them."""
    T, H, dn, dr, dv = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    pos = torch.arange(T)
    q = low_rank_queries(h, W, p, eps).view(T, H, dn + dr)
    q = torch.cat([q[..., :dn], turn_halves(q[..., dn:], pos, c["rot"])], -1)
    if c.get("kv_from") is None:
        kv = h @ W[p + "dkv"].T
        lat = rms_norm(kv[:, : c["kv_rank"]], W[p + "dkv.norm"], eps)
        kr = turn_halves(kv[:, None, c["kv_rank"]:], pos, c["rot"])[:, 0]
        kept[p] = (lat, kr)
    else:
        lat, kr = kept[f"l{c['kv_from']}.mix."]
    k = torch.cat([(lat @ W[p + "uk"].T).view(T, H, dn), kr[:, None].expand(T, H, dr)], -1)
    v = (lat @ W[p + "uv"].T).view(T, H, dv)
    o = banded_attention(q, k, v, c["scale"], (c.get("mask") or {}).get("size")).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def key_value_attention(h, W, p, c):
    """The values are the keys before their rotation."""
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    pos = torch.arange(T)
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, c["dim"])
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, c["dim"])
    o = banded_attention(turn_pairs(q, pos, c["rot"]), turn_pairs(k, pos, c["rot"]), k, c["scale"], plus_one=True)
    return o.reshape(T, H * c["vdim"]) @ W[p + "o"].T


def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def poly_ff(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T + W[p + "up.b"], W[p + "act"], eps) @ W[p + "down"].T + W[p + "down.b"]


def forward_zigivik(cfg, W, tokens, dtype=torch.float64, trace=None):
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = one_number_norm(W["embed"][torch.as_tensor(tokens, dtype=torch.long)], W["embed.norm"], eps)
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = one_number_norm(x, W[p + "norm1"], eps)
        g = input_conv(h, W[p + "canon1"])
        y = (key_value_attention(g, W, p + "mix.", L["mixer"]) if L["type"] == "attention"
             else window_latent_attention(g, W, p + "mix.", L["mixer"], eps, kept))
        if L["mlp"] is not None:
            y = y + poly_ff(h, W, p + "mlp.", eps)
        x = x + m * y
        if trace is not None:
            trace.append(x)
    return one_number_norm(x, W["final.norm"], eps) @ W["head"].T


def forward(cfg, W, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) receives the stream after every layer."""
    if cfg["architecture"] == "Lebedra":
        return forward_lebedra(cfg, W, tokens, dtype, trace)
    if cfg["architecture"] == "Dogozen":
        return forward_dogozen(cfg, W, tokens, dtype, trace)
    if cfg["architecture"] == "Zigivik":
        return forward_zigivik(cfg, W, tokens, dtype, trace)
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][tok] * cfg["embedding"]["scale"] + W["pos"][: tok.numel()]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[L["type"]](rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", L["mixer"], eps)
        x = x + rms_norm(y, W[p + "norm1b"], eps)
        if L["mlp"] is not None:
            y = dense_ff(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
            x = x + rms_norm(y, W[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]
