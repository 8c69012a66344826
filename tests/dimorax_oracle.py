"""Plain, slow statement of the Dimorax design: one function per mechanism, one whole sequence at a time, written for reading.

Shares no code with the package.  `w` maps checkpoint names to tensors (any float dtype; everything is computed in the dtype
of `embed`, so a float64 copy of the weights gives a float64 oracle); `cfg` is the parsed config.json.

The design in short.  Every layer reads the residual stream twice, through two norms of the SAME x, and adds both results with one
fixed factor: x <- x + m (mixer(norm1(x)) + ff(norm2(x))).  The norms store their weight as its distance from one.  Mixers: a gated
delta rule with a decay per head and key channel (q, k and v through short causal convolutions over time, q and k made unit
vectors), softmax attention with half-split rotary positions under YaRN scaling, soft-capped scores and a learned sink per head (a layer may
read the keys and values of an earlier attention layer), and latent attention inside a sliding window, also with sinks.  Feed-forward:
tanh-gelu gated, or a mixture of silu-gated experts with a sigmoid router limited to groups, plus a shared expert behind a gate of one
number per token.
"""
import math
from typing import Dict, List, Optional

import torch


def unit_rms(x, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, w, eps: float):
    return unit_rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


# ------------------------------------------------------------------------------------------------ rotation
def frequencies(rot: dict):
    """([dims / 2] float64 angles per position, factor on cos and sin)."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def dim_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(float(sc["fast"]))), 0), min(math.ceil(dim_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x, rot: dict):
    """x [T, heads, dim], row t at position t: entries i and i + dims / 2 turn together, entries >= dims pass unchanged."""
    f, mag = frequencies(rot)
    half = len(f)
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    c, s = (mag * ang.cos()).to(x.dtype)[:, None], (mag * ang.sin()).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


# ------------------------------------------------------------------------------------------------ mixers
def attend(q, k, v, scale: float, window: Optional[int], sink, softcap: float = 0.0):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e].  sink [H]: one more term exp(sink) in every denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = (j <= i) & (i - j < window if window is not None else torch.ones(1, dtype=torch.bool))
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~seen, -math.inf)
        m = s.max(-1, keepdim=True).values.clamp(min=sink[h])
        p = torch.exp(s - m)
        out.append((p @ v[:, g]) / (p.sum(-1, keepdim=True) + torch.exp(sink[h] - m)))
    return torch.stack(out, 1)


def attention(hs, w: Dict[str, torch.Tensor], p: str, a: dict, eps: float, kv):
    """kv: (keys after rotation, values) of an earlier layer, or None.  Returns (output, (keys, values))."""
    T = hs.shape[0]
    H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    q = rotate_halves((hs @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d), a["rot"])
    if kv is None:
        k = rotate_halves((hs @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d), a["rot"])
        kv = (k, (hs @ w[p + "v"].T + w[p + "v.b"]).view(T, G, e))
    o = attend(q, kv[0], kv[1], float(a["scale"]), None, w[p + "sink"], float(a.get("softcap") or 0.0))
    return o.reshape(T, H * e) @ w[p + "o"].T, kv


def latent_attention(hs, w: Dict[str, torch.Tensor], p: str, a: dict, eps: float):
    T = hs.shape[0]
    H, d, r, e, n = a["heads"], a["dim"], a["rot_dim"], a["vdim"], a["kv_rank"]
    rot = dict(a["rot"], dims=a["rot"].get("dims", r))
    q = (hs @ w[p + "q"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate_halves(q[..., d:], rot)], -1)
    y = hs @ w[p + "dkv"].T
    c = unit_rms(y[:, :n], eps) * w[p + "dkv.norm"]
    kr = rotate_halves(y[:, None, n:], rot)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), kr.expand(T, H, r)], -1)
    v = (c @ w[p + "uv"].T).view(T, H, e)
    mask = a.get("mask")
    o = attend(q, k, v, float(a["scale"]), int(mask["size"]) if mask else None, w[p + "sink"])
    return o.reshape(T, H * e) @ w[p + "o"].T


def causal_conv_silu(xs, taps):
    """xs [T, channels], taps [channels, n]: the last column meets the current token, nothing before the first one; then silu."""
    T, n = xs.shape[0], taps.shape[1]
    acc = torch.zeros_like(xs)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            acc[back:] = acc[back:] + taps[:, j] * xs[: T - back]
    return silu(acc)


def delta_rule(q, k, v, beta, g):
    """q, k [T, H, d], v [T, H, e], beta [T, H], g [T, H, d] -> o [T, H, e]: per head, S from zero,
    S <- diag(g) S; S <- S + k (beta (v - S^T k))^T; o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out)


def delta_decay(hs, w, p: str, H: int, d: int):
    z = (hs @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    softplus = torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus.view(-1, H, d))


def channel_delta(hs, w: Dict[str, torch.Tensor], p: str, a: dict, eps: float):
    T = hs.shape[0]
    H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    q = causal_conv_silu(hs @ w[p + "q"].T, w[p + "q.conv"]).view(T, G, d)
    k = causal_conv_silu(hs @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, d)
    v = causal_conv_silu(hs @ w[p + "v"].T, w[p + "v.conv"]).view(T, H, e)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * d ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    src = [h // (H // G) for h in range(H)]
    beta = torch.sigmoid(hs @ w[p + "b"].T)
    o = delta_rule(q[:, src], k[:, src], v, beta, delta_decay(hs, w, p, H, d))
    gate = torch.sigmoid((hs @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (unit_rms(o, eps) * w[p + "norm"]).reshape(T, H * e) * gate @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated(h, w, p: str, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p: str, r: dict):
    """[(expert, weight)] of one token h [width]."""
    s = torch.sigmoid(w[p + "router"] @ h)
    choice = (s + w[p + "correction"]).tolist()
    E, grp = int(r["experts"]), r.get("groups") or {"count": 1, "keep": 1}
    n, size = int(grp["count"]), E // int(grp["count"])
    score = [sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(n)]
    best = sorted(range(n), key=lambda g: -score[g])[: int(grp["keep"])]
    allowed = [e for e in range(E) if e // size in best]
    chosen = sorted(allowed, key=lambda e: -choice[e])[: int(r["top"])]
    total = sum(s[e] for e in chosen) + 1e-20
    return [(e, s[e] / total * float(r.get("scale", 1.0))) for e in chosen]


def moe(hs, w, p: str, f: dict):
    out = []
    for t in range(hs.shape[0]):
        out.append(sum(wt * gated(hs[t], w, f"{p}e{e}.", silu) for e, wt in route(hs[t], w, p, f["router"])))
    y = torch.stack(out)
    if f.get("shared"):
        y = y + torch.sigmoid(hs @ w[p + "shared.sg"].T) * gated(hs, w, p + "shared.", silu)
    return y


# ------------------------------------------------------------------------------------------------ model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None, mixer_taps: Optional[list] = None):
    """Logits [T, vocab] of one sequence.  taps: gets the stream after every layer; mixer_taps: the raw mixer outputs."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][torch.tensor(tokens)]
    kvs: Dict[int, tuple] = {}
    for i, L in enumerate(cfg["layers"]):
        p, a = f"l{i}.", L["mixer"]
        h = norm_around_one(x, w[p + "norm1"], eps)
        if L["type"] == "attention":
            y, kv = attention(h, w, p + "mix.", a, eps, kvs[a["kv_from"]] if a.get("kv_from") is not None else None)
            kvs[i] = kv
        else:
            y = {"latent_attention": latent_attention, "channel_delta": channel_delta}[L["type"]](h, w, p + "mix.", a, eps)
        if mixer_taps is not None:
            mixer_taps.append(y)
        f = L.get("mlp")
        if f:
            h2 = norm_around_one(x, w[p + "norm2"], eps)
            y = y + (moe(h2, w, p + "mlp.", f) if f["kind"] == "moe" else gated(h2, w, p + "mlp.", gelu_tanh))
        x = x + m * y
        if taps is not None:
            taps.append(x)
    return norm_around_one(x, w["final.norm"], eps) @ w["head"].T
