"""Plain, slow statement of the Pukarax design: one function per mechanism, one whole sequence at a time, written for reading.

Shares no code with the package.  `w` maps checkpoint names to tensors (any float dtype; everything is computed in the dtype
of `embed`, so a float64 copy of the weights gives a float64 oracle); `cfg` is the parsed config.json.

The design in short.  Every sublayer reads the normed stream and is normed again before it is added.  Both mixers are softmax attention
inside chunks of fixed size: a token sees the keys of its own chunk up to itself.  "attention" takes the difference of two softmax maps over
one set of values (a weighted difference, each head then brought to unit root mean square), with biases on its four projections, rotary
positions on neighbouring entries and a sigmoid gate of one number per head.  "attention_2" has no value projection -- the raw key
projection is also the value -- and turns entry i with entry i + dims / 2 at slowed-down positions, brings every rotated query and key to unit
root mean square and gates every entry of its output.  Feed-forward: silu-gated, or a mixture of such experts weighted by a softmax over the
chosen logits, plus a shared expert.  A span of layers may run several times; the head is the embedding table.
"""
import math
from typing import Dict, List, Optional

import torch


def unit_rms(x, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps: float):
    return unit_rms(x, eps) * w


def silu(x):
    return x * torch.sigmoid(x)


# ------------------------------------------------------------------------------------------------ rotation
def turn(u, v, angle):
    c, s = angle.cos().to(u.dtype), angle.sin().to(u.dtype)
    return u * c - v * s, v * c + u * s


def angles(T: int, rot: dict, slow: float = 1.0):
    """float64 [T, 1, dims / 2]"""
    n = int(rot["dims"]) // 2
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / int(rot["dims"])) / slow for i in range(n)], dtype=torch.float64)
    return (torch.arange(T, dtype=torch.float64)[:, None] * f)[:, None]


def rotate_neighbours(x, rot: dict):
    """x [T, heads, dim], row t at position t: entries 2i and 2i + 1 turn together."""
    n = int(rot["dims"])
    out = x.clone()
    out[..., 0:n:2], out[..., 1:n:2] = turn(x[..., 0:n:2], x[..., 1:n:2], angles(x.shape[0], rot))
    return out


def rotate_halves(x, rot: dict):
    """Entries i and i + dims / 2 turn together, every frequency divided by the scaling factor."""
    n = int(rot["dims"])
    out = x.clone()
    out[..., :n // 2], out[..., n // 2:n] = turn(x[..., :n // 2], x[..., n // 2:n], angles(x.shape[0], rot, float((rot.get("scaling") or {}).get("factor", 1.0))))
    return out


# ------------------------------------------------------------------------------------------------ mixers
def softmax_map(q, k, v, scale: float, size: Optional[int]):
    """q, k [T, d], v [T, e] of one head: token i averages the values of the keys j <= i in its own chunk of `size` positions."""
    i, j = torch.arange(q.shape[0])[:, None], torch.arange(q.shape[0])[None]
    seen = j <= i
    if size is not None:
        seen = seen & (i // size == j // size)
    return torch.softmax(((q @ k.T) * scale).masked_fill(~seen, -math.inf), -1) @ v


def mix_size(a: dict) -> Optional[int]:
    return int(a["mask"]["size"]) if a.get("mask") else None


def lam_of(w, p: str, diff: float):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def difference(a1, a2, lam, diff: float, eps: float):
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention(hs, w: Dict[str, torch.Tensor], p: str, a: dict, eps: float):
    T, H, G, d, e = hs.shape[0], a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    q = rotate_neighbours((hs @ w[p + "q"].T + w[p + "q.b"]).view(T, H * 2, d), a["rot"]).view(T, H, 2, d)
    k = rotate_neighbours((hs @ w[p + "k"].T + w[p + "k.b"]).view(T, G * 2, d), a["rot"]).view(T, G, 2, d)
    v = (hs @ w[p + "v"].T + w[p + "v.b"]).view(T, G, e)
    lam, gate = lam_of(w, p, a["diff"]), torch.sigmoid(hs @ w[p + "g"].T)
    out = []
    for h in range(H):
        g = h // (H // G)
        a1, a2 = (softmax_map(q[:, h, m], k[:, g, m], v[:, g], a["scale"], mix_size(a)) for m in (0, 1))
        out.append(difference(a1, a2, lam, a["diff"], eps) * gate[:, h:h + 1])
    return torch.cat(out, -1) @ w[p + "o"].T + w[p + "o.b"]


def attention_2(hs, w: Dict[str, torch.Tensor], p: str, a: dict, eps: float):
    T, H, G, d = hs.shape[0], a["heads"], a["kv_heads"], a["dim"]
    v = (hs @ w[p + "k"].T).view(T, G, d)
    q = unit_rms(rotate_halves((hs @ w[p + "q"].T).view(T, H, d), a["rot"]), eps)
    k = unit_rms(rotate_halves(v, a["rot"]), eps)
    out = [softmax_map(q[:, h], k[:, h // (H // G)], v[:, h // (H // G)], a["scale"], mix_size(a)) for h in range(H)]
    return (torch.cat(out, -1) * torch.sigmoid(hs @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"attention": attention, "attention_2": attention_2}


# ------------------------------------------------------------------------------------------------ feed-forward
def gated(hs, w: Dict[str, torch.Tensor], p: str):
    return (silu(hs @ w[p + "gate"].T) * (hs @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w: Dict[str, torch.Tensor], p: str, r: dict):
    """[(expert, weight)] of one token, the largest logit first."""
    z = w[p + "router"] @ h + w[p + "router.b"]
    order = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[: r["top"]]
    total = sum(math.exp(float(z[e] - z[order[0]])) for e in order)
    return [(e, math.exp(float(z[e] - z[order[0]])) / total) for e in order]


def moe(hs, w: Dict[str, torch.Tensor], p: str, f: dict):
    rows = []
    for h in hs:
        y = sum(s * gated(h[None], w, f"{p}e{e}.")[0] for e, s in route(h, w, p, f["router"]))
        rows.append(y + (gated(h[None], w, p + "shared.")[0] if f.get("shared") else 0.0))
    return torch.stack(rows)


def feed_forward(hs, w: Dict[str, torch.Tensor], p: str, f: dict):
    return gated(hs, w, p) if f["kind"] == "dense" else moe(hs, w, p, f)


# ------------------------------------------------------------------------------------------------ model
def layer_order(cfg: dict) -> List[int]:
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None):
    """Logits [T, vocab] of one sequence from position 0; `taps` collects the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i in layer_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        x = x + norm(MIXERS[L["type"]](norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps), w[p + "norm1b"], eps)
        if L.get("mlp"):
            x = x + norm(feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"]), w[p + "norm2b"], eps)
        if taps is not None:
            taps.append(x)
    return norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
