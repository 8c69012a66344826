"""Small random Dimorax models for the tests: configurations, weights with the checkpoint's names, folders on disk."""
import json
import math
from pathlib import Path
from typing import Dict, Optional

import torch


def attn_cfg(heads=4, kv_heads=2, dim=12, vdim=10, scale=0.4, rot=(1000.0, 8), scaling=(3.0, 64, 6.0, 1.5), softcap=7.0, kv_from: Optional[int] = None) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": rot[0], "dims": rot[1]}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if softcap:
        m["softcap"] = softcap
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def latent_cfg(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=14, scale=0.35, base=300.0, window: Optional[int] = 5) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m}


def delta_cfg(heads=4, kv_heads=2, dim=12, vdim=10, conv=3, ranks=(5, 7)) -> dict:
    # `ranks` are not part of config.json (the checkpoint's tensors give them)
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "_ranks": ranks}


def dense_cfg(ff=24) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_cfg(ff=12, experts=6, top=2, groups=3, keep=2, scale=1.7, shared: Optional[int] = 20) -> dict:
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def make_config(width=40, vocab=50, layers=None, eps=1e-4, mult=0.6) -> dict:
    """layers: list of (mixer entry from attn_cfg / latent_cfg / delta_cfg, mlp dict or None)."""
    cfg = {"architecture": "Dimorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
           "layers": [{"type": m["type"], "mixer": m["mixer"], "mlp": f} for m, f in layers]}
    cfg["_ranks"] = [m.get("_ranks") for m, _ in layers]
    return cfg


def on_disk(cfg: dict) -> dict:
    return {k: v for k, v in cfg.items() if not k.startswith("_")}


def make_weights(cfg: dict, seed: int = 0, dtype=torch.float32, router_gain: float = 4.0, long_memory: bool = False) -> Dict[str, torch.Tensor]:
    """long_memory: decays close to 1, so that what a state took in hundreds of tokens ago still shows in the output."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * s / math.sqrt(i)).to(dtype)

    def vec(n, mean=0.0, s=0.3):
        return (mean + s * torch.randn(n, generator=g)).to(dtype)

    def glu(q, ff):
        w[q + "gate"], w[q + "up"], w[q + "down"] = mat(ff, W, 2.0), mat(ff, W, 2.0), mat(W, ff)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g).to(dtype), "final.norm": vec(W), "head": mat(cfg["vocab"], W, 3.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        w[f"l{i}.norm1"] = vec(W)
        H = m["heads"]
        if L["type"] == "attention":
            G, d, e = m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * d),) + ((("k", G * d), ("v", G * e)) if m.get("kv_from") is None else ()):
                w[p + n], w[p + n + ".b"] = mat(rows, W, 1.5), vec(rows)
            w[p + "sink"], w[p + "o"] = vec(H, 1.0, 1.0), mat(W, H * e, 2.0)
        elif L["type"] == "latent_attention":
            d, r, e, n = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w[p + "q"], w[p + "dkv"], w[p + "dkv.norm"] = mat(H * (d + r), W, 1.5), mat(n + r, W, 1.5), vec(n, 1.0)
            w[p + "uk"], w[p + "uv"] = mat(H * d, n, 1.5), mat(H * e, n, 1.5)
            w[p + "sink"], w[p + "o"] = vec(H, 1.0, 1.0), mat(W, H * e, 2.0)
        else:
            G, d, e, taps = m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            ra, rg = cfg["_ranks"][i]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                w[p + n], w[p + n + ".conv"] = mat(rows, W, 2.0), (0.6 * torch.randn(rows, taps, generator=g)).to(dtype)
            w[p + "b"], w[p + "a1"], w[p + "a2"], w[p + "g1"], w[p + "g2"] = mat(H, W, 2.0), mat(ra, W), mat(H * d, ra), mat(rg, W, 2.0), mat(H * e, rg, 2.0)
            w[p + "A_log"], w[p + "dt_bias"] = vec(H, -4.0 if long_memory else -0.5, 0.5), vec(H * d, -3.0 if long_memory else -1.0, 0.5)
            w[p + "norm"], w[p + "o"] = vec(e, 1.0), mat(W, H * e, 2.0)
        f = L["mlp"]
        if f:
            q = f"l{i}.mlp."
            w[f"l{i}.norm2"] = vec(W)
            if f["kind"] == "dense":
                glu(q, f["ff"])
                continue
            E = f["router"]["experts"]
            w[q + "router"], w[q + "correction"] = mat(E, W, router_gain), vec(E, -0.4, 0.3)  # many choice scores below zero
            for e in range(E):
                glu(f"{q}e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                glu(q + "shared.", f["shared"]["ff"])
                w[q + "shared.sg"] = mat(1, W, 2.0)
    return w


def write_folder(path: Path, cfg: dict, weights: Dict[str, torch.Tensor]) -> Path:
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(on_disk(cfg)))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(path / "model.safetensors"))
    return path


def f32(weights: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    return {k: v.float() for k, v in weights.items()}
