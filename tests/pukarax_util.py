"""Small random Pukarax models for the tests: configurations, weights with the checkpoint's names, folders on disk."""
import json
import math
from pathlib import Path
from typing import Dict, Optional, Tuple

import torch


def diff_cfg(heads=4, kv_heads=2, dim=6, vdim=10, scale=0.5, rot=(1000.0, 4), size: Optional[int] = 7, diff=0.35) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": rot[0], "dims": rot[1]}, "diff": diff}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "attention", "mixer": m}


def keyval_cfg(heads=3, kv_heads=1, dim=12, scale=0.4, rot=(300.0, 8), factor: Optional[float] = 2.5, size: Optional[int] = 5) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": {"base": rot[0], "dims": rot[1]}}
    if factor is not None:
        m["rot"]["scaling"] = {"factor": factor}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "attention_2", "mixer": m}


def dense_cfg(ff=24) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_cfg(ff=12, experts=6, top=2, shared: Optional[int] = 20) -> dict:
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def make_config(width=40, vocab=50, layers=None, eps=1e-4, embed_scale=1.7, logit_scale=0.8, loop: Optional[Tuple[int, int, int]] = None) -> dict:
    """layers: list of (mixer entry from diff_cfg / keyval_cfg, mlp dict or None)."""
    cfg = {"architecture": "Pukarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "logit_scale": logit_scale,
           "layers": [{"type": m["type"], "mixer": m["mixer"], "mlp": f} for m, f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def make_weights(cfg: dict, seed: int = 0, dtype=torch.float32, router_gain: float = 4.0) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * s / math.sqrt(i)).to(dtype)

    def vec(n, mean=0.0, s=0.3):
        return (mean + s * torch.randn(n, generator=g)).to(dtype)

    def glu(q, ff):
        w[q + "gate"], w[q + "up"], w[q + "down"] = mat(ff, W, 2.0), mat(ff, W, 2.0), mat(W, ff)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g).to(dtype), "final.norm": vec(W, 1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[f"l{i}.norm1"], w[f"l{i}.norm1b"] = vec(W, 1.0), vec(W, 0.7)
        if L["type"] == "attention":
            for n, rows in (("q", 2 * H * d), ("k", 2 * G * d), ("v", G * e)):
                w[p + n], w[p + n + ".b"] = mat(rows, W, 1.5), vec(rows)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + n] = vec(d, 0.0, 0.4)
            w[p + "g"], w[p + "o"], w[p + "o.b"] = mat(H, W, 2.0), mat(W, H * e, 2.0), vec(W)
        else:
            w[p + "q"], w[p + "k"] = mat(H * d, W, 1.5), mat(G * d, W, 1.5)
            w[p + "g"], w[p + "o"] = mat(H * d, W, 2.0), mat(W, H * d, 2.0)
        f = L["mlp"]
        if f:
            q = f"l{i}.mlp."
            w[f"l{i}.norm2"], w[f"l{i}.norm2b"] = vec(W, 1.0), vec(W, 0.7)
            if f["kind"] == "dense":
                glu(q, f["ff"])
                continue
            E = f["router"]["experts"]
            w[q + "router"], w[q + "router.b"] = mat(E, W, router_gain), vec(E, 0.0, 1.5)
            for e in range(E):
                glu(f"{q}e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                glu(q + "shared.", f["shared"]["ff"])
    return w


def write_folder(path: Path, cfg: dict, weights: Dict[str, torch.Tensor]) -> Path:
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(path / "model.safetensors"))
    return path


def f32(weights: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    return {k: v.float() for k, v in weights.items()}
