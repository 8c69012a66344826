"""`bench.py --design fesenex|taruvik|lotazen|viladra|dimorax|pukarax`: prefill and decode throughput of the layered decoder at layer sizes of real models (random
weights), beside the dense `Transformer` of equal width / heads / feed-forward size / depth / vocabulary, plus the time of each
hybrid kernel at those shapes against its roofline (bf16 tensor peak or HBM copy bandwidth from MEASURED_PEAKS.json).
For `taruvik` (latent attention, mixture of experts) the neighbour is the `Transformer` with a mixture of experts of equal
width / heads / experts / depth; for `lotazen` (rotary window attention beside a gated recurrence, matrix memories, experts with scaled
input) it is the Fesenex design at equal width / heads / depth, and every new kernel is timed next to the like kernel at the same shape;
for `viladra` (convolution on the stream, norms after the sublayers with a depth average, retention, gated linear attention,
sigmoid-weight window attention, ungated experts) the neighbour is the Lotazen design at equal width / heads / experts / depth; for
`dimorax` (gated delta rule, soft-capped attention with sinks, windowed latent attention, group-limited experts) too; for `pukarax` (differential attention and attention
with keys as values, both inside chunks, softmax over the chosen experts) it is the Dimorax design with rotary attention in every layer.  Timed with CUDA events after warm-up; the prompt batch and the weights exceed L2 at the larger size, and L2 is flushed between
timed kernel launches.  Prints one JSON line."""
import json
import math
import time

import torch

SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, ff=8192, vocab=32768, layers=8, lin_heads=16),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, ff=14336, vocab=32768, layers=4, lin_heads=32),
}


def layered_config(s: dict) -> dict:
    att = {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
                                          "bias_max": 4096, "q_temp": {"coef": 0.1, "every": 1024}, "v_mix": True},
           "mlp": {"kind": "dense", "ff": s["ff"], "limit": 7.0}}
    lin = {"type": "lightning", "mixer": {"heads": s["lin_heads"], "dim": s["dim"], "vdim": s["dim"],
                                          "decay": [math.exp(-1.0 / (4 + 8 * h)) for h in range(s["lin_heads"])]},
           "mlp": {"kind": "dense", "ff": s["ff"], "limit": 7.0}}
    return {"architecture": "Fesenex", "vocab": s["vocab"], "width": s["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5},
            "layers": [lin if (i in s["lightning_at"] if "lightning_at" in s else i % 4 == 3) else att for i in range(s["layers"])]}


def build_layered(s: dict, dev):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer
    from mistral_inference_b200.transformer_layers import BiasedAttention

    m = LayeredTransformer.empty(LayeredArgs.from_dict(layered_config(s)), dev, torch.bfloat16)
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for blk in m.layers:
            if isinstance(blk.mix, BiasedAttention):
                blk.mix.rel = torch.nn.Parameter(torch.empty(32, blk.mix.a.heads, dtype=torch.bfloat16, device=dev), requires_grad=False)
        for n, p in m.named_parameters():
            if p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            elif "norm" in n:
                p.fill_(1.0)
            else:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.1)
    return m.eval()


def build_dense(s: dict, dev):
    import mistral_inference_b200 as mi
    from mistral_inference_b200.transformer import Transformer

    args = mi.TransformerArgs(dim=s["width"], n_layers=s["layers"], head_dim=s["dim"], hidden_dim=s["ff"], n_heads=s["heads"], n_kv_heads=s["kv_heads"],
                              norm_eps=1e-5, vocab_size=s["vocab"], max_batch_size=8)
    m = Transformer.empty(args, dev, torch.bfloat16)
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            if p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            else:
                p.fill_(1.0)
    return m.eval()


def _time(fn, warmup: int, steps: int, flush=None) -> float:
    """Median milliseconds of fn() over `steps` runs."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(steps):
        if flush is not None:
            flush.add_(1.0)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    ts.sort()
    return ts[len(ts) // 2]


def _experts_used(idx) -> int:
    """Experts that some token of the step chose: each one's weights have to be read once."""
    return len(set(idx.flatten().tolist()))


def end_to_end(model, vocab: int, T: int, ctx: int, batches, warmup: int, steps: int, dev) -> dict:
    out = {}
    ids = torch.randint(0, vocab, (T,), device=dev)
    cache = model.make_cache(max(batches), ctx + 64 + warmup + steps)

    def prefill():
        cache.reset()
        model.forward(ids, [T], cache)

    ms = _time(prefill, max(3, warmup // 4), max(3, steps // 8))
    out["prefill"] = {"tokens": T, "ms": round(ms, 3), "tok_s": round(T / ms * 1e3, 1)}
    for B in batches:
        cache.reset()
        n = ctx // 2 if B > 1 else ctx
        model.forward(ids[:n].repeat(B), [n] * B, cache)
        tok = torch.randint(0, vocab, (B,), device=dev)
        ms = _time(lambda: model.next_token_logits(tok, cache), warmup, steps)
        out[f"decode_b{B}"] = {"context": n, "ms": round(ms, 4), "tok_s": round(B / ms * 1e3, 1)}
    return out


def kernel_table(s: dict, T: int, ctx: int, peaks: dict, dev) -> dict:
    """Every hybrid kernel alone at this size: time, achieved rate, fraction of the measured roofline."""
    from mistral_inference_b200 import _abi_hybrid as h

    bf = torch.bfloat16
    W, H, G, d, ff = s["width"], s["heads"], s["kv_heads"], s["dim"], s["ff"]
    flush = torch.zeros(160 << 20, dtype=torch.float32, device=dev)  # 640 MB > L2
    rows = {}

    def rec(name, ms, flops=0.0, bytes_=0.0):
        r = {"ms": round(ms, 4)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["of_bf16_peak"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 3)
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["of_hbm_peak"] = round(bytes_ / ms / 1e6 / peaks["hbm_gbs"], 3)
        rows[name] = r

    x = torch.randn(T, W, device=dev).to(bf)
    w13 = torch.randn(2 * ff, W, device=dev).to(bf) * 0.02
    rec("prompt linear gate/up+glu (tcgen05 GEMM + epilogue pass)", _time(lambda: h.linear(x, w13, epi=h.EPI_GLU, limit=7.0, alpha=1.702), 3, 8, flush), flops=2.0 * T * 2 * ff * W)
    for M in (1, 8):
        xs = x[:M].contiguous()
        rec(f"linear_skinny gate/up+glu M={M}", _time(lambda: h.linear(xs, w13, epi=h.EPI_GLU, limit=7.0, alpha=1.702), 3, 8, flush), bytes_=w13.numel() * 2.0)
    # attention: a prompt of T tokens, then one token per sequence at context ctx
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec
    B = 8
    cache = BufferCache(1, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d)]).to(dev, bf)
    cache.cache_k[0].normal_(); cache.cache_v[0].normal_()
    tab = torch.zeros(64, H, device=dev)
    md = cache.get_input_metadata([T])[0]
    q = torch.randn(T, H * d, device=dev).to(bf)
    o = torch.empty_like(q)
    att = lambda: h.attn_bias(q, cache.cache_k[0], cache.cache_v[0], tab, md.positions, md.q_start, md.slots, o, 1, ctx + 8, H, G, d, d, d ** -0.5,
                              n_tiles=(T + 63) // 64)  # noqa: E731
    rec("attn_bias_flash prompt", _time(att, 2, 5, flush), flops=4.0 * d * H * T * (T + 1) / 2)
    cache.reset(); cache.init_kvseqlens(B); cache.update_seqlens([ctx] * B)
    md2 = cache.get_input_metadata([1] * B)[0]
    q2, o2 = q[:B].contiguous(), torch.empty(B, H * d, device=dev, dtype=bf)
    dec = lambda: h.attn_bias(q2, cache.cache_k[0], cache.cache_v[0], tab, md2.positions, md2.q_start, md2.slots, o2, B, ctx + 8, H, G, d, d, d ** -0.5,
                              splits=h.attn_splits(B, H, ctx + 8))  # noqa: E731
    rec(f"attn_bias decode B={B} ctx={ctx}", _time(dec, 3, 8, flush), bytes_=2.0 * B * (ctx + 1) * G * d * 2)
    # lightning: prompt and decode
    LH = s["lin_heads"]
    qkvg = torch.randn(T, 4 * LH * d, device=dev).to(bf) * 0.1
    state = torch.zeros(B, LH, d, d, device=dev)
    dec_ = torch.full((LH,), 0.97, device=dev)
    o32 = torch.empty(T, LH * d, device=dev)
    zero = torch.zeros(1, dtype=torch.int32, device=dev)
    rec("lightning_scan prompt", _time(lambda: h.lightning_scan(qkvg, state, dec_, md.q_start, zero, md.slots, o32, 1, LH, d, d), 2, 5, flush),
        flops=4.0 * T * LH * d * d)
    one = torch.ones(B, dtype=torch.int32, device=dev)
    rec(f"lightning_scan decode B={B}", _time(lambda: h.lightning_scan(qkvg, state, dec_, md2.q_start, one, md2.slots, o32, B, LH, d, d), 3, 8, flush),
        bytes_=2.0 * state.numel() * 4)
    return rows


# ----------------------------------------------------------------------------------------------- Taruvik
TARUVIK_SIZES = {
    "w2048": dict(width=2048, heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512, experts=16, identity=4, top=4, groups=4, keep=2,
                  ff=1408, vocab=32768, layers=4),
    "w4096": dict(width=4096, heads=32, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512, experts=8, identity=0, top=2, groups=1, keep=1,
                  ff=14336, vocab=32768, layers=2),
}


def taruvik_config(s: dict) -> dict:
    mix = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot_dim"], "vdim": s["vdim"], "q_rank": s["q_rank"], "kv_rank": s["kv_rank"],
           "scale": (s["dim"] + s["rot_dim"]) ** -0.5,
           "rot": {"base": 10000.0, "dims": s["rot_dim"], "scaling": {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]},
           "router": {"experts": s["experts"], "identity": s["identity"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["keep"]}}}
    return {"architecture": "Taruvik", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5},
            "layers": [{"type": "latent_attention", "mixer": mix, "mlp": mlp} for _ in range(s["layers"])]}


def build_taruvik(s: dict, dev):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer

    m = LayeredTransformer.empty(LayeredArgs.from_dict(taruvik_config(s)), dev, torch.bfloat16)
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            if p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            elif n.endswith("weight") or "norm" in n.rsplit(".", 1)[-1]:
                p.fill_(1.0)
            else:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.01)
    return m.eval()


def build_moe_transformer(s: dict, dev):
    import mistral_inference_b200 as mi
    from mistral_inference_b200.args import MoeArgs
    from mistral_inference_b200.transformer import Transformer

    args = mi.TransformerArgs(dim=s["width"], n_layers=s["layers"], head_dim=s["dim"], hidden_dim=s["ff"], n_heads=s["heads"], n_kv_heads=s["heads"],
                              norm_eps=1e-5, vocab_size=s["vocab"], max_batch_size=8, moe=MoeArgs(num_experts=s["experts"], num_experts_per_tok=s["top"]))
    m = Transformer.empty(args, dev, torch.bfloat16)
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            if p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            else:
                p.fill_(1.0)
    return m.eval()


def taruvik_kernel_table(s: dict, T: int, ctx: int, peaks: dict, dev) -> dict:
    """Every kernel that the design added, alone at this size: time, achieved rate, fraction of the measured roofline (bytes and
    FLOPs are the algorithm's: what a perfect kernel would have to move or compute)."""
    from mistral_inference_b200 import _abi_hybrid as h
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec
    from mistral_inference_b200.rope import scaled_frequencies

    bf = torch.bfloat16
    W, H, dn, dr, dv, rq, rk, E, ff, top = (s[k] for k in ("width", "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "experts", "ff", "top"))
    n_routed = E + s["identity"]
    flush = torch.zeros(160 << 20, dtype=torch.float32, device=dev)
    rows = {}

    def rec(name, ms, flops=0.0, bytes_=0.0, note=None):
        r = {"ms": round(ms, 4)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 1)
            r["of_bf16_peak"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 3)
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["of_hbm_peak"] = round(bytes_ / ms / 1e6 / peaks["hbm_gbs"], 3)
        if note:
            r["note"] = note
        rows[name] = r

    B = 8
    x32 = torch.randn(T, W, device=dev)
    wv, bv = torch.ones(W, device=dev).to(bf), torch.zeros(W, device=dev).to(bf)
    rec("layernorm prompt", _time(lambda: h.layernorm(x32, wv, bv, 1e-5), 3, 8, flush), bytes_=T * W * 6.0)
    acc = torch.zeros(T, W, device=dev)
    rec("layernorm + residual add prompt", _time(lambda: h.layernorm(x32, wv, bv, 1e-5, add_to=acc), 3, 8, flush), bytes_=T * W * 12.0)
    # latent attention
    freq, mag = scaled_frequencies(dr, 10000.0, None)
    freq = freq.to(dev)
    n_in = rq + rk + dr + H
    cache = BufferCache(1, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=1, k_dim=rk + dr, v_dim=0)]).to(dev, bf)
    cache.cache_k[0].normal_()
    md = cache.get_input_metadata([T])[0]
    y = torch.randn(T, n_in, device=dev).to(bf)
    qn, cn = torch.ones(rq, device=dev).to(bf), torch.ones(rk, device=dev).to(bf)
    rec("latent_prep prompt", _time(lambda: h.latent_prep(y, qn, cn, freq, md.positions, md.cache_rows, cache.cache_k[0], rq, rk, dr, dr, 1e-5, mag), 3, 8, flush),
        bytes_=T * (n_in + rq + rk + dr) * 2.0)
    q = torch.randn(T, H * (dn + dr), device=dev).to(bf)
    w_uk = (torch.randn(H * dn, rk, device=dev) / math.sqrt(rk)).to(bf)
    rec("latent_absorb prompt", _time(lambda: h.latent_absorb(q, w_uk, freq, md.positions, H, dn, dr, dr, rk, mag), 2, 5, flush), flops=2.0 * T * H * dn * rk)
    qa = torch.randn(T, H * (rk + dr), device=dev).to(bf)
    Tp = min(T, 1024)  # the exact kernel on a prompt: a shorter one keeps the run short
    mdp = cache.get_input_metadata([Tp])[0]
    qp = qa[:Tp].contiguous()
    rec(f"attn_latent (latent form, portions of prompts and fp32) T={Tp}", _time(lambda: h.attn_latent(qp, cache.cache_k[0], mdp.positions, mdp.q_start, mdp.slots, 1, ctx + 8, H, rk, dr, 0.07,
                                                                 splits=h.attn_splits(Tp, H, ctx + 8)), 1, 3, flush),
        flops=2.0 * H * (2 * rk + dr) * Tp * (Tp + 1) / 2, note="exact fp32 FMA kernel, no tensor cores")
    cache.reset(); cache.init_kvseqlens(B); cache.update_seqlens([ctx] * B)
    md2 = cache.get_input_metadata([1] * B)[0]
    q2 = qa[:B].contiguous()
    rec(f"attn_latent (a CTA per head) decode B={B} ctx={ctx}", _time(lambda: h.attn_latent(q2, cache.cache_k[0], md2.positions, md2.q_start, md2.slots, B, ctx + 8, H, rk, dr, 0.07,
                                                                            splits=h.attn_splits(B, H, ctx + 8)), 3, 8, flush),
        bytes_=B * (ctx + 1) * (rk + dr) * 2.0, note="bytes: every latent row once; each head's CTAs re-read them through L2")
    rec(f"attn_latent_decode (rows shared by the heads) B={B} ctx={ctx}",
        _time(lambda: h.attn_latent_decode(q2, cache.cache_k[0], md2.positions, md2.slots, B, ctx + 8, H, rk, dr, 0.07), 3, 8, flush),
        bytes_=B * (ctx + 1) * (rk + dr) * 2.0)
    if (dn + dr, dv) in h.FLASH_SIZES:  # whole prompts: multi-head attention over written-out keys and values
        kf = torch.randn(T, H, dn + dr, device=dev).to(bf)
        vf = torch.randn(T, H, dv, device=dev).to(bf)
        qr = torch.randn(T, H * (dn + dr), device=dev).to(bf)
        of = torch.empty(T, H * dv, device=dev, dtype=bf)
        rec(f"prompt attention over written-out keys (attn_bias_flash, {dn + dr}/{dv}) T={T}",
            _time(lambda: h.attn_bias(qr, kf, vf, None, md.positions, md.q_start, h.iota(1, dev), of, 1, T, H, H, dn + dr, dv, 0.07, n_tiles=(T + 63) // 64), 2, 5, flush),
            flops=2.0 * H * (dn + dr + dv) * T * (T + 1) / 2)
    o_lat = torch.randn(T, H * rk, device=dev).to(bf)
    w_uv = (torch.randn(H * dv, rk, device=dev) / math.sqrt(rk)).to(bf)
    rec("latent_vup prompt", _time(lambda: h.latent_vup(o_lat, w_uv, y, n_in, rq + rk + dr, H, dv, rk), 2, 5, flush), flops=2.0 * T * H * dv * rk)
    ob = o_lat[:B].contiguous()
    rec(f"latent_vup decode B={B}", _time(lambda: h.latent_vup(ob, w_uv, y, n_in, rq + rk + dr, H, dv, rk), 3, 8, flush), bytes_=w_uv.numel() * 2.0)
    qb = q[:B].contiguous()
    rec(f"latent_absorb decode B={B}", _time(lambda: h.latent_absorb(qb, w_uk, freq, md2.positions, H, dn, dr, dr, rk, mag), 3, 8, flush), bytes_=w_uk.numel() * 2.0)
    # mixture of experts
    x = torch.randn(T, W, device=dev).to(bf)
    wr = (torch.randn(n_routed, W, device=dev) / math.sqrt(W) * 4).to(bf)
    corr = torch.zeros(n_routed, device=dev).to(bf)
    rec("moe_route prompt", _time(lambda: h.moe_route(x, wr, corr, s["groups"], s["keep"], top), 3, 8, flush), bytes_=T * W * 2.0)
    dense, idx, wsel = h.moe_route(x, wr, corr, s["groups"], s["keep"], top)
    w13 = (torch.randn(E * 2 * ff, W, device=dev) * 0.02).to(bf)
    w2 = (torch.randn(W, E * ff, device=dev) * 0.02).to(bf)

    def dense_form():
        act = h.linear_swiglu(x, w13, rowscale=dense, group=ff)
        return h.linear(act, w2, epi=h.EPI_F32)

    rec("experts prompt (all experts, masked)", _time(dense_form, 2, 5, flush), flops=6.0 * T * top * ff * W,
        note=f"useful FLOPs (top {top} of {E}); the kernels compute all {E} experts")
    for M in (1, B):
        xs, ii, ww = x[:M].contiguous(), idx[:M].contiguous(), wsel[:M].contiguous()
        live = len({e for e in ii.flatten().tolist() if e < E})
        rec(f"experts decode (chosen only) M={M}", _time(lambda: h.moe_sparse(xs, w13, w2, ii, ww, E, ff), 3, 8, flush), bytes_=live * 3.0 * ff * W * 2)
    return rows


def run_taruvik(a, peaks: dict) -> dict:
    dev = torch.device("cuda", torch.cuda.current_device())
    T, ctx = a.prefill, a.prefill
    res = {"design": "Taruvik", "dtype": "bf16", "data": "synthetic", "prompt_tokens": T, "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    for name, s in TARUVIK_SIZES.items():
        t0 = time.time()
        m = build_taruvik(s, dev)
        new = end_to_end(m, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del m
        torch.cuda.empty_cache()
        try:
            d = build_moe_transformer(s, dev)
            old = end_to_end(d, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
            del d
        except Exception as e:  # the neighbour's kernels may not take this size
            old = {"unavailable": f"{type(e).__name__}: {e}"[:300]}
        torch.cuda.empty_cache()
        res["sizes"][name] = {"config": s, "layered": new, "moe_transformer": old, "kernels": taruvik_kernel_table(s, T, ctx, peaks, dev),
                              "seconds": round(time.time() - t0, 1)}
    return res


# ----------------------------------------------------------------------------------------------- Lotazen
LOTAZEN_SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, window=1024, rec_heads=16, experts=16, top=2, ff=1408, shared_ff=2816, vocab=32768,
                  order="ppmp", lin_heads=16),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, window=2048, rec_heads=32, experts=8, top=2, ff=3584, shared_ff=7168, vocab=32768,
                  order="pm", lin_heads=32),
}


def lotazen_config(s: dict) -> dict:
    d = s["dim"]
    side = {"type": "parallel", "mixer": {
        "left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": s["window"]},
                 "rot": {"base": 500000.0, "dims": d, "scaling": {"factor": 2.0}}},
        "right": {"heads": s["rec_heads"], "dim": d, "vdim": d}, "left_scale": 0.6, "right_scale": 0.5}}
    mem = {"type": "mlstm", "mixer": {"heads": s["rec_heads"], "dim": d, "vdim": d, "gate_cap": 12.0}}
    mlp = {"kind": "moe", "expert": {"ff": s["ff"], "limit": 7.0}, "router": {"experts": s["experts"], "top": s["top"]},
           "shared": {"ff": s["shared_ff"], "limit": 7.0}}
    return {"architecture": "Lotazen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "max_positions": 8192, "logit_softcap": 30.0,
            "layers": [{**(side if c == "p" else mem), "mlp": mlp} for c in s["order"]]}


def build_lotazen(s: dict, dev):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer

    m = LayeredTransformer.empty(LayeredArgs.from_dict(lotazen_config(s)), dev, torch.bfloat16)
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            last = n.rsplit(".", 1)[-1]
            if p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            elif last in ("weight", "norm"):
                p.fill_(1.0)
            elif last == "lower":
                p.copy_(torch.rand(p.shape, generator=g, device=dev) * 0.9)
            else:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.1)
    return m.eval()


def fesenex_like(s: dict) -> dict:
    """The closest existing design at equal size: attention layers of the same heads where Lotazen has attention beside a recurrence,
    a lightning layer where it has a matrix memory, a dense feed-forward of the size of the experts one token uses."""
    return dict(width=s["width"], heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"], ff=s["top"] * s["ff"] + s["shared_ff"], vocab=s["vocab"],
                layers=len(s["order"]), lin_heads=s["lin_heads"], lightning_at=[i for i, c in enumerate(s["order"]) if c == "m"])


def lotazen_kernel_table(s: dict, T: int, ctx: int, peaks: dict, dev) -> dict:
    """Every kernel the design added, alone at this size, each next to the like kernel of the closest design at the same shape."""
    from mistral_inference_b200 import _abi_hybrid as h
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec

    bf = torch.bfloat16
    W, H, G, d, win, RH, E, ff, top = (s[k] for k in ("width", "heads", "kv_heads", "dim", "window", "rec_heads", "experts", "ff", "top"))
    flush = torch.zeros(160 << 20, dtype=torch.float32, device=dev)
    rows = {}

    def rec(name, ms, flops=0.0, bytes_=0.0, note=None):
        r = {"ms": round(ms, 4)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 2)
            r["of_bf16_peak"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["of_hbm_peak"] = round(bytes_ / ms / 1e6 / peaks["hbm_gbs"], 3)
        if note:
            r["note"] = note
        rows[name] = r

    B = 8
    # ---- attention: a prompt through the window, then one token per sequence
    ring = BufferCache(1, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d, window=win)]).to(dev, bf)
    full = BufferCache(1, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d)]).to(dev, bf)
    for c in (ring, full):
        c.cache_k[0].normal_(); c.cache_v[0].normal_()
    md = ring.get_input_metadata([T])[0]
    mdf = full.get_input_metadata([T])[0]
    qkv = torch.randn(T, (H + 2 * G) * d, device=dev).to(bf)
    freq = (torch.tensor(500000.0, dtype=torch.float64) ** (-torch.arange(0, d, 2, dtype=torch.float64) / d) / 2.0).to(dev)
    rec("rot_prep prompt", _time(lambda: h.rot_prep(qkv, freq, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True), 3, 8, flush),
        bytes_=2.0 * qkv.numel() * 2)
    q, k, v = h.rot_prep(qkv, freq, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True)
    o = torch.empty(T, H * d, device=dev, dtype=bf)
    nt = (T + 63) // 64
    pairs = sum(min(p + 1, win) for p in range(T))  # (query, key) pairs inside the window
    rec(f"attn_window prompt (tensor-core kernel, window {win})",
        _time(lambda: h.attn_window(q, ring.cache_k[0], ring.cache_v[0], md.positions, md.q_start, md.slots, o, 1, md.window, H, G, d, d, 0.09, win, own_k=k, own_v=v,
                                    seqpos=md.seqpos, n_tiles=nt), 2, 5, flush), flops=4.0 * d * H * pairs)
    tab = torch.zeros(64, H, device=dev)
    rec("like: attn_bias_flash prompt (all keys)",
        _time(lambda: h.attn_bias(q, full.cache_k[0], full.cache_v[0], tab, mdf.positions, mdf.q_start, mdf.slots, o, 1, ctx + 8, H, G, d, d, 0.09, n_tiles=nt), 2, 5, flush),
        flops=4.0 * d * H * T * (T + 1) / 2)
    rec("kv_scatter prompt", _time(lambda: h.kv_scatter(k, v, md.cache_rows, ring.cache_k[0], ring.cache_v[0]), 3, 8, flush), bytes_=2.0 * min(T, win) * 2 * G * d * 2)
    for c in (ring, full):
        c.reset(); c.init_kvseqlens(B); c.update_seqlens([ctx] * B)
    md2, md2f = ring.get_input_metadata([1] * B)[0], full.get_input_metadata([1] * B)[0]
    q2, o2 = q[:B].contiguous(), torch.empty(B, H * d, device=dev, dtype=bf)
    rec(f"attn_window decode B={B} (ring of {md2.window})",
        _time(lambda: h.attn_window(q2, ring.cache_k[0], ring.cache_v[0], md2.positions, md2.q_start, md2.slots, o2, B, md2.window, H, G, d, d, 0.09, win,
                                    splits=h.window_decode_plan(B, H, md2.window)[0], chunk=h.window_decode_plan(B, H, md2.window)[1]), 3, 8, flush),
        bytes_=2.0 * B * min(ctx + 1, win) * G * d * 2)
    q1, o1 = q[:1].contiguous(), torch.empty(1, H * d, device=dev, dtype=bf)
    ring.reset(); ring.init_kvseqlens(1); ring.update_seqlens([ctx])
    md1 = ring.get_input_metadata([1])[0]
    for label, (sp, ch) in (("128-key chunks", (h.attn_splits(1, H, md1.window), 0)), ("planned chunks", h.window_decode_plan(1, H, md1.window))):
        rec(f"attn_window decode B=1 (ring of {md1.window}), {label}: {sp} splits",
            _time(lambda: h.attn_window(q1, ring.cache_k[0], ring.cache_v[0], md1.positions, md1.q_start, md1.slots, o1, 1, md1.window, H, G, d, d, 0.09, win,
                                        splits=sp, chunk=ch), 3, 8, flush), bytes_=2.0 * min(ctx + 1, win) * G * d * 2)
    rec(f"like: attn_bias decode B={B} ctx={ctx}",
        _time(lambda: h.attn_bias(q2, full.cache_k[0], full.cache_v[0], tab, md2f.positions, md2f.q_start, md2f.slots, o2, B, ctx + 8, H, G, d, d, 0.09,
                                  splits=h.attn_splits(B, H, ctx + 8)), 3, 8, flush), bytes_=2.0 * B * (ctx + 1) * G * d * 2)
    # ---- recurrences
    Hd = RH * d
    qfv = (torch.randn(T, 3 * Hd, device=dev) * 0.3).to(bf)
    lower = (torch.rand(Hd, device=dev) * 0.9).to(bf)
    rec("hgrn2_gates prompt", _time(lambda: h.hgrn2_gates(qfv, lower, Hd), 3, 8, flush), bytes_=T * Hd * (2 * 2 + 3 * 4.0))
    qab = h.hgrn2_gates(qfv, lower, Hd)
    state = torch.zeros(B, RH, d, d, device=dev)
    zero = torch.zeros(1, dtype=torch.int32, device=dev)
    rec("gated_scan prompt (HGRN2)", _time(lambda: h.gated_scan(qab, qfv, 3 * Hd, 2 * Hd, state, md.q_start, zero, md.slots, 1, RH, d, d, ones=False), 2, 5, flush),
        flops=4.0 * T * RH * d * d, note="one CTA column walks the sequence, fp32 FMA")
    rec("gated_scan prompt (HGRN2), chunk-parallel",
        _time(lambda: h.gated_scan(qab, qfv, 3 * Hd, 2 * Hd, state, md.q_start, zero, md.slots, 1, RH, d, d, ones=False, max_seqlen=T), 2, 5, flush),
        flops=4.0 * T * RH * d * d, note="useful FLOPs; the chunks run twice (local state, then outputs), fp32 FMA")
    qkvg = torch.randn(T, 4 * Hd, device=dev).to(bf) * 0.1
    lstate = torch.zeros(B, RH, d, d, device=dev)
    decay = torch.full((RH,), 0.97, device=dev)
    o32 = torch.empty(T, Hd, device=dev)
    rec("like: lightning_scan prompt", _time(lambda: h.lightning_scan(qkvg, lstate, decay, md.q_start, zero, md.slots, o32, 1, RH, d, d), 2, 5, flush),
        flops=4.0 * T * RH * d * d, note="sequential in the tokens, fp32 FMA")
    mstate = torch.zeros(B, RH * d * (d + 1) + RH, device=dev)
    gif = torch.randn(T, 2 * RH, device=dev)
    rec("mlstm_gates prompt", _time(lambda: h.mlstm_gates(qkvg, gif, mstate, RH * d * (d + 1), md.q_start, zero, md.slots, 1, RH, d, 12.0, d ** -0.5), 3, 8, flush),
        bytes_=T * Hd * (2 * 2 + 3 * 4.0), note="includes the running maximum, one warp per head over all tokens")
    gates, qab2 = h.mlstm_gates(qkvg, gif, mstate, RH * d * (d + 1), md.q_start, zero, md.slots, 1, RH, d, 12.0, d ** -0.5)
    rec("gated_scan prompt (mLSTM, normaliser column)",
        _time(lambda: h.gated_scan(qab2, qkvg, 4 * Hd, 2 * Hd, mstate, md.q_start, zero, md.slots, 1, RH, d, d, ones=True), 2, 5, flush), flops=4.0 * T * RH * d * (d + 1))
    rec("gated_scan prompt (mLSTM, normaliser column), chunk-parallel",
        _time(lambda: h.gated_scan(qab2, qkvg, 4 * Hd, 2 * Hd, mstate, md.q_start, zero, md.slots, 1, RH, d, d, ones=True, max_seqlen=T), 2, 5, flush),
        flops=4.0 * T * RH * d * (d + 1))
    om, nq = h.gated_scan(qab2, qkvg, 4 * Hd, 2 * Hd, mstate, md.q_start, zero, md.slots, 1, RH, d, d, ones=True)
    nw = torch.ones(Hd, device=dev).to(bf)
    rec("scan_post prompt (mLSTM)", _time(lambda: h.scan_post(om, gates, nw, True, qkvg, 4 * Hd, 3 * Hd, RH, d, True, 1e-5, nq=nq), 3, 8, flush), bytes_=T * Hd * (4 + 4 + 2 + 2.0))
    rec("like: gated_headnorm prompt", _time(lambda: h.gated_headnorm(o32, nw, qkvg, 4 * Hd, 3 * Hd, 1e-5), 3, 8, flush), bytes_=T * Hd * (4 + 2 + 2.0))
    one = torch.ones(B, dtype=torch.int32, device=dev)
    qabB = qab[:B].contiguous()
    rec(f"gated_scan decode B={B} (HGRN2)", _time(lambda: h.gated_scan(qabB, qfv, 3 * Hd, 2 * Hd, state, md2.q_start, one, md2.slots, B, RH, d, d, ones=False), 3, 8, flush),
        bytes_=2.0 * state.numel() * 4)
    rec(f"like: lightning_scan decode B={B}", _time(lambda: h.lightning_scan(qkvg, lstate, decay, md2.q_start, one, md2.slots, o32, B, RH, d, d), 3, 8, flush),
        bytes_=2.0 * lstate.numel() * 4)
    # ---- experts
    x = torch.randn(T, W, device=dev).to(bf)
    wr = (torch.randn(E, W, device=dev) / math.sqrt(W) * 4).to(bf)
    rec("moe_route prompt (sigmoid)", _time(lambda: h.moe_route(x, wr, None, 1, 1, top, score=1), 3, 8, flush), bytes_=T * W * 2.0)
    dense, idx, wsel = h.moe_route(x, wr, None, 1, 1, top, score=1)
    w13 = (torch.randn(E * 2 * ff, W, device=dev) * 0.02).to(bf)
    w2 = (torch.randn(W, E * ff, device=dev) * 0.02).to(bf)
    x32 = torch.zeros(T, W, device=dev)

    def dense_form():
        act = h.linear_glu(x, w13, 7.0, 1.702, rowscale=dense, group=ff)
        return h.linear(act, w2, epi=h.EPI_RESIDUAL, residual=x32)

    def dense_like():
        act = h.linear_swiglu(x, w13, rowscale=dense, group=ff)
        return h.linear(act, w2, epi=h.EPI_F32)

    rec("experts prompt (all experts, scaled input, masked)", _time(dense_form, 2, 5, flush), flops=6.0 * T * top * ff * W,
        note=f"useful FLOPs (top {top} of {E}); the kernels compute all {E} experts")
    rec("like: experts prompt of the softmax-routed mixture", _time(dense_like, 2, 5, flush), flops=6.0 * T * top * ff * W)
    for M in (1, B):
        xs, ii, ww = x[:M].contiguous(), idx[:M].contiguous(), wsel[:M].contiguous()
        rec(f"experts decode (chosen only, scaled input) M={M}", _time(lambda: h.moe_sparse(xs, w13, w2, ii, ww, E, ff, glu=True, limit=7.0, alpha=1.702), 3, 8, flush),
            bytes_=_experts_used(ii) * 3.0 * ff * W * 2)
        rec(f"like: experts decode of the softmax-routed mixture M={M}", _time(lambda: h.moe_sparse(xs, w13, w2, ii, ww, E, ff), 3, 8, flush),
            bytes_=_experts_used(ii) * 3.0 * ff * W * 2)
    return rows


def run_lotazen(a, peaks: dict) -> dict:
    dev = torch.device("cuda", torch.cuda.current_device())
    T, ctx = a.prefill, a.prefill
    res = {"design": "Lotazen", "dtype": "bf16", "data": "synthetic", "prompt_tokens": T, "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    for name, s in LOTAZEN_SIZES.items():
        t0 = time.time()
        m = build_lotazen(s, dev)
        new = end_to_end(m, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del m
        torch.cuda.empty_cache()
        f = fesenex_like(s)
        d = build_layered(f, dev)
        old = end_to_end(d, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del d
        torch.cuda.empty_cache()
        res["sizes"][name] = {"config": s, "layered": new, "fesenex_equal_size": old, "kernels": lotazen_kernel_table(s, T, ctx, peaks, dev),
                              "seconds": round(time.time() - t0, 1)}
    return res

# ----------------------------------------------------------------------------------------------- Viladra
VILADRA_SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, window=1024, rec_heads=16, experts=16, top=2, ff=1408, shared_ff=2816, vocab=32768,
                  order="grag", rank=64, taps=4),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, window=2048, rec_heads=32, experts=8, top=2, ff=3584, shared_ff=7168, vocab=32768,
                  order="ar", rank=128, taps=4),
}


def viladra_config(s: dict) -> dict:
    d, RH = s["dim"], s["rec_heads"]
    mixers = {
        "a": {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": s["window"]}}},
        "r": {"type": "retention", "mixer": {"heads": RH, "dim": d, "vdim": d, "decay": [1.0 - 2.0 ** (-5 - 5 * i / max(RH - 1, 1)) for i in range(RH)],
                                             "rot": {"base": 500000.0, "dims": d}}},
        "g": {"type": "gla", "mixer": {"heads": RH, "dim": d, "vdim": d, "tau": 16.0}},
    }
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"], "scale": 1.5}, "shared": {"ff": s["shared_ff"]}}
    return {"architecture": "Viladra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "canon": {"taps": s["taps"]},
            "embedding": {"scale": 1.0}, "logit_softcap": 30.0, "layers": [{**mixers[c], "mlp": mlp} for c in s["order"]]}


def build_viladra(s: dict, dev):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer
    from mistral_inference_b200.transformer_layers import GlaMixer

    m = LayeredTransformer.empty(LayeredArgs.from_dict(viladra_config(s)), dev, torch.bfloat16)
    for blk in m.layers:  # the rank of the decay projection comes with a checkpoint; here it is the size table's
        if isinstance(blk.mix, GlaMixer):
            blk.mix.prepare("a1", (s["rank"], s["width"]))
            blk.mix.prepare("a2", (blk.mix.nqk, s["rank"]))
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            last = n.rsplit(".", 1)[-1]
            if last == "dwa":
                p.fill_(1.0 / p.numel())
            elif last == "weight" and p.dim() == 2:  # convolution taps
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.2)
            elif p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            elif last in ("weight", "norm", "q_norm", "k_norm"):
                p.fill_(1.0)
            elif last == "ba2":
                p.fill_(3.0)
            else:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.1)
    return m.eval()


def lotazen_like(s: dict) -> dict:
    """The closest existing design at equal size: rotary window attention beside a gated recurrence where Viladra has sigmoid-weight
    window attention, a matrix memory where it has retention or gated linear attention, the same experts (gated there)."""
    return dict(width=s["width"], heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"], window=s["window"], rec_heads=s["rec_heads"], experts=s["experts"],
                top=s["top"], ff=s["ff"], shared_ff=s["shared_ff"], vocab=s["vocab"], order="".join("p" if c == "a" else "m" for c in s["order"]),
                lin_heads=s["rec_heads"])


def viladra_kernel_table(s: dict, T: int, ctx: int, peaks: dict, dev) -> dict:
    """Every kernel the design added or extended, alone at this size, each next to the like kernel of the closest design at the same shape."""
    from mistral_inference_b200 import _abi_hybrid as h
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec

    bf = torch.bfloat16
    W, H, G, d, win, RH, E, ff, top, taps, rank = (s[k] for k in ("width", "heads", "kv_heads", "dim", "window", "rec_heads", "experts", "ff", "top", "taps", "rank"))
    flush = torch.zeros(160 << 20, dtype=torch.float32, device=dev)
    rows = {}

    def rec(name, ms, flops=0.0, bytes_=0.0, note=None):
        r = {"ms": round(ms, 4)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 2)
            r["of_bf16_peak"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["of_hbm_peak"] = round(bytes_ / ms / 1e6 / peaks["hbm_gbs"], 3)
        if note:
            r["note"] = note
        rows[name] = r

    B = 8
    ring = BufferCache(1, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d, window=win)]).to(dev, bf)
    ring.cache_k[0].normal_(); ring.cache_v[0].normal_()
    md = ring.get_input_metadata([T])[0]
    zero = torch.zeros(1, dtype=torch.int32, device=dev)
    # ---- the stream: convolution in, norm and depth average out
    x32 = torch.randn(T, W, device=dev)
    cw = (torch.randn(W, taps, device=dev) * 0.2).to(bf)
    cstate = torch.zeros(B, 2, taps - 1, W, device=dev)
    nw = torch.ones(W, device=dev).to(bf)
    rec("canon_conv prompt", _time(lambda: h.canon_conv(x32, cw, cstate, 0, md.q_start, zero, md.slots, 1, False), 3, 8, flush), bytes_=T * W * (4 + 2.0),
        note="reads the fp32 stream, writes bf16; includes the state write-back launch")
    rec("like: rmsnorm prompt", _time(lambda: h.rmsnorm(x32, nw, 1e-5), 3, 8, flush), bytes_=T * W * (4 + 2.0))
    n_mix = 5
    stack = torch.randn(n_mix + 1, T, W, device=dev)
    y32 = torch.randn(T, W, device=dev)
    coef = torch.full((n_mix,), 1.0 / n_mix, device=dev).to(bf)
    rec("rmsnorm_add prompt", _time(lambda: h.rmsnorm_add(y32, nw, stack[n_mix - 1], 1e-5), 3, 8, flush), bytes_=T * W * 12.0)
    rec(f"rmsnorm_add + depth average over {n_mix} prompt", _time(lambda: h.rmsnorm_add(y32, nw, stack[n_mix - 1], 1e-5, stack, n_mix, coef, stack[n_mix]), 3, 8, flush),
        bytes_=T * W * 4.0 * (3 + n_mix))
    rec("like: layernorm add prompt", _time(lambda: h.layernorm(y32, nw, nw, 1e-5, add_to=stack[0]), 3, 8, flush), bytes_=T * W * 12.0)
    # ---- attention
    qkv = torch.randn(T, (H + 2 * G) * d, device=dev).to(bf)
    qn, kn = torch.ones(H * d, device=dev).to(bf), torch.ones(G * d, device=dev).to(bf)
    rec("whole_norm_prep prompt", _time(lambda: h.whole_norm_prep(qkv, qn, kn, None, None, None, H * d, G * d, G * d, 1e-5, own=True), 3, 8, flush),
        bytes_=2.0 * qkv.numel() * 2)
    freq = (torch.tensor(500000.0, dtype=torch.float64) ** (-torch.arange(0, d, 2, dtype=torch.float64) / d)).to(dev)
    rec("like: rot_prep prompt", _time(lambda: h.rot_prep(qkv, freq, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True), 3, 8, flush),
        bytes_=2.0 * qkv.numel() * 2)
    q, k, v = h.whole_norm_prep(qkv, qn, kn, None, None, None, H * d, G * d, G * d, 1e-5, own=True)
    o = torch.empty(T, H * d, device=dev, dtype=bf)
    nt = (T + 63) // 64
    pairs = sum(min(p + 1, win) for p in range(T))
    pb = torch.zeros(H, device=dev)
    for label, hb in (("attn_window prompt, sigmoid weights", pb), ("like: attn_window prompt, softmax", None)):
        rec(f"{label} (tensor-core kernel, window {win})",
            _time(lambda: h.attn_window(q, ring.cache_k[0], ring.cache_v[0], md.positions, md.q_start, md.slots, o, 1, md.window, H, G, d, d, 0.09, win, own_k=k,
                                        own_v=v, seqpos=md.seqpos, n_tiles=nt, head_bias=hb), 2, 5, flush), flops=4.0 * d * H * pairs)
    ring.reset(); ring.init_kvseqlens(B); ring.update_seqlens([ctx] * B)
    md2 = ring.get_input_metadata([1] * B)[0]
    q2, o2 = q[:B].contiguous(), torch.empty(B, H * d, device=dev, dtype=bf)
    sp, ch = h.window_decode_plan(B, H, md2.window)
    for label, hb in (("attn_window decode, sigmoid weights", pb), ("like: attn_window decode, softmax", None)):
        rec(f"{label} B={B} (ring of {md2.window})",
            _time(lambda: h.attn_window(q2, ring.cache_k[0], ring.cache_v[0], md2.positions, md2.q_start, md2.slots, o2, B, md2.window, H, G, d, d, 0.09, win,
                                        splits=sp, chunk=ch, head_bias=hb), 3, 8, flush), bytes_=2.0 * B * min(ctx + 1, win) * G * d * 2)
    # ---- recurrences
    Hd = RH * d
    qkvg = (torch.randn(T, 4 * Hd, device=dev) * 0.1).to(bf)
    decay = torch.full((RH,), 0.97, device=dev)
    rec("retention_qab prompt", _time(lambda: h.retention_qab(qkvg, freq, decay, md.positions, RH, d, d, d ** -0.5), 3, 8, flush), bytes_=T * Hd * (2 * 2 + 3 * 4.0))
    z32 = torch.randn(T, Hd, device=dev)
    rec("gla_qab prompt", _time(lambda: h.gla_qab(qkvg, z32, Hd, d ** -0.5, 1 / 16.0), 3, 8, flush), bytes_=T * Hd * (2 * 2 + 4 + 3 * 4.0))
    lower = (torch.rand(Hd, device=dev) * 0.9).to(bf)
    rec("like: hgrn2_gates prompt", _time(lambda: h.hgrn2_gates(qkvg, lower, Hd), 3, 8, flush), bytes_=T * Hd * (2 * 2 + 3 * 4.0))
    qab = h.gla_qab(qkvg, z32, Hd, d ** -0.5, 1 / 16.0)
    state = torch.zeros(B, RH, d, d, device=dev)
    rec("gated_scan prompt (gated linear attention), chunk-parallel",
        _time(lambda: h.gated_scan(qab, qkvg, 4 * Hd, 2 * Hd, state, md.q_start, zero, md.slots, 1, RH, d, d, ones=False, max_seqlen=T), 2, 5, flush),
        flops=4.0 * T * RH * d * d, note="the kernel of the closest design's recurrences, same launch; useful FLOPs, the chunks run twice, fp32 FMA")
    o32 = h.gated_scan(qab, qkvg, 4 * Hd, 2 * Hd, state, md.q_start, zero, md.slots, 1, RH, d, d, ones=False, max_seqlen=T)
    hw = torch.ones(d, device=dev).to(bf)
    rec("scan_post prompt (shared weight, SiLU gate)", _time(lambda: h.scan_post(o32, None, hw, False, qkvg, 4 * Hd, 3 * Hd, RH, d, False, 1e-5, silu_gate=True), 3, 8, flush),
        bytes_=T * Hd * (4 + 2 + 2.0))
    rec("scan_post prompt (no weight, SiLU gate)", _time(lambda: h.scan_post(o32, None, None, False, qkvg, 4 * Hd, 3 * Hd, RH, d, False, 1e-5, silu_gate=True), 3, 8, flush),
        bytes_=T * Hd * (4 + 2 + 2.0))
    rec("like: scan_post prompt (shared weight, no gate)", _time(lambda: h.scan_post(o32, None, hw, False, None, 0, 0, RH, d, False, 1e-5), 3, 8, flush), bytes_=T * Hd * (4 + 2.0))
    one = torch.ones(B, dtype=torch.int32, device=dev)
    qabB = qab[:B].contiguous()
    rec(f"gated_scan decode B={B}", _time(lambda: h.gated_scan(qabB, qkvg, 4 * Hd, 2 * Hd, state, md2.q_start, one, md2.slots, B, RH, d, d, ones=False), 3, 8, flush),
        bytes_=2.0 * state.numel() * 4, note="the closest design's kernel")
    # ---- experts
    x = torch.randn(T, W, device=dev).to(bf)
    wr = (torch.randn(E, W, device=dev) / math.sqrt(W) * 4).to(bf)
    rec("moe_route prompt (softmax, scaled weights)", _time(lambda: h.moe_route(x, wr, None, 1, 1, top, score=0, scale=1.5), 3, 8, flush), bytes_=T * W * 2.0)
    rec("like: moe_route prompt (sigmoid)", _time(lambda: h.moe_route(x, wr, None, 1, 1, top, score=1), 3, 8, flush), bytes_=T * W * 2.0)
    dense, idx, wsel = h.moe_route(x, wr, None, 1, 1, top, score=0, scale=1.5)
    w_up = (torch.randn(E * ff, W, device=dev) * 0.02).to(bf)
    w13 = (torch.randn(E * 2 * ff, W, device=dev) * 0.02).to(bf)
    w2 = (torch.randn(W, E * ff, device=dev) * 0.02).to(bf)
    xr = torch.zeros(T, W, device=dev)

    def dense_form():
        return h.linear(h.linear_relu2(x, w_up, rowscale=dense, group=ff), w2, epi=h.EPI_F32)

    def dense_like():
        return h.linear(h.linear_glu(x, w13, 7.0, 1.702, rowscale=dense, group=ff), w2, epi=h.EPI_RESIDUAL, residual=xr)

    rec("experts prompt (all experts, ungated, masked)", _time(dense_form, 2, 5, flush), flops=4.0 * T * top * ff * W,
        note=f"useful FLOPs (top {top} of {E}); the kernels compute all {E} experts")
    rec("like: experts prompt of the scaled-input gated mixture", _time(dense_like, 2, 5, flush), flops=6.0 * T * top * ff * W)
    for M in (1, B):
        xs, ii, ww = x[:M].contiguous(), idx[:M].contiguous(), wsel[:M].contiguous()
        rec(f"experts decode (chosen only, ungated) M={M}", _time(lambda: h.moe_sparse(xs, w_up, w2, ii, ww, E, ff, glu=2), 3, 8, flush),
            bytes_=_experts_used(ii) * 2.0 * ff * W * 2)
        rec(f"like: experts decode of the scaled-input gated mixture M={M}", _time(lambda: h.moe_sparse(xs, w13, w2, ii, ww, E, ff, glu=1, limit=7.0, alpha=1.702), 3, 8, flush),
            bytes_=_experts_used(ii) * 3.0 * ff * W * 2)
    # ---- one decode step's convolution and norms
    xB = x32[:B].contiguous()
    rec(f"canon_conv decode B={B}", _time(lambda: h.canon_conv(xB, cw, cstate, 0, md2.q_start, one, md2.slots, B, True), 3, 8, flush),
        bytes_=B * W * (4 + 2 + 2 * (taps - 1) * 4.0), note="latency: a few KB")
    rec(f"like: rmsnorm decode B={B}", _time(lambda: h.rmsnorm(xB, nw, 1e-5), 3, 8, flush), bytes_=B * W * (4 + 2.0))
    return rows


def run_viladra(a, peaks: dict) -> dict:
    dev = torch.device("cuda", torch.cuda.current_device())
    T, ctx = a.prefill, a.prefill
    res = {"design": "Viladra", "dtype": "bf16", "data": "synthetic", "prompt_tokens": T, "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    for name, s in VILADRA_SIZES.items():
        t0 = time.time()
        m = build_viladra(s, dev)
        new = end_to_end(m, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del m
        torch.cuda.empty_cache()
        d = build_lotazen(lotazen_like(s), dev)
        old = end_to_end(d, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del d
        torch.cuda.empty_cache()
        res["sizes"][name] = {"config": s, "layered": new, "lotazen_equal_size": old, "kernels": viladra_kernel_table(s, T, ctx, peaks, dev),
                              "seconds": round(time.time() - t0, 1)}
    return res


# ----------------------------------------------------------------------------------------------- Dimorax
DIMORAX_SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, lat_heads=16, lat_dim=128, rot_dim=64, kv_rank=512, window=1024, rec_heads=16, rec_kv_heads=16, taps=4, rank=64,
                  experts=16, top=2, groups=4, keep=2, ff=1408, shared_ff=2816, dense_ff=5632, vocab=32768, order="dald"),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, lat_heads=32, lat_dim=128, rot_dim=64, kv_rank=512, window=2048, rec_heads=32, rec_kv_heads=16, taps=4, rank=128,
                  experts=8, top=2, groups=4, keep=2, ff=3584, shared_ff=7168, dense_ff=14336, vocab=32768, order="adl"),
}


def dimorax_config(s: dict) -> dict:
    d = s["dim"]
    mixers = {
        "a": {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "softcap": 30.0,
                                             "rot": {"base": 500000.0, "dims": d // 2, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}},
        "l": {"type": "latent_attention", "mixer": {"heads": s["lat_heads"], "dim": s["lat_dim"], "rot_dim": s["rot_dim"], "vdim": s["lat_dim"], "kv_rank": s["kv_rank"],
                                                    "scale": (s["lat_dim"] + s["rot_dim"]) ** -0.5, "mask": {"size": s["window"]}, "rot": {"base": 10000.0, "dims": s["rot_dim"]}}},
        "d": {"type": "channel_delta", "mixer": {"heads": s["rec_heads"], "kv_heads": s["rec_kv_heads"], "dim": d, "vdim": d, "conv": s["taps"]}},
    }
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"], "scale": 1.5, "groups": {"count": s["groups"], "keep": s["keep"]}},
           "shared": {"ff": s["shared_ff"]}}
    return {"architecture": "Dimorax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "residual_mult": 0.7,
            "layers": [{**mixers[c], "mlp": moe if i % 3 != 2 else {"kind": "dense", "ff": s["dense_ff"]}} for i, c in enumerate(s["order"])]}


def build_dimorax(s: dict, dev):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer
    from mistral_inference_b200.transformer_layers import DeltaMixer

    m = LayeredTransformer.empty(LayeredArgs.from_dict(dimorax_config(s)), dev, torch.bfloat16)
    for blk in m.layers:  # the ranks of the low-rank projections come with a checkpoint; here they are the size table's
        if isinstance(blk.mix, DeltaMixer):
            blk.mix.resize(s["rank"], s["rank"])
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            last = n.rsplit(".", 1)[-1]
            if p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            elif last in ("norm", "c_norm"):
                p.fill_(1.0)
            elif last in ("dt_bias", "a_log"):
                p.fill_(-2.0)
            else:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.1)
    return m.eval()


def lotazen_like_dimorax(s: dict) -> dict:
    """The closest existing design at equal size: rotary window attention beside a gated recurrence where Dimorax has attention, a matrix memory
    elsewhere, gated experts of the same sizes in every layer."""
    return dict(width=s["width"], heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"], window=s["window"], rec_heads=s["rec_heads"], experts=s["experts"],
                top=s["top"], ff=s["ff"], shared_ff=s["shared_ff"], vocab=s["vocab"], order="".join("p" if c == "a" else "m" for c in s["order"]),
                lin_heads=s["rec_heads"])


def dimorax_kernel_table(s: dict, T: int, ctx: int, peaks: dict, dev) -> dict:
    """Every kernel the design added or extended, alone at this size, each next to the like kernel of an existing design at the same shape."""
    from mistral_inference_b200 import _abi_hybrid as h
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec
    from mistral_inference_b200.rope import scaled_frequencies

    bf = torch.bfloat16
    W, H, G, d, E, ff, top, RH, RG, taps, rank = (s[k] for k in ("width", "heads", "kv_heads", "dim", "experts", "ff", "top", "rec_heads", "rec_kv_heads", "taps", "rank"))
    LH, dn, dr, rk, win = (s[k] for k in ("lat_heads", "lat_dim", "rot_dim", "kv_rank", "window"))
    flush = torch.zeros(160 << 20, dtype=torch.float32, device=dev)
    rows = {}

    def rec(name, fn, flops=0.0, bytes_=0.0, note=None, n=(3, 8)):
        ms = _time(fn, n[0], n[1], flush)
        r = {"ms": round(ms, 4)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 2)
            r["of_bf16_peak"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["of_hbm_peak"] = round(bytes_ / ms / 1e6 / peaks["hbm_gbs"], 3)
        if note:
            r["note"] = note
        rows[name] = r

    def rnd(*shape, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(bf)

    B, nt = 8, (T + 63) // 64
    zero, one = torch.zeros(1, dtype=torch.int32, device=dev), torch.ones(B, dtype=torch.int32, device=dev)
    # ---- norms
    x32, nw = torch.randn(T, W, device=dev), torch.ones(W, device=dev).to(bf)
    rec("rmsnorm_pair prompt (two norms, one pass)", lambda: h.rmsnorm_pair(x32, nw, nw, 1e-5, 1.0), bytes_=T * W * 8.0)
    rec("like: rmsnorm prompt", lambda: h.rmsnorm(x32, nw, 1e-5), bytes_=T * W * 6.0)
    # ---- attention
    ring = BufferCache(1, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d)]).to(dev, bf)
    ring.cache_k[0].normal_(); ring.cache_v[0].normal_()
    md = ring.get_input_metadata([T])[0]
    qkv = rnd(T, (H + 2 * G) * d)
    fh, fd = scaled_frequencies(d // 2, 5e5, None)[0].to(dev), scaled_frequencies(d, 5e5, None)[0].to(dev)
    rec("rot_prep prompt (halves, half of each head)", lambda: h.rot_prep(qkv, fh, md.positions, None, None, None, H, G, d, d, d // 2, False, 0.0, own=True, halves=True, mag=1.2),
        bytes_=4.0 * qkv.numel())
    rec("like: rot_prep prompt (neighbours, unit norm)", lambda: h.rot_prep(qkv, fd, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True), bytes_=4.0 * qkv.numel())
    q, k, v = h.rot_prep(qkv, fh, md.positions, None, None, None, H, G, d, d, d // 2, False, 0.0, own=True, halves=True)
    o, sink = torch.empty(T, H * d, device=dev, dtype=bf), torch.zeros(H, device=dev)
    for label, kw in (("attn_window prompt, soft cap and sinks", dict(softcap=30.0, sink=sink)), ("like: attn_window prompt, softmax", {})):
        rec(f"{label} (tensor-core kernel)", lambda: h.attn_window(q, ring.cache_k[0], ring.cache_v[0], md.positions, md.q_start, md.slots, o, 1, md.window, H, G, d, d, 0.09, 0,
                                                                   own_k=k, own_v=v, seqpos=md.seqpos, n_tiles=nt, **kw), flops=4.0 * d * H * T * (T + 1) / 2, n=(2, 5))
    ring.reset(); ring.init_kvseqlens(B); ring.update_seqlens([ctx] * B)
    md2 = ring.get_input_metadata([1] * B)[0]
    q2, o2 = q[:B].contiguous(), torch.empty(B, H * d, device=dev, dtype=bf)
    sp, ch = h.window_decode_plan(B, H, md2.window)
    for label, kw in (("attn_window decode, soft cap and sinks", dict(softcap=30.0, sink=sink)), ("like: attn_window decode, softmax", {})):
        rec(f"{label} B={B}", lambda: h.attn_window(q2, ring.cache_k[0], ring.cache_v[0], md2.positions, md2.q_start, md2.slots, o2, B, md2.window, H, G, d, d, 0.09, 0, splits=sp,
                                                    chunk=ch, **kw), bytes_=2.0 * B * (ctx + 1) * G * d * 2)
    # ---- latent attention
    lat = BufferCache(2, B, ctx + 8, 0, 0, None, layer_specs=[LayerCacheSpec(kind="ring", n_kv_heads=1, k_dim=rk + dr, v_dim=0, window=w) for w in (win, None)]).to(dev, bf)
    lat.cache_k[0].normal_(); lat.cache_k[1].normal_()
    mw, mf = lat.get_input_metadata([T])
    freq = scaled_frequencies(dr, 1e4, None)[0].to(dev)
    nq = LH * (dn + dr)
    y, cn, qn = rnd(T, nq + rk + dr), torch.ones(rk, device=dev).to(bf), torch.ones(rk, device=dev).to(bf)
    rec("latent_prep prompt (rows beside the ring)", lambda: h.latent_prep(y, None, cn, freq, mw.positions, None, lat.cache_k[0], 0, rk, dr, dr, 1e-5, 1.0, kv_off=nq, halves=True, own=True),
        bytes_=T * (rk + dr) * 4.0)
    y2 = rnd(T, 2 * rk + dr)
    rec("like: latent_prep prompt (query latent, ring)", lambda: h.latent_prep(y2, qn, cn, freq, mf.positions, mf.cache_rows, lat.cache_k[1], rk, rk, dr, dr, 1e-5, 1.0),
        bytes_=T * (2 * rk + dr) * 4.0)
    kf, vf, qr, of = rnd(T, LH, dn + dr), rnd(T, LH, dn), rnd(T, nq), torch.empty(T, LH * dn, device=dev, dtype=bf)
    lsink, iota = torch.zeros(LH, device=dev), h.iota(1, dev)
    pairs = sum(min(p + 1, win) for p in range(T))
    for label, w, kw, n_pairs in ((f"latent prompt attention, window {win}, sinks", win, dict(sink=lsink), pairs), ("like: latent prompt attention, whole", 0, {}, T * (T + 1) / 2)):
        rec(f"{label} (tensor-core kernel)", lambda: h.attn_window(qr, kf, vf, md.positions, md.q_start, iota, of, 1, 1, LH, LH, dn + dr, dn, 0.07, w, own_k=kf, own_v=vf, seqpos=zero,
                                                                   n_tiles=nt, **kw), flops=2.0 * LH * (2 * dn + dr) * n_pairs, n=(2, 5))
    kn, rows_ = rnd(T, LH * dn), rnd(T, rk + dr)
    rec("latent_expand prompt", lambda: h.latent_expand(kn, rows_, LH, dn, dr, rk), bytes_=T * 2.0 * (LH * dn + dr + nq))
    lat.reset(); lat.init_kvseqlens(B); lat.update_seqlens([ctx] * B)
    mw2, mf2 = lat.get_input_metadata([1] * B)
    qa = rnd(B, LH * (rk + dr))
    for label, m_, i, w, kw, n in ((f"attn_latent_decode, window {win}, sinks", mw2, 0, win, dict(sink=lsink), min(ctx + 1, win)), ("like: attn_latent_decode, whole", mf2, 1, 0, {}, ctx + 1)):
        rec(f"{label} B={B}", lambda: h.attn_latent_decode(qa, lat.cache_k[i], m_.positions, m_.slots, B, m_.window, LH, rk, dr, 0.07, w, **kw), bytes_=B * n * (rk + dr) * 2.0)
    # ---- gated delta rule
    Nk, He, Hd = RG * d, RH * d, RH * d
    ch_, N = 2 * Nk + He, 2 * Nk + He + RH + 2 * rank
    N = (N + 127) // 128 * 128
    yd, conv = rnd(T, N), rnd(ch_, taps, scale=0.3)
    cstate, state = torch.zeros(B, taps, ch_, device=dev), torch.zeros(B, RH, d, d, device=dev)
    wa2, wg2, dtb, alog, hw = rnd(Hd, rank, scale=0.1), rnd(He, rank, scale=0.1), torch.full((Hd,), -2.0, device=dev).to(bf), torch.full((RH,), -2.0, device=dev).to(bf), torch.ones(d, device=dev).to(bf)
    prep = lambda: h.delta_prep(yd, conv, cstate, md.positions, md.q_start, zero, md.slots, 1, RH, RG, d, d)  # noqa: E731
    rec("delta_prep prompt (convolutions, unit norms; incl. the carried inputs' launch)", prep, bytes_=T * ch_ * (2 + 4.0))
    z32 = torch.randn(T, Hd, device=dev)
    qkvg = rnd(T, 4 * Hd, scale=0.1)
    rec("like: gla_qab prompt", lambda: h.gla_qab(qkvg, z32, Hd, d ** -0.5, 1 / 16.0), bytes_=T * Hd * (2 * 2 + 4 + 3 * 4.0))
    xa = yd[:, ch_ + RH: ch_ + RH + rank]
    rec(f"linear_decay prompt (rank {rank} -> decays, fp32 out)", lambda: h.linear_decay(xa, wa2, dtb, alog, d), bytes_=T * (rank * 2 + Hd * 4.0))
    xc = xa.contiguous()
    rec(f"like: linear prompt (rank {rank}, fp32 out)", lambda: h.linear(xc, wa2, dtb, epi=h.EPI_F32), bytes_=T * (rank * 2 + Hd * 4.0))
    qk, kq, vv, beta = prep()
    g = h.linear_decay(xa, wa2, dtb, alog, d)
    rec("delta_scan prompt", lambda: h.delta_scan(qk, kq, vv, beta, g, state, md.q_start, zero, md.slots, 1, RH, RG, d, d), flops=6.0 * T * RH * d * d, n=(2, 5),
        note="useful FLOPs, fp32 FMA, one dependent step per token")
    qab = h.gla_qab(qkvg, z32, Hd, d ** -0.5, 1 / 16.0)
    gst = torch.zeros(B, RH, d, d, device=dev)
    rec("like: gated_scan prompt, chunk-parallel", lambda: h.gated_scan(qab, qkvg, 4 * Hd, 2 * Hd, gst, md.q_start, zero, md.slots, 1, RH, d, d, ones=False, max_seqlen=T),
        flops=4.0 * T * RH * d * d, n=(2, 5), note="useful FLOPs, the chunks run twice, fp32 FMA")
    ydB, qabB = yd[:B].contiguous(), qab[:B].contiguous()
    rec(f"delta_step decode B={B} (convolutions, decays, state, norm, gate in one)",
        lambda: h.delta_step(ydB, rank, rank, conv, cstate, state, wa2, dtb, alog, wg2, hw, md2.positions, one, md2.slots, RH, RG, d, d, 1e-5), bytes_=2.0 * state.numel() * 4)
    rec(f"like: gated_scan decode B={B} (the state only)", lambda: h.gated_scan(qabB, qkvg, 4 * Hd, 2 * Hd, gst, md2.q_start, one, md2.slots, B, RH, d, d, ones=False),
        bytes_=2.0 * gst.numel() * 4)
    # ---- feed-forward
    x = rnd(T, W)
    w13, w2, wr, corr = rnd(E * 2 * ff, W, scale=0.02), rnd(W, E * ff, scale=0.02), rnd(E, W, scale=4 / math.sqrt(W)), torch.zeros(E, device=dev).to(bf)
    route = lambda t: h.moe_route(t, wr, corr, s["groups"], s["keep"], top, score=1, scale=1.5, group_two=True, renorm=True)  # noqa: E731
    rec("moe_route prompt (groups by two, renormalised)", lambda: route(x), bytes_=T * W * 2.0)
    rec("like: moe_route prompt (sigmoid)", lambda: h.moe_route(x, wr, None, 1, 1, top, score=1), bytes_=T * W * 2.0)
    dense, idx, wsel = route(x)
    xr = torch.zeros(T, W, device=dev)
    rec("experts prompt (all experts, masked)", lambda: h.linear(h.linear_swiglu(x, w13, rowscale=dense, group=ff), w2, epi=h.EPI_RESIDUAL, residual=xr), flops=6.0 * T * top * ff * W,
        note=f"useful FLOPs (top {top} of {E}); the kernels compute all {E} experts", n=(2, 5))
    rec("like: experts prompt of the scaled-input gated mixture", lambda: h.linear(h.linear_glu(x, w13, 7.0, 1.702, rowscale=dense, group=ff), w2, epi=h.EPI_RESIDUAL, residual=xr),
        flops=6.0 * T * top * ff * W, n=(2, 5))
    for M in (1, B):
        xs, ii, ww, xm = x[:M].contiguous(), idx[:M].contiguous(), wsel[:M].contiguous(), xr[:M].contiguous()
        rec(f"experts decode (chosen only) M={M}", lambda: h.moe_sparse(xs, w13, w2, ii, ww, E, ff, add_to=xm), bytes_=_experts_used(ii) * 3.0 * ff * W * 2)
        rec(f"like: experts decode of the scaled-input gated mixture M={M}", lambda: h.moe_sparse(xs, w13, w2, ii, ww, E, ff, glu=1, limit=7.0, alpha=1.702, add_to=xm),
            bytes_=_experts_used(ii) * 3.0 * ff * W * 2)
    wd = rnd(2 * s["dense_ff"], W, scale=0.02)
    rec("linear_swiglu prompt (gelu)", lambda: h.linear_swiglu(x, wd, gelu=True), flops=4.0 * T * s["dense_ff"] * W, n=(2, 5))
    rec("like: linear prompt (clamped gated unit)", lambda: h.linear_glu(x, wd, 7.0, 1.702), flops=4.0 * T * s["dense_ff"] * W, n=(2, 5))
    return rows


def run_dimorax(a, peaks: dict) -> dict:
    dev = torch.device("cuda", torch.cuda.current_device())
    T, ctx = a.prefill, a.prefill
    res = {"design": "Dimorax", "dtype": "bf16", "data": "synthetic", "prompt_tokens": T, "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    for name, s in DIMORAX_SIZES.items():
        t0 = time.time()
        m = build_dimorax(s, dev)
        new = end_to_end(m, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del m
        torch.cuda.empty_cache()
        d = build_lotazen(lotazen_like_dimorax(s), dev)
        old = end_to_end(d, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del d
        torch.cuda.empty_cache()
        res["sizes"][name] = {"config": s, "layered": new, "lotazen_equal_size": old, "kernels": dimorax_kernel_table(s, T, ctx, peaks, dev),
                              "seconds": round(time.time() - t0, 1)}
    return res


# ----------------------------------------------------------------------------------------------- Pukarax
PUKARAX_SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, map_dim=64, chunk_a=2048, chunk_b=1024, experts=16, top=2, ff=1408, shared_ff=2816, dense_ff=5632, vocab=32768,
                  order="kdkd", loop=(1, 3, 2)),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, map_dim=64, chunk_a=4096, chunk_b=2048, experts=8, top=2, ff=3584, shared_ff=7168, dense_ff=14336, vocab=32768,
                  order="dkd", loop=None),
}


def pukarax_config(s: dict) -> dict:
    d = s["dim"]
    mixers = {
        "d": {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["map_dim"], "vdim": d, "scale": s["map_dim"] ** -0.5, "diff": 0.5,
                                             "mask": {"size": s["chunk_a"]}, "rot": {"base": 500000.0, "dims": s["map_dim"]}}},
        "k": {"type": "attention_2", "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": s["chunk_b"]},
                                               "rot": {"base": 10000.0, "dims": d, "scaling": {"factor": 8.0}}}},
    }
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}, "shared": {"ff": s["shared_ff"]}}
    cfg = {"architecture": "Pukarax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0}, "logit_scale": 0.5,
           "layers": [{**mixers[c], "mlp": moe if i % 3 != 2 else {"kind": "dense", "ff": s["dense_ff"]}} for i, c in enumerate(s["order"])]}
    if s["loop"]:
        cfg["loop"] = dict(zip(("start", "stop", "times"), s["loop"]))
    return cfg


def build_pukarax(s: dict, dev):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer

    m = LayeredTransformer.empty(LayeredArgs.from_dict(pukarax_config(s)), dev, torch.bfloat16)
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for n, p in m.named_parameters():
            if "norm" in n:
                p.fill_(1.0)
            elif p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) / math.sqrt(p.shape[-1]))
            else:
                p.copy_(torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32) * 0.1)
    return m.eval()


def dimorax_like_pukarax(s: dict) -> dict:
    """The closest existing design at equal size: rotary softmax attention (over the whole sequence, one map of the value size per head) in every
    layer run, silu-gated experts with a shared expert and dense layers of the same sizes in the same places."""
    n = len(s["order"]) + ((s["loop"][1] - s["loop"][0]) * (s["loop"][2] - 1) if s["loop"] else 0)
    return dict(width=s["width"], heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"], lat_heads=1, lat_dim=64, rot_dim=32, kv_rank=64, window=64, rec_heads=1, rec_kv_heads=1,
                taps=1, rank=1, experts=s["experts"], top=s["top"], groups=1, keep=1, ff=s["ff"], shared_ff=s["shared_ff"], dense_ff=s["dense_ff"], vocab=s["vocab"], order="a" * n)


def pukarax_kernel_table(s: dict, T: int, ctx: int, peaks: dict, dev) -> dict:
    """Every kernel the design added or extended, alone at this size, each next to the like kernel of an existing design at the same shape."""
    from mistral_inference_b200 import _abi_hybrid as h
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec
    from mistral_inference_b200.rope import scaled_frequencies

    bf = torch.bfloat16
    W, H, G, d, dm, E, ff, sff, top, ca, cb = (s[k] for k in ("width", "heads", "kv_heads", "dim", "map_dim", "experts", "ff", "shared_ff", "top", "chunk_a", "chunk_b"))
    flush = torch.zeros(160 << 20, dtype=torch.float32, device=dev)
    rows = {}

    def rec(name, fn, flops=0.0, bytes_=0.0, note=None, n=(3, 8)):
        ms = _time(fn, n[0], n[1], flush)
        r = {"ms": round(ms, 4)}
        if flops:
            r["tflops"] = round(flops / ms / 1e9, 2)
            r["of_bf16_peak"] = round(flops / ms / 1e9 / peaks["bf16_tflops"], 4)
        if bytes_:
            r["gb_s"] = round(bytes_ / ms / 1e6, 1)
            r["of_hbm_peak"] = round(bytes_ / ms / 1e6 / peaks["hbm_gbs"], 3)
        if note:
            r["note"] = note
        rows[name] = r

    def rnd(*shape, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(bf)

    B, nt = 8, (T + 63) // 64
    # ---- norms
    x32, y32, nw = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev), torch.ones(W, device=dev).to(bf)
    rec("rmsnorm_add_norm prompt (add, then the next norm)", lambda: h.rmsnorm_add(y32, nw, x32, 1e-5, w_next=nw), bytes_=T * W * 14.0)
    rec("like: rmsnorm_add prompt", lambda: h.rmsnorm_add(y32, nw, x32, 1e-5), bytes_=T * W * 12.0)
    yB, xB = y32[:B].contiguous(), x32[:B].contiguous()
    rec(f"rmsnorm_add_norm decode B={B}", lambda: h.rmsnorm_add(yB, nw, xB, 1e-5, w_next=nw), bytes_=B * W * 14.0, note="latency")
    rec(f"like: rmsnorm_add, then rmsnorm, decode B={B}", lambda: (h.rmsnorm_add(yB, nw, xB, 1e-5), h.rmsnorm(xB, nw, 1e-5)), bytes_=B * W * 18.0, note="latency, two launches")
    # ---- rotation
    specs = {"diff": LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=2 * dm, v_dim=d, window=ca), "keyval": LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d, window=cb),
             "like": LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d, window=ca), "like_b": LayerCacheSpec(kind="ring", n_kv_heads=G, k_dim=d, v_dim=d, window=cb)}
    ring = BufferCache(4, B, ctx + 8, 0, 0, None, layer_specs=list(specs.values())).to(dev, bf)
    for i in range(4):
        ring.cache_k[i].normal_()
        ring.cache_v[i].normal_()
    mds = dict(zip(specs, ring.get_input_metadata([T])))
    md = mds["like"]
    fm, fd = scaled_frequencies(dm, 5e5, None)[0].to(dev), scaled_frequencies(d, 1e4, None)[0].to(dev)
    qkv_d, qkv_k, qkv = rnd(T, (2 * H + 2 * G) * dm + G * d + 64), rnd(T, (H + G) * d + H * d), rnd(T, (H + 2 * G) * d)
    rot_d = lambda: h.rot_prep(qkv_d, fm, md.positions, None, None, None, 2 * H, 2 * G, dm, d, dm, False, 0.0, own=True, v_heads=G)  # noqa: E731
    rot_k = lambda: h.rot_prep(qkv_k, fd, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True, halves=True, v_off=H * d)  # noqa: E731
    rec("rot_prep prompt (two maps, neighbours)", rot_d, bytes_=T * 4.0 * ((2 * H + 2 * G) * dm + G * d))
    rec("rot_prep prompt (keys as values, halves, unit norm)", rot_k, bytes_=T * 2.0 * ((H + G) * d + (H + 2 * G) * d))
    rec("like: rot_prep prompt (neighbours, unit norm)", lambda: h.rot_prep(qkv, fd, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True), bytes_=4.0 * qkv.numel())
    # ---- attention
    qd, kd, vd = rot_d()
    qk, kk, vk = rot_k()
    ql, kl, vl = h.rot_prep(qkv, fd, md.positions, None, None, None, H, G, d, d, d, True, 1e-5, own=True)
    o, lam, gates = torch.empty(T, H * d, device=dev, dtype=bf), torch.full((1,), 0.5, device=dev), rnd(T, H * d)
    diff = dict(lam=lam, out_scale=0.5, norm_eps=1e-5)
    pairs_chunk = lambda c: sum(p % c + 1 for p in range(T))  # noqa: E731
    pairs_win = lambda c: sum(min(p + 1, c) for p in range(T))  # noqa: E731

    def prompt(name, q, k, v, key, dk, c, flops, **kw):
        m_, i = mds[key], list(specs).index(key)
        rec(name, lambda: h.attn_window(q, ring.cache_k[i], ring.cache_v[i], m_.positions, m_.q_start, m_.slots, o, 1, m_.window, H, G, dk, d, 0.09, c, own_k=k, own_v=v,
                                        seqpos=m_.seqpos, n_tiles=nt, **kw), flops=flops, n=(2, 5))

    prompt(f"differential attention prompt, chunks of {ca}, head gate", qd, kd, vd, "diff", dm, ca, 4.0 * H * (dm + d) * pairs_chunk(ca), chunked=True, gate=gates[:, :H], **diff)
    prompt(f"like: softmax attention prompt, window {ca}", ql, kl, vl, "like", d, ca, 4.0 * H * d * pairs_win(ca))
    prompt(f"attention prompt, chunks of {cb}, entry gate", qk, kk, vk, "keyval", d, cb, 4.0 * H * d * pairs_chunk(cb), chunked=True, gate=gates, gate_entry=True)
    prompt(f"like: softmax attention prompt, window {cb}", ql, kl, vl, "like_b", d, cb, 4.0 * H * d * pairs_win(cb))
    at = ca - 1 if ca - 1 <= ctx else ctx  # the last token of a chunk: it sees the whole chunk
    ring.reset(); ring.init_kvseqlens(B); ring.update_seqlens([at] * B)
    md2 = dict(zip(specs, ring.get_input_metadata([1] * B)))
    oB = torch.empty(B, H * d, device=dev, dtype=bf)

    def decode(name, q, key, dk, c, **kw):
        m_, i, qB = md2[key], list(specs).index(key), q[:B].contiguous()
        rec(f"{name} B={B}", lambda: h.attn_decode(qB, ring.cache_k[i], ring.cache_v[i], m_.positions, m_.slots, oB, B, m_.window, H, G, dk, d, 0.09, c, **kw),
            bytes_=B * min(at + 1, c) * G * 2.0 * (d + dk * (2 if "lam" in kw else 1)))

    decode(f"differential attention decode, chunks of {ca}, head gate", qd, "diff", dm, ca, chunked=True, gate=gates[:B, :H], **diff)
    decode(f"like: softmax attention decode, window {ca}", ql, "like", d, ca)
    decode(f"attention decode, chunks of {cb}, entry gate", qk, "keyval", d, cb, chunked=True, gate=gates[:B], gate_entry=True)
    decode(f"like: softmax attention decode, window {cb}", ql, "like_b", d, cb)
    m_, sp_ch = md2["like"], h.window_decode_plan(B, H, md2["like"].window)
    qB = ql[:B].contiguous()
    rec(f"like: softmax attention decode, window {ca}, a CTA per query head B={B}",
        lambda: h.attn_window(qB, ring.cache_k[2], ring.cache_v[2], m_.positions, m_.q_start, m_.slots, oB, B, m_.window, H, G, d, d, 0.09, ca, splits=sp_ch[0], chunk=sp_ch[1]),
        bytes_=B * min(at + 1, ca) * G * 4.0 * d)
    # ---- feed-forward
    x = rnd(T, W)
    al = sff // ff
    w13, w2, wr, wb = rnd((E + al) * 2 * ff, W, scale=0.02), rnd(W, (E + al) * ff, scale=0.02), rnd(E, W, scale=4 / math.sqrt(W)), torch.zeros(E, device=dev).to(bf)
    route = lambda t: h.moe_route(t, wr, None, 1, 1, top, score=2, w_bias=wb, always=al)  # noqa: E731
    rec("moe_route prompt (softmax over the chosen)", lambda: route(x), bytes_=T * W * 2.0)
    rec("like: moe_route prompt (sigmoid)", lambda: h.moe_route(x, wr, None, 1, 1, top, score=1), bytes_=T * W * 2.0)
    dense, idx, wsel = route(x)
    l13, l2, s13, s2 = w13[: E * 2 * ff], w2[:, : E * ff].contiguous(), w13[E * 2 * ff:], w2[:, E * ff:].contiguous()
    d_like, i_like, w_like = h.moe_route(x, wr, None, 1, 1, top, score=1)
    ones = torch.ones(T, 1, device=dev)
    fl = 6.0 * T * (top * ff + sff) * W

    def like_prompt():
        y = h.linear(h.linear_swiglu(x, l13, rowscale=d_like, group=ff), l2, epi=h.EPI_F32)
        return h.linear(h.linear_swiglu(x, s13, rowscale=ones, group=sff), s2, epi=h.EPI_RESIDUAL, residual=y)

    rec("experts prompt (shared expert among them)", lambda: h.linear(h.linear_swiglu(x, w13, rowscale=dense, group=ff), w2, epi=h.EPI_F32), flops=fl, n=(2, 5),
        note=f"useful FLOPs (top {top} of {E} + shared); the kernels compute all {E} experts")
    rec("like: experts prompt, shared expert of its own", like_prompt, flops=fl, n=(2, 5))
    for M in (1, B):
        xs, ii, ww, il, wl = (t[:M].contiguous() for t in (x, idx, wsel, i_like, w_like))

        def like_decode():
            y = h.moe_sparse(xs, l13, l2, il, wl, E, ff)
            return h.linear(h.linear_swiglu(xs, s13), s2, epi=h.EPI_RESIDUAL, residual=y)

        by = 3.0 * W * 2 * ff * (len(set(ii[:, :top].flatten().tolist())) + al)
        rec(f"experts decode (chosen and shared) M={M}", lambda: h.moe_sparse(xs, w13, w2, ii, ww, E + al, ff), bytes_=by, note="bytes: every weight that is used, once")
        rec(f"like: experts decode, shared expert of its own M={M}", like_decode, bytes_=by)
    return rows


def run_pukarax(a, peaks: dict) -> dict:
    dev = torch.device("cuda", torch.cuda.current_device())
    T, ctx = a.prefill, a.prefill - 128  # decode steps near the end of a chunk, where they read most of it (both models at the same place)
    res = {"design": "Pukarax", "dtype": "bf16", "data": "synthetic", "prompt_tokens": T, "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    for name, s in PUKARAX_SIZES.items():
        t0 = time.time()
        m = build_pukarax(s, dev)
        new = end_to_end(m, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del m
        torch.cuda.empty_cache()
        d = build_dimorax(dimorax_like_pukarax(s), dev)
        old = end_to_end(d, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del d
        torch.cuda.empty_cache()
        res["sizes"][name] = {"config": s, "layered": new, "dimorax_equal_size": old, "kernels": pukarax_kernel_table(s, T, ctx, peaks, dev),
                              "seconds": round(time.time() - t0, 1)}
    return res


def run(a, peaks: dict) -> dict:
    if a.design == "pukarax":
        return run_pukarax(a, peaks)
    if a.design == "dimorax":
        return run_dimorax(a, peaks)
    if a.design == "viladra":
        return run_viladra(a, peaks)
    if a.design == "taruvik":
        return run_taruvik(a, peaks)
    if a.design == "lotazen":
        return run_lotazen(a, peaks)
    dev = torch.device("cuda", torch.cuda.current_device())
    T, ctx = a.prefill, a.prefill
    res = {"design": "Fesenex", "dtype": "bf16", "data": "synthetic", "prompt_tokens": T, "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    for name, s in SIZES.items():
        t0 = time.time()
        m = build_layered(s, dev)
        new = end_to_end(m, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del m
        torch.cuda.empty_cache()
        d = build_dense(s, dev)
        old = end_to_end(d, s["vocab"], T, ctx, (1, 8), a.warmup, a.steps, dev)
        del d
        torch.cuda.empty_cache()
        res["sizes"][name] = {"config": s, "layered": new, "dense_transformer": old, "kernels": kernel_table(s, T, ctx, peaks, dev),
                              "seconds": round(time.time() - t0, 1)}
    return res
