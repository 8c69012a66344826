"""The Pukarax design on the GPU against the plain statement in tests/pukarax_oracle.py: every mechanism alone (router, experts with the shared
expert among or beside them, scaled logits, the chained norms, rotation with values out of the keys, attention in chunks with one and two maps
and output gates), then whole models of several shapes through the cache: prompts against token-by-token decoding, portions, ragged batches,
reused rows, chunk edges, far keys, looped layers, long decoding, and greedy generation through `generate()`.  fp32 runs are compared tightly,
bf16 runs by an error norm per token."""
import math

import pytest
import torch

from tests import pukarax_oracle as O
from tests.pukarax_util import dense_cfg, diff_cfg, f32, keyval_cfg, make_config, make_weights, moe_cfg, write_folder

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]

SHAPES = {
    # nothing a multiple of 8 or 32 where it need not be; query heads in groups of 2 and 3; a layer without chunks, one without feed-forward; the
    # shared expert beside the experts, among them (twice their size), and none
    "odd": dict(width=40, vocab=50, loop=(1, 3, 2), layers=[
        (keyval_cfg(), moe_cfg()), (diff_cfg(), dense_cfg()), (keyval_cfg(4, 2, 10, size=3, factor=None), None), (diff_cfg(6, 2, 5, 9, size=None), moe_cfg(shared=24)),
        (diff_cfg(2, 2, 8, 3, rot=(40.0, 8), size=11), moe_cfg(ff=10, experts=3, top=1, shared=None))]),
    # head sizes of the tensor-core prompt kernels, chunks across and along their 64-key tiles
    "tc": dict(width=64, vocab=70, layers=[
        (diff_cfg(4, 2, 32, 64, 0.2, (1e4, 24), size=50), moe_cfg(ff=32, experts=8, top=3, shared=64)), (keyval_cfg(4, 1, 64, 0.15, (1e4, 32), 4.0, size=64), dense_cfg(32)),
        (diff_cfg(2, 1, 64, 128, 0.15, (1e4, 64), size=None), None), (keyval_cfg(2, 2, 32, 0.2, (5e3, 32), None, size=96), moe_cfg(ff=16, experts=4, top=4, shared=16))]),
    # odd width and vocabulary, a value size below 8, three query heads on one key head, a span of one layer that runs four times
    "awkward": dict(width=31, vocab=17, loop=(0, 1, 4), layers=[
        (diff_cfg(3, 1, 7, 5, 0.5, (50.0, 6)), moe_cfg(ff=7, experts=3, top=2, shared=5)), (keyval_cfg(3, 1, 9, 0.5, (20.0, 2), 1.5, size=2), dense_cfg(7))]),
    # everything 1: one head, one expert, chunks of one token, factors of 1, a loop that runs once
    "one": dict(width=24, vocab=20, embed_scale=1.0, logit_scale=1.0, loop=(0, 2, 1), layers=[
        (diff_cfg(1, 1, 4, 4, 1.0, (10.0, 2), size=1, diff=0.0), moe_cfg(ff=8, experts=1, top=1, shared=8)), (keyval_cfg(1, 1, 8, 1.0, (10.0, 8), 1.0, size=1), dense_cfg(8)),
        (keyval_cfg(1, 1, 2, 1.0, (10.0, 2), 1.0, size=4), None)]),
}
MIXER_LAYERS = {
    "diff": diff_cfg(), "diff_whole": diff_cfg(size=None), "diff_tc": diff_cfg(4, 1, 64, 64, 0.15, (1e4, 48), size=40), "diff_tc_whole": diff_cfg(2, 2, 32, 32, 0.2, (1e4, 16), size=None),
    "diff_wide": diff_cfg(2, 1, 20, 200, 0.3, (1e3, 20), size=30), "diff_large_diff": diff_cfg(3, 3, 12, 16, 0.4, (1e3, 6), size=25, diff=0.9), "diff_128": diff_cfg(2, 1, 128, 128, 0.1, (1e4, 96), size=70),
    "keyval": keyval_cfg(), "keyval_whole": keyval_cfg(size=None), "keyval_tc": keyval_cfg(6, 2, 96, 0.1, (1e4, 96), 3.0, size=65), "keyval_unscaled": keyval_cfg(4, 4, 16, 0.4, (100.0, 16), None, size=33),
    "keyval_256": keyval_cfg(2, 1, 256, 0.1, (1e4, 128), 8.0, size=20), "keyval_odd": keyval_cfg(3, 3, 11, 0.5, (30.0, 6), 1.25, size=31),
}


def _model(tmp_path, name, dtype, seed=0, weights=None, **over):
    from mistral_inference_b200.registry import load_model

    cfg = make_config(**{**SHAPES[name], **over}) if isinstance(name, str) else name
    w = weights if weights is not None else make_weights(cfg, seed)
    m = load_model(write_folder(tmp_path / "m", cfg, w), device=DEV, dtype=dtype)
    if dtype == torch.bfloat16:  # the oracle sees the rounded weights
        w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    return m, cfg, f32(w)


def _tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _close(got, ref, dtype, what="", tol=3e-4):
    got, ref = got.float().cpu(), ref.float().cpu()
    if dtype == torch.float32:
        torch.testing.assert_close(got, ref, rtol=tol, atol=tol, msg=lambda m: f"{what}: {m}")
    else:
        # per token: most are within bf16 rounding; a near tie of a router turns the other way for a few tokens in a hundred
        got, ref = got.reshape(-1, got.shape[-1]), ref.reshape(-1, ref.shape[-1])
        err = (got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean(-1).sqrt().clamp_min(1e-6)
        assert err.median() < 0.04, f"{what}: median relative rms error {err.median():.4f}"
        assert int((err > 0.25).sum()) <= max(1, len(err) // 10), f"{what}: {int((err > 0.25).sum())} of {len(err)} tokens are far off ({err.max():.3f})"


def _run(m, pieces, cache=None, taps=None):
    """Feeds one sequence in `pieces` (lists of tokens) through one cache row; returns the logits of all tokens."""
    cache = cache or m.make_cache(1, sum(len(p) for p in pieces))
    m._tap = (lambda r, x: taps.setdefault(r, []).append(x.clone())) if taps is not None else None
    try:
        out = [m.forward(torch.tensor(p, device=DEV), [len(p)], cache) for p in pieces]
    finally:
        m._tap = None
    return torch.cat(out)


def _cut(toks, sizes):
    out, o = [], 0
    for c in sizes:
        out.append(toks[o:o + c])
        o += c
    assert o == len(toks)
    return out


def _i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device=DEV)


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 40])
@pytest.mark.parametrize("D", [37, 40, 516, 2048, 5000, 9000])
def test_norm_that_adds_and_the_next_one(dtype, T, D):
    """The norm of a sublayer's output added to the stream, and the next norm of the result, in one kernel."""
    from mistral_inference_b200.transformer_layers import Norm

    g = torch.Generator().manual_seed(D)
    a, b = Norm(D, 1e-3, "rms").to(DEV).to(dtype), Norm(D, 1e-3, "rms").to(DEV).to(dtype)
    for n in (a, b):
        n.load_weight((1 + 0.3 * torch.randn(D, generator=g)).to(dtype))
    y, x = torch.randn(T, D, generator=g) * torch.logspace(-3, 3, T)[:, None], torch.randn(T, D, generator=g)
    acc = x.to(DEV)
    nxt = a(y.to(DEV), add_to=acc, then=b)
    want = x + O.norm(y, a.weight.float().cpu(), 1e-3)
    _close(acc, want, torch.float32, tol=1e-5)
    _close(nxt, O.norm(want, b.weight.float().cpu(), 1e-3).to(dtype), torch.float32, tol=1e-5 if dtype == torch.float32 else 2e-2)
    acc2 = x.to(DEV)
    a(y.to(DEV), add_to=acc2)
    torch.testing.assert_close(acc, acc2, rtol=1e-6, atol=1e-6)


@pytest.mark.parametrize("E,top,always,T", [(6, 2, 0, 60), (12, 5, 2, 7), (40, 6, 1, 33), (7, 7, 3, 1), (1, 1, 0, 5), (200, 9, 40, 4)])
def test_router_softmax_over_the_chosen(E, top, always, T):
    """Biases that decide, weights that leave the unchosen logits out, large logits (no overflow), further experts for every token."""
    from mistral_inference_b200 import _abi_hybrid as h

    g = torch.Generator().manual_seed(E)
    x, wr, b = torch.randn(T, 24, generator=g) * 8, torch.randn(E, 24, generator=g), torch.randn(E, generator=g) * 30
    dense, idx, wsel = h.moe_route(x.to(DEV), wr.to(DEV), None, 1, 1, top, score=2, w_bias=b.to(DEV), always=always)
    assert dense.shape == (T, E + always) and idx.shape == wsel.shape == (T, top + always)
    for t in range(T):
        ref = O.route(x[t].double(), {"router": wr.double(), "router.b": b.double()}, "", {"top": top})
        assert idx[t].tolist() == [e for e, _ in ref] + list(range(E, E + always)), t
        vals = torch.tensor([v for _, v in ref] + [1.0] * always)
        _close(wsel[t], vals, torch.float32, tol=2e-5)
        row = torch.zeros(E + always)
        row[idx[t].long().cpu()] = vals
        _close(dense[t], row, torch.float32, tol=2e-5)
    assert abs(float(wsel[:, :top].sum()) - T) < 1e-4 * T


def test_router_leaves_the_unchosen_out():
    """With equal logits a softmax over all outputs and one over the chosen ones differ by a factor of E / top."""
    from mistral_inference_b200 import _abi_hybrid as h

    x, wr, b = torch.ones(1, 4, device=DEV), torch.zeros(8, 4, device=DEV), torch.zeros(8, device=DEV)
    b[5] = 1.0
    _, idx, wsel = h.moe_route(x, wr, None, 1, 1, 2, score=2, w_bias=b)
    assert idx.tolist() == [[5, 0]]
    _close(wsel[0], torch.softmax(torch.tensor([1.0, 0.0]), 0), torch.float32, tol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 5, 16, 17, 150])
@pytest.mark.parametrize("f", [moe_cfg(), moe_cfg(ff=32, experts=4, top=1, shared=None), moe_cfg(ff=16, experts=3, top=3, shared=16), moe_cfg(ff=10, experts=5, top=2, shared=30)])
def test_experts(dtype, T, f):
    """The feed-forward alone, dense (prompts) and sparse (few tokens), behind a norm and straight into the stream."""
    from mistral_inference_b200.args import ChosenSoftmaxMoeArgs
    from mistral_inference_b200.transformer_layers import ChosenSoftmaxMoe, Norm

    cfg = make_config(layers=[(diff_cfg(), f)])
    w = {k: v.to(dtype) for k, v in make_weights(cfg, 5).items()}
    ff = ChosenSoftmaxMoe(40, ChosenSoftmaxMoeArgs.from_dict(f)).to(DEV).to(dtype)
    for n in ff.checkpoint_names():
        assert ff.assign(n, lambda dst: dst.copy_(w["l0.mlp." + n]))
    hs, x0 = torch.randn(T, 40).to(dtype), torch.randn(T, 40)
    want = O.moe(hs.float(), f32(w), "l0.mlp.", f)
    x32 = x0.to(DEV)
    ff.run(hs.to(DEV), x32, None)
    _close(x32 - x0.to(DEV), want, dtype, f"T={T}")
    post = Norm(40, 1e-3, "rms").to(DEV).to(dtype)
    post.load_weight(w["l0.norm2b"])
    x32 = x0.to(DEV)
    ff.run(hs.to(DEV), x32, post)
    _close(x32 - x0.to(DEV), O.norm(want, w["l0.norm2b"].float(), 1e-3), dtype, f"T={T}, normed")


@pytest.mark.parametrize("glu", [0, 1, 2])
@pytest.mark.parametrize("T", [2, 3, 8, 9, 16])
@pytest.mark.parametrize("E,top,ff,width,identity", [(4, 2, 24, 40, 0), (3, 3, 8, 304, 0), (40, 2, 16, 72, 2), (1, 1, 72, 24, 0)])
def test_experts_of_several_tokens(glu, T, E, top, ff, width, identity):
    """Expert by expert on tensor cores against one token at a time: experts that nobody, one or all tokens chose, identity experts, results stored
    and added."""
    from mistral_inference_b200 import _abi_hybrid as h

    g = torch.Generator().manual_seed(T * E)
    bf = lambda *sh: torch.randn(*sh, generator=g).to(torch.bfloat16).to(DEV)  # noqa: E731
    x, w13, w2 = bf(T, width), bf(E * ff * (1 if glu == 2 else 2), width) * 0.2, bf(width, E * ff) * 0.2
    idx = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(T)]).to(torch.int32).to(DEV)
    wsel, base = torch.rand(T, top, generator=g).to(DEV), torch.randn(T, width, generator=g).to(DEV)
    kw = dict(glu=glu, limit=1.5, alpha=1.7)
    for add in (False, True):
        got = h.moe_sparse(x, w13, w2, idx, wsel, E, ff, add_to=base.clone() if add else None, **kw)
        one = torch.cat([h.moe_sparse(x[t:t + 1], w13, w2, idx[t:t + 1].contiguous(), wsel[t:t + 1].contiguous(), E, ff, add_to=base[t:t + 1].clone() if add else None, **kw)
                         for t in range(T)])
        torch.testing.assert_close(got, one, rtol=3e-2, atol=3e-2 * float(one.abs().max().clamp_min(1.0)))
        assert (got - one).norm() < 1e-2 * one.norm()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 6, 70])
def test_silu_feed_forward(dtype, T):
    from mistral_inference_b200.args import SiluGluArgs
    from mistral_inference_b200.transformer_layers import SiluGlu

    cfg = make_config(layers=[(diff_cfg(), dense_cfg(27))])
    w = {k: v.to(dtype) for k, v in make_weights(cfg, 2).items()}
    ff = SiluGlu(40, SiluGluArgs(27)).to(DEV).to(dtype)
    for n in ff.checkpoint_names():
        assert ff.assign(n, lambda dst: dst.copy_(w["l0.mlp." + n]))
    hs, x0 = torch.randn(T, 40).to(dtype), torch.randn(T, 40)
    x32 = x0.to(DEV)
    ff.run(hs.to(DEV), x32, None)
    _close(x32 - x0.to(DEV), O.gated(hs.float(), f32(w), "l0.mlp."), dtype, f"T={T}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M", [1, 5, 60, 200])
@pytest.mark.parametrize("N", [96, 128, 51])
def test_scaled_logits(dtype, M, N):
    """The factor on the logits, alone and behind a soft cap, in every Linear kernel and behind the prompt GEMM (128 columns, 200 rows)."""
    from mistral_inference_b200 import _abi_hybrid as h

    g = torch.Generator().manual_seed(M)
    x, w = torch.randn(M, 64, generator=g).to(dtype), (torch.randn(N, 64, generator=g) * 0.3).to(dtype)
    z = x.double() @ w.double().T
    for kw, want in ((dict(alpha=-1.6), -1.6 * z), (dict(alpha=0.5, limit=2.0), torch.tanh(z / 2.0)), ({}, z)):
        got = h.linear(x.to(DEV), w.to(DEV), epi=h.EPI_F32, **kw)
        _close(got, want, torch.float32, str(kw), tol=1e-4 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dims,halves,norm", [(17, 8, True, True), (12, 12, True, True), (64, 32, True, True), (7, 6, False, False), (48, 48, False, False), (250, 2, False, True)])
def test_rotation_with_keys_as_values(dtype, d, dims, halves, norm):
    """Queries and keys rotated (and normed), values the keys as projected; the gate's columns behind them are left alone.  Far positions."""
    from mistral_inference_b200 import _abi_hybrid as h

    H, G, T, start, extra, eps = 3, 2, 20, 3000, 9, 1e-2
    f = torch.tensor([500.0 ** (-2.0 * i / dims) / 2.5 for i in range(dims // 2)], dtype=torch.float64, device=DEV)
    x = torch.randn(T, (H + G) * d + extra, generator=torch.Generator().manual_seed(d)).to(dtype)
    ring_k, ring_v = torch.zeros(40, G * d, dtype=dtype, device=DEV), torch.zeros(40, G * d, dtype=dtype, device=DEV)
    rows = [i if i % 3 else -1 for i in range(T)]
    q, k, v = h.rot_prep(x.to(DEV), f, _i32(range(start, start + T)), _i32(rows), ring_k, ring_v, H, G, d, d, dims, norm, eps, own=True, halves=halves, v_off=H * d)

    def ref(t, heads):
        full = torch.cat([torch.zeros(start, heads, d), t.float().view(T, heads, d)]).double()
        rot = {"base": 500.0, "dims": dims}
        y = (O.rotate_halves(full, {**rot, "scaling": {"factor": 2.5}}) if halves else _slow_neighbours(full, rot, 2.5))[start:]
        return (O.unit_rms(y, eps) if norm else y).reshape(T, -1)

    tol = 1e-5 if dtype == torch.float32 else 2e-2
    _close(q, ref(x[:, : H * d], H), torch.float32, tol=tol)
    _close(k, ref(x[:, H * d: (H + G) * d], G), torch.float32, tol=tol)
    assert torch.equal(v.cpu(), x[:, H * d: (H + G) * d])
    for i, r in enumerate(rows):
        if r >= 0:
            assert torch.equal(ring_k[r], k[i]) and torch.equal(ring_v[r], v[i])
        else:
            assert float(ring_k[i].abs().sum()) == 0.0


def _slow_neighbours(x, rot, factor):
    out, n = x.clone(), rot["dims"]
    out[..., 0:n:2], out[..., 1:n:2] = O.turn(x[..., 0:n:2], x[..., 1:n:2], O.angles(x.shape[0], rot, factor))
    return out


def _attend(q, k, v, H, G, d, e, scale, size, gate, entry, lam, diff, eps):
    """q [T, H*maps*d], k [T, G*maps*d], v [T, G*e] -> [T, H*e] from the plain statement."""
    T, maps = q.shape[0], 1 if lam is None else 2
    q, k, v = q.float().view(T, H, maps, d), k.float().view(T, G, maps, d), v.float().view(T, G, e)
    rows = []
    for h in range(H):
        g = h // (H // G)
        m = [O.softmax_map(q[:, h, i], k[:, g, i], v[:, g], scale, size) for i in range(maps)]
        o = m[0] if maps == 1 else O.difference(m[0], m[1], lam, diff, eps)
        if gate is not None:
            o = o * torch.sigmoid(gate.float()[:, h * e: (h + 1) * e] if entry else gate.float()[:, h: h + 1])
        rows.append(o)
    return torch.cat(rows, -1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("gate", [None, "head", "entry"])
@pytest.mark.parametrize("d,e,H,G", [(12, 10, 4, 2), (64, 64, 4, 1), (32, 64, 6, 3), (64, 128, 2, 1), (96, 96, 2, 2), (128, 128, 2, 1), (200, 130, 1, 1), (5, 256, 2, 1)])
def test_attention_core(dtype, maps, gate, d, e, H, G):
    """Chunks, two maps and gates in the exact kernel (one CTA and split keys) and in the tensor-core one: a prompt, and its last tokens alone over
    a ring (token 129 opens a chunk of 43, token 128 closes one)."""
    for size in (None, 1, 20, 43, 64, 65, 100):
        _attention_core(dtype, maps, gate, d, e, H, G, size)


def _attention_core(dtype, maps, gate, d, e, H, G, size):
    from mistral_inference_b200 import _abi_hybrid as h

    T, eps, diff = 150, 1e-3, 0.4
    g = torch.Generator().manual_seed(d)
    q, k, v = (torch.randn(T, n, generator=g).to(dtype) for n in (H * maps * d, G * maps * d, G * e))
    wide = torch.randn(T, 6 + H * e, generator=g).to(dtype)  # the gate is some columns of a wider matrix
    gt = None if gate is None else wide[:, 4: 4 + (H * e if gate == "entry" else H)]
    scale = 3.0 / math.sqrt(d)
    lam = torch.tensor([0.7]) if maps == 2 else None
    ref = _attend(q, k, v, H, G, d, e, scale, size, gt, gate == "entry", lam, diff, eps)
    W = min(size or T, T)
    ck, cv = torch.zeros(2, W, G, maps * d, dtype=dtype, device=DEV), torch.zeros(2, W, G, e, dtype=dtype, device=DEV)
    kw = dict(chunked=size is not None, lam=lam.to(DEV) if maps == 2 else None, out_scale=1 - diff, norm_eps=eps, gate_entry=gate == "entry")
    wide = wide.to(DEV)
    gd = None if gate is None else wide[:, 4: 4 + gt.shape[1]]
    slots = _i32([1])
    for tiles in (0, (T + 63) // 64):
        out = torch.empty(T, H * e, dtype=dtype, device=DEV)
        h.attn_window(q.to(DEV), ck, cv, _i32(range(T)), _i32([0, T]), slots, out, 1, W, H, G, d, e, scale, size or 0, own_k=k.to(DEV), own_v=v.to(DEV), seqpos=_i32([0]),
                      n_tiles=tiles, gate=gd, **kw)
        _close(out, ref, dtype, f"prompt, {tiles} tiles", tol=3e-5)
    for n in (T, 130, 129):  # the ring as it is when token n - 1 asks
        rows = [W + (p % W) if n - W <= p < n else -1 for p in range(T)]
        h.kv_scatter(k.to(DEV), v.to(DEV), _i32(rows), ck, cv)
        for splits, chunk in ((1, 0), (1, 7), (3, 16), (9, 32)):
            out = torch.empty(1, H * e, dtype=dtype, device=DEV)
            h.attn_window(q[n - 1: n].to(DEV), ck, cv, _i32([n - 1]), _i32([0, 1]), slots, out, 1, W, H, G, d, e, scale, size or 0, splits=splits, chunk=chunk,
                          gate=None if gd is None else gd[n - 1: n], **kw)
            _close(out, ref[n - 1: n], dtype, f"decode at {n - 1}, {splits} splits", tol=3e-5)
        if h.attn_decode_ok(q, H, G, d, e, maps):
            for splits in (1, 3, 64):
                out = torch.full((1, H * e), 9.0, dtype=dtype, device=DEV)
                h.attn_decode(q[n - 1: n].to(DEV), ck, cv, _i32([n - 1]), slots, out, 1, W, H, G, d, e, scale, size or 0, gate=None if gd is None else gd[n - 1: n], splits=splits, **kw)
                _close(out, ref[n - 1: n], dtype, f"grouped decode at {n - 1}, {splits} splits", tol=3e-5)


@pytest.mark.parametrize("H,G,d,e,W,window,chunked,softcap", [(16, 1, 64, 64, 300, 0, False, 0.0), (6, 2, 96, 64, 40, 40, False, 5.0), (4, 4, 32, 32, 7, 7, True, 0.0), (9, 1, 128, 128, 1000, 600, True, 2.0),
                                                              (8, 1, 64, 32, 5, 3, False, 0.0), (2, 1, 128, 64, 1, 1, True, 0.0)])
def test_grouped_decode_attention(H, G, d, e, W, window, chunked, softcap):
    """Sequences of unequal length in scattered rows of a ring against the exact kernel: sliding windows, chunks, soft caps, sinks, rings shorter than
    a piece of keys, groups of up to 16 query heads; keys outside a window are poisoned."""
    from mistral_inference_b200 import _abi_hybrid as h

    g = torch.Generator().manual_seed(W)
    pos, rows = [0, W // 2, W - 1, 3 * W + 1, 7 * W + W // 3], [4, 0, 6, 1, 3]
    if window == 0:
        pos = [min(p, W - 1) for p in pos]
    B = len(pos)
    ck, cv = torch.full((7, W, G, d), 30.0).to(torch.bfloat16), torch.full((7, W, G, e), 1e4).to(torch.bfloat16)
    for p, r in zip(pos, rows):
        lo = 0 if window == 0 else p - p % window if chunked else max(0, p - window + 1)
        for j in range(lo, p + 1):
            ck[r, j % W], cv[r, j % W] = torch.randn(G, d, generator=g), torch.randn(G, e, generator=g)
    q = torch.randn(B, H * d, generator=g).to(torch.bfloat16).to(DEV)
    sink = None if chunked else torch.randn(H, generator=g).to(DEV)
    outs = []
    for fn, extra in ((h.attn_decode, {}), (h.attn_window, dict(splits=3, chunk=32))):
        out = torch.empty(B, H * e, dtype=torch.bfloat16, device=DEV)
        pre = (q, ck.to(DEV), cv.to(DEV), _i32(pos)) + (() if fn is h.attn_decode else (_i32(range(B + 1)),))
        fn(*pre, _i32(rows), out, B, W, H, G, d, e, 2.0 / math.sqrt(d), window, chunked=chunked, softcap=softcap, sink=sink, **extra)
        outs.append(out)
    torch.testing.assert_close(outs[0].float(), outs[1].float(), rtol=2e-2, atol=2e-2)


def test_attention_rejects():
    """Combinations that have no meaning end in an error from the host, before any launch."""
    from mistral_inference_b200 import _abi_hybrid as h

    q, kv, out, one = torch.zeros(1, 16, device=DEV), torch.zeros(1, 4, 1, 8, device=DEV), torch.zeros(1, 8, device=DEV), _i32([0])
    lam = torch.ones(1, device=DEV)
    bad = [dict(window=0, chunked=True), dict(window=4, lam=lam, softcap=3.0), dict(window=4, lam=lam, sink=torch.zeros(1, device=DEV)), dict(window=4, lam=lam, head_bias=torch.zeros(1, device=DEV))]
    for kw in bad:
        with pytest.raises(h.Mb200Error):
            h.attn_window(q if "lam" in kw else q[:, :8].contiguous(), kv, kv, one, _i32([0, 1]), one, out, 1, 4, 1, 1, 8, 8, 1.0, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(MIXER_LAYERS))
def test_mixer_alone(tmp_path, dtype, kind):
    """A model of one layer without feed-forward: the stream after the layer, for a prompt, a prompt with decoded tokens and portions."""
    cfg = make_config(width=48, vocab=30, layers=[(MIXER_LAYERS[kind], None)])
    m, _, w = _model(tmp_path, cfg, dtype, seed=7)
    toks = _tokens(cfg, 90, 1)
    ref = []
    O.forward(cfg, w, toks, ref)
    for pieces in ([toks], [toks[:60]] + [[t] for t in toks[60:]], _cut(toks, [2, 17, 64, 7]), _cut(toks, [1, 1, 1, 1, 30, 56])):
        taps = {}
        _run(m, pieces, taps=taps)
        _close(torch.cat(taps[0]), ref[0], dtype, f"{kind} in {len(pieces)} pieces")


# ----------------------------------------------------------------------------- whole models through the cache
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SHAPES))
def test_prompt_decode_portions(tmp_path, dtype, name):
    m, cfg, w = _model(tmp_path, name, dtype)
    toks = _tokens(cfg, 150, 2)
    ref_taps = []
    ref = O.forward(cfg, w, toks, ref_taps)
    taps = {}
    whole = _run(m, [toks], taps=taps)
    assert len(taps) == len(ref_taps) == len(O.layer_order(cfg))
    for r in range(len(ref_taps)):
        _close(taps[r][0], ref_taps[r], dtype, f"{name} layer run {r}")
    _close(whole, ref, dtype, f"{name} whole")
    by_token = _run(m, [toks[:100]] + [[t] for t in toks[100:]])
    _close(by_token, ref, dtype, f"{name} prompt + 50 decoded")
    tol = dict(tol=2e-4) if dtype == torch.float32 else {}
    _close(by_token, whole, dtype, f"{name} decoded against whole", **tol)
    _close(_run(m, [[t] for t in toks]), whole, dtype, f"{name} from the first token on", **tol)
    for cuts in ([2] * 75, [7, 64, 3, 65, 11], [149, 1], [1, 149], [70, 80]):
        _close(_run(m, _cut(toks, cuts)), whole, dtype, f"{name} portions {cuts[:5]}", **tol)


def test_blocks_with_and_without_chained_norms(tmp_path):
    """The layers one by one, each computing its own norms, leave the same stream as the chain."""
    m, cfg, w = _model(tmp_path, "odd", torch.float32)
    toks = torch.tensor(_tokens(cfg, 60, 3), device=DEV)
    chained = m.forward(toks, [60], m.make_cache(1, 60))
    assert m._chained
    m._chained = False
    torch.testing.assert_close(m.forward(toks, [60], m.make_cache(1, 60)), chained, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "tc"])
def test_ragged_batch_retire_and_reuse(tmp_path, dtype, name):
    """Three unequal requests as one batch: prompts together (the second in portions), then token by token; the shorter ones end first.  Then
    other requests in the same rows (the rings of the first batch must not show)."""
    m, cfg, w = _model(tmp_path, name, dtype)
    cache = m.make_cache(3, 140)
    tol = dict(tol=2e-4) if dtype == torch.float32 else {}
    for round_, (portions, dec) in enumerate([([(70, 3, 100)], (20, 5, 30)), ([(1, 60, 33), (5, 40, 2)], (40, 3, 8))]):
        lens = [sum(p[i] for p in portions) for i in range(3)]
        reqs = [_tokens(cfg, n + d, 10 * round_ + i) for i, (n, d) in enumerate(zip(lens, dec))]
        alone = [_run(m, [r]) for r in reqs]
        if round_ == 0:
            _close(alone[0], O.forward(cfg, w, reqs[0]), dtype, "alone against the oracle")
        cache.reset()
        cache.init_kvseqlens(3)
        got, at = [[] for _ in reqs], [0, 0, 0]
        for p in portions:
            flat = [t for i in range(3) for t in reqs[i][at[i]: at[i] + p[i]]]
            lg = m.forward(torch.tensor(flat, device=DEV), list(p), cache)
            o = 0
            for i in range(3):
                got[i].append(lg[o:o + p[i]])
                o += p[i]
                at[i] += p[i]
        live, step = [0, 1, 2], 0
        while live:
            ended = [k for k, i in enumerate(live) if step >= dec[i]]
            if ended:
                cache.retire(ended)
                live = [i for k, i in enumerate(live) if k not in ended]
                if not live:
                    break
            lg = m.forward(torch.tensor([reqs[i][lens[i] + step] for i in live], device=DEV), [1] * len(live), cache)
            for k, i in enumerate(live):
                got[i].append(lg[k:k + 1])
            step += 1
        for i in range(3):
            _close(torch.cat(got[i]), alone[i], dtype, f"{name} round {round_} request {i}", **tol)


@pytest.mark.parametrize("phase", ["prompt", "decoded", "portions"])
@pytest.mark.parametrize("kind", ["diff", "keyval"])
@pytest.mark.parametrize("size,d", [(1, 6), (2, 6), (7, 6), (64, 32), (65, 32), (100, 32)])
def test_chunk_edges(tmp_path, phase, kind, size, d):
    """A marked token at the end of a chunk shows in its own chunk's tokens (there is one: itself) and not in the next chunk's first token; at the
    start of a chunk it shows up to the chunk's last token and not one further."""
    layer = diff_cfg(2, 1, d, 2 * d, 0.3, (100.0, d), size=size) if kind == "diff" else keyval_cfg(2, 1, d, 0.3, (100.0, d), 2.0, size=size)
    cfg = make_config(width=48, vocab=12, embed_scale=1.0, layers=[(layer, None)])
    w = make_weights(cfg, 3)
    w["embed"][:, 5] = 0
    w["embed"][11, 5] = 6.0               # token 11 is the mark, along one direction of the stream
    w["l0.mix.q"][:, 5] = 0
    w["l0.mix.q"] *= 0.1                  # nearly even attention
    w["l0.mix.g"].zero_()
    if kind == "diff":
        w["l0.mix.k"][:, 5] = 0
        w["l0.mix.v"][:, 5] *= 12.0       # ... that the values see
        w["l0.mix.lq1"].zero_()           # lambda = diff: the maps do not cancel
        w["l0.mix.lq2"].zero_()
    else:
        w["l0.mix.k"][:, 5] = 12.0 * torch.randn(d, generator=torch.Generator().manual_seed(1)) / 7
    first = 40 // size * size             # a chunk in the middle of the sequence
    n = first + 2 * size + 40
    for at in sorted({first, first + size - 1}):
        toks = [t % 11 for t in _tokens(cfg, n, size)]
        toks[at] = 11
        inside, outside = first + size - 1, first + size
        pieces = {"prompt": [toks], "decoded": [toks[: at + 1]] + [[t] for t in toks[at + 1:]],
                  "portions": [p for p in (toks[:at], toks[at: inside + 1], toks[inside + 1: inside + 3], toks[inside + 3:]) if p]}[phase]
        for dtype in DTYPES:
            m, _, wf = _model(tmp_path / f"{dtype}{at}", cfg, dtype, weights={k: v.clone() for k, v in w.items()})
            ref, plain = [], []
            O.forward(cfg, wf, toks, ref)
            O.forward(cfg, wf, [3 if i == at else t for i, t in enumerate(toks)], plain)
            show_in = (ref[0][inside] - plain[0][inside]).norm() if inside != at else (ref[0][at] - plain[0][at]).norm()
            assert show_in > 0.15 and torch.equal(ref[0][outside], plain[0][outside]), "the mark shows to the end of its chunk and not beyond"
            taps = {}
            _run(m, pieces, taps=taps)
            got = torch.cat(taps[0]).cpu()
            _close(got, ref[0], dtype, f"chunk {size} mark {at}")
            for i in (inside, outside):
                err = (got[i] - ref[0][i]).norm()
                assert err < 0.25 * show_in, (i, err, show_in)


@pytest.mark.parametrize("kind", ["diff", "keyval"])
@pytest.mark.parametrize("phase", ["prompt", "decoded"])
def test_far_key(tmp_path, kind, phase):
    """One query whose score with one key hundreds of tokens back stands out: it must be found, in a prompt and from the ring; and with the two
    maps of a head exchanged, or the second one left out, the result would be another."""
    n, size, at, ask = 560, 500, 3, 480
    d = 32
    layer = diff_cfg(2, 1, d, 64, 1.0, (1e4, 16), size=size, diff=0.3) if kind == "diff" else keyval_cfg(2, 1, d, 6.0, (1e4, 16), 4.0, size=size)
    cfg = make_config(width=48, vocab=40, embed_scale=1.0, layers=[(layer, None)])
    w = make_weights(cfg, 9)
    w["embed"] *= 0.5
    w["embed"][:38, [7, 9]] = 0
    w["embed"][38, 7], w["embed"][39, 9] = 8.0, 8.0          # 38 is the key, 39 asks for it
    free = 20                                                # an entry that no rotation touches
    maps = 2 if kind == "diff" else 1
    q, k = w["l0.mix.q"].view(2, maps, d, 48), w["l0.mix.k"].view(1, maps, d, 48)
    q *= 0.1
    k *= 0.3
    q[:, 0, free, 9] = 6.0                                   # in the first map only
    k[:, 0, free, 7] = 6.0
    toks = [t % 38 for t in _tokens(cfg, n, 1)]
    toks[at], toks[ask] = 38, 39
    for dtype in DTYPES:
        m, _, wf = _model(tmp_path / str(dtype), cfg, dtype, weights={kk: v.clone() for kk, v in w.items()})
        ref, without, other = [], [], []
        O.forward(cfg, wf, toks, ref)
        O.forward(cfg, wf, [5 if i == at else t for i, t in enumerate(toks)], without)
        delta = (ref[0][ask] - without[0][ask]).norm()
        assert delta > 0.5
        if kind == "diff":
            swapped = dict(wf)
            for nm in ("q", "q.b", "k", "k.b"):
                swapped["l0.mix." + nm] = wf["l0.mix." + nm].view(-1, 2, d, *wf["l0.mix." + nm].shape[1:]).flip(1).reshape(wf["l0.mix." + nm].shape)
            O.forward(cfg, swapped, toks, other)
            assert (other[-1][ask] - ref[0][ask]).norm() > 0.5
        taps = {}
        _run(m, [toks] if phase == "prompt" else [toks[:470]] + [[t] for t in toks[470:]], taps=taps)
        got = torch.cat(taps[0]).cpu()
        _close(got, ref[0], dtype, kind)
        assert (got[ask] - ref[0][ask]).norm() < 0.15 * delta


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path, dtype):
    """A prompt of 200 and 500 decoded tokens: the rings go round many times, and one layer keeps the whole sequence."""
    layers = [(keyval_cfg(size=40), moe_cfg()), (diff_cfg(size=None), None), (diff_cfg(2, 1, 8, 8, size=33), dense_cfg())]
    cfg = make_config(width=40, vocab=50, layers=layers, loop=(1, 3, 2))
    m, _, w = _model(tmp_path, cfg, dtype, seed=4)
    toks = _tokens(cfg, 700, 4)
    ref = O.forward(cfg, w, toks)
    _close(_run(m, [toks[:200]] + [[t] for t in toks[200:]]), ref, dtype, "long", tol=1e-3)
    _close(_run(m, [toks]), ref, dtype, "long prompt", tol=1e-3)


def test_passes_of_a_loop(tmp_path):
    """A looped span repeats its layers with the same weights and nothing in between: the unrolled model is the same."""
    cfg = make_config(**{**SHAPES["odd"], "loop": (1, 3, 3)})
    w = make_weights(cfg, 6)
    order = O.layer_order(cfg)
    flat = {**cfg, "layers": [cfg["layers"][i] for i in order]}
    del flat["loop"]
    wf = {k: v for k, v in w.items() if not k.startswith("l")}
    for r, i in enumerate(order):
        wf.update({f"l{r}." + k.split(".", 1)[1]: v.clone() for k, v in w.items() if k.startswith(f"l{i}.")})
    a, _, _ = _model(tmp_path / "a", cfg, torch.float32, weights=w)
    b, _, _ = _model(tmp_path / "b", flat, torch.float32, weights=wf)
    toks = _tokens(cfg, 60, 8)
    pieces = [toks[:40]] + [[t] for t in toks[40:]]
    torch.testing.assert_close(_run(a, pieces), _run(b, pieces), rtol=0, atol=0)


def test_first_tokens_and_rows_far_apart(tmp_path):
    """Sequences of 1, 2 and 3 tokens, and a sequence in the last row of a large cache."""
    m, cfg, w = _model(tmp_path, "odd", torch.float32)
    for n in (1, 2, 3):
        toks = _tokens(cfg, n, n)
        _close(_run(m, [toks]), O.forward(cfg, w, toks), torch.float32, f"{n} tokens")
        _close(_run(m, [[t] for t in toks]), O.forward(cfg, w, toks), torch.float32, f"{n} tokens, one by one")
    cache = m.make_cache(6, 64)
    cache.init_kvseqlens(1)
    cache._rows = [5]
    toks = _tokens(cfg, 40, 9)
    _close(_run(m, [toks[:30]] + [[t] for t in toks[30:]], cache=cache), O.forward(cfg, w, toks), torch.float32, "row 5")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tc", "odd"])
def test_generate_greedy(tmp_path, dtype, name):
    """Greedy generation through generate() (chunked prompts, the CUDA-graph decode step) repeats the oracle's choices wherever the
    oracle's best two logits are not close."""
    from mistral_inference_b200.generate import generate

    m, cfg, w = _model(tmp_path, name, dtype)
    m.args.max_batch_size = 2
    prompts = [_tokens(cfg, 70, 1), _tokens(cfg, 80, 2)]
    for chunk in (None, 16):
        out, lps = generate(prompts, m, max_tokens=12, temperature=0.0, chunk_size=chunk)
        checked = 0
        for p, o in zip(prompts, out):
            lg = O.forward(cfg, w, p + o)
            for i, tok in enumerate(o):
                row = lg[len(p) - 1 + i]
                top2 = torch.topk(row, 2).values
                if top2[0] - top2[1] > (0.02 if dtype == torch.float32 else 0.5):
                    assert tok == int(row.argmax()), (chunk, i)
                    checked += 1
        assert checked >= 8 and len(lps[0]) == len(prompts[0]) - 1 + 12


def test_command_line_and_trace_runner(tmp_path):
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    cfg = make_config(**SHAPES["odd"])
    w = make_weights(cfg, 0)
    folder = write_folder(tmp_path / "m", cfg, {k: v.to(torch.bfloat16) for k, v in w.items()})
    repo = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "mistral_inference_b200.main", "generate", str(folder), "--prompt", "1 2 3 4", "--max-tokens", "5", "--dtype", "float32"],
                       cwd=repo, capture_output=True, text=True)
    assert r.returncode == 0 and len(r.stdout.split()) == 5, r.stderr[-2000:]
    a, b = _tokens(cfg, 30, 1), _tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:25], "want": [0, 24]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[25:26], "want": []}, {"id": "b", "tokens": b[8:9], "want": [0]}], "end": ["b"]}]
    steps += [{"step": 2 + i, "entries": [{"id": "a", "tokens": [a[26 + i]], "want": [0]}], "end": ["a"] if i == 3 else []} for i in range(4)]
    steps += [{"step": 6, "entries": [{"id": "c", "tokens": b, "want": [8]}], "end": ["c"]}]
    r = subprocess.run([os.path.join(repo, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == [f"done {i}" for i in range(7)]
    wf = f32({k: v.to(torch.bfloat16) for k, v in w.items()})
    ra, rb = O.forward(cfg, wf, a), O.forward(cfg, wf, b)

    def rows(i):
        return torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))

    _close(rows(0), torch.stack([ra[0], ra[24], rb[7]]), torch.float32, "step 0")
    _close(rows(1), rb[8:9], torch.float32, "step 1")
    for i in range(4):
        _close(rows(2 + i), ra[26 + i:27 + i], torch.float32, f"step {2 + i}")
    _close(rows(6), rb[8:9], torch.float32, "a new batch in used rows")
