"""Host-side logic of the Pukarax design: configuration, registry, checkpoint packing, cache layout; and the plain statement's own sanity."""
import copy
import random

import pytest
import torch

from tests import pukarax_oracle as O
from tests.pukarax_util import dense_cfg, diff_cfg, keyval_cfg, make_config, make_weights, moe_cfg, write_folder


def _cfg():
    return make_config(layers=[(keyval_cfg(), moe_cfg()), (diff_cfg(), dense_cfg()), (diff_cfg(2, 1, 8, 12, rot=(50.0, 8), size=None), None),
                               (keyval_cfg(4, 2, 10, factor=None, size=3), moe_cfg(ff=8, experts=5, top=5, shared=24)), (keyval_cfg(2, 2, 6, rot=(9.0, 6)), moe_cfg(shared=None))],
                       loop=(1, 3, 2))


def _layered(cfg):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer

    return LayeredTransformer(LayeredArgs.from_dict(cfg))


def test_config():
    from mistral_inference_b200.args import ChosenSoftmaxMoeArgs, DifferentialAttentionArgs, KeyValueAttentionArgs, LayeredArgs, SiluGluArgs

    a = LayeredArgs.from_dict(_cfg())
    assert a.norm == "rms" and a.post_norm and a.pre_norm and a.tied_head and not a.parallel_block and not a.loop_adds_embedding
    assert a.embedding_scale == 1.7 and a.logit_scale == 0.8 and a.layer_runs() == [0, 1, 2, 1, 2, 3, 4]
    L0, L1, L2, L3, L4 = a.layers
    assert isinstance(L0.mixer, KeyValueAttentionArgs) and L0.mixer.rot_halves and L0.mixer.rot_factor == 2.5 and L0.mixer.unit_norm and L0.mixer.values_are_keys
    assert L0.mixer.chunked and L0.mixer.window == 5 and L0.mixer.out_gate == "entry" and not L0.mixer.qkv_bias and not L0.mixer.out_bias and L0.mixer.maps == 1
    assert isinstance(L0.mlp, ChosenSoftmaxMoeArgs) and (L0.mlp.ff, L0.mlp.experts, L0.mlp.top, L0.mlp.shared_ff) == (12, 6, 2, 20)
    assert isinstance(L1.mixer, DifferentialAttentionArgs) and (L1.mixer.maps, L1.mixer.diff, L1.mixer.out_gate) == (2, 0.35, "head") and not L1.mixer.rot_halves
    assert L1.mixer.qkv_bias and L1.mixer.out_bias and not L1.mixer.unit_norm and not L1.mixer.values_are_keys and L1.mixer.rot_dims == 4
    assert isinstance(L1.mlp, SiluGluArgs) and L2.mlp is None and L2.mixer.window is None and L3.mixer.rot_factor == 1.0 and L4.mlp.shared_ff == 0
    d = _cfg()
    del d["logit_scale"], d["loop"]
    assert LayeredArgs.from_dict(d).logit_scale == 1.0 and LayeredArgs.from_dict(d).loop is None


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "mixer", "kv_heads"), 2), (("layers", 0, "mixer", "vdim"), 11), (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "rot", "dims"), 3),
    (("layers", 1, "mixer", "rot", "dims"), 8), (("layers", 0, "mlp", "router", "top"), 7), (("layers", 0, "mlp", "router", "top"), 0), (("loop", "stop"), 6), (("loop", "times"), 0)])
def test_rejected_config(path, value):
    from mistral_inference_b200.args import LayeredArgs

    bad = copy.deepcopy(_cfg())
    node = bad
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(AssertionError):
        LayeredArgs.from_dict(bad)


def test_registry_and_packing(tmp_path):
    from mistral_inference_b200.registry import ARCHITECTURES, architecture_of

    cfg = _cfg()
    w = make_weights(cfg, 1)
    assert architecture_of(write_folder(tmp_path / "m", cfg, w)) == "Pukarax" and "Pukarax" in ARCHITECTURES
    m = _layered(cfg)
    keys = list(w)
    assert sorted(m.checkpoint_keys()) == sorted(keys)
    for p in m.parameters():
        p.data.fill_(7.0)
    random.Random(1).shuffle(keys)
    m.load_state_dict({k: w[k] for k in keys})
    kv, df = m.layers[0].mix, m.layers[1].mix
    assert torch.equal(kv.wqkv, torch.cat([w["l0.mix." + n] for n in ("q", "k", "g")])) and kv.bqkv is None and kv.nv == 0 and kv.lambdas is None
    assert torch.equal(df.wqkv, torch.cat([w["l1.mix." + n] for n in ("q", "k", "v", "g")])) and torch.equal(df.bo, w["l1.mix.o.b"])
    assert torch.equal(df.bqkv, torch.cat([w[f"l1.mix.{n}.b"] for n in "qkv"] + [torch.zeros(4)])), "the gate has no bias, whatever the memory held"
    assert torch.equal(df.lambdas, torch.stack([w["l1.mix." + n] for n in ("lq1", "lk1", "lq2", "lk2")]))
    assert abs(float(df.difference_weight()) - float(O.lam_of({k: v.double() for k, v in w.items()}, "l1.mix.", 0.35))) < 1e-6
    # a shared expert of another size beside the experts; one of three times their size among them; none
    m0, m3, m4 = m.layers[0].mlp, m.layers[3].mlp, m.layers[4].mlp
    assert m0.always == 0 and torch.equal(m0.shared.w2, w["l0.mlp.shared.down"]) and torch.equal(m0.router_bias, w["l0.mlp.router.b"])
    assert m3.always == 3 and m3.shared is None and torch.equal(m3.w2[:, 40:], w["l3.mlp.shared.down"]) and torch.equal(m3.w2[:, 16:24], w["l3.mlp.e2.down"])
    assert torch.equal(m3.w13.view(-1, 2, 40)[40:, 0], w["l3.mlp.shared.gate"]) and torch.equal(m3.w13.view(-1, 2, 40)[8:16, 1], w["l3.mlp.e1.up"])
    assert m4.always == 0 and m4.shared is None and m.layers[2].norm2 is None and m.layers[2].norm1b is not None and m.head is None
    for k in ("l3.norm2b", "l1.mix.lk2", "l0.mix.g", "l1.mix.o.b", "l3.mlp.shared.up", "l0.mlp.router.b"):
        with pytest.raises(AssertionError):
            _layered(cfg).load_state_dict({n: t for n, t in w.items() if n != k})
    for k in ("l0.mix.v", "l0.mix.q.b", "l0.mix.lq1", "l2.norm2", "l4.mlp.shared.up", "head", "l0.mix.o.b", "l0.mlp.e6.up"):
        with pytest.raises(ValueError):
            m.load_state_dict({k: w["l0.norm1"]}, strict=False)


def test_large_input_projection_is_padded_with_zeros():
    from mistral_inference_b200.args import DifferentialAttentionArgs
    from mistral_inference_b200.transformer_layers import RotaryWindowAttention

    at = RotaryWindowAttention(16, DifferentialAttentionArgs.from_dict(diff_cfg(8, 4, 48, 40, rot=(50.0, 48))["mixer"]), 1e-5)
    used = 2 * 8 * 48 + 2 * 4 * 48 + 4 * 40 + 8
    assert at.g_off + at.ng == used and at.wqkv.shape[0] == 1408 == at.bqkv.shape[0]
    at.wqkv.data.fill_(7.0)
    at.bqkv.data.fill_(7.0)
    at.assign("g", lambda dst: dst.zero_())
    at.assign("q.b", lambda dst: dst.zero_())
    assert float(at.wqkv[used:].abs().sum()) == 0.0 and float(at.bqkv[used - 8:].abs().sum()) == 0.0


def test_cache_layout():
    """An entry per layer run; chunks need a ring of one chunk; two maps are twice the key size."""
    m = _layered(_cfg())
    c = m.make_cache(3, 64)
    assert [tuple(c.cache_k[r].shape) for r in range(7)] == [(3, 5, 1, 12), (3, 7, 2, 12), (3, 64, 1, 16), (3, 7, 2, 12), (3, 64, 1, 16), (3, 3, 2, 10), (3, 5, 2, 6)]
    assert tuple(c.cache_v[1].shape) == (3, 7, 2, 10) and tuple(c.cache_v[5].shape) == (3, 3, 2, 10) and not c.cache_state
    assert c.cache_k[1].data_ptr() != c.cache_k[3].data_ptr(), "every pass of a looped layer has its own ring"
    assert tuple(m.make_cache(1, 4).cache_k[1].shape) == (1, 4, 2, 12)


def test_norms_are_handed_on_only_where_nothing_comes_between():
    """Blocks hand on the norm of the stream; designs that touch the stream between layers or have other norms do not."""
    m = _layered(_cfg())
    assert m._chained and all(b.chains() for b in m.layers)
    m.args.loop_adds_embedding = True
    assert not type(m)(m.args)._chained


def test_plain_statement():
    """Facts of the mechanisms that do not need a second implementation."""
    g = torch.Generator().manual_seed(0)
    x = torch.randn(9, 2, 8, generator=g, dtype=torch.float64)
    rot = {"base": 100.0, "dims": 6, "scaling": {"factor": 3.0}}
    for fn in (O.rotate_halves, O.rotate_neighbours):
        y = fn(x, rot)
        assert torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0]) and torch.allclose(y.norm(dim=-1), x.norm(dim=-1))
    slow, plain = O.rotate_halves(x, rot), O.rotate_halves(torch.stack([x[0], x[3]]), {"base": 100.0, "dims": 6})
    assert torch.allclose(slow[3], plain[1]), "position 3 at a third of the speed is position 1"
    q, k, v = (torch.randn(20, n, generator=g, dtype=torch.float64) for n in (4, 4, 3))
    out = O.softmax_map(q, k, v, 0.5, 6)
    assert torch.equal(out[6], v[6]) and torch.equal(out[12], v[12]), "the first token of a chunk sees itself alone"
    assert torch.allclose(out[6:12], O.softmax_map(q[6:12], k[6:12], v[6:12], 0.5, None)), "chunks do not see one another"
    d = O.difference(out, out * 0.5, 0.4, 0.25, 0.0)
    assert torch.allclose(d.pow(2).mean(-1), torch.full((20,), 0.75 ** 2, dtype=torch.float64))
    w = {"router": torch.eye(4, dtype=torch.float64), "router.b": torch.tensor([0.0, 3.0, 0.0, -9.0], dtype=torch.float64)}
    got = O.route(torch.tensor([2.0, 0.0, 1.0, 5.0], dtype=torch.float64), w, "", {"top": 2})
    assert [e for e, _ in got] == [1, 0] and abs(got[0][1] - 1 / (1 + 2.718281828 ** -1)) < 1e-6
