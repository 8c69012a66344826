"""Host-side logic of the Dimorax design: configuration, registry, checkpoint packing, cache layout."""
import copy
import random

import pytest
import torch

from tests.dimorax_util import attn_cfg, delta_cfg, dense_cfg, latent_cfg, make_config, make_weights, moe_cfg, on_disk


def _cfg():
    return make_config(layers=[(delta_cfg(), moe_cfg()), (attn_cfg(), dense_cfg()), (latent_cfg(), None), (attn_cfg(6, 2, 12, 10, 0.3, softcap=0, kv_from=1), moe_cfg(shared=None)),
                               (latent_cfg(window=None), dense_cfg(9)), (attn_cfg(2, 1, 16, 24, scaling=None), moe_cfg(groups=1, keep=1))])


def _layered(cfg):
    from mistral_inference_b200.args import LayeredArgs
    from mistral_inference_b200.layered import LayeredTransformer

    return LayeredTransformer(LayeredArgs.from_dict(on_disk(cfg)))


def test_config():
    from mistral_inference_b200.args import CappedAttentionArgs, DeltaArgs, GeluGluArgs, GroupedMoeArgs, LayeredArgs, SinkLatentAttentionArgs

    a = LayeredArgs.from_dict(on_disk(_cfg()))
    assert a.norm == "rms_around_one" and a.parallel_block and a.parallel_norms == 2 and a.residual_mult == 0.6 and not a.tied_head
    L0, L1, L2, L3, L4, L5 = a.layers
    assert isinstance(L0.mixer, DeltaArgs) and (L0.mixer.heads, L0.mixer.kv_heads, L0.mixer.conv) == (4, 2, 3)
    assert isinstance(L0.mlp, GroupedMoeArgs) and (L0.mlp.groups, L0.mlp.keep, L0.mlp.router_scale, L0.mlp.shared_ff) == (3, 2, 1.7, 20)
    assert isinstance(L1.mixer, CappedAttentionArgs) and L1.mixer.rot_scaling.factor == 3.0 and L1.mixer.rot_factor == 1.0 and L1.mixer.softcap == 7.0
    assert L1.mixer.rot_halves and L1.mixer.qkv_bias and L1.mixer.sink and not L1.mixer.unit_norm and isinstance(L1.mlp, GeluGluArgs)
    assert isinstance(L2.mixer, SinkLatentAttentionArgs) and L2.mixer.window == 5 and L2.mixer.q_rank == 0 and not L2.mixer.head_gate and L2.mlp is None
    assert L3.mixer.kv_from == 1 and L3.mixer.softcap == 0.0 and L3.mlp.shared_ff == 0 and L4.mixer.window is None and L5.mixer.rot_scaling is None


@pytest.mark.parametrize("path,value", [
    (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "kv_from"), 0), (("layers", 3, "mixer", "vdim"), 9), (("layers", 3, "mixer", "kv_heads"), 3),
    (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "conv"), 0), (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "rot", "dims"), 14),
    (("layers", 2, "mixer", "mask", "size"), 0), (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 0, "mlp", "router", "groups", "keep"), 4),
    (("layers", 0, "mlp", "router", "top"), 5)])
def test_rejected_config(path, value):
    from mistral_inference_b200.args import LayeredArgs

    bad = copy.deepcopy(on_disk(_cfg()))
    node = bad
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(AssertionError):
        LayeredArgs.from_dict(bad)


def test_registry_and_packing(tmp_path):
    from mistral_inference_b200.registry import ARCHITECTURES, architecture_of
    from tests.dimorax_util import write_folder

    cfg = _cfg()
    w = make_weights(cfg, 1)
    assert architecture_of(write_folder(tmp_path / "m", cfg, w)) == "Dimorax" and "Dimorax" in ARCHITECTURES
    keys = list(w)
    for seed in range(3):  # the ranks of the low-rank projections come with the tensors, in whatever order those arrive
        m = _layered(cfg)
        assert sorted(m.checkpoint_keys()) == sorted(keys)
        random.Random(seed).shuffle(keys)
        m.load_state_dict({k: w[k] for k in keys})
        d = m.layers[0].mix
        assert (d.ra, d.rg) == (5, 7) and d.wa2.shape == (48, 5) and d.wg2.shape == (40, 7)
        want = torch.cat([w["l0.mix." + n] for n in ("q", "k", "v", "b", "a1", "g1")])
        assert torch.equal(d.w_in[: len(want)], want) and torch.equal(d.conv, torch.cat([w[f"l0.mix.{n}.conv"] for n in "qkv"]))
    at, sh, la = m.layers[1].mix, m.layers[3].mix, m.layers[2].mix
    assert torch.equal(at.wqkv[48:72], w["l1.mix.k"]) and torch.equal(at.bqkv[72:], w["l1.mix.v.b"]) and torch.equal(at.sink, w["l1.mix.sink"])
    assert sh.wqkv.shape[0] == 72 and torch.equal(sh.bqkv, w["l3.mix.q.b"])
    assert torch.equal(la.w_in[:48], w["l2.mix.q"]) and torch.equal(la.w_in[48:68], w["l2.mix.dkv"]) and la.w_uq is None
    mo = m.layers[0].mlp
    assert torch.equal(mo.w13.view(6, 12, 2, 40)[3, :, 1], w["l0.mlp.e3.up"]) and torch.equal(mo.w2.view(40, 6, 12)[:, 4], w["l0.mlp.e4.down"])
    assert torch.equal(mo.shared_gate, w["l0.mlp.shared.sg"]) and m.layers[3].mlp.shared is None
    assert m.layers[2].norm2 is None and m.layers[1].norm2 is not None and m.layers[0].residual_mult == 0.6
    for k in ("l3.norm2", "l1.mix.sink", "l0.mix.k.conv"):
        with pytest.raises(AssertionError):
            _layered(cfg).load_state_dict({n: t for n, t in w.items() if n != k})
    for k in ("l3.mix.k", "l2.norm2", "l3.mlp.shared.sg"):  # no keys of its own, no feed-forward, no shared expert
        with pytest.raises(ValueError):
            m.load_state_dict({k: w["l0.norm1"]}, strict=False)


def test_input_projection_padding():
    """A large packed projection is padded to the prompt GEMM's tile; the padding is zero whatever the memory held."""
    from mistral_inference_b200.args import DeltaArgs, SinkLatentAttentionArgs
    from mistral_inference_b200.transformer_layers import DeltaMixer, LatentAttention, padded_rows

    assert [padded_rows(n) for n in (1, 1000, 1024, 1025)] == [1, 1000, 1024, 1152]
    d = DeltaMixer(16, DeltaArgs(heads=8, kv_heads=4, dim=64, vdim=64, conv=4), 1e-5)
    d.resize(20, 12)
    assert d.w_in.shape == (1152, 16) and float(d.w_in[2 * 256 + 512 + 8 + 32:].abs().sum()) == 0.0
    la = LatentAttention(16, SinkLatentAttentionArgs.from_dict(latent_cfg(8, 96, 32, 64, 40)["mixer"]), 1e-5)
    la.w_in.data.fill_(7.0)
    la.assign("q", lambda dst: dst.zero_())
    assert la.n_used == 1024 + 72 and la.w_in.shape[0] == 1152 and float(la.w_in[la.n_used:].abs().sum()) == 0.0


def test_cache_layout():
    m = _layered(_cfg())
    c = m.make_cache(3, 64)
    assert [sp.kind for sp in c.layer_specs] == ["state", "ring", "ring", "shared", "ring", "ring"]
    assert c.cache_state[0].shape == (3, 4, 10, 12) and c.cache_conv[0].shape == (3, 3, 48 + 40) and c.cache_conv[0].dtype == torch.float32
    assert c.cache_k[1].shape == (3, 64, 2, 12) and c.cache_k[2].shape == (3, 5, 1, 20) and c.cache_k[4].shape == (3, 64, 1, 20)
    assert 3 not in c.cache_k and 3 not in c.cache_state
    c.init_kvseqlens(2)
    md = c.get_input_metadata([7, 2])
    v1, v3 = c.get_view(1, md[1]), c.get_view(3, md[3])
    assert v3.cache_k is v1.cache_k and v3.cache_v is v1.cache_v and md[3].window == 64 and md[2].window == 5
    one = _layered(make_config(layers=[(delta_cfg(conv=1), None)]))
    assert one.make_cache(2, 8).cache_conv[0].shape == (2, 1, 88)


def test_shared_cache_entry_needs_a_whole_ring():
    from mistral_inference_b200.cache import BufferCache, LayerCacheSpec

    ring = LayerCacheSpec(kind="ring", n_kv_heads=1, k_dim=4, v_dim=4)
    for first, source in ((LayerCacheSpec(kind="ring", n_kv_heads=1, k_dim=4, v_dim=4, window=3), 0), (LayerCacheSpec(kind="state", state_shape=(1, 2, 2)), 0), (ring, 1)):
        with pytest.raises(AssertionError):
            BufferCache(2, 1, 8, 0, 0, None, layer_specs=[first, LayerCacheSpec(kind="shared", source=source)])
