"""Host-side tests of the Sizudra decoder's configuration, specification, weight map and cache needs, of the cache manager's
kept first keys, and of the plain implementation against itself (causality, windows, kept keys, blended values)."""
import os
import random

import pytest
import torch

import helpers
from plain import sizudra_plain as plain
from return_b200.cache.manager import CacheManager, GroupSpec
from return_b200.cache.storage import CacheStorage
from return_b200.config import registry
from return_b200.config.model_config import ConfigError
from return_b200.config.sizudra_config import SizudraConfig
from return_b200.models import sizudra
from return_b200.models.decoder import DecoderModel
from return_b200.parts.base import BLOCKS, FEED_FORWARDS, MIXERS, BuildEnv, KVCacheNeed, StateNeed
from return_b200.parts.spec import (AttentionSpec, DenseMLPSpec, MoESpec, NormSpec, PostNormBlockSpec, SwiGLUSpec, TanhNormSpec)
from return_b200.weights import loader

CPU = BuildEnv(torch.float32, torch.device("cpu"))


def raw_config():
    att = {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.4, "rot": {"base": 500.0, "dims": 8}, "v_mix": True}
    windowed = {**att, "heads": 6, "dim": 24, "mask": {"size": 9, "keep_first": 5}, "softcap": 4.0}
    moe = {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 24}, "shared": {"ff": 10}}
    return {"architecture": "Sizudra", "vocab": 83, "width": 40, "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": 37, "mul_prev": 11, "mul_cur": 3}}, "layers": [
                {"type": "attention", "mixer": {**att, "v_mix": False}, "mlp": moe},
                {"type": "attention_2", "mixer": windowed, "mlp": {"kind": "dense", "ff": 56}},
                {"type": "attention", "mixer": att, "mlp": None},
                {"type": "attention_2", "mixer": {**windowed, "mask": {"size": 9}, "v_mix": False}, "mlp": {"kind": "dense", "ff": 33}},
                {"type": "attention", "mixer": {**att, "rot": {"base": 500.0, "dims": 0}}, "mlp": {**moe, "shared": None}}]}


def test_registry_finds_the_architecture_by_its_name():
    arch = registry.resolve({"architecture": "Sizudra"})
    assert arch.config_cls is SizudraConfig and "Sizudra" in registry.architectures()


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "attention_3"), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "vdim"), 0),
    (("layers", 0, "mixer", "scale"), 0.0), (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "rot", "dims"), 14),
    (("layers", 1, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "mask", "keep_first"), -1), (("layers", 1, "mixer", "mask"), {}),
    (("layers", 1, "mixer", "softcap"), -1.0), (("layers", 2, "mixer", "vdim"), 16), (("layers", 4, "mixer", "kv_heads"), 1),
    (("layers", 0, "mlp", "router", "top"), 6), (("layers", 0, "mlp", "expert", "ff"), 0), (("layers", 0, "mlp", "shared"), {"ff": 0}),
    (("layers", 1, "mlp", "kind"), "gated"), (("layers", 1, "mlp", "ff"), 0), (("embedding", "bigram", "buckets"), 0),
    (("embedding", "bigram"), {"buckets": 3}), (("norm", "eps"), 0.0), (("width",), 0), (("layers",), [])])
def test_configuration_rejects_what_the_design_does_not_have(path, value):
    raw = raw_config()
    d = raw
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError):
        SizudraConfig(raw)


def test_keys_that_must_be_there_and_keys_that_may_be_absent():
    for key in ("heads", "kv_heads", "dim", "vdim", "scale"):
        raw = raw_config()
        del raw["layers"][1]["mixer"][key]
        with pytest.raises(ConfigError):
            SizudraConfig(raw)
    raw = raw_config()
    for key in ("rot", "mask", "softcap", "v_mix"):
        del raw["layers"][1]["mixer"][key]
    del raw["embedding"]
    spec = sizudra.decoder_spec(SizudraConfig(raw))
    m = spec.layers[1].mixer
    assert (m.position, m.window, m.keep_first, m.softcap, m.value_mix) == (None, None, 0, None, None) and m.sink
    assert spec.embedding_pairs is None


def test_specification_follows_the_configuration():
    spec = sizudra.decoder_spec(SizudraConfig(raw_config()), 128)
    assert [e.cache_of for e in spec.schedule] == [None] * 5 and not spec.tie_embeddings and spec.embedding_pairs == (37, 11, 3)
    mixers = [b.mixer for b in spec.layers]
    assert [m.value_mix for m in mixers] == [None, "source", "blend", None, "blend"]
    assert [m.sink for m in mixers] == [False, True, False, True, False]
    assert [(m.window, m.keep_first, m.softcap) for m in mixers] == [(None, 0, None), (9, 5, 4.0), (None, 0, None), (9, 0, 4.0), (None, 0, None)]
    assert [m.head_dim for m in mixers] == [32] * 5 and mixers[1].qk_norm == NormSpec(24, 1e-5) and mixers[0].qk_norm == NormSpec(12, 1e-5)
    assert mixers[0].position.rotary_dim == 8 and mixers[0].position.theta == 500.0 and mixers[4].position is None
    ff = spec.layers[0].feed_forward
    assert (ff.top, ff.renorm_tiny, ff.score, ff.shared_gate, ff.expert) == (2, 0.0, "softmax", True, DenseMLPSpec(40, 24, "relu2"))
    assert ff.shared == DenseMLPSpec(40, 10, "relu2") and spec.layers[4].feed_forward.shared is None
    assert not spec.layers[4].feed_forward.shared_gate and spec.layers[2].feed_forward is None
    assert spec.layers[1].feed_forward == SwiGLUSpec(40, 56, 8, activation="gelu_tanh") and spec.layers[3].feed_forward.interleave == 0
    lone = raw_config()
    for i in (2, 4):
        lone["layers"][i]["mixer"]["v_mix"] = False
    assert sizudra.decoder_spec(SizudraConfig(lone)).layers[1].mixer.value_mix is None      # nobody blends its values in


def test_parameters_checkpoint_names_and_caches_fit_together(tmp_path):
    cfg = SizudraConfig(raw_config())
    arch = registry.resolve(cfg.to_dict())
    model = DecoderModel(arch.decoder_spec(cfg, 64), CPU)
    params, sources, shapes = model.params(), arch.weight_sources(cfg), loader.checkpoint_shapes(arch, cfg)
    assert set(params) == set(sources)
    assert {n for s in sources.values() for n in s.names} == set(shapes)
    assert shapes["l2.mix.vmix"][0] == () and "l1.mix.vmix" not in shapes and "l0.mix.vmix" not in shapes
    assert "l0.mix.sink" not in shapes and shapes["l1.mix.sink"][0] == (6,) and "l2.norm2" not in shapes
    assert arch.ignorable_tensors(cfg) == {"l0.mix.vmix", "l1.mix.vmix", "l3.mix.vmix", "l2.norm2"}
    d = loader.write_random_model(str(tmp_path / "m"), cfg, 1, torch.bfloat16)
    expected = {n: s for n, (s, _) in shapes.items()}
    loaded = loader.load_parameters(params, sources, expected, d, torch.float32, "cpu", arch.ignorable_tensors(cfg))
    assert {n: tuple(t.shape) for n, t in loaded.items()} == {n: tuple(p.shape) for n, p in params.items()}
    w = plain.read_safetensors(os.path.join(d, "model.safetensors"))
    qkv = loaded["layers.1.mixer.qkv"].view(10, 32, 40)                     # 6 + 2 + 2 heads, padded to the cache's 32
    assert torch.equal(qkv[:6, :24].reshape(144, 40), w["l1.mix.q"].float()) and torch.equal(qkv[8:, :20].reshape(40, 40), w["l1.mix.v"].float())
    assert float(qkv[:8, 24:].abs().max()) == 0.0 and float(qkv[8:, 20:].abs().max()) == 0.0
    assert torch.equal(loaded["layers.1.mixer.k_norm.weight"][:24], w["l1.mix.k.norm"].float())
    o = loaded["layers.0.mixer.o"].view(40, 4, 32)
    assert torch.equal(o[:, :, :20].reshape(40, 80), w["l0.mix.o"].float()) and float(o[:, :, 20:].abs().max()) == 0.0
    router = loaded["layers.0.feed_forward.router"]
    assert torch.equal(router[:5], w["l0.mlp.router"].float()) and torch.equal(router[5:], w["l0.mlp.shared.sg"].float())
    model.bind(loaded)
    assert model.blocks[0].feed_forward.up.shape == (5, 24, 40) and float(model.blocks[2].mixer.value_share) == float(w["l2.mix.vmix"])
    assert model.cache_needs() == [KVCacheNeed(2, 32), KVCacheNeed(2, 32, 9, 5), KVCacheNeed(2, 32), KVCacheNeed(2, 32, 9, 0),
                                   KVCacheNeed(2, 32), StateNeed((1,), torch.int32)]
    storage = CacheStorage(model.cache_needs(), 4, 64, 3, CPU, longest_append=8)
    assert [(g.window, g.keep_first) for g in storage.group_specs] == [(None, 0), (9, 5), (9, 0)]
    assert storage.group_specs[1].num_pages == storage.group_specs[2].num_pages + 3 * 2       # two pages of kept keys a request
    assert not storage.make_manager().truncatable                                             # a request's last token is state


def test_a_file_may_hold_the_share_that_nothing_reads(tmp_path):
    from return_b200.weights.safetensors_io import write_safetensors
    cfg = SizudraConfig(raw_config())
    arch = registry.resolve(cfg.to_dict())
    model = DecoderModel(arch.decoder_spec(cfg, 64), CPU)
    d = loader.write_random_model(str(tmp_path / "m"), cfg, 1, torch.bfloat16)
    path = os.path.join(d, "model.safetensors")
    tensors = plain.read_safetensors(path)
    expected = {n: s for n, (s, _) in loader.checkpoint_shapes(arch, cfg).items()}

    def load(extra):
        write_safetensors(path, list({**tensors, **extra}.items()))
        return loader.load_parameters(model.params(), arch.weight_sources(cfg), expected, d, torch.float32, "cpu", arch.ignorable_tensors(cfg))
    load({"l1.mix.vmix": torch.tensor(0.5).bfloat16()})
    with pytest.raises(loader.WeightError, match="l0.mix.sink"):
        load({"l0.mix.sink": torch.zeros(4).bfloat16()})


def test_parts_reject_options_that_do_not_fit():
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=16, scale=0.25)
    for bad in (dict(keep_first=3), dict(window=4, keep_first=-1), dict(softcap=0.0), dict(value_mix="first"),
                dict(qk_norm=NormSpec(12, 1e-6))):
        with pytest.raises(ValueError):
            MIXERS.build(AttentionSpec(**base, **bad), CPU)
    unit = DenseMLPSpec(16, 8, "relu2")
    moe = dict(hidden_size=16, num_experts=4, top=2)
    for bad in (dict(expert=unit, weigh_input=True), dict(expert=unit, shared_gate=True),
                dict(expert=SwiGLUSpec(16, 8, activation="gelu_tanh"))):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(MoESpec(**moe, **bad), CPU)
    with pytest.raises(ValueError):
        FEED_FORWARDS.build(SwiGLUSpec(16, 8, activation="relu2"), CPU)
    with pytest.raises(ValueError):
        BLOCKS.build(PostNormBlockSpec(AttentionSpec(**base), None, TanhNormSpec(16)), CPU)


# ------------------------------------------------------------------------------- pages of a window that keeps first keys

@pytest.mark.parametrize("page,window,keep", [(4, 7, 1), (4, 7, 4), (4, 7, 6), (8, 5, 20), (4, 30, 3), (2, 1, 5), (16, 40, 16)])
def test_no_block_goes_back_that_a_query_still_needs(page, window, keep):
    m = CacheManager([GroupSpec("win", page, 400, window=window, keep_first=keep)], max_requests=1)
    m.add("r")
    rng, length = random.Random(page + window + keep), 0
    kept_pages = None
    while length < 260:
        n = rng.choice([1, 1, 2, 3, 5, 13])
        assert m.append("r", n) == length
        bt = m.block_table("r", 0)
        for q in range(length, length + n):
            for k in [*range(min(keep, q + 1)), *range(max(0, q - window + 1), q + 1)]:
                assert bt[k // page] >= 0, (q, k)
        length += n
        if length >= keep:
            kept_pages = kept_pages or list(bt[:(keep + page - 1) // page])
            assert bt[:len(kept_pages)] == kept_pages                        # the same pages as long as the request lives
        assert m.pages_used()[0] <= (window + 13) // page + 3 + (keep + page - 1) // page
        m.check()
    assert m.pages_used()[0] < 260 // page or keep > 100
    m.free("r")
    assert m.pages_used() == [0]
    m.check()


def test_pages_needed_agrees_with_what_append_takes():
    m = CacheManager([GroupSpec("full", 4, 64), GroupSpec("win", 4, 64, window=6, keep_first=5)], max_requests=2)
    m.add("r")
    rng = random.Random(3)
    for _ in range(40):
        n = rng.choice([1, 2, 3, 7])
        if not m.fits("r", n):
            break
        need, used = m.pages_needed("r", n), m.pages_used()
        m.append("r", n)
        assert [u + x for u, x in zip(used, need)] == m.pages_used()
    bt = m.block_table("r", 1)
    assert bt[0] >= 0 and bt[1] >= 0 and bt[2] == -1                        # keys 0..4 lie in the first two blocks


def test_a_group_without_a_window_keeps_everything_anyway():
    g = GroupSpec("full", 4, 8, None, 3)
    assert g.kept_blocks == 0
    m = CacheManager([g], 1)
    m.add("r")
    m.append("r", 20)
    m.append("r", 5)
    assert all(p >= 0 for p in m.block_table("r", 0))


# ------------------------------------------------------------------------------- the plain implementation against itself

def _random_plain(tmp_path, raw=None, seed=2):
    d = loader.write_random_model(str(tmp_path / "m"), SizudraConfig(raw or raw_config()), seed, torch.bfloat16)
    return plain.read_model(d)


def test_plain_is_causal_and_starts_over_for_every_sequence(tmp_path):
    c, w = _random_plain(tmp_path)
    ids = helpers.random_ids(c["vocab"], 40, 5)
    full = plain.forward(c, w, ids)
    for n in (1, 2, 17, 39):
        assert torch.allclose(plain.forward(c, w, ids[:n]), full[:n], atol=1e-10)
    other = list(ids)
    other[20] = (other[20] + 1) % c["vocab"]
    assert (plain.forward(c, w, other)[20:] - full[20:]).abs().amax(1).min() > 1e-3


def test_plain_pieces():
    assert plain.pair_rows([4, 6, 1], 10, 3, 2) == [10, (4 * 3 + 6 * 2) % 10, (6 * 3 + 1 * 2) % 10]
    ok = plain.visible(12, {"size": 3, "keep_first": 2})
    assert ok[9].nonzero().flatten().tolist() == [0, 1, 7, 8, 9] and ok[1].nonzero().flatten().tolist() == [0, 1]
    assert plain.visible(5, None).sum() == 15
    x = torch.randn(7, 2, 10, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    y = plain.rotate_halves(x, 100.0, 6)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    assert torch.allclose(y.pow(2).sum(-1), x.pow(2).sum(-1))                            # turning keeps lengths
    s = torch.zeros(1, 2, 2, dtype=torch.float64)
    p = plain.softmax_with_sink(s, plain.visible(2, None), torch.zeros(1, dtype=torch.float64))
    assert torch.allclose(p[0], torch.tensor([[1 / 2, 0.0], [1 / 3, 1 / 3]], dtype=torch.float64))
    z = torch.linspace(-4, 4, 33, dtype=torch.float64)
    gate = z * torch.sigmoid(2 * (2 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3))          # the form the kernels use
    assert torch.allclose(plain.gelu_tanh(z), gate)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
