"""Host-side tests of the Losorax decoder's configuration, specification, weight map and cache needs, and of the plain
implementation against itself (causality, the distance buckets, the temperature, the router, shared keys)."""
import copy
import math
import os

import pytest
import torch

import helpers
from plain import losorax_plain as plain
from return_b200.cache.storage import CacheStorage
from return_b200.config import registry
from return_b200.config.losorax_config import LosoraxConfig
from return_b200.config.model_config import ConfigError
from return_b200.models import losorax
from return_b200.models.decoder import DecoderModel
from return_b200.parts.attention import distance_rows
from return_b200.parts.base import BuildEnv, KVCacheNeed, StateNeed
from return_b200.parts.spec import GatedAttentionSpec, MixerSumSpec, NormSpec, SandwichBlockSpec, TanhNormSpec
from return_b200.weights import loader

CPU = BuildEnv(torch.float32, torch.device("cpu"))


def raw_config():
    att = {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.4, "conv": 3, "bias_rows": 10, "bias_max": 33,
           "q_temp": {"coef": 0.4, "every": 16}}
    moe = {"kind": "moe", "router": {"experts": 6, "top": 2}, "expert": {"ff": 24}}
    return {"architecture": "Losorax", "vocab": 97, "width": 40, "norm": {"eps": 1e-5}, "layers": [
        {"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": 56}},
        {"type": "general_delta", "mixer": {"heads": 3, "dim": 10, "decay_rank": 6}, "mlp": moe},
        {"type": "attention", "mixer": {**att, "heads": 2, "conv": 4, "kv_from": 0, "bias_rows": 8}, "mlp": None},
        {"type": "general_delta", "mixer": {"heads": 2, "dim": 16, "decay_rank": 5}, "mlp": {"kind": "dense", "ff": 33}}]}


def test_registry_finds_the_architecture_by_its_name():
    arch = registry.resolve({"architecture": "Losorax"})
    assert arch.config_cls is LosoraxConfig and "Losorax" in registry.architectures()


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "retention"), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "vdim"), 0),
    (("layers", 0, "mixer", "conv"), 40), (("layers", 0, "mixer", "bias_max"), 5), (("layers", 0, "mixer", "bias_rows"), 1),
    (("layers", 0, "mixer", "q_temp", "every"), 0), (("layers", 0, "mixer", "q_temp", "every"), 2.5),
    (("layers", 0, "mixer", "q_temp"), {"coef": 1.0}), (("layers", 2, "mixer", "kv_from"), 1), (("layers", 2, "mixer", "kv_from"), 2),
    (("layers", 2, "mixer", "dim"), 16), (("layers", 1, "mixer", "decay_rank"), 0), (("layers", 1, "mlp", "router", "top"), 7),
    (("layers", 0, "mlp", "kind"), "gated"), (("layers", 0, "mlp", "ff"), 0), (("norm", "eps"), 0.0), (("width",), 0), (("layers",), [])])
def test_configuration_rejects_what_the_design_does_not_have(path, value):
    raw = raw_config()
    d = raw
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError):
        LosoraxConfig(raw)


def test_keys_that_must_be_there_and_keys_that_may_be_absent():
    for i, key in ((0, "bias_max"), (0, "scale"), (1, "heads")):
        raw = raw_config()
        del raw["layers"][i]["mixer"][key]
        with pytest.raises(ConfigError):
            LosoraxConfig(raw)
    raw = raw_config()
    for key in ("conv", "q_temp"):
        del raw["layers"][0]["mixer"][key]
    m = losorax.decoder_spec(LosoraxConfig(raw)).layers[0].mixer
    assert m.conv_taps is None and m.temperature is None
    del raw["layers"][0]["mixer"]["bias_rows"]                    # a size that is only the shape of a tensor
    with pytest.raises(ConfigError, match="bias_rows"):
        losorax.decoder_spec(LosoraxConfig(raw))


def test_specification_follows_the_configuration():
    spec = losorax.decoder_spec(LosoraxConfig(raw_config()), 128)
    assert [e.cache_of for e in spec.schedule] == [None, None, 0, None] and not spec.tie_embeddings
    first, reader = spec.layers[0].mixer, spec.layers[2].mixer
    assert (first.conv_taps, first.head_norm_eps, first.temperature, first.distance_bias, first.fixed_sink) == (3, 1e-5, (0.4, 16), (10, 33.0), 0.0)
    assert first.own_cache and not reader.own_cache and reader.num_heads == 2 and reader.distance_bias == (8, 33.0) and first.window is None
    delta = spec.layers[1].mixer
    assert (delta.num_heads, delta.key_dim, delta.decay_rank, delta.unit_eps) == (3, 10, 6, 1e-6)
    assert delta.decay_scale == math.exp(-0.5)
    ff = spec.layers[1].feed_forward
    assert (ff.score, ff.renormalize, ff.weigh_input, ff.top, ff.groups) == ("sigmoid", False, True, 2, 1)
    assert spec.layers[0].feed_forward.interleave == 8 and spec.layers[3].feed_forward.interleave == 0
    assert spec.layers[2].feed_forward is None and all(b.layer_scale and b.token_shift for b in spec.layers)
    assert spec.final_norm == TanhNormSpec(40)


def test_parameters_checkpoint_names_and_what_runs_keep_fit_together(tmp_path):
    cfg = LosoraxConfig(raw_config())
    arch = registry.resolve(cfg.to_dict())
    model = DecoderModel(arch.decoder_spec(cfg, 64), CPU)
    params, sources, shapes = model.params(), arch.weight_sources(cfg), loader.checkpoint_shapes(arch, cfg)
    assert set(params) == set(sources)
    assert {n for s in sources.values() for n in s.names} == set(shapes)
    assert "l2.mix.k" not in shapes and "l2.mix.v.conv" not in shapes and "l2.norm2" not in shapes and "l2.ls2" not in shapes
    assert shapes["l0.norm1.alpha"][0] == () and shapes["l2.mix.rel"][0] == (8, 2) and shapes["l1.mix.w1"][0] == (6, 40)
    d = loader.write_random_model(str(tmp_path / "m"), cfg, 1, torch.bfloat16)
    loaded = loader.load_parameters(params, sources, {n: s for n, (s, _) in shapes.items()}, d, torch.float32, "cpu",
                                    arch.ignorable_tensors(cfg))
    assert {n: tuple(t.shape) for n, t in loaded.items()} == {n: tuple(p.shape) for n, p in params.items()}
    w = plain.read_safetensors(os.path.join(d, "model.safetensors"))
    o = loaded["layers.0.mixer.o"].view(40, 4, 32)                           # heads of 20 values padded to the cache's 32
    assert torch.equal(o[:, :, :20].reshape(40, 80), w["l0.mix.o"].float()) and float(o[:, :, 20:].abs().max()) == 0.0
    assert float(loaded["layers.3.mixer_post_norm.alpha"]) == float(w["l3.norm1b.alpha"])
    model.bind(loaded)
    post = model.blocks[0]._post["mixer"]                                    # the layer's scale lies in the norm behind the sublayer
    assert torch.equal(post[1], (w["l0.norm1b"].float() * w["l0.ls1"].float())) and float(post[0]) == float(w["l0.norm1b.alpha"])
    assert model.cache_needs() == [KVCacheNeed(2, 32, None), StateNeed((3 * 10 * 12,)), None, StateNeed((2 * 16 * 16,))]
    # the last inputs of the convolutions (q, k, v where the layer has them), then the last normed row; a layer that reads
    # another's keys keeps its own
    assert model.kept_needs() == [StateNeed(((48 + 24 + 40) * 2 + 40,)), StateNeed((40,)), StateNeed((24 * 3 + 40,)), StateNeed((40,))]


def test_sizes_that_only_shapes_give_are_read_from_the_folder(tmp_path):
    d = loader.write_random_model(str(tmp_path / "m"), LosoraxConfig(raw_config()), 1, torch.bfloat16)
    raw = raw_config()
    for layer in raw["layers"]:
        layer["mixer"].pop("bias_rows", None)
        layer["mixer"].pop("decay_rank", None)
    cfg = LosoraxConfig.from_model_dir(d, raw)
    assert cfg.to_dict() == LosoraxConfig(raw_config()).to_dict()
    raw["layers"].append(copy.deepcopy(raw["layers"][1]))
    with pytest.raises(ConfigError, match="l4.mix.w1"):
        LosoraxConfig.from_model_dir(d, raw)


def test_a_slot_taken_again_keeps_nothing_of_the_request_before():
    model = DecoderModel(losorax.decoder_spec(LosoraxConfig(raw_config()), 64), CPU)
    st = CacheStorage(model.cache_needs(), page_size=8, num_pages=16, max_reside=2, env=CPU, kept=model.kept_needs())
    manager = st.make_manager()
    st.allocate()
    assert len(st.group_specs) == 1 and not manager.truncatable
    assert st.kept(0).shape == (3, 264) and st.kept(2).shape == (3, 112) and st.kept(4) is None
    manager.add("a")
    slot = manager.slot("a")
    for t in st.states.values():
        t.fill_(5.0)
    manager.free("a")
    manager.add("b")
    assert manager.slot("b") == slot
    assert all(float(t[slot].abs().max()) == 0.0 and float(t[1 - slot].min()) == 5.0 for t in st.states.values())


def test_random_parameters_follow_the_same_map():
    cfg = LosoraxConfig(raw_config())
    arch = registry.resolve(cfg.to_dict())
    params = DecoderModel(arch.decoder_spec(cfg, 64), CPU).params()
    got = loader.random_parameters(params, arch.weight_sources(cfg), loader.checkpoint_shapes(arch, cfg), 3, torch.float32, "cpu")
    assert {n: tuple(t.shape) for n, t in got.items()} == {n: tuple(p.shape) for n, p in params.items()}
    assert 0.5 <= float(got["layers.0.mixer_norm.alpha"]) <= 1.0


def test_parts_refuse_what_they_cannot_do():
    from return_b200.parts.base import BLOCKS, MIXERS
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, key_dim=8, value_dim=8, scale=1.0)
    for extra in (dict(conv_taps=3, bias=True), dict(head_norm_eps=1e-5, values_are_keys=True), dict(conv_taps=34),
                  dict(temperature=(0.1, 0)), dict(distance_bias=(1, 8)), dict(distance_bias=(16, 8)), dict(sink=True, fixed_sink=0.0)):
        with pytest.raises(ValueError):
            MIXERS.build(GatedAttentionSpec(**base, **extra), CPU)
    plain_att = GatedAttentionSpec(**base)
    with pytest.raises(ValueError, match="keep"):
        MIXERS.build(MixerSumSpec(("a", "b"), (plain_att, GatedAttentionSpec(**base, conv_taps=3)), (1.0, 1.0)), CPU)
    with pytest.raises(ValueError, match="norms"):
        BLOCKS.build(SandwichBlockSpec(plain_att, None, TanhNormSpec(16), NormSpec(16, 1e-5)), CPU)


# ------------------------------------------------------------------------------- distances

@pytest.mark.parametrize("rows,reach", [(2, 3), (8, 40), (9, 64), (16, 128), (32, 1000), (12, 7)])
def test_distance_rows(rows, reach):
    """One row a distance in the first half, never a step back, at most one new row a distance from where the spans are
    shorter than one, the last row at the end; and the plain walk's own formula, distance by distance."""
    table = distance_rows(rows, reach)
    half = rows // 2
    assert table[:half] == list(range(half)) and table[-1] == rows - 1 and rows - 1 not in table[:-1]
    assert all(b >= a for a, b in zip(table, table[1:])) and len(table) <= reach + 1
    for n in range(3 * reach):
        assert plain.bucket(n, rows, reach) == table[min(n, len(table) - 1)]


# ------------------------------------------------------------------------------- the plain implementation against itself

def test_plain_small_pieces():
    a = torch.tensor([[1.0, 2.0], [3.0, 5.0], [0.0, 1.0]])
    assert torch.equal(plain.blend_with_previous(a, torch.tensor([0.0, 1.0])), torch.tensor([[1.0, 0.0], [3.0, 2.0], [0.0, 5.0]]))
    t = plain.temperature(10, 0.5, 4, torch.float64)                          # steps at positions 3 and 7
    assert t[0] == t[2] == 1.0 and t[3] == t[6] == 1.0 + 0.5 * math.log(2) and t[7] == 1.0 + 0.5 * math.log(3)
    ok = torch.tensor([[True, True, False]])
    p = plain.softmax_plus_one(torch.tensor([[1.0, -2.0, 9.0]]), ok)
    den = 1.0 + math.exp(1.0) + math.exp(-2.0)
    assert torch.allclose(p, torch.tensor([[math.exp(1.0) / den, math.exp(-2.0) / den, 0.0]]))
    z = plain.causal_conv(torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 1.0]]))
    assert z.flatten().tolist() == [1.0, 12.0, 24.0]
    picked, weight = plain.route(torch.tensor([[0.0, 3.0, -1.0, 1.0]]), 2)
    assert picked.tolist() == [[1, 3]] and torch.allclose(weight, torch.sigmoid(torch.tensor([[3.0, 1.0]])))


def test_plain_general_delta_removes_along_the_key_it_is_given():
    """With no decay and a rate of one the removal is the projection that clears the key's direction, whatever its length."""
    D = 4
    eye = torch.eye(D, dtype=torch.float64)
    w = {"r": eye, "k": eye, "v": eye, "g": torch.zeros(D, D, dtype=torch.float64), "o": eye, "norm": torch.full((D,), 2.0, dtype=torch.float64),
         "a": 0 * eye, "a.b": torch.full((D,), 50.0, dtype=torch.float64), "w1": torch.zeros(1, D, dtype=torch.float64),
         "w2": torch.zeros(D, 1, dtype=torch.float64), "w0": torch.full((D,), -60.0, dtype=torch.float64)}
    a = torch.tensor([[3.0, 0, 0, 0], [0, 2.0, 0, 0], [1.0, 0, 0, 0]], dtype=torch.float64)
    out = plain.general_delta(w, "", {"heads": 1, "dim": D}, a, 0.0)
    # row 2: S held 9 at (0, 0) and 4 at (1, 1); key e0 clears row 0 and writes 1 there; the read-out is e0 times one,
    # over its root mean square (1/2), times the weight 2 and the open-half gate
    assert torch.allclose(out[2], torch.tensor([2.0, 0, 0, 0], dtype=torch.float64), atol=1e-5)


def test_plain_model_is_causal_and_its_parts_matter(tmp_path):
    d = loader.write_random_model(str(tmp_path / "m"), LosoraxConfig(raw_config()), 2, torch.bfloat16)
    c, w = plain.read_model(d)
    ids = helpers.random_ids(97, 60, 3)
    full = plain.forward(c, w, ids)
    assert torch.allclose(plain.forward(c, w, ids[:31]), full[:31], atol=1e-9)            # nothing looks ahead
    for i, change in ((0, lambda m: m["q_temp"].update(coef=0.0)), (0, lambda m: m["q_temp"].update(every=17)),
                      (0, lambda m: m.update(bias_max=40)), (0, lambda m: m.update(scale=0.5)), (0, lambda m: m.update(conv=0))):
        c2 = copy.deepcopy(c)
        change(c2["layers"][i]["mixer"])
        assert not torch.allclose(plain.forward(c2, w, ids), full, atol=1e-6)
    for name in ("l0.shift", "l1.ls1", "l3.ls2", "l2.mix.rel", "l1.mix.a.b", "l3.mix.w0", "l2.norm1b.b", "final.norm.alpha"):
        w2 = dict(w)
        w2[name] = w[name] * 0.5 + 0.1
        assert not torch.allclose(plain.forward(c, w2, ids), full, atol=1e-6), name
