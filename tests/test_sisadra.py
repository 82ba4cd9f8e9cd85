"""Sisadra without a GPU: the configuration reader, the model as data (what every layer keeps, tensor names and shapes),
the random-weights folder, and properties of the plain implementation that the GPU tests rely on."""
import copy
import math

import pytest
import torch

import plain_sisadra as ps
import sisadra_tiny as st

F64 = torch.float64


def spec_of(cfg):
    from flambeau_b200 import models  # noqa: F401
    from flambeau_b200.config.registry import resolve
    arch = resolve("Sisadra")
    return arch.build_spec(arch.config_class.from_dict(cfg))


def changed(cfg, path, value):
    out = copy.deepcopy(cfg)
    at = out
    for k in path[:-1]:
        at = at[k]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return out


def test_config_round_trip_and_errors():
    from flambeau_b200.config.base import BadValue, MissingKey
    from flambeau_b200.config.sisadra import SisadraConfig
    for cfg in st.CONFIGS.values():
        c = SisadraConfig.from_dict(cfg)
        assert SisadraConfig.from_dict(c.to_dict()) == c and c.to_dict()["layers"] == cfg["layers"]
    c = SisadraConfig.from_dict(st.CONFIG_DA)
    assert (c.vocab, c.width, c.norm_eps, c.embedding_scale, c.logit_softcap) == (200, 64, 1e-5, 2.5, 12.0)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur) == (53, 5, 11)
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.scale, a.diff) == (4, 2, 32, 48, 20, 0.3, 0.4)
    assert (a.rot.base, a.rot.dims, a.rot.scaling) == (1e4, 8, {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 64.0})
    b = SisadraConfig.from_dict(st.CONFIG_DB)
    assert b.bigram is None and b.logit_softcap == 0.0 and b.layers[3].mixer.chunk == 0 and b.layers[3].mixer.rot.scaling is None
    assert c.layers[3].mixer.rot is None and c.layers[2].ff == 0 and c.layers[4].ff == 56
    bare = copy.deepcopy(st.CONFIG_DC)
    del bare["embedding"], bare["logit_softcap"], bare["layers"][0]["mixer"]["kv_heads"], bare["layers"][0]["mixer"]["vdim"]
    bare["layers"][1]["mixer"]["rot"]["dims"] = 0
    d = SisadraConfig.from_dict(bare)
    assert (d.embedding_scale, d.bigram, d.layers[0].mixer.kv_heads, d.layers[0].mixer.vdim, d.layers[1].mixer.rot) == (1.0, None, 3, 10, None)
    for path, value in [(("layers", 0, "mixer", "rot", "dims"), 34), (("layers", 0, "mixer", "rot", "dims"), 7),
                        (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 2, "mixer", "kv_heads"), 4),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 2, "mixer", "conv"), 0),
                        (("layers", 0, "mixer", "rot", "scaling", "low"), 5.0), (("layers", 1, "mixer", "scale"), 0.0),
                        (("layers", 1, "type"), "attention_2"), (("layers", 1, "mlp", "kind"), "moe"),
                        (("embedding", "bigram", "buckets"), 0), (("logit_softcap",), -1.0), (("layers",), [])]:
        with pytest.raises(BadValue):
            SisadraConfig.from_dict(changed(st.CONFIG_DA, path, value))
    for path in [("layers", 0, "mixer", "diff"), ("layers", 0, "mixer", "rot", "scaling", "high"), ("norm", "eps"),
                 ("layers", 1, "mixer", "kv_rank"), ("layers", 2, "mixer", "conv"), ("embedding", "bigram", "mul_prev")]:
        with pytest.raises(MissingKey):
            SisadraConfig.from_dict(changed(st.CONFIG_DA, path, KeyError))


def test_what_every_layer_keeps():
    from flambeau_b200.models.decoder import DecoderModel
    plans = DecoderModel(spec_of(st.CONFIG_DA), runtime=None).cache_plans()
    assert len(plans) == 6 and all(p.cache_from is None for p in plans)
    a, lat, rec = plans[0].kv, plans[1].kv, plans[2]
    assert (a.kv_heads, a.head_dim, a.value_dim, a.window, a.chunk, a.release_window) == (2, 64, 48, 0, 20, 20)
    assert (lat.kv_heads, lat.head_dim, lat.values_in_keys, lat.chunk, lat.release_window) == (1, 48, True, 0, 0), "c alone"
    channels = 2 * 2 * 24 + 6 * 16
    assert rec.kv is None and rec.state.dtype == "float32" and rec.state.shape[0] >= 6 * 24 * 16 + 3 * channels
    assert plans[3].kv.chunk == 1 and plans[4].state.shape[0] >= 3 * 16 * 32
    assert plans[5].kv is None and plans[5].state.shape == (1,) and plans[5].state.dtype == "int32", "the token before"
    assert len(DecoderModel(spec_of(st.CONFIG_DB), runtime=None).cache_plans()) == 4, "no pairs: nothing beside the caches"


def test_tensor_names_and_shapes():
    from flambeau_b200.models.decoder import DecoderModel
    specs = DecoderModel(spec_of(st.CONFIG_DA), runtime=None).tensor_specs()
    want = {"embed": (200, 64), "bigram": (54, 64), "head": (200, 64), "final.norm": (64,), "l0.norm1": (64,), "l0.norm2": (64,),
            "l0.mix.q": (256, 64), "l0.mix.q.b": (256,), "l0.mix.k": (128, 64), "l0.mix.k.b": (128,), "l0.mix.v": (96, 64),
            "l0.mix.v.b": (96,), "l0.mix.q.norm": (32,), "l0.mix.k.norm": (32,), "l0.mix.lq1": (32,), "l0.mix.lk2": (32,),
            "l0.mix.o": (64, 192), "l0.mix.o.b": (64,), "l0.mlp.up": (80, 64), "l0.mlp.down": (64, 80),
            "l1.mix.q": (48, 64), "l1.mix.dkv": (48, 64), "l1.mix.dkv.norm": (48,), "l1.mix.uk": (48, 48),
            "l1.mix.uv": (72, 48), "l1.mix.sink": (3,), "l1.mix.o": (64, 72),
            "l2.mix.q": (48, 64), "l2.mix.q.conv": (48, 4), "l2.mix.v": (96, 64), "l2.mix.v.conv": (96, 4), "l2.mix.b": (6, 64),
            "l2.mix.A_log": (6,), "l2.mix.dt_bias": (144,), "l2.mix.norm": (16,), "l2.mix.o": (64, 96)}
    for name, shape in want.items():
        assert name in specs and tuple(specs[name].shape) == shape, name
    for name, fixed, free in (("a1", (1, 64), 0), ("a2", (0, 144), 1), ("g1", (1, 64), 0), ("g2", (0, 96), 1)):
        ts = specs["l2.mix." + name]
        assert ts.free_axes == (free,) and ts.shape[fixed[0]] == fixed[1], "the file says how wide a narrow middle is"
    assert not any(n in specs for n in ("l2.norm2", "l2.mlp.up", "l1.mix.g", "l1.mix.dq", "l0.mix.g", "l2.mix.a", "l2.mix.g"))
    assert len([n for n in specs if n.startswith("l1.")]) == 2 + 7 + 2 and len([n for n in specs if n.startswith("l2.")]) == 1 + 15


def test_random_folder_is_read_back_by_the_oracle(tmp_path):
    for name, dtype in (("DC", "bfloat16"), ("DA", "float32")):
        cfg, w = ps.read_folder(st.make_folder(tmp_path / name, st.CONFIGS[name], seed=5, dtype=dtype))
        runs = []
        logits = ps.forward(cfg, w, [1, 2, 3, 4, 5, 6, 7], runs)
        assert logits.shape == (7, cfg["vocab"]) and bool(torch.isfinite(logits).all()) and len(runs) == len(cfg["layers"])
        assert float(logits.abs().max()) < cfg["logit_softcap"]
        assert any(w[n].shape[0] != w[n.replace("a1", "g1")].shape[0] for n in w if n.endswith(".a1"))


def test_middles_that_do_not_fit_are_refused():
    from flambeau_b200.parts.gated_delta import GatedDeltaRule
    kw = dict(width=8, num_heads=2, num_qk_heads=1, key_dim=4, value_dim=4, conv=2, decay="channel", gate="sigmoid",
              low_rank_gate=True, rank=3)
    part = GatedDeltaRule(None, "m.", **kw)
    t = {n: torch.zeros(s.shape) for n, s in part.tensor_specs().items()}
    part.bind(t)
    t["m.a1"] = torch.zeros(5, 8)
    with pytest.raises(ValueError, match="a1"):
        part.bind(t)
    for bad in (dict(decay="row"), dict(gate="tanh"), dict(num_qk_heads=3), dict(conv=0)):
        with pytest.raises(ValueError):
            GatedDeltaRule(None, "m.", **dict(kw, **bad))


def test_parts_refuse_what_does_not_fit():
    from flambeau_b200.parts.diff_attention import DifferentialAttention
    from flambeau_b200.parts.embedding import LMHead
    from flambeau_b200.parts.spec import PartSpec
    kw = dict(width=16, num_heads=2, num_kv_heads=1, key_dim=8, value_dim=8)
    rot = PartSpec("position", "rotary_half", dict(head_dim=16, theta=10.0))
    for bad in (dict(position=rot, head_gate=False), dict(qk_norm=True, head_gate=True), dict(num_kv_heads=3)):
        with pytest.raises(ValueError):
            DifferentialAttention(None, "a.", **dict(kw, **bad))
    with pytest.raises(ValueError):
        LMHead(None, "h.", vocab=4, width=4, softcap=-1.0)


def test_command_line_makes_and_inspects_a_model(tmp_path):
    import json
    from flambeau_b200.cli import main
    (tmp_path / "c.json").write_text(json.dumps(st.CONFIG_DC))
    assert main(["random-model", "--config", str(tmp_path / "c.json"), "--out", str(tmp_path / "m"), "--seed", "3"]) == 0
    assert main(["inspect", "--model", str(tmp_path / "m")]) == 0
    cfg, w = ps.read_folder(tmp_path / "m")
    assert cfg["architecture"] == "Sisadra" and w["l2.mix.uv"].shape == (20, 20)


@pytest.mark.parametrize("rot", [st.rotation(1e4, 64, 8.0, 1.0, 4.0, 64), st.rotation(500.0, 16, 4.0, 0.5, 2.0, 200),
                                 st.rotation(50.0, 2, 3.0, 2.0, 2.0, 7), st.rotation(5e5, 96, 1.0, 1.0, 4.0, 4096),
                                 st.rotation(1e5, 40, 16.0, 1.0, 32.0, 512), st.rotation(1e4, 16)], ids=str)
def test_frequencies_in_bands(rot):
    from flambeau_b200.parts.positions import RotaryHalf, RotaryNeighbours
    want = ps.frequencies(rot)
    for cls in (RotaryHalf, RotaryNeighbours):
        part = cls(None, "", head_dim=rot["dims"], theta=rot["base"], rotary_dim=rot["dims"], stretch=rot.get("scaling"))
        assert torch.allclose(torch.tensor(part.frequencies, dtype=F64), want, rtol=1e-12) and part.magnitude == 1.0
    if "scaling" in rot:
        plain = ps.frequencies({"base": rot["base"], "dims": rot["dims"]})
        f = rot["scaling"]["factor"]
        assert bool((want <= plain * (1 + 1e-12)).all()) and bool((want >= plain / f * (1 - 1e-12)).all())
    if rot["base"] == 1e4 and "scaling" in rot:       # all three bands are there
        plain = ps.frequencies({"base": rot["base"], "dims": rot["dims"]})
        ratio = want / plain
        assert bool((ratio == 1.0).any()) and bool(((ratio - 0.125).abs() < 1e-12).any()) and bool(((ratio > 0.13) & (ratio < 0.99)).any())


# ---- properties of the plain implementation ----------------------------------------------------------------------
def test_what_a_position_sees():
    seen = ps.same_chunk(9, 3)
    assert seen[5].nonzero().flatten().tolist() == [3, 4, 5] and seen[6].nonzero().flatten().tolist() == [6]
    assert bool((ps.same_chunk(5, 1) == torch.eye(5, dtype=torch.bool)).all())
    assert bool((ps.same_chunk(6, None) == torch.tril(torch.ones(6, 6, dtype=torch.bool))).all())


def test_a_sink_takes_its_share_and_no_more():
    s = torch.tensor([[0.0, 1.0, 500.0]], dtype=F64)
    seen = torch.tensor([[True, True, False]])
    p = ps.sink_softmax(s, seen, torch.tensor(2.0, dtype=F64))
    z = 1.0 + math.e + math.exp(2.0)
    assert torch.allclose(p, torch.tensor([[1.0 / z, math.e / z, 0.0]], dtype=F64))


def test_the_delta_rule_by_hand():
    """A key written twice: the second write corrects towards its value; rows decay each by their own factor."""
    one, q = torch.tensor([1.0, 0.0], dtype=F64), torch.tensor([1.0, 1.0], dtype=F64)
    k = torch.stack([one, torch.tensor([0.0, 1.0], dtype=F64), one])
    v = torch.tensor([[4.0], [6.0], [10.0]], dtype=F64)
    g = torch.tensor([[1.0, 1.0], [0.5, 0.25], [0.5, 0.5]], dtype=F64)
    o = ps.delta_rule(torch.stack([q] * 3), k, v, torch.tensor([1.0, 1.0, 0.5], dtype=F64), g)
    # after 1: rows (4, 0); after 2: (2, 6); decayed to (1, 3), then the first row moves half-way from 1 to 10
    assert o.flatten().tolist() == [4.0, 8.0, 8.5]


def test_decays_lie_between_nought_and_one_and_differ_by_channel():
    g = torch.Generator().manual_seed(0)
    w = {"a1": torch.randn(3, 8, generator=g, dtype=F64), "a2": torch.randn(12, 3, generator=g, dtype=F64),
         "dt_bias": torch.randn(12, generator=g, dtype=F64), "A_log": torch.randn(2, generator=g, dtype=F64)}
    d = ps.channel_decays(torch.randn(5, 8, generator=g, dtype=F64), w, "", 2, 6)
    assert d.shape == (5, 2, 6) and bool(((d > 0) & (d < 1)).all()) and float(d.std(dim=-1).min()) > 0.0


def test_the_difference_of_two_equal_maps():
    a = torch.tensor([[3.0, -4.0]], dtype=F64)
    assert torch.allclose(ps.difference_of_maps(a, a, 0.25, 0.2, 0.0), 0.8 * a / math.sqrt(12.5))
    assert torch.equal(ps.difference_of_maps(a, a, 1.0, 0.2, 1e-6), torch.zeros_like(a))
