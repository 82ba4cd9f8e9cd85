"""Saropel without a GPU: the configuration reader, the model as data (run order, one cache per pass of the looped
stretch, what is kept per request, tensor names), the random-weights folder, and properties of the plain implementation
that the GPU tests rely on."""
import copy
import math

import pytest
import torch

import plain_saropel as ps
import saropel_tiny as st

F64 = torch.float64


def spec_of(cfg):
    from flambeau_b200 import models  # noqa: F401
    from flambeau_b200.config.registry import resolve
    arch = resolve("Saropel")
    return arch.build_spec(arch.config_class.from_dict(cfg))


def test_config_round_trip_and_errors():
    from flambeau_b200.config.base import BadValue, MissingKey
    from flambeau_b200.config.saropel import SaropelConfig
    for cfg in st.CONFIGS.values():
        c = SaropelConfig.from_dict(cfg)
        assert SaropelConfig.from_dict(c.to_dict()) == c
    c = SaropelConfig.from_dict(st.CONFIG_SA)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur, c.side_dim) == (53, 5, 11, 12)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 3)
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.softcap, a.rot) == (4, 2, 16, 24, 9, 2.5, None)
    m = c.layers[0].mlp
    assert (m.experts, m.top, m.groups, m.keep_groups, m.expert.limit, m.shared.ff, m.shared.limit) == (6, 3, 3, 2, 0.8, 40, 0.5)
    assert c.layers[1].mixer.rot.scaling["factor"] == 3.0 and c.layers[3].mixer.rot.scaling is None
    assert c.layers[2].mlp is None and c.layers[3].mlp.shared is None and c.layers[3].mlp.keep_groups == 0
    b = SaropelConfig.from_dict(st.CONFIG_SB)
    assert b.bigram is None and b.loop is None and b.layers[3].mixer.window == 0
    assert SaropelConfig.from_dict(st.CONFIG_SC).side_dim == 0
    for path, value, err in [(("layers", 1, "mixer", "rot", "dims"), 34, BadValue),           # more than a head has
                             (("layers", 1, "mixer", "rot", "dims"), 7, BadValue),            # odd
                             (("layers", 1, "mixer", "vdim"), 16, BadValue),                  # the values are the keys
                             (("layers", 0, "mixer", "kv_heads"), 3, BadValue),
                             (("layers", 0, "mixer", "softcap"), 0.0, BadValue),
                             (("layers", 0, "mlp", "router", "groups", "count"), 4, BadValue),  # 6 experts in 4 groups
                             (("layers", 0, "mlp", "router", "groups", "keep"), 4, BadValue),
                             (("layers", 0, "mlp", "router", "top"), 5, BadValue),            # 2 groups hold 4 experts
                             (("layers", 0, "mlp", "expert", "limit"), -1.0, BadValue),
                             (("layers", 1, "type"), "attention_3", BadValue),
                             (("layers", 3, "mlp", "kind"), "sparse", BadValue),
                             (("embedding", "bigram", "buckets"), 0, BadValue),
                             (("loop", "stop"), 5, BadValue)]:
        bad = copy.deepcopy(st.CONFIG_SA)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(err):
            SaropelConfig.from_dict(bad)
    for path in [("layers", 0, "mixer", "scale"), ("layers", 1, "mixer", "rot", "scaling", "slow"), ("norm", "eps"),
                 ("layers", 0, "mlp", "expert", "limit"), ("embedding", "bigram", "mul_cur")]:
        bad = copy.deepcopy(st.CONFIG_SA)
        at = bad
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(MissingKey):
            SaropelConfig.from_dict(bad)


def test_run_order_and_what_is_kept_per_request():
    from flambeau_b200.models.decoder import DecoderModel
    spec = spec_of(st.CONFIG_SA)
    assert [c.layer for c in spec.order] == [0, 1, 2, 1, 2, 1, 2, 3] == [i for i, _ in ps.run_order(st.CONFIG_SA)]
    assert [c.pass_index if c.reenter else None for c in spec.order] == [t for _, t in ps.run_order(st.CONFIG_SA)]
    plans = DecoderModel(spec, runtime=None).cache_plans()
    assert len(plans) == 9 and all(p.cache_from is None and p.state is None for p in plans[:8]), "a cache for every pass"
    assert plans[8].kv is None and plans[8].state.shape == (1,) and plans[8].state.dtype == "int32", "the token before"
    kv = plans[0].kv
    assert (kv.kv_heads, kv.head_dim, kv.value_dim, kv.window) == (2, 16, 24, 9)
    assert plans[1].kv == plans[3].kv == plans[5].kv and plans[1].kv.head_dim == plans[1].kv.value_dim == 32
    assert plans[7].kv.window == 0
    assert len(DecoderModel(spec_of(st.CONFIG_SB), runtime=None).cache_plans()) == 4, "no pairs: nothing beside the caches"
    assert spec.layers[0].kind == "token_input" and spec_of(st.CONFIG_SC).layers[0].kind == "parallel"
    assert spec_of(st.CONFIG_SB).reentry is None


def test_tensor_names_and_shapes():
    from flambeau_b200.models.decoder import DecoderModel
    model = DecoderModel(spec_of(st.CONFIG_SA), runtime=None)
    specs = model.tensor_specs()
    want = {"embed": (200, 64), "bigram": (54, 64), "side.embed": (200, 48), "loop.step": (3, 64), "head": (200, 64),
            "final.norm": (64,), "l0.norm1": (64,), "l0.mix.q": (64, 64), "l0.mix.k": (32, 64), "l0.mix.v": (48, 64),
            "l0.mix.o": (64, 96), "l0.mlp.router": (6, 64), "l0.mlp.e5.gate": (24, 64), "l0.mlp.e5.down": (64, 24),
            "l0.mlp.shared.up": (40, 64), "l0.mlp.shared.sg": (1, 64), "l0.side.gate": (12, 64), "l0.side.proj": (64, 12),
            "l0.side.norm": (64,), "l1.mix.q": (128, 64), "l1.mix.k": (64, 64), "l1.mix.q.norm": (32,),
            "l1.mix.k.norm": (32,), "l1.mix.g": (4, 64), "l1.mix.o": (64, 128), "l1.mlp.gate": (48, 64),
            "l1.mlp.down": (64, 48), "l3.mlp.e3.up": (32, 64)}
    for name, shape in want.items():
        assert name in specs and tuple(specs[name].shape) == shape, name
    assert not any(n.startswith("l2.mlp.") or n.endswith(".norm2") for n in specs), "one norm a layer, one without feed-forward"
    assert not any(n in specs for n in ("l1.mix.v", "l0.mix.g", "l0.mix.q.norm", "l3.mlp.shared.sg", "l0.mlp.router.b"))
    assert model.shared_tensor_names() == {"side.embed"}, "the layers' columns lie in one table"
    assert not any(n.startswith(("bigram", "loop")) for n in DecoderModel(spec_of(st.CONFIG_SB), runtime=None).tensor_specs())
    assert not any("side" in n for n in DecoderModel(spec_of(st.CONFIG_SC), runtime=None).tensor_specs())


def test_random_folder_is_read_back_by_the_oracle(tmp_path):
    for name, dtype in (("SC", "bfloat16"), ("SA", "float32")):
        folder = st.make_folder(tmp_path / name, st.CONFIGS[name], seed=5, dtype=dtype, steady_router=dtype == "bfloat16")
        cfg, w = ps.read_folder(folder)
        assert cfg["width"] == st.CONFIGS[name]["width"] and "l1.mix.k.norm" in w
        runs = []
        logits = ps.forward(cfg, w, [1, 2, 3, 4, 5, 6, 7], collect=runs)
        assert logits.shape == (7, cfg["vocab"]) and bool(torch.isfinite(logits).all())
        assert len(runs) == len(ps.run_order(cfg))


def test_command_line_makes_and_inspects_a_model(tmp_path):
    import json
    from flambeau_b200.cli import main
    (tmp_path / "c.json").write_text(json.dumps(st.CONFIG_SC))
    assert main(["random-model", "--config", str(tmp_path / "c.json"), "--out", str(tmp_path / "m"), "--seed", "3"]) == 0
    assert main(["inspect", "--model", str(tmp_path / "m")]) == 0
    cfg, w = ps.read_folder(tmp_path / "m")
    assert cfg["architecture"] == "Saropel" and w["l1.mlp.e1.down"].shape == (36, 16)


def test_parts_refuse_what_does_not_fit():
    from flambeau_b200.kernels.library import KernelError
    from flambeau_b200.parts.attention import PagedAttention
    from flambeau_b200.parts.block import TokenInputBlock
    from flambeau_b200.parts.feedforward import GatedMLP
    from flambeau_b200.parts.moe import RoutedExperts
    from flambeau_b200.parts.spec import PartSpec
    kw = dict(width=16, num_heads=2, num_kv_heads=1, head_dim=8)
    for bad in (dict(gate="row"), dict(softcap=-1.0), dict(values_from_keys=True, value_dim=4)):
        with pytest.raises(ValueError):
            PagedAttention(None, "a.", **kw, **bad)
    with pytest.raises(KernelError):
        GatedMLP(None, "m.", width=16, inner=8, activation="limited")          # no limit
    base = dict(width=16, inner=8, experts=6, top=3, gated=True, activation="silu")
    for bad in (dict(groups=4), dict(rule="softmax_of_all", groups=3, keep_groups=1), dict(groups=3, keep_groups=2),
                dict(rule="softmax_of_all", groups=3, keep_groups=4), dict(shared_gate=True)):
        with pytest.raises(ValueError):
            RoutedExperts(None, "m.", **base, **bad)
    block = PartSpec("block", "parallel", dict(mixer=PartSpec("mixer", "attention", kw, "a."),
                                               norm=PartSpec("norm", "rmsnorm", dict(width=16, eps=1e-5), "n.")), "")
    with pytest.raises(ValueError):
        TokenInputBlock(None, "s.", block=block, norm=PartSpec("norm", "rmsnorm", dict(width=16, eps=1e-5), "s."), width=16,
                        dim=4, offset=6, vocab=10, table="t", table_width=8)


@pytest.mark.parametrize("rot", [st.rotation(2e4, 40, 6.0, 300), st.rotation(100.0, 6, 2.0), st.rotation(1e3, 64, 8.0, 32, 4.0, 0.5),
                                 st.rotation(5e5, 128, 1.0, 4096), st.rotation(1e4, 16), st.rotation(50.0, 2, 3.0, 7, 2.0, 1.9)],
                         ids=str)
def test_stretched_frequencies_of_both_pairings(rot):
    from flambeau_b200.parts.positions import RotaryHalf, RotaryNeighbours
    want, magnitude = ps.frequencies(rot)
    for cls in (RotaryHalf, RotaryNeighbours):
        part = cls(None, "", head_dim=rot["dims"], theta=rot["base"], rotary_dim=rot["dims"], stretch=rot.get("scaling"))
        assert torch.allclose(torch.tensor(part.frequencies, dtype=F64), want, rtol=1e-12) and math.isclose(part.magnitude, magnitude)
    if "scaling" in rot and rot["scaling"]["factor"] > 1.0:
        plain, one = ps.frequencies({"base": rot["base"], "dims": rot["dims"]})
        assert magnitude > one and bool((want <= plain).all())
        assert bool((want >= plain / rot["scaling"]["factor"] - 1e-15).all())


# ---- properties of the plain implementation ----------------------------------------------------------------------
def test_rows_of_the_pair_table():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 4}
    assert ps.pair_rows([5, 1, 2], b).tolist() == [10, (15 + 4) % 10, (3 + 8) % 10]
    assert ps.pair_rows([7], b).tolist() == [10]
    assert ps.pair_rows([1, 2], b).tolist() != ps.pair_rows([2, 1], b).tolist()


def test_what_a_position_sees():
    seen = ps.visible(8, 3)
    assert seen[7].nonzero().flatten().tolist() == [5, 6, 7] and seen[0].nonzero().flatten().tolist() == [0]
    assert bool((ps.visible(5, 1) == torch.eye(5, dtype=torch.bool)).all())
    assert bool((ps.visible(6, None) == torch.tril(torch.ones(6, 6, dtype=torch.bool))).all())


def test_a_cap_bends_large_scores_and_leaves_small_ones():
    s = torch.tensor([-1e3, -0.01, 0.0, 0.01, 2.0, 1e3], dtype=F64)
    c = ps.capped(s, 5.0)
    assert float(c.abs().max()) <= 5.0 and torch.allclose(c[1:4], s[1:4], atol=1e-7) and 1.8 < float(c[4]) < 2.0
    assert torch.equal(ps.capped(s, None), s)


def test_experts_are_chosen_within_the_best_groups():
    scores = torch.tensor([[0.30, 0.01, 0.20, 0.19, 0.25, 0.05]], dtype=F64)
    router = {"top": 2, "groups": {"count": 3, "keep": 1}}
    chosen, weights = ps.choose(scores, router)
    assert chosen.tolist() == [[0, 1]] and torch.allclose(weights, torch.tensor([[0.30, 0.01]], dtype=F64)), \
        "the group of the largest score, though its second is the smallest of all; weights as they are"
    assert ps.choose(scores, {"top": 3, "groups": {"count": 3, "keep": 2}})[0].tolist() == [[0, 4, 5]]
    assert ps.choose(scores, {"top": 3})[0].tolist() == [[0, 4, 2]]
    assert ps.choose(scores, {"top": 3, "groups": {"count": 3, "keep": 3}})[0].tolist() == [[0, 4, 2]]


def test_an_expert_cuts_its_operands_off():
    w = {"gate": torch.tensor([[1.0]], dtype=F64), "up": torch.tensor([[1.0]], dtype=F64), "down": torch.tensor([[1.0]], dtype=F64)}
    big, low = (float(ps.limited_expert(torch.tensor([[v]], dtype=F64), w, "", 2.0)) for v in (50.0, -50.0))
    assert math.isclose(big, 2.0 / (1.0 + math.exp(-3.404)) * 3.0)
    assert math.isclose(low, -50.0 / (1.0 + math.exp(85.1)) * -1.0), "the gate is cut from above only, the up side from both"


def test_the_values_are_the_keys_before_norm_and_rotation():
    g = torch.Generator().manual_seed(0)
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0, "mask": {"size": 1}, "rot": st.rotation(10.0, 4, 2.0)}
    w = {n: torch.randn(s, generator=g, dtype=F64) for n, s in (("q", (4, 4)), ("k", (4, 4)), ("o", (4, 4)), ("g", (1, 4)),
                                                                ("q.norm", (4,)), ("k.norm", (4,)))}
    h = torch.randn(3, 4, generator=g, dtype=F64)
    want = ((h @ w["k"].T) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T         # a window of one key: its own value
    assert torch.allclose(ps.shared_kv_attention(h, w, "", m, 1e-5, range(3)), want)


def test_passes_add_the_embedding_but_for_the_first_and_a_vector_each():
    cfg = {"norm": {"eps": 1e-5}, "vocab": 5, "width": 4, "loop": {"start": 0, "stop": 1, "times": 3},
           "layers": [dict(st.capped(1, 1, 4, 4, 2, 1.0), mlp=None)]}
    g = torch.Generator().manual_seed(1)
    w = {n: torch.randn(s, generator=g, dtype=F64) for n, s in (
        ("embed", (5, 4)), ("head", (5, 4)), ("final.norm", (4,)), ("loop.step", (3, 4)), ("l0.norm1", (4,)),
        ("l0.mix.q", (4, 4)), ("l0.mix.k", (4, 4)), ("l0.mix.v", (4, 4)))}
    w["l0.mix.o"] = torch.zeros(4, 4, dtype=F64)
    runs = []
    ps.forward(cfg, w, [3], runs)
    x0 = w["embed"][3]
    for t, want in enumerate((x0, 2 * x0, 3 * x0)):
        assert torch.allclose(runs[t][0], want + w["loop.step"][:t + 1].sum(0))
