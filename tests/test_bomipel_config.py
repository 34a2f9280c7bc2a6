"""The Bomipel configuration on the CPU: the reader of its keys, what it refuses, the model it describes, frequencies in bands,
pages that a sequence keeps from its start, and the plain implementation's own premises."""

import copy
import math
import random

import pytest
import torch

from bomipel_tools import CONFIGS, draw_weights
from plain import plain_bomipel as plain
from quantinfer_b200.cache import CacheManager, PagedKVNeed
from quantinfer_b200.config import BomipelConfig, RotarySpec, config_from_dict
from quantinfer_b200.engine.model import tensor_needs_of_spec
from quantinfer_b200.errors import ConfigError
from quantinfer_b200.parts.position import direct_frequencies


def test_the_registry_finds_the_class_and_the_dictionary_comes_back():
    for cfg in CONFIGS.values():
        c = config_from_dict(cfg)
        assert isinstance(c, BomipelConfig) and c.to_dict() == cfg
        rebuilt = BomipelConfig(**{k: getattr(c, k) for k in ("vocab", "width", "norm_eps", "layers", "logit_softcap")})
        assert BomipelConfig.from_dict(rebuilt.to_dict()) == c


def test_the_model_it_describes():
    s = config_from_dict(CONFIGS["P"]).to_model_spec()
    assert [(c.layer, c.cache, c.writes_cache) for c in s.order] == [(i, i, True) for i in range(6)]
    assert (s.head.tied, s.head.softcap, s.embedding.weight_name, s.final_norm.kind, s.final_norm.prefix, s.final_norm.eps) == (
        True, 9.0, "embed", "rmsnorm_named", "final.norm", 3e-6)
    assert all(l.kind == "parallel" and l.norm.prefix == f"l{i}.norm1" for i, l in enumerate(s.layers))
    a, b = s.layers[0].mixer, s.layers[1].mixer
    assert (a.q_rank, a.kv_rank, a.rot_dim, a.window, a.sink, a.norm_eps, a.position.pairing, a.position.bands) == (13, 12, 6, None, False, 3e-6, "half_split", None)
    assert (b.num_heads, b.num_kv_heads, b.head_dim, b.value_dim, b.window, b.keep_first, b.value_mix, b.bias, b.out_gate) == (
        6, 3, 10, 7, 9, 3, "first", False, False)
    assert b.position == RotarySpec(4, 300.0, "interleaved", bands=(3.0, 1.0, 3.0, 60.0))
    assert [l.mixer.value_mix for l in s.layers if hasattr(l.mixer, "value_mix")] == ["first", None, "mix", "mix"]
    f = s.layers[3].ffn
    assert (f.experts, f.top, f.expert.intermediate_size, f.expert.activation, f.scoring, f.has_correction, f.normalize, f.weight_on, f.router_scale) == (
        7, 3, 12, "silu", "sigmoid", False, False, "input", 1.0)
    assert s.layers[2].ffn is None
    for cfg in CONFIGS.values():          # the tensors that the tests draw are the tensors that the model asks for
        needs = tensor_needs_of_spec(config_from_dict(cfg).to_model_spec())
        assert {k: tuple(v.shape) for k, v in draw_weights(cfg, 1).items()} == {k: tuple(n.shape) for k, n in needs.items()}


@pytest.mark.parametrize("edit, word", [
    (lambda d: d["layers"][0].update(type="mamba2"), "latent_attention"),
    (lambda d: d["layers"][1]["mixer"].update(heads=5), "multiple"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=0), "positive"),
    (lambda d: d["layers"][1]["mixer"].update(dim=300), "256"),
    (lambda d: d["layers"][1]["mixer"].update(scale=0.0), "scale"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda d: d["layers"][4]["mixer"].update(vdim=9), "layer 1"),
    (lambda d: d["layers"][1]["mixer"].update(v_mix="yes"), "v_mix"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=12), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(base=0.0), "rot.base"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("high"), "high"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high at least low"),
    (lambda d: d["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][0]["mixer"].update(kv_rank=600), "512"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "moe"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda d: d["layers"][0]["mlp"]["expert"].update(ff=0), "ff"),
    (lambda d: d.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda d: d["norm"].update(eps=0.0), "eps"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_what_it_refuses(edit, word):
    d = copy.deepcopy(CONFIGS["P"])
    edit(d)
    with pytest.raises(ConfigError) as err:
        config_from_dict(d)
    assert word in str(err.value)


@pytest.mark.parametrize("dims, base, bands", [(64, 10000.0, (8.0, 1.0, 4.0, 512)), (6, 50.0, (3.0, 1.0, 2.0, 40)), (32, 500000.0, (32.0, 1.0, 4.0, 8192)),
                                               (16, 100.0, (2.0, 2.0, 2.0, 64)), (8, 1000.0, (4.0, 1.0, 4.0, 1)), (8, 3.0, (4.0, 1.0, 4.0, 10 ** 9))])
def test_frequencies_in_bands(dims, base, bands):
    """All three bands against the plain rule; low equal to high (no pair in between); everything slowed, nothing slowed."""
    got, factor = direct_frequencies(RotarySpec(dims, base, "interleaved", bands=bands))
    want = plain.pair_frequencies(dims, base, dict(zip(("factor", "low", "high", "original"), bands)))
    assert factor == 1.0 and got.dtype == torch.float32
    assert torch.allclose(got.double(), want, rtol=1e-7, atol=0)
    as_is = plain.pair_frequencies(dims, base)
    ratio = got.double() / as_is
    length = 2 * math.pi / as_is
    assert torch.allclose(ratio[length < bands[3] / bands[2]], torch.ones(1).double(), rtol=1e-6)
    assert torch.allclose(ratio[length > bands[3] / bands[1]], torch.ones(1).double() / bands[0], rtol=1e-6)
    assert torch.all(ratio <= 1 + 1e-6) and torch.all(ratio >= 1 / bands[0] - 1e-6)


def test_rotations_that_cannot_be_are_refused():
    for spec in (RotarySpec(8, 100.0, bands=(0.0, 1.0, 4.0, 64)), RotarySpec(8, 100.0, bands=(2.0, 4.0, 1.0, 64)),
                 RotarySpec(8, 100.0, bands=(2.0, 1.0, 4.0, 64), stretch=(2.0, 64, 4.0, 1.0))):
        with pytest.raises(ConfigError):
            direct_frequencies(spec)


@pytest.mark.parametrize("keep, window, page", [(3, 9, 4), (4, 9, 4), (5, 6, 4), (11, 1, 4), (0, 7, 4), (1, 5, 8), (40, 4, 8)])
def test_pages_of_kept_first_positions_stay(keep, window, page):
    """At every length: the table holds exactly the pages in which the next query can see a position; closing gives all back."""
    m = CacheManager([PagedKVNeed(2, 8, window, keep_first=keep)], page, 40, 2, 128, device=None)
    m.open("a")
    rng, length = random.Random(keep), 0
    while length < 100:
        n = min(rng.choice([1, 1, 2, 5, 13]), 100 - length)
        m.prepare("a", n)
        m.commit("a")
        length += n
        m.check_invariants()
        table = m.table_row("a", 0)
        for b, p in enumerate(table):
            held = range(b * page, min((b + 1) * page, length))
            seen = any(j < keep or length - j < window for j in held)
            assert (p >= 0) == (seen or (b + 1) * page > length), (length, b)        # (a page with room is written next)
        assert m.live_length(0, length) == min(length, min(length, window) + keep)
    m.close("a")
    assert m.free_pages() == 40


def test_needs_with_and_without_kept_positions():
    a, b = PagedKVNeed(2, 8, 16, keep_first=4), PagedKVNeed(2, 8, 24, keep_first=2)
    assert a != PagedKVNeed(2, 8, 16) and a.merged(b) == PagedKVNeed(2, 8, 24, keep_first=4)
    groups = CacheManager([a, PagedKVNeed(2, 8, 16), a], 8, 4, 1, 64, device=None).groups
    assert [g.entries for g in groups] == [[0, 2], [1]]


def test_the_rules_on_small_numbers():
    """Each plain rule on a case worked out by hand."""
    ok = plain.visible(6, 2, 1)
    assert ok[5].tolist() == [True, False, False, False, True, True] and ok[0].tolist() == [True] + [False] * 5
    assert plain.visible(3).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    assert plain.mix_values(torch.tensor(2.0), torch.tensor(10.0), 0.25) == 4.0
    s, e = plain.route(torch.tensor([[1.0]]).double(), torch.tensor([[0.0], [2.0], [-1.0]]), 2)
    assert e.tolist() == [[1, 0]] and s[0].tolist() == pytest.approx([1 / (1 + math.exp(-2)), 0.5])
    w = {"e0.gate": torch.tensor([[1.0]]), "e0.up": torch.tensor([[3.0]]), "e0.down": torch.tensor([[2.0]]), "router": torch.tensor([[0.0]])}
    y = plain.mixture(torch.tensor([[4.0]]).double(), {"router": {"top": 1}}, w, "")
    assert float(y) == pytest.approx(2.0 / (1 + math.exp(-2)) * 6.0 * 2.0)          # the expert reads 0.5 * 4
    f = plain.pair_frequencies(4, 100.0, {"factor": 2.0, "low": 1.0, "high": 4.0, "original": 2 * math.pi * 20})
    assert f.tolist() == pytest.approx([1.0, (1 - 1 / 3) * 0.05 + 0.1 / 3])         # wavelengths 2 pi (kept) and 20 pi (a third of the way)


def test_random_tensors_of_the_design():
    from quantinfer_b200.weights import random_tensors

    t = random_tensors(tensor_needs_of_spec(config_from_dict(CONFIGS["Q"]).to_model_spec()), 3)
    assert t["l0.mix.vmix"].shape == () and 0.4 <= float(t["l2.mix.vmix"]) <= 0.6 and t["l1.mix.uq"].shape == (4 * 48, 48)


def test_the_comparison_of_the_bench():
    """`bench.py --compare bomipel`: the stacks are valid configurations of their designs; the Kiruvik stack holds the same
    weights to 6 % (its attention has an output gate), and the arithmetic's count is the count of the tensors."""
    import bench

    for size in bench.BOMIPEL_SIZES:
        new, kir, beb = bench.bomipel_entries(size)
        a, b, _ = (bench.model_arithmetic(c, c.to_model_spec()) for c in (config_from_dict(e["config"]) for e in (new, kir, beb)))
        assert abs(a["weight_bytes"] / b["weight_bytes"] - 1.0) < 0.06
        needs = tensor_needs_of_spec(config_from_dict(new["config"]).to_model_spec())
        stored = sum(math.prod(n.shape) for k, n in needs.items() if len(n.shape) == 2 and k != "embed")
        assert abs(stored / a["stored_params"] - 1.0) < 0.001
