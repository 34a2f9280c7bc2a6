"""The Siditar configuration on the CPU: the reader of its keys, what it refuses, the model it describes, the rows that a
distance bias reads, and the plain implementation's own premises."""

import copy
import math

import pytest
import torch

from plain import plain_siditar as plain
from siditar_tools import CONFIGS, clean, draw_weights
from quantinfer_b200.config import SiditarConfig, config_from_dict
from quantinfer_b200.engine.model import tensor_needs_of_spec
from quantinfer_b200.errors import ConfigError
from quantinfer_b200.parts.position import distance_buckets


def test_the_registry_finds_the_class_and_the_dictionary_comes_back():
    for name, cfg in CONFIGS.items():
        c = config_from_dict(clean(cfg))
        assert isinstance(c, SiditarConfig)
        assert c.to_dict() == clean(cfg)
        rebuilt = SiditarConfig(**{k: getattr(c, k) for k in ("vocab", "width", "streams", "norm_eps", "layers", "loop")})
        assert SiditarConfig.from_dict(rebuilt.to_dict()) == c


def test_the_model_it_describes():
    s = config_from_dict(clean(CONFIGS["P"])).to_model_spec()
    assert [call.layer for call in s.order] == [0, 1, 2, 1, 2, 3]
    assert [(call.cache, call.writes_cache, call.reenter) for call in s.order] == [(i, True, False) for i in range(6)]     # a cache a pass
    assert (s.embedding.copies, s.embedding.sinusoid_base, s.final_norm.kind, s.final_norm.streams, s.final_norm.norm.kind) == (
        3, 10000.0, "stream_sum", 3, "layernorm_nobias")
    b = s.layers[0]
    assert (b.kind, b.streams, b.names, b.mixer_norm.eps) == ("hyper", 3, ("l0.hc1", "l0.hc2"), 3e-6)
    assert (b.ffn.intermediate_size, b.ffn.limit, b.ffn.alpha) == (56, 1.5, 1.702)
    assert b.mixer.branch_scales == (0.8, 1.3)
    l, r = b.mixer.left, b.mixer.right
    assert (l.num_heads, l.num_kv_heads, l.head_dim, l.value_dim, l.scale, l.window, l.chunk, l.sink, l.qk_norm, l.qk_norm_eps, l.q_temp,
            l.distance_bias, l.position, l.bias, l.out_gate) == (
        6, 3, 10, 7, 1.0 / math.sqrt(10), None, None, "learned", "head", 3e-6, (0.4, 16), 40.0, None, False, False)
    assert (r.heads, r.head_dim, r.value_dim, r.tau, r.norm_eps) == (4, 5, 7, 8.0, 3e-6)
    assert s.layers[1].ffn is None and s.layers[1].names == ("l1.hc1",) and s.layers[3].mixer.left.q_temp is None
    needs = tensor_needs_of_spec(s)
    assert "l1.norm2" not in needs and "l1.hc2.in" not in needs and needs["l0.hc2.mix"].shape == (3, 3)
    assert needs["l0.mix.left.rel"].shape == (None, 6) and needs["l0.mix.left.q.norm"].shape == (10,) and needs["l0.mix.left.v"].shape == (21, 44)
    assert needs["l0.mix.right.a1"].shape == (None, 44) and needs["l0.mix.right.a2"].shape == (20, None) and needs["l0.mix.right.a2.b"].shape == (20,)
    for name, cfg in CONFIGS.items():          # the tensors that the tests draw are the tensors that the model asks for
        needs = tensor_needs_of_spec(config_from_dict(clean(cfg)).to_model_spec())
        w = draw_weights(cfg, 1)
        assert set(w) == set(needs)
        assert all(len(needs[k].shape) == w[k].dim() and all(a is None or a == b for a, b in zip(needs[k].shape, w[k].shape)) for k in w)
    assert [c.layer for c in config_from_dict(clean(CONFIGS["S"])).to_model_spec().order] == [0, 0, 0]


@pytest.mark.parametrize("edit, word", [
    (lambda d: d["layers"][0].update(type="attention"), "parallel"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(heads=5), "multiple"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(dim=0), "positive"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(vdim=300), "256"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(scale=0.0), "scale"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(bias_max=0), "bias_max"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("bias_max"), "bias_max"),
    (lambda d: d["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(tau=0.0), "tau"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(dim=257), "256"),
    (lambda d: d["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda d: d["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "dense"),
    (lambda d: d["loop"].update(stop=9), "stretch"),
    (lambda d: d["loop"].update(times=0), "at least once"),
    (lambda d: d.update(streams=0), "streams"),
    (lambda d: d.pop("streams"), "streams"),
    (lambda d: d["norm"].update(eps=0.0), "eps"),
])
def test_what_it_refuses(edit, word):
    d = copy.deepcopy(clean(CONFIGS["P"]))
    edit(d)
    with pytest.raises(ConfigError) as err:
        config_from_dict(d)
    assert word in str(err.value)


@pytest.mark.parametrize("rows, reach", [(8, 40), (16, 128), (10, 160), (2, 9), (4, 25), (32, 333), (6, 100.5)])
def test_the_row_that_a_distance_reads(rows, reach):
    """The engine's list against the plain rule for every distance well past the reach; whole numbers against the logarithms,
    which agree wherever the logarithms are not within rounding of an edge."""
    table = distance_buckets(rows, reach)
    h = rows // 2
    assert table[:h] == list(range(h)) and table[-1] == rows - 1 and (len(table) < 2 or table[-2] < rows - 1)
    for n in range(3 * int(reach)):
        want = plain.distance_bucket(n, rows, reach)
        assert table[min(n, len(table) - 1)] == want
        if n >= h:
            x = math.log(n / h) / math.log(reach / h) * (rows - h)
            if abs(x - round(x)) > 1e-9:
                assert want == min(rows - 1, h + math.floor(x))


def test_edges_of_the_distance_rows_that_logarithms_miss():
    """Sixteen rows up to 128: the edges 8 * 2^(k / 2) of even k are whole numbers; ten rows up to 160: 5 * 2^k."""
    assert [distance_buckets(16, 128)[n] for n in (15, 16, 31, 32, 63, 64)] == [9, 10, 11, 12, 13, 14]
    assert [distance_buckets(10, 160)[n] for n in (9, 10, 19, 20, 39, 40, 79, 80)] == [5, 6, 6, 7, 7, 8, 8, 9]


def test_a_bias_that_cannot_be_is_refused():
    for rows, reach in ((1, 40), (16, 8), (16, 5)):
        with pytest.raises(ConfigError):
            distance_buckets(rows, reach)


def test_the_rules_on_small_numbers():
    """Each plain rule on a case worked out by hand."""
    assert plain.query_temperature(8, 0.5, 4).tolist() == pytest.approx([1.0, 1.0, 1.0, 1 + 0.5 * math.log(2)] + [1 + 0.5 * math.log(2)] * 3 + [1 + 0.5 * math.log(3)])
    assert torch.allclose(plain.decay(torch.zeros(1, dtype=torch.float64), 2.0), torch.tensor([0.5 ** 0.5], dtype=torch.float64))
    s = plain.sinusoid(3, 4)
    assert s[2].tolist() == pytest.approx([math.sin(2), math.cos(2), math.sin(0.02), math.cos(0.02)])
    w = {"h.in": torch.tensor([1.0, 2.0]), "h.out": torch.tensor([3.0, 5.0]), "h.mix": torch.tensor([[1.0, 10.0], [100.0, 1000.0]])}
    x = torch.tensor([[[1.0]], [[7.0]]], dtype=torch.float64)
    out = plain.hyper_step(w, "h.", x, lambda u: 2.0 * u)          # u = 15, y = 30
    assert out.flatten().tolist() == [1 + 700 + 90, 10 + 7000 + 150]
    ok = torch.ones(1, 1, 1, dtype=torch.bool)
    assert float(plain.softmax_with_sink(torch.zeros(1, 1, 1, dtype=torch.float64), ok, torch.zeros(1, dtype=torch.float64))) == 0.5
    assert plain.run_order({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3, 4]


def test_random_tensors_of_the_design():
    from quantinfer_b200.weights import random_tensors

    needs = tensor_needs_of_spec(config_from_dict(clean(CONFIGS["R"])).to_model_spec())
    t = random_tensors(needs, 3)
    mix = t["l0.hc1.mix"]
    assert mix.shape == (4, 4) and float((mix - torch.eye(4)).abs().max()) <= 0.1 and t["l0.mix.left.rel"].shape[1] == 2


def test_the_comparison_of_the_bench_holds_equal_weights():
    """`bench.py --compare siditar`: both stacks are valid configurations of their designs and hold the same weights to 3 %."""
    import bench

    for size in bench.SIDITAR_SIZES:
        new, old = bench.siditar_entries(size)
        a, b = (bench.model_arithmetic(c, c.to_model_spec()) for c in (config_from_dict(new["config"]), config_from_dict(old["config"])))
        assert abs(a["weight_bytes"] / b["weight_bytes"] - 1.0) < 0.03
        needs = tensor_needs_of_spec(config_from_dict(new["config"]).to_model_spec())
        stored = sum(math.prod(16 if d is None else d for d in n.shape) for k, n in needs.items()
                     if len(n.shape) == 2 and ".rel" not in k and ".hc" not in k and k != "embed")
        assert abs(2 * stored / a["weight_bytes"] - 1.0) < 0.01       # the count of the arithmetic is the count of the tensors
