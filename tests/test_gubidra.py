"""Host-side tests of the Gubidra design: configuration, the model description (declared tensors, run order, caches), the rows
of the distance bias, and facts of the plain implementation that the GPU tests lean on."""
import copy
import math

import pytest
import torch

from tests.gubidra_cases import CASES, case, complete, write_folder
from tests.helpers import random_tokens
from tests.plain import gubidra_plain as plain

F64 = torch.float64


def _model(key, dtype=torch.float32):
    from microllm_rocm_b200.config import get_architecture
    from microllm_rocm_b200.config.gubidra import GubidraConfig
    from microllm_rocm_b200.parts.base import Runtime
    from microllm_rocm_b200.parts.build import build_model
    arch = get_architecture("Gubidra")
    return build_model(arch.build_spec(GubidraConfig.from_dict(complete(*case(key)))), Runtime(torch.device("cpu"), dtype))


@pytest.mark.parametrize("key", sorted(CASES))
def test_declared_tensors_are_the_checkpoints(key):
    _, weights = case(key)
    expected = _model(key).expected_tensors()
    assert set(expected) == set(weights)
    for name, spec in expected.items():
        assert tuple(spec.shape) == tuple(weights[name].shape), name


def test_configuration_round_trip_and_sizes_from_the_weight_file(tmp_path):
    from microllm_rocm_b200.config.gubidra import GubidraConfig
    from microllm_rocm_b200.config.qwen2 import ConfigError
    from microllm_rocm_b200.config.registry import load_config
    for key in CASES:
        raw, weights = case(key)
        folder = write_folder(str(tmp_path / key), raw, weights)
        arch, cfg = load_config(folder)
        assert arch.name == "Gubidra"
        again = GubidraConfig.from_dict(cfg.to_dict())
        assert again == cfg and hash(again) == hash(cfg)
        assert [l["mixer"].get("bias_rows") for l in cfg.layers] == [l.get("_rows") for l in CASES[key]["layers"]]
    with pytest.raises(ConfigError):                        # config.json alone does not know the rows of the bias table
        GubidraConfig.from_dict(case("a")[0])


def test_presets_build():
    from microllm_rocm_b200.config import find_preset
    for name in ("gubidra-tiny", "gubidra-small", "gubidra-3b-layers"):
        arch, cfg = find_preset(name)
        spec = arch.build_spec(cfg)
        assert arch.name == "Gubidra" and len(spec.layers) == len(cfg.layers) and spec.streams == cfg.streams


def test_refusals():
    from microllm_rocm_b200.config.gubidra import GubidraConfig
    from microllm_rocm_b200.config.qwen2 import ConfigError
    raw = complete(*case("a"))

    def broken(change):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ConfigError):
            GubidraConfig.from_dict(bad)
    broken(lambda r: r.pop("streams"))
    broken(lambda r: r.__setitem__("streams", 0))
    broken(lambda r: r.__setitem__("streams", 17))
    broken(lambda r: r["norm"].__setitem__("eps", 0))
    broken(lambda r: r["layers"][0].__setitem__("type", "mamba"))
    broken(lambda r: r["layers"][0]["mixer"].__setitem__("decay", [0.5, 0.9]))            # three heads
    broken(lambda r: r["layers"][0]["mixer"]["rot"].__setitem__("dims", 18))              # more than a head has
    broken(lambda r: r["layers"][1]["mixer"].__setitem__("kv_heads", 3))                  # 4 heads
    broken(lambda r: r["layers"][1]["mixer"].__setitem__("bias_max", 5))                  # not beyond half of ten rows
    broken(lambda r: r["layers"][1]["mixer"]["mask"].__setitem__("size", 0))
    broken(lambda r: r["layers"][2]["mixer"].__setitem__("gate_cap", -1.0))
    broken(lambda r: r["layers"][2]["mlp"]["router"]["groups"].__setitem__("count", 4))   # six experts
    broken(lambda r: r["layers"][2]["mlp"]["router"].__setitem__("top", 5))               # four are open
    broken(lambda r: r["layers"][2]["mlp"].__setitem__("kind", "dense"))
    broken(lambda r: r["loop"].__setitem__("stop", 4))
    broken(lambda r: r["loop"].__setitem__("times", "2"))


def test_run_order_and_caches():
    from microllm_rocm_b200.parts.base import FixedStateNeed, PagedKVNeed
    model = _model("a")
    assert [r.layer for r in model.spec.order] == [0, 1, 0, 1, 2] == plain.run_order(case("a")[0])
    # every pass has a state or pages of its own; the matrix memory keeps a matrix, a vector and a maximum
    assert set(model.cache_entries) == {"run0.state", "run1", "run2.state", "run3", "run4.state", "run4.n", "run4.m"}
    need = model.cache_entries["run1"].need
    assert isinstance(need, PagedKVNeed) and (need.head_dim, need.value_dim, need.window) == (16, 24, 24)
    shapes = {n: model.cache_entries[n].need.shape for n in ("run0.state", "run4.state", "run4.n", "run4.m")}
    assert shapes == {"run0.state": (3, 16, 24), "run4.state": (2, 20, 12), "run4.n": (2, 20), "run4.m": (2,)}
    assert all(isinstance(model.cache_entries[n].need, FixedStateNeed) and model.cache_entries[n].need.dtype == torch.float32 for n in shapes)
    assert [r.layer for r in _model("c").spec.order] == [0, 1, 2, 3, 3, 3]
    assert [r.layer for r in _model("d").spec.order] == [0, 1, 2, 3, 4]


def test_streams_and_blocks_must_agree():
    from dataclasses import replace
    from microllm_rocm_b200.parts.base import Runtime
    from microllm_rocm_b200.parts.build import build_model
    spec = _model("a").spec
    with pytest.raises(ValueError):
        build_model(replace(spec, streams=None), Runtime(torch.device("cpu"), torch.float32))


@pytest.mark.parametrize("buckets,far", [(10, 60), (7, 21.5), (2, 9), (32, 128), (16, 300), (9, 40), (3, 2.5), (32, 16.5), (64, 1000)])
def test_rows_of_the_distance_bias(buckets, far):
    from microllm_rocm_b200.parts.attention import distance_rows
    rows = distance_rows(buckets, far)
    assert rows == [plain.bucket(n, buckets, far) for n in range(len(rows))]
    assert rows[-1] == buckets - 1 and rows.count(buckets - 1) == 1           # it ends at the first distance of the last row
    assert all(plain.bucket(n, buckets, far) == buckets - 1 for n in range(len(rows), len(rows) + 2000, 7))
    assert rows[:buckets // 2] == list(range(buckets // 2)) and rows == sorted(rows)


def test_distance_table_repeats_its_ends():
    from microllm_rocm_b200.kernels.ops import DISTANCE_PAD, DistanceBias
    values = torch.arange(10.0).view(2, 5)
    bias = DistanceBias(values)
    assert bias.last == 4 and bias.table.shape == (2, 5 + 2 * DISTANCE_PAD)
    for h in range(2):
        row = bias.table[h]
        assert torch.equal(row[DISTANCE_PAD:DISTANCE_PAD + 5], values[h])
        assert bool((row[:DISTANCE_PAD] == values[h, 0]).all()) and bool((row[DISTANCE_PAD + 5:] == values[h, 4]).all())


def test_recorded_runs_are_only_issued_again_where_addresses_stand_for_one_another():
    from microllm_rocm_b200.parts.build import _one_to_one
    assert _one_to_one([1, 2, 1, 0], [5, 6, 5, 9])
    assert not _one_to_one([1, 2, 1], [5, 6, 7])             # one recorded tensor would have to become two


def test_plain_routing_by_hand():
    logit = lambda s: math.log(s / (1 - s))
    z = torch.tensor([[logit(s) for s in (0.9, 0.1, 0.6, 0.55, 0.3, 0.5)]], dtype=F64)
    # groups (0.9, 0.1), (0.6, 0.55), (0.3, 0.5): sums 1.0, 1.15, 0.8.  The best single expert is in the second-best group.
    chosen, w = plain.route(z, 2, 3, 1, 3.0)
    assert chosen.tolist() == [[2, 3]] and torch.allclose(w, torch.tensor([[0.6, 0.55]], dtype=F64) / 1.15 * 3.0)
    chosen, w = plain.route(z, 3, 3, 2, 1.0)
    assert chosen.tolist() == [[0, 2, 3]] and torch.allclose(w, torch.tensor([[0.9, 0.6, 0.55]], dtype=F64) / 2.05)
    assert plain.route(z, 1, 1, 1, 1.0)[0].tolist() == [[0]]                  # one group: no limit
    assert plain.route(z, 2, 6, 2, 1.0)[0].tolist() == [[0, 2]]               # groups of one expert: its own score


def test_plain_bias_window_and_bucket_edges():
    q = torch.zeros(6, 1, 2, dtype=F64)
    v = torch.eye(6, dtype=F64)[:, None, :]
    rel = torch.tensor([[0.3], [-1.0], [2.0], [0.5]], dtype=F64)              # near rows 0, 1; rows 2, 3 beyond
    o = plain.biased_attention(q, q, v, 1.0, rel, 8, None)
    rows = [plain.bucket(n, 4, 8) for n in range(6)]
    assert rows == [0, 1, 2, 2, 3, 3]
    want = torch.softmax(torch.tensor([rel[rows[5 - j], 0] for j in range(6)]), 0)
    assert torch.allclose(o[5, 0], want)
    o = plain.biased_attention(q, q, v, 7.0, rel, 8, 3)                       # three keys; the scale leaves the bias alone
    assert torch.allclose(o[5, 0], torch.cat([torch.zeros(3, dtype=F64), torch.softmax(torch.tensor([2.0, -1.0, 0.3], dtype=F64), 0)]))


def test_plain_matrix_memory_does_not_depend_on_its_running_maximum():
    """With the maximum's exponentials undone: S_t = sum_j e^(i_j + sum_(l>j) f_l) k_j v_j^T, o = S^T q / max(|n . q|, 1)."""
    torch.manual_seed(0)
    q, k, v = torch.randn(7, 1, 3, dtype=F64), torch.randn(7, 1, 3, dtype=F64), torch.randn(7, 1, 4, dtype=F64)
    i, f = torch.randn(7, 1, dtype=F64) * 2, torch.nn.functional.logsigmoid(torch.randn(7, 1, dtype=F64))
    got = plain.matrix_memory(q, k, v, i, f)
    for t in range(7):
        e = torch.stack([torch.exp(i[j, 0] + f[j + 1:t + 1, 0].sum()) for j in range(t + 1)])
        s = e * (k[:t + 1, 0] @ q[t, 0])
        # max(|n q| e^-m, e^-m) = e^-m max(|n q|, 1), and the 1e-6 is tiny beside it
        assert torch.allclose(got[t, 0], (s[:, None] * v[:t + 1, 0]).sum(0) / max(float(s.sum().abs()), 1.0), rtol=1e-4)


def test_plain_retention_by_hand():
    torch.manual_seed(1)
    q, k, v = (torch.randn(9, 2, 3, dtype=F64) for _ in range(3))
    whole = plain.retain(q, k, v, [0.5, 1.0])
    for h, d in enumerate((0.5, 1.0)):
        want = sum(d ** (8 - j) * float(q[8, h] @ k[j, h]) * v[j, h] for j in range(9))
        assert torch.allclose(whole[8, h], want)
    x = torch.randn(4, 1, 6, dtype=F64)
    y = plain.rotate_halves(x, 4, 100.0)
    a = 3 * 100.0 ** -0.5                                                     # pair 1 of position 3: elements 1 and 3
    assert torch.allclose(y[3, 0, 1], x[3, 0, 1] * math.cos(a) - x[3, 0, 3] * math.sin(a))
    assert torch.allclose(y[3, 0, 3], x[3, 0, 3] * math.cos(a) + x[3, 0, 1] * math.sin(a))
    assert torch.equal(y[..., 4:], x[..., 4:])


def test_plain_streams_by_hand():
    x = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)                          # two streams, one token, one column
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64)                   # from, to
    assert plain.read_streams(x, torch.tensor([2.0, -1.0], dtype=F64)).item() == -8.0
    assert plain.write_streams(x, torch.tensor([[100.0]], dtype=F64), mix, torch.tensor([1.0, 0.5], dtype=F64)).flatten().tolist() == \
        [1 + 30 + 100, 2 + 40 + 50]


@pytest.mark.parametrize("key", ["a", "c"])
def test_a_wrong_window_bias_pass_or_stream_would_show(key):
    """What a comparison of logits sees when one mechanism is taken the wrong way: the plain implementation with that
    mistake lands hundreds of the fp32 tests' tolerances away."""
    raw, weights = case(key, seed=11, sharp=3.0, bias=3.0)
    tokens = random_tokens(200, raw["vocab"], 3)
    ref = plain.forward(raw, weights, tokens)
    distance = lambda r, w: float((plain.forward(r, w, tokens) - ref).abs().amax() / ref.abs().max())
    wrong = copy.deepcopy(raw)
    for layer in wrong["layers"]:
        if layer["type"] == "attention":
            layer["mixer"]["mask"]["size"] -= 1                                 # a window that is one key short
    assert distance(wrong, weights) > 0.01
    wrong = copy.deepcopy(raw)
    wrong["loop"]["times"] += 1
    assert distance(wrong, weights) > 0.01
    for change in (lambda n, t: t.T.contiguous() if n.endswith(".mix") and ".hc" in n else t,             # from and to exchanged
                   lambda n, t: torch.roll(t, 1, 0) if n.endswith("mix.rel") else t,                      # a bias one row off
                   lambda n, t: t - 3.0 if n.endswith("f.b") else t):                                     # other forget gates
        assert distance(raw, {n: change(n, t) for n, t in weights.items()}) > 0.01
