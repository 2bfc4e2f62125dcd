"""Host-side tests of the Naburax design: configuration, the model description (declared tensors, caches, state of the
embedding), the books of a window that keeps its first tokens, and facts of the plain implementation that the GPU tests lean on."""
import copy
import math

import pytest
import torch

from tests.naburax_cases import CASES, case, write_folder
from tests.plain import naburax_plain as plain

F64 = torch.float64


def _model(raw, dtype=torch.float32):
    from microllm_rocm_b200.config import get_architecture
    from microllm_rocm_b200.config.naburax import NaburaxConfig
    from microllm_rocm_b200.parts.base import Runtime
    from microllm_rocm_b200.parts.build import build_model
    arch = get_architecture("Naburax")
    return build_model(arch.build_spec(NaburaxConfig.from_dict(raw)), Runtime(torch.device("cpu"), dtype))


@pytest.mark.parametrize("key", sorted(CASES))
def test_declared_tensors_are_the_checkpoints(key):
    raw, weights = case(key)
    model = _model(raw)
    expected = model.expected_tensors()
    assert set(expected) == set(weights)
    for name, spec in expected.items():
        assert tuple(spec.shape) == tuple(weights[name].shape), name
    # a layer without a feed-forward may still carry the norm that would stand behind one
    assert set(model.tolerated_extra_tensors()) == {f"l{i}.norm2" for i, l in enumerate(raw["layers"]) if l["mlp"] is None}


def test_padded_and_fused_tensors_cover_their_pieces():
    """The projections' rows are padded to a multiple of 8; every checkpoint tensor has a place in one device tensor."""
    model = _model(case("b")[0])
    destinations, pieces = model.placements()
    expected = model.expected_tensors()
    assert set(pieces) == set(expected)
    for name, (dest, row) in pieces.items():
        assert row + expected[name].shape[0] <= destinations[dest].shape[0], name
    right = destinations["l1.mix.right.in_proj.padded"].shape[0]
    assert right % 8 == 0 and right >= expected["l1.mix.right.in"].shape[0] and expected["l1.mix.right.in"].shape[0] % 8
    assert destinations["l0.mix.in_proj.weight"].shape[0] % 8 == 0


def test_configuration_round_trip_and_choice_by_name(tmp_path):
    from microllm_rocm_b200.config.naburax import NaburaxConfig
    from microllm_rocm_b200.config.registry import load_config
    for key in CASES:
        raw, weights = case(key)
        arch, cfg = load_config(write_folder(str(tmp_path / key), raw, weights))
        assert arch.name == "Naburax"
        again = NaburaxConfig.from_dict(cfg.to_dict())
        assert again == cfg and hash(again) == hash(cfg)
        assert (cfg.bigram is None) == ("bigram" not in raw["embedding"])
        assert (cfg.embedding_scale, cfg.logit_scale) == (raw["embedding"]["scale"], raw["logit_scale"])
    bare = case("b")[0]
    del bare["embedding"], bare["logit_scale"]
    cfg = NaburaxConfig.from_dict(bare)
    assert (cfg.embedding_scale, cfg.logit_scale, cfg.bigram) == (1.0, 1.0, None)


def test_presets_build():
    from microllm_rocm_b200.config import find_preset
    for name in ("naburax-tiny", "naburax-small", "naburax-3b-layers"):
        arch, cfg = find_preset(name)
        assert arch.name == "Naburax" and len(arch.build_spec(cfg).layers) == len(cfg.layers)


def test_refusals():
    from microllm_rocm_b200.config.naburax import NaburaxConfig
    from microllm_rocm_b200.config.qwen2 import ConfigError
    raw = case("a")[0]

    def broken(change):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ConfigError):
            NaburaxConfig.from_dict(bad)
    mixer = lambda r, i: r["layers"][i]["mixer"]
    broken(lambda r: r.pop("norm"))
    broken(lambda r: r["layers"][0].__setitem__("type", "attention"))
    broken(lambda r: mixer(r, 0)["left"].__setitem__("kv_heads", 3))                     # 4 heads, 3 kv heads
    broken(lambda r: mixer(r, 0)["left"]["mask"].__setitem__("size", 0))
    broken(lambda r: mixer(r, 0)["left"]["mask"].__setitem__("keep_first", -1))
    broken(lambda r: mixer(r, 0)["right"].__setitem__("groups", 3))                      # 4 heads
    broken(lambda r: mixer(r, 0)["right"].__setitem__("norm_groups", 5))                 # 48 columns
    broken(lambda r: mixer(r, 0)["right"].pop("conv"))
    broken(lambda r: mixer(r, 0).pop("right_scale"))
    broken(lambda r: mixer(r, 1).pop("q_rank"))
    broken(lambda r: mixer(r, 1)["mask"].__setitem__("keep_first", 4))                   # only keys per head are kept
    broken(lambda r: mixer(r, 1)["rot"].__setitem__("dims", 10))                         # rot_dim is 8
    broken(lambda r: mixer(r, 1)["rot"]["scaling"].pop("slow"))
    broken(lambda r: r["layers"][0]["mlp"].__setitem__("kind", "dense"))
    broken(lambda r: r["layers"][0]["mlp"]["router"].__setitem__("top", 6))              # five experts
    broken(lambda r: r["embedding"]["bigram"].__setitem__("buckets", 0))
    broken(lambda r: r.__setitem__("logit_scale", "big"))


def test_caches_of_each_layer():
    from microllm_rocm_b200.parts.base import FixedStateNeed, PagedKVNeed, PagedRowsNeed
    entries = {n: e.need for n, e in _model(case("a")[0]).cache_entries.items()}
    assert set(entries) == {"embedding", "run0.left", "run0.right.state", "run0.right.conv", "run1", "run2"}
    kv = entries["run0.left"]
    assert isinstance(kv, PagedKVNeed) and (kv.head_dim, kv.value_dim, kv.window, kv.keep_first) == (16, 24, 20, 5)
    assert entries["run0.right.state"] == FixedStateNeed((4, 20, 12)) and entries["run0.right.conv"] == FixedStateNeed((2, 48 + 80))
    assert entries["run1"] == PagedRowsNeed(28, 33) and entries["run2"] == PagedRowsNeed(28, None)
    one_tap = {n: e.need for n, e in _model(case("b")[0]).cache_entries.items()}
    assert "run1.right.conv" not in one_tap and "embedding" not in one_tap                # one tap keeps nothing; no pair table, no state
    # bf16: unequal widths are stored with zeros to one width
    assert _model(case("a")[0], torch.bfloat16).cache_entries["run0.left"].need.head_dim == 32


def test_pages_of_kept_tokens_stay():
    """A window of 20 in front of which 37 tokens stay: their pages (three of 16) are never given back, those between them and the
    window are, and a request that ends gives back all."""
    from microllm_rocm_b200.cache.manager import RELEASED, CacheManager, group_key
    from microllm_rocm_b200.parts.base import PagedKVNeed
    need, plain_window = PagedKVNeed(1, 8, 20, keep_first=37), PagedKVNeed(1, 8, 20)
    assert group_key(need) != group_key(plain_window) and group_key(PagedKVNeed(1, 8, None, keep_first=37)) == "full"
    cache = CacheManager({"kept": need, "plain": plain_window}, page_size=16, num_pages=20, max_requests=2)
    assert cache.add("x")
    for n in range(1, 201):
        assert cache.reserve("x", n)
        cache.commit("x", n)
        kept, gone = cache.requests["x"].tables[group_key(need)], cache.requests["x"].tables[group_key(plain_window)]
        first_needed = n - 20 + 1                                        # the next query's window starts here
        for b, (page, other) in enumerate(zip(kept, gone)):
            dead = (b + 1) * 16 <= first_needed
            assert (other == RELEASED) == dead
            assert (page == RELEASED) == (dead and b >= 3)
        cache.check()
    cache.release("x")
    cache.check()
    assert all(g.pool.used_count == 0 for g in cache.groups.values())
    # with a promise of at most 8 tokens a step the pool holds every request's window and its kept blocks
    small = CacheManager({"kept": need}, page_size=16, num_pages=100, max_requests=3, max_step_tokens=8)
    group = small.groups[group_key(need)]
    assert group.pool.num_pages == 3 * (2 + 1 + 3)
    for r in "xyz":
        assert small.add(r)
    for n in range(8, 400, 8):
        for r in "xyz":
            assert small.reserve(r, n)
            small.commit(r, n)
    assert group.pool.peak_used <= group.pool.num_pages


# ------------------------------------------------------------------------------------------- the plain implementation by hand
def test_plain_visibility():
    assert plain.visible(3, None) == [0, 1, 2, 3]
    assert plain.visible(10, 3) == [8, 9, 10]
    assert plain.visible(10, 3, 2) == [0, 1, 8, 9, 10]
    assert plain.visible(4, 3, 4) == [0, 1, 2, 3, 4] and plain.visible(2, 1, 9) == [0, 1, 2]


def test_plain_attention_over_a_kept_token():
    # equal scores: the mean of the visible values
    q, k = torch.zeros(6, 1, 2, dtype=F64), torch.randn(6, 1, 2, dtype=F64)
    v = torch.arange(6, dtype=F64).view(6, 1, 1)
    o = plain.softmax_attention(q, k, v, 1.0, 2, 1)
    assert torch.allclose(o[:, 0, 0], torch.tensor([0.0, 0.5, 1.0, 5 / 3, 7 / 3, 3.0], dtype=F64))


def test_plain_convolution_and_state_by_hand():
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=F64)
    assert plain.causal_conv(u, torch.tensor([[3.0, 5.0]]), torch.tensor([0.5])).flatten().tolist() == [5.5, 13.5, 26.5]
    # one head: y_t = sum_j exp(-a sum_{j<i<=t} dt_i) dt_j (C_t . B_j) x_j + D x_t
    torch.manual_seed(0)
    T, H, P, G, N = 7, 4, 3, 2, 5
    x, B, C = torch.randn(T, H, P, dtype=F64), torch.randn(T, G, N, dtype=F64), torch.randn(T, G, N, dtype=F64)
    dt, a, D = torch.rand(T, H, dtype=F64), torch.randn(H, dtype=F64), torch.randn(H, dtype=F64)
    y = plain.selective_state(x, B, C, dt, a, D)
    for h in range(H):
        g = h // 2
        want = D[h] * x[6, h]
        for j in range(T):
            want = want + torch.exp(-torch.exp(a[h]) * dt[j + 1:, h].sum()) * dt[j, h] * (C[6, g] @ B[j, g]) * x[j, h]
        assert torch.allclose(y[6, h], want)


def test_plain_gate_comes_before_the_grouped_norm():
    raw, w = case("a", seed=3)
    m, p = raw["layers"][0]["mixer"]["right"], "l0.mix.right."
    h = torch.randn(5, raw["width"], dtype=F64)
    y = plain.right_mamba(m, w, p, h, 1e-5)
    # scaling one part of the gated row (through z, where silu is nearly linear) would leave it as it is, were it not for the others:
    # with three parts of 16 columns, each has a root mean square of one before the weight
    o = torch.linalg.lstsq(w[p + "o"].to(F64), y.T).solution.T / w[p + "norm"].to(F64)
    assert torch.allclose((o.view(5, 3, 16) ** 2).mean(-1), torch.ones(5, 3, dtype=F64), atol=1e-2)


def test_plain_rotation():
    x = torch.tensor([[[1.0, 0.0, 0.0, 1.0]]] * 3, dtype=F64)
    out = plain.rotate_pairs(x, [0.5, 0.25], 2.0)
    assert torch.allclose(out[2, 0], 2.0 * torch.tensor([math.cos(1.0), math.sin(1.0), -math.sin(0.5), math.cos(0.5)], dtype=F64))
    freq, magnitude = plain.rotation_table(8, 10000.0, None)
    assert freq == [10000.0 ** (-i / 4) for i in range(4)] and magnitude == 1.0
    # the product's table, made in float64 and stored in fp32
    from microllm_rocm_b200.parts.rotary import stretched_frequencies
    for scaling in ({"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}, {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}):
        for dims, base in ((8, 5000.0), (16, 1e4), (64, 2e5)):
            freq, magnitude = plain.rotation_table(dims, base, scaling)
            got, factor = stretched_frequencies(base, dims, scaling)
            assert torch.allclose(torch.from_numpy(got).double(), torch.tensor(freq, dtype=F64), rtol=1e-6) and abs(factor - magnitude) < 1e-12
            plain_freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
            assert freq != plain_freq and all(f <= g for f, g in zip(freq, plain_freq))


def test_plain_routing_by_hand():
    z = torch.tensor([[0.0, math.log(3.0), -50.0, math.log(9.0)]], dtype=F64)
    chosen, w = plain.route(z, 2)
    assert chosen.tolist() == [[3, 1]] and torch.allclose(w, torch.tensor([[0.9, 0.75]], dtype=F64))       # as they are: no sum of one
    assert plain.route(torch.zeros(1, 3, dtype=F64), 2)[0].tolist() == [[0, 1]]
    # the weight goes in: silu(w g) (w u), which no factor on the result makes up for
    mlp = {"router": {"experts": 1, "top": 1}, "expert": {"ff": 1}}
    weights = {"m.router": torch.zeros(1, 1), "m.e0.gate": torch.ones(1, 1), "m.e0.up": torch.ones(1, 1), "m.e0.down": torch.ones(1, 1)}
    y = plain.routed_ff(mlp, weights, "m.", torch.tensor([[4.0]], dtype=F64))
    assert abs(float(y) - 2.0 / (1 + math.exp(-2.0)) * 2.0) < 1e-12


def test_pair_rows_of_the_plain_embedding():
    assert plain.pair_rows([5, 9, 9, 0], 7, 3, 2) == [7, (5 * 3 + 9 * 2) % 7, (9 * 3 + 9 * 2) % 7, (9 * 3) % 7]
    assert plain.pair_rows([4], 11, 100, 100) == [11]


def test_mistakes_would_show_in_the_logits():
    """How far a mistake in a mechanism moves the logits of the sharp cases: each far beyond the GPU tests' tolerances."""
    from tests.helpers import random_tokens

    def moved(key, change_raw=None, change_weights=None, n=70, seed=11):
        raw, w = case(key, seed=seed, sharp=3.0)
        toks = random_tokens(n, raw["vocab"], 21)
        a = plain.forward(raw, w, toks)
        raw, w = copy.deepcopy(raw), dict(w)
        if change_raw:
            change_raw(raw)
        if change_weights:
            change_weights(w)
        b = plain.forward(raw, w, toks)
        return float((a - b)[n // 2:].abs().max() / a.abs().max())
    left = lambda r, i=0: r["layers"][i]["mixer"]["left"]["mask"]
    assert moved("a", lambda r: left(r).__setitem__("size", 21)) > 0.15                  # a window one token off
    assert moved("a", lambda r: left(r).__setitem__("size", 19)) > 0.15
    assert moved("a", lambda r: left(r).__setitem__("keep_first", 4)) > 0.15             # a kept token left out, or one too many
    assert moved("a", lambda r: left(r).__setitem__("keep_first", 6)) > 0.15
    assert moved("a", lambda r: r["layers"][1]["mixer"]["mask"].__setitem__("size", 32)) > 0.15
    assert moved("a", lambda r: r["layers"][1]["mixer"]["rot"].pop("scaling")) > 0.15
    assert moved("a", lambda r: r["embedding"]["bigram"].__setitem__("mul_prev", 14)) > 0.15
    assert moved("a", lambda r: r["embedding"].__setitem__("scale", 1.6)) > 0.15
    assert moved("a", None, lambda w: w.__setitem__("l0.mix.right.dt_bias", w["l0.mix.right.dt_bias"] + 0.1)) > 0.05
    assert moved("a", None, lambda w: w.__setitem__("l0.mix.right.conv.b", torch.zeros_like(w["l0.mix.right.conv.b"]))) > 0.15
    assert moved("a", None, lambda w: w.__setitem__("l0.mix.right.D", torch.zeros_like(w["l0.mix.right.D"]))) > 0.15
