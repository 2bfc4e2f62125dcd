"""The Naburax decoder on the GPU against its plain float64 restatement: each mechanism alone, then whole models cut in
every way (whole prompts, a tail decoded token by token, portions down to two tokens, mixed batches over a pool so small
that pages and state slots are used again), in true fp32 and in bf16, and greedy generation through the scheduler."""
import math
from types import SimpleNamespace

import pytest
import torch

from tests.helpers import collect, random_tokens, steps_mixed, steps_portions, steps_prefill_then_decode, steps_whole
from tests.naburax_cases import CASES, case, write_folder
from tests.plain import naburax_plain as plain

pytestmark = pytest.mark.gpu

FP32_TOL = 3e-5          # of the largest |logit|
BF16_TOL = 0.05          # of the largest |logit|
DEV = "cuda:0"
LENGTHS = {"a": [1, 2, 37, 130], "b": [5, 64, 99], "c": [3, 50, 290], "d": [17, 80]}
F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for key in CASES:
        raw, weights = case(key)
        out[key] = (write_folder(str(tmp_path_factory.mktemp("naburax_" + key)), raw, weights), raw, weights)
    return out


def engine_for(folder, dtype, max_tokens=1024, page_size=16, max_requests=4, **more):
    from microllm_rocm_b200.engine.loading import load_engine
    return load_engine(folder, dtype=dtype, page_size=page_size, max_tokens=max_tokens, max_requests=max_requests, **more)


_plain = {}


def plain_logits(raw, weights, tokens):
    k = (id(weights), tuple(tokens))
    if k not in _plain:
        _plain[k] = (weights, plain.forward(raw, weights, list(tokens)).float())     # (the weights stay alive: their id is the key)
    return _plain[k][1]


def compare(got, key, raw, weights, requests, dtype, share=0.15, fp32_tol=FP32_TOL, median=0.4):
    """fp32: every position within the tolerance.  bf16 rounds the router's input: where two scores are a rounding error apart the
    choice flips, that position lands far off, and the recurrence and the attention carry a little of it to later positions of
    the request.  So bf16 is held, over all positions of a case, to a small median error and to at most `share` of them over the
    tolerance."""
    errs = []
    for rid, toks in requests.items():
        ref = plain_logits(raw, weights, toks)
        rows = torch.stack([got[(rid, p)] for p in range(len(toks))])
        assert torch.isfinite(rows).all(), f"case {key} request {rid}: logits that are not finite"
        err = (rows - ref).abs().amax(dim=1) / ref.abs().max()
        if dtype == "float32" and bool((err > fp32_tol).any()):
            pos = int((err > fp32_tol).nonzero()[0])
            raise AssertionError(f"case {key} request {rid}: position {pos} of {len(toks)} is over the tolerance {fp32_tol} "
                                 f"(error {float(err[pos]):.3e} of the largest |logit|)")
        errs.append(err)
    err = torch.cat(errs)
    over = int((err > BF16_TOL).sum())
    print(f"[naburax parity] case {key} {dtype}: median error {float(err.median()):.3e}, worst {float(err.max()):.3e} of the largest |logit|, {over} over")
    if dtype != "float32":
        assert over <= max(2, int(share * err.numel())) and float(err.median()) <= median * BF16_TOL, \
            f"case {key}: {over} of {err.numel()} positions over the tolerance {BF16_TOL}, median error {float(err.median()):.3e}"


def requests_for(raw, lengths, seed=0):
    return {f"r{i}": random_tokens(n, raw["vocab"], seed + 100 * i + n) for i, n in enumerate(lengths)}


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def step_of(lengths, pos0, slots, tokens=None):
    """The per-sequence arrays a kernel sees of a step whose sequences bring `lengths` tokens from positions `pos0`."""
    starts = [0]
    for n in lengths:
        starts.append(starts[-1] + n)
    return SimpleNamespace(
        seq_starts=i32(starts), seq_pos0=i32(pos0), num_seqs=len(lengths), error_flag=torch.zeros(1, dtype=torch.int32, device=DEV),
        token_seq=i32([a for a, n in enumerate(lengths) for _ in range(n)]), token_ids=i32(tokens if tokens is not None else [0] * starts[-1]),
        positions=i32([p + i for p, n in zip(pos0, lengths) for i in range(n)])), i32(slots)


# ------------------------------------------------------------------------------------------- mechanisms alone
def test_scaled_token_row_plus_pair_row_in_one_pass():
    from microllm_rocm_b200.kernels import ops
    torch.manual_seed(2)
    buckets, a, b, W = 53, 40009, 7919, 40
    for dt in (torch.float32, torch.bfloat16):
        table, token_table = torch.randn(buckets + 1, W, device=DEV).to(dt), torch.randn(60000, W, device=DEV).to(dt)
        toks = random_tokens(9, 60000, 1)
        state = torch.full((2, 1), 123456, dtype=torch.int32, device=DEV)
        want = token_table.double()[torch.tensor(toks)] * 2.75 + table.double()[torch.tensor(plain.pair_rows(toks, buckets, a, b))]
        at = 0
        for n in (4, 1, 4):
            ctx, slots = step_of([n], [at], [1], toks[at:at + n])
            x = torch.full((n, W), float("nan"), device=DEV)
            ops.bigram_add(x, table, ctx, state, slots, buckets, a % buckets, b % buckets, token_table=token_table, scale=2.75)
            assert torch.allclose(x.double(), want[at:at + n], atol=1e-5)
            at += n
        assert state[:, 0].tolist() == [123456, toks[-1]]


@pytest.mark.parametrize("width", [40, 256, 1000, 4100])
def test_normed_result_added_with_a_copy_of_the_stream(width):
    """x += norm(weighted terms), terms as partial results, and the copy of the new stream in bf16."""
    from microllm_rocm_b200.kernels import ops
    torch.manual_seed(3)
    for terms in ([(1.0, torch.randn(3, 5, width, device=DEV))], [(0.8, torch.randn(5, width, device=DEV)), (-1.3, torch.randn(2, 5, width, device=DEV))]):
        x, w = torch.randn(5, width, device=DEV), 1 + 0.2 * torch.randn(width, device=DEV)
        d = sum(s * (t.double().sum(0) if t.dim() == 3 else t.double()) for s, t in terms)
        want = x.double() + plain.rms_norm(d, w.double(), 1e-3)
        for dt in (None, torch.bfloat16, torch.float32):
            y = x.clone()
            copy = None if dt is None else torch.full((5, width), float("nan"), dtype=dt, device=DEV)
            ops.normed_add_rmsnorm(y, terms, w, 1e-3, out=copy)
            assert torch.allclose(y.double(), want, atol=2e-5)
            if copy is not None:
                assert torch.equal(copy, y.to(dt))


def test_norm_factor_is_taken_into_the_weight():
    from microllm_rocm_b200.parts.base import Runtime
    from microllm_rocm_b200.parts.norm import RMSNorm
    norm = RMSNorm(dict(size=24, eps=1e-4, scale=0.3), Runtime(torch.device(DEV), torch.float32))
    w, x = torch.rand(24, device=DEV) + 0.5, torch.randn(6, 24, device=DEV)
    norm.bind({"weight": w})
    out = torch.empty_like(x)
    norm.forward(x, out)
    assert torch.allclose(out.double(), plain.rms_norm(x.double(), w.double(), 1e-4) * 0.3, atol=1e-6)


# ---- a window that keeps the first tokens
def spiky(n, nh, nkv, d, window, keep, seed):
    """Queries, keys and values of n tokens, q and k so that for every query some one key stands out: in turn the last kept one,
    the first one behind those, the window's first, the one just outside it, the query's own, the first of all, and one in the
    middle of the gap (those that the query may not see must not show)."""
    g = torch.Generator().manual_seed(seed)
    k, v = torch.randn(n, nkv, d, generator=g), torch.randn(n, nkv, d, generator=g)
    q = torch.randn(n, nh, d, generator=g) * 0.3
    for i in range(n):
        places = [keep - 1, keep, i - window + 1, i - window, i, 0, (keep + i - window) // 2]
        j = places[i % len(places)]
        if 0 <= j <= i:
            for h in range(nh):
                q[i, h] = k[j, h // (nh // nkv)] * (4.0 / d ** 0.5)
    return q, k, v


@pytest.mark.parametrize("window, keep", [(20, 5), (3, 40), (33, 16), (16, 17), (1, 1), (50, 0), (64, 64)])
@pytest.mark.parametrize("page_size", [8, 16])
def test_kept_tokens_on_the_kernel_of_two_widths(window, keep, page_size):
    """fp32, over scattered pages whose blocks between the kept tokens and the window are gone from the table; a prompt in one
    step and as decoded tokens, bit for bit the same."""
    from microllm_rocm_b200.kernels import attention_kv
    n, nh, nkv, dk = 150, 4, 2, 24
    q, k, v = spiky(n, nh, nkv, dk, window, keep, 5)
    want = plain.softmax_attention(q.double(), k.double(), v.double(), 1.0, window, keep)
    blocks = -(-n // page_size)
    order = torch.randperm(blocks + 2, generator=torch.Generator().manual_seed(1))[:blocks]
    pages = torch.full((blocks + 2, nkv * page_size * 2 * dk), float("nan"))
    for t in range(n):
        page, slot = pages[order[t // page_size]], t % page_size
        page[:nkv * page_size * dk].view(nkv, page_size, dk)[:, slot] = k[t]
        page[nkv * page_size * dk:].view(nkv, page_size, dk)[:, slot] = v[t]
    pages = pages.to(DEV)
    qd = q.reshape(n, nh * dk).contiguous().to(DEV)

    def run(first, count, drop):
        table = order.to(torch.int32).clone().view(1, -1)
        if drop:                                          # what the cache manager has given back before this step
            for b in range(-(-keep // page_size), max(0, first - window + 1) // page_size):
                table[0, b] = -1
        out = torch.full((count, nh * dk), float("nan"), device=DEV)
        flag = torch.zeros(1, dtype=torch.int32, device=DEV)
        attention_kv.paged_attention_kv(qd[first:first + count].contiguous(), pages, out, i32(list(range(first, first + count))), i32([0] * count),
                                        table.to(DEV), page_size, nh, nkv, dk, dk, 1.0, window, None, 0, flag, keep_first=keep)
        assert int(flag.item()) == 0
        return out
    whole = run(0, n, False)
    assert float((whole.double().cpu().view(n, nh, dk) - want).abs().max()) < 1e-5
    for first, count in ((0, 1), (1, 2), (keep, 1), (window, 3), (60, 7), (97, 2), (111, 39), (n - 1, 1)):
        assert torch.equal(run(first, count, True), whole[first:first + count]), (first, count)


def one_width_step(pages, table, lens, q_list, news, nh, nkv, d, scale, window, keep):
    """One step on the attention kernels of one width: sequence s brings news[s] queries at its last positions."""
    from microllm_rocm_b200.kernels import attention
    from microllm_rocm_b200.parts.base import StepContext
    pos0 = [l - n for l, n in zip(lens, news)]
    starts = [0]
    for n in news:
        starts.append(starts[-1] + n)
    q = torch.cat([x.reshape(x.shape[0], nh * d) for x in q_list]).contiguous()
    positions = torch.cat([torch.arange(p, p + n, dtype=torch.int32) for p, n in zip(pos0, news)]).to(DEV)
    token_seq = torch.cat([torch.full((n,), s, dtype=torch.int32) for s, n in enumerate(news)]).to(DEV)
    flag = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full(q.shape, float("nan"), dtype=torch.bfloat16, device=DEV)
    ctx = StepContext(num_tokens=q.shape[0], num_seqs=len(news), token_ids=positions, positions=positions, token_seq=token_seq,
                      seq_starts=i32(starts), seq_pos0=i32(pos0), seq_lens=i32(lens), block_tables={}, state_slots=None,
                      logit_rows=None, error_flag=flag, seq_starts_host=starts, seq_pos0_host=pos0,
                      max_new_tokens=max(news), max_seq_len=max(lens))
    attention.paged_attention(q, pages, out, ctx, table, nh, nkv, d, scale, window, keep_first=keep)
    torch.cuda.synchronize()
    assert int(flag.item()) == 0
    return out.float().reshape(-1, nh, d)


@pytest.mark.parametrize("d, page, nh, nkv", [(64, 16, 4, 2), (128, 64, 6, 1), (128, 16, 16, 1), (32, 16, 4, 2), (256, 16, 4, 2)])
@pytest.mark.parametrize("window, keep", [(130, 37), (300, 128), (48, 200), (17, 1), (128, 129), (100, 0)])
def test_kept_tokens_on_the_kernels_of_one_width(d, page, nh, nkv, window, keep):
    """bf16, the tensor-core kernels (prompt portions, every decode form, decoded tokens beside portions) against the formula over
    the same bf16 keys and values.  The pages that nobody reads any more are gone from the tables, and what stands in the pool's
    other pages is not a number."""
    from microllm_rocm_b200.kernels import attention
    n = 700
    q, k, v = spiky(n, nh, nkv, d, window, keep, d + nh)
    q, k, v = q.bfloat16(), k.bfloat16(), v.bfloat16()
    want = plain.softmax_attention(q.double(), k.double(), v.double(), 1.0, window, keep)
    blocks = -(-n // page)
    order = torch.randperm(blocks + 3, generator=torch.Generator().manual_seed(d))[:blocks]
    pages = torch.full((blocks + 3, 2, nkv, page, d), float("nan")).bfloat16()
    filled = torch.cat([k, torch.full((blocks * page - n, nkv, d), float("nan")).bfloat16()])
    pages[order, 0] = filled.view(blocks, page, nkv, d).transpose(1, 2)
    filled = torch.cat([v, torch.full((blocks * page - n, nkv, d), float("nan")).bfloat16()])
    pages[order, 1] = filled.view(blocks, page, nkv, d).transpose(1, 2)
    pages, q = pages.to(DEV), q.to(DEV)

    def table_for(*firsts):
        rows = []
        for first in firsts:                              # the first new position of each sequence
            row = order.to(torch.int32).clone()
            row[-(-keep // page):max(-(-keep // page), max(0, first - window + 1) // page)] = -1
            rows.append(row)
        return torch.stack(rows).contiguous().to(DEV)

    def check(out, rows, what):
        ref = want[rows]
        err = (out.double().cpu() - ref).abs().amax(-1) / ref.abs().amax(-1).clamp_min(0.05)
        assert torch.isfinite(out).all() and float(err.max()) < 0.04, (what, float(err.max()), int(err.amax(-1).argmax()))

    def step(lens, starts, what):
        outs = one_width_step(pages, table_for(*starts), lens, [q[s:l] for s, l in zip(starts, lens)], [l - s for s, l in zip(starts, lens)],
                              nh, nkv, d, 1.0, window, keep)
        at = 0
        for s, l in zip(starts, lens):
            check(outs[at:at + l - s], slice(s, l), f"{what}: {s}..{l}")
            at += l - s
    step([n], [0], "whole prompt")
    step([n], [301], "portion")
    step([n], [n - 2], "portion of two")
    step([300], [255], "portion")
    for pos in (0, 1, keep, window, keep + window, 127, 128, 511, n - 1):
        step([pos + 1], [pos], "decoded token")
    step([1, 130, 500, n], [0, 129, 499, n - 1], "batched decode")
    step([400, n], [250, n - 1], "portion beside a decoded token")
    if d == 128 and nh // nkv <= 8:                       # the kernel that brings keys through a ring
        attention.DECODE_RING = True
        try:
            step([1, 130, 500, n], [0, 129, 499, n - 1], "batched decode through the ring")
            step([400, n], [250, n - 1], "portion beside a decoded token, through the ring")
        finally:
            attention.DECODE_RING = None


# ---- the selective state space
@pytest.mark.parametrize("H, P, N, G, taps, norm_groups", [(4, 12, 20, 2, 3, 3), (1, 10, 12, 1, 1, 1), (6, 7, 9, 3, 2, 6), (4, 64, 64, 2, 4, 2),
                                                            (2, 20, 136, 1, 6, 4), (8, 136, 40, 8, 5, 1)])
def test_state_space_kernels_over_steps_with_slots_used_again(H, P, N, G, taps, norm_groups):
    """Convolution with bias, step sizes and decays, recurrence, skip, gate and grouped norm, each against the plain formula,
    over three steps of unequal portions; the projection comes as two partial results; a sequence starts in the slot another one
    left; slots hold a pattern at first."""
    from microllm_rocm_b200.kernels import recurrent, state_space
    torch.manual_seed(7)
    inner, bc = H * P, G * N
    C = inner + 2 * bc
    width = inner + C + H + 3
    w, bias = (torch.randn(C, taps) * 0.6).float(), torch.randn(C) * 0.3
    dt_bias, a_log, D, weight = torch.randn(H) - 1, torch.randn(H) * 0.5 - 1, 1 + torch.randn(H), 1 + 0.2 * torch.randn(inner)
    seqs = {0: torch.randn(60, width), 1: torch.randn(7, width), 2: torch.randn(44, width)}
    want = {}
    for s, proj in seqs.items():
        z, u, dt, _ = torch.split(proj.double(), [inner, C, H, 3], -1)
        u = plain.silu(plain.causal_conv(u, w, bias))
        x, B, c = torch.split(u, [inner, bc, bc], -1)
        T = proj.shape[0]
        dt = torch.log1p(torch.exp(dt + dt_bias.double()))
        y = plain.selective_state(x.view(T, H, P), B.view(T, G, N), c.view(T, G, N), dt, a_log, D).reshape(T, inner)
        want[s] = (u, dt, plain.rms_norm((y * plain.silu(z)).view(T, norm_groups, -1), None, 1e-4).reshape(T, inner) * weight.double())
    state = torch.full((4, H, N, P), 77.0, device=DEV)
    conv_state = torch.full((4, taps - 1, C), -55.0, device=DEV) if taps > 1 else None
    dev = lambda t: t.contiguous().to(DEV)
    w, bias, dt_bias, a_log, D, weight = (dev(t) for t in (w, bias, dt_bias, a_log, D, weight))
    plan = [[(0, 2, 0, 4), (1, 0, 0, 1)], [(0, 2, 4, 1), (1, 0, 1, 6)], [(0, 2, 5, 2), (2, 0, 0, 33)], [(2, 0, 33, 11), (0, 2, 7, 53)]]
    for step in plan:
        rows = torch.cat([seqs[s][p:p + n] for s, _, p, n in step])
        part = torch.randn_like(rows)
        proj = dev(torch.stack([rows - part, part]))
        ctx, slots = step_of([n for *_, n in step], [p for _, _, p, _ in step], [sl for _, sl, _, _ in step])
        T = rows.shape[0]
        u, dt, decay, o = (torch.full((T, c), float("nan"), device=DEV) for c in (C, H, H, inner))
        recurrent.short_conv(proj, inner, w, conv_state, slots, ctx, u, silu=True, update_state=False, bias=bias)
        state_space.steps(proj, inner + C, dt_bias, a_log, dt, decay, ctx, conv_col=inner, conv_state=conv_state, slots=slots if taps > 1 else None)
        recurrent.head_scan(u[:, inner + bc:], u[:, inner:inner + bc], decay, u[:, :inner], o, state, slots, ctx, H, N, P, weight=dt, kv_heads=G)
        for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 0.02)):
            out = torch.full((T, inner), float("nan"), dtype=dtype, device=DEV)
            state_space.gated_group_norm(o, u[:, :inner], D, proj, 0, weight, out, H, P, norm_groups, 1e-4)
            at = 0
            for s, _, p, n in step:
                ref = want[s][2][p:p + n]
                assert float((out[at:at + n].double().cpu() - ref).abs().max()) < tol * float(ref.abs().max()), (s, p, dtype)
                at += n
        assert int(ctx.error_flag.item()) == 0
        at = 0
        for s, _, p, n in step:
            assert torch.allclose(u[at:at + n].double().cpu(), want[s][0][p:p + n], atol=1e-5)
            assert torch.allclose(dt[at:at + n].double().cpu(), want[s][1][p:p + n], atol=1e-6, rtol=1e-5)
            at += n
    for slot in (1, 3):                                                      # other slots are not touched
        assert bool((state[slot] == 77.0).all()) and (conv_state is None or bool((conv_state[slot] == -55.0).all()))


def test_states_do_not_depend_on_cuts():
    """Bit for bit the same outputs and states, whatever the portions."""
    from microllm_rocm_b200.kernels import recurrent
    torch.manual_seed(1)
    H, P, N, G, n = 4, 24, 40, 2, 90
    u, dt, decay = torch.randn(n, H * P + 2 * G * N, device=DEV), torch.rand(n, H, device=DEV), torch.rand(n, H, device=DEV)
    results = []
    for cuts in ([n], [1] * n, [2, 31, 1, 33, 16, 7]):
        state = torch.full((1, H, N, P), 9.0, device=DEV)
        o = torch.empty(n, H * P, device=DEV)
        at = 0
        for m in cuts:
            ctx, slots = step_of([m], [at], [0])
            part = u[at:at + m]
            out = torch.empty(m, H * P, device=DEV)
            recurrent.head_scan(part[:, H * P + G * N:], part[:, H * P:H * P + G * N], decay[at:at + m].contiguous(), part[:, :H * P], out, state, slots,
                                ctx, H, N, P, weight=dt[at:at + m].contiguous(), kv_heads=G)
            o[at:at + m] = out
            at += m
        results.append((o, state))
    for o, state in results[1:]:
        assert torch.equal(o, results[0][0]) and torch.equal(state, results[0][1])


def test_step_sizes_at_both_ends():
    """softplus without overflow or underflow, and decays of exactly zero and one."""
    from microllm_rocm_b200.kernels import state_space
    z = torch.tensor([[-90.0, -20.0, -1.0, 0.0, 1.0, 19.9, 20.1, 90.0]], device=DEV)
    H = z.shape[1]
    dt, decay = torch.empty(1, H, device=DEV), torch.empty(1, H, device=DEV)
    ctx, _ = step_of([1], [0], [0])
    zero = torch.zeros(H, device=DEV)
    state_space.steps(z, 0, zero, zero, dt, decay, ctx)
    want = torch.nn.functional.softplus(z.double(), threshold=60.0)
    assert torch.allclose(dt.double(), want, rtol=1e-5, atol=1e-30) and torch.allclose(decay.double(), torch.exp(-want), rtol=2e-5, atol=1e-37)


# ---- latent attention with a latent for the queries
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, d, r, dv, rq, R, window, scaled", [(3, 16, 8, 24, 28, 20, 33, True), (1, 20, 6, 28, 18, 30, None, False),
                                                                (4, 64, 16, 64, 64, 64, 41, True), (2, 24, 32, 40, 40, 160, 5, False),
                                                                (5, 32, 16, 16, 24, 96, 64, True)])
def test_latent_attention_alone(H, d, r, dv, rq, R, window, scaled, dtype):
    """The mixer over scattered pages: a prompt, then portions and single tokens, one query and one far key made to point the same
    way just inside and just outside the window.  Rotated parts matter (their share of the scores is large)."""
    from microllm_rocm_b200.config.spec import PartSpec
    from microllm_rocm_b200.parts.base import PagedKVView, Runtime, StepContext
    from microllm_rocm_b200.parts.latent_attention import LatentAttention
    from microllm_rocm_b200.parts.rotary import RotaryEmbedding
    from microllm_rocm_b200.kernels import build, ops
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    rt = Runtime(torch.device(DEV), dt)
    W, n, page = 48, 140, 16
    rot = {"dims": r, "base": 900.0}
    if scaled:
        rot["scaling"] = {"factor": 4.0, "original": 48, "fast": 6.0, "slow": 1.0}
    position = RotaryEmbedding(dict(head_dim=r, theta=rot["base"], layout="interleaved", **({"stretch": rot["scaling"]} if scaled else {})), rt)
    m = {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "q_rank": rq, "kv_rank": R, "scale": 4.0 * (d + r) ** -0.5, "rot": rot}
    if window:
        m["mask"] = {"size": window}
    names = dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", o="o")
    mixer = LatentAttention(dict(hidden_size=W, num_heads=H, dim=d, rot_dim=r, vdim=dv, q_rank=rq, kv_rank=R, scale=m["scale"], eps=1e-4,
                                 window=window, names=names), rt, position)
    build.compile_many(ops.base_sources() + mixer.kernel_sources())
    g = torch.Generator().manual_seed(H + R)
    weights = {}
    for name, spec in mixer.weight_specs().items():
        t = torch.randn(spec.shape, generator=g)
        weights[name] = (1 + 0.2 * t if name.endswith("norm") else t * spec.shape[-1] ** -0.5).bfloat16().float()
    mixer.bind({k: v.to(DEV, torch.float32 if k.endswith("norm") else dt) for k, v in weights.items()})
    h = torch.randn(n, W, generator=g)
    for i in range(40, n, 7):                             # twins: the query at i is the token at an edge of its window again
        j = i - (window or 30) + (1 if i % 2 else 0)
        if j >= 0:
            h[i] = h[j]
    h = h.bfloat16().float()
    want = plain.mixer_latent(m, {"m." + k: v for k, v in weights.items()}, "m.", h.double(), 1e-4)
    blocks = -(-n // page)
    pages = torch.full((blocks + 2, page, R + r), float("nan"), dtype=dt, device=DEV)
    table = torch.randperm(blocks + 2, generator=g)[:blocks].to(torch.int32)
    at, errs = 0, []
    for count in (61, 1, 2, 1, 30, 1, 17, 1, 1, 25):
        row = table.clone()
        if window:
            row[:max(0, at - window + 1) // page] = -1
        flag = torch.zeros(1, dtype=torch.int32, device=DEV)
        ctx = StepContext(num_tokens=count, num_seqs=1, token_ids=i32([0] * count), positions=i32(list(range(at, at + count))), token_seq=i32([0] * count),
                          seq_starts=i32([0, count]), seq_pos0=i32([at]), seq_lens=i32([at + count]), block_tables={}, state_slots=None, logit_rows=None,
                          error_flag=flag, seq_starts_host=[0, count], seq_pos0_host=[at], max_new_tokens=count, max_seq_len=at + count)
        out = mixer.forward(h[at:at + count].to(DEV, dt).contiguous(), ctx, PagedKVView(pages, row.view(1, -1).to(DEV), page, True))
        assert int(flag.item()) == 0
        out = out.sum(0) if out.dim() == 3 else out
        errs.append((out.double().cpu() - want[at:at + count]).abs().amax(-1) / want.abs().max())
        at += count
    err = torch.cat(errs)
    assert at == n and float(err.max()) < (2e-5 if dtype == "float32" else 0.04), (float(err.max()), int(err.argmax()))
    # the rotation and the window do show
    for key in ("rot", "mask"):
        other = {k: v for k, v in m.items() if k != key}
        if key in m:
            off = plain.mixer_latent(other, {"m." + k: v for k, v in weights.items()}, "m.", h.double(), 1e-4)
            assert float((off - want).abs().max() / want.abs().max()) > 0.15, key


# ---- routing
@pytest.mark.parametrize("experts, top, T", [(5, 2, 33), (3, 3, 7), (3, 1, 1), (40, 6, 90), (130, 32, 20)])
def test_sigmoid_scores_as_they_are(experts, top, T):
    from microllm_rocm_b200.kernels import moe
    torch.manual_seed(experts)
    parts = torch.randn(2, T, experts + 3, device=DEV)
    ids, weights = torch.full((T, top), -1, dtype=torch.int32, device=DEV), torch.full((T, top), float("nan"), device=DEV)
    moe.select(parts, experts, None, top, ids, weights, scoring="sigmoid")
    chosen, w = plain.route(parts.double().sum(0)[:, :experts].cpu(), top)
    assert ids.cpu().tolist() == chosen.tolist() and torch.allclose(weights.double().cpu(), w, atol=1e-6)
    # scores that round to 1 and to the same tiny number: the logits still tell the experts apart
    far = torch.tensor([[30.0, 31.0, 29.0, -200.0, -199.0]], device=DEV)
    ids1, w1 = torch.empty(1, 4, dtype=torch.int32, device=DEV), torch.empty(1, 4, device=DEV)
    moe.select(far, 5, None, 4, ids1, w1, scoring="sigmoid")
    assert ids1.tolist() == [[1, 0, 2, 4]] and w1[0, :3].tolist() == [1.0, 1.0, 1.0]
    # every place's row in the layout of `top` partial results
    offsets, order, dest = (torch.full((k,), -1, dtype=torch.int32, device=DEV) for k in (experts + 1, T * top, T * top))
    moe.align(ids, experts, offsets, order, dest=dest)
    pair = order.cpu().long()
    assert torch.equal(dest.cpu().long(), (pair % top) * T + pair // top) and sorted(pair.tolist()) == list(range(T * top))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W, ff, experts, top, T", [(64, 24, 5, 2, 33), (72, 36, 3, 3, 7), (72, 36, 3, 1, 50), (50, 18, 4, 2, 9), (128, 64, 4, 3, 700)])
def test_weights_on_the_experts_input(W, ff, experts, top, T, dtype):
    """The whole feed-forward on both grouped products (sizes that 16-byte pieces suit, and sizes they do not), with and without a
    factor per column on the result; the same with the weights on the output gives something else."""
    from microllm_rocm_b200.kernels import build, ops
    from microllm_rocm_b200.parts.base import Runtime
    from microllm_rocm_b200.parts.routed import RoutedExperts
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    params = dict(hidden_size=W, experts=experts, top=top, expert_size=ff, expert_names=("e{}.gate", "e{}.up", "e{}.down"), router_name="router",
                  scoring="sigmoid")
    g = torch.Generator().manual_seed(W + top)
    part = RoutedExperts(dict(params, weight_on="input"), Runtime(torch.device(DEV), dt))
    build.compile_many(ops.base_sources() + part.kernel_sources())
    weights = {name: (torch.randn(spec.shape, generator=g) * spec.shape[-1] ** -0.5 * 2.0).bfloat16().float() for name, spec in part.weight_specs().items()}
    h = torch.randn(T, W, generator=g).bfloat16().float()
    on_dev = {k: v.to(DEV, dt) for k, v in weights.items()}
    part.bind(on_dev)
    mlp = {"router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    want = plain.routed_ff(mlp, {"m." + k: v for k, v in weights.items()}, "m.", h.double())
    x = h.to(DEV, dt)
    tol = 1e-5 if dtype == "float32" else 0.02
    out = part.forward(x, None)
    got = (out.double().sum(0) if out.dim() == 3 else out.double()).cpu()
    assert float((got - want).abs().max() / want.abs().max()) < tol
    scale = torch.rand(W, generator=g) + 0.5
    got = part.forward(x, None, out_scale=scale.to(DEV)).double().cpu()
    assert float((got - want * scale.double()).abs().max() / want.abs().max()) < tol
    other = RoutedExperts(params, Runtime(torch.device(DEV), dt))
    other.bind(on_dev)
    assert float((other.forward(x, None).double().cpu() - want).abs().max() / want.abs().max()) > 0.05


# ------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", sorted(CASES))
def test_every_layer_against_the_plain_residual_stream(folders, key, dtype):
    from microllm_rocm_b200.engine.step import StepEntry
    folder, raw, weights = folders[key]
    tokens = random_tokens(41, raw["vocab"], 5)
    want = []
    plain.forward(raw, weights, tokens, want)
    engine = engine_for(folder, dtype)
    got = {}
    engine.cache.add("x")
    engine.step([StepEntry("x", tokens, [])], tensor_sink=lambda name, t: got.__setitem__(name, None if t is None else t.float().cpu().clone()))
    engine.check_device_errors()
    for i, ref in enumerate(want):
        name = [n for n in got if n.startswith(f"run{i}.") and n.endswith(".residual")][0]
        err = (got[name].double() - ref).abs().amax(1) / ref.abs().max()              # per token
        if dtype == "float32":
            assert float(err.max()) < 2e-5, f"layer {i}: {float(err.max()):.3e}"
        else:
            assert float(err.median()) < 0.02 and int((err > 0.05).sum()) <= len(tokens) // 4, f"layer {i}: {err.tolist()}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", sorted(CASES))
@pytest.mark.parametrize("cut", ["whole", "tail", "portions"])
def test_one_request_at_a_time(folders, key, dtype, cut):
    folder, raw, weights = folders[key]
    reqs = requests_for(raw, LENGTHS[key])
    steps = {"whole": steps_whole, "tail": steps_prefill_then_decode, "portions": steps_portions}[cut](reqs)
    got = collect(engine_for(folder, dtype), steps)
    compare(got, key, raw, weights, reqs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["a", "b", "c"])
def test_mixed_batches_over_a_tight_pool(folders, key, dtype):
    """Up to four live requests, portions beside single tokens, some left out of a step; the pool holds just the peak and
    there are four state slots for ten requests, so pages and slots go from one request to the next (a slot's old state,
    convolution inputs and previous token must not leak into the request that takes it).  Guard pages around every pool."""
    folder, raw, weights = folders[key]
    reqs = requests_for(raw, [60, 33, 150, 90, 47, 128, 75, 20, 101, 64], seed=9)
    steps, peak = steps_mixed(reqs, max_live=4, seed=3)
    engine = engine_for(folder, dtype, max_tokens=peak, max_requests=4, guard_pages=True)
    got = collect(engine, steps)
    compare(got, key, raw, weights, reqs, dtype)
    engine.cache.check_guards()
    for name, group in engine.cache.groups.items():
        if group.window is None:
            assert group.pool.total_allocations > group.pool.num_pages, "the pool was never tight enough to use a page again"
    assert engine.cache.pages_released_by_window > 0
    assert engine.cache.slots.total_allocations > 4, "no state slot was used again"


def test_fp32_does_not_depend_on_cuts_batches_or_pages(folders):
    for key in ("a", "c"):
        folder, raw, weights = folders[key]
        reqs = requests_for(raw, [70, 133, 20, 45], seed=4)
        whole = collect(engine_for(folder, "float32"), steps_whole(reqs))
        portions = collect(engine_for(folder, "float32", page_size=8), steps_portions(reqs, sizes=(2, 9, 2, 30, 1, 5)))
        steps, peak = steps_mixed(reqs, max_live=3, seed=1)
        mixed = collect(engine_for(folder, "float32", max_tokens=peak), steps)
        for k in whole:
            assert torch.equal(whole[k], portions[k]) and torch.equal(whole[k], mixed[k]), f"case {key}: {k} differs between schedules"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["a", "c", "d"])
def test_far_keys_edges_and_page_borders_decide_the_output(tmp_path_factory, dtype, key):
    """Peaky softmax (its scale multiplied): single keys, far back, among the kept first ones, at a window's edge and at page
    borders, carry a position's output, in a prompt of several hundred tokens and in the tokens decoded after it, with two page
    sizes and portions of many sizes.  Scores three times as large carry three times the rounding error into the exponentials."""
    raw, weights = case(key, seed=11, sharp=3.0)
    folder = write_folder(str(tmp_path_factory.mktemp("naburax_sharp")), raw, weights)
    reqs = {"long": random_tokens(430, raw["vocab"], 21), "short": random_tokens(67, raw["vocab"], 22)}
    for page_size, steps in ((16, steps_prefill_then_decode(reqs, tail=40)), (32, steps_portions(reqs, sizes=(63, 1, 2, 1, 127, 2, 33, 1, 64, 300)))):
        got = collect(engine_for(folder, dtype, max_tokens=1200, page_size=page_size), steps)
        compare(got, key + "-sharp", raw, weights, reqs, dtype, share=0.25, fp32_tol=1e-4, median=0.8)


def test_recorded_layers_against_call_by_call(folders):
    """Layers of equal structure (two latent ones in a row in case c) are issued from a recording: the same bits either way."""
    folder, raw, weights = folders["c"]
    reqs = requests_for(raw, [90, 33], seed=6)
    for dtype in ("float32", "bfloat16"):
        engine = engine_for(folder, dtype)
        engine.model.replay_layers = False
        plain_calls = collect(engine, steps_portions(reqs, sizes=(40, 1, 7)))
        engine = engine_for(folder, dtype)
        recorded = collect(engine, steps_portions(reqs, sizes=(40, 1, 7)))
        for k in plain_calls:
            assert torch.equal(plain_calls[k], recorded[k]), k


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["b", "d"])
def test_long_decoding_from_the_first_token(folders, dtype, key):
    """One token per step from position 0 on, over many pages: every step reads and writes the state slots (the recurrence's
    matrices, the convolution's inputs and the embedding's previous token)."""
    folder, raw, weights = folders[key]
    reqs = {"d": random_tokens(150, raw["vocab"], 8)}
    got = collect(engine_for(folder, dtype, page_size=8), steps_prefill_then_decode(reqs, tail=149))
    compare(got, key, raw, weights, reqs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(folders, dtype):
    from microllm_rocm_b200.engine.llm import LLM
    from microllm_rocm_b200.sampling import GenerationConfig
    folder, raw, weights = folders["a"]
    prompts = [random_tokens(n, raw["vocab"], 50 + n) for n in (9, 40, 3)]
    llm = LLM(folder, dtype=dtype, page_size=16, max_tokens=512)
    outs = llm.generate(prompts, GenerationConfig(max_new_tokens=40, temperature=0.0))
    for prompt, got in zip(prompts, outs):
        assert len(got) == 40
        ref = plain.forward(raw, weights, list(prompt) + got[:-1])[len(prompt) - 1:]
        gaps = [float(ref[i].max() - ref[i, token]) / float(ref.abs().max()) for i, token in enumerate(got)]
        if dtype == "float32":
            assert got == ref.argmax(-1).tolist(), "fp32 greedy tokens differ from the plain implementation"
        else:       # bf16 may leave the fp32 choice at a near tie (or where it flips an expert): nearly every pick is a near maximum
            assert sum(gap > 0.05 for gap in gaps) <= 4, gaps


def test_random_config_from_the_command_line_presets():
    """The tiny preset with seeded random weights through the same entry the command line uses."""
    from microllm_rocm_b200.config import find_preset
    from microllm_rocm_b200.engine.loading import random_engine
    from microllm_rocm_b200.engine.step import StepEntry
    arch, cfg = find_preset("naburax-tiny")
    engine = random_engine(cfg, seed=3, dtype="float32", max_tokens=256, max_requests=2)
    tokens = random_tokens(33, cfg.vocab, 4)
    engine.cache.add("x")
    logits = engine.step([StepEntry("x", tokens, list(range(33)))]).cpu()
    engine.check_device_errors()
    assert torch.isfinite(logits).all() and math.isfinite(float(logits.abs().max()))
