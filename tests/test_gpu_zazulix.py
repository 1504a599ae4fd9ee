"""The Zazulix decoder on the GPU against the plain implementation (``plain_zazulix.py``): every mechanism alone, then
whole models through the engine: prompts, token-by-token decoding, portions, unequal batches, slots and pages used
again, marked keys far away, at page borders and at a window's edges, a mark carried by a recurrent state, first tokens,
long decoding, drawn configurations, greedy generation, and the trace replay program."""

import dataclasses
import os

import pytest
import torch

import helpers
import plain_zazulix as plain
from idempotent_llm_b200 import api
from idempotent_llm_b200.cache import SequenceCache
from idempotent_llm_b200.config import (DifferentialAttentionSpec, GatedMLPSpec, LatentAttentionSpec, NormSpec, RetentionSpec,
                                        RotarySpec, RoutedExpertsSpec)
from idempotent_llm_b200.config.specs import GatedMLPNames
from idempotent_llm_b200.engine.batch import context_from_packed, pack_step_host
from idempotent_llm_b200.parts import FEED_FORWARDS, MIXERS, NORMS, Runtime
from idempotent_llm_b200.weights import random_weights

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# against the 64-bit plain implementation, relative to the largest value: 32-bit sums of a few hundred terms; bfloat16
# rounds activations (8 bits of mantissa) a handful of times per layer
TOL = {"float32": 1e-4, "bfloat16": 4e-2}


def _close(got, want, dtype):
    if dtype == "float32":
        return helpers.rel_err(got, want) < TOL[dtype]
    g, w = got.detach().double().cpu(), want.detach().double().cpu()
    rms = float((g - w).pow(2).mean().sqrt() / w.pow(2).mean().sqrt())
    return rms < TOL[dtype] and helpers.rel_err(got, want) < 0.25


def _close_rows(got, want, dtype):
    """For a routed feed-forward alone in bfloat16: a token whose two best scores lie within the rounding of the router's
    input may take another expert than the 64-bit witness, so a row in thirty may be off; every other row is held to
    the type's tolerance.  32-bit is held as ever."""
    if dtype == "float32":
        return _close(got, want, dtype)
    g, w = got.detach().double().cpu(), want.detach().double().cpu()
    rows = ((g - w).pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt())
    return int((rows > TOL[dtype]).sum()) <= max(1, rows.numel() // 30) and float(rows.median()) < TOL[dtype] / 2


def _rt(dtype):
    from idempotent_llm_b200.kernels import Kernels
    dev = torch.device("cuda:0")
    return Runtime(device=dev, dtype=DT[dtype], kernels=Kernels(DT[dtype], dev))


def _ctx(slots, starts, lens, tokens=None):
    toks = tokens if tokens is not None else [[0] * L for L in lens]
    packed, n, q_lens = pack_step_host(slots, starts, toks)
    return context_from_packed(packed.cuda(), n, slots, q_lens, starts, host_tokens=toks)


def _w64(w):
    return {k: v.double().cpu() for k, v in w.items()}


def _cuts(T, sizes):
    out, lo, i = [], 0, 0
    while lo < T:
        n = sizes[min(i, len(sizes) - 1)]
        out.append((lo, min(T, lo + n)))
        lo, i = lo + n, i + 1
    return out


def _run_mixer(part, cls, spec, x, cuts, dtype, pages=24, residual=False):
    """The part alone over ``x`` cut as ``cuts`` says, in a cache of its own, in a slot that held another sequence before;
    the rows one after another.  ``residual``: the part adds into a stream of ones."""
    cache = SequenceCache({0: cls.cache_need(spec)}, 64 * pages, DT[dtype], "cuda:0", max_seqs=2)
    cache.alloc_slot()
    slot = cache.alloc_slot()
    cache.reserve([(slot, 5)]); cache.flush()
    part.forward(x[:5].contiguous().cuda(), _ctx([slot], [0], [5]), cache.view(0), cache.state_of(0), True)
    cache.set_length(slot, 5)
    cache.free_slot(slot)
    slot = cache.alloc_slot()
    outs = []
    for lo, hi in cuts:
        cache.reserve([(slot, hi)]); cache.flush()
        kw = {"residual": torch.ones((hi - lo, spec.hidden), device="cuda")} if residual else {}
        y = part.forward(x[lo:hi].contiguous().cuda(), _ctx([slot], [lo], [hi - lo]), cache.view(0), cache.state_of(0), True, **kw)
        outs.append(kw["residual"] - 1.0 if y is None else y.sum(0))
        cache.set_length(slot, hi)
    return torch.cat(outs)


def _rows_of(seed, n, width, dtype, scale=1.5):
    return (torch.randn(n, width, generator=torch.Generator().manual_seed(seed)) * scale).to(DT[dtype])


# ----------------------------------------------------------------------------------- the differential attention, alone
def _diff_spec(rot=6, base=3000.0, **kw):
    d = dict(hidden=40, n_heads=6, n_kv_heads=2, key_dim=12, value_dim=16, softmax_scale=0.5, diff=0.35, eps=1e-5, conv_taps=3)
    d.update(kw)
    if rot:
        d["position"] = RotarySpec(theta=base, dim=rot, max_positions=1 << 20, variant="half_partial")
    return DifferentialAttentionSpec(**d)


def _plain_diff(x, w, s, p):
    m = dict(heads=s.n_heads, kv_heads=s.n_kv_heads, dim=s.key_dim, vdim=s.value_dim, scale=s.softmax_scale, diff=s.diff,
             rot=dict(base=s.position.theta, dims=s.position.dim) if s.position else None, conv=s.conv_taps)
    if not s.head_gate:                       # (a gate of 1/2 everywhere, taken out again: the output projection is linear)
        return 2.0 * plain.differential_mixer(x, {**w, p + "g": torch.zeros(s.n_heads, s.hidden, dtype=x.dtype)}, p, m, s.eps)
    return plain.differential_mixer(x, w, p, m, s.eps)


def _diff_weights(cls, spec, dtype, seed):
    """Sharp scores, and vectors whose products move the maps' weight well away from its constant."""
    w = random_weights(cls.declare(spec, "M."), seed, 0.25, dtype=DT[dtype], device="cuda")
    w["M.q"] = (w["M.q"].float() * 2.0).to(DT[dtype])
    for n in ("lq1", "lk1", "lq2", "lk2"):
        w["M." + n] = (w["M." + n].float() * 2.0).to(DT[dtype])
    return w


DIFF_VARIANTS = {
    "grouped": lambda: _diff_spec(),
    "one_head": lambda: _diff_spec(n_heads=1, n_kv_heads=1, key_dim=5, value_dim=7, rot=0, conv_taps=2),
    "no_filter": lambda: _diff_spec(conv_taps=None, rot=12),
    "one_tap": lambda: _diff_spec(conv_taps=1, n_kv_heads=6),
    "long_filter": lambda: _diff_spec(conv_taps=8, rot=2, hidden=36, value_dim=40),
    "no_gate": lambda: _diff_spec(head_gate=False, diff=0.0),
    # twice the map's size is the values': head sizes the tensor cores have
    "tc_64": lambda: _diff_spec(n_heads=4, n_kv_heads=2, key_dim=32, value_dim=64, softmax_scale=0.25, conv_taps=4, rot=16),
    "tc_128_long": lambda: _diff_spec(n_heads=3, n_kv_heads=1, key_dim=64, value_dim=128, softmax_scale=0.15, rot=64),
    "tc_64_eight": lambda: _diff_spec(n_heads=8, n_kv_heads=1, key_dim=32, value_dim=64, softmax_scale=0.25, rot=32, diff=0.8),
    # keys of 64 beside values of another size
    "uneven": lambda: _diff_spec(n_heads=4, n_kv_heads=4, key_dim=32, value_dim=48, softmax_scale=0.25, rot=32),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(DIFF_VARIANTS))
def test_the_differential_attention_alone_prompt_portions_single_tokens(dtype, variant):
    spec = DIFF_VARIANTS[variant]()
    cls = MIXERS.get(spec.kind)
    w = _diff_weights(cls, spec, dtype, 5)
    part = cls(spec, w, "M.", _rt(dtype))
    T, pre = (1300, 1205) if variant.endswith("long") else (150, 125)
    x = _rows_of(3, T, spec.hidden, dtype)
    ref = _plain_diff(x.double(), _w64(w), spec, "M.")
    whole = _run_mixer(part, cls, spec, x, [(0, T)], dtype)
    cut = _run_mixer(part, cls, spec, x, [(0, 70), (70, 72), (72, 73), (73, pre)] + [(i, i + 1) for i in range(pre, T)], dtype, residual=True)
    assert _close(whole, ref, dtype) and _close(cut, ref, dtype)
    if dtype == "float32":
        assert helpers.rel_err(cut, whole) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_map_counts_and_so_does_their_weight(dtype):
    """Turning nothing, swapping the maps, filtering nothing or reading their weight another way is far outside the tolerance."""
    spec = DIFF_VARIANTS["tc_64"]()
    cls = MIXERS.get(spec.kind)
    w = _diff_weights(cls, spec, dtype, 6)
    x = _rows_of(4, 90, spec.hidden, dtype)
    got = _run_mixer(cls(spec, w, "M.", _rt(dtype)), cls, spec, x, [(0, 90)], dtype)
    W = _w64(w)
    assert _close(got, _plain_diff(x.double(), W, spec, "M."), dtype)
    for change in ("lq1", "lk2"):
        other = dict(W); other["M." + change] = -W["M." + change]
        assert not _close(got, _plain_diff(x.double(), other, spec, "M."), dtype), change
    swapped = dict(W)
    swapped["M.q"] = W["M.q"].view(4, 2, 32, -1)[:, [1, 0]].reshape(W["M.q"].shape)
    assert not _close(got, _plain_diff(x.double(), swapped, spec, "M."), dtype)
    for s in (dataclasses.replace(spec, diff=spec.diff + 0.2), dataclasses.replace(spec, position=None), dataclasses.replace(spec, conv_taps=None)):
        assert not _close(got, _plain_diff(x.double(), W, s, "M."), dtype)


def test_two_sequences_in_a_step_keep_their_filters_and_keys():
    """Unequal sequences side by side, one of them a single token beside a portion: filters read their own sequence's
    inputs, from the step and from the state."""
    spec = DIFF_VARIANTS["tc_64"]()
    cls = MIXERS.get(spec.kind)
    w = _diff_weights(cls, spec, "bfloat16", 7)
    part = cls(spec, w, "M.", _rt("bfloat16"))
    lens = (80, 40)
    x = [_rows_of(10 + n, n, spec.hidden, "bfloat16").cuda() for n in lens]
    cache = SequenceCache({0: cls.cache_need(spec)}, 64 * 8, torch.bfloat16, "cuda:0", max_seqs=2)
    slots, at, got = [cache.alloc_slot(), cache.alloc_slot()], [0, 0], [[], []]
    for step in [(1, 30), (60, 1), (2, 3), (1, 1), (16, 5)]:
        hi = [a + n for a, n in zip(at, step)]
        cache.reserve(list(zip(slots, hi))); cache.flush()
        y = part.forward(torch.cat([x[i][at[i]:hi[i]] for i in (0, 1)]), _ctx(slots, at, list(step)), cache.view(0), cache.state_of(0), True).sum(0)
        got[0].append(y[:step[0]]); got[1].append(y[step[0]:])
        at = hi
        for s, n in zip(slots, at):
            cache.set_length(s, n)
    for i in (0, 1):
        assert at[i] == lens[i] and _close(torch.cat(got[i]), _plain_diff(x[i].double().cpu(), _w64(w), spec, "M."), "bfloat16")


# ----------------------------------------------------------------------------------- the latent attention, alone
def _latent_spec(**kw):
    d = dict(hidden=40, n_heads=3, plain_dim=16, rot_dim=0, value_dim=24, kv_rank=40, softmax_scale=0.5, eps=1e-5, window=37, gate=True)
    d.update(kw)
    return LatentAttentionSpec(**d)


def _plain_latent(x, w, s, p):
    m = dict(heads=s.n_heads, dim=s.plain_dim, vdim=s.value_dim, kv_rank=s.kv_rank, scale=s.softmax_scale,
             mask=dict(size=s.window) if s.window else None)
    return plain.latent_mixer(x, w, p, m, s.eps)


LATENT_VARIANTS = {
    "three_heads": lambda: _latent_spec(),
    "one_head": lambda: _latent_spec(n_heads=1, plain_dim=8, value_dim=8, kv_rank=8, window=1),
    "odd": lambda: _latent_spec(n_heads=5, plain_dim=6, value_dim=10, kv_rank=22, hidden=20, window=65),
    "no_window": lambda: _latent_spec(window=None, n_heads=9),
    "window_2": lambda: _latent_spec(window=2),
    # latents the fragment kernel has; heads that fill, or do not fill, the tensor-core attention's
    "fragments_64": lambda: _latent_spec(n_heads=4, plain_dim=64, value_dim=64, kv_rank=64, softmax_scale=0.2, window=64),
    "fragments_padded": lambda: _latent_spec(n_heads=20, plain_dim=48, value_dim=72, kv_rank=160, softmax_scale=0.2, window=100),
    "values_padded": lambda: _latent_spec(n_heads=2, plain_dim=128, value_dim=40, kv_rank=96, softmax_scale=0.15, window=128),
    "long": lambda: _latent_spec(n_heads=2, plain_dim=64, value_dim=64, kv_rank=96, softmax_scale=0.2, window=600),
    "long_plain": lambda: _latent_spec(n_heads=2, plain_dim=20, value_dim=12, kv_rank=40, window=300),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(LATENT_VARIANTS))
def test_the_windowed_latent_attention_alone_prompt_portions_single_tokens(dtype, variant):
    spec = LATENT_VARIANTS[variant]()
    cls = MIXERS.get(spec.kind)
    w = random_weights(cls.declare(spec, "M."), 5, 0.25, dtype=DT[dtype], device="cuda")
    w["M.q"] = (w["M.q"].float() * 2.0).to(DT[dtype])
    part = cls(spec, w, "M.", _rt(dtype))
    T, pre = (1300, 1205) if variant.startswith("long") else (170, 130)
    x = _rows_of(3, T, spec.hidden, dtype)
    W = _w64(w)
    ref = _plain_latent(x.double(), W, spec, "M.")
    whole = _run_mixer(part, cls, spec, x, [(0, T)], dtype)
    cut = _run_mixer(part, cls, spec, x, [(0, 70), (70, 72), (72, pre)] + [(i, i + 1) for i in range(pre, T)], dtype, residual=True)
    assert _close(whole, ref, dtype) and _close(cut, ref, dtype)
    if spec.window and spec.window > 2 and dtype == "float32":               # one key more or less is far outside the tolerance
        for off in (-1, 1):
            assert not _close(whole, _plain_latent(x.double(), W, dataclasses.replace(spec, window=spec.window + off), "M."), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_tokens_of_many_sequences_share_the_window_kernel(dtype):
    """Forty sequences of unlike lengths decode side by side (steps of many tokens walk their keys in one run, steps of
    few in several): every row against its own sequence's plain result."""
    spec = LATENT_VARIANTS["fragments_64"]()
    cls = MIXERS.get(spec.kind)
    w = random_weights(cls.declare(spec, "M."), 8, 0.25, dtype=DT[dtype], device="cuda")
    part = cls(spec, w, "M.", _rt(dtype))
    W, n = _w64(w), 40
    lens = [1 + 7 * i % 193 for i in range(n)]
    x = [_rows_of(100 + i, L + 1, spec.hidden, dtype) for i, L in enumerate(lens)]
    cache = SequenceCache({0: cls.cache_need(spec)}, 64 * 4 * n, DT[dtype], "cuda:0", max_seqs=n)
    slots = [cache.alloc_slot() for _ in range(n)]
    for i, (s, L) in enumerate(zip(slots, lens)):
        cache.reserve([(s, L)]); cache.flush()
        part.forward(x[i][:L].cuda(), _ctx([s], [0], [L]), cache.view(0), None, True)
        cache.set_length(s, L)
    for live in (range(n), range(0, n, 13)):
        cache.reserve([(slots[i], lens[i] + 1) for i in live]); cache.flush()
        y = part.forward(torch.cat([x[i][-1:] for i in live]).cuda(), _ctx([slots[i] for i in live], [lens[i] for i in live], [1] * len(live)),
                         cache.view(0), None, True).sum(0)
        want = torch.stack([_plain_latent(x[i].double(), W, spec, "M.")[-1] for i in live])
        assert _close(y, want, dtype)


# ----------------------------------------------------------------------------------- the retention, alone
def _ret_spec(rot=10, base=3000.0, **kw):
    d = dict(hidden=40, heads=3, key_dim=16, value_dim=12, decay=(0.9, 0.999, 0.5), eps=1e-5)
    d.update(kw)
    if rot:
        d["position"] = RotarySpec(theta=base, dim=rot, max_positions=1 << 20, variant="half_partial")
    return RetentionSpec(**d)


def _plain_ret(x, w, s, p):
    m = dict(heads=s.heads, dim=s.key_dim, vdim=s.value_dim, decay=list(s.decay),
             rot=dict(base=s.position.theta, dims=s.position.dim) if s.position else None)
    return plain.retention_mixer(x, w, p, m, s.eps)


RET_VARIANTS = {
    "three_heads": lambda: _ret_spec(),
    "one_head": lambda: _ret_spec(heads=1, key_dim=5, value_dim=7, decay=(0.97,), rot=0, hidden=20),
    "extremes": lambda: _ret_spec(heads=4, decay=(0.0, 1.0, 1e-3, 0.9999), rot=16),
    "wide_values": lambda: _ret_spec(heads=2, key_dim=24, value_dim=130, decay=(0.99, 0.95), rot=24),
    "wide_keys": lambda: _ret_spec(heads=2, key_dim=200, value_dim=20, decay=(0.99, 0.95), rot=64),
    "tiles": lambda: _ret_spec(heads=2, key_dim=128, value_dim=192, decay=(0.98, 0.999), rot=128),
    "off_borders": lambda: _ret_spec(heads=3, key_dim=34, value_dim=66, hidden=36, rot=2),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(RET_VARIANTS))
def test_the_retention_alone_in_portions(dtype, variant):
    """Whole, one by one, and in portions on both sides of where chunks begin; chunks of fewer tokens than a whole one and
    one token more than a whole one."""
    spec = RET_VARIANTS[variant]()
    cls = MIXERS.get(spec.kind)
    w = random_weights(cls.declare(spec, "M."), 7, 0.2, dtype=DT[dtype], device="cuda")
    part = cls(spec, w, "M.", _rt(dtype))
    T = 210
    x = _rows_of(8, T, spec.hidden, dtype, 1.2)
    ref = _plain_ret(x.double(), _w64(w), spec, "M.")
    for sizes in ([T], [1], [2], [64, 65], [3, 1, 70, 8, 9, 2, 17, 128]):
        got = _run_mixer(part, cls, spec, x, _cuts(T, sizes), dtype, residual=sizes[0] == 64)
        assert _close(got, ref, dtype), f"portions of {sizes}"
    if variant == "three_heads":
        for other in (dataclasses.replace(spec, decay=(0.9, 0.995, 0.5)), dataclasses.replace(spec, position=None)):
            assert not _close(got, _plain_ret(x.double(), _w64(w), other, "M."), dtype)


def test_both_forms_of_the_recurrence_on_the_same_numbers():
    """Token by token against chunks, in 32-bit, for unequal sequences in one step: read-outs and the states left behind;
    a sequence of few tokens runs in a chunk of its own beside long ones."""
    K = _rt("float32").kernels
    H, dk, dv, lens = 3, 40, 72, [130, 3, 64, 65, 1]
    decay = torch.tensor([0.97, 1.0, 0.3], device="cuda")
    g = torch.Generator().manual_seed(3)
    proj = torch.randn(sum(lens), H * (2 * dk + dv) + 4, generator=g).cuda()
    out, states = {}, {}
    for form in ("walk", "chunks"):
        K.RETENTION_WALK = 10 ** 9 if form == "walk" else 0
        ctx = _ctx(list(range(5)), [0] * 5, lens)
        state = torch.randn(5, H * dk * dv + 7, generator=torch.Generator().manual_seed(4)).cuda()
        cs = K.rope_table(ctx.positions, (1e4 ** (-2.0 * torch.arange(0, 9, dtype=torch.float64) / 18)).cuda())
        out[form] = K.retention(proj.clone(), (0, H * dk, 2 * H * dk), cs, dk ** -0.5, decay, state[:, 7:], ctx, H, dk, dv)
        states[form] = state
    assert helpers.rel_err(out["chunks"], out["walk"]) < 1e-5 and helpers.rel_err(states["chunks"], states["walk"]) < 1e-5


# ----------------------------------------------------------------------------------- norm and feed-forwards, alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_norms_offset(dtype):
    rt = _rt(dtype)
    spec = NormSpec(size=72, eps=1e-5, weight="", weight_offset=1.0)
    cls = NORMS.get(spec.kind)
    w = random_weights(cls.declare(spec, "n"), 3, 0.3, dtype=DT[dtype], device="cuda")
    x = torch.randn(9, 72, generator=torch.Generator().manual_seed(5)).cuda()
    got = cls(spec, w, "n", rt).forward(x.clone(), None, _ctx([0], [0], [9]))
    assert _close(got, plain.norm(x.double().cpu(), 1e-5, w["n"].double().cpu()), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,inter,limit", [(32, 56, 0.8), (20, 30, 0.3), (64, 200, 7.0), (24, 8, 0.0)])
def test_the_clamped_feed_forward_in_every_kernel(dtype, hidden, inter, limit):
    """One token (few-token products) to 600 (the persistent kernels' epilogue); inputs on both sides of the limit."""
    rt = _rt(dtype)
    spec = GatedMLPSpec(hidden=hidden, intermediate=inter, activation="clamped", limit=limit, slope=1.702, names=GatedMLPNames("gate", "up", "down"))
    cls = FEED_FORWARDS.get(spec.kind)
    w = random_weights(cls.declare(spec, "F."), 3, 0.3, dtype=DT[dtype], device="cuda")
    part = cls(spec, w, "F.", rt)
    for n in (1, 7, 130, 600):
        x = _rows_of(n, n, hidden, dtype)
        ref = plain.clamped_ff(x.double(), _w64(w), "F.", limit)
        assert _close(part.forward(x.cuda(), None).sum(0), ref, dtype), n
        h = torch.ones(n, hidden, device="cuda")
        d = part.forward(x.cuda(), None, residual=h)
        assert _close((h if d is None else h + d.sum(0)) - 1.0, ref, dtype), n


ROUTER_SHAPES = [
    # experts, per token, groups, kept groups, the group's score: a sum of so many
    (18, 2, 3, 1, 2), (7, 3, 1, 1, 2), (64, 6, 8, 3, 2), (3, 3, 1, 1, 2), (12, 4, 4, 4, 2), (40, 1, 5, 1, 3), (96, 8, 3, 2, 2), (4, 1, 4, 2, 2), (6, 2, 2, 1, 1),
]


@pytest.mark.parametrize("E,top,groups,keep,group_top", ROUTER_SHAPES)
@pytest.mark.parametrize("shift", [0.0, -3.0])
def test_the_router_kernel_against_plain(E, top, groups, keep, group_top, shift):
    """With ``shift`` every choice score is negative: an expert that is shut out must lose to all of them.  The column behind
    the logits is the shared expert's gate."""
    K = _rt("float32").kernels
    g = torch.Generator().manual_seed(E * 7 + top)
    z = (torch.randn(300, E + 1, generator=g) * 2.0).cuda()
    corr = (torch.randn(E, generator=g) * 0.3 + shift).cuda()
    chosen, weight, gate = K.route(z, corr, top, groups, keep, 1.7, sigmoid=True, group_top=group_top, n_experts=E)
    z64, c64 = z.double().cpu(), corr.double().cpu()
    s = torch.sigmoid(z64[:, :E]) + c64
    parts = s.view(300, groups, -1)
    scores = parts.topk(min(group_top, E // groups), dim=-1).values.sum(-1)
    open_ = torch.zeros_like(parts, dtype=torch.bool)
    for t in range(300):
        open_[t, scores[t].topk(keep).indices] = True
    want = s.masked_fill(~open_.view(300, E), -float("inf")).topk(top, dim=-1).indices
    assert torch.equal(chosen.cpu().long(), want)
    if group_top == 2:
        assert torch.equal(want, plain.route(z64[:, :E], c64, dict(top=top, groups=dict(count=groups, keep=keep)))[0])
    assert helpers.rel_err(weight, plain.weigh(z64[:, :E], want, 1.7)) < 1e-5
    assert helpers.rel_err(gate, torch.sigmoid(z64[:, E])) < 1e-6


def test_equal_choice_scores_in_a_group_count_each():
    """Two experts with the same score add up like two; the lower index is taken first."""
    K = _rt("float32").kernels
    s = torch.tensor([[0.6, 0.6, 0.1, 0.95, 0.2, 0.1]])
    z = torch.log(s / (1 - s)).cuda()
    chosen, _ = K.route(z, torch.zeros(6, device="cuda"), 2, 2, 1, 1.0, sigmoid=True, group_top=2)
    assert chosen.tolist() == [[0, 1]]


def _moe_spec(shared=40, **kw):
    base = dict(hidden=32, intermediate=24, n_experts=8, top=3, groups=4, groups_keep=2, group_top=2, scale=1.5, scores="sigmoid")
    base.update(kw)
    if shared:
        base["shared"] = GatedMLPSpec(hidden=base["hidden"], intermediate=shared, names=GatedMLPNames("shared.gate", "shared.up", "shared.down"))
        base["shared_gate"] = "shared.sg"
    return RoutedExpertsSpec(**base)


MOE_VARIANTS = {
    "groups_shared": lambda: _moe_spec(),
    "one_of_three": lambda: _moe_spec(n_experts=3, top=1, groups=1, groups_keep=1, scale=1.0, shared=None),
    "off_borders": lambda: _moe_spec(hidden=20, intermediate=12, n_experts=6, top=2, groups=3, groups_keep=3, shared=28),
    "many": lambda: _moe_spec(hidden=64, intermediate=32, n_experts=16, top=2, groups=2, groups_keep=1, scale=2.5, shared=72),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(MOE_VARIANTS))
def test_routed_experts_alone_in_steps_of_every_size(dtype, variant):
    """3 tokens (every pair streams its expert), 30 and 100, 300 (rows grouped by expert on the host), and 300 without the
    host's help (a captured step's way), as a delta and added into the stream: the same sums."""
    spec = MOE_VARIANTS[variant]()
    cls = FEED_FORWARDS.get(spec.kind)
    w = random_weights(cls.declare(spec, "F."), 11, 0.2, dtype=DT[dtype], device="cuda")
    w["F.router"] = (w["F.router"].float() * 6.0).to(DT[dtype])          # decisive choices: few calls close enough to round over
    if spec.shared is not None:
        w["F.shared.sg"] = (w["F.shared.sg"].float() * 4.0).to(DT[dtype])
    part = cls(spec, w, "F.", _rt(dtype))
    c = dict(kind="moe", expert=dict(ff=spec.intermediate), shared=dict(ff=1) if spec.shared else None,
             router=dict(experts=spec.n_experts, top=spec.top, scale=spec.scale, groups=dict(count=spec.groups, keep=spec.groups_keep)))
    for n, host in ((3, True), (30, True), (100, True), (300, True), (300, False)):
        x = _rows_of(n, n, spec.hidden, dtype, 1.3)
        ctx = _ctx([0], [0], [n])
        if not host:
            ctx.host_tokens = None
        ref = plain.experts_ff(x.double(), _w64(w), "F.", c)
        assert _close_rows(part.forward(x.cuda(), ctx).sum(0), ref, dtype), n
        h = torch.ones(n, spec.hidden, device="cuda")
        assert part.forward(x.cuda(), ctx, residual=h) is None and _close_rows(h - 1.0, ref, dtype), n


# ----------------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def zazulix_dirs(tmp_path_factory):
    made = {}

    def get(name, dtype="bfloat16", seed=1):
        key = (name, dtype, seed)
        if key not in made:
            d = str(tmp_path_factory.mktemp(f"zazulix-{name}-{dtype}-{seed}"))
            helpers.make_zazulix_dir(helpers.ZAZULIX[name](), d, seed=seed, dtype=DT[dtype], edit=_sharpen)
            made[key] = d
        return made[key]
    return get


def _sharpen(n, t):
    """Maps' weights away from their constant, decisive routers."""
    if n.split(".")[-1] in ("lq1", "lk1", "lq2", "lk2"):
        return (t.float() * 2.0).to(t.dtype)
    if n.endswith("mlp.router"):
        return (t.float() * 3.0).to(t.dtype)
    return t


class RouteTap:
    """Writes down, per routed layer and sequence, the experts the model gave each token and what its router read
    (steps called from Python only: a captured step's choices stay on the device).  In bfloat16 the stream a router
    reads is a few parts in a thousand off the 64-bit one, so a choice may fall another way than in 64-bit, and what
    the token and those behind it then compute is another function.  So the 64-bit witness is given the model's choices
    (``plain.forward(routes=...)``: weights, experts and everything else stay its own), and the choices themselves are
    held against the plain router run on the very rows the model's router read: there they must be the same but for
    ties.  32-bit models are compared with nothing handed over."""

    def __init__(self, lm):
        self.seen, self.layout = {}, None
        for li, b in enumerate(lm.model.blocks):
            if hasattr(b.feed_forward, "route"):
                b.feed_forward.route = self._wrap(b.feed_forward.route, li)
        inner = lm.engine.step

        def step(entries, want=None):
            self.layout = [(int(s), len(t)) for s, t in entries]
            return inner(entries, want)
        lm.engine.step = step

    def _wrap(self, inner, li):
        def route(x):
            chosen, *rest = inner(x)
            rows, xs, off = chosen.cpu(), x.double().cpu(), 0
            for slot, n in self.layout:
                self.seen.setdefault(slot, {}).setdefault(li, []).append((rows[off:off + n], xs[off:off + n]))
                off += n
            return (chosen, *rest)
        return route

    def routes(self, slot, cfg, w):
        """{layer: [T, top]} of a sequence, checked against the plain router on the same inputs."""
        out = {}
        for li, parts in self.seen.pop(slot, {}).items():
            chosen, x = torch.cat([p[0] for p in parts]).long(), torch.cat([p[1] for p in parts])
            out[li] = chosen
            z, corr, r = x @ w[f"l{li}.mlp.router"].T, w[f"l{li}.mlp.correction"], cfg["layers"][li]["mlp"]["router"]
            own, margin = plain.route(z, corr, r)[0], plain.route_margin(z, corr, r)
            off = [t for t in range(x.shape[0]) if sorted(own[t].tolist()) != sorted(chosen[t].tolist())]
            assert all(float(margin[t]) < 1e-3 for t in off), f"layer {li}: tokens {off[:5]} were given other experts than their scores name"
        return out


def _load(d, dtype, **kw):
    """The model and, in bfloat16, the tap on its routers (with steps called from Python)."""
    if dtype == "bfloat16":
        lm = api.load(d, dtype=dtype, use_graph=False, **kw)
        return lm, RouteTap(lm)
    return api.load(d, dtype=dtype, **kw), None


def _close_model(got, want, dtype):
    """Whole models, row by row: the worst row in twenty is left out of the root mean square, which is held to the type's
    tolerance, and no row may be lost.  (A norm divides a short vector's rounding by its own length: a sequence's first
    read-out is one value row times q . k, and where q . k is small 32-bit arithmetic of any order is 1e-4 off there.)"""
    g, w = got.detach().double().cpu(), want.detach().double().cpu()
    rows = (g - w).pow(2).mean(-1) / w.pow(2).mean()
    kept = rows.sort().values[:rows.numel() - max(2, rows.numel() // 20)] if rows.numel() > 4 else rows
    return float(kept.mean().sqrt()) < TOL[dtype] and float(rows.max().sqrt()) < (5e-3 if dtype == "float32" else 0.5)


def _plain_logits(model_dir, tokens, tap=None, slot=None, layers=None):
    cfg, w = plain.load(model_dir)
    if tap is None:
        return plain.forward(cfg, w, tokens, layers)
    flips = []
    out = plain.forward(cfg, w, tokens, layers, routes=tap.routes(slot, cfg, w), flips=flips)
    assert len(flips) <= max(3, len(tokens) // 4), f"{len(flips)} choices of {len(tokens)} tokens fell another way than in 64-bit"
    return out


def _step_all(lm, slot, tokens, lo, hi):
    return lm.engine.step([(slot, tokens[lo:hi])], [list(range(hi - lo))])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "T"])
def test_whole_prompt_and_every_layer_against_plain(zazulix_dirs, name, dtype):
    d = zazulix_dirs(name, dtype)
    lm, tap = _load(d, dtype, max_tokens=512)
    toks = helpers.rand_ids(190, lm.spec.vocab_size, 5)
    seen = []

    def recording(inner):
        def forward(h, *a, **k):
            out = inner(h, *a, **k)
            seen.append(out[0].clone() if out[1] is None else out[0] + out[1].sum(0))
            return out
        return forward
    for b in lm.model.blocks:
        b.forward = recording(b.forward)
    s = lm.engine.open()
    got = _step_all(lm, s, toks, 0, len(toks))
    layers = []
    want = _plain_logits(d, toks, tap, s, layers)
    assert len(seen) == len(layers)
    for i, h in enumerate(seen):
        assert h.dtype == torch.float32 and _close_model(h, layers[i], dtype), f"stream after layer {i}"
    assert _close_model(got, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "T"])
def test_token_by_token_from_the_first_token_equals_the_prompt(zazulix_dirs, name, dtype):
    d = zazulix_dirs(name, dtype)
    lm, tap = _load(d, dtype, max_tokens=512)
    toks = helpers.rand_ids(140, lm.spec.vocab_size, 9)
    s = lm.engine.open()
    whole = _step_all(lm, s, toks, 0, len(toks))
    assert _close_model(whole, _plain_logits(d, toks, tap, s), dtype)
    lm.engine.close(s)
    s = lm.engine.open()
    one = torch.cat([_step_all(lm, s, toks, i, i + 1) for i in range(len(toks))])
    assert _close_model(one, _plain_logits(d, toks, tap, s), dtype)
    if dtype == "float32":
        assert _close_model(one, whole, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,sizes", [("A", [2]), ("A", [3, 2, 64, 1, 2]), ("A", [20, 13, 20, 2, 1, 64]), ("T", [64, 65]), ("T", [63, 2, 128, 2])])
def test_portions_of_several_sizes(zazulix_dirs, name, dtype, sizes):
    d = zazulix_dirs(name, dtype)
    lm, tap = _load(d, dtype, max_tokens=512)
    toks = helpers.rand_ids(45 if sizes == [2] else 200, lm.spec.vocab_size, 21)
    s = lm.engine.open()
    got = torch.cat([_step_all(lm, s, toks, lo, hi) for lo, hi in _cuts(len(toks), sizes)])
    assert _close_model(got, _plain_logits(d, toks, tap, s), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "T"])
def test_unequal_batch_against_each_alone_with_slots_and_pages_used_again(zazulix_dirs, name, dtype):
    """Three requests of unlike lengths start in one step and decode together, the short ones leaving early; then
    the slots, states and pages they gave back serve other requests."""
    d = zazulix_dirs(name, dtype)
    lm, tap = _load(d, dtype, max_tokens=64 * 7, max_seqs=3)
    V = lm.spec.vocab_size
    rounds = [[helpers.rand_ids(n, V, 30 + n) for n in (1, 67, 158)], [helpers.rand_ids(n, V, 50 + n) for n in (129, 3, 64)]]
    extra = [12, 5, 9]
    for reqs in rounds:
        full = [r + helpers.rand_ids(e, V, len(r)) for r, e in zip(reqs, extra)]
        slots = [lm.engine.open() for _ in reqs]
        got = [[] for _ in reqs]
        lg = lm.engine.step([(s, r) for s, r in zip(slots, reqs)], [list(range(len(r))) for r in reqs])
        off = 0
        for i, r in enumerate(reqs):
            got[i].append(lg[off:off + len(r)]); off += len(r)
        for step in range(max(extra)):
            live = [i for i in range(len(reqs)) if step < extra[i]]
            lg = lm.engine.step([(slots[i], [full[i][len(reqs[i]) + step]]) for i in live])
            for row, i in enumerate(live):
                got[i].append(lg[row:row + 1])
            for i in range(len(reqs)):
                if step == extra[i] - 1:
                    lm.engine.close(slots[i])
        for i in range(len(reqs)):
            assert _close_model(torch.cat(got[i]), _plain_logits(d, full[i], tap, slots[i]), dtype), f"request {i}"
    assert lm.engine.cache.pages_held() == 0


def _marked_model(tmp, dtype, kind, window=None, dim=8, which=0, decay=0.99):
    """A one-layer model that finds ONE token.  The stream's first coordinate is -1 for every token but token 1 (+1), the
    second 1 for all.  Attentions: a head's query is minus the first coordinate and its key plus it, in a dim that is not
    turned, so that any other token's query takes the marked key alone; without it the softmax is spread over all keys
    (``which``: the differential attention's map that looks for it; the other stays spread).  Retention: keys are the sum of
    the two coordinates, zero but for the mark, so the state holds the marked token's value and nothing else, which the
    norm behind it brings back to full size however far it has faded."""
    if kind == "attention":
        layer = helpers.zazulix_attention(heads=2, kv_heads=1, dim=dim, vdim=2 * dim, scale=1.0, diff=0.5, conv=2, rot_dims=2, mlp=None)
    elif kind == "latent_attention":
        layer = helpers.zazulix_latent(heads=2, dim=dim, vdim=dim, kv_rank=32, scale=1.0, window=window, mlp=None)
    else:
        layer = helpers.zazulix_retention(heads=2, dim=dim, vdim=dim, decay=(decay, 1.0), rot_dims=2, mlp=None)
    cfg = helpers.zazulix_config([layer], vocab=16, width=16)
    p = "l0.mix."

    def edit(n, t):
        t = t.float()
        if n == "embed":
            t[:, 0] = -1.0; t[1, 0] = 1.0; t[:, 1] = 1.0
        elif n.endswith("norm1"):
            t = torch.zeros_like(t)
        elif n == p + "q":
            t = torch.zeros_like(t)
            if kind == "retention":
                t[4, 1] = 1.0; t[dim + 4, 1] = 1.0
            else:
                t[which * dim + 4, 0] = -10.0
        elif n == p + "k":
            t = torch.zeros_like(t)
            if kind == "retention":
                t[4, :2] = 1.0; t[dim + 4, :2] = 1.0
            else:
                t[which * dim + 4, 0] = 2.0
        elif n.endswith("q.conv") or n.endswith("k.conv"):
            t = torch.zeros_like(t); t[:, -1] = 1.0             # (the values keep their filters)
        elif n == p + "dkv":
            t[0] = 0.0; t[0, 0] = 1.0
        elif n == p + "dkv.norm":
            t = torch.ones_like(t)
        elif n == p + "uk":
            t = torch.zeros_like(t); t[4, 0] = 4.0
        elif n in (p + "o", p + "uv", p + "v"):
            t = t * (8.0 if kind == "attention" else 4.0)     # (the mixer's output weighs against the stream)
        return t.to(DT[dtype])
    return helpers.make_zazulix_dir(cfg, tmp, seed=3, dtype=DT[dtype], edit=edit)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("where", [0, 63, 64, 65, 127, 255, 300])
@pytest.mark.parametrize("kind", ["latent_attention", "attention", "second map", "tensor cores", "retention"])
def test_one_far_token_among_hundreds_in_prompts_and_in_decoding(tmp_path, kind, dtype, where):
    """The marked token sits at a page's, a run's or a chunk's first or last place, or far back; every later token finds it,
    in a prompt, across portions and when decoding alone.  Without the mark the logits differ, so a lost key or a lost
    state shows."""
    d = (_marked_model(str(tmp_path), dtype, "attention", dim=8, which=1) if kind == "second map" else
         _marked_model(str(tmp_path), dtype, "attention", dim=32) if kind == "tensor cores" else _marked_model(str(tmp_path), dtype, kind))
    lm = api.load(d, dtype=dtype, max_tokens=512)
    T = 330
    toks = [2 + (i % 13) for i in range(T)]
    toks[where] = 1
    want = _plain_logits(d, toks)
    lost = list(toks); lost[where] = 2
    assert helpers.rel_err(_plain_logits(d, lost)[-1:], want[-1:]) > 0.05        # the mark matters to the last token
    portions = _cuts(T, [where + 1, 2, 250])[:3]               # up to the mark, two tokens, up to 250, the rest alone
    for cuts in ([(0, T)], portions + [(i, i + 1) for i in range(portions[-1][1], T)], [(0, 280)] + [(i, i + 1) for i in range(280, T)]):
        s = lm.engine.open()
        got = torch.cat([_step_all(lm, s, toks, lo, hi) for lo, hi in cuts])
        lm.engine.close(s)
        assert _close(got, want, dtype), f"cuts {cuts[:4]}"
        assert _close(got[-1:], want[-1:], dtype), f"the last token, cuts {cuts[:4]}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,where", [(2, 4), (7, 3), (33, 40), (64, 0), (64, 63), (64, 100), (65, 64), (100, 150), (129, 1), (300, 31)])
@pytest.mark.parametrize("dim", [8, 64])
def test_a_marked_key_just_inside_and_just_outside_the_window(tmp_path, dtype, window, where, dim):
    """The last query that sees the mark finds it, the next one does not: as a prompt, cut into portions at the edge, and
    decoded token by token across it."""
    d = _marked_model(str(tmp_path), dtype, "latent_attention", window=window, dim=dim)
    lm = api.load(d, dtype=dtype, max_tokens=512)
    inside, outside = where + window - 1, where + window
    T = outside + 6
    toks = [2 + (i % 13) for i in range(T)]
    toks[where] = 1
    want = _plain_logits(d, toks)
    lost = list(toks); lost[where] = 2
    miss = _plain_logits(d, lost)
    assert helpers.rel_err(miss[inside:inside + 1], want[inside:inside + 1]) > 0.05
    assert helpers.rel_err(miss[outside:outside + 1], want[outside:outside + 1]) < 1e-9
    schedules = [[(0, T)], _cuts(T, [inside, 1, 1, 2]), _cuts(T, [outside, 2]), _cuts(T, [where + 1, 3, 2, 5]),
                 [(0, max(1, inside - 3))] + [(i, i + 1) for i in range(max(1, inside - 3), T)]]
    for cuts in schedules:
        s = lm.engine.open()
        got = torch.cat([_step_all(lm, s, toks, lo, hi) for lo, hi in cuts])
        lm.engine.close(s)
        assert _close(got, want, dtype), f"cuts {cuts[:4]}"
        assert _close(got[inside:outside + 1], want[inside:outside + 1], dtype), f"edge, cuts {cuts[:4]}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_of_a_sequence(zazulix_dirs, dtype):
    """Sequences of one, two and three tokens, alone and as a batch, after the slot held a longer request."""
    d = zazulix_dirs("T", dtype)
    lm, tap = _load(d, dtype, max_tokens=256, max_seqs=3)
    V = lm.spec.vocab_size
    s = lm.engine.open()
    lm.engine.step([(s, helpers.rand_ids(90, V, 1))])
    lm.engine.close(s)
    if tap is not None:
        tap.seen.clear()
    reqs = [helpers.rand_ids(n, V, 70 + n) for n in (1, 2, 3)]
    slots = [lm.engine.open() for _ in reqs]
    lg = lm.engine.step(list(zip(slots, reqs)), [list(range(len(r))) for r in reqs])
    off = 0
    for r, s in zip(reqs, slots):
        assert _close_model(lg[off:off + len(r)], _plain_logits(d, r, tap, s), dtype)
        off += len(r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,graph", [("A", True), ("A", False), ("T", True)])
def test_long_decoding_of_a_batch(zazulix_dirs, name, dtype, graph):
    """200 single-token steps of two sequences (captured graphs or not): pages carry on, windows pass over decoded tokens,
    states are carried.  In bfloat16 the steps called from Python are held against the plain implementation and the
    captured ones against those."""
    d = zazulix_dirs(name, dtype)
    V = helpers.ZAZULIX[name]()["vocab"]
    full = [helpers.rand_ids(40 + 200, V, 3), helpers.rand_ids(3 + 200, V, 4)]
    starts = [40, 3]

    def run(lm):
        slots = [lm.engine.open(), lm.engine.open()]
        lm.engine.step([(s, f[:n]) for s, f, n in zip(slots, full, starts)])
        rows = [[], []]
        for k in range(200):
            last = lm.engine.step([(s, [f[n + k]]) for s, f, n in zip(slots, full, starts)])
            if k >= 150:
                rows[0].append(last[0:1].clone()); rows[1].append(last[1:2].clone())
        return slots, [torch.cat(r) for r in rows]
    if dtype == "float32":
        lm = api.load(d, dtype=dtype, max_tokens=1024, max_seqs=2, use_graph=graph)
        _, rows = run(lm)
        for row, f in enumerate(full):
            assert _close_model(rows[row], _plain_logits(d, f)[-50:], dtype)
        return
    lm, tap = _load(d, dtype, max_tokens=1024, max_seqs=2)
    slots, rows = run(lm)
    for row, f in enumerate(full):
        assert _close_model(rows[row], _plain_logits(d, f, tap, slots[row])[-50:], dtype)
    if graph:
        _, captured = run(api.load(d, dtype=dtype, max_tokens=1024, max_seqs=2, use_graph=True))
        for row in (0, 1):
            assert _close(captured[row], rows[row], "bfloat16")               # (grids of another size: equal up to rounding)


@pytest.mark.parametrize("seed", list(range(1, 15)))
def test_drawn_configurations_in_a_batch_and_decoding(tmp_path, seed):
    """Configurations drawn at random (sizes, head counts, windows, rotations, filters, decays, layer order, experts): a
    prompt of 200 tokens beside a short one, then six single tokens each, in both types."""
    cfg = helpers.zazulix_random_config(seed)
    d = helpers.make_zazulix_dir(cfg, str(tmp_path), seed=seed, std=0.08, edit=_sharpen)
    V = cfg["vocab"]
    a, b = helpers.rand_ids(206, V, seed), helpers.rand_ids(9, V, seed + 100)
    for dtype in ("float32", "bfloat16"):
        lm, tap = _load(d, dtype, max_tokens=512)
        sa, sb = lm.engine.open(), lm.engine.open()
        g = lm.engine.step([(sa, a[:200]), (sb, b[:3])], [list(range(200)), [0, 1, 2]])
        ga, gb = [g[:200]], [g[200:]]
        for k in range(6):
            g = lm.engine.step([(sa, [a[200 + k]]), (sb, [b[3 + k]])])
            ga.append(g[0:1]); gb.append(g[1:2])
        assert _close_model(torch.cat(ga), _plain_logits(d, a, tap, sa), dtype), f"{dtype}: {cfg}"
        assert _close_model(torch.cat(gb), _plain_logits(d, b, tap, sb), dtype), f"{dtype}: {cfg}"
        del lm


def test_greedy_generation_through_the_entry_point(zazulix_dirs):
    """``LM.generate`` (scheduler, batching, sampling, captured steps) against greedy decoding with the plain
    implementation, in 32-bit, where a choice of experts cannot fall another way; and bfloat16 generates what its own
    steps called one by one would."""
    d = zazulix_dirs("A", "float32")
    lm = api.load(d, dtype="float32", max_tokens=256)
    V = lm.spec.vocab_size
    prompts = [helpers.rand_ids(n, V, 80 + n) for n in (5, 1, 19)]
    toks, _ = lm.generate(prompts, max_new=40)                 # (more new tokens than the windows hold)
    cfg, w = plain.load(d)
    for p, row in zip(prompts, toks.tolist()):
        lg = plain.forward(cfg, w, list(p) + row)
        for i, t in enumerate(row):
            top2 = torch.topk(lg[len(p) - 1 + i], 2).values
            if float(top2[0] - top2[1]) > 1e-3:                # a near tie may fall either way
                assert t == int(lg[len(p) - 1 + i].argmax())
    d = zazulix_dirs("A", "bfloat16")
    lm = api.load(d, dtype="bfloat16", max_tokens=256)
    toks, _ = lm.generate(prompts, max_new=40)
    eager = api.load(d, dtype="bfloat16", max_tokens=256, use_graph=False)
    for p, row in zip(prompts, toks.tolist()):
        s = eager.engine.open()
        lg = eager.engine.step([(s, p)])
        for t in row:
            top2 = torch.topk(lg[0], 2).values
            if float(top2[0] - top2[1]) > 0.05 * float(lg[0].abs().max()):
                assert t == int(lg[0].argmax())
            lg = eager.engine.step([(s, [t])])


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("T", "bfloat16")])
def test_the_device_side_decode_loop_gives_the_tokens_generation_gives(zazulix_dirs, name, dtype):
    """``Engine.decode_session`` (model, greedy pick and feedback in one captured graph): states and filters are carried by
    replays that the host never sees, and its warm-up runs leave them as they were."""
    d = zazulix_dirs(name, dtype)
    lm = api.load(d, dtype=dtype, max_tokens=64 * 24, max_seqs=8)
    eng = lm.engine
    prompts = [helpers.rand_ids(n, lm.spec.vocab_size, 500 + n) for n in (5, 61, 30)]
    steps = 70
    toks, _ = lm.generate(prompts, steps)
    assert eng.cache.slots.n_held == 0 and eng.cache.pages_held() == 0
    slots = [eng.open() for _ in prompts]
    first = eng.sample(eng.step(list(zip(slots, prompts))), 0.0, 0, list(range(len(prompts))), [0] * len(prompts))
    assert first == toks[:, 0].tolist()
    sess = eng.decode_session(slots, first, steps - 1)
    sess.run(steps - 1)
    got = sess.tokens()
    sess.finish()
    assert torch.equal(got.T.long(), toks[:, 1:].long()), "the device-side loop chose other tokens than generation"
    if dtype == "float32":                                     # and the sequences go on from where the session left them
        more = eng.step([(s, [int(t)]) for s, t in zip(slots, got[-1])])
        whole = torch.stack([_plain_logits(d, list(p) + toks[i].tolist())[-1] for i, p in enumerate(prompts)])
        assert helpers.rel_err(more, whole) < TOL[dtype]
    for s in slots:
        eng.close(s)


def test_sampling_with_a_temperature_is_the_same_in_any_batch(zazulix_dirs):
    d = zazulix_dirs("A", "float32")
    lm = api.load(d, dtype="float32", max_tokens=512)
    V = lm.spec.vocab_size
    prompts = [helpers.rand_ids(n, V, 90 + n) for n in (7, 2, 33)]
    together = lm.generate_requests(prompts, 12, temperature=0.8, seed=5)
    alone = lm.generate_requests(prompts[:1], 12, temperature=0.8, seed=5)
    assert together[0].tokens == alone[0].tokens and len(set(together[0].tokens)) > 3


def test_what_the_parts_cannot_mean_is_refused():
    rt = _rt("float32")
    turn = lambda dim, variant: RotarySpec(theta=1e4, dim=dim, max_positions=99, variant=variant)
    for spec in (_diff_spec(n_heads=5), dataclasses.replace(_diff_spec(), position=turn(14, "half_partial")),
                 dataclasses.replace(_diff_spec(), position=turn(6, "interleaved")), _ret_spec(decay=(0.5,)),
                 dataclasses.replace(_ret_spec(), position=turn(18, "half_partial")), _moe_spec(group_top=0),
                 dataclasses.replace(_moe_spec(), shared=None),
                 GatedMLPSpec(hidden=8, intermediate=8, activation="clamped", limit=-1.0, names=GatedMLPNames("gate", "up", "down"))):
        cls = (FEED_FORWARDS if isinstance(spec, (GatedMLPSpec, RoutedExpertsSpec)) else MIXERS).get(spec.kind)
        w = random_weights(cls.declare(spec, "M."), 1, 0.1, dtype=torch.float32, device="cuda")
        with pytest.raises(ValueError):
            cls(spec, w, "M.", rt)


def test_the_command_line_replays_a_trace(zazulix_dirs, tmp_path):
    """``bin/trace_run`` on a Zazulix folder: whole, decoded and batched give the plain implementation's logits."""
    import json
    import subprocess
    import sys
    import numpy as np
    d = zazulix_dirs("A", "float32")
    V = helpers.ZAZULIX["A"]()["vocab"]
    a, b = helpers.rand_ids(70, V, 1), helpers.rand_ids(9, V, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []}]
    for k in range(4):
        steps.append({"step": k + 1, "entries": [{"id": "a", "tokens": [a[66 + k]], "want": [0]}, {"id": "b", "tokens": [b[5 + k]], "want": [0] if k == 3 else []}],
                      "end": ["a", "b"] if k == 3 else []})
    steps.append({"step": 5, "entries": [{"id": "c", "tokens": b, "want": [8]}], "end": ["c"]})
    p = subprocess.run([sys.executable, os.path.join(helpers.ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-3000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(6)]
    read = lambda i: torch.from_numpy(np.fromfile(os.path.join(str(tmp_path), f"{i}.f32"), dtype="<f4").reshape(-1, V).copy())
    wa, wb = _plain_logits(d, a), _plain_logits(d, b)
    assert helpers.rel_err(read(0), torch.stack([wa[0], wa[65], wb[4]])) < TOL["float32"]
    assert helpers.rel_err(read(4), torch.stack([wa[69], wb[8]])) < TOL["float32"]
    assert helpers.rel_err(read(5), wb[8:9]) < TOL["float32"]
    assert helpers.rel_err(read(5), read(4)[1:2]) < 1e-5
