"""The Tosodra decoder on the GPU against the plain implementation (``plain_tosodra.py``): every mechanism alone, then
whole models through the engine: prompts, token-by-token decoding, portions, unequal batches, slots and pages used
again, marked keys far away, at page borders and at a chunk's edges, first tokens, long decoding, drawn configurations,
greedy generation, and the trace replay program."""

import dataclasses
import os

import pytest
import torch

import helpers
import plain_tosodra as plain
from idempotent_llm_b200 import api
from idempotent_llm_b200.cache import SequenceCache
from idempotent_llm_b200.config import GatedMLPSpec, HeadAttentionSpec, LatentAttentionSpec, RotarySpec, RoutedExpertsSpec
from idempotent_llm_b200.config.specs import GatedMLPNames
from idempotent_llm_b200.engine.batch import context_from_packed, pack_step_host
from idempotent_llm_b200.parts import FEED_FORWARDS, MIXERS, Runtime
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


def _run_mixer(part, cls, spec, x, cuts, dtype, pages=24):
    """The part alone over ``x`` cut as ``cuts`` says, in a cache of its own; the rows one after another."""
    cache = SequenceCache({0: cls.cache_need(spec)}, 64 * pages, DT[dtype], "cuda:0", max_seqs=2)
    cache.alloc_slot()
    slot = cache.alloc_slot()
    outs = []
    for lo, hi in cuts:
        cache.reserve([(slot, hi)]); cache.flush()
        outs.append(part.forward(x[lo:hi].contiguous().cuda(), _ctx([slot], [lo], [hi - lo]), cache.view(0), cache.state_of(0), True).sum(0))
        cache.set_length(slot, hi)
    return torch.cat(outs)


# ----------------------------------------------------------------------------------- the attention of sigmoids, alone
def _att_spec(rot=8, base=3000.0, **kw):
    d = dict(hidden=40, n_heads=6, n_kv_heads=2, key_dim=24, value_dim=16, softmax_scale=0.4, eps=1e-5, bias_in=True,
             qk_norm_over="projection", value_norm=True, channel_gate=True, weights="sigmoid", chunk=37)
    d.update(kw)
    if rot:
        d["position"] = RotarySpec(theta=base, dim=rot, max_positions=1 << 20, variant="interleaved")
    return HeadAttentionSpec(**d)


def _plain_att(x, w, s, p):
    m = dict(heads=s.n_heads, kv_heads=s.n_kv_heads, dim=s.key_dim, vdim=s.value_dim, scale=s.softmax_scale,
             rot=dict(base=s.position.theta if s.position else 1.0, dims=s.position.dim if s.position else 0),
             mask=dict(size=s.chunk) if s.chunk else None)
    return plain.chunked_mixer(x, w, p, m, s.eps)


def _att_weights(cls, spec, dtype, seed):
    """Random weights with sharp scores (large query norm weights) and biases that keep most weights small."""
    w = random_weights(cls.declare(spec, "M."), seed, 0.25, dtype=DT[dtype], device="cuda")
    w["M.q.norm"] = (w["M.q.norm"].float() * 2.0).to(DT[dtype])
    w["M.pb"] = (w["M.pb"].float() - 2.0).to(DT[dtype])
    return w


ATT_VARIANTS = {
    "grouped": lambda: _att_spec(),
    # chunks of one key, of a page, of a page and one, of less than a block of 32 keys; none at all
    "chunk_1": lambda: _att_spec(chunk=1),
    "chunk_64": lambda: _att_spec(chunk=64, n_kv_heads=1),
    "chunk_65": lambda: _att_spec(chunk=65, value_dim=40),
    "chunk_9": lambda: _att_spec(chunk=9, n_kv_heads=6),
    "no_chunk": lambda: _att_spec(chunk=None, rot=24),
    # one head, odd sizes, nothing turned; two dims turned
    "one_head": lambda: _att_spec(n_heads=1, n_kv_heads=1, key_dim=10, value_dim=7, rot=0),
    "rot_2": lambda: _att_spec(n_heads=3, n_kv_heads=3, key_dim=18, value_dim=24, rot=2, hidden=36),
    # head sizes the tensor cores have
    "tc_64": lambda: _att_spec(n_heads=4, n_kv_heads=2, key_dim=64, value_dim=64, softmax_scale=0.2, chunk=100, rot=16),
    "tc_128_long": lambda: _att_spec(n_heads=2, n_kv_heads=1, key_dim=128, value_dim=128, softmax_scale=0.12, chunk=700, rot=128),
    "tc_64_sixteen": lambda: _att_spec(n_heads=16, n_kv_heads=1, key_dim=64, value_dim=64, softmax_scale=0.2, chunk=128, rot=64),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(ATT_VARIANTS))
def test_the_attention_alone_prompt_then_portions_then_single_tokens(dtype, variant):
    spec = ATT_VARIANTS[variant]()
    rt = _rt(dtype)
    cls = MIXERS.get(spec.kind)
    w = _att_weights(cls, spec, dtype, 5)
    part = cls(spec, w, "M.", rt)
    T, pre = (1500, 1405) if variant.endswith("long") else (150, 125)
    x = (torch.randn(T, spec.hidden, generator=torch.Generator().manual_seed(3)) * 1.5).to(DT[dtype])
    ref = _plain_att(x.double(), _w64(w), spec, "M.")
    whole = _run_mixer(part, cls, spec, x, [(0, T)], dtype)
    cut = _run_mixer(part, cls, spec, x, [(0, 70), (70, 72), (72, pre)] + [(i, i + 1) for i in range(pre, T)], dtype)
    assert helpers.rel_err(whole, ref) < TOL[dtype] and helpers.rel_err(cut, ref) < TOL[dtype]
    if variant.startswith("tc") or dtype == "float32":
        assert torch.equal(whole, cut), "a row's bits depend on how its sequence was cut"


@pytest.mark.parametrize("shape", [(64, 8, 1, 600), (128, 4, 2, 1100), (64, 4, 1, 64), (64, 2, 2, 65), (128, 2, 2, None), (64, 6, 2, 513)])
def test_sigmoids_and_chunks_on_the_tensor_cores_against_the_general_kernel(shape):
    """bfloat16 with head sizes of 64 and 128 runs on the tensor cores; the general kernel is the witness.  Two unequal
    sequences in the same steps: a long prompt (tiles shared by several blocks), a portion behind it, single tokens, and
    portions of a few tokens whose rows lie on both sides of a chunk's edge."""
    hd, H, G, chunk = shape
    spec = _att_spec(hidden=32, n_heads=H, n_kv_heads=G, key_dim=hd, value_dim=hd, softmax_scale=hd ** -0.5, chunk=chunk, rot=32)
    cls = MIXERS.get(spec.kind)
    w = _att_weights(cls, spec, "bfloat16", 9)
    lens = (2900, 1500)
    x = [(torch.randn(n, 32, generator=torch.Generator().manual_seed(3 + n)) * 1.5).to(torch.bfloat16).cuda() for n in lens]
    outs = {}
    for impl in ("generic", "tcgen05", "tcgen05 without the kernel for few rows"):
        rt = _rt("bfloat16")
        rt.kernels.attention_impl = impl.split()[0]
        few = rt.kernels.attention_tc_few_rows(not impl.endswith("rows"))
        calls, inner = [], rt.kernels.attention_tc
        rt.kernels.attention_tc = lambda *a, _f=inner, **k: (calls.append(1), _f(*a, **k))[1]
        part = cls(spec, w, "M.", rt)
        cache = SequenceCache({0: cls.cache_need(spec)}, 64 * 80, torch.bfloat16, "cuda:0", max_seqs=2)
        slots = [cache.alloc_slot(), cache.alloc_slot()]
        got, at = [[], []], [0, 0]
        steps = [(2497, 1200), (383, 290)] + [(1, 1)] * 5 + [(5, 0), (2, 3), (8, 2)]
        for step in steps:
            live = [i for i in (0, 1) if step[i]]
            hi = [at[i] + step[i] for i in live]
            cache.reserve([(slots[i], h) for i, h in zip(live, hi)]); cache.flush()
            ctx = _ctx([slots[i] for i in live], [at[i] for i in live], [step[i] for i in live])
            y = part.forward(torch.cat([x[i][at[i]:h] for i, h in zip(live, hi)]), ctx, cache.view(0), None, True).sum(0)
            off = 0
            for i, h in zip(live, hi):
                got[i].append(y[off:off + step[i]]); off += step[i]
                cache.set_length(slots[i], h); at[i] = h
        rt.kernels.attention_tc_few_rows(few)
        assert rt.kernels.attention_tc_status() == 0 and (len(calls) == len(steps)) == impl.startswith("tcgen05")
        outs[impl] = [torch.cat(g) for g in got]
    for i in (0, 1):
        ref = _plain_att(x[i][:outs["generic"][i].shape[0]].double().cpu(), _w64(w), spec, "M.")
        assert helpers.rel_err(outs["generic"][i], ref) < TOL["bfloat16"]
        assert helpers.rel_err(outs["tcgen05"][i], ref) < TOL["bfloat16"]
        assert helpers.rel_err(outs["tcgen05"][i], outs["generic"][i]) < 2e-2
        assert torch.equal(outs["tcgen05"][i], outs["tcgen05 without the kernel for few rows"][i])


@pytest.mark.parametrize("hd,dtype", [(64, "bfloat16"), (128, "bfloat16"), (24, "bfloat16"), (24, "float32")])
def test_chunks_go_with_a_softmax_too(hd, dtype):
    """The chunk is an option beside the sigmoids: a softmax over the keys of the query's chunk, with a sink, in prompts,
    few rows and single tokens; the same bits however the sequence is cut."""
    spec = _att_spec(n_heads=4, n_kv_heads=2, key_dim=hd, value_dim=hd, chunk=90, weights="softmax", sink=True, qk_norm_over="head",
                     value_norm=False, bias_in=False)
    cls = MIXERS.get(spec.kind)
    rt = _rt(dtype)
    w = random_weights(cls.declare(spec, "M."), 4, 0.25, dtype=DT[dtype], device="cuda")
    part = cls(spec, w, "M.", rt)
    T = 700
    x = (torch.randn(T, spec.hidden, generator=torch.Generator().manual_seed(8)) * 1.5).to(DT[dtype])
    W = _w64(w)
    h = x.double()
    q = plain.unit_rms((h @ W["M.q"].T).view(T, 4, hd), spec.eps, W["M.q.norm"])
    k = plain.unit_rms((h @ W["M.k"].T).view(T, 2, hd), spec.eps, W["M.k.norm"])
    v = (h @ W["M.v"].T).view(T, 2, hd)
    pos = torch.arange(T)
    q, k = plain.turn_neighbours(q, pos, 8, 3000.0), plain.turn_neighbours(k, pos, 8, 3000.0)
    seen, o = plain.chunk_mask(T, 90), torch.zeros(T, 4, hd, dtype=torch.float64)
    for i in range(4):
        s = ((q[:, i] @ k[:, i // 2].T) * spec.softmax_scale).masked_fill(~seen, float("-inf"))
        both = torch.cat([s, W["M.sink"][i].expand(T, 1)], dim=1)
        o[:, i] = torch.softmax(both, dim=-1)[:, :T] @ v[:, i // 2]
    ref = (o.reshape(T, -1) * torch.sigmoid(h @ W["M.g"].T)) @ W["M.o"].T
    whole = _run_mixer(part, cls, spec, x, [(0, T)], dtype)
    cut = _run_mixer(part, cls, spec, x, [(0, 600), (600, 603), (603, 660)] + [(i, i + 1) for i in range(660, T)], dtype)
    assert helpers.rel_err(whole, ref) < TOL[dtype] and torch.equal(whole, cut)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_heads_number_moves_its_weights(dtype):
    """A number far below every score leaves nothing of the values; one far above makes every visible key's weight 1:
    the plain sum of the values of the chunk."""
    spec = _att_spec(rot=0)
    rt = _rt(dtype)
    cls = MIXERS.get(spec.kind)
    w = _att_weights(cls, spec, dtype, 6)
    x = (torch.randn(60, spec.hidden, generator=torch.Generator().manual_seed(4)) * 1.5).to(DT[dtype])
    out = {}
    for name, value in (("high", 60.0), ("low", -60.0)):
        w["M.pb"] = torch.full_like(w["M.pb"], value)
        out[name] = _run_mixer(cls(spec, w, "M.", rt), cls, spec, x, [(0, 60)], dtype)
    W, h = _w64(w), x.double()
    v = plain.unit_rms((h @ W["M.v"].T + W["M.v.b"]).view(60, 2, 16), spec.eps)
    sums = torch.einsum("tj,jgd->tgd", plain.chunk_mask(60, 37).double(), v)
    o = sums[:, [0, 0, 0, 1, 1, 1]].reshape(60, -1) * torch.sigmoid(h @ W["M.g"].T)
    assert helpers.rel_err(out["high"], o @ W["M.o"].T) < TOL[dtype]
    assert float(out["low"].abs().max()) < 1e-9 * float(out["high"].abs().max())


# ----------------------------------------------------------------------------------- the latent attention, alone
def _latent_spec(rot=None, base=3e4, **kw):
    d = dict(hidden=40, n_heads=3, plain_dim=16, rot_dim=8, value_dim=24, kv_rank=40, softmax_scale=0.3, eps=1e-5)
    d.update(kw)
    dims = d["rot_dim"] if rot is None else rot
    return LatentAttentionSpec(position=RotarySpec(theta=base, dim=dims, max_positions=1 << 20, variant="half_partial"), **d)


LATENT_VARIANTS = {
    "three_heads": lambda: _latent_spec(),
    "one_head": lambda: _latent_spec(n_heads=1, plain_dim=8, rot_dim=2, value_dim=8, kv_rank=8),
    "odd": lambda: _latent_spec(n_heads=5, plain_dim=6, rot_dim=10, value_dim=10, kv_rank=22, hidden=20),
    "part_turned": lambda: _latent_spec(rot_dim=12, rot=6),
    "fragments_64": lambda: _latent_spec(n_heads=4, plain_dim=48, rot_dim=16, value_dim=64, kv_rank=64, softmax_scale=0.15),
    "fragments_128": lambda: _latent_spec(n_heads=20, plain_dim=96, rot_dim=32, value_dim=128, kv_rank=160, softmax_scale=0.1),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(LATENT_VARIANTS))
def test_the_latent_attention_alone_turned_by_halves(dtype, variant):
    spec = LATENT_VARIANTS[variant]()
    rt = _rt(dtype)
    cls = MIXERS.get(spec.kind)
    w = random_weights(cls.declare(spec, "M."), 5, 0.25, dtype=DT[dtype], device="cuda")
    part = cls(spec, w, "M.", rt)
    T, pre = 330, 300
    x = (torch.randn(T, spec.hidden, generator=torch.Generator().manual_seed(3)) * 1.5).to(DT[dtype])
    m = dict(heads=spec.n_heads, dim=spec.plain_dim, rot_dim=spec.rot_dim, vdim=spec.value_dim, kv_rank=spec.kv_rank,
             scale=spec.softmax_scale, rot=dict(base=spec.position.theta, dims=spec.position.dim))
    ref = plain.latent_mixer(x.double(), _w64(w), "M.", m, spec.eps)
    for cuts in ([(0, T)], [(0, 64), (64, 66), (66, pre)] + [(i, i + 1) for i in range(pre, T)], [(i, i + 1) for i in range(T)][:40]):
        got = _run_mixer(part, cls, spec, x, cuts, dtype)
        assert _close(got, ref[:got.shape[0]], dtype), f"cuts {cuts[:3]}"


# ----------------------------------------------------------------------------------- router and experts, alone
@pytest.mark.parametrize("E,top", [(6, 2), (1, 1), (40, 1), (7, 7), (96, 8), (2, 1)])
def test_the_router_of_sigmoids_against_plain(E, top):
    """Chosen by the logits (sigmoids of large logits round to 1 alike), weights the sigmoids as they are."""
    K = _rt("float32").kernels
    z = (torch.randn(300, E, generator=torch.Generator().manual_seed(E * 7 + top)) * 2.0)
    z[100:] *= 20.0                                                   # logits beyond where a 32-bit sigmoid tells them apart
    chosen, weight = K.route(z.cuda(), None, top, 1, 1, 1.0, sigmoid=True, renorm=False)
    want = z.double().topk(top, dim=-1).indices
    assert torch.equal(chosen.cpu().long(), want)
    assert helpers.rel_err(weight, torch.sigmoid(z.double()).gather(1, want)) < 1e-5
    # the options apart: renormalized sigmoids, a correction, softmax weights left as they are
    _, weight = K.route(z.cuda(), None, top, 1, 1, 1.5, sigmoid=True, renorm=True)
    s = torch.sigmoid(z.double()).gather(1, want)
    assert helpers.rel_err(weight, s / (s.sum(-1, keepdim=True) + 1e-20) * 1.5) < 1e-5
    corr = torch.randn(E, generator=torch.Generator().manual_seed(1)) * 0.2
    chosen, weight = K.route(z[:100].cuda(), corr.cuda(), top, 1, 1, 1.0, sigmoid=True, renorm=False)
    want = (torch.sigmoid(z[:100].double()) + corr.double()).topk(top, dim=-1).indices
    assert torch.equal(chosen.cpu().long(), want)
    _, weight = K.route(z[:100].cuda(), None, top, 1, 1, 1.0, sigmoid=False, renorm=False)
    assert helpers.rel_err(weight, torch.softmax(z[:100].double(), -1).topk(top, dim=-1).values) < 1e-5


def _moe_spec(shared=40, **kw):
    d = dict(hidden=32, intermediate=24, n_experts=6, top=3, scores="sigmoid", renormalize=False, weight_on="input", correction=None)
    d.update(kw)
    if shared:
        d["shared"] = GatedMLPSpec(hidden=d["hidden"], intermediate=shared, names=GatedMLPNames("shared.gate", "shared.up", "shared.down"))
    return RoutedExpertsSpec(**d)


MOE_VARIANTS = {
    "shared": lambda: _moe_spec(),
    "one_of_many": lambda: _moe_spec(n_experts=24, top=1),
    "one_of_one": lambda: _moe_spec(n_experts=1, top=1, shared=None),
    "off_borders": lambda: _moe_spec(hidden=20, intermediate=12, n_experts=5, top=2, shared=28),
    "wide": lambda: _moe_spec(hidden=256, intermediate=192, n_experts=8, top=2, shared=64),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("variant", sorted(MOE_VARIANTS))
def test_experts_weighed_at_their_input_in_steps_of_every_size(dtype, variant):
    """3 tokens (every pair streams its expert), 30 and 100 (expert by expert, or every expert over all tokens), 300 and
    1500 (rows grouped by expert on the host), and 300 without the host's help (a captured step's way): the same sums.
    The weights lie between a fifth and one, so a weight on the output instead would show."""
    spec = MOE_VARIANTS[variant]()
    rt = _rt(dtype)
    cls = FEED_FORWARDS.get(spec.kind)
    w = random_weights(cls.declare(spec, "F."), 11, 0.2 if spec.hidden < 200 else 0.1, dtype=DT[dtype], device="cuda")
    w["F.router"] = (w["F.router"].float() * 3.0).to(DT[dtype])
    part = cls(spec, w, "F.", rt)
    w64 = _w64(w)
    c = dict(kind="moe", expert=dict(ff=spec.intermediate), shared=dict(ff=1) if spec.shared else None,
             router=dict(experts=spec.n_experts, top=spec.top))
    for n, host in ((3, True), (30, True), (100, True), (300, True), (300, False), (1500, True)):
        x = (torch.randn(n, spec.hidden, generator=torch.Generator().manual_seed(n)) * 1.3).to(DT[dtype])
        ctx = _ctx([0], [0], [n])
        if not host:
            ctx.host_tokens = None
        got = part.forward(x.cuda(), ctx).sum(0)
        chosen, weight = part.route(x.cuda())
        forced = None if dtype == "float32" else chosen.cpu()
        want = plain.experts_ff(x.double(), w64, "F.", c, forced)
        assert _close(got, want, dtype), f"{n} tokens, host {host}"
        own, own_w = plain.route(x.double() @ w64["F.router"].T, spec.top)
        if dtype == "float32":                                           # the choices themselves
            assert torch.equal(chosen.cpu().long(), own) and helpers.rel_err(weight, own_w) < 1e-4
        else:
            assert _close_rows(got, plain.experts_ff(x.double(), w64, "F.", c), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("weight_on", ["input", "output"])
@pytest.mark.parametrize("hidden,ff,E,top", [(32, 24, 6, 3), (264, 776, 5, 4), (20, 12, 3, 1), (1032, 520, 4, 2)])
def test_every_way_a_step_of_few_tokens_runs_its_experts(dtype, weight_on, hidden, ff, E, top):
    """The same step pair by pair, expert by expert and every expert over all tokens, whatever the step would take by
    itself; rows of lengths that are whole and not whole multiples of a warp's pieces."""
    spec = _moe_spec(hidden=hidden, intermediate=ff, n_experts=E, top=top, shared=None, weight_on=weight_on)
    rt = _rt(dtype)
    cls = FEED_FORWARDS.get(spec.kind)
    w = random_weights(cls.declare(spec, "F."), 12, 2.0 * hidden ** -0.5, dtype=DT[dtype], device="cuda")
    part = cls(spec, w, "F.", rt)
    w64 = _w64(w)
    c = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=E, top=top))
    for n in (1, 21):
        x = torch.randn(n, hidden, generator=torch.Generator().manual_seed(n)).to(DT[dtype])
        chosen, weight = part.route(x.cuda())
        if weight_on == "input":
            want = plain.experts_ff(x.double(), w64, "F.", c, chosen.cpu())
        else:
            want = torch.stack([sum(weight[t, k].double().cpu() * plain.gated_ff(x.double()[t:t + 1], w64, f"F.e{int(chosen[t, k])}.")[0]
                                    for k in range(top)) for t in range(n)])
        for dense_from, major_from in ((1 << 30, 1 << 30), (1 << 30, 0), (0, 0)):
            part.dense_from, rt.kernels.EXPERT_MAJOR_FROM = dense_from, major_from
            assert _close(part.forward(x.cuda(), _ctx([0], [0], [n])).sum(0), want, dtype), f"{n} tokens, {dense_from}, {major_from}"


def test_the_products_epilogue_takes_a_factor_per_row():
    """The gated product with a factor per row, in every kernel it may run on (few tokens, many): gate and up times the
    factor before the activation; factors of 1 change no bit."""
    K = _rt("bfloat16").kernels
    g = torch.Generator().manual_seed(2)
    for M, Kd, inter in ((1, 64, 24), (40, 128, 96), (128, 256, 200), (300, 256, 128), (2100, 512, 320)):
        x = torch.randn(M, Kd, generator=g).bfloat16().cuda()
        gate, up = (torch.randn(inter, Kd, generator=g).mul(0.1).bfloat16().cuda() for _ in range(2))
        wt = K.tile_gate_up(gate, up)
        rw = (torch.rand(M, generator=g) + 0.2).cuda()
        y, ones, none = (torch.empty(M, inter, dtype=torch.bfloat16, device="cuda") for _ in range(3))
        for out, factor in ((y, rw), (ones, torch.ones_like(rw)), (none, None)):
            K._check(K.lib.idm_gemm_bf16_gated_rows(x.data_ptr(), wt.data_ptr(), out.data_ptr(), M, inter, Kd, 0,
                                                    None if factor is None else factor.data_ptr(), K._stream()))
        a, b = (rw.double()[:, None] * (x.double() @ t.double().T) for t in (gate, up))
        assert helpers.rel_err(y, plain.silu(a) * b) < 1e-2 and torch.equal(ones, none)
        assert K.gemm_status() == 0


# ----------------------------------------------------------------------------------- the norm of the sum, alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden,groups", [(18, 2), (20, 5), (96, 1), (96, 8), (1024, 4), (1028, 1), (2048, 1), (2048, 2), (4096, 1),
                                           (4096, 4), (5200, 1), (5202, 3), (6, 6)])
def test_the_norm_of_stream_and_output_together(dtype, hidden, groups):
    K = _rt(dtype).kernels
    g = torch.Generator().manual_seed(hidden)
    w = (torch.randn(hidden, generator=g) + 1.0).cuda()
    scale = torch.linspace(0.2, 30.0, groups).repeat_interleave(hidden // groups)      # parts of unlike sizes: each its own root
    tol = 1e-5 if dtype == "float32" else 1e-2
    for n in (3, 70):
        h0 = (torch.randn(n, hidden, generator=g) * scale).cuda()
        y = (torch.randn(1, n, hidden, generator=g) * scale).cuda()
        h = h0.clone()
        x = K.sum_norm(h, y, 2.5, w, 1e-5, groups)
        want = plain.grouped_norm(2.5 * h0.double().cpu() + y[0].double().cpu(), groups, 1e-5, w.double().cpu())
        assert helpers.rel_err(h, want) < 1e-5 and helpers.rel_err(x, want) < tol
        h = h0.clone()
        K.sum_norm(h, torch.cat([y, y]), -0.5, w, 1e-5, groups, cast=False)            # two partial sums, a negative constant
        assert helpers.rel_err(h, plain.grouped_norm(-0.5 * h0.double().cpu() + 2 * y[0].double().cpu(), groups, 1e-5, w.double().cpu())) < 1e-5
        rows = torch.tensor([n - 1, 0], dtype=torch.int32).cuda()
        h = h0.clone()
        got = K.grouped_rmsnorm(h, None, w, 1e-5, groups, rows=rows)
        assert torch.equal(h, h0)                                                       # the stream is left alone
        assert helpers.rel_err(got, plain.grouped_norm(h0.double().cpu()[[n - 1, 0]], groups, 1e-5, w.double().cpu())) < tol
        got = K.grouped_rmsnorm(h, y, w, 1e-5, groups)
        assert helpers.rel_err(got, plain.grouped_norm((h0 + y[0]).double().cpu(), groups, 1e-5, w.double().cpu())) < tol
    y = torch.randn(1, 70, hidden, generator=g).cuda()
    a, c = torch.ones(70, hidden).cuda(), torch.ones(3, hidden).cuda()
    K.sum_norm(a, y, 1.5, w, 1e-5, groups)
    K.sum_norm(c, y[:, :3].contiguous(), 1.5, w, 1e-5, groups)
    assert torch.equal(a[:3], c), "a row's bits depend on how many rows the step holds"


# ----------------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def tosodra_dirs(tmp_path_factory):
    made = {}

    def get(name, dtype="bfloat16", seed=1):
        key = (name, dtype, seed)
        if key not in made:
            d = str(tmp_path_factory.mktemp(f"tosodra-{name}-{dtype}-{seed}"))
            helpers.make_tosodra_dir(helpers.TOSODRA[name](), d, seed=seed, dtype=DT[dtype], edit=_sharpen)
            made[key] = d
        return made[key]
    return get


def _sharpen(n, t):
    """Sharper attention (single far keys carry real weight) and decisive routers."""
    if n.endswith("q.norm"):
        return (t.float() * 2.0).to(t.dtype)
    if n.endswith("mix.pb"):
        return (t.float() - 2.0).to(t.dtype)
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
            chosen, weight = inner(x)
            rows, xs, off = chosen.cpu(), x.double().cpu(), 0
            for slot, n in self.layout:
                self.seen.setdefault(slot, {}).setdefault(li, []).append((rows[off:off + n], xs[off:off + n]))
                off += n
            return chosen, weight
        return route

    def routes(self, slot, cfg, w):
        """{layer: [T, top]} of a sequence, checked against the plain router on the same inputs."""
        out = {}
        for li, parts in self.seen.pop(slot, {}).items():
            chosen, x = torch.cat([p[0] for p in parts]).long(), torch.cat([p[1] for p in parts])
            out[li] = chosen
            z, top = x @ w[f"l{li}.mlp.router"].T, cfg["layers"][li]["mlp"]["router"]["top"]
            own, margin = plain.route(z, top)[0], plain.route_margin(z, top)
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
    """Whole models.  32-bit: as everywhere.  bfloat16: row by row; the worst row in twenty is left out of the root mean
    square, which is held to the type's tolerance, and no row may be lost (a norm divides a short vector's rounding by
    its own length)."""
    if dtype == "float32":
        return _close(got, want, dtype)
    g, w = got.detach().double().cpu(), want.detach().double().cpu()
    rows = (g - w).pow(2).mean(-1) / w.pow(2).mean()
    kept = rows.sort().values[:rows.numel() - max(2, rows.numel() // 20)] if rows.numel() > 4 else rows
    return float(kept.mean().sqrt()) < TOL[dtype] and float(rows.max().sqrt()) < 0.5


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
def test_whole_prompt_and_every_layer_against_plain(tosodra_dirs, name, dtype):
    d = tosodra_dirs(name, dtype)
    lm, tap = _load(d, dtype, max_tokens=512)
    toks = helpers.rand_ids(190, lm.spec.vocab_size, 5)
    seen = []

    def recording(inner):
        def forward(h, *a, **k):
            out = inner(h, *a, **k)
            seen.append(out[0].clone())                  # (what such a layer hands on adds nothing)
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
def test_token_by_token_from_the_first_token_equals_the_prompt(tosodra_dirs, name, dtype):
    d = tosodra_dirs(name, dtype)
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
        assert helpers.rel_err(one, whole) < TOL[dtype] / 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,sizes", [("A", [2]), ("A", [3, 2, 64, 1, 2]), ("A", [20, 13, 20, 2, 1, 64]), ("T", [64, 65]), ("T", [63, 2, 128, 2])])
def test_portions_of_several_sizes(tosodra_dirs, name, dtype, sizes):
    d = tosodra_dirs(name, dtype)
    lm, tap = _load(d, dtype, max_tokens=512)
    toks = helpers.rand_ids(45 if sizes == [2] else 200, lm.spec.vocab_size, 21)
    s = lm.engine.open()
    got = torch.cat([_step_all(lm, s, toks, lo, hi) for lo, hi in _cuts(len(toks), sizes)])
    assert _close_model(got, _plain_logits(d, toks, tap, s), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "T"])
def test_unequal_batch_against_each_alone_with_slots_and_pages_used_again(tosodra_dirs, name, dtype):
    """Three requests of unlike lengths start in one step and decode together, the short ones leaving early; then
    the slots and pages they gave back serve other requests."""
    d = tosodra_dirs(name, dtype)
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


def _marked_model(tmp, dtype, kind, chunk=None, dim=8):
    """A one-layer model whose first head looks for ONE key.  The stream's first coordinate is -1 for every token but
    token 1 (+1); the head's query is minus that coordinate and its key plus it, in a dim that is not turned, so that any
    other token's query scores far above everything on the marked key and far below on every other.  ``attention``: the
    heads' numbers of -8 make the weights of unmarked keys vanish.  ``latent_attention``: the softmax is the marked key's
    alone; without it, it is spread over all keys.  No feed-forward."""
    if kind == "attention":
        layer = helpers.tosodra_attention(heads=2, kv_heads=1, dim=dim, vdim=dim, scale=24.0 / dim, chunk=chunk, rot_dims=2, mlp=None)
    else:
        layer = helpers.tosodra_latent(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=32, scale=1.0, mlp=None)
    cfg = helpers.tosodra_config([layer], vocab=16, width=16, groups=2, alpha=1.0, emb_scale=1.0)
    p = "l0.mix."

    def edit(n, t):
        t = t.float()
        if n == "embed":
            t[:, 0] = -1.0; t[1, 0] = 1.0
        elif kind == "attention" and n in (p + "q", p + "k"):
            t = torch.zeros_like(t); t[4, 0] = -1.0 if n.endswith("q") else 1.0
        elif n in (p + "q.b", p + "k.b"):
            t = torch.zeros_like(t)
        elif n in (p + "q.norm", p + "k.norm"):
            t = torch.ones_like(t)
        elif n == p + "pb":
            t = torch.full_like(t, -8.0)
        elif kind == "latent_attention" and n == p + "q":
            t = torch.zeros_like(t); t[0, 0] = -10.0
        elif n == p + "dkv":
            t[0] = 0.0; t[0, 0] = 1.0
        elif n == p + "dkv.norm":
            t = torch.ones_like(t)
        elif n == p + "uk":
            t = torch.zeros_like(t); t[0, 0] = 4.0
        elif n in (p + "o", p + "uv", p + "v"):
            t = t * 4.0                                       # (the mixer's output weighs against the stream)
        return t.to(DT[dtype])
    return helpers.make_tosodra_dir(cfg, tmp, seed=3, dtype=DT[dtype], edit=edit)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("where", [0, 63, 64, 65, 127, 255, 300])
@pytest.mark.parametrize("kind", ["latent_attention", "attention"])
def test_one_far_key_among_hundreds_in_prompts_and_in_decoding(tmp_path, kind, dtype, where):
    """The marked token sits at a page's (or a run's) first or last place, or far back; every later query finds it, in a
    prompt, across portions and when decoding alone.  Without the mark the logits differ, so a lost key shows.  The
    attention of sigmoids has one chunk for all of it."""
    d = _marked_model(str(tmp_path), dtype, kind, chunk=400)
    lm = api.load(d, dtype=dtype, max_tokens=512)
    T = 330
    toks = [2 + (i % 13) for i in range(T)]
    toks[where] = 1
    want = _plain_logits(d, toks)
    lost = list(toks); lost[where] = 2
    assert helpers.rel_err(_plain_logits(d, lost)[-1:], want[-1:]) > 0.05        # the key matters to the last query
    portions = _cuts(T, [where + 1, 2, 250])[:3]               # up to the mark, two tokens, up to 250, the rest alone
    for cuts in ([(0, T)], portions + [(i, i + 1) for i in range(portions[-1][1], T)], [(0, 280)] + [(i, i + 1) for i in range(280, T)]):
        s = lm.engine.open()
        got = torch.cat([_step_all(lm, s, toks, lo, hi) for lo, hi in cuts])
        lm.engine.close(s)
        assert _close(got, want, dtype), f"cuts {cuts[:4]}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,where", [(2, 4), (7, 3), (7, 6), (64, 0), (64, 63), (64, 100), (65, 64), (100, 150), (129, 1), (129, 130)])
@pytest.mark.parametrize("dim", [8, 64])
def test_a_marked_key_at_the_edges_of_its_chunk(tmp_path, dtype, chunk, where, dim):
    """The chunk's last query sees the mark, the next chunk's first does not, whatever the distance; a mark at a chunk's
    first place is seen by that chunk and not by the one before.  As a prompt, cut into portions at the edge (a cut
    starts no chunk), and decoded token by token across it."""
    d = _marked_model(str(tmp_path), dtype, "attention", chunk=chunk, dim=dim)
    lm = api.load(d, dtype=dtype, max_tokens=512)
    inside, outside = where // chunk * chunk + chunk - 1, where // chunk * chunk + chunk
    T = outside + 6
    toks = [2 + (i % 13) for i in range(T)]
    toks[where] = 1
    want = _plain_logits(d, toks)
    lost = list(toks); lost[where] = 2
    miss = _plain_logits(d, lost)
    if inside != where:                                       # (a query at the mark itself looks for the other sign)
        assert helpers.rel_err(miss[inside:inside + 1], want[inside:inside + 1]) > 0.05
    assert helpers.rel_err(miss[outside:outside + 1], want[outside:outside + 1]) < 1e-9
    schedules = [[(0, T)], _cuts(T, [max(1, inside), 1, 1, 2]), _cuts(T, [outside, 2]), _cuts(T, [where + 1, 3, 2, 5]),
                 [(0, max(1, inside - 3))] + [(i, i + 1) for i in range(max(1, inside - 3), T)]]
    for cuts in schedules:
        s = lm.engine.open()
        got = torch.cat([_step_all(lm, s, toks, lo, hi) for lo, hi in cuts])
        lm.engine.close(s)
        assert _close(got, want, dtype), f"cuts {cuts[:4]}"
        assert _close(got[inside:outside + 1], want[inside:outside + 1], dtype), f"edge, cuts {cuts[:4]}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_of_a_sequence(tosodra_dirs, dtype):
    """Sequences of one, two and three tokens, alone and as a batch, after the slot held a longer request."""
    d = tosodra_dirs("T", dtype)
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
def test_long_decoding_of_a_batch(tosodra_dirs, name, dtype, graph):
    """200 single-token steps of two sequences (captured graphs or not): pages carry on and chunks pass by.  In bfloat16
    the steps called from Python are held against the plain implementation and the captured ones against those."""
    d = tosodra_dirs(name, dtype)
    V = helpers.TOSODRA[name]()["vocab"]
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
            assert helpers.rel_err(captured[row], rows[row]) < 1e-5       # the same kernels on the same numbers


@pytest.mark.parametrize("seed", list(range(1, 11)))
def test_drawn_configurations_in_a_batch_and_decoding(tmp_path, seed):
    """Configurations drawn at random (sizes, head counts, chunks, rotations, layer order, norms' parts, experts): a
    prompt of 200 tokens beside a short one, then six single tokens each, in both types."""
    cfg = helpers.tosodra_random_config(seed)
    d = helpers.make_tosodra_dir(cfg, str(tmp_path), seed=seed, std=0.08, edit=_sharpen)
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


def test_greedy_generation_through_the_entry_point(tosodra_dirs):
    """``LM.generate`` (scheduler, batching, sampling, captured steps) against greedy decoding with the plain
    implementation, in 32-bit, where a choice of experts cannot fall another way; and bfloat16 generates what its own
    steps called one by one would."""
    d = tosodra_dirs("A", "float32")
    lm = api.load(d, dtype="float32", max_tokens=256)
    V = lm.spec.vocab_size
    prompts = [helpers.rand_ids(n, V, 80 + n) for n in (5, 1, 19)]
    toks, _ = lm.generate(prompts, max_new=40)                 # (more new tokens than the chunks hold)
    cfg, w = plain.load(d)
    for p, row in zip(prompts, toks.tolist()):
        seq = list(p)
        for t in row:
            lg = plain.forward(cfg, w, seq)[-1]
            top2 = torch.topk(lg, 2).values
            if float(top2[0] - top2[1]) > 1e-3:                # a near tie may fall either way
                assert t == int(lg.argmax())
            seq.append(t)
    d = tosodra_dirs("A", "bfloat16")
    lm = api.load(d, dtype="bfloat16", max_tokens=256)
    toks, _ = lm.generate(prompts, max_new=40)
    eager = api.load(d, dtype="bfloat16", max_tokens=256, use_graph=False)
    for p, row in zip(prompts, toks.tolist()):
        s = eager.engine.open()
        lg = eager.engine.step([(s, p)])
        for t in row:
            top2 = torch.topk(lg[0], 2).values
            if float(top2[0] - top2[1]) > 0.05:
                assert t == int(lg[0].argmax())
            lg = eager.engine.step([(s, [t])])


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("T", "bfloat16")])
def test_the_device_side_decode_loop_gives_the_tokens_generation_gives(tosodra_dirs, name, dtype):
    """``Engine.decode_session`` (model, greedy pick and feedback in one captured graph): experts are chosen for a token
    that was picked on the device one replay earlier and never seen by the host."""
    d = tosodra_dirs(name, dtype)
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


def test_sampling_with_a_temperature_is_the_same_in_any_batch(tosodra_dirs):
    """Tokens drawn at temperature 0.8 for a request alone and beside two others: the same (the draw is keyed by seed,
    request and step; the logits do not depend on the batch beyond rounding, which no draw here rests on)."""
    d = tosodra_dirs("A", "float32")
    lm = api.load(d, dtype="float32", max_tokens=512)
    V = lm.spec.vocab_size
    prompts = [helpers.rand_ids(n, V, 90 + n) for n in (7, 2, 33)]
    together = lm.generate_requests(prompts, 12, temperature=0.8, seed=5)
    alone = lm.generate_requests(prompts[:1], 12, temperature=0.8, seed=5)
    assert together[0].tokens == alone[0].tokens and len(set(together[0].tokens)) > 3


def test_options_that_do_not_go_together_are_refused():
    rt = _rt("float32")
    for spec in (_att_spec(sink=True), _att_spec(window=9), _att_spec(head_gate=True), _att_spec(weights="tanh"),
                 _att_spec(qk_norm_over="row"), dataclasses.replace(_moe_spec(), n_identity=1), dataclasses.replace(_moe_spec(), scores="relu")):
        cls = (MIXERS if isinstance(spec, HeadAttentionSpec) else FEED_FORWARDS).get(spec.kind)
        w = random_weights(cls.declare(spec, "M."), 1, 0.1, dtype=torch.float32, device="cuda")
        with pytest.raises(ValueError):
            cls(spec, w, "M.", rt)


def test_the_command_line_replays_a_trace(tosodra_dirs, tmp_path):
    """``bin/trace_run`` on a Tosodra folder: whole, decoded and batched give the plain implementation's logits."""
    import json
    import subprocess
    import sys
    import numpy as np
    d = tosodra_dirs("A", "float32")
    V = helpers.TOSODRA["A"]()["vocab"]
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
