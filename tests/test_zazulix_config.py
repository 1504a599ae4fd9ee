"""Zazulix on the CPU: its configuration (every key read per layer, absent options, refusals by key), the tensors it
declares, what its parts ask of the cache, a random folder loaded by name, and the plain implementation's mechanisms
against closed forms of their own."""

import math

import pytest
import torch

import helpers
import plain_zazulix as plain
from idempotent_llm_b200.config import (ConfigError, DifferentialAttentionSpec, GatedMLPSpec, LatentAttentionSpec, LayerSpec, NormSpec,
                                        RetentionSpec, RoutedExpertsSpec, ZazulixConfig)
from idempotent_llm_b200.engine.assembly import cache_needs, declare_weights
from idempotent_llm_b200.registry import read_config, registered_architectures

F64 = torch.float64


# ----------------------------------------------------------------------------------- configuration
def test_every_key_is_read_per_layer():
    spec = ZazulixConfig.from_dict(helpers.ZAZULIX["A"]()).to_model_spec()
    assert "Zazulix" in registered_architectures()
    assert spec.tie_embeddings and spec.embed_scale == 1.0 and (spec.vocab_size, spec.hidden) == (91, 32)
    assert isinstance(spec.final_norm, NormSpec) and (spec.final_norm.eps, spec.final_norm.weight_offset, spec.final_norm.size) == (1e-5, 1.0, 32)
    assert all(isinstance(L, LayerSpec) and L.kind == "prenorm" and L.mixer_norm.weight_offset == 1.0 for L in spec.layers)
    kinds = [DifferentialAttentionSpec, RetentionSpec, LatentAttentionSpec, RetentionSpec, DifferentialAttentionSpec, LatentAttentionSpec]
    assert [type(L.mixer) for L in spec.layers] == kinds
    a = spec.layers[0].mixer
    assert (a.n_heads, a.n_kv_heads, a.key_dim, a.value_dim, a.softmax_scale, a.diff, a.conv_taps, a.eps, a.head_gate) == (4, 2, 12, 20, 0.3, 0.4, 3, 1e-5, True)
    assert (a.position.theta, a.position.dim, a.position.variant) == (5000.0, 8, "half_partial")
    assert (spec.layers[4].mixer.conv_taps, spec.layers[4].mixer.diff, spec.layers[4].mixer.position.dim) == (2, 0.1, 2)
    r = spec.layers[1].mixer
    assert (r.heads, r.key_dim, r.value_dim, r.decay, r.eps) == (3, 16, 12, (0.9, 0.995, 0.5), 1e-5)
    assert (r.position.theta, r.position.dim) == (7e3, 10) and spec.layers[3].mixer.decay == (0.97, 1.0)
    m = spec.layers[2].mixer
    assert (m.n_heads, m.plain_dim, m.rot_dim, m.value_dim, m.kv_rank, m.softmax_scale, m.window, m.gate, m.sink, m.position) == \
        (3, 16, 0, 24, 40, 0.3, 20, True, False, None)
    assert spec.layers[5].mixer.window == 70
    d = spec.layers[1].feed_forward
    assert isinstance(d, GatedMLPSpec) and (d.intermediate, d.activation, d.limit, d.slope) == (56, "clamped", 0.8, 1.702)
    ff = spec.layers[4].feed_forward
    assert isinstance(ff, RoutedExpertsSpec) and (ff.n_experts, ff.top, ff.intermediate, ff.groups, ff.groups_keep, ff.group_top) == (8, 4, 40, 2, 1, 2)
    assert (ff.scores, ff.renormalize, ff.weight_on, ff.correction, ff.scale, ff.activation) == ("sigmoid", True, "output", "mlp.correction", 1.4, "silu")
    assert ff.shared.intermediate == 16 and ff.shared.activation == "silu" and ff.shared_gate == "mlp.shared.sg"
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_norm is None


def test_declared_tensors_and_what_a_sequence_keeps():
    spec = ZazulixConfig.from_dict(helpers.ZAZULIX["A"]()).to_model_spec()
    decl = {d.name: d for d in declare_weights(spec)}
    for n, shape in {"embed": (91, 32), "final.norm": (32,), "l0.norm1": (32,), "l0.norm2": (32,), "l0.mix.q": (96, 32), "l0.mix.k": (48, 32),
                     "l0.mix.v": (40, 32), "l0.mix.q.conv": (96, 3), "l0.mix.k.conv": (48, 3), "l0.mix.v.conv": (40, 3), "l0.mix.lq1": (12,),
                     "l0.mix.lk2": (12,), "l0.mix.g": (4, 32), "l0.mix.o": (32, 80),
                     "l1.mix.q": (48, 32), "l1.mix.k": (48, 32), "l1.mix.v": (36, 32), "l1.mix.g": (36, 32), "l1.mix.o": (32, 36),
                     "l1.mlp.gate": (56, 32), "l1.mlp.down": (32, 56),
                     "l2.mix.q": (48, 32), "l2.mix.dkv": (40, 32), "l2.mix.dkv.norm": (40,), "l2.mix.uk": (48, 40), "l2.mix.uv": (72, 40),
                     "l2.mix.g": (72, 32), "l2.mix.o": (32, 72), "l2.mlp.router": (9, 32), "l2.mlp.correction": (9,),
                     "l2.mlp.e8.down": (32, 24), "l2.mlp.shared.up": (40, 32), "l2.mlp.shared.sg": (1, 32)}.items():
        assert decl[n].shape == shape, n
    for absent in ("l3.norm2", "l3.mlp.router", "l2.mix.sink", "l2.mlp.e9.gate", "l1.mix.q.conv", "l0.mix.q.norm"):
        assert absent not in decl
    assert decl["head"].optional
    needs = cache_needs(spec)
    assert needs[0].kind == "full" and needs[0].key_row() == (2, 24) and needs[0].value_row() == (2, 20) and needs[0].state_shape == (2 * 184,)
    assert needs[1].kind == "none" and needs[1].state_shape == (3 * 16 * 12,)
    assert needs[2].key_row() == (1, 40) and needs[2].value_row() == (1, 0) and needs[2].state_shape is None


def test_absent_options():
    spec = ZazulixConfig.from_dict(helpers.ZAZULIX["B"]()).to_model_spec()
    L = [x.mixer for x in spec.layers]
    assert (L[0].window, L[4].window) == (1, None)
    assert (L[1].conv_taps, L[3].conv_taps, L[1].position, L[2].position, L[3].position.dim) == (1, None, None, None, 2)
    ff = spec.layers[0].feed_forward
    assert (ff.groups, ff.groups_keep, ff.scale) == (1, 1, 1.0)
    assert spec.layers[1].feed_forward.shared is None and spec.layers[1].feed_forward.shared_gate is None
    decl = {d.name for d in declare_weights(spec)}
    assert "l1.mix.q.conv" in decl and "l3.mix.q.conv" not in decl and "l1.mlp.shared.sg" not in decl
    needs = cache_needs(spec)
    assert needs[1].state_shape is None and needs[3].state_shape is None


@pytest.mark.parametrize("edit,word", [
    (lambda c: c["layers"][0].update(type="delta"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"].update(conv=-1), "conv"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "dims"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 1.5, 0.1]), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("decay"), "decay"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"].update(limit=-2), "limit"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=-3), "size"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=7), "chosen"),
    (lambda c: c["layers"][2]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][2]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "empty"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_refusals_by_key(edit, word):
    cfg = helpers.ZAZULIX["A"]()
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        ZazulixConfig.from_dict(cfg)
    assert word in str(e.value)


def test_random_folder_round_trip(tmp_path):
    from idempotent_llm_b200.weights import load_weights
    cfg = helpers.ZAZULIX["C"]()
    d = helpers.make_zazulix_dir(cfg, str(tmp_path), seed=4)
    arch, typed = read_config(d)
    assert arch.name == "Zazulix" and typed.to_dict()["layers"] == cfg["layers"]
    w = load_weights(d, declare_weights(typed.to_model_spec()), "cpu")
    c2, w2 = plain.load(d)
    assert c2["layers"] == cfg["layers"] and set(w) == set(w2)
    assert torch.equal(w2["l1.mix.k.conv"], w["l1.mix.k.conv"].double()) and torch.equal(w2["embed"], w["embed"].double())
    assert float(w2["l0.norm1"].abs().mean()) < 0.5                          # offsets from one, not weights around one


def test_presets_name_the_design():
    from idempotent_llm_b200.config.presets import preset
    for n in ("zazulix-tiny", "zazulix-0.6b", "zazulix-8b"):
        c = preset(n)
        assert c.architecture == "Zazulix" and {L.type for L in c.layers} == {"attention", "latent_attention", "retention"}


# ----------------------------------------------------------------------------------- plain mechanisms, by hand
def test_the_norms_tensor_is_an_offset_from_one():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    r = math.sqrt(25 / 2 + 0.5)
    assert torch.allclose(plain.norm(x, 0.5, torch.tensor([0.0, -0.25], dtype=F64)), torch.tensor([[3 / r, 3 / r]], dtype=F64), atol=1e-14)


def test_rotation_is_complex_multiplication():
    g = torch.Generator().manual_seed(1)
    x, pos = torch.randn(7, 2, 10, generator=g, dtype=F64), torch.tensor([0, 1, 5, 64, 300, 1000, 31])
    f = 100.0 ** (-2.0 * torch.arange(3, dtype=F64) / 6)
    z = torch.complex(x[..., 0:3], x[..., 3:6]) * torch.exp(1j * pos[:, None].to(F64) * f[None, :])[:, None, :]
    got = plain.turn_if(x, pos, dict(base=100.0, dims=6))
    assert torch.allclose(got[..., 0:3], z.real, atol=1e-12) and torch.allclose(got[..., 3:6], z.imag, atol=1e-12)
    assert torch.equal(got[..., 6:], x[..., 6:]) and plain.turn_if(x, pos, None) is x


def test_filter_is_a_padded_correlation():
    g = torch.Generator().manual_seed(2)
    for taps in (1, 2, 5):
        u, w = torch.randn(9, 4, generator=g, dtype=F64), torch.randn(4, taps, generator=g, dtype=F64)
        padded = torch.cat([torch.zeros(taps - 1, 4, dtype=F64), u])
        want = torch.nn.functional.conv1d(padded.T[None], w[:, None], groups=4)[0].T
        assert torch.allclose(plain.short_filter(u, w), want, atol=1e-13)
    assert torch.allclose(plain.short_filter(u[:2], w), want[:2], atol=1e-13)           # shorter than the filter


def test_window_mask_by_hand():
    m = plain.window_mask(5, 2)
    assert m[0].tolist() == [True] + [False] * 4 and m[3].tolist() == [False, False, True, True, False]
    assert plain.window_mask(4, 1).tolist() == torch.eye(4).bool().tolist()
    assert plain.window_mask(4, None).tolist() == torch.tril(torch.ones(4, 4)).bool().tolist()


def test_two_maps_subtract_before_the_norm():
    lam = plain.map_weight(*(torch.tensor(v, dtype=F64) for v in ([1.0, 2.0], [0.5, 0.25], [0.0, 1.0], [3.0, 0.1])), 0.6)
    assert abs(float(lam) - (math.exp(1.0) - math.exp(0.1) + 0.6)) < 1e-12
    a1, a2 = torch.tensor([[[2.0, 0.0]]], dtype=F64), torch.tensor([[[1.0, 1.0]]], dtype=F64)
    r = math.sqrt((1.5 ** 2 + 0.5 ** 2) / 2 + 0.1)
    got = plain.difference_of_maps(a1, a2, torch.tensor(0.5, dtype=F64), 0.2, 0.1)
    assert torch.allclose(got, torch.tensor([[[1.5 / r * 0.8, -0.5 / r * 0.8]]], dtype=F64), atol=1e-14)


def test_the_maps_are_laid_out_head_by_head():
    """A head's rows are [map 1, map 2], and both maps of kv-head g serve the same query heads and values."""
    g = torch.Generator().manual_seed(4)
    m = dict(heads=4, kv_heads=2, dim=3, vdim=5, scale=0.7, diff=0.3)
    w = {n: torch.randn(*s, generator=g, dtype=F64) for n, s in dict(q=(24, 6), k=(12, 6), v=(10, 6), g=(4, 6), o=(6, 20), lq1=(3,), lk1=(3,),
                                                                    lq2=(3,), lk2=(3,)).items()}
    h = torch.randn(7, 6, generator=g, dtype=F64)
    lam = math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + 0.3
    rows = []
    for i in range(4):
        t, kv = 6, i // 2
        v = h @ w["v"][kv * 5:kv * 5 + 5].T
        a = []
        for mp in (0, 1):
            q = w["q"][i * 6 + mp * 3:i * 6 + mp * 3 + 3] @ h[t]
            s = torch.tensor([0.7 * float(q @ (w["k"][kv * 6 + mp * 3:kv * 6 + mp * 3 + 3] @ h[j])) for j in range(t + 1)], dtype=F64)
            a.append(torch.softmax(s, 0) @ v[:t + 1])
        o = a[0] - lam * a[1]
        o = o / math.sqrt(float((o * o).mean()) + 1e-5) * 0.7
        rows.append(o / (1 + math.exp(-float(w["g"][i] @ h[t]))))
    assert torch.allclose(plain.differential_mixer(h, w, "", m, 1e-5)[6], w["o"] @ torch.cat(rows), atol=1e-10)


def test_retention_is_a_decayed_sum():
    g = torch.Generator().manual_seed(5)
    q, k, v = torch.randn(8, 2, 3, generator=g, dtype=F64), torch.randn(8, 2, 3, generator=g, dtype=F64), torch.randn(8, 2, 4, generator=g, dtype=F64)
    got = plain.retain(q, k, v, torch.tensor([0.9, 0.0], dtype=F64))
    for t in range(8):
        assert torch.allclose(got[t, 0], sum(0.9 ** (t - s) * (q[t, 0] @ k[s, 0]) * v[s, 0] for s in range(t + 1)), atol=1e-12)
        assert torch.allclose(got[t, 1], (q[t, 1] @ k[t, 1]) * v[t, 1], atol=1e-12)


def test_the_dense_feed_forward_clamps_both_branches():
    w = {"gate": torch.eye(3, dtype=F64), "up": torch.eye(3, dtype=F64), "down": torch.eye(3, dtype=F64)}
    got = plain.clamped_ff(torch.tensor([[5.0, -9.0, 1.0]], dtype=F64), w, "", 2.0)[0]
    f = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert torch.allclose(got, torch.tensor([f(2.0, 2.0), f(-9.0, -2.0), f(1.0, 1.0)], dtype=F64), atol=1e-14)


def test_groups_score_by_their_best_pair():
    """Group 0 has the single largest score, group 1 the largest pair: one group kept is group 1; negative choice scores
    do not lose to closed experts; the weights are the uncorrected sigmoids."""
    s = torch.tensor([[0.9, 0.1, 0.2, 0.8, 0.7, 0.1]], dtype=F64)
    z = torch.log(s / (1 - s))
    zero = torch.zeros(6, dtype=F64)
    chosen, weight = plain.route(z, zero, dict(top=2, scale=3.0, groups=dict(count=2, keep=1)))
    assert chosen.tolist() == [[3, 4]] and torch.allclose(weight, torch.tensor([[0.8 / 1.5 * 3, 0.7 / 1.5 * 3]], dtype=F64))
    chosen, _ = plain.route(z, zero - 5.0, dict(top=3, scale=1.0, groups=dict(count=2, keep=1)))
    assert chosen.tolist() == [[3, 4, 5]]
    assert plain.route(z, zero, dict(top=1, scale=1.0))[0].tolist() == [[0]]
    corr = torch.tensor([0.0, 0.0, 1.0, 0.0, 0.0, 0.0], dtype=F64)
    chosen, weight = plain.route(z, corr, dict(top=2, scale=1.0, groups=dict(count=2, keep=1)))
    assert chosen.tolist() == [[2, 0]] and torch.allclose(weight, torch.tensor([[0.2 / 1.1, 0.9 / 1.1]], dtype=F64))


def test_the_shared_expert_is_gated():
    g = torch.Generator().manual_seed(3)
    W, E, F = 5, 4, 3
    c = dict(kind="moe", expert=dict(ff=F), router=dict(experts=E, top=2, scale=2.0), shared=dict(ff=2))
    w = {"router": torch.randn(E, W, generator=g, dtype=F64), "correction": torch.zeros(E, dtype=F64), "shared.sg": torch.randn(1, W, generator=g, dtype=F64)}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = (torch.randn(*s, generator=g, dtype=F64) for s in ((F, W), (F, W), (W, F)))
    w["shared.gate"], w["shared.up"], w["shared.down"] = (torch.randn(*s, generator=g, dtype=F64) for s in ((2, W), (2, W), (W, 2)))
    h = torch.randn(6, W, generator=g, dtype=F64)
    out = plain.experts_ff(h, w, "", c)
    for t in range(6):
        s = torch.sigmoid(w["router"] @ h[t])
        best = sorted(range(E), key=lambda e: -float(s[e]))[:2]
        want = plain.gated_ff(h[t:t + 1], w, "shared.")[0] / (1 + math.exp(-float(w["shared.sg"][0] @ h[t])))
        for e in best:
            want = want + 2.0 * s[e] / (s[best[0]] + s[best[1]]) * plain.gated_ff(h[t:t + 1], w, f"e{e}.")[0]
        assert torch.allclose(out[t], want, atol=1e-12)
