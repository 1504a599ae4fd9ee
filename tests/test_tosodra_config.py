"""Tosodra on the CPU: its configuration (every key read per layer, absent options, refusals by key), the tensors it
declares, what its parts ask of the cache, a random folder loaded by name, and the plain implementation's mechanisms
against closed forms of their own."""

import math

import pytest
import torch

import helpers
import plain_tosodra as plain
from idempotent_llm_b200.config import (ConfigError, GroupedRMSNormSpec, HeadAttentionSpec, LatentAttentionSpec, RoutedExpertsSpec,
                                        SumNormLayerSpec, TosodraConfig)
from idempotent_llm_b200.engine.assembly import cache_needs, declare_weights
from idempotent_llm_b200.registry import read_config, registered_architectures

F64 = torch.float64


# ----------------------------------------------------------------------------------- configuration
def test_every_key_is_read_per_layer():
    cfg = TosodraConfig.from_dict(helpers.TOSODRA["A"]())
    spec = cfg.to_model_spec()
    assert "Tosodra" in registered_architectures()
    assert spec.tie_embeddings and spec.embed_scale == 3.0 and (spec.vocab_size, spec.hidden) == (97, 32)
    assert isinstance(spec.final_norm, GroupedRMSNormSpec) and (spec.final_norm.groups, spec.final_norm.eps, spec.final_norm.size) == (4, 1e-5, 32)
    assert all(isinstance(L, SumNormLayerSpec) and L.alpha == 1.7 and L.mixer_norm.groups == 4 for L in spec.layers)
    assert [type(L.mixer) for L in spec.layers] == [HeadAttentionSpec, LatentAttentionSpec, HeadAttentionSpec, HeadAttentionSpec]
    a = spec.layers[0].mixer
    assert (a.n_heads, a.n_kv_heads, a.key_dim, a.value_dim, a.softmax_scale, a.chunk, a.window) == (4, 2, 24, 16, 0.3, 20, None)
    assert (a.weights, a.qk_norm_over, a.value_norm, a.channel_gate, a.bias_in, a.head_gate, a.sink) == ("sigmoid", "projection", True, True, True, False, False)
    assert (a.position.theta, a.position.dim, a.position.variant) == (5000.0, 8, "interleaved")
    assert (spec.layers[2].mixer.chunk, spec.layers[2].mixer.position.dim, spec.layers[3].mixer.n_heads) == (33, 24, 6)
    m = spec.layers[1].mixer
    assert (m.n_heads, m.plain_dim, m.rot_dim, m.value_dim, m.kv_rank, m.softmax_scale, m.eps, m.sink) == (3, 16, 8, 24, 40, 0.25, 1e-5, False)
    assert (m.position.theta, m.position.dim, m.position.variant) == (3e4, 8, "half_partial")
    ff = spec.layers[3].feed_forward
    assert isinstance(ff, RoutedExpertsSpec) and (ff.n_experts, ff.top, ff.intermediate, ff.n_identity, ff.groups) == (9, 4, 40, 0, 1)
    assert (ff.scores, ff.renormalize, ff.weight_on, ff.correction, ff.scale, ff.activation) == ("sigmoid", False, "input", None, 1.0, "silu")
    assert ff.shared.intermediate == 16 and ff.shared.activation == "silu"
    assert spec.layers[2].feed_forward is None and spec.layers[2].feed_forward_norm is None


def test_declared_tensors_and_cache_rows():
    spec = TosodraConfig.from_dict(helpers.TOSODRA["A"]()).to_model_spec()
    decl = {d.name: d for d in declare_weights(spec)}
    for n, shape in {"embed": (97, 32), "final.norm": (32,), "l0.norm1": (32,), "l0.norm2": (32,), "l0.mix.q": (96, 32), "l0.mix.q.b": (96,),
                     "l0.mix.k": (48, 32), "l0.mix.k.b": (48,), "l0.mix.v": (32, 32), "l0.mix.v.b": (32,), "l0.mix.q.norm": (96,),
                     "l0.mix.k.norm": (48,), "l0.mix.pb": (4,), "l0.mix.g": (64, 32), "l0.mix.o": (32, 64),
                     "l1.mix.q": (72, 32), "l1.mix.dkv": (48, 32), "l1.mix.dkv.norm": (40,), "l1.mix.uk": (48, 40), "l1.mix.uv": (72, 40),
                     "l1.mix.o": (32, 72), "l1.mlp.router": (6, 32), "l1.mlp.e5.down": (32, 24), "l1.mlp.shared.up": (40, 32),
                     "l3.mlp.e8.gate": (40, 32)}.items():
        assert decl[n].shape == shape, n
    for absent in ("l0.mlp.correction", "l2.norm2", "l2.mlp.router", "l0.mix.sink", "l1.mix.sink", "l1.mlp.e6.gate"):
        assert absent not in decl
    assert decl["head"].optional
    needs = cache_needs(spec)
    assert needs[0].kind == "full" and needs[0].key_row() == (2, 24) and needs[0].value_row() == (2, 16) and needs[0].state_shape is None
    assert needs[1].key_row() == (1, 48) and needs[1].value_row() == (1, 0)


def test_absent_options():
    c = helpers.TOSODRA["A"]()
    del c["embedding"], c["norm"]["groups"], c["layers"][0]["mixer"]["mask"], c["layers"][0]["mixer"]["rot"], c["layers"][0]["mlp"]["shared"]
    spec = TosodraConfig.from_dict(c).to_model_spec()
    assert spec.embed_scale == 1.0 and spec.final_norm.groups == 1
    assert spec.layers[0].mixer.chunk is None and spec.layers[0].mixer.position is None and spec.layers[0].feed_forward.shared is None


@pytest.mark.parametrize("edit,word", [
    (lambda c: c["layers"][0].update(type="delta"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-3), "size"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "dims"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "chosen"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c.pop("postln_alpha"), "postln_alpha"),
    (lambda c: c["norm"].update(groups=5), "groups"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "empty"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_refusals_by_key(edit, word):
    cfg = helpers.TOSODRA["A"]()
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        TosodraConfig.from_dict(cfg)
    assert word in str(e.value)


def test_random_folder_round_trip(tmp_path):
    from idempotent_llm_b200.weights import load_weights
    cfg = helpers.TOSODRA["C"]()
    d = helpers.make_tosodra_dir(cfg, str(tmp_path), seed=4)
    arch, typed = read_config(d)
    assert arch.name == "Tosodra" and typed.to_dict()["layers"] == cfg["layers"]
    w = load_weights(d, declare_weights(typed.to_model_spec()), "cpu")
    c2, w2 = plain.load(d)
    assert c2["layers"] == cfg["layers"] and set(w) == set(w2)
    assert torch.equal(w2["l0.mix.pb"], w["l0.mix.pb"].double()) and torch.equal(w2["embed"], w["embed"].double())


def test_presets_name_the_design():
    from idempotent_llm_b200.config.presets import preset
    for n in ("tosodra-tiny", "tosodra-0.6b", "tosodra-8b"):
        c = preset(n)
        assert c.architecture == "Tosodra" and {L.type for L in c.layers} == {"attention", "latent_attention"}


# ----------------------------------------------------------------------------------- plain mechanisms, by hand
def test_grouped_norm_by_hand():
    x = torch.tensor([[3.0, 4.0, 1.0, 0.0]], dtype=F64)
    w = torch.tensor([1.0, 2.0, 1.0, 5.0], dtype=F64)
    a, b = math.sqrt((9 + 16) / 2 + 0.5), math.sqrt(1 / 2 + 0.5)
    assert torch.allclose(plain.grouped_norm(x, 2, 0.5, w), torch.tensor([[3 / a, 8 / a, 1 / b, 0.0]], dtype=F64), atol=1e-14)
    one = math.sqrt(26 / 4 + 0.5)
    assert torch.allclose(plain.grouped_norm(x, 1, 0.5, w), x / one * w, atol=1e-14)


def test_rotations_are_complex_multiplications():
    g = torch.Generator().manual_seed(1)
    x, pos = torch.randn(7, 2, 10, generator=g, dtype=F64), torch.tensor([0, 1, 5, 64, 300, 1000, 31])
    f = 100.0 ** (-2.0 * torch.arange(3, dtype=F64) / 6)
    turn = torch.exp(1j * pos[:, None].to(F64) * f[None, :])[:, None, :]
    z = torch.complex(x[..., 0:6:2], x[..., 1:6:2]) * turn
    got = plain.turn_neighbours(x, pos, 6, 100.0)
    assert torch.allclose(got[..., 0:6:2], z.real, atol=1e-12) and torch.allclose(got[..., 1:6:2], z.imag, atol=1e-12)
    z = torch.complex(x[..., 0:3], x[..., 3:6]) * turn
    got2 = plain.turn_halves(x, pos, 6, 100.0)
    assert torch.allclose(got2[..., 0:3], z.real, atol=1e-12) and torch.allclose(got2[..., 3:6], z.imag, atol=1e-12)
    assert torch.equal(got[..., 6:], x[..., 6:]) and torch.equal(got2[..., 6:], x[..., 6:])


def test_chunk_mask_by_hand():
    m = plain.chunk_mask(7, 3)
    assert m[2].tolist() == [True] * 3 + [False] * 4 and m[3].tolist() == [False] * 3 + [True] + [False] * 3
    assert m[5].tolist() == [False] * 3 + [True] * 3 + [False] and m[6].tolist() == [False] * 6 + [True]
    assert plain.chunk_mask(4, 1).tolist() == torch.eye(4).bool().tolist()
    assert plain.chunk_mask(4, None).tolist() == torch.tril(torch.ones(4, 4)).bool().tolist()


def test_sigmoid_weights_have_no_denominator():
    g = torch.Generator().manual_seed(2)
    q, k, v = torch.randn(9, 4, 6, generator=g, dtype=F64), torch.randn(9, 2, 6, generator=g, dtype=F64), torch.randn(9, 2, 3, generator=g, dtype=F64)
    bias = torch.tensor([0.3, -2.0, 0.0, 1.5], dtype=F64)
    got = plain.sigmoid_attention(q, k, v, 0.7, bias, 4)
    for h in range(4):
        for t in range(9):
            want = sum(v[j, h // 2] / (1 + math.exp(-(0.7 * float(q[t, h] @ k[j, h // 2]) + float(bias[h])))) for j in range(t // 4 * 4, t + 1))
            assert torch.allclose(got[t, h], want, atol=1e-12)


def test_route_keeps_the_sigmoids():
    z = torch.tensor([[0.0, 2.0, -1.0, 3.0], [30.0, 31.0, 29.0, -5.0]], dtype=F64)
    chosen, weights = plain.route(z, 2)
    assert chosen.tolist() == [[3, 1], [1, 0]]
    assert torch.allclose(weights[0], torch.sigmoid(torch.tensor([3.0, 2.0], dtype=F64)), atol=1e-15)


def test_the_weight_scales_an_experts_input():
    g = torch.Generator().manual_seed(3)
    W, E, F = 5, 4, 3
    c = dict(kind="moe", expert=dict(ff=F), router=dict(experts=E, top=2), shared=dict(ff=2))
    w = {"router": torch.randn(E, W, generator=g, dtype=F64)}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = (torch.randn(*s, generator=g, dtype=F64) for s in ((F, W), (F, W), (W, F)))
    w["shared.gate"], w["shared.up"], w["shared.down"] = (torch.randn(*s, generator=g, dtype=F64) for s in ((2, W), (2, W), (W, 2)))
    h = torch.randn(6, W, generator=g, dtype=F64)
    out = plain.experts_ff(h, w, "", c)
    for t in range(6):
        s = torch.sigmoid(w["router"] @ h[t])
        best = sorted(range(E), key=lambda e: -float(s[e]))[:2]
        want = plain.gated_ff(h[t:t + 1], w, "shared.")[0]
        scaled = want.clone()
        for e in best:
            x = s[e] * h[t]
            gate = w[f"e{e}.gate"] @ x
            want = want + w[f"e{e}.down"] @ (gate / (1 + torch.exp(-gate)) * (w[f"e{e}.up"] @ x))
            scaled = scaled + s[e] * plain.gated_ff(h[t:t + 1], w, f"e{e}.")[0]
        assert torch.allclose(out[t], want, atol=1e-12) and not torch.allclose(out[t], scaled, atol=1e-3)
