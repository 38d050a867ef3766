"""Nomudra without a GPU: the registry, the generator of made-up checkpoints, argument checks of the modules, and the plain
restatement's mechanisms on cases with closed forms (what the GPU tests compare the kernels with)."""

import json
import math

import pytest
import torch

from oracle import nomudra as O
from tiny_llm_b200.layer_norm import TanhNorm
from tiny_llm_b200.linear_attention import MatrixMemory
from tiny_llm_b200.mlp import GatedMLP, MixtureOfExperts, TopKRouter
from tiny_llm_b200.models import ARCHITECTURES
from tiny_llm_b200.synthetic import nomudra_config, save_nomudra, synthetic_nomudra

D64 = torch.float64


def test_registry_names_the_design():
    assert ARCHITECTURES["Nomudra"] == ("tiny_llm_b200.nomudra", "NomudraModel")


def test_generator_spells_the_stack_and_round_trips_through_a_directory(tmp_path):
    config = nomudra_config(pattern="MmAnAmMn", chunks=(10, 30))
    assert [l["type"] for l in config["layers"]] == ["mlstm", "attention", "attention", "mlstm"]
    assert [l["mixer"]["mask"]["size"] for l in config["layers"][1:3]] == [10, 30] and config["layers"][1]["mlp"] is None
    tensors = synthetic_nomudra(config, seed=3)
    assert tensors["l0.norm1b.alpha"].shape == () and "l1.norm2" not in tensors and "l1.mix.v" not in tensors and tensors["l1.mix.g"].shape == (64, 96)
    assert tensors["l0.mlp.router"].shape == (8, 96) and "l0.mlp.e6.up" not in tensors and tensors["l0.mlp.shared.sg"].shape == (1, 96)
    assert tensors["l0.mix.norm"].shape == (72,) and tensors["l3.mix.f.b"].shape == (3,)
    save_nomudra(config, tensors, tmp_path / "m")
    from tiny_llm_b200.checkpoint import read_tensors

    again = read_tensors(tmp_path / "m")
    assert set(again) == set(tensors) and json.loads((tmp_path / "m" / "config.json").read_text()) == config
    assert all(torch.equal(again[k], tensors[k]) for k in tensors)
    plain = nomudra_config(pattern="Am", groups=None, shared_ff=0, rot_dims=0)["layers"][0]
    assert "groups" not in plain["mlp"]["router"] and "shared" not in plain["mlp"] and "rot" not in plain["mixer"]
    for bad in ("Xm", "Md", "A"):
        with pytest.raises(ValueError):
            nomudra_config(pattern=bad)


def test_modules_refuse_tensors_that_do_not_fit():
    z = torch.zeros
    assert TanhNorm(z(4), z(4), torch.tensor(0.5)).alpha == 0.5
    for args in ((z(4), z(5), z(())), (z(4), z(4), z(2)), (z(2, 2), z(2, 2), z(()))):
        with pytest.raises(ValueError, match="tanh norm"):
            TanhNorm(*args)
    good = dict(heads=2, dim=3, vdim=4, gate_cap=5.0, w_i=z(2, 6), b_i=z(2), w_f=z(2, 6), b_f=z(2), norm_weight=z(8), w_o=z(6, 8))
    m = MatrixMemory(**good)
    assert m.state_shape == (2, 3, 5) and m.peak_shape == (2,) and m.w_gates.shape == (4, 6)
    for wrong in (dict(gate_cap=0.0), dict(w_f=z(1, 6)), dict(b_i=z(3)), dict(norm_weight=z(4)), dict(w_o=z(6, 6))):
        with pytest.raises(ValueError, match="matrix memory"):
            MatrixMemory(**{**good, **wrong})
    router = TopKRouter(z(6, 8), None, 2, scoring="softmax_all", groups=(3, 2))
    for groups in ((4, 1), (3, 4), (6, 1)):
        with pytest.raises(ValueError, match="groups"):
            TopKRouter(z(6, 8), None, 2, scoring="softmax_all", groups=groups)
    experts = z(4, 5, 8), z(4, 5, 8), z(4, 8, 5)
    shared = GatedMLP(z(7, 8), z(7, 8), z(8, 7), "clamped_swish", limit=1.0)
    MixtureOfExperts(router, *experts, "clamped_swish", shared, identity=2, limit=1.0, shared_gate=z(1, 8))
    for wrong in (dict(identity=1, limit=1.0), dict(identity=2), dict(identity=2, limit=1.0, shared_gate=z(1, 9)), dict(identity=2, limit=1.0, shared_gate=z(1, 8), shared=None)):
        with pytest.raises(ValueError):
            MixtureOfExperts(router, *experts, "clamped_swish", **{"shared": shared, **wrong})


# ---------------------------------------------------------------------------------------------- the plain restatement
def test_tanh_norm_knows_no_row():
    w = {"n": torch.tensor([2.0, -1.0], dtype=D64), "n.b": torch.tensor([0.5, 0.0], dtype=D64), "n.alpha": torch.tensor(3.0, dtype=D64)}
    y = O.tanh_norm(torch.tensor([[0.1, 100.0], [0.1, 0.0]], dtype=D64), w, "n")
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(0.3) + 0.5, -1.0], [2 * math.tanh(0.3) + 0.5, 0.0]], dtype=D64))


def test_chunks_are_counted_from_nought():
    assert [j for j in range(20) if O.visible(12, j, 5)] == [10, 11, 12] and [j for j in range(20) if O.visible(9, j, 5)] == [5, 6, 7, 8, 9]
    assert [j for j in range(20) if O.visible(10, j, 5)] == [10] and [j for j in range(20) if O.visible(3, j, 100)] == [0, 1, 2, 3]


def test_attention_of_one_token_hands_its_unturned_key_on():
    spec = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0, "mask": {"size": 1}, "rot": {"dims": 2, "base": 10.0}}
    g = torch.Generator().manual_seed(0)
    w = {n: torch.randn(*s, generator=g, dtype=D64) for n, s in (("q", (8, 6)), ("q.b", (8,)), ("k", (4, 6)), ("k.b", (4,)), ("g", (8, 6)), ("o", (6, 8)), ("o.b", (6,)))}
    h = torch.randn(5, 6, generator=g, dtype=D64)
    v = h @ w["k"].t() + w["k.b"]          # chunks of one token: every token sees itself alone
    want = (torch.cat([v, v], dim=1) * torch.sigmoid(h @ w["g"].t())) @ w["o"].t() + w["o.b"]
    assert torch.allclose(O.attention_mixer(h, w, "", spec), want)


def test_rotation_pairs_halves_and_leaves_the_rest():
    x = torch.zeros(3, 1, 6, dtype=D64)
    x[:, 0] = torch.tensor([1.0, 0, 0, 0, 5.0, 6.0], dtype=D64)
    assert torch.allclose(O.rotate(x, 4, 100.0)[2, 0], torch.tensor([math.cos(2.0), 0, math.sin(2.0), 0, 5.0, 6.0], dtype=D64))


def test_matrix_memory_equals_the_sums_it_stabilises():
    """o_t = sum_s a_ts (k_s.q_t) v_s / (max(|sum_s a_ts k_s.q_t|, 1) + 1e-6 e^m), a_ts = exp(i_s + f_(s+1) + .. + f_t)."""
    g = torch.Generator().manual_seed(2)
    T, H, dk, dv = 25, 2, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=D64) for n in (dk, dk, dv))
    li, lf = 2 * torch.randn(T, H, generator=g, dtype=D64) - 1, O.log_sigmoid(2 + torch.randn(T, H, generator=g, dtype=D64))
    got = O.matrix_memory(q, k, v, li, lf)
    for h in range(H):
        m = 0.0
        for t in range(T):
            m = max(m + lf[t, h].item(), li[t, h].item())
            a = torch.stack([li[s, h] + lf[s + 1 : t + 1, h].sum() for s in range(t + 1)]).exp() * (k[: t + 1, h] @ q[t, h])
            want = (a[:, None] * v[: t + 1, h]).sum(0) / (a.sum().abs().clamp(min=1.0) + 1e-6 * math.exp(m))
            assert torch.allclose(got[t, h], want, rtol=1e-9, atol=1e-12)


def test_gates_of_the_memory():
    z = torch.tensor([-1e3, -2.0, 0.0, 1e3], dtype=D64)
    assert torch.allclose(O.soft_bound(z, 5.0), torch.tensor([-5.0, 5 * math.tanh(-0.4), 0.0, 5.0], dtype=D64))
    assert torch.allclose(O.log_sigmoid(torch.tensor([-50.0, 0.0, 3.0], dtype=D64)), torch.tensor([-50.0, math.log(0.5), -math.log1p(math.exp(-3.0))], dtype=D64))


def test_choice_among_the_best_groups_with_scores_below_nought():
    s = torch.tensor([0.30, 0.05, 0.20, 0.25, 0.10, 0.10], dtype=D64)
    c = torch.tensor([-0.9, -0.5, -0.5, -0.6, -0.35, -0.8], dtype=D64)   # choice: -.60 -.45 | -.30 -.35 | -.25 -.70
    assert O.choose(s, c, 2) == [4, 2] and O.choose(s, c, 2, {"count": 3, "keep": 1}) == [4, 5] and O.choose(s, c, 3, {"count": 3, "keep": 2}) == [4, 2, 3]
    assert O.choose(s, c, 2, {"count": 1, "keep": 1}) == [4, 2] and O.choose(s, torch.zeros(6, dtype=D64), 1, {"count": 2, "keep": 1}) == [0]


def test_expert_mixture_weights_identity_and_shared():
    D = 3
    w = {"router": torch.zeros(3, D, dtype=D64), "correction": torch.tensor([0.0, 0.2, 0.1], dtype=D64), "shared.sg": torch.zeros(1, D, dtype=D64)}
    for name in ("e0.", "e1.", "shared."):
        for part in ("gate", "up", "down"):
            w[name + part] = torch.eye(D, dtype=D64) * (2.0 if name == "e1." else 1.0)
    spec = {"router": {"experts": 2, "identity": 1, "top": 2}, "expert": {"limit": 1.0}, "shared": {"limit": 0.5}}
    h = torch.tensor([[3.0, -4.0, 0.25]], dtype=D64)
    inner = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    e1 = torch.tensor([inner(1, 1), inner(-8, -1), inner(0.5, 0.5)], dtype=D64) * 2
    sh = torch.tensor([inner(0.5, 0.5), inner(-4, -0.5), inner(0.25, 0.25)], dtype=D64)
    assert torch.allclose(O.expert_mixture(h, w, "", spec)[0], 0.5 * e1 + 0.5 * h[0] + 0.5 * sh)   # outputs 1 and 2 (identity), equal scores


def test_every_sublayer_is_normed_on_both_sides():
    config = nomudra_config(pattern="AmMn", width=24, vocab=30, heads=2, kv_heads=1, dim=6, rot_dims=4, mem_heads=2, mem_dim=5, mem_vdim=4, expert_ff=9, shared_ff=11)
    t = {n: x.to(D64) for n, x in synthetic_nomudra(config, seed=2).items()}
    ids = torch.randint(0, 30, (20,), generator=torch.Generator().manual_seed(3)).tolist()
    tap = []
    full = O.forward(ids, t, config, tap=tap)
    assert full.shape == (20, 30) and len(tap) == 2 and torch.isfinite(full).all()
    assert torch.allclose(O.forward(ids[:9], t, config), full[:9], atol=1e-9)        # causal
    x = O.tanh_norm(t["embed"][ids], t, "embed.norm")
    x = x + O.tanh_norm(O.attention_mixer(O.tanh_norm(x, t, "l0.norm1"), t, "l0.mix.", config["layers"][0]["mixer"]), t, "l0.norm1b")
    x = x + O.tanh_norm(O.expert_mixture(O.tanh_norm(x, t, "l0.norm2"), t, "l0.mlp.", config["layers"][0]["mlp"]), t, "l0.norm2b")
    assert torch.allclose(tap[0], x)
    x = x + O.tanh_norm(O.matrix_memory_mixer(O.tanh_norm(x, t, "l1.norm1"), t, "l1.mix.", config["layers"][1]["mixer"], 1e-5), t, "l1.norm1b")
    assert torch.allclose(tap[1], x) and torch.allclose(full, O.tanh_norm(x, t, "final.norm") @ t["head"].t())
