"""Zalazen without a GPU: the registry, the generator of made-up checkpoints, the token history that the pair embedding reads,
the joined projection, the stretched rotation's ramp, and the plain restatement's mechanisms on cases with closed forms (what
the GPU tests compare the kernels with)."""

import json
import math

import pytest
import torch

from oracle import zalazen as O
from tiny_llm_b200.latent_kv_cache import LatentPagedCache, LatentPagedPool
from tiny_llm_b200.models import ARCHITECTURES
from tiny_llm_b200.positional_encoding import yarn_ramp
from tiny_llm_b200.ragged import RaggedEntry, RaggedPlan
from tiny_llm_b200.state_cache import HybridPagedCache, StateSlotPool
from tiny_llm_b200.synthetic import save_zalazen, synthetic_zalazen, zalazen_config

D64 = torch.float64


def test_registry_names_the_design():
    assert ARCHITECTURES["Zalazen"] == ("tiny_llm_b200.zalazen", "ZalazenModel")


def test_generator_spells_the_stack_and_round_trips_through_a_directory(tmp_path):
    config = zalazen_config(pattern="AdSnAdSdSd", windows=((10, 2), (30, 0)))
    assert [l["mixer"].get("kv_from") for l in config["layers"]] == [None, 0, None, 2, 2]
    assert [l["mixer"]["mask"]["size"] for l in config["layers"]] == [10, 30, 10, 30, 10]
    assert config["layers"][1]["mlp"] is None and config["layers"][2]["mlp"]["kind"] == "dense"
    tensors = synthetic_zalazen(config, seed=3)
    assert "l1.norm2" not in tensors and "l1.mix.k" not in tensors and "l3.mix.k.norm" not in tensors and "l2.mix.v" in tensors
    assert tensors["bigram"].shape == (510, 96) and tensors["l3.mix.q.norm"].shape == (64,) and tensors["l0.mix.g"].shape == (4, 96)
    save_zalazen(config, tensors, tmp_path / "m")
    from tiny_llm_b200.checkpoint import read_tensors

    again = read_tensors(tmp_path / "m")
    assert set(again) == set(tensors) and json.loads((tmp_path / "m" / "config.json").read_text()) == config
    assert all(torch.equal(again[k], tensors[k]) for k in tensors)
    plain = zalazen_config(pattern="Ad", buckets=0, scaling=None)
    assert "bigram" not in plain["embedding"] and "scaling" not in plain["layers"][0]["mixer"]["rot"] and "bigram" not in synthetic_zalazen(plain)
    for bad in ("Xd", "Sd", "Az", "A"):
        with pytest.raises(ValueError):
            zalazen_config(pattern=bad)


# ---------------------------------------------------------------------------------------------- the token before, in the cache
@pytest.mark.parametrize("hybrid", [False, True])
def test_plan_hands_every_sequence_its_previous_token(hybrid):
    pool = LatentPagedPool([8], page_size=4, device="cpu", dtype=torch.float32)
    states = StateSlotPool(3, device="cpu")
    make = lambda: HybridPagedCache(pool, states) if hybrid else LatentPagedCache(pool)
    a, b = make(), make()
    plan = RaggedPlan([RaggedEntry([5, 6, 7, 8, 9], [a])], "cpu", 4)
    assert plan.seq_prev.tolist() == [-1] and list(a.tokens) == [5, 6, 7, 8, 9]
    plan = RaggedPlan([RaggedEntry([1], [b]), RaggedEntry([2, 3], [a])], "cpu", 4)
    assert plan.seq_prev.tolist() == [-1, 9] and plan.seq_info[:, 2].tolist() == [0, 5]
    plan = RaggedPlan([RaggedEntry([4], [a]), RaggedEntry([11, 12], [b])], "cpu", [2, 4])
    assert plan.seq_prev.tolist() == [3, 1]
    assert plan.total_ints == RaggedPlan.block_ints(3, 2, 2, plan.max_pages, 4)
    a.release()
    assert len(a.tokens) == 0
    plan = RaggedPlan([RaggedEntry([30], [a])], "cpu", 4)        # the same cache object starts a new sequence
    assert plan.seq_prev.tolist() == [-1] and list(a.tokens) == [30]
    a.release()
    b.release()


def test_history_follows_a_rewind_and_a_step_that_was_refused():
    pool = LatentPagedPool([8], page_size=4, device="cpu", dtype=torch.float32, max_pages=3)
    a, b = LatentPagedCache(pool), LatentPagedCache(pool)
    RaggedPlan([RaggedEntry([5, 6, 7, 8, 9, 10], [a])], "cpu", 4)
    a.rewind(2)
    assert list(a.tokens) == [5, 6, 7, 8]
    assert RaggedPlan([RaggedEntry([40], [a])], "cpu", 4).seq_prev.tolist() == [8]
    with pytest.raises(RuntimeError, match="exhausted"):
        RaggedPlan([RaggedEntry([1, 2], [a]), RaggedEntry([3] * 8, [b])], "cpu", 4)
    assert list(a.tokens) == [5, 6, 7, 8, 40] and a.offset == 5 and len(b.tokens) == 0
    with pytest.raises(ValueError, match="wanted place"):           # refused before anything is appended
        RaggedPlan([RaggedEntry([1, 2], [a], want=[2])], "cpu", 4)
    with pytest.raises(ValueError, match="once per step"):
        RaggedPlan([RaggedEntry([1], [a]), RaggedEntry([2], [a])], "cpu", 4)
    with pytest.raises(ValueError, match="at least one token"):
        RaggedPlan([RaggedEntry([1], [a]), RaggedEntry([], [b])], "cpu", 4)
    assert list(a.tokens) == [5, 6, 7, 8, 40] and a.offset == 5 and b.offset == 0
    a.append_slots(2)                                             # filled by something that is no step: no ids known
    assert RaggedPlan([RaggedEntry([50], [a])], "cpu", 4).seq_prev.tolist() == [-1]
    assert list(a.tokens) == [5, 6, 7, 8, 40, -1, -1, 50]


def test_plan_rows_of_unequal_entries():
    pool = LatentPagedPool([8], page_size=4, device="cpu", dtype=torch.float32)
    a, b, c = (LatentPagedCache(pool) for _ in range(3))
    RaggedPlan([RaggedEntry([9] * 6, [b])], "cpu", 4)
    plan = RaggedPlan([RaggedEntry([1, 2, 3, 4, 5], [a], want=[4, 0]), RaggedEntry([6], [b], want=[]), RaggedEntry([7, 8], [c])], "cpu", [2, 4])
    assert plan.ids.tolist() == [1, 2, 3, 4, 5, 6, 7, 8] and plan.tok_pos.tolist() == [0, 1, 2, 3, 4, 6, 0, 1] and plan.tok_seq.tolist() == [0] * 5 + [1, 2, 2]
    assert plan.want_rows.tolist() == [4, 0, 7] and plan.want_counts == [2, 0, 1] and not plan.all_wanted and plan.max_tokens == 5 and plan.max_context == 7
    assert plan.tiles_for(2).tolist() == [[0, 2, 0], [2, 2, 0], [4, 1, 0], [5, 1, 1], [6, 2, 2]]
    assert plan.tiles_for(4).tolist() == [[0, 4, 0], [4, 1, 0], [5, 1, 1], [6, 2, 2]]
    assert plan.seq_info.tolist() == [[0, 5, 0, -1], [5, 1, 6, -1], [6, 2, 0, -1]] and plan.seq_prev.tolist() == [-1, 9, -1]
    assert plan.block_table.tolist() == [a.page_ids, b.page_ids, c.page_ids + [-1]]
    plan = RaggedPlan([RaggedEntry([1], [c]), RaggedEntry([3], [a], want=[0, 0]), RaggedEntry([2], [b], want=[])], "cpu", [2, 4])
    assert plan.tok_pos.tolist() == [2, 5, 7] and plan.want_rows.tolist() == [0, 1, 1] and plan.tiles_for(4).tolist() == [[0, 1, 0], [1, 1, 1], [2, 1, 2]]
    assert not plan.all_wanted and RaggedPlan([RaggedEntry([1, 2], [a], want=range(2)), RaggedEntry([1], [b])], "cpu", 4).all_wanted
    assert not RaggedPlan([RaggedEntry([1, 2], [a], want=[1, 0])], "cpu", 4).all_wanted


# ---------------------------------------------------------------------------------------------- small product parts
def test_joined_projection_keeps_one_copy_and_sums_its_parts():
    from tiny_llm_b200.paged_attention import JoinedProjection

    g = torch.Generator().manual_seed(1)
    w1, w2 = torch.randn(6, 10, generator=g), torch.randn(6, 7, generator=g)
    j = JoinedProjection([("a", w1), ("b", w2)])
    assert torch.equal(j.part("a"), w1) and torch.equal(j.part("b"), w2)
    assert j.part("b").untyped_storage().data_ptr() == j.weight.untyped_storage().data_ptr()
    x, part = j.operand(3)
    u, v = torch.randn(3, 10, generator=g), torch.randn(3, 7, generator=g)
    part["a"].copy_(u)
    part["b"].copy_(v)
    assert torch.allclose(j(x), u @ w1.t() + v @ w2.t(), atol=1e-5)
    assert torch.equal(JoinedProjection([("a", w1)]).part("a"), w1)


@pytest.mark.parametrize("dims,base,scaling", [(8, 3e4, (4.0, 512, 16.0, 1.0)), (64, 1e4, (8.0, 4096, 32.0, 1.0)), (2, 500.0, (3.0, 64, 8.0, 2.0)),
                                               (32, 1e6, (1.0, 1024, 32.0, 1.0)), (16, 100.0, (2.0, 100000, 64.0, 60.0)), (16, 1e5, (16.0, 8, 32.0, 1.0))])
def test_ramp_of_the_stretched_rotation(dims, base, scaling):
    names = dict(zip(("factor", "original", "fast", "slow"), scaling))
    factor, lo, hi, gain = yarn_ramp(dims, base, **names)
    freqs, want_gain = O.frequencies({"dims": dims, "base": base, "scaling": names})
    assert gain == pytest.approx(want_gain) and gain == pytest.approx(0.1 * math.log(names["factor"]) + 1)
    for i, want in enumerate(freqs):
        f = base ** (-2 * i / dims)
        r = min(max((i - lo) / max(hi - lo, 0.001), 0), 1)
        assert f / factor * r + f * (1 - r) == pytest.approx(want, rel=1e-12)
    turns = [names["original"] * base ** (-2 * i / dims) / (2 * math.pi) for i in range(dims // 2)]
    for i, n in enumerate(turns):                                # far from the ramp: kept, or divided
        if n > names["fast"] * base ** (2 / dims):
            assert freqs[i] == pytest.approx(base ** (-2 * i / dims))
        if n < names["slow"] / base ** (2 / dims) and i > 0:
            assert freqs[i] == pytest.approx(base ** (-2 * i / dims) / factor)


# ---------------------------------------------------------------------------------------------- the plain restatement
def test_pair_rows():
    assert O.bigram_row(None, 9, mul_prev=7, mul_cur=3, buckets=50) == 50
    assert O.bigram_row(0, 9, mul_prev=7, mul_cur=3, buckets=50) == 27      # token 0 before is not "nothing before"
    assert O.bigram_row(8, 9, mul_prev=7, mul_cur=3, buckets=50) == (56 + 27) % 50
    config = zalazen_config(pattern="Ad", vocab=20, width=8)
    tensors = {n: t.to(D64) for n, t in synthetic_zalazen(config, seed=1).items()}
    x = O.embed([4, 4, 7], tensors, config)
    assert torch.allclose(x[0], tensors["embed"][4] * 5.0 + tensors["bigram"][509])
    assert torch.allclose(x[2], tensors["embed"][7] * 5.0 + tensors["bigram"][(4 * 19 + 7 * 11) % 509])
    assert not torch.allclose(x[0], x[1])


def test_window_and_kept_first_positions_at_their_edges():
    see = lambda i, j: O.visible(i, j, 5, 2)
    assert [j for j in range(12) if see(10, j)] == [0, 1, 6, 7, 8, 9, 10]
    assert [j for j in range(12) if see(5, j)] == [0, 1, 2, 3, 4, 5] and [j for j in range(12) if see(0, j)] == [0]
    assert [j for j in range(12) if O.visible(10, j, 5, 0)] == [6, 7, 8, 9, 10]
    assert [j for j in range(12) if O.visible(3, j, 1, 9)] == [0, 1, 2, 3]     # nothing from the future is kept


def test_sink_counts_once_unscaled_and_gives_no_value():
    q, k = torch.zeros(3, 1, 2, dtype=D64), torch.zeros(3, 1, 2, dtype=D64)
    v = torch.tensor([2.0, 4.0, 9.0], dtype=D64).reshape(3, 1, 1)
    out = O.sink_window_attention(q, k, v, torch.tensor([math.log(8.0)], dtype=D64), scale=100.0, size=2, keep_first=0)
    assert torch.allclose(out.reshape(-1), torch.tensor([2.0 / 9, 6.0 / 10, 13.0 / 10], dtype=D64))
    out = O.sink_window_attention(q, k, v, torch.tensor([math.log(8.0)], dtype=D64), scale=100.0, size=2, keep_first=1)
    assert torch.allclose(out.reshape(-1), torch.tensor([2.0 / 9, 6.0 / 10, 15.0 / 11], dtype=D64))


def test_rotation_pairs_halves_and_leaves_the_rest():
    x = torch.zeros(3, 1, 6, dtype=D64)
    x[:, 0] = torch.tensor([1.0, 0, 0, 0, 5.0, 6.0], dtype=D64)
    y = O.rotate(x, {"dims": 4, "base": 100.0})
    assert torch.allclose(y[2, 0], torch.tensor([math.cos(2.0), 0, math.sin(2.0), 0, 5.0, 6.0], dtype=D64))
    y = O.rotate(x, {"dims": 4, "base": 100.0, "scaling": {"factor": math.e, "original": 1000, "fast": 1e9, "slow": 1e8}})
    gain = 1.1                                                   # every pair below `slow` turns: all but pair 0 divided, pair 0 at the ramp's start
    assert torch.allclose(y[2, 0, :4], gain * torch.tensor([math.cos(2.0), 0, math.sin(2.0), 0], dtype=D64))


def test_branches_read_the_same_stream_and_shared_keys_come_from_the_source_layer():
    config = zalazen_config(pattern="AdSdAn", width=24, vocab=30, heads=2, kv_heads=1, dim=6, vdim=5, rot_dims=4, ff=20)
    tensors = {n: t.to(D64) for n, t in synthetic_zalazen(config, seed=2).items()}
    ids = torch.randint(0, 30, (40,), generator=torch.Generator().manual_seed(3)).tolist()
    tap = []
    full = O.forward(ids, tensors, config, tap=tap)
    assert full.shape == (40, 30) and len(tap) == 3 and torch.isfinite(full).all()
    assert torch.allclose(O.forward(ids[:17], tensors, config), full[:17], atol=1e-9)        # causal
    x = O.embed(ids, tensors, config)
    m, eps = config["layers"][0]["mixer"], 1e-6
    h1, h2 = O.rms_unit(x, eps) * tensors["l0.norm1"], O.rms_unit(x, eps) * tensors["l0.norm2"]
    kv = O.keys_values(h1, tensors, "l0.mix.", m, eps=eps)
    assert torch.allclose(tap[0], x + O.attention_mixer(h1, tensors, "l0.mix.", m, kv, eps=eps) + O.gated_ff(h2, tensors, "l0.mlp."))
    h1 = O.rms_unit(tap[0], eps) * tensors["l1.norm1"]
    h2 = O.rms_unit(tap[0], eps) * tensors["l1.norm2"]
    y = O.attention_mixer(h1, tensors, "l1.mix.", config["layers"][1]["mixer"], kv, eps=eps)
    assert torch.allclose(tap[1], tap[0] + y + O.gated_ff(h2, tensors, "l1.mlp."))
