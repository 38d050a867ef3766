"""Nomudra on a B200 against the plain CPU restatement (oracle/nomudra.py, float64): each mechanism that the design added to
the blocks library alone, then the model through every way of cutting and batching a sequence, the schedulers and the
entry points.  Small made-up configurations and random weights; where random weights would hide a fault (a far key among
hundreds, the edge of a chunk, a memory that outlives hundreds of tokens, a normaliser's floor) the inputs are built so that it shows.

Tolerances: relative root-mean-square error of a logits row (mean taken off) below 5e-5 in float32 mode - every product in
true fp32, so only summation order differs.  In bfloat16 mode a router's close call can go the other way for a token (its row
then differs by more than rounding), so whole schedules are held to a median of 4e-2, 90 % of the rows below 2e-1; the
float32 run is the sharp test.
"""

import math

import pytest
import torch

from oracle import nomudra as O
from extensions_b200.tiny_llm_ext_b200 import blocks
from tiny_llm_b200 import BatchingKvCache, ContinuousBatcher, greedy_generate_ids
from tiny_llm_b200.layer_norm import TanhNorm
from tiny_llm_b200.linear_attention import MatrixMemory
from tiny_llm_b200.mlp import GatedMLP, MixtureOfExperts, TopKRouter
from tiny_llm_b200.models import load_model, model_class
from tiny_llm_b200.paged_attention import PagedGroupedAttention
from tiny_llm_b200.ragged import RaggedEntry
from tiny_llm_b200.synthetic import nomudra_config, save_nomudra, synthetic_nomudra

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def dev(cuda_device):
    return cuda_device


def row_errors(got, want):
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def row_error(got, want):
    return row_errors(got, want).max().item()


def rows_match(got, want, dtype):
    err = row_errors(got, want)
    if dtype == torch.float32:
        return err.max().item() < 5e-5
    return err.median().item() < 4e-2 and err.quantile(0.9).item() < 2e-1


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs().max().item()
    scale = want.abs().max().item() + 1e-9
    assert err <= tol * scale, (err, scale)


def ids_for(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def ints(dev, rows):
    return torch.tensor(rows, dtype=torch.int32, device=dev)


def tile_list(dev, count, tile):
    return ints(dev, [(t, min(tile, count - t), 0) for t in range(0, count, tile)])


# ---------------------------------------------------------------------------------------------- tanh norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [8, 50, 77, 2112])
def test_tanh_norms_around_the_stream(dev, dtype, D):
    g = torch.Generator().manual_seed(D)
    rows, tol = 19, 3e-6 if dtype == torch.float32 else 1e-2
    w = {}
    for name, alpha in (("a", 0.7), ("b", 1.9), ("c", 0.25)):
        w[name], w[name + ".b"], w[name + ".alpha"] = (1 + 0.3 * torch.randn(D, generator=g)).to(dtype), (0.4 * torch.randn(D, generator=g)).to(dtype), torch.tensor(alpha).to(dtype)
    a, b, c = (TanhNorm(w[n].to(dev), w[n + ".b"].to(dev), w[n + ".alpha"].to(dev)) for n in "abc")
    w = {n: t.double() for n, t in w.items()}
    table = (2 * torch.randn(30, D, generator=g)).to(dtype)
    ids = ids_for(rows, 30, 1)
    x, h = a.embed(ints(dev, ids), table.to(dev), b)
    want = O.tanh_norm(table[ids].double(), w, "a")
    assert x.dtype == torch.float32 and h.dtype == dtype
    close(x, want, 3e-6)
    close(h, O.tanh_norm(want, w, "b"), tol)
    # a sublayer's output, with and without its projection's bias, into the stream; the next norm, or none
    y, bias = 3 * torch.randn(rows, D, generator=g), torch.randn(D, generator=g).to(dtype)
    h = b.follow(x, y.to(dev), c, y_bias=bias.to(dev))
    want = want + O.tanh_norm(y.double() + bias.double(), w, "b")
    close(x, want, 3e-6)
    close(h, O.tanh_norm(want, w, "c"), tol)
    assert c.follow(x, y.to(dev), None) is None
    want = want + O.tanh_norm(y.double(), w, "c")
    close(x, want, 3e-6)
    # the norm alone, on all rows and on some in any order; the stream stays as it is
    before = x.clone()
    close(a.rows(x), O.tanh_norm(want, w, "a"), tol)
    pick = [7, 0, 7, 18]
    close(a.rows(x, ints(dev, pick)), O.tanh_norm(want, w, "a")[pick], tol)
    assert torch.equal(x, before)
    # large inputs saturate instead of overflowing
    big = torch.full((rows, D), 1e30, device=dev)
    a.follow(x, big, None)
    close(x, want + w["a"] + w["a.b"], 3e-6)


# ---------------------------------------------------------------------------------------------- attention
def cached(dev, dtype, k, v, page=32, seed=0):
    """Keys and values of one sequence in pages that are out of order -> (slab, block table)."""
    S, G, dk = k.shape
    pages = -(-S // page)
    order = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(seed))[:pages]
    slab = torch.full((pages + 2, page, G * (dk + v.shape[2])), 7.0, dtype=dtype)
    flat = torch.cat([k.reshape(S, -1), v.reshape(S, -1)], dim=1).to(dtype)
    for p in range(pages):
        part = flat[p * page : (p + 1) * page]
        slab[order[p], : part.shape[0]] = part
    return slab.to(dev), order.to(torch.int32).reshape(1, -1).to(dev)


def kernels_for(dtype, heads, kv_heads, dk, dv):
    """Every kernel that serves these sizes, with the most tokens an entry of its work list may hold."""
    out = {"general": blocks.paged_attention_tile_tokens(heads, kv_heads)}
    name, tile = blocks.paged_attention_kernel(dtype, heads, kv_heads, dk, dv, 32)
    out[name] = tile
    out.update(blocks.paged_attention_flash_forms(dtype, heads, kv_heads, dk, dv, 32))
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dk,size", [(4, 2, 16, 37), (6, 2, 10, 50), (3, 3, 64, 64), (8, 1, 128, 100), (2, 1, 72, 1), (40, 1, 24, 33)])
def test_an_entry_wise_gate_in_every_attention_kernel(dev, dtype, heads, kv_heads, dk, size):
    g = torch.Generator().manual_seed(heads * dk + size)
    S = 150
    q, k, v = torch.randn(S, heads, dk, generator=g), torch.randn(S, kv_heads, dk, generator=g), torch.randn(S, kv_heads, dk, generator=g)
    wide = torch.randn(S, heads * dk + 11, generator=g)  # the gate is a view into a wider product
    q, k, v, wide = (t.to(dtype) for t in (q, k, v, wide))
    want = O.chunk_attention(q.double(), k.double(), v.double(), scale=dk ** -0.5, size=size)
    want = want * torch.sigmoid(wide[:, 3 : 3 + heads * dk].double()).view(S, heads, dk)
    slab, table = cached(dev, dtype, k, v)
    gate = wide.to(dev)[:, 3 : 3 + heads * dk]
    kernels = kernels_for(dtype, heads, kv_heads, dk, dk)
    assert dtype == torch.float32 or dk % 8 or len(kernels) >= 3
    pos = torch.arange(S, dtype=torch.int32, device=dev)
    for name, tile in kernels.items():
        run = lambda lo, hi, ctx=0: blocks.paged_attention(q[lo:hi].to(dev), slab, table, tile_list(dev, hi - lo, tile), pos[lo:hi], kv_heads=kv_heads, dv=dk,
                                                           mask=blocks.MASK_CHUNK, mask_size=size, scale=dk ** -0.5, gate=gate[lo:hi], kernel=name, max_context=ctx)
        close(run(0, S), want, 3e-6 if dtype == torch.float32 else 2e-2)
        close(run(S - 9, S), want[S - 9 :], 3e-6 if dtype == torch.float32 else 2e-2)
        close(run(S - 1, S, S), want[S - 1 :], 3e-6 if dtype == torch.float32 else 2e-2)  # the key range may be split over CTAs
    per_head = wide.to(dev)[:, :heads]  # one logit per head is still that
    want = O.chunk_attention(q.double(), k.double(), v.double(), scale=dk ** -0.5, size=size) * torch.sigmoid(wide[:, :heads].double())[:, :, None]
    for name, tile in kernels.items():
        got = blocks.paged_attention(q.to(dev), slab, table, tile_list(dev, S, tile), pos, kv_heads=kv_heads, dv=dk, mask=blocks.MASK_CHUNK, mask_size=size,
                                     scale=dk ** -0.5, gate=per_head, kernel=name)
        close(got, want, 3e-6 if dtype == torch.float32 else 2e-2)


def test_a_gate_is_merged_once_when_the_older_tensor_core_kernel_splits_the_keys(dev):
    g = torch.Generator().manual_seed(3)
    S, heads, kv_heads, dk, bf = 900, 4, 2, 32, torch.bfloat16
    q, k, v = (torch.randn(S, n, dk, generator=g).to(bf) for n in (heads, kv_heads, kv_heads))
    gate = torch.randn(S, heads * dk, generator=g).to(bf)
    want = O.chunk_attention(q.double(), k.double(), v.double(), scale=dk ** -0.5, size=880)[[879, 899]] * torch.sigmoid(gate.double()).view(S, heads, dk)[[879, 899]]
    slab, table = cached(dev, bf, k, v)
    for name in ("mma", "flash_split"):
        rows = [blocks.paged_attention(q[i : i + 1].to(dev), slab, table, ints(dev, [(0, 1, 0)]), ints(dev, [i]), kv_heads=kv_heads, dv=dk, mask=blocks.MASK_CHUNK,
                                       mask_size=880, scale=dk ** -0.5, gate=gate[i : i + 1].to(dev), kernel=name, max_context=i + 1) for i in (879, 899)]
        close(torch.cat(rows), want, 2e-2)


class OnePlan:
    """What an attention layer asks of a step's plan, for one sequence's tokens [lo, hi)."""

    def __init__(self, dev, lo, hi, table):
        self.dev, self.count = dev, hi - lo
        self.tok_pos = torch.arange(lo, hi, dtype=torch.int32, device=dev)
        self.tok_seq = torch.zeros_like(self.tok_pos)
        self.block_table, self.max_context, self.max_tokens = table, hi, hi - lo

    def tiles_for(self, size):
        return tile_list(self.dev, self.count, size)

    def rope_tables(self, dims, base, factor=1.0, ramp=None):
        return blocks.rope_table(self.tok_pos, dims=dims, base=base, factor=factor, ramp=ramp)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,d,dims,size", [(4, 2, 16, 8, 24), (6, 3, 10, 10, 31), (4, 1, 64, 32, 64), (2, 2, 40, 0, 17), (3, 1, 7, 4, 50)])
def test_values_are_the_keys_before_their_rotation(dev, dtype, heads, kv_heads, d, dims, size):
    """Projections through the module: the cache holds turned keys beside the keys as projected, the projection itself stays,
    and the rows are the plain ones - whole, in portions and one by one."""
    g = torch.Generator().manual_seed(d)
    T, page, base = 100, 32, 77.0
    H, G = heads, kv_heads
    y = torch.randn(T, (H + G + H) * d, generator=g).to(dtype)
    layer = PagedGroupedAttention(heads=H, kv_heads=G, dim=d, vdim=d, scale=0.3, mask="chunk", mask_size=size, w_o=torch.zeros(8, H * d, dtype=dtype, device=dev),
                                  page_size=page, values="keys", rot={"dims": dims, "base": base} if dims else None)
    q, k, gate = (t.double() for t in y.split([H * d, G * d, H * d], dim=1))
    turn = lambda x, n: O.rotate(x.view(T, n, d), dims, base) if dims else x.view(T, n, d)
    want = O.chunk_attention(turn(q, H), turn(k, G), k.view(T, G, d), scale=0.3, size=size) * torch.sigmoid(gate).view(T, H, d)
    tol = 5e-6 if dtype == torch.float32 else 3e-2
    table = ints(dev, [[3, 0, 4, 1]])
    for cuts in ([0, 100], [0, 2, 31, 33, 97, 100], list(range(0, 40)) + [100]):
        slab = torch.full((5, page, G * 2 * d), 7.0, dtype=dtype, device=dev)
        got = []
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            yd = y[lo:hi].to(dev)
            qd, kd, gd = yd.split([H * d, G * d, H * d], dim=1)
            got.append(layer.attend(qd, kd, None, gd, OnePlan(dev, lo, hi, table), slab))
            assert torch.equal(kd.cpu(), y[lo:hi, H * d : (H + G) * d])
        close(torch.cat(got), want, tol)
        rows = torch.stack([slab[table[0, t // page], t % page] for t in range(T)]).cpu()
        close(rows[:, : G * d], turn(k, G).reshape(T, -1), 3e-6 if dtype == torch.float32 else 1e-2)
        assert torch.equal(rows[:, G * d :], y[:, H * d : (H + G) * d])
    with pytest.raises(ValueError, match="values"):
        PagedGroupedAttention(heads=H, kv_heads=G, dim=d, vdim=d + 1, scale=1.0, mask="chunk", mask_size=size, w_o=torch.zeros(8, H * (d + 1), device=dev), values="keys")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [1, 5, 31, 32, 64, 70])
def test_one_key_that_matters_just_inside_and_just_outside_a_chunk(dev, dtype, size):
    """All keys are noise but one that the probing query scores far above the rest: the output is that key's value exactly when
    both lie in the same chunk.  Prompt rows and single tokens, pages of 32."""
    g = torch.Generator().manual_seed(size)
    S, d = 300, 16
    for target in (0, size - 1, size, 31, 32, 2 * size, 3 * size - 1, 160):
        if not 0 <= target < S:
            continue
        k, v = 0.05 * torch.randn(S, 1, d, generator=g), torch.randn(S, 1, d, generator=g)
        k[target, 0, 3], v[target] = 40.0, 5.0
        q = torch.zeros(S, 2, d)
        q[:, :, 3] = 1.0
        slab, table = cached(dev, dtype, k, v, seed=target)
        pos = torch.arange(S, dtype=torch.int32, device=dev)
        for name, tile in kernels_for(dtype, 2, 1, d, d).items():
            run = lambda lo, hi: blocks.paged_attention(q[lo:hi].to(dtype).to(dev), slab, table, tile_list(dev, hi - lo, tile), pos[lo:hi], kv_heads=1, dv=d,
                                                        mask=blocks.MASK_CHUNK, mask_size=size, scale=1.0, kernel=name).float().cpu()
            whole = run(0, S)
            last = (target // size + 1) * size - 1
            for i in sorted({target - 1, target, target + 1, last, last + 1, last + size, S - 1}):
                if not 0 <= i < S:
                    continue
                sees = O.visible(i, target, size)
                one = run(i, i + 1)[0]
                for row in (whole[i], one):
                    assert (row - 5.0).abs().max() < 2e-2 if sees else (row - 5.0).abs().min() > 0.2, (name, i, target)


# ---------------------------------------------------------------------------------------------- matrix memory
def memory_case(dtype, heads, dk, dv, T, seed, width=40):
    g = torch.Generator().manual_seed(seed)
    w = {"i": torch.randn(heads, width, generator=g), "f": torch.randn(heads, width, generator=g), "i.b": torch.randn(heads, generator=g) - 1.0,
         "f.b": 4.0 + 2.0 * torch.randn(heads, generator=g), "norm": 1 + 0.2 * torch.randn(heads * dv, generator=g),
         "o": torch.eye(heads * dv)}
    y = {"q": torch.randn(T, heads * dk, generator=g), "k": torch.randn(T, heads * dk, generator=g), "v": torch.randn(T, heads * dv, generator=g),
         "g": torch.randn(T, heads * dv, generator=g), "h": torch.randn(T, width, generator=g)}
    return {n: t.to(dtype) for n, t in w.items()}, {n: t.to(dtype) for n, t in y.items()}


def memory_want(w, y, heads, dk, dv, cap, eps):
    T = y["q"].shape[0]
    w, y = {n: t.double() for n, t in w.items()}, {n: t.double() for n, t in y.items()}
    log_in = O.soft_bound(y["h"] @ w["i"].t() + w["i.b"], cap)
    log_forget = O.log_sigmoid(O.soft_bound(y["h"] @ w["f"].t() + w["f.b"], cap))
    o = O.matrix_memory(y["q"].view(T, heads, dk) / math.sqrt(dk), y["k"].view(T, heads, dk), y["v"].view(T, heads, dv), log_in, log_forget)
    return O.rms_unit(o, eps).reshape(T, -1) * w["norm"] * torch.sigmoid(y["g"])


class MemoryPlan:
    def __init__(self, dev, rows):
        self.seq_info, self.max_tokens = ints(dev, rows), max(r[1] for r in rows)


class MemoryBench:
    """A MatrixMemory over slots that are wider than its share and hold stale numbers."""

    def __init__(self, dev, dtype, w, heads, dk, dv, cap, eps, slots=4):
        self.dev = dev
        w = {n: t.to(dev) for n, t in w.items()}
        self.m = MatrixMemory(heads=heads, dim=dk, vdim=dv, gate_cap=cap, w_i=w["i"], b_i=w["i.b"], w_f=w["f"], b_f=w["f.b"], norm_weight=w["norm"], w_o=w["o"], eps=eps)
        n = heads * dk * (dv + 1)
        self.pool = torch.full((slots, 3 + n + heads + 2), 9.0, device=dev)
        self.state, self.peak = self.pool[:, 3 : 3 + n].unflatten(1, self.m.state_shape), self.pool[:, 3 + n : 3 + n + heads]

    def run(self, y, spans):
        """``spans``: [(first row, count, position of the first row, slot)]; their rows form one step."""
        rows, at = [], 0
        for _, count, start, slot in spans:
            rows.append((at, count, start, slot))
            at += count
        part = {n: torch.cat([t[lo : lo + count] for lo, count, _, _ in spans]).to(self.dev) for n, t in y.items()}
        out = self.m(part["h"], part["q"], part["k"], part["v"], part["g"], MemoryPlan(self.dev, rows), self.state, self.peak)
        assert float(self.pool[:, :3].min()) == 9.0 and float(self.pool[:, -2:].min()) == 9.0  # the neighbours' columns
        return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dk,dv,cap", [(2, 16, 32, 9.0), (3, 12, 40, 15.0), (1, 64, 31, 4.0), (2, 33, 7, 30.0), (1, 200, 64, 6.0), (5, 8, 1, 1.0)])
def test_matrix_memory_whole_in_portions_token_by_token_and_in_a_batch(dev, dtype, heads, dk, dv, cap):
    w, y = memory_case(dtype, heads, dk, dv, 300, dk)
    eps = 1e-5
    a = memory_want(w, {n: t[:230] for n, t in y.items()}, heads, dk, dv, cap, eps)   # rows 0..229 are one sequence, 230..299 another
    b = memory_want(w, {n: t[230:] for n, t in y.items()}, heads, dk, dv, cap, eps)
    tol = 5e-5 if dtype == torch.float32 else 2e-2  # bf16: the normed rows and the identity product round
    bench = MemoryBench(dev, dtype, w, heads, dk, dv, cap, eps)
    close(bench.run(y, [(0, 230, 0, 2)]), a, tol)                                     # segments, from a stale slot
    both = bench.run(y, [(230, 60, 0, 1), (0, 100, 0, 3)])                            # unequal, in one step
    close(both[:60], b[:60], tol), close(both[60:], a[:100], tol)
    rest = bench.run(y, [(100, 130, 100, 3), (290, 1, 60, 1)])                        # each goes on from its slot, the order turned round
    close(rest[:130], a[100:], tol), close(rest[130:], b[60:61], tol)
    at = 0
    for n in [2, 2, 3, 64, 5, 1, 63, 65, 25]:                                         # slot 3 again, by a new sequence
        close(bench.run(y, [(at, n, at, 3)]), a[at : at + n], tol)
        at += n
    rows = [bench.run(y, [(230 + t, 1, t, 3), (t, 1, t, 0)]) for t in range(70)]      # two sequences, a token each
    close(torch.cat([r[:1] for r in rows]), b, tol), close(torch.cat([r[1:] for r in rows]), a[:70], tol)


@pytest.mark.parametrize("inline", [True, False])
def test_the_running_maximum_starts_at_nought_and_lives_in_the_slot(dev, inline):
    """Gates far below 0 everywhere: m follows f down from 0 until i catches it, and the floor exp(-m), not the normaliser, divides."""
    heads, cap, T, D = 3, 8.0, 700, 24
    g = torch.Generator().manual_seed(5)
    z = torch.cat([-6 + 3 * torch.randn(T, heads, generator=g), 3 + 3 * torch.randn(T, heads, generator=g)], dim=1)
    z[350, 0] = 100.0                      # one input gate at the cap
    z[400:420, heads:] = -100.0            # everything is forgotten
    h, w = torch.randn(T, D, generator=g), torch.zeros(2 * heads, D)
    if inline:                             # the projection that gives z, to fp32 accuracy: columns of z in h, picked by w
        h[:, : 2 * heads], w = z, torch.eye(2 * heads, D)
    bias = torch.randn(2 * heads, generator=g)
    li = O.soft_bound(z[:, :heads].double() + bias[:heads].double(), cap)
    lf = O.log_sigmoid(O.soft_bound(z[:, heads:].double() + bias[heads:].double(), cap))
    m, want = torch.zeros(heads, dtype=torch.float64), []
    for t in range(T):
        top = torch.maximum(lf[t] + m, li[t])
        want.append(torch.stack([torch.exp(lf[t] + m - top), torch.exp(li[t] - top), torch.exp(-top)], dim=-1))
        m = top
    want = torch.stack(want)
    state = torch.full((2, heads + 1), 9.0, device=dev)
    for cuts in ([0, 1, 2, 250, 251, 300, 700], [0, 700], list(range(0, 60)) + [700]):
        got = []
        for lo, hi in zip(cuts[:-1], cuts[1:]):
            args = dict(h=h[lo:hi].to(dev), w=w.to(dev)) if inline else {}
            step, floor = blocks.matrix_memory_gates(None if inline else z[lo:hi].to(dev), **args, bias=bias.to(dev), cap=cap, heads=heads, seq_info=ints(dev, [[0, hi - lo, lo, 1]]),
                                                     state=state[:, :heads], max_tokens=hi - lo)
            got.append(torch.cat([step, floor[..., None]], dim=-1))
        got = torch.cat(got).double().cpu()
        assert float(((got - want).abs() / want.abs().clamp_min(1e-3)).max()) < 2e-4   # a log of rounding eps times the largest log weight
        close(state[1, :heads], m, 1e-5)
        assert float(state[0].min()) == 9.0 and float(state[1, heads]) == 9.0
    assert want[0, :, 2].max() < 1.5 and want[:350, :, 2].max() > 20.0                  # the floor starts near exp(0) and rises


def test_one_write_is_read_hundreds_of_tokens_later_and_gone_after_a_forget(dev):
    """Input gates shut but one token's: its value comes back for every later query that meets its key, until a token forgets."""
    heads, dk, dv, T, D, cap, eps = 1, 8, 16, 600, 6, 12.0, 1e-6
    y = {n: torch.zeros(T, s) for n, s in (("q", dk), ("k", dk), ("v", dv), ("g", dv), ("h", D))}
    g = torch.Generator().manual_seed(1)
    y["k"], y["v"], y["g"] = torch.randn(T, dk, generator=g), torch.randn(T, dv, generator=g), torch.full((T, dv), 20.0)
    y["q"][:, 0] = 3.0
    y["h"][:, 0], y["h"][:, 1] = -100.0, 100.0         # input gate at -cap, forget gate at +cap
    y["h"][37, 0] = 100.0
    y["k"][37], y["v"][37] = torch.eye(dk)[0], torch.linspace(-2, 3, dv)
    y["h"][500:504, 1] = -100.0       # e^-12 each: one would leave it as large as the writes that follow
    w = {"i": torch.eye(1, D), "f": torch.eye(2, D)[1:], "i.b": torch.zeros(1), "f.b": torch.zeros(1), "norm": torch.ones(dv), "o": torch.eye(dv)}
    want = memory_want(w, y, heads, dk, dv, cap, eps)
    stored = O.rms_unit(y["v"][37].double(), eps)
    assert (want[37:500] - stored).abs().max() < 5e-2 and (want[510] - stored).abs().max() > 0.3
    bench = MemoryBench(dev, torch.float32, w, heads, dk, dv, cap, eps)
    close(bench.run(y, [(0, 600, 0, 0)]), want, 5e-5)
    close(torch.cat([bench.run(y, [(0, 30, 0, 1)])] + [bench.run(y, [(t, 1, t, 1)]) for t in range(30, 600)]), want, 5e-5)


# ---------------------------------------------------------------------------------------------- experts
def expert_case(dtype, D, experts, identity, expert_ff, shared_ff, seed):
    g = torch.Generator().manual_seed(seed)
    n = experts + identity
    mat = lambda r, c, gain=1.0: (torch.randn(r, c, generator=g) * gain / c ** 0.5).to(dtype)
    w = {"router": mat(n, D, 2.0), "correction": (-0.3 + 0.15 * torch.randn(n, generator=g)).to(dtype)}  # most choice scores below 0
    for name, ff in [(f"e{e}.", expert_ff) for e in range(experts)] + ([("shared.", shared_ff)] if shared_ff else []):
        w[name + "gate"], w[name + "up"], w[name + "down"] = mat(ff, D, 2.5), mat(ff, D, 2.5), mat(D, ff)
    if shared_ff:
        w["shared.sg"] = mat(1, D, 3.0)
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,identity,top,groups,T", [(6, 2, 2, (2, 1), 70), (12, 4, 3, (4, 2), 300), (5, 1, 1, (6, 3), 40), (3, 3, 4, None, 33), (40, 32, 5, (36, 4), 64),
                                                           (7, 0, 7, (1, 1), 9)])
def test_grouped_choice_clamped_experts_and_a_gated_shared_expert(dev, dtype, experts, identity, top, groups, T):
    D, ff, sff, n = 48, 24, 56, experts + identity
    w = expert_case(dtype, D, experts, identity, ff, sff, experts * 31 + top)
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(top)).to(dtype)
    spec = {"router": {"experts": experts, "identity": identity, "top": top}, "expert": {"limit": 0.9}, "shared": {"limit": 1.6}}
    if groups:
        spec["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    wd = {k: t.double() for k, t in w.items()}
    scores = torch.softmax(h.double() @ wd["router"].t(), dim=-1)
    chosen = torch.tensor([O.choose(s, wd["correction"], top, spec["router"].get("groups")) for s in scores])
    router = TopKRouter(w["router"].to(dev), None, top, scoring="softmax_all", choice_bias=w["correction"].to(dev), groups=groups)
    idx, gate, side = router(h.to(dev), w["shared.sg"].to(dev))
    assert torch.equal(idx.cpu().long(), chosen)  # fp32 scores of rounded inputs: no close calls in these draws
    picked = scores.gather(1, chosen)
    close(gate, picked / picked.sum(1, keepdim=True), 1e-5)
    close(side, torch.sigmoid(h.double() @ wd["shared.sg"].t())[:, 0], 1e-5)
    if groups and groups[1] < groups[0] and top > groups[1]:
        free = torch.tensor([O.choose(s, wd["correction"], top) for s in scores])
        assert (free != chosen).any(1).float().mean() > 0.1  # the groups matter
    stack = lambda part: torch.stack([w[f"e{e}.{part}"] for e in range(experts)]).to(dev)
    shared = GatedMLP(*(w["shared." + part].to(dev) for part in ("gate", "up", "down")), "clamped_swish", limit=1.6, slope=1.702)
    moe = MixtureOfExperts(router, stack("gate"), stack("up"), stack("down"), "clamped_swish", shared, identity=identity, limit=0.9, slope=1.702, shared_gate=w["shared.sg"].to(dev))
    want = O.expert_mixture(h.double(), wd, "", spec)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    close(moe(h.to(dev)), want, tol)
    if dtype == torch.float32:  # the limits bind, and which of the two belongs to whom
        assert row_error(moe(h.to(dev)), O.expert_mixture(h.double(), wd, "", dict(spec, expert={"limit": 1.6}))) > 1e-3
        assert row_error(moe(h.to(dev)), O.expert_mixture(h.double(), wd, "", dict(spec, shared={"limit": 0.9}))) > 1e-3
    # the fused end of the sublayer: the sum through a tanh norm into the stream, and the norm that reads it next
    g = torch.Generator().manual_seed(9)
    norms = {}
    for name, alpha in (("post", 0.9), ("next", 0.5)):
        norms[name], norms[name + ".b"], norms[name + ".alpha"] = (1 + 0.3 * torch.randn(D, generator=g)).to(dtype), (0.3 * torch.randn(D, generator=g)).to(dtype), torch.tensor(alpha).to(dtype)
    post, following = (TanhNorm(norms[name].to(dev), norms[name + ".b"].to(dev), norms[name + ".alpha"].to(dev)) for name in ("post", "next"))
    x0 = torch.randn(T, D, generator=g)
    nd = {k: t.double() for k, t in norms.items()}
    x1 = x0.double() + O.tanh_norm(want, nd, "post")
    x = x0.to(dev)
    out = moe(h.to(dev), into=(x, post, following))
    close(x, x1, tol)
    close(out, O.tanh_norm(x1, nd, "next"), tol)
    x = x0.to(dev)
    assert moe(h.to(dev), into=(x, post, None)) is None
    close(x, x1, tol)


def test_router_rejects_groups_that_cannot_give_the_choices(dev):
    w = torch.zeros(8, 16, device=dev)
    for groups, top in (((3, 1), 1), ((4, 5), 1), ((4, 0), 1), ((4, 1), 3), ((0, 0), 1)):
        with pytest.raises(ValueError, match="groups"):
            TopKRouter(w, None, top, scoring="softmax_all", groups=groups)
    assert TopKRouter(w, None, 2, scoring="softmax_all", groups=(4, 1)).groups == (4, 1)


# ---------------------------------------------------------------------------------------------- the model
CONFIGS = {
    # both mixers, a layer without feed-forward, chunks of several sizes, a sharp softmax
    "mixed": dict(pattern="MmAmMnAmAn", width=96, vocab=160, chunks=(24, 70, 33)),
    # what usually differs made equal, or 1: one key/value head per head, all of every head rotated, one memory head with dim = vdim, the chunk a page,
    # one group, top 1, no identity experts, expert and shared expert alike
    "equal": dict(pattern="AmMm", width=64, vocab=97, heads=2, kv_heads=2, dim=32, rot_dims=32, chunks=(64,), scale=1.0, mem_heads=1, mem_dim=32, mem_vdim=32, experts=4,
                  identity=0, top=1, groups=(1, 1), expert_ff=64, shared_ff=64, limit=1.0, shared_limit=1.0),
    # sizes that are multiples of nothing: the general attention kernel, groups of three heads, no 16-byte access fits
    "odd": dict(pattern="MnAmAnMm", width=54, vocab=131, heads=6, kv_heads=2, dim=10, rot_dims=6, rot_base=77.0, chunks=(29, 31), mem_heads=3, mem_dim=9, mem_vdim=14,
                gate_cap=4.0, experts=7, identity=2, top=3, groups=(3, 2), expert_ff=10, shared_ff=22, limit=0.7, shared_limit=3.0, eps=1e-3),
    # neither groups nor a shared expert nor a rotation; more identity experts than real ones; one key/value head for more query heads than a CTA holds
    "plain": dict(pattern="AmMm", width=72, vocab=90, heads=40, kv_heads=1, dim=8, rot_dims=0, chunks=(50,), experts=2, identity=4, top=4, groups=None, shared_ff=0),
    # no attention layer at all (no pages are ever read)
    "recurrent": dict(pattern="MmMn", width=50, vocab=91, mem_heads=2, mem_dim=70, mem_vdim=40, gate_cap=15.0),
    # no recurrent layer at all (no state slots), chunks of one token and far beyond the prompt
    "attention": dict(pattern="AmAnAm", width=56, vocab=80, chunks=(1, 4096, 65), dim=24, rot_dims=24, top=1, experts=3, identity=1, groups=(2, 1)),
}
_models = {}


def model_and_oracle(dev, name, dtype, max_tokens=None, max_requests=None):
    key = (name, dtype, max_tokens, max_requests)
    if key not in _models:
        config = nomudra_config(**CONFIGS[name])
        tensors = synthetic_nomudra(config, seed=len(name), sharp=2.0 if name == "mixed" else 1.0)
        model = model_class("Nomudra").from_checkpoint(config, tensors, dtype=dtype, device=dev, max_tokens=max_tokens, max_requests=max_requests)
        _models[key] = (model, config, tensors)
    return _models[key]


def run_schedule(model, prompts, schedule):
    """``schedule``: steps of [(request, count)]; every position's logits are collected.  Requests end (and give their
    pages and state slot back) with their last token."""
    caches, at, got = {}, {r: 0 for r in prompts}, {r: [] for r in prompts}
    for step in schedule:
        entries = []
        for r, n in step:
            caches.setdefault(r, model.create_kv_cache())
            entries.append(RaggedEntry(prompts[r][at[r] : at[r] + n], caches[r], want=range(n)))
        logits = model.forward_ragged(entries).cpu()
        k = 0
        for r, n in step:
            got[r].append(logits[k : k + n])
            k += n
            at[r] += n
            if at[r] == len(prompts[r]):
                caches.pop(r)[0].release()
    return {r: torch.cat(v) for r, v in got.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_matches_the_plain_model(dev, name, dtype):
    model, config, tensors = model_and_oracle(dev, name, dtype)
    prompt = ids_for(150, config["vocab"], 1)
    want = O.forward(prompt, tensors, config)
    got = run_schedule(model, {"a": prompt}, [[("a", len(prompt))]])["a"]
    assert rows_match(got, want, dtype)
    cache = model.create_kv_cache()                                      # some rows wanted, in any order; none at all
    some = model.forward_ragged([RaggedEntry(prompt, cache, want=[149, 3, 80])])
    assert row_error(some, got[[149, 3, 80]].double()) < (2e-5 if dtype == torch.float32 else 2e-2)
    cache[0].release()
    cache = model.create_kv_cache()
    assert model.forward_ragged([RaggedEntry(prompt[:140], cache, want=[])]).shape == (0, config["vocab"])
    rest = model.forward_ragged([RaggedEntry(prompt[140:], cache, want=range(10))])
    cache[0].release()
    if dtype == torch.float32:  # in bfloat16 ten rows say little: a close router call moves a token and, through the memory, those after it
        assert row_error(rest, want[140:]) < 5e-5
    else:
        assert row_errors(rest, want[140:]).median().item() < 1.5e-1


@pytest.mark.parametrize("name", list(CONFIGS))
def test_layers_one_by_one(dev, name):
    """The residual sum after every layer (float32 mode), tapped from the model's own step."""
    model, config, tensors = model_and_oracle(dev, name, torch.float32)
    prompt = ids_for(70, config["vocab"], 2)
    want = []
    O.forward(prompt, tensors, config, tap=want)
    cache = model.create_kv_cache()
    model.stream_tap = []
    try:
        model.forward_ragged([RaggedEntry(prompt, cache)])
        assert len(model.stream_tap) == len(want) == len(config["layers"])
        for x, w in zip(model.stream_tap, want):
            close(x, w, 2e-5)
    finally:
        model.stream_tap = None
        cache[0].release()


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_every_mechanism_of_the_configuration_shows_in_the_logits(dev, name):
    """A plain model with one thing planted wrong differs from the framework's logits by far more than the tolerance."""
    import copy

    model, config, tensors = model_and_oracle(dev, name, torch.float32)
    prompt = ids_for(120, config["vocab"], 1)
    got = run_schedule(model, {"a": prompt}, [[("a", len(prompt))]])["a"]

    def differs(change_config=lambda c: None, change_tensors=lambda t: None):
        c, t = copy.deepcopy(config), {n: w.clone() for n, w in tensors.items()}
        change_config(c)
        change_tensors(t)
        return row_error(got, O.forward(prompt, t, c)) > 1e-3

    each = lambda kind, change: lambda c: [change(l["mixer"]) for l in c["layers"] if l["type"] == kind]
    routed = lambda change: lambda c: [change(l["mlp"]) for l in c["layers"] if l["mlp"]]
    zero = lambda *ends: lambda t: [t[n].zero_() for n in t if n.endswith(ends)]
    assert differs(each("attention", lambda m: m["mask"].update(size=m["mask"]["size"] + 1)))
    assert differs(each("attention", lambda m: m["rot"].update(base=2 * m["rot"]["base"])))
    assert differs(each("attention", lambda m: m.update(scale=1.2 * m["scale"])))
    assert differs(each("mlstm", lambda m: m.update(gate_cap=0.7 * m["gate_cap"])))
    for end in ("q.b", "k.b", "o.b", "i.b", "f.b", ".correction", "shared.sg", "mix.g", "norm1b.b", "norm2b.b", "embed.norm.b"):
        assert differs(change_tensors=zero(end)), end
    assert differs(change_tensors=lambda t: [t[n].mul_(1.3) for n in t if n.endswith(".alpha")])
    assert differs(routed(lambda f: f["router"].pop("groups")))
    assert differs(routed(lambda f: f["expert"].update(limit=9.0))) and differs(routed(lambda f: f["shared"].update(limit=0.5 * f["shared"]["limit"])))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "equal", "odd", "recurrent"])
def test_prefill_then_token_by_token_decoding_across_pages_and_chunks(dev, name, dtype):
    model, config, tensors = model_and_oracle(dev, name, dtype)
    prompt = ids_for(100 + 120, config["vocab"], 3)  # 120 decoded tokens: page borders and chunks pass by
    want = O.forward(prompt, tensors, config)
    replays = model.graph_replays
    got = run_schedule(model, {"a": prompt}, [[("a", 100)]] + [[("a", 1)]] * 120)["a"]
    assert rows_match(got, want, dtype)
    assert model.graph_replays - replays >= 110  # single-token steps replay a captured graph from their third step on
    model.use_decode_graph = False
    try:
        eager = run_schedule(model, {"a": prompt}, [[("a", 100)]] + [[("a", 1)]] * 120)["a"]
    finally:
        model.use_decode_graph = None
    assert row_error(eager, got.double()) < 1e-6
    alone = run_schedule(model, {"a": prompt[:40]}, [[("a", 1)]] * 40)["a"]  # the first tokens, one by one from nothing
    # in bfloat16 against the same tokens run as a prompt: a close router call goes the same way in both
    assert rows_match(alone, want[:40] if dtype == torch.float32 else got[:40].double(), dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_of_every_size_down_to_two(dev, name):
    model, config, tensors = model_and_oracle(dev, name, torch.float32)
    prompt = ids_for(203, config["vocab"], 4)
    want = O.forward(prompt, tensors, config)
    for sizes in ([2] * 20 + [3, 5, 64, 23, 2, 33, 31, 2], [63, 1, 64, 2, 62, 11], [7] * 29, [128, 75]):
        assert sum(sizes) == len(prompt)
        got = run_schedule(model, {"a": prompt}, [[("a", n)] for n in sizes])["a"]
        assert row_error(got, want) < 5e-5, sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_equal_each_alone_and_pages_and_slots_are_reused(dev, dtype):
    model, config, tensors = model_and_oracle(dev, "mixed", dtype, max_tokens=5 * 64, max_requests=3)  # 5 pages, 3 state slots in all
    prompts = {"a": ids_for(130, 160, 5), "b": ids_for(61, 160, 6), "c": ids_for(3, 160, 7), "d": ids_for(100, 160, 8), "e": ids_for(64, 160, 9)}
    want = {r: O.forward(p, tensors, config) for r, p in prompts.items()}
    schedule = [[("a", 60), ("b", 2)], [("a", 2), ("b", 58), ("c", 1)], [("a", 1), ("b", 1), ("c", 2)],   # b and c end: 2 pages and 2 slots back
                [("a", 30), ("d", 50)], [("a", 37), ("d", 1)],                                           # a ends (3 pages), d in a reused page and slot
                [("d", 49), ("e", 64)]]                                                                  # e fills a whole reused page
    got = run_schedule(model, prompts, schedule)
    pool, states = model.page_pool, model.state_pool
    assert pool.reused_page_allocations >= 3 and pool.capacity == 5 and not pool.used_page_ids
    assert states.reused_slot_allocations >= 2 and states.capacity == 3 and not states.used_slots
    for r in prompts:
        assert rows_match(got[r], want[r], dtype), r
    if dtype == torch.float32:  # and the same as alone up to the summation order of the library products (which follows the row count)
        alone = run_schedule(model, {"d": prompts["d"]}, [[("d", 50)], [("d", 1)], [("d", 49)]])["d"]
        assert row_error(alone, got["d"].double()) < 2e-5
    with pytest.raises(RuntimeError, match="exhausted"):
        run_schedule(model, {"x": ids_for(330, 160, 1)}, [[("x", 330)]])
    assert not pool.used_page_ids and not states.used_slots  # the refused step took nothing
    live = [model.create_kv_cache() for _ in range(4)]
    with pytest.raises(RuntimeError, match="state slots exhausted"):
        model.forward_ragged([RaggedEntry([1, 2], c) for c in live])
    assert not pool.used_page_ids and not states.used_slots


def test_a_request_left_out_of_steps_goes_on_from_its_slot(dev):
    model, config, tensors = model_and_oracle(dev, "mixed", torch.float32)
    a, b = ids_for(60, 160, 41), ids_for(50, 160, 42)
    wa, wb = O.forward(a, tensors, config), O.forward(b, tensors, config)
    ca, cb = model.create_kv_cache(), model.create_kv_cache()
    model.forward_ragged([RaggedEntry(a[:30], ca), RaggedEntry(b[:7], cb)])
    for t in range(7, 20):                                            # only b runs
        assert row_error(model.forward_ragged([RaggedEntry(b[t : t + 1], cb)]), wb[t : t + 1]) < 5e-5
    got = model.forward_ragged([RaggedEntry(b[20:21], cb), RaggedEntry(a[30:33], ca, want=range(3))])
    assert row_error(got, torch.cat([wb[20:21], wa[30:33]])) < 5e-5
    assert row_error(model.forward_ragged([RaggedEntry(a[33:], ca, want=range(27))]), wa[33:]) < 5e-5
    with pytest.raises(NotImplementedError):
        ca[0].rewind(1)
    ca[0].release(), cb[0].release()


@pytest.mark.parametrize("seed", range(12))
def test_random_stacks_and_sizes_in_random_schedules(dev, seed):
    """Layer order, head counts, sizes, chunks, rotations, caps, routers and the schedule all drawn at random (float32): one
    request whole and in random portions, three requests interleaved."""
    import random

    rng = random.Random(seed)
    pattern = "".join(rng.choice("AM") + rng.choice("mmn") for _ in range(rng.randint(1, 5)))
    kv, dim = rng.choice([1, 2, 3]), rng.choice([6, 8, 10, 16, 24, 40])
    count = rng.choice([1, 2, 3, 4])
    size = rng.randint(1, 4)
    outputs = count * size
    keep = rng.randint(1, count)
    identity = rng.randint(0, outputs - 1)
    config = nomudra_config(pattern=pattern, width=rng.choice([40, 50, 64, 72, 100, 136]), vocab=rng.choice([61, 128, 301]), heads=kv * rng.choice([1, 2, 3]), kv_heads=kv,
                            dim=dim, chunks=tuple(rng.choice([1, 2, 17, 31, 32, 33, 64, 100, 128, 1000]) for _ in range(3)), rot_dims=rng.choice([0, 2, dim // 4 * 2, dim]),
                            rot_base=rng.choice([50.0, 1e4, 1e6]), scale=rng.choice([None, 0.15, 1.0]), mem_heads=rng.randint(1, 5),
                            mem_dim=rng.choice([3, 8, 16, 33, 64]), mem_vdim=rng.choice([2, 16, 31, 32, 33, 70]), gate_cap=rng.choice([1.0, 5.0, 15.0, 30.0]),
                            experts=outputs - identity, identity=identity, top=rng.randint(1, keep * size), groups=rng.choice([(count, keep), (count, keep), None]),
                            expert_ff=rng.choice([10, 24, 32]), limit=rng.choice([0.5, 1.5, 7.0]), shared_ff=rng.choice([0, 20, 64]), shared_limit=rng.choice([0.5, 1.5, 7.0]),
                            eps=rng.choice([1e-6, 1e-5, 1e-3]))
    tensors = synthetic_nomudra(config, seed=seed, sharp=rng.choice([1.0, 2.0]))
    model = model_class("Nomudra").from_checkpoint(config, tensors, dtype=torch.float32, device=dev, max_tokens=8 * 64, max_requests=3)
    V, T = config["vocab"], rng.choice([70, 131, 200])
    prompts = {"a": ids_for(T, V, seed), "b": ids_for(45, V, seed + 50), "c": ids_for(90, V, seed + 99)}
    want = {r: O.forward(p, tensors, config) for r, p in prompts.items()}
    assert row_error(run_schedule(model, {"a": prompts["a"]}, [[("a", T)]])["a"], want["a"]) < 5e-5, config
    sizes, left = [], T
    while left:
        n = min(left, rng.choice([1, 2, 2, 3, 7, 30, 64, 70]))
        sizes.append(n)
        left -= n
    assert row_error(run_schedule(model, {"a": prompts["a"]}, [[("a", n)] for n in sizes])["a"], want["a"]) < 5e-5, (config, sizes)
    at, schedule = {r: 0 for r in prompts}, []
    while any(at[r] < len(prompts[r]) for r in prompts):
        step = []
        for r in prompts:
            room = len(prompts[r]) - at[r]
            if room and rng.random() < 0.7:
                n = min(room, rng.choice([1, 1, 2, 5, 40]))
                step.append((r, n))
                at[r] += n
        if step:
            schedule.append(step)
    got = run_schedule(model, prompts, schedule)
    for r in prompts:
        assert row_error(got[r], want[r]) < 1e-4, (r, config)
    assert not model.page_pool.used_page_ids and not model.state_pool.used_slots


@pytest.mark.parametrize("seed", range(4))
def test_random_stacks_in_the_serving_dtype(dev, seed):
    """Sizes that take the register-softmax kernel's forms and sizes that do not, in bfloat16: whole, and decoded after a prompt."""
    import random

    rng = random.Random(100 + seed)
    kv, dim = rng.choice([1, 2, 3]), rng.choice([8, 24, 32, 64, 128, 136])
    config = nomudra_config(pattern=rng.choice(["AmMm", "MnAmMm", "AmAm"]), width=rng.choice([56, 96, 128]), vocab=rng.choice([64, 101]), heads=kv * rng.choice([1, 3, 4, 20]),
                            kv_heads=kv, dim=dim, chunks=(rng.choice([3, 31, 64, 65, 128]),), rot_dims=rng.choice([2, dim // 8 * 8, dim // 4 * 2]),
                            mem_heads=rng.randint(1, 3), mem_dim=rng.choice([16, 48, 128]), mem_vdim=rng.choice([8, 64, 96]))
    tensors = synthetic_nomudra(config, seed=seed)
    model = model_class("Nomudra").from_checkpoint(config, tensors, dtype=torch.bfloat16, device=dev, max_tokens=6 * 64)
    prompt = ids_for(200, config["vocab"], seed)
    want = O.forward(prompt, tensors, config)
    assert rows_match(run_schedule(model, {"a": prompt}, [[("a", 200)]])["a"], want, torch.bfloat16), config
    got = run_schedule(model, {"a": prompt}, [[("a", 97)], [("a", 2)], [("a", 65)]] + [[("a", 1)]] * 36)["a"]
    assert rows_match(got, want, torch.bfloat16), config


def test_long_decoding(dev):
    """500 single-token steps after a two-token prompt (graph replays over growing block tables, chunks beginning anew), against
    the plain model."""
    model, config, tensors = model_and_oracle(dev, "mixed", torch.float32)
    prompt = ids_for(502, config["vocab"], 12)
    want = O.forward(prompt, tensors, config)
    got = run_schedule(model, {"a": prompt}, [[("a", 2)]] + [[("a", 1)]] * 500)["a"]
    assert row_error(got, want) < 5e-5


def test_rectangular_call_scheduler_slots_and_offsets(dev):
    model, config, tensors = model_and_oracle(dev, "mixed", torch.float32)
    p0, p1 = ids_for(9, 160, 10), ids_for(5, 160, 11)
    c0, c1 = model.create_kv_cache(), model.create_kv_cache()
    l0 = model(torch.tensor([p0], dtype=torch.int32, device=dev), 0, c0)                 # all rows
    l1 = model(torch.tensor([p1], dtype=torch.int32, device=dev), 0, c1, logits_to_keep=1)
    assert l0.shape == (1, 9, 160) and l1.shape == (1, 1, 160)
    assert row_error(l0[0], O.forward(p0, tensors, config)) < 2e-5
    with pytest.raises(ValueError, match="offset"):
        model(torch.tensor([[1]], dtype=torch.int32, device=dev), 3, c0)
    tables = [BatchingKvCache(max_active_requests=3) for _ in range(model.num_hidden_layers)]
    for t, a, b in zip(tables, c0, c1):
        t.add_request(a, 2)
        t.add_request(b, 0)
    out = model(torch.tensor([[7], [0], [8]], dtype=torch.int32, device=dev), [5, 0, 9], tables, logits_to_keep=1)
    assert out.shape == (3, 1, 160) and float(out[1].abs().max()) == 0.0               # the idle slot
    assert row_error(out[2, 0], O.forward(p0 + [8], tensors, config)[-1]) < 2e-5
    assert row_error(out[0, 0], O.forward(p1 + [7], tensors, config)[-1]) < 2e-5
    for t in tables:
        t.remove_request(0), t.remove_request(2)
    assert not model.page_pool.used_page_ids and not model.state_pool.used_slots


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_points(dev, dtype, tmp_path):
    """greedy_generate_ids and the continuous batcher (mixed steps, 2 slots, 5 requests, pages reused) produce the plain model's
    greedy tokens; the checkpoint goes through a directory and load_model."""
    config = nomudra_config(**CONFIGS["mixed"])
    tensors = synthetic_nomudra(config, seed=21)
    save_nomudra(config, tensors, tmp_path / "ckpt")
    model = load_model(tmp_path / "ckpt", device=dev, dtype=dtype, max_tokens=6 * 64, max_requests=3)
    prompts = [ids_for(n, 160, 30 + n) for n in (5, 70, 2, 33, 64)]
    new = 20
    want = [O.greedy(p, tensors, config, new) for p in prompts]
    if dtype == torch.float32:
        assert greedy_generate_ids(model, prompts[1], new, device=dev) == want[1]
    batcher = ContinuousBatcher(model, None, prompts, max_seq_len=128, batch_size=2, prefill_step=16, verbose=False, device=dev,
                                max_new_tokens=[new] * len(prompts))
    results = dict(batcher.run())
    got = [[int(t) for t in results[i].split()] for i in range(len(prompts))]
    if dtype == torch.float32:
        assert got == want
    else:  # bf16: the same tokens until a near-tie, at least the first one of most requests
        assert sum(g[:1] == w[:1] for g, w in zip(got, want)) >= len(prompts) - 1
    assert batcher.mixed and batcher.mixed_steps > 0 and model.page_pool.reused_page_allocations > 0
    assert not model.page_pool.used_page_ids and not model.state_pool.used_slots and model.state_pool.reused_slot_allocations > 0


def test_trace_program_replays_steps_and_writes_logits(dev, tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np

    config = nomudra_config(**CONFIGS["odd"])
    tensors = synthetic_nomudra(config, seed=4)
    save_nomudra(config, tensors, tmp_path / "ckpt")
    V = config["vocab"]
    a, b = ids_for(70, V, 1), ids_for(9, V, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:], "want": [0, 3]}, {"id": "b", "tokens": b, "want": [8]}], "end": ["a", "b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": b, "want": [0]}], "end": ["c"]}]
    root = Path(__file__).resolve().parent.parent
    run = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path / "ckpt"), "--dtype", "float32",
                          "--out", str(tmp_path / "out"), "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "out" / "0.f32").exists()
    got = torch.from_numpy(np.fromfile(tmp_path / "out" / "1.f32", dtype="<f4").reshape(3, V))
    wa, wb = O.forward(a, tensors, config), O.forward(b, tensors, config)
    assert row_error(got, torch.stack([wa[66], wa[69], wb[8]])) < 2e-5
    got = torch.from_numpy(np.fromfile(tmp_path / "out" / "2.f32", dtype="<f4").reshape(1, V))
    assert row_error(got, wb[:1]) < 2e-5


def test_command_line_generates_and_batches(dev, tmp_path, capsys):
    from tiny_llm_b200 import cli

    config = nomudra_config(**CONFIGS["equal"])
    tensors = synthetic_nomudra(config, seed=8)
    save_nomudra(config, tensors, tmp_path / "ckpt")
    prompt = ids_for(11, 97, 5)
    want = O.greedy(prompt, tensors, config, 6)
    assert cli.main(["generate", "--model", str(tmp_path / "ckpt"), "--dtype", "float32", "--prompt-ids", ",".join(map(str, prompt)),
                     "--max-new-tokens", "6"]) == 0
    assert [int(t) for t in capsys.readouterr().out.split()] == want
    assert cli.main(["batch", "--model", str(tmp_path / "ckpt"), "--dtype", "float32", "--quiet", "--batch-size", "2", "--prefill-step", "4",
                     "--max-new-tokens", "6", "--prompt-ids", ";".join(",".join(map(str, ids_for(n, 97, n))) for n in (11, 3, 7))]) == 0
    out = capsys.readouterr().out
    assert out.count("--- request") == 3
    first = out.split("--- request 0\n")[1].split("\n")[0]
    assert [int(t) for t in first.split()] == O.greedy(ids_for(11, 97, 11), tensors, config, 6)
    assert cli.main(["generate", "--synthetic", "nomudra:MmAn", "--prompt-ids", "5,17,3", "--max-new-tokens", "4"]) == 0
    assert len(capsys.readouterr().out.split()) == 4
