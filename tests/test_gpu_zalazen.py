"""Zalazen on a B200 against the plain CPU restatement (oracle/zalazen.py, float64): each mechanism that the design added to
the blocks library alone, then the model through every way of cutting and batching a sequence, the schedulers and the
entry points.  Small made-up configurations and random weights; where random weights would hide a fault (a far key among
hundreds, a sink, the edge of a window, a kept first position) the inputs are built so that it shows.

Tolerances: relative root-mean-square error of a logits row (mean taken off) below 5e-5 in float32 mode - every product in
true fp32, so only summation order differs.  In bfloat16 mode whole schedules are held to a median of 3e-2 and 95 % of the
rows below 1.5e-1; the float32 run is the sharp test.
"""

import pytest
import torch

from oracle import zalazen as O
from extensions_b200.tiny_llm_ext_b200 import blocks
from tiny_llm_b200 import BatchingKvCache, ContinuousBatcher, greedy_generate_ids
from tiny_llm_b200.models import load_model, model_class
from tiny_llm_b200.positional_encoding import yarn_ramp
from tiny_llm_b200.ragged import RaggedEntry
from tiny_llm_b200.synthetic import save_zalazen, synthetic_zalazen, zalazen_config

pytestmark = pytest.mark.gpu
D64 = torch.float64
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
    return err.median().item() < 3e-2 and err.quantile(0.95).item() < 1.5e-1


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs().max().item()
    scale = want.abs().max().item() + 1e-9
    assert err <= tol * scale, (err, scale)


def ids_for(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def ints(dev, values):
    return torch.tensor(values, dtype=torch.int32).to(dev)


# ---------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,buckets,mul_prev,mul_cur", [(96, 61, 7, 3), (50, 1, 5, 9), (7, 1000, 10**12 + 39, 10**11 + 3), (4100, 37, 40, 100), (2048, 300, 0, 1),
                                                          (256, (1 << 20) + 7, (1 << 20) + 6, (1 << 20) + 5)])
def test_embedding_rows_with_the_token_before(dev, dtype, dim, buckets, mul_prev, mul_cur):
    """Two sequences that continue (one by a single token), two that start; the token before from the batch, from the cache's
    history, or none; ids large enough that the products leave 32 bits."""
    g = torch.Generator().manual_seed(dim)
    vocab, scale, eps = 5000, 3.5, 1e-5
    table = torch.randn(vocab, dim, generator=g).to(dtype)
    rows = min(buckets, 2000) + 1
    pairs = torch.randn(rows, dim, generator=g).to(dtype)
    if buckets + 1 > rows:                                       # a table too big to fill at random: its rows repeat
        pairs = pairs.repeat(-(-(buckets + 1) // rows), 1)[: buckets + 1].contiguous()
    w1, w2 = (1 + 0.3 * torch.randn(dim, generator=g)).to(dtype), (1 + 0.3 * torch.randn(dim, generator=g)).to(dtype)
    ids = [4999, 4998, 0, 17, 17, 4999, 3, 0]
    seq, pos, prev = [0, 0, 0, 1, 2, 2, 3, 3], [70, 71, 72, 5, 0, 1, 0, 1], [0, 4997, -1, -1]
    want = []
    for t, i in enumerate(ids):
        before = None if pos[t] == 0 else (ids[t - 1] if t and seq[t - 1] == seq[t] else prev[seq[t]])
        want.append(table[i].double() * scale + pairs[O.bigram_row(before, i, mul_prev=mul_prev, mul_cur=mul_cur, buckets=buckets)].double())
    want = torch.stack(want)
    d = lambda t: t.to(dev)
    x, h1, h2 = blocks.embed_pairs(ints(dev, ids), d(table), scale, pairs=d(pairs), mul_prev=mul_prev, mul_cur=mul_cur, tok_pos=ints(dev, pos),
                                   tok_seq=ints(dev, seq), seq_prev=ints(dev, prev), weight=d(w1), weight2=d(w2), eps=eps)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    close(x, want, 1e-6)
    close(h1, O.rms_unit(want, eps) * w1.double(), tol)
    close(h2, O.rms_unit(want, eps) * w2.double(), tol)
    x1, h, none = blocks.embed_pairs(ints(dev, ids), d(table), scale, pairs=d(pairs), mul_prev=mul_prev, mul_cur=mul_cur, tok_pos=ints(dev, pos),
                                     tok_seq=ints(dev, seq), seq_prev=ints(dev, prev), weight=d(w1), eps=eps)
    assert torch.equal(x1, x) and torch.equal(h, h1) and none is None
    x, h, none = blocks.embed_pairs(ints(dev, ids), d(table), 1.0)                 # no pair table, no norms
    assert h is None and none is None and torch.equal(x.cpu(), table[ids].float())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [7, 50, 256, 1024, 2050, 2300, 9000])
def test_residual_sum_with_two_norms(dev, dtype, dim):
    g = torch.Generator().manual_seed(dim)
    rows, eps = 5, 1e-5
    res, a, b, row = (torch.randn(rows, dim, generator=g) for _ in range(3)), None, None, torch.randn(dim, generator=g)
    res, a, b = res
    w1, w2 = (1 + 0.3 * torch.randn(dim, generator=g)).to(dtype), (1 + 0.3 * torch.randn(dim, generator=g)).to(dtype)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    for first, second in ((a, b), (a, None), (row, None), (row, b)):
        x = res.to(dev)
        h1, h2 = blocks.add_norm(x, first.to(dev), None if second is None else second.to(dev), w1.to(dev), eps, w2.to(dev))
        want = res.double() + first.double() + (0 if second is None else second.double())
        close(x, want, 1e-6)
        close(h1, O.rms_unit(want, eps) * w1.double(), tol)
        close(h2, O.rms_unit(want, eps) * w2.double(), tol)
        again = res.to(dev)
        one = blocks.add_norm(again, first.to(dev), None if second is None else second.to(dev), w1.to(dev), eps)
        assert torch.equal(one, h1) and torch.equal(again, x)
        assert blocks.add_norm(again, first.to(dev), None, None, eps) is None


@pytest.mark.parametrize("dims,base,scaling", [(8, 3e4, (4.0, 512, 16.0, 1.0)), (64, 1e4, (8.0, 4096, 32.0, 1.0)), (2, 500.0, (3.0, 64, 8.0, 2.0)),
                                               (16, 100.0, (2.0, 100000, 64.0, 60.0)), (130, 1e6, (1.0, 1024, 32.0, 1.0)), (12, 1e4, None)])
def test_rotation_tables_stretched_by_frequency(dev, dims, base, scaling):
    names = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    freqs, gain = O.frequencies({"dims": dims, "base": base, "scaling": names})
    pos = [0, 1, 2, 63, 64, 1000, 131071, 1 << 20]
    cs, sn = blocks.rope_table(ints(dev, pos), dims=dims, base=base, ramp=None if names is None else yarn_ramp(dims, base, **names))
    a = torch.tensor(pos, dtype=D64)[:, None] * torch.tensor(freqs, dtype=D64)
    close(cs, torch.cos(a) * gain, 1e-6)
    close(sn, torch.sin(a) * gain, 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("first,width", [(16, 24), (9, 24), (5, 13), (0, 40)])
def test_gated_activation_and_attention_meet_in_one_product(dev, dtype, first, width):
    """The activation lands in columns of a wider matrix (neighbours untouched); the joined product equals the sum of both."""
    from tiny_llm_b200.paged_attention import JoinedProjection

    g = torch.Generator().manual_seed(first * 100 + width)
    T, D = 11, 32
    gu = torch.randn(T, 2 * width, generator=g).to(dtype)
    u = torch.randn(T, max(first, 1), generator=g).to(dtype)
    w_a, w_b = torch.randn(D, max(first, 1), generator=g).to(dtype), torch.randn(D, width, generator=g).to(dtype)
    parts = ([("a", w_a.to(dev))] if first else []) + [("b", w_b.to(dev))]
    joined = JoinedProjection(parts)
    x, part = joined.operand(T)
    x.fill_(7.0)
    if first:
        part["a"].copy_(u.to(dev))
    out = blocks.gated_act(gu.to(dev), blocks.ACT_SILU, out=part["b"])
    assert out.data_ptr() == part["b"].data_ptr()
    inner = O.silu(gu.double()[:, :width]) * gu.double()[:, width:]
    close(part["b"], inner, 2e-6 if dtype == torch.float32 else 1e-2)
    if first:
        assert torch.equal(part["a"].cpu(), u)
    want = part["b"].double().cpu() @ w_b.double().t() + (u.double() @ w_a.double().t() if first else 0)
    tf32 = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        got = joined(x)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = tf32
    assert got.dtype == torch.float32
    close(got, want, 2e-6)


def fill_cache(dev, rows, page_size, dtype):
    """rows [T, width] -> (slab, block_table) with the tokens' pages in a scrambled order."""
    T, width = rows.shape
    pages = -(-T // page_size)
    order = torch.randperm(pages + 3, generator=torch.Generator().manual_seed(T))[:pages]
    slab = torch.full((pages + 3, page_size, width), 50.0, dtype=dtype, device=dev)     # stale numbers in every unused slot
    for p in range(pages):
        part = rows[p * page_size : (p + 1) * page_size]
        slab[order[p], : part.shape[0]] = part.to(dev)
    return slab, order.to(torch.int32).reshape(1, -1).to(dev)


def tiles_for(dev, first, count, size):
    return ints(dev, [(first + lo, min(size, count - lo), 0) for lo in range(0, count, size)])


WINDOWS = [(24, 0), (24, 1), (24, 5), (31, 32), (20, 33), (64, 64), (70, 3), (1, 4), (1, 0), (33, 100), (5, 700), (1000, 2)]


def attention_choices(dtype, heads, kv_heads, dk, dv):
    """(kernel, most tokens of a work-list entry) of every kernel that serves these sizes."""
    return [blocks.paged_attention_kernel(dtype, heads, kv_heads, dk, dv, 64)] + list(blocks.paged_attention_flash_forms(dtype, heads, kv_heads, dk, dv, 64).items())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dk,dv", [(4, 2, 16, 24), (6, 2, 12, 10), (40, 1, 8, 16)])
@pytest.mark.parametrize("size,keep", WINDOWS)
def test_window_with_kept_first_positions_and_sinks_at_every_edge(dev, dtype, heads, kv_heads, dk, dv, size, keep):
    """One key carries nearly all the weight: by its head, a query asks for the oldest position of its window (inside), the one
    before that (outside, unless kept), the last kept position, the first one that is not kept, position 0, or itself.  Whole
    prompts, single decoded tokens, portions of two; the output written into columns of a wider matrix."""
    g = torch.Generator().manual_seed(heads + size + keep)
    T, scale, group = 420, 0.5, heads // kv_heads
    k = torch.randn(T, kv_heads, dk, generator=g)
    k = 4.0 * k / k.norm(dim=2, keepdim=True)
    v = torch.randn(T, kv_heads, dv, generator=g)
    q = 0.1 * torch.randn(T, heads, dk, generator=g)
    for p in range(T):
        for h in range(heads):
            target = (p - size + 1, p - size, keep - 1, keep, 0, p)[h % 6]
            if 0 <= target < T:
                q[p, h] = 3.0 * k[target, h // group]
    sink, gate = torch.randn(heads, generator=g), torch.randn(T, heads, generator=g)
    q, k, v, gate = q.to(dtype), k.to(dtype), v.to(dtype), gate.to(dtype)
    plain = lambda keep: O.sink_window_attention(q.double(), k.double(), v.double(), sink.double(), scale=scale, size=size, keep_first=keep)
    want = plain(keep) * torch.sigmoid(gate.double())[:, :, None]
    slab, table = fill_cache(dev, torch.cat([k.reshape(T, -1), v.reshape(T, -1)], dim=1), 64, dtype)
    pos = torch.arange(T, dtype=torch.int32, device=dev)
    qd, gd, tol = q.to(dev), gate.to(dev), 2e-5 if dtype == torch.float32 else 3e-2

    for kernel, tile in attention_choices(dtype, heads, kv_heads, dk, dv):
        def run(lo, hi, keep=keep, sink_on=True, split=True):
            wide = torch.full((hi - lo, heads * dv + 5), 3.0, dtype=dtype, device=dev)
            blocks.paged_attention(qd[lo:hi], slab, table, tiles_for(dev, 0, hi - lo, tile), pos[lo:hi], kv_heads=kv_heads, dv=dv, mask=blocks.MASK_WINDOW,
                                   mask_size=size, keep_first=keep, scale=scale, sink=sink_on, head_bias=sink.to(dev) if sink_on else None, gate=gd[lo:hi],
                                   kernel=kernel, max_context=hi if split else 0, out=wide[:, : heads * dv].unflatten(1, (heads, dv)))
            assert float(wide[:, -5:].float().sub(3.0).abs().max()) == 0.0
            return wide[:, : heads * dv].unflatten(1, (heads, dv))

        whole = run(0, T)
        close(whole, want, tol)
        cut = torch.cat([run(lo, min(lo + 170, T), split=False) for lo in range(0, T, 170)])
        assert torch.equal(cut, run(0, T, split=False))                      # where a prompt was cut leaves no trace (one CTA per tile)
        close(torch.cat([run(p, p + 1) for p in list(range(0, 70, 3)) + list(range(380, T))]), torch.cat([want[0:70:3], want[380:]]), tol)
        close(torch.cat([run(p, p + 2) for p in range(180, 240, 2)]), want[180:240], tol)
        if heads >= 6:                                                       # the construction shows what it is meant to show
            assert (run(0, T, sink_on=False).double().cpu() - want).abs().max() > 0.05
        if 0 < keep < 300 and size < 200 and (heads >= 4 or keep == 1):
            assert (plain(keep - 1) * torch.sigmoid(gate.double())[:, :, None] - want).abs().max() > 0.05
            assert (run(0, T, keep=keep - 1).double().cpu() - want).abs().max() > 0.05


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_kept_position_thousands_of_keys_back(dev, dtype):
    """A step of one token over a long context: pages between the kept ones and the window are never read (they hold
    not-a-number), whatever the split of the key range."""
    T, heads, kv_heads, dk, dv, size, keep = 5000, 4, 2, 16, 16, 700, 40
    g = torch.Generator().manual_seed(9)
    k, v, q = torch.randn(T, kv_heads, dk, generator=g), torch.randn(T, kv_heads, dv, generator=g), torch.randn(1, heads, dk, generator=g)
    k[37] *= 3.0
    q[0] = k[37].repeat_interleave(2, 0)
    rows = torch.cat([k.reshape(T, -1), v.reshape(T, -1)], dim=1).to(dtype)
    see = [j for j in range(T) if O.visible(T - 1, j, size, keep)]
    assert len(see) == size + keep
    want = torch.zeros(1, heads, dv, dtype=D64)
    sink = torch.randn(heads, generator=g)
    qd, kd, vd = q.to(dtype).double(), k.to(dtype).double(), v.to(dtype).double()
    for h in range(heads):
        e = torch.exp(0.25 * kd[see, h // 2] @ qd[0, h])
        want[0, h] = (e / (e.sum() + torch.exp(sink[h].double()))) @ vd[see, h // 2]
    slab, table = fill_cache(dev, rows, 64, dtype)
    dead = [p for p in range(-(-T // 64)) if p * 64 + 63 < T - size - 64 and p * 64 >= 64]
    slab[table[0, dead].long()] = float("nan")
    choices = attention_choices(dtype, heads, kv_heads, dk, dv)
    assert len(choices) == (1 if dtype == torch.float32 else 3)
    for (kernel, tile), max_context in [(c, m) for c in choices for m in (0, T)]:   # one CTA per tile, or the key range split over several
        out = blocks.paged_attention(q.to(dtype).to(dev), slab, table, tiles_for(dev, 0, 1, tile), ints(dev, [T - 1]), kv_heads=kv_heads, dv=dv,
                                     mask=blocks.MASK_WINDOW, mask_size=size, keep_first=keep, scale=0.25, sink=True, head_bias=sink.to(dev), kernel=kernel,
                                     max_context=max_context)
        close(out, want, 2e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dk,dv,dims", [(4, 2, 16, 24, 8), (6, 3, 12, 10, 6), (1, 1, 64, 8, 2), (16, 2, 128, 64, 32), (3, 1, 24, 24, 24)])
@pytest.mark.parametrize("tokens", [70, 2600])
def test_whole_projection_norms_with_a_stretched_rotation_into_the_cache(dev, dtype, heads, kv_heads, dk, dv, dims, tokens):
    """Norm over all heads at once, partial rotation by ramped tables, keys and values into pages in reverse order; aligned and
    odd column starts; small steps and steps of thousands of tokens (both forms of the kernel)."""
    g = torch.Generator().manual_seed(heads * 31 + dk)
    eps, base, page, start = 1e-5, 5e4, 32, 1000
    rot = {"dims": dims, "base": base, "scaling": {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 0.5}}
    ramp = yarn_ramp(dims, base, **rot["scaling"])
    wq, wk = (1 + 0.3 * torch.randn(heads * dk, generator=g)).to(dtype), (1 + 0.3 * torch.randn(kv_heads * dk, generator=g)).to(dtype)
    check = list(range(0, tokens, max(1, tokens // 40)))
    freqs, gain = O.frequencies(rot)

    def turned(x, w, n):
        y = (O.rms_unit(x.double(), eps) * w.double()).view(-1, n, dk)[check]
        a = torch.tensor([start + t for t in check], dtype=D64)[:, None, None] * torch.tensor(freqs, dtype=D64)
        c, s, half = torch.cos(a) * gain, torch.sin(a) * gain, dims // 2
        u, v = y[..., :half], y[..., half:dims]
        return torch.cat([u * c - v * s, v * c + u * s, y[..., dims:]], dim=-1).reshape(len(check), n * dk)

    for gap in (0, 3):                                                   # the parts' first columns aligned, or not
        cols = [heads * dk, kv_heads * dk, kv_heads * dv]
        wide = torch.randn(tokens, sum(cols) + 2 * gap + 8, generator=g).to(dtype)
        at = [0, cols[0] + gap, cols[0] + cols[1] + 2 * gap]
        take = lambda m: [m[:, a : a + c] for a, c in zip(at, cols)]
        q, k, v = take(wide)
        wd = wide.to(dev)
        qd, kd, vd = take(wd)
        pages = (start + tokens) // page + 1
        slab = torch.zeros((pages, page, kv_heads * (dk + dv)), dtype=dtype, device=dev)
        table = torch.arange(pages - 1, -1, -1, dtype=torch.int32, device=dev).reshape(1, -1)
        pos = torch.arange(start, start + tokens, dtype=torch.int32, device=dev)
        blocks.qk_whole_prepare(qd, kd, vd, heads=heads, kv_heads=kv_heads, q_norm=wq.to(dev), k_norm=wk.to(dev), eps=eps, rot_dims=dims, base=base,
                                tok_pos=pos, tok_seq=torch.zeros_like(pos), block_table=table, slab=slab,
                                rope=blocks.rope_table(pos, dims=dims, base=base, ramp=ramp))
        tol = 3e-6 if dtype == torch.float32 else 1e-2
        close(qd[check], turned(q, wq, heads), tol)
        rows = torch.stack([slab[pages - 1 - (start + t) // page, (start + t) % page] for t in check])
        close(rows[:, : kv_heads * dk], turned(k, wk, kv_heads), tol)
        assert torch.equal(rows[:, kv_heads * dk :].cpu(), v[check])
        assert torch.equal(wd[:, heads * dk :].cpu(), wide[:, heads * dk :])  # keys, values and neighbours untouched
        alone = wide.to(dev)                                              # queries only: a layer that reads another layer's cache
        blocks.qk_whole_prepare(take(alone)[0], None, None, heads=heads, kv_heads=kv_heads, q_norm=wq.to(dev), eps=eps, rot_dims=dims, base=base, tok_pos=pos,
                                rope=blocks.rope_table(pos, dims=dims, base=base, ramp=ramp))
        assert torch.equal(alone, wd)


# ---------------------------------------------------------------------------------------------- the model
CONFIGS = {
    # own and shared caches, layers without a feed-forward, windows and kept positions of several sizes, a sharp softmax
    "mixed": dict(pattern="AdSdAnSnAd", width=96, vocab=160, windows=((24, 3), (40, 0), (70, 37), (1, 2))),
    # what usually differs made equal, or 1: one key/value head per head, dim = vdim, all of every head rotated, window = kept = page, one bucket
    "equal": dict(pattern="AdAd", width=64, vocab=97, heads=2, kv_heads=2, dim=32, vdim=32, rot_dims=32, windows=((64, 64),), ff=64, buckets=1, embed_scale=1.0,
                  scale=1.0, scaling=(1.0, 64, 4.0, 1.0)),
    # sizes that are multiples of nothing: the general attention kernel, groups of three, widths no 16-byte access fits
    "odd": dict(pattern="AnSdSdAd", width=54, vocab=131, heads=6, kv_heads=2, dim=10, vdim=7, rot_dims=6, windows=((29, 5), (33, 1)), ff=50, buckets=77,
                mul_prev=1000003, mul_cur=998244353, eps=1e-5, scaling=(16.0, 100, 30.0, 0.5)),
    # neither pair table nor stretched rotation nor kept positions
    "plain": dict(pattern="AdSd", width=64, vocab=120, buckets=0, scaling=None, windows=((50, 0),)),
    # one key/value head for many query heads, more than a CTA's 32 rows hold
    "group": dict(pattern="AdSd", width=72, vocab=90, heads=40, kv_heads=1, dim=8, vdim=16, rot_dims=4, windows=((30, 33),)),
}
_models = {}


def model_and_oracle(dev, name, dtype, max_tokens=None, max_requests=None):
    key = (name, dtype, max_tokens, max_requests)
    if key not in _models:
        config = zalazen_config(**CONFIGS[name])
        tensors = synthetic_zalazen(config, seed=len(name), sharp=2.5 if name == "mixed" else 1.0)
        model = model_class("Zalazen").from_checkpoint(config, tensors, dtype=dtype, device=dev, max_tokens=max_tokens, max_requests=max_requests)
        _models[key] = (model, config, tensors)
    return _models[key]


def run_schedule(model, prompts, schedule):
    """``schedule``: steps of [(request, count)]; every position's logits are collected.  Requests end (and give their
    pages back) with their last token."""
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


@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_mechanism_of_the_configuration_shows_in_the_logits(dev, name):
    """A plain model with one thing planted wrong differs from the framework's logits by far more than the tolerance."""
    import copy

    model, config, tensors = model_and_oracle(dev, name, torch.float32)
    prompt = ids_for(150, config["vocab"], 1)
    got = run_schedule(model, {"a": prompt}, [[("a", len(prompt))]])["a"]

    def differs(change_config=lambda c: None, change_tensors=lambda t: None):
        c, t = copy.deepcopy(config), {n: w.clone() for n, w in tensors.items()}
        change_config(c)
        change_tensors(t)
        return row_error(got, O.forward(prompt, t, c)) > 1e-3

    def every_mask(key, by):
        return lambda c: [l["mixer"]["mask"].__setitem__(key, max(0, l["mixer"]["mask"][key] + by)) for l in c["layers"]]

    assert differs(every_mask("size", 1))
    assert differs(every_mask("keep_first", 1))
    assert differs(change_tensors=lambda t: [t[n].fill_(-100.0) for n in t if n.endswith(".sink")])
    assert differs(change_tensors=lambda t: [t[n].fill_(0.0) for n in t if n.endswith(".mix.g")])
    assert differs(lambda c: [l["mixer"]["rot"].__setitem__("base", 2 * l["mixer"]["rot"]["base"]) for l in c["layers"]])
    if CONFIGS[name].get("scaling", (4.0,)) and CONFIGS[name].get("scaling", (4.0,))[0] != 1.0:
        assert differs(lambda c: [l["mixer"]["rot"].pop("scaling") for l in c["layers"]])
    if config["embedding"].get("bigram", {}).get("buckets", 0) > 1:
        assert differs(lambda c: c["embedding"]["bigram"].__setitem__("mul_prev", c["embedding"]["bigram"]["mul_prev"] + 1))
    if any("kv_from" in l["mixer"] for l in config["layers"]) and name in ("mixed", "odd"):
        last = max(i for i, l in enumerate(config["layers"]) if "kv_from" not in l["mixer"])
        assert differs(change_tensors=lambda t: t[f"l{last}.mix.k"].mul_(1.0 + 0.5 * torch.arange(t[f"l{last}.mix.k"].shape[0])[:, None] % 2))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "equal", "odd"])
def test_prefill_then_token_by_token_decoding_across_pages_and_windows(dev, name, dtype):
    model, config, tensors = model_and_oracle(dev, name, dtype)
    prompt = ids_for(100 + 120, config["vocab"], 3)  # 120 decoded tokens: page borders and windows pass by
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
    assert rows_match(alone, want[:40], dtype)


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
def test_unequal_requests_in_one_batch_equal_each_alone_and_pages_are_reused(dev, dtype):
    model, config, tensors = model_and_oracle(dev, "mixed", dtype, max_tokens=5 * 64, max_requests=3)
    V = config["vocab"]
    prompts = {"a": ids_for(130, V, 5), "b": ids_for(3, V, 6), "c": ids_for(66, V, 7), "d": ids_for(90, V, 8), "e": ids_for(40, V, 9)}
    want = {r: O.forward(p, tensors, config) for r, p in prompts.items()}
    schedule = [[("a", 60), ("b", 1)], [("a", 2), ("b", 2), ("c", 30)], [("a", 68), ("c", 36)],  # a, b, c end: 3 + 1 + 2 pages come back
                [("d", 64), ("e", 1)], [("d", 1), ("e", 38)], [("d", 25), ("e", 1)]]
    got = run_schedule(model, prompts, schedule)
    for r in prompts:
        assert rows_match(got[r], want[r], dtype), r
    assert model.page_pool.reused_page_allocations > 0 and not model.page_pool.used_page_ids
    if dtype == torch.float32:  # alone, through other pages: the same numbers up to the library products' tile choice
        alone = run_schedule(model, {"d": prompts["d"]}, [[("d", 90)]])["d"]
        assert row_error(alone, got["d"].double()) < 2e-5
    # a step that finds no pages leaves nothing behind, neither in the page list nor in the history of tokens
    caches = [model.create_kv_cache() for _ in range(2)]
    model.forward_ragged([RaggedEntry([1, 2], c) for c in caches])
    with pytest.raises(RuntimeError, match="exhausted"):
        model.forward_ragged([RaggedEntry([4], caches[1]), RaggedEntry(list(range(150)) * 3, caches[0])])
    assert [c[0].offset for c in caches] == [2, 2] and [list(c[0].tokens) for c in caches] == [[1, 2], [1, 2]]
    for c in caches:
        c[0].release()
    assert not model.page_pool.used_page_ids


def test_a_request_left_out_of_steps_and_one_taken_back_keep_their_token_before(dev):
    model, config, tensors = model_and_oracle(dev, "mixed", torch.float32)
    V = config["vocab"]
    a, b = ids_for(60, V, 41), ids_for(50, V, 42)
    wa, wb = O.forward(a, tensors, config), O.forward(b, tensors, config)
    ca, cb = model.create_kv_cache(), model.create_kv_cache()
    model.forward_ragged([RaggedEntry(a[:30], ca), RaggedEntry(b[:7], cb)])
    for t in range(7, 20):                                            # only b runs
        got = model.forward_ragged([RaggedEntry(b[t : t + 1], cb)])
        assert row_error(got, wb[t : t + 1]) < 5e-5
    got = model.forward_ragged([RaggedEntry(b[20:21], cb), RaggedEntry(a[30:33], ca, want=range(3))])
    assert row_error(got, torch.cat([wb[20:21], wa[30:33]])) < 5e-5
    model.forward_ragged([RaggedEntry([1, 2, 3, 4], ca)])               # tokens that are taken back again
    ca[0].rewind(4)
    got = model.forward_ragged([RaggedEntry(a[33:], ca, want=range(27))])
    assert row_error(got, wa[33:]) < 5e-5
    ca[0].release(), cb[0].release()


@pytest.mark.parametrize("seed", range(10))
def test_random_stacks_and_sizes_in_random_schedules(dev, seed):
    """Layer order, shared caches, head counts and groups, sizes, windows, kept positions, rotations and pair tables drawn at
    random; the prompt whole, in random portions, and as three interleaved requests, in float32."""
    g = torch.Generator().manual_seed(1000 + seed)
    pick = lambda *options: options[int(torch.randint(0, len(options), (1,), generator=g))]
    layers = int(pick(2, 3, 4))
    pattern = "A" + pick("d", "d", "n") + "".join(pick("A", "S") + pick("d", "d", "n") for _ in range(layers - 1))
    kv_heads, dim = pick(1, 2, 3), pick(8, 10, 16, 24)
    config = zalazen_config(pattern=pattern, width=pick(36, 56, 96, 130), vocab=pick(64, 101), heads=kv_heads * pick(1, 2, 4), kv_heads=kv_heads, dim=dim,
                            vdim=pick(8, 12, 16, 40), windows=tuple((pick(1, 3, 31, 64, 65, 128), pick(0, 1, 4, 32, 65)) for _ in range(3)),
                            rot_dims=pick(2, dim // 2 * 2, dim // 4 * 2 or 2), rot_base=pick(50.0, 1e4, 1e6),
                            scaling=pick(None, (2.0, 64, 8.0, 1.0), (40.0, 4096, 32.0, 1.0), (8.0, 128, 100.0, 0.01)), scale=pick(None, 0.1, 1.0),
                            ff=pick(24, 64, 75), embed_scale=pick(0.5, 1.0, 7.0), buckets=pick(0, 1, 64, 1009), mul_prev=pick(1, 31, 70001), mul_cur=pick(1, 17, 99991),
                            eps=pick(1e-6, 1e-5, 1e-3))
    tensors = synthetic_zalazen(config, seed=seed, sharp=pick(1.0, 2.0))
    model = model_class("Zalazen").from_checkpoint(config, tensors, dtype=torch.float32, device=dev, max_tokens=6 * 64, max_requests=3)
    V = config["vocab"]
    prompts = {"a": ids_for(160, V, seed), "b": ids_for(45, V, seed + 50), "c": ids_for(90, V, seed + 99)}
    want = {r: O.forward(p, tensors, config) for r, p in prompts.items()}
    assert row_error(run_schedule(model, {"a": prompts["a"]}, [[("a", 160)]])["a"], want["a"]) < 5e-5, config
    sizes, left = [], 160
    while left:
        n = min(left, int(pick(1, 2, 2, 3, 7, 30, 64, 70)))
        sizes.append(n)
        left -= n
    assert row_error(run_schedule(model, {"a": prompts["a"]}, [[("a", n)] for n in sizes])["a"], want["a"]) < 5e-5, (config, sizes)
    at, schedule = {r: 0 for r in prompts}, []
    while any(at[r] < len(prompts[r]) for r in prompts):
        step = []
        for r in prompts:
            room = len(prompts[r]) - at[r]
            if room and pick(True, True, False):
                n = min(room, int(pick(1, 1, 2, 5, 40)))
                step.append((r, n))
                at[r] += n
        if step:
            schedule.append(step)
    got = run_schedule(model, prompts, schedule)
    for r in prompts:
        assert row_error(got[r], want[r]) < 1e-4, (r, config)
    assert not model.page_pool.used_page_ids


@pytest.mark.parametrize("seed", range(8))
def test_random_stacks_in_the_serving_dtype(dev, seed):
    """Sizes that take the register-softmax kernel's forms and sizes that do not, in bfloat16: whole, and decoded after a prompt."""
    g = torch.Generator().manual_seed(2000 + seed)
    pick = lambda *options: options[int(torch.randint(0, len(options), (1,), generator=g))]
    kv_heads, dim = pick(1, 2, 3), pick(8, 24, 32, 64, 128, 144)
    config = zalazen_config(pattern=pick("AdSd", "AnAdSd", "AdAd"), width=pick(56, 96, 128), vocab=pick(64, 101), heads=kv_heads * pick(1, 3, 4, 20), kv_heads=kv_heads,
                            dim=dim, vdim=pick(8, 12, 32, 64, 104, 128, 200), windows=tuple((pick(3, 31, 64, 65, 128), pick(0, 1, 32, 65)) for _ in range(3)),
                            rot_dims=pick(2, dim // 8 * 8, dim // 4 * 2), ff=pick(24, 64, 75), buckets=pick(0, 64, 1009))
    tensors = synthetic_zalazen(config, seed=seed)
    model = model_class("Zalazen").from_checkpoint(config, tensors, dtype=torch.bfloat16, device=dev, max_tokens=6 * 64)
    prompt = ids_for(200, config["vocab"], seed)
    want = O.forward(prompt, tensors, config)
    whole = run_schedule(model, {"a": prompt}, [[("a", 200)]])["a"]
    assert rows_match(whole, want, torch.bfloat16), config
    got = run_schedule(model, {"a": prompt}, [[("a", 97)], [("a", 2)], [("a", 65)]] + [[("a", 1)]] * 36)["a"]
    assert rows_match(got, want, torch.bfloat16), config


def test_long_decoding(dev):
    """500 single-token steps after a two-token prompt (graph replays over growing block tables, windows sliding along), against
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
    assert not model.page_pool.used_page_ids


def test_a_cache_must_come_from_a_layer_that_has_one_of_the_same_sizes(dev):
    config = zalazen_config(pattern="AdSdSd")
    tensors = synthetic_zalazen(config)
    for wrong in (1, 2, 5):                                            # a layer without keys of its own, itself, none
        config["layers"][2]["mixer"]["kv_from"] = wrong
        with pytest.raises(ValueError, match="kv_from"):
            model_class("Zalazen").from_checkpoint(config, tensors, device=dev)
    config["layers"][2]["mixer"].update(kv_from=0, vdim=8)
    with pytest.raises(ValueError, match="kv_from"):
        model_class("Zalazen").from_checkpoint(config, tensors, device=dev)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_points(dev, dtype, tmp_path):
    """greedy_generate_ids and the continuous batcher (mixed steps, 2 slots, 5 requests, pages reused) produce the plain model's
    greedy tokens; the checkpoint goes through a directory and load_model."""
    config = zalazen_config(**CONFIGS["mixed"])
    tensors = synthetic_zalazen(config, seed=21)
    save_zalazen(config, tensors, tmp_path / "ckpt")
    model = load_model(tmp_path / "ckpt", device=dev, dtype=dtype, max_tokens=6 * 64, max_requests=3)
    prompts = [ids_for(n, 160, 30 + n) for n in (5, 70, 2, 33, 64)]
    new = 30
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
    assert batcher.mixed and batcher.mixed_steps > 0 and model.page_pool.reused_page_allocations > 0 and not model.page_pool.used_page_ids


def test_trace_program_replays_steps_and_writes_logits(dev, tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np

    config = zalazen_config(**CONFIGS["odd"])
    tensors = synthetic_zalazen(config, seed=4)
    save_zalazen(config, tensors, tmp_path / "ckpt")
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

    config = zalazen_config(**CONFIGS["equal"])
    tensors = synthetic_zalazen(config, seed=8)
    save_zalazen(config, tensors, tmp_path / "ckpt")
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
    assert cli.main(["generate", "--synthetic", "zalazen:AdSn", "--prompt-ids", "5,17,3", "--max-new-tokens", "4"]) == 0
    assert len(capsys.readouterr().out.split()) == 4
