"""The register-softmax form of grouped-query attention (``flash``: 64 query rows per CTA, ``flash_split``: 16 rows whose keys
the warps share) against the plain restatements, over every mask and weight function, head sizes and groups, page sizes,
alignments, splits of the key range over a cluster, and cuts of a prompt."""

import pytest
import torch

from oracle import bapovik as OB
from oracle import norusun as ON
from extensions_b200.tiny_llm_ext_b200 import blocks

pytestmark = pytest.mark.gpu
BF = torch.bfloat16
MASK = {"causal": blocks.MASK_CAUSAL, "window": blocks.MASK_WINDOW, "chunk": blocks.MASK_CHUNK}


@pytest.fixture(scope="module")
def dev(cuda_device):
    return cuda_device


def close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    err, scale = (got - want).abs().max().item(), want.abs().max().item() + 1e-9
    assert err <= tol * scale, (err, scale)


def paged(dev, rows, page_size, seed):
    """rows [T, width] into pages in a scrambled order; unused slots hold stale numbers."""
    T, width = rows.shape
    pages = -(-T // page_size)
    order = torch.randperm(pages + 3, generator=torch.Generator().manual_seed(seed))[:pages]
    slab = torch.full((pages + 3, page_size, width), 50.0, dtype=BF, device=dev)
    for p in range(pages):
        part = rows[p * page_size : (p + 1) * page_size]
        slab[order[p], : part.shape[0]] = part.to(dev)
    return slab, order.to(torch.int32).reshape(1, -1).to(dev)


def tiles(dev, count, size):
    return torch.tensor([(lo, min(size, count - lo), 0) for lo in range(0, count, size)], dtype=torch.int32).to(dev)


SIZES = [(4, 4, 16, 16), (6, 2, 24, 40), (8, 1, 8, 72), (2, 2, 64, 32), (36, 1, 16, 24), (70, 1, 8, 8), (3, 1, 200, 256), (8, 2, 128, 128), (4, 2, 96, 64),
         (5, 1, 192, 128), (16, 1, 40, 96), (17, 1, 32, 160)]
KINDS = [("causal", 0, 0.0, None), ("window", 37, 0.0, None), ("window", 64, 0.0, "learned"), ("chunk", 50, 4.0, "zero"), ("window", 1, 2.0, "zero"), ("chunk", 64, 0.0, "sigmoid"),
         ("causal", 0, 0.0, "sigmoid"), ("chunk", 33, 0.0, "learned")]


@pytest.mark.parametrize("heads,kv_heads,dk,dv", SIZES)
@pytest.mark.parametrize("kind,size,softcap,extra", KINDS)
def test_every_mask_and_weight_function(dev, heads, kv_heads, dk, dv, kind, size, softcap, extra):
    g = torch.Generator().manual_seed(heads * dk + size)
    page = (32, 64, 96)[(heads + dk + size) % 3]
    S, scale, group = 146, dk ** -0.5, heads // kv_heads
    q, k, v = (2 * torch.randn(S, heads, dk, generator=g)).to(BF), torch.randn(S, kv_heads, dk, generator=g).to(BF), torch.randn(S, kv_heads, dv, generator=g).to(BF)
    gate, bias = torch.randn(S, heads, generator=g).to(BF), torch.randn(heads, generator=g)
    kk, vv = k.double().repeat_interleave(group, 1), v.double().repeat_interleave(group, 1)
    if extra == "sigmoid":
        want = ON.sigmoid_attention(q.double(), kk, vv, bias.double(), scale=scale, kind=kind, size=size)
    elif extra == "learned":
        want = ON.sink_softmax_attention(q.double(), kk, vv, bias.double(), scale=scale, kind=kind, size=size)
    else:
        want = OB.masked_attention(q.double(), k.double(), v.double(), scale=scale, kind=kind, size=size, softcap=softcap or None, sink=extra == "zero")
    want = want * torch.sigmoid(gate.double())[:, :, None]
    slab, table = paged(dev, torch.cat([k.reshape(S, -1), v.reshape(S, -1)], dim=1), page, seed=size)
    pos = torch.arange(S, dtype=torch.int32, device=dev)
    args = dict(kv_heads=kv_heads, dv=dv, mask=MASK[kind], mask_size=size, scale=scale, softcap=softcap, sink=extra in ("zero", "learned"),
                head_bias=bias.to(dev) if extra in ("learned", "sigmoid") else None, weights=blocks.WEIGHTS_SIGMOID if extra == "sigmoid" else blocks.WEIGHTS_SOFTMAX)
    forms = blocks.paged_attention_flash_forms(BF, heads, kv_heads, dk, dv, page)
    assert ("flash_split" in forms) == (group <= 16) and forms["flash"] == max(1, 64 // group)
    wide = torch.zeros((S, heads * dk + 3), dtype=BF, device=dev)              # queries whose rows start at odd places
    wide[:, 1 : 1 + heads * dk] = q.reshape(S, -1).to(dev)
    odd = wide[:, 1 : 1 + heads * dk].unflatten(1, (heads, dk))
    qd, gd = q.to(dev), gate.to(dev)
    for kernel, tile in forms.items():
        run = lambda lo, hi, qq=qd, ctx=0, out=None: blocks.paged_attention(qq[lo:hi], slab, table, tiles(dev, hi - lo, tile), pos[lo:hi], gate=gd[lo:hi], kernel=kernel,
                                                                            max_context=ctx, out=out, **args)
        whole = run(0, S)
        close(whole, want, 2e-2)
        for lo in (0, 63, 141, S - 1):                                          # the same rows from a portion that starts anywhere
            assert torch.equal(run(lo, S), whole[lo:]), (kernel, lo)
        assert torch.equal(run(0, S, odd), whole)
        out = torch.full((S, heads * dv + 5), 9.0, dtype=BF, device=dev)         # and into columns that start at an odd place
        run(0, S, out=out[:, 3 : 3 + heads * dv].unflatten(1, (heads, dv)))
        assert torch.equal(out[:, 3 : 3 + heads * dv].reshape(S, heads, dv), whole) and float(out[:, :3].float().min()) == 9.0 and float(out[:, -2:].float().min()) == 9.0
        close(run(S - 1, S, ctx=S), want[S - 1 :], 2e-2)                         # the key range shared by a cluster
        close(run(70, 90, ctx=S), want[70:90], 2e-2)


@pytest.mark.parametrize("kernel", ["flash", "flash_split"])
@pytest.mark.parametrize("kind,size,sink", [("causal", 0, True), ("window", 300, False), ("chunk", 512, True), ("window", 40, True)])
def test_a_cluster_shares_the_key_range(dev, kernel, kind, size, sink):
    """Few rows over a long range, cut over one to eight CTAs (also more than there are tiles): the sink counted once, parts
    without a visible key weigh nothing."""
    g = torch.Generator().manual_seed(size)
    S, heads, kv_heads, dk, dv = 700, 4, 2, 32, 48
    q, k, v = torch.randn(S, heads, dk, generator=g).to(BF), torch.randn(S, kv_heads, dk, generator=g).to(BF), torch.randn(S, kv_heads, dv, generator=g).to(BF)
    gate = torch.randn(S, heads, generator=g).to(BF)
    want = OB.masked_attention(q.double(), k.double(), v.double(), scale=dk ** -0.5, kind=kind, size=size, softcap=5.0, sink=sink) * torch.sigmoid(gate.double())[:, :, None]
    slab, table = paged(dev, torch.cat([k.reshape(S, -1), v.reshape(S, -1)], dim=1), 32, seed=1)
    tile = blocks.paged_attention_flash_forms(BF, heads, kv_heads, dk, dv, 32)[kernel]
    original = blocks.flash_splits
    try:
        for splits in range(1, 9):
            blocks.flash_splits = lambda *_: splits
            for lo, n in ((S - 1, 1), (640, 3), (511, 2), (0, 1), (130, 40)):
                pos = torch.arange(lo, lo + n, dtype=torch.int32, device=dev)
                got = blocks.paged_attention(q[lo : lo + n].to(dev), slab, table, tiles(dev, n, tile), pos, kv_heads=kv_heads, dv=dv, mask=MASK[kind], mask_size=size,
                                             scale=dk ** -0.5, softcap=5.0, sink=sink, gate=gate[lo : lo + n].to(dev), kernel=kernel, max_context=lo + n)
                close(got, want[lo : lo + n], 2e-2)
    finally:
        blocks.flash_splits = original
    assert blocks.flash_splits(1, 700, None, dev) == 8 and blocks.flash_splits(1, 700, 65, dev) == 2 and blocks.flash_splits(10**6, 10**6, None, dev) == 1
    assert {blocks.flash_splits(1, n, None, dev) for n in (1, 5, 128, 256)} == {4}   # the same over a captured step's range of contexts


@pytest.mark.parametrize("kernel", ["flash", "flash_split"])
@pytest.mark.parametrize("kind,size", [("window", 70), ("window", 64), ("chunk", 70), ("chunk", 64), ("causal", 0)])
def test_one_key_that_matters_far_away_at_page_borders_and_mask_edges(dev, kernel, kind, size):
    """All keys are noise but one, which the probing query scores far above the rest: the output is that key's value exactly
    when the mask lets the query see it.  Prompt rows and single decoded tokens, bit for bit the same."""
    g = torch.Generator().manual_seed(size)
    S, dk, dv = 400, 16, 8
    tile = blocks.paged_attention_flash_forms(BF, 2, 1, dk, dv, 32)[kernel]
    for target in (0, 31, 32, 63, 64, 200, 329, 330, 331, 398, 399):
        k, v = 0.05 * torch.randn(S, 1, dk, generator=g), torch.randn(S, 1, dv, generator=g)
        k[target, 0, 3] = 40.0
        v[target] = 5.0
        q = torch.zeros(S, 2, dk)
        q[:, :, 3] = 1.0
        slab, table = paged(dev, torch.cat([k.reshape(S, -1), v.reshape(S, -1)], dim=1).to(BF), 32, seed=target)
        q = q.to(BF).to(dev)
        run = lambda lo, hi: blocks.paged_attention(q[lo:hi], slab, table, tiles(dev, hi - lo, tile), torch.arange(lo, hi, dtype=torch.int32, device=dev), kv_heads=1,
                                                    dv=dv, mask=MASK[kind], mask_size=size, scale=1.0, kernel=kernel).float().cpu()
        whole = run(0, S)
        for i in sorted({target, target + 1, target + size - 2, target + size - 1, target + size, target + size + 1, (target // max(size, 1) + 1) * max(size, 1) - 1,
                         (target // max(size, 1) + 1) * max(size, 1), S - 1}):
            if 0 <= i < S:
                sees = OB.visible(i, target, kind, size)
                assert (whole[i, 0] - 5.0).abs().max().item() < 2e-2 if sees else (whole[i, 0] - 5.0).abs().min().item() > 1.0, (target, i)
                assert torch.equal(run(i, i + 1)[0], whole[i])


def test_several_sequences_of_unequal_lengths_in_one_launch(dev):
    """Portions beside single tokens, each over its own pages; a table entry that names no page reads as zeros."""
    g = torch.Generator().manual_seed(3)
    heads, kv_heads, dk, dv, page = 8, 2, 32, 32, 64
    lengths, news = [300, 5, 130, 64], [100, 5, 1, 1]
    ks = [torch.randn(n, kv_heads, dk, generator=g).to(BF) for n in lengths]
    vs = [torch.randn(n, kv_heads, dv, generator=g).to(BF) for n in lengths]
    qs = [torch.randn(n, heads, dk, generator=g).to(BF) for n in news]
    pages = [-(-n // page) for n in lengths]
    order = torch.randperm(sum(pages), generator=g)
    slab = torch.full((sum(pages), page, kv_heads * (dk + dv)), 50.0, dtype=BF, device=dev)
    table = torch.full((4, max(pages) + 1), -1, dtype=torch.int32)
    at = 0
    for s, (k, v) in enumerate(zip(ks, vs)):
        rows = torch.cat([k.reshape(len(k), -1), v.reshape(len(v), -1)], dim=1)
        for p in range(pages[s]):
            table[s, p] = order[at]
            part = rows[p * page : (p + 1) * page]
            slab[order[at], : part.shape[0]] = part.to(dev)
            at += 1
    want = []
    for k, v, q, n in zip(ks, vs, qs, news):
        full = torch.zeros(len(k), heads, dk, dtype=torch.float64)
        full[len(k) - n :] = q.double()
        want.append(OB.masked_attention(full, k.double(), v.double(), scale=0.3, kind="window", size=90, softcap=None, sink=False)[len(k) - n :])
    pos = torch.cat([torch.arange(n - m, n, dtype=torch.int32) for n, m in zip(lengths, news)]).to(dev)
    for kernel, tile in blocks.paged_attention_flash_forms(BF, heads, kv_heads, dk, dv, page).items():
        work, first = [], 0
        for s, n in enumerate(news):
            work += [(first + lo, min(tile, n - lo), s) for lo in range(0, n, tile)]
            first += n
        for ctx in (0, 300):
            got = blocks.paged_attention(torch.cat(qs).to(dev), slab, table.to(dev), torch.tensor(work, dtype=torch.int32).to(dev), pos, kv_heads=kv_heads, dv=dv,
                                         mask=blocks.MASK_WINDOW, mask_size=90, scale=0.3, kernel=kernel, max_context=ctx)
            close(got, torch.cat(want), 2e-2)
