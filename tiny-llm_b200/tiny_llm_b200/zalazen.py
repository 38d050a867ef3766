"""Zalazen: a decoder-only model whose layers add a windowed attention and a gated feed-forward, each behind an RMS norm of
its own and both reading the SAME fp32 residual stream: ``x <- x + (mixer(norm1(x)) + ff(norm2(x)))``.

- Embedding: ``embed[token] * embedding.scale``, plus a row of ``bigram`` chosen by the token and the one before it
  (``embedding.bigram``: ``buckets``, ``mul_prev``, ``mul_cur``; the last row for a sequence's first token).
- Mixer (``type`` ``attention``): grouped-query attention.  Queries and keys are RMS-normed over the whole projection (weights
  ``q.norm``, ``k.norm`` of that size), then rotated on the first ``rot.dims`` entries of every head (pairs ``(i, i + dims/2)``,
  base ``rot.base``, stretched by frequency when ``rot.scaling`` gives ``factor``, ``original``, ``fast``, ``slow``).  A position
  sees the last ``mask.size`` positions up to its own and the sequence's first ``mask.keep_first``; the softmax's denominator
  holds one more term, ``exp(sink[h])``; head h's output is multiplied by ``sigmoid(g[h])``, ``g`` a projection of the mixer's
  input.  A layer with ``kv_from = j`` has no keys and values of its own and reads layer j's cache.
- Feed-forward (``mlp`` ``dense``, or null): ``down(silu(gate h) * (up h))``.
- Output: ``head(norm(x))``.

Everything that can differ between models of the design is read from ``config.json`` (``vocab``, ``width``, ``norm.eps``,
``embedding``, the list ``layers`` with ``heads kv_heads dim vdim scale rot mask kv_from`` and ``mlp.ff``).  Weights: ``embed``,
``bigram``, ``l<i>.norm1``, ``l<i>.mix.{q,k,v,q.norm,k.norm,sink,g,o}``, ``l<i>.norm2``, ``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``head``.

The model is the framework's usual object (``RaggedDecoderModel``).  A request holds one page list for all layers
(``LatentPagedPool``: one slab per layer with keys of its own, rows of ``kv_heads * (dim + vdim)``) and the ids it has run,
whose newest one the pair embedding of its next portion reads.  Compute dtype bf16 (serving) or fp32 (every product in true
fp32); embedding sum, residual, norms, scores, softmax and rotation angles are fp32 in both.  A layer's two branches meet in
one product (``JoinedProjection``), whose fp32 accumulator makes their sum; small steps run them on two streams.
"""

from __future__ import annotations

import torch

from extensions_b200.tiny_llm_ext_b200 import blocks

from .basics import linear_wide
from .embedding import PairEmbedding
from .latent_kv_cache import LatentCacheView, LatentPagedCache, LatentPagedPool
from .mlp import GatedMLP
from .paged_attention import FusedProjection, JoinedProjection, PagedGroupedAttention
from .ragged import RaggedPlan
from .ragged_model import RaggedDecoderModel


BESIDE_TOKENS = 128  # steps of up to this many tokens run a layer's two branches side by side: neither fills the GPU


class ZalazenLayer:
    def __init__(self, norm1, proj: FusedProjection, attention: PagedGroupedAttention, slab_index: int, norm2, mlp, out: JoinedProjection):
        self.norm1, self.proj, self.attention, self.slab_index, self.norm2, self.mlp, self.out = norm1, proj, attention, slab_index, norm2, mlp, out


class ZalazenModel(RaggedDecoderModel):
    architecture = "Zalazen"
    graph_env = "TL_ZALAZEN_GRAPH"

    def __init__(self, config: dict, tensors: dict, dtype=torch.bfloat16, device="cuda", page_size: int = 64, max_tokens: int | None = None,
                 max_requests: int | None = None):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Zalazen runs in bfloat16 or float32")
        self.config, self.precision, self.device = config, dtype, torch.device(device)
        self.vocab_size, self.hidden_size = int(config["vocab"]), int(config["width"])
        self.eps = float(config["norm"]["eps"])
        self.num_hidden_layers = len(config["layers"])
        self.page_size = page_size
        self.stream_tap: list | None = None  # a list here receives a copy of the residual stream after every layer
        self._init_step()

        def take(name: str) -> torch.Tensor:
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            t = tensors[name]
            return t.to(device=self.device, dtype=dtype if t.is_floating_point() else t.dtype).contiguous()

        embedding = config.get("embedding") or {}
        bigram = embedding.get("bigram")
        self.embedding = PairEmbedding(take("embed"), embedding.get("scale", 1.0), take("bigram") if bigram else None, **(bigram or {}))
        if tuple(self.embedding.weight.shape) != (self.vocab_size, self.hidden_size):
            raise ValueError("embed does not match vocab x width")
        self.layers: list[ZalazenLayer] = []
        slab_of: dict[int, int] = {}  # caching layer -> slab index
        widths: list[int] = []
        for i, spec in enumerate(config["layers"]):
            if spec["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {spec['type']!r}")
            m, p = spec["mixer"], f"l{i}.mix."
            source = m.get("kv_from")
            own = source is None
            if not own:
                src = config["layers"][source]["mixer"] if source in slab_of else None
                if src is None or (src["kv_heads"], src["dim"], src["vdim"]) != (m["kv_heads"], m["dim"], m["vdim"]):
                    raise ValueError(f"layer {i}: kv_from={source} must name an earlier layer with its own keys and values of the same sizes")
            attention = PagedGroupedAttention(
                heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], mask="window", mask_size=m["mask"]["size"],
                keep_first=m["mask"].get("keep_first") or 0, w_o=take(p + "o"), sink=True, head_bias=take(p + "sink"), q_norm=take(p + "q.norm"),
                k_norm=take(p + "k.norm") if own else None, eps=self.eps, caches=own, page_size=page_size, qk_norm="whole", rot=self._rotation(m.get("rot")))
            names = ("q", "k", "v", "g") if own else ("q", "g")
            proj = FusedProjection([(n, take(p + n), None) for n in names], dtype, self.device)
            if own:
                slab_of[i] = len(widths)
                widths.append(attention.cache_width)
            mlp, norm2 = self._feed_forward(spec.get("mlp"), f"l{i}.mlp.", take), None
            out = JoinedProjection([("o", attention.w_o)] + ([("down", mlp.w_down)] if mlp is not None else []))
            attention.w_o = out.part("o")  # one copy of the weights
            if mlp is not None:
                mlp.w_down, norm2 = out.part("down"), take(f"l{i}.norm2")
            self.layers.append(ZalazenLayer(take(f"l{i}.norm1"), proj, attention, slab_of[i if own else source], norm2, mlp, out))
        self.final_norm = take("final.norm")
        self.head = take("head")
        max_pages = None if max_tokens is None else -(-int(max_tokens) // page_size)
        self.page_pool = LatentPagedPool(widths, page_size=page_size, dtype=dtype, device=self.device, max_pages=max_pages)
        self.tile_sizes = sorted({size for layer in self.layers for size in layer.attention.tile_sizes})

    @staticmethod
    def _rotation(rot):
        if not rot:
            return None
        scaling = rot.get("scaling")
        yarn = {key: float(scaling[key]) for key in ("factor", "original", "fast", "slow")} if scaling else None
        return {"dims": int(rot["dims"]), "base": float(rot["base"]), "interleaved": False, "yarn": yarn}

    @staticmethod
    def _feed_forward(spec, prefix: str, take):
        if not spec:
            return None
        if spec["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {spec['kind']!r}")
        return GatedMLP(take(prefix + "gate"), take(prefix + "up"), take(prefix + "down"), "silu")

    @classmethod
    def from_checkpoint(cls, config: dict, tensors: dict, **kwargs) -> "ZalazenModel":
        return cls(config, tensors, **kwargs)

    # ---- cache ---------------------------------------------------------------------
    def create_kv_cache(self) -> list:
        """One entry per layer (what the schedulers expect); all are faces of ONE page list, held by entry 0."""
        owner = LatentPagedCache(self.page_pool)
        return [owner] + [LatentCacheView(owner, layer.slab_index) for layer in self.layers[1:]]

    # ---- the layers over one plan ------------------------------------------------------
    def _layer(self, layer: ZalazenLayer, h1: torch.Tensor, h2: torch.Tensor | None, plan: RaggedPlan) -> torch.Tensor:
        """What the layer adds to the stream, fp32 ``[T, width]``."""
        T, a = h1.shape[0], layer.attention
        operand, part = layer.out.operand(T)
        with self._beside(layer.mlp is not None and T <= BESIDE_TOKENS):
            if layer.mlp is not None:
                layer.mlp.inner(h2, out=part["down"])
        y = layer.proj(h1)
        a.attend(y["q"], y.get("k"), y.get("v"), y["g"], plan, self.page_pool.slabs[layer.slab_index], out=part["o"].unflatten(1, (a.heads, a.vdim)))
        self._join()
        return layer.out(operand)

    def _forward_plan(self, plan: RaggedPlan) -> torch.Tensor:
        exact = self.precision == torch.float32
        tf32 = torch.backends.cuda.matmul.allow_tf32
        if exact:
            torch.backends.cuda.matmul.allow_tf32 = False  # fp32 means fp32
        try:
            x32, h1, h2 = self.embedding(plan, self.eps, self.layers[0].norm1, self.layers[0].norm2)
            for i, layer in enumerate(self.layers):
                delta = self._layer(layer, h1, h2, plan)
                # the layer's sum, fused with the next layer's norms (the model's norm runs on the wanted rows only)
                following = self.layers[i + 1] if i + 1 < len(self.layers) else None
                if following is None:
                    h1 = blocks.add_norm(x32, delta, None, self.final_norm if plan.all_wanted else None, self.eps)
                elif following.norm2 is None:
                    h1, h2 = blocks.add_norm(x32, delta, None, following.norm1, self.eps), None
                else:
                    h1, h2 = blocks.add_norm(x32, delta, None, following.norm1, self.eps, following.norm2)
                if self.stream_tap is not None:
                    self.stream_tap.append(x32.clone())
            if plan.num_want == 0:  # a portion whose logits nobody asked for: the cache is filled, that is all
                return torch.empty((0, self.vocab_size), dtype=torch.float32, device=self.device)
            if not plan.all_wanted:
                h1 = blocks.norm_residual(x32.index_select(0, plan.want_rows), self.final_norm, self.eps)
            return linear_wide(h1, self.head)
        finally:
            if exact:
                torch.backends.cuda.matmul.allow_tf32 = tf32
