"""Nomudra: a decoder-only model with elementwise bounded norms before AND behind every sublayer, ``x <- x + n1b(mixer(n1(x)))``,
``x <- x + n2b(ff(n2(x)))``, every norm ``n(x) = w tanh(alpha x) + b`` (``layer_norm.TanhNorm``); the embedding passes one too.

Mixers (``layers[i].type``):

- ``attention``: grouped-query attention within chunks of ``mask.size`` positions counted from 0.  Queries and keys (biased
  projections) are rotated on the first ``rot.dims`` entries of every head (pairs ``(i, i + dims/2)``); the values are the keys
  before that rotation.  Every entry of the concatenated heads is multiplied by the sigmoid of a projection of the mixer's
  input, and the output projection has a bias (``paged_attention.PagedGroupedAttention``).
- ``mlstm``: a matrix memory with exponential gates and a normaliser (``linear_attention.MatrixMemory``).

Feed-forward (``mlp``, null = none; ``kind`` ``moe``): ``router.top`` of ``router.experts`` clamped experts (``g = min(W_gate h, limit)``,
``u = clamp(W_up h, -limit, limit)``, ``W_down (g sigmoid(1.702 g) (u + 1))``) and ``router.identity`` identity experts, scores a
softmax over all router outputs, chosen by score + ``correction`` among the best ``groups.keep`` of ``groups.count`` groups of
neighbours, weights the chosen scores renormalised; plus a shared expert times ``sigmoid(W_sg h)``.  Everything that can differ
between models of the design is read from ``config.json`` (``vocab``, ``width``, ``norm.eps``, the layers' sizes, scales, rotations, masks,
caps, limits and routers) or from a tensor's shape.

The model is the framework's usual object (``RaggedDecoderModel``).  A request holds one page list for all attention layers
(``LatentPagedPool``: one slab per attention layer, rows of ``kv_heads * (dim + vdim)``) and one slot of the ``StateSlotPool`` with two blocks
per recurrent layer (memory with its normaliser, running maximum).  Compute dtype bf16 (serving) or fp32 (every product in
true fp32); norms, scores, softmax, router, gates, memory, rotation angles and the residual sum are fp32 in both.  A sublayer's
post norm, the residual sum and the norm that reads the stream next are one launch, for the feed-forward together with the
weighted sum of the experts; small steps run the shared expert on a second stream.
"""

from __future__ import annotations

import torch

from extensions_b200.tiny_llm_ext_b200 import blocks

from .basics import linear_wide
from .latent_kv_cache import LatentCacheView, LatentPagedPool
from .layer_norm import TanhNorm
from .linear_attention import MatrixMemory
from .mlp import GatedMLP, MixtureOfExperts, TopKRouter
from .paged_attention import FusedProjection, PagedGroupedAttention
from .ragged import RaggedPlan
from .ragged_model import RaggedDecoderModel
from .state_cache import HybridPagedCache, StateSlotPool

MIXERS = ("attention", "mlstm")
SWISH_SLOPE = 1.702    # the design's sigmoid approximation of GELU inside the experts' gate
BESIDE_TOKENS = 128    # steps of up to this many tokens run the shared expert beside the routed ones: neither fills the GPU


class NomudraLayer:
    def __init__(self, kind: str):
        self.kind = kind
        self.norm1 = self.norm1b = self.norm2 = self.norm2b = self.mlp = None
        self.proj = self.attention = self.out_bias = self.memory = None
        self.slab_index = 0
        self.state_offset = self.peak_offset = 0


class NomudraModel(RaggedDecoderModel):
    architecture = "Nomudra"
    graph_env = "TL_NOMUDRA_GRAPH"

    def __init__(self, config: dict, tensors: dict, dtype=torch.bfloat16, device="cuda", page_size: int = 64, max_tokens: int | None = None,
                 max_requests: int | None = None):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Nomudra runs in bfloat16 or float32")
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

        def norm(name: str) -> TanhNorm:
            n = TanhNorm(take(name), take(name + ".b"), take(name + ".alpha"))
            if n.weight.numel() != self.hidden_size:
                raise ValueError(f"{name} does not match the width")
            return n

        self.embed = take("embed")
        if tuple(self.embed.shape) != (self.vocab_size, self.hidden_size):
            raise ValueError("embed does not match vocab x width")
        self.embed_norm = norm("embed.norm")
        self.layers: list[NomudraLayer] = []
        widths: list[int] = []
        state_floats = 0
        for i, spec in enumerate(config["layers"]):
            kind, m, p = spec["type"], spec["mixer"], f"l{i}.mix."
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            layer = NomudraLayer(kind)
            layer.norm1, layer.norm1b = norm(f"l{i}.norm1"), norm(f"l{i}.norm1b")
            if kind == "attention":
                rot = m.get("rot") or {}
                layer.attention = PagedGroupedAttention(
                    heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], mask="chunk", mask_size=m["mask"]["size"],
                    w_o=take(p + "o"), eps=self.eps, page_size=page_size, values="keys",
                    rot={"dims": int(rot["dims"]), "base": float(rot["base"]), "interleaved": False} if rot.get("dims") else None)
                layer.out_bias = take(p + "o.b")
                layer.proj = FusedProjection([("q", take(p + "q"), take(p + "q.b")), ("k", take(p + "k"), take(p + "k.b")), ("g", take(p + "g"), None)],
                                             dtype, self.device)
                layer.slab_index = len(widths)
                widths.append(layer.attention.cache_width)
            else:
                layer.memory = MatrixMemory(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], gate_cap=m["gate_cap"], w_i=take(p + "i"), b_i=take(p + "i.b"),
                                            w_f=take(p + "f"), b_f=take(p + "f.b"), norm_weight=take(p + "norm"), w_o=take(p + "o"), eps=self.eps)
                layer.proj = FusedProjection([(n, take(p + n), None) for n in ("q", "k", "v", "g")], dtype, self.device)
                layer.state_offset = state_floats
                state_floats += layer.memory.heads * layer.memory.dim * (layer.memory.vdim + 1)
                layer.peak_offset = state_floats
                state_floats += layer.memory.heads
            layer.mlp = self._feed_forward(spec.get("mlp"), f"l{i}.mlp.", take)
            if layer.mlp is not None:
                layer.norm2, layer.norm2b = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
            self.layers.append(layer)
        self.final_norm = norm("final.norm")
        self.head = take("head")
        max_pages = None if max_tokens is None else -(-int(max_tokens) // page_size)
        self.page_pool = LatentPagedPool(widths, page_size=page_size, dtype=dtype, device=self.device, max_pages=max_pages)
        self.state_pool = StateSlotPool(state_floats, device=self.device, max_slots=max_requests)
        self.tile_sizes = sorted({size for layer in self.layers if layer.attention is not None for size in layer.attention.tile_sizes}) or [blocks.ATTENTION_TILE_TOKENS]

    @staticmethod
    def _feed_forward(spec, prefix: str, take):
        if not spec:
            return None
        if spec["kind"] != "moe":
            raise ValueError(f"unknown feed-forward kind {spec['kind']!r}")
        r = spec["router"]
        experts, top, identity, groups = int(r["experts"]), int(r["top"]), int(r.get("identity") or 0), r.get("groups")
        router = TopKRouter(take(prefix + "router"), None, top, scoring="softmax_all", choice_bias=take(prefix + "correction"),
                            groups=(groups["count"], groups["keep"]) if groups else None)
        stack = lambda part: torch.stack([take(f"{prefix}e{k}.{part}") for k in range(experts)]).contiguous()
        shared = side = None
        if spec.get("shared"):
            shared = GatedMLP(*(take(f"{prefix}shared.{part}") for part in ("gate", "up", "down")), "clamped_swish", limit=float(spec["shared"]["limit"]), slope=SWISH_SLOPE)
            side = take(prefix + "shared.sg")
        return MixtureOfExperts(router, stack("gate"), stack("up"), stack("down"), "clamped_swish", shared, identity=identity,
                                limit=float(spec["expert"]["limit"]), slope=SWISH_SLOPE, shared_gate=side)

    @classmethod
    def from_checkpoint(cls, config: dict, tensors: dict, **kwargs) -> "NomudraModel":
        return cls(config, tensors, **kwargs)

    # ---- cache ---------------------------------------------------------------------
    def create_kv_cache(self) -> list:
        """One entry per layer (what the schedulers expect); all are faces of ONE page list + state slot, held by entry 0."""
        owner = HybridPagedCache(self.page_pool, self.state_pool)
        return [owner] + [LatentCacheView(owner, layer.slab_index) for layer in self.layers[1:]]

    def _storage_version(self):
        return (self.page_pool.slab_version, self.state_pool.version)

    # ---- the layers over one plan ------------------------------------------------------
    def _mixer(self, layer: NomudraLayer, h: torch.Tensor, plan: RaggedPlan) -> torch.Tensor:
        y = layer.proj(h)
        if layer.kind == "attention":
            return layer.attention(y["q"], y["k"], None, y["g"], plan, self.page_pool.slabs[layer.slab_index])
        m, view = layer.memory, self.state_pool.layer_view
        return m(h, y["q"], y["k"], y["v"], y["g"], plan, view(layer.state_offset, m.state_shape), view(layer.peak_offset, m.peak_shape))

    def _forward_plan(self, plan: RaggedPlan) -> torch.Tensor:
        exact = self.precision == torch.float32
        tf32 = torch.backends.cuda.matmul.allow_tf32
        if exact:
            torch.backends.cuda.matmul.allow_tf32 = False  # fp32 means fp32
        try:
            x32, h = self.embed_norm.embed(plan.ids, self.embed, self.layers[0].norm1)
            beside = self if plan.num_tokens <= BESIDE_TOKENS else None
            for i, layer in enumerate(self.layers):
                mixed = self._mixer(layer, h, plan)
                # the model's norm joins the last sum when every row's logits are wanted, else it runs on the wanted rows only
                following = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else self.final_norm if plan.all_wanted else None
                h = layer.norm1b.follow(x32, mixed, layer.norm2 if layer.mlp is not None else following, y_bias=layer.out_bias)
                if layer.mlp is not None:
                    h = layer.mlp(h, into=(x32, layer.norm2b, following), beside=beside)
                if self.stream_tap is not None:
                    self.stream_tap.append(x32.clone())
            if plan.num_want == 0:  # a portion whose logits nobody asked for: caches and states are filled, that is all
                return torch.empty((0, self.vocab_size), dtype=torch.float32, device=self.device)
            return linear_wide(h if plan.all_wanted else self.final_norm.rows(x32, plan.want_rows), self.head)
        finally:
            if exact:
                torch.backends.cuda.matmul.allow_tf32 = tf32
