"""A routed mixture of gated feed-forward experts, with an optional always-on shared expert."""
from __future__ import annotations

import torch

from ..kernels import linear, ops
from .base import FeedForward
from .registry import register
from .spec import TensorSpec


@register("feed_forward", "routed_experts")
class RoutedExperts(FeedForward):
    """`n_experts` experts of the form down(silu(gate x) * (up x)), of which every token uses `top`.

    Router: s = sigmoid(W_router x) in float32; c = s + correction ranks the experts.  Experts e with the same
    e // (n_experts / n_groups) form a group, ranked by its top-2 sum of c; only the `group_keep` highest groups
    remain candidates (the rest are removed from the ranking, whatever the sign of their c).  The `top`
    candidates with the highest c run, weighted by s / (sum of the chosen s + 1e-20).  A shared expert of
    width `shared_size` (None: none) runs for every token and is added times sigmoid(w_sg . x).

    Other forms, as parameters: `router_kind` "softmax" (s = softmax(W_router x) over all router outputs instead of
    sigmoids); `normalise` False (the weights are the chosen s as they are); `identity` (so many more router outputs
    after the experts', which stand for experts without tensors whose output is their input x itself, times the
    weight); `expert_form` / `shared_form` (a dict with limit and optionally alpha, shift: the bounded gate
    g' sigmoid(alpha g') (u' + shift) of `bounded_glu` instead of SiLU); `shared_gate` False (the shared expert has no
    learned gate and is added as it is); `out_scale` (a factor on the part's whole result, applied in float32 as it
    joins the stream); `correction` False (no such tensor: the scores rank the experts by themselves); `group_score` "max" (a
    group is ranked by its largest c alone instead of the sum of its two largest); `router_bias` (a vector of its own added
    to W_router x before the sigmoid or softmax: it moves the ranking and the weights alike.  Softmax scores of all experts
    divided by the sum of the chosen ones are the softmax over the chosen logits).

    Everything from the router to the sum runs on the device (`csrc/moe.cu`), so decode steps stay
    inside captured graphs.  Experts are kept stacked: gate, up [experts, ff, hidden], down [experts,
    hidden, ff].  `names` gives the tensors' names below the part's prefix; "{e}" is the expert's number."""

    _NAMES = {"router": "router.weight", "correction": "router.correction", "router_bias": "router.bias", "gate": "experts.{e}.gate_proj.weight",
              "up": "experts.{e}.up_proj.weight", "down": "experts.{e}.down_proj.weight",
              "shared_gate": "shared.gate_proj.weight", "shared_up": "shared.up_proj.weight",
              "shared_down": "shared.down_proj.weight", "shared_mix": "shared.mix.weight"}

    ROUTERS = ("sigmoid", "softmax")
    GROUP_SCORES = ("top2_sum", "max")

    def __init__(self, *, n_experts: int, top: int, expert_size: int, n_groups: int = 1, group_keep: int = 1,
                 shared_size: int | None = None, names: dict | None = None, router_kind: str = "sigmoid",
                 normalise: bool = True, identity: int = 0, expert_form: dict | None = None,
                 shared_form: dict | None = None, shared_gate: bool = True, out_scale: float = 1.0,
                 correction: bool = True, group_score: str = "top2_sum", router_bias: bool = False, hidden_size: int, dtype, device):
        super().__init__(hidden_size=hidden_size, dtype=dtype, device=device)
        if router_kind not in self.ROUTERS:
            raise ValueError(f"routed_experts: unknown router {router_kind!r}; known: {', '.join(self.ROUTERS)}")
        if group_score not in self.GROUP_SCORES:
            raise ValueError(f"routed_experts: unknown group score {group_score!r}; known: {', '.join(self.GROUP_SCORES)}")
        self.has_router_bias, self.router_bias = bool(router_bias), None
        self.has_correction, self.group_max = bool(correction), group_score == "max"
        if identity < 0 or (identity and n_groups != 1):
            raise ValueError(f"{identity} experts without tensors (not negative; not combined with groups)")
        if not 0 < top <= n_experts + identity:
            raise ValueError(f"{top} of {n_experts + identity} experts cannot be chosen")
        self.router_kind, self.normalise, self.identity = router_kind, bool(normalise), int(identity)
        self.shared_gate, self.out_scale = bool(shared_gate), float(out_scale)
        self.expert_form = self._form(expert_form, device)
        self.shared_form = self._form(shared_form, device)
        if n_groups <= 0 or n_experts % n_groups or not 0 < group_keep <= n_groups:
            raise ValueError(f"{n_experts} experts do not form {n_groups} equal groups of which {group_keep} are kept")
        if group_keep * (n_experts // n_groups) + identity < top:
            raise ValueError(f"{group_keep} groups of {n_experts // n_groups} experts cannot give {top} choices")
        self.n_experts, self.top, self.expert_size = n_experts, top, expert_size
        self.n_groups, self.group_keep = n_groups, group_keep
        self.shared_size = shared_size
        # so many slices of an expert's width a shared expert without a gate of its own consists of, where it is a whole number
        # of them and the experts' activation is its own (0: it always runs as matrices of its own)
        self.in_lists = 0
        if shared_size is not None and not self.shared_gate and not self.identity and expert_form is None and shared_form is None:
            slices = shared_size // expert_size
            self.in_lists = slices if slices * expert_size == shared_size and slices <= self.MOST_SLICES else 0
        self.names = dict(self._NAMES, **(names or {}))
        self.router = self.correction = self.w_gate = self.w_up = self.w_down = None
        self.shared = self.shared_mix = self.w_router = None

    @staticmethod
    def _form(form, device):
        """The bounded gate's constants on the device (None: SiLU)."""
        if form is None:
            return None
        limit = float(form["limit"])
        if not limit > 0:
            raise ValueError(f"the bound of a bounded gate is positive, found {limit}")
        return torch.tensor([float(form.get("alpha", 1.702)), limit, float(form.get("shift", 1.0)), 0.0, 1.0],
                            dtype=torch.float32, device=device)

    def tensor_specs(self):
        h, f, nm = self.hidden_size, self.expert_size, self.names
        outputs = self.n_experts + self.identity
        specs = {nm["router"]: TensorSpec((outputs, h), role="vector")}
        if self.has_correction:
            specs[nm["correction"]] = TensorSpec((outputs,), role="vector", init="zeros")
        if self.has_router_bias:
            specs[nm["router_bias"]] = TensorSpec((outputs,), role="vector", init="zeros")
        for e in range(self.n_experts):
            specs[nm["gate"].format(e=e)] = TensorSpec((f, h))
            specs[nm["up"].format(e=e)] = TensorSpec((f, h))
            specs[nm["down"].format(e=e)] = TensorSpec((h, f))
        if self.shared_size is not None:
            s = self.shared_size
            specs[nm["shared_gate"]] = TensorSpec((s, h))
            specs[nm["shared_up"]] = TensorSpec((s, h))
            specs[nm["shared_down"]] = TensorSpec((h, s))
            if self.shared_gate:
                specs[nm["shared_mix"]] = TensorSpec((1, h), role="vector")
        return specs

    def set_tensors(self, tensors):
        nm, n = self.names, self.n_experts
        self.router = tensors[nm["router"]].contiguous()
        self.correction = tensors[nm["correction"]].contiguous() if self.has_correction else None
        self.router_bias = tensors[nm["router_bias"]].contiguous() if self.has_router_bias else None
        self.shared_mix = tensors[nm["shared_mix"]].reshape(-1).contiguous() if self.shared_size is not None and self.shared_gate else None
        self.w_router, self.router_terms = self._router_matrix()
        # an ungated shared expert that is a whole number of experts wide stands behind the experts as that many slices
        slices = lambda key: (tensors[nm["shared_" + key]].chunk(self.in_lists, dim=1 if key == "down" else 0) if self.in_lists else ())
        stack = lambda key: torch.stack([tensors[nm[key].format(e=e)] for e in range(n)] + list(slices(key))).contiguous()
        self.w_gate, self.w_up, self.w_down = stack("gate"), stack("up"), stack("down")
        if self.shared_size is not None:
            # (its gate and up rows are those slices' storage; its down matrix lies the other way round and is kept twice)
            whole = lambda w, key: w[n:].view(self.shared_size, -1) if self.in_lists else tensors[nm["shared_" + key]]
            self.shared = (linear.Weight(whole(self.w_gate, "gate")), linear.Weight(whole(self.w_up, "up")),
                           linear.Weight(tensors[nm["shared_down"]]))

    def _router_matrix(self):
        """The router's rows (and the shared expert's gate row) for bfloat16 runs as bfloat16 matrices that add up to them, one
        below the other: a float32 number is the sum of three bfloat16 ones (8 bits of its 24 each), and one that is stored as
        bfloat16 is the first of them alone.  Products of a bfloat16 input with bfloat16 weights are exact in float32, so a
        tensor-core product with float32 accumulators forms the same 32-bit logits as the float32 rows would."""
        if self.dtype != torch.bfloat16:
            return None, 0
        rows = self.router if self.shared_mix is None else torch.cat([self.router, self.shared_mix[None]], dim=0)
        rest, terms = torch.cat([rows, rows.new_zeros(-len(rows) % 8, rows.shape[1])], dim=0), []
        while len(terms) < 3 and (not terms or bool(rest.any())):
            terms.append(rest.to(torch.bfloat16))
            rest = rest - terms[-1].float()
        return linear.Weight(torch.cat(terms, dim=0)), len(terms)

    def get_tensors(self):
        nm = self.names
        out = {nm["router"]: self.router}
        if self.has_correction:
            out[nm["correction"]] = self.correction
        if self.has_router_bias:
            out[nm["router_bias"]] = self.router_bias
        for e in range(self.n_experts):
            out[nm["gate"].format(e=e)] = self.w_gate[e]
            out[nm["up"].format(e=e)] = self.w_up[e]
            out[nm["down"].format(e=e)] = self.w_down[e]
        if self.shared_size is not None:
            out[nm["shared_gate"]], out[nm["shared_up"]], out[nm["shared_down"]] = (w.t for w in self.shared)
            if self.shared_gate:
                out[nm["shared_mix"]] = self.shared_mix.view(1, -1)
        return out

    # steps of more tokens than this run the experts' products on the tensor cores (tiles of 128 rows of one
    # expert, their weights streamed by TMA) when the sizes allow; the FFMA form is the 32-bit path and
    # the fallback for other sizes
    TENSOR_CORE_MIN_TOKENS = 0
    SHARED_IN_LISTS_TOKENS, MOST_SLICES = 64, 8     # steps of up to so many tokens; slices of a shared expert
    GATHER_IN_ARRANGE_PAIRS = 256       # up to so many (token, choice) pairs the arranging block also gathers their rows
    ROUTE_PRODUCT_TOKENS = 256          # steps of at least so many tokens: the router's logits as a product
    ROUTE_SPLIT_TOKENS, ROUTE_SPLIT_BLOCKS, ROUTE_SPLIT_MOST = 64, 148, 16     # steps of up to 64 tokens: the router's rows
    #                                     over up to 16 blocks per token, about one block per SM in all

    def _on_tensor_cores(self, x) -> bool:
        if x.dtype != torch.bfloat16 or x.shape[0] <= self.TENSOR_CORE_MIN_TOKENS:
            return False
        from ..kernels import tcgen05
        return (tcgen05.grouped_supports(x.dtype, self.w_gate) and tcgen05.grouped_supports(x.dtype, self.w_down)
                and self.hidden_size % 8 == 0)

    def route_cut(self, x, ctx) -> dict:
        """Keyword arguments of `ops.moe_route` for the step's input x: a step of few tokens cuts the router's rows over several
        blocks per token, so that more SMs than tokens read them; one of many forms the logits as a product on the
        tensor cores (scratch from the step's workspace)."""
        n = x.shape[0]
        if n >= self.ROUTE_PRODUCT_TOKENS and self.w_router is not None and linear.on_tensor_cores(x, self.w_router):
            sums = ctx.buffer("moe_route_logits", (n, self.w_router.n), torch.float32)
            linear.logits(x, self.w_router, sums, ctx)
            return dict(sums=(sums, self.router_terms))
        outputs = self.router.shape[0] + (1 if self.shared_mix is not None else 0)
        if n > self.ROUTE_SPLIT_TOKENS:
            return {}
        split = min(self.ROUTE_SPLIT_MOST, self.ROUTE_SPLIT_BLOCKS // n, outputs // 4)
        if split <= 1:
            return {}
        return dict(split=split, split_sums=ctx.buffer("moe_route_sums", (n, self.router.shape[0] + 1), torch.float32),
                    split_count=ctx.zeroed_buffer("moe_route_count", (n,), torch.int32))

    def forward(self, x, residual, ctx):
        r = self._run(x, ctx)
        # ids at or beyond the experts with tensors were left out of the lists: their rows are the input itself
        through = dict(ids=r["ids"], x=x, n_real=self.n_experts) if self.identity else {}
        ops.moe_combine(residual, r["y"], r["weights"], top=r["top"], shared_y=r["shared"], gate=r["gate"], place=r["place"],
                        scale=self.out_scale, **through)

    def forward_unsummed(self, x, ctx):
        if self.identity or self.shared_mix is not None or self.top + self.in_lists > ops.MAX_SUMMED_EXPERTS:
            return None
        r = self._run(x, ctx)
        return {**{k: r[k] for k in ("y", "weights", "top", "place", "shared")}, "factor": self.out_scale}

    def _run(self, x, ctx) -> dict:
        """Everything up to the sum: the experts' rows y, a token's weights and the places of its rows, the shared expert's result."""
        n, h, experts = x.shape[0], self.hidden_size, self.n_experts
        # a step of few tokens lists the shared expert's slices as experts that every token uses
        extra = self.in_lists if n <= self.SHARED_IN_LISTS_TOKENS and self._on_tensor_cores(x) else 0
        chosen, top = self.top, self.top + extra
        listed = experts + extra
        pairs = n * top
        ids = ctx.buffer("moe_ids", (n, top), torch.int32)
        weights = ctx.buffer("moe_weights", (n, top), torch.float32)
        gate = ctx.buffer("moe_shared_gate", (n,), torch.float32) if self.shared_mix is not None else None
        cut = self.route_cut(x, ctx)
        ops.moe_route(x, self.router, self.correction, ids, weights, top=chosen, always=extra, groups=self.n_groups,
                      keep=self.group_keep, gate_weight=self.shared_mix, gate_out=gate,
                      softmax=self.router_kind == "softmax", normalise=self.normalise, group_max=self.group_max, bias=self.router_bias, **cut)
        fast = self._on_tensor_cores(x)
        if fast:
            from ..kernels import tcgen05
            rows = tcgen05.GROUPED_TILE_ROWS
        else:
            rows = ops.moe_tile_rows()
        offsets = ctx.buffer("moe_offsets", (listed + 1,), torch.int32)
        order = ctx.buffer("moe_order", (pairs,), torch.int32)
        tiles = ctx.buffer("moe_tiles", (2 * (-(-pairs // rows) + listed),), torch.int32)
        n_tiles = ctx.buffer("moe_n_tiles", (1,), torch.int32)
        place = ctx.buffer("moe_place", (pairs,), torch.int32) if fast else None
        # an expert's rows consecutive: the activations are gathered into the lists' order (by the arranging
        # kernel itself when the pairs are few); act and y stay in that order
        xs = ctx.buffer("moe_x_sorted", (pairs, h), self.dtype) if fast else None
        small = fast and pairs <= self.GATHER_IN_ARRANGE_PAIRS
        ops.moe_arrange(ids, pairs, listed, rows, offsets, order, tiles, n_tiles, place,
                        gather=(x, xs, top) if small else None)
        act = ctx.buffer("moe_act", (pairs, self.expert_size), self.dtype)
        y = ctx.buffer("moe_y", (pairs, h), torch.float32)
        w_gate, w_up, w_down = (w[:listed] for w in (self.w_gate, self.w_up, self.w_down))
        if fast:
            if not small:
                ops.moe_gather(x, xs, order, n_pairs=pairs, top=top,
                               listed=offsets[listed:listed + 1] if self.identity else None)
            tcgen05.grouped_gemm(xs, w_gate, w_up, act, offsets, tiles, n_tiles, n_pairs=pairs,
                                 gate_form=self.expert_form)
            tcgen05.grouped_gemm(act, w_down, None, y, offsets, tiles, n_tiles, n_pairs=pairs)
        else:
            ops.moe_grouped_simt(x, w_gate, w_up, act, offsets, order, tiles, n_tiles, n_pairs=pairs, top=top,
                                 gate_form=self.expert_form)
            ops.moe_grouped_simt(act, w_down, None, y, offsets, order, tiles, n_tiles, n_pairs=pairs, top=top)
        shared_y = None
        if self.shared is not None and not extra:
            w_gate, w_up, w_down = self.shared
            sact = ctx.buffer("moe_shared_act", (n, self.shared_size), self.dtype)
            linear.gated(x, w_gate, w_up, sact, ctx, form=self.shared_form)
            shared_y = ctx.buffer("moe_shared_y", (n, h), torch.float32)
            linear.logits(sact, w_down, shared_y, ctx)
        return dict(y=y, weights=weights, top=top, place=place, shared=shared_y, gate=gate, ids=ids)
