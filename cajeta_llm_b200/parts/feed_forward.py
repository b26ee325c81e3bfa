"""Feed-forward parts: the dense gated MLP (SwiGLU and its like), a dense one with a squared ReLU, and the sparse mixture of experts.

``dense_swiglu``: ``W_d (silu(W_g x) * (W_u x))``, ``silu(x) = x / (1 + exp(-x))``
(model/Prim.cajeta:1822-1847, model/CausalLM.cajeta:1556-1566).  Parameters:
``hidden_size``, ``intermediate_size``, ``names`` (optional: the tensor names of
``gate``, ``up`` and ``down`` under the part's prefix).  ``dense_gated`` is the same part with its two options:
``activation`` (``silu``, the default, or ``gelu_tanh``, gelu's tanh form) and ``bias`` (every projection has one, under its
weight's name with ``.b`` added; gate's and up's are added before the activation, in the product's epilogue).

``dense_relu2``: ``W_d max(W_u x, 0)^2``, a feed-forward without a gate whose activation is the square of the
rectified sum.  Parameters: ``hidden_size``, ``intermediate_size``, ``names`` (``up``, ``down``), ``bias`` (optional: both products
have a bias, under the weight's name with ``.b`` added).  A block may set ``out_scale`` (multiplies the result as it is added)
and ``allow_pending`` (few rows: partial sums are handed back instead of added).  The square is the up-product's epilogue (the
float32 sum squared, then rounded).

``sparse_moe``: router logits ``l_e = Wr[e] . x`` in float32, softmax over all experts,
top-k by repeated strict-``>`` argmax (ties to the lower index), weights = the picked
probabilities, optionally renormalised with the divisor clamped at 2^-14
(model/MoeFfn.cajeta:908-988); each picked expert is a SwiGLU MLP of
``expert_intermediate_size``, summed per token in selection order
(model/MoeFfn.cajeta:1849-1916); an optional shared expert of
``shared_intermediate_size`` is added, scaled by ``sigma(g . x)`` when it has a gate
(model/MoeFfn.cajeta:1925-1964).  Tokens are grouped by expert with a counting sort and
each expert multiplies its own rows (model/MoeFfn.cajeta:2064-2099,2644-2777).  When the
shared expert's width is a multiple of the experts' width it is cut into chunks of that
width which ride through the same two grouped products as extra groups that every token
belongs to (their partial down-projections are summed in chunk order by the combine):
one launch streams all expert weights of the layer.
Parameters: ``hidden_size``, ``num_experts``, ``top_k``, ``expert_intermediate_size``,
``shared_intermediate_size`` (0 = none), ``shared_gate``, ``norm_topk_prob``;
``score`` (``softmax`` over all experts, the default, or ``sigmoid``: each expert's own
sigma(l_e); the order of the experts is the same, the weights differ); ``weight_on``
(``output``, the default: y = sum_j w_j expert_j(x); or ``input``: y = sum_j expert_j(w_j x),
the weight multiplying the float32 row before it is rounded for the products);
``names`` (optional tensor-name templates under the part's prefix: ``router``, and
``gate`` / ``up`` / ``down`` with ``{e}`` for the expert's index; ``shared_gate`` / ``shared_up`` /
``shared_down`` and ``shared_sg``, the shared expert's tensors and its sigmoid gate);
``act_limit`` L > 0 with ``act_alpha`` a: an expert is the capped form ``g = min(W_g x, L)``,
``u = clamp(W_u x, -L, L)``, ``W_d (g sigmoid(a g) (u + 1))`` instead of SwiGLU; ``shared_act_limit`` /
``shared_act_alpha``: the same for the shared expert (default: the experts');
``route_groups`` ``(count, keep)``: the experts form ``count`` equal groups of neighbours, a group's
score is its largest score (``group_score`` ``top2``: the sum of its two largest), and only experts of the ``keep`` best groups
can be picked;
``activation`` ``relu2``: an expert has no gate, ``W_d max(W_u x, 0)^2`` (tensors ``up`` and ``down`` only;
built with the weight on the output); ``gelu``: the same with gelu by the error function.  A shared expert has the experts' form;
``correction``: a tensor name, ``[num_experts]``: a number per expert that is added to its score for the CHOICE of the
``top_k`` experts alone, a pick's weight staying its score without it; ``route_scale``: multiplies the picks'
weights (after a renormalisation, when one is asked for); ``norm_floor`` e > 0: a renormalisation divides by the picks' sum plus
e instead of by the clamped sum.

The file stores one tensor per expert and projection
(``experts.{e}.gate_proj.weight`` ...); they are stacked into ``[E, I, H]`` and
``[E, H, I]`` slabs at load, as the reference binds merged slabs
(model/ExpertBank.cajeta:243-308).
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..csrc import kernels as K
from .base import Part, register_part
from .linear import project, project_split, splits_few_rows
from .plan import ParamSpec


GATES = {"silu": (1.0, 0.0), "gelu_tanh": K.GELU_TANH}      # (alpha, cubic): g sigmoid(alpha g + cubic g^3)


@register_part("feed_forward", "dense_gated")
@register_part("feed_forward", "dense_swiglu")
class DenseSwiGLU(Part):
    needs_f32_input = False

    def __init__(self, spec, prefix, runtime):
        super().__init__(spec, prefix, runtime)
        self.hidden = int(spec["hidden_size"])
        self.inter = int(spec["intermediate_size"])
        names = dict(spec.get("names") or {})
        self.n_gate = self.name(names.get("gate", "gate_proj.weight"))
        self.n_up = self.name(names.get("up", "up_proj.weight"))
        self.n_down = self.name(names.get("down", "down_proj.weight"))
        self.bias = bool(spec.get("bias", False))
        activation = str(spec.get("activation", "silu"))
        if activation not in GATES:
            raise ValueError(f"activation must be one of {', '.join(sorted(GATES))}, found '{activation}'")
        self.gate_alpha, self.gate_cubic = GATES[activation]
        self.w_gate = self.w_up = self.w_down = None
        self.b_gate = self.b_up = self.b_down = None

    def params(self) -> Dict[str, ParamSpec]:
        p = {
            self.n_gate: ParamSpec((self.inter, self.hidden)),
            self.n_up: ParamSpec((self.inter, self.hidden)),
            self.n_down: ParamSpec((self.hidden, self.inter)),
        }
        if self.bias:
            for n in (self.n_gate, self.n_up):
                p[n + ".b"] = ParamSpec((self.inter,), role="vector")
            p[self.n_down + ".b"] = ParamSpec((self.hidden,), role="vector")
        return p

    def libraries(self) -> set:
        libs = {"gemm_simt"}
        if self.runtime.fast_kernels and self.hidden >= 128:
            libs |= {"gemm_tc", "gemm_tc2"}
        return libs

    def load(self, source) -> None:
        self.w_gate = self.fetch(source, self.n_gate)
        self.w_up = self.fetch(source, self.n_up)
        self.w_down = self.fetch(source, self.n_down)
        if self.bias:
            self.b_gate, self.b_up, self.b_down = (self.fetch(source, n + ".b") for n in (self.n_gate, self.n_up, self.n_down))

    def forward(self, x: torch.Tensor, x_f32: Optional[torch.Tensor], residual: torch.Tensor, ctx) -> None:
        T = x.shape[0]
        act = torch.empty((T, self.inter), dtype=self.runtime.act_dtype, device=x.device)
        K.tag = "dense gate/up"
        project(self.runtime, x, self.w_gate, act, w_up=self.w_up, bias=self.b_gate, bias_up=self.b_up, act_alpha=self.gate_alpha,
                act_cubic=self.gate_cubic)
        K.tag = "dense down"
        project(self.runtime, act, self.w_down, residual, bias=self.b_down, accumulate=True)
        K.tag = None


@register_part("feed_forward", "dense_relu2")
class DenseRelu2(Part):
    needs_f32_input = False

    def __init__(self, spec, prefix, runtime):
        super().__init__(spec, prefix, runtime)
        self.hidden = int(spec["hidden_size"])
        self.inter = int(spec["intermediate_size"])
        names = dict(spec.get("names") or {})
        self.n_up = self.name(names.get("up", "up_proj.weight"))
        self.n_down = self.name(names.get("down", "down_proj.weight"))
        self.bias = bool(spec.get("bias", False))
        self.out_scale = 1.0
        self.allow_pending = False         # a block that takes partial sums from its feed-forward sets this True
        self.w_up = self.w_down = self.b_up = self.b_down = None

    def params(self) -> Dict[str, ParamSpec]:
        p = {self.n_up: ParamSpec((self.inter, self.hidden)), self.n_down: ParamSpec((self.hidden, self.inter))}
        if self.bias:
            p[self.n_up + ".b"] = ParamSpec((self.inter,), role="vector")
            p[self.n_down + ".b"] = ParamSpec((self.hidden,), role="vector")
        return p

    def libraries(self) -> set:
        libs = {"gemm_simt"}
        if self.runtime.fast_kernels and self.hidden >= 128:
            libs |= {"gemm_tc", "gemm_tc2"}
        return libs

    def load(self, source) -> None:
        self.w_up = self.fetch(source, self.n_up)
        self.w_down = self.fetch(source, self.n_down)
        if self.bias:
            self.b_up = self.fetch(source, self.n_up + ".b")
            self.b_down = self.fetch(source, self.n_down + ".b")

    def defers(self, rows: int) -> bool:
        return self.allow_pending and splits_few_rows(self.runtime, rows, self.w_down)

    def forward(self, x: torch.Tensor, x_f32: Optional[torch.Tensor], residual: torch.Tensor, ctx) -> Optional[torch.Tensor]:
        rt = self.runtime
        T = x.shape[0]
        act = torch.empty((T, self.inter), dtype=rt.act_dtype, device=x.device)
        K.tag = "dense up"
        project(rt, x, self.w_up, act, bias=self.b_up, act="relu2")
        K.tag = "dense down"
        parts = project_split(rt, act, self.w_down, bias=self.b_down, out_scale=self.out_scale) if self.allow_pending else None
        if parts is None:
            project(rt, act, self.w_down, residual, bias=self.b_down, accumulate=True, out_scale=self.out_scale)
        K.tag = None
        return parts


@register_part("feed_forward", "sparse_moe")
class SparseMoE(Part):
    needs_f32_input = True      # the router reads the normed row in float32

    def __init__(self, spec, prefix, runtime):
        super().__init__(spec, prefix, runtime)
        self.hidden = int(spec["hidden_size"])
        self.num_experts = int(spec["num_experts"])
        self.top_k = int(spec["top_k"])
        self.inter = int(spec["expert_intermediate_size"])
        self.shared_inter = int(spec.get("shared_intermediate_size", 0) or 0)
        self.shared_gate = bool(spec.get("shared_gate", False)) and self.shared_inter > 0
        self.norm_topk = bool(spec.get("norm_topk_prob", False))
        self.score = str(spec.get("score", "softmax"))
        self.weight_on = str(spec.get("weight_on", "output"))
        if self.score not in ("softmax", "sigmoid"):
            raise ValueError(f"score must be 'softmax' or 'sigmoid', found '{self.score}'")
        if self.weight_on not in ("output", "input"):
            raise ValueError(f"weight_on must be 'output' or 'input', found '{self.weight_on}'")
        names = dict(spec.get("names") or {})
        self.act_limit = float(spec.get("act_limit", 0.0) or 0.0)
        self.act_alpha = float(spec.get("act_alpha", 1.0))
        self.shared_act_limit = float(spec.get("shared_act_limit", self.act_limit) or 0.0)
        self.shared_act_alpha = float(spec.get("shared_act_alpha", self.act_alpha))
        self.activation = str(spec.get("activation", "swiglu"))
        if self.activation not in ("swiglu", "relu2", "gelu"):
            raise ValueError(f"activation must be 'swiglu', 'relu2' or 'gelu', found '{self.activation}'")
        self.gated = self.activation == "swiglu"
        if not self.gated and (self.weight_on != "output" or self.act_limit > 0.0):
            raise ValueError("ungated experts are built without capped gates or the weight on the input")
        self.projections = ("gate", "up", "down") if self.gated else ("up", "down")
        self.group_score = str(spec.get("group_score", "largest"))
        if self.group_score not in ("largest", "top2"):
            raise ValueError(f"group_score must be 'largest' or 'top2', found '{self.group_score}'")
        self.norm_floor = float(spec.get("norm_floor", 0.0) or 0.0)
        self.n_correction = self.name(str(spec["correction"])) if spec.get("correction") else None
        self.route_scale = float(spec.get("route_scale", 1.0))
        self.correction = None
        groups = spec.get("route_groups")
        self.route_groups = (int(groups[0]), int(groups[1])) if groups and int(groups[0]) > 1 else None
        if self.route_groups:
            count, keep = self.route_groups
            if self.num_experts % count != 0 or not 1 <= keep <= count:
                raise ValueError(f"route_groups {self.route_groups}: {self.num_experts} experts must form equal groups, 1 <= keep <= count")
            if keep * (self.num_experts // count) < self.top_k:
                raise ValueError(f"route_groups {self.route_groups}: the kept groups hold fewer than top_k = {self.top_k} experts")
        self.n_shared = {proj: self.name(names.get(f"shared_{proj}", f"shared_expert.{proj}_proj.weight")) for proj in ("gate", "up", "down")}
        self.n_shared_sg = self.name(names.get("shared_sg", "shared_expert_gate.weight"))
        self.n_router = self.name(names.get("router", "gate.weight"))
        self.n_expert = {proj: names.get(proj, f"experts.{{e}}.{proj}_proj.weight") for proj in ("gate", "up", "down")}
        if not 1 <= self.top_k <= self.num_experts:
            raise ValueError(f"top_k must be between 1 and num_experts ({self.num_experts}), found {self.top_k}")
        if self.num_experts > 1024:
            raise ValueError(f"num_experts {self.num_experts} is more than the router kernel takes (1024)")
        self.router = None
        self.w_gate = self.w_up = self.w_down = None
        self.ws_gate = self.ws_up = self.ws_down = None
        self.shared_gate_w = None
        self.router_split = None        # [cols, 3 hidden] bfloat16: router rows (and the gate's) three times over
        # chunks of the shared expert that run as extra groups of the grouped products
        self.shared_chunks = 0
        same_act = (self.act_limit, self.act_alpha) == (self.shared_act_limit, self.shared_act_alpha)
        if self.shared_inter > 0 and self.shared_inter % self.inter == 0 and self.shared_inter // self.inter <= 64 and same_act:
            self.shared_chunks = self.shared_inter // self.inter

    def params(self) -> Dict[str, ParamSpec]:
        p = {self.n_router: ParamSpec((self.num_experts, self.hidden), role="vector")}
        if self.n_correction:
            p[self.n_correction] = ParamSpec((self.num_experts,), role="vector", std=0.05)
        for e in range(self.num_experts):
            if self.gated:
                p[self.expert_name("gate", e)] = ParamSpec((self.inter, self.hidden))
            p[self.expert_name("up", e)] = ParamSpec((self.inter, self.hidden))
            p[self.expert_name("down", e)] = ParamSpec((self.hidden, self.inter))
        if self.shared_inter > 0:
            if self.gated:
                p[self.n_shared["gate"]] = ParamSpec((self.shared_inter, self.hidden))
            p[self.n_shared["up"]] = ParamSpec((self.shared_inter, self.hidden))
            p[self.n_shared["down"]] = ParamSpec((self.hidden, self.shared_inter))
            if self.shared_gate:
                p[self.n_shared_sg] = ParamSpec((1, self.hidden), role="vector")
        return p

    def expert_name(self, proj: str, e: int) -> str:
        return self.name(self.n_expert[proj].format(e=e))

    def libraries(self) -> set:
        libs = {"rowwise", "moe_route", "gemm_simt"} | ({"recurrent"} if self.weight_on == "input" else set())
        if self.runtime.fast_kernels and self.hidden >= 128:
            libs |= {"gemm_tc", "gemm_tc2"}
        return libs

    def load(self, source) -> None:
        rt = self.runtime
        self.router = self.fetch(source, self.n_router)
        if self.n_correction:
            self.correction = self.fetch(source, self.n_correction)

        E, C, I = self.num_experts, self.shared_chunks, self.inter

        def slab(proj: str, rows: int, cols: int) -> torch.Tensor:
            out = torch.empty((E + C, rows, cols), dtype=rt.matrix_dtype, device=rt.device)
            for e in range(E):
                out[e].copy_(self.fetch(source, self.expert_name(proj, e)))
            return out

        self.w_gate = slab("gate", I, self.hidden) if self.gated else None
        self.w_up = slab("up", I, self.hidden)
        self.w_down = slab("down", self.hidden, I)
        if self.shared_inter > 0:
            ws_gate = self.fetch(source, self.n_shared["gate"]) if self.gated else None
            ws_up = self.fetch(source, self.n_shared["up"])
            ws_down = self.fetch(source, self.n_shared["down"])
            if C > 0:
                # chunk c of the shared expert: rows [c I, (c + 1) I) of gate and up, columns of down
                if self.gated:
                    self.w_gate[E:].copy_(ws_gate.view(C, I, self.hidden))
                self.w_up[E:].copy_(ws_up.view(C, I, self.hidden))
                self.w_down[E:].copy_(ws_down.view(self.hidden, C, I).permute(1, 0, 2))
                if rt.fast_kernels:
                    # steps with many rows run the shared expert as dense products of its own (see
                    # forward): gate and up are then the chunks' rows seen as one matrix, the down
                    # projection is held a second time, whole
                    self.ws_down = ws_down
            else:
                self.ws_gate, self.ws_up, self.ws_down = ws_gate, ws_up, ws_down
            if self.shared_gate:
                self.shared_gate_w = self.fetch(source, self.n_shared_sg).reshape(-1).contiguous()

        self._prepare_split_router()

    # Router logits on the tensor cores, float32-grade.  The normed row arrives as three
    # bfloat16 terms hi | mid | lo (their sum is the float32 value to 2^-24); the router's
    # weights, when they are exactly representable in bfloat16 (a bfloat16 checkpoint), are
    # laid three times side by side, so one bfloat16 product over K = 3 hidden, accumulated in
    # float32 and cut along K into partial sums, gives sum_j w[e, j] (hi + mid + lo)[j] with
    # every product exact.  Used for many rows; few rows take the fused float32 kernel.
    SPLIT_ROUTER_MIN_ROWS = 64

    def _prepare_split_router(self) -> None:
        rt = self.runtime
        self.router_split = None
        if not rt.fast_kernels or self.hidden % 8 != 0 or self.hidden < 128:
            return
        rows = [self.router]
        if self.shared_gate:
            rows.append(self.shared_gate_w.view(1, -1))
        w = torch.cat(rows, dim=0)
        wb = w.to(torch.bfloat16)
        if not torch.equal(wb.to(torch.float32), w):
            return                              # weights with more than 8 bits of mantissa: the float32 kernel
        cols = -(-w.shape[0] // 16) * 16
        padded = torch.zeros((cols, self.hidden), dtype=torch.bfloat16, device=w.device)
        padded[:w.shape[0]] = wb
        self.router_split = torch.cat([padded, padded, padded], dim=1).contiguous()

    # From this many rows on, the shared expert leaves the grouped products: as extra groups it
    # costs a copy of every row per chunk in the gather, a float32 partial result per chunk out of
    # the down product and as many reads in the combine - bytes that a step with few rows does not
    # notice beside the weights, and a step with many rows does.
    SHARED_DENSE_MIN_ROWS = 512

    def wants_split_input(self, rows: int) -> bool:
        # with the weight on the expert's input the float32 row itself is needed, not its three-term form
        return self.router_split is not None and rows >= self.SPLIT_ROUTER_MIN_ROWS and self.weight_on == "output"

    def _route(self, x_exact: torch.Tensor, sel, wts, shared_scale, pin=None, gap=None) -> None:
        k = self.top_k
        if x_exact.dtype == torch.bfloat16:
            # the three-term form: one tensor-core product, cut along K so that the machine is
            # occupied and the float32 sums stay short
            T = x_exact.shape[0]
            cols, Kd = self.router_split.shape
            k_blocks = Kd // 64
            tiles = -(-T // 128) * -(-cols // 128)
            rt_sms = self.runtime.sm_count
            splits = max(1, min(8, k_blocks // 8, -(-rt_sms // tiles)))
            logits = torch.empty((splits, T, cols), dtype=torch.float32, device=x_exact.device)
            K.gemm_tc(x_exact, self.router_split, logits if splits > 1 else logits[0], K.EPI_STORE_F32, False, 128,
                      k_splits=splits)
            K.router_select(logits, self.num_experts, k, self.norm_topk, sel, wts, shared_scale, pin=pin, gap=gap,
                            sigmoid_scores=self.score == "sigmoid", groups=self.route_groups, correction=self.correction,
                            weight_scale=self.route_scale, group_top2=self.group_score == "top2", norm_floor=self.norm_floor)
        else:
            K.router_topk(x_exact, self.router, self.shared_gate_w, k, self.norm_topk, sel, wts, shared_scale, pin=pin, gap=gap,
                          sigmoid_scores=self.score == "sigmoid", groups=self.route_groups, correction=self.correction,
                          weight_scale=self.route_scale, group_top2=self.group_score == "top2", norm_floor=self.norm_floor)

    def forward(self, x: torch.Tensor, x_exact: torch.Tensor, residual: torch.Tensor, ctx) -> None:
        rt = self.runtime
        dev = x.device
        T = x.shape[0]
        k, E = self.top_k, self.num_experts
        sel = torch.empty((T, k), dtype=torch.int32, device=dev)
        wts = torch.empty((T, k), dtype=torch.float32, device=dev)
        shared_scale = torch.empty((T,), dtype=torch.float32, device=dev) if self.shared_gate else None
        # a step may bring the experts of its rows with it (``ctx.routing_pin``: this part's tensor-name
        # prefix -> int32 [rows, k]; the weights stay the rows' own probabilities), or ask for what was
        # picked and how narrowly (``ctx.routing_dump``: prefix -> (experts, margins))
        pins, dump = getattr(ctx, "routing_pin", None), getattr(ctx, "routing_dump", None)
        # a layer that runs several times a step (a looped stretch) is '<prefix>' the first time and
        # '<prefix>#1', '<prefix>#2', ... after that, in both dictionaries
        key = self.prefix
        if pins is not None or dump is not None:
            seen = ctx.routing_seen.get(self.prefix, 0)
            ctx.routing_seen[self.prefix] = seen + 1
            if seen:
                key = f"{self.prefix}#{seen}"
        pin = pins.get(key) if pins else None
        gap = torch.empty((T,), dtype=torch.float32, device=dev) if dump is not None and pin is None else None
        K.tag = "router"
        self._route(x_exact, sel, wts, shared_scale, pin, gap)
        if dump is not None:
            dump[key] = (sel, gap)

        shared_dense = self.ws_down is not None and self.shared_chunks > 0 and T >= self.SHARED_DENSE_MIN_ROWS
        C = 0 if shared_dense else self.shared_chunks
        n_slots = T * k + C * T
        offsets = torch.empty((E + C + 1,), dtype=torch.int32, device=dev)
        slot_token = torch.empty((n_slots,), dtype=torch.int32, device=dev)
        slot_of_pick = torch.empty((T * k,), dtype=torch.int32, device=dev)
        K.tag = "grouping"
        K.moe_group(sel, k, E, offsets, slot_token, slot_of_pick, extra_groups=C)

        act = torch.empty((n_slots, self.inter), dtype=rt.act_dtype, device=dev)
        G = E + C
        if self.weight_on == "input":
            # a pick's score multiplies the float32 row; the product then reads the scaled rows in
            # the grouped order, and the combine adds the experts' results unweighted
            if C > 0 or self.shared_inter > 0:
                raise ValueError("weight_on='input' with a shared expert is not built")
            scaled = torch.empty((n_slots, self.hidden), dtype=rt.act_dtype, device=dev)
            K.tag = "row gather"
            K.scale_rows_gather(x_exact, slot_of_pick, wts, k, scaled)
            K.tag = "experts gate/up"
            project(rt, scaled, self.w_gate[:G], act, w_up=self.w_up[:G], group_offsets=offsets, max_group_rows=T,
                    offsets_settled=True, act_limit=self.act_limit, act_alpha=self.act_alpha)
            wts = torch.ones_like(wts)
        elif not self.gated:
            # an expert without a gate: the activation of the float32 sum in the product's epilogue, then rounded
            K.tag = "experts up"
            project(rt, x, self.w_up[:G], act, group_offsets=offsets, a_row_index=slot_token, max_group_rows=T, act=self.activation)
        else:
            K.tag = "experts gate/up"
            project(rt, x, self.w_gate[:G], act, w_up=self.w_up[:G], group_offsets=offsets, a_row_index=slot_token,
                    max_group_rows=T, act_limit=self.act_limit, act_alpha=self.act_alpha)
        y = torch.empty((n_slots, self.hidden), dtype=torch.float32, device=dev)
        K.tag = "experts down"
        project(rt, act, self.w_down[:G], y, group_offsets=offsets, max_group_rows=T, offsets_settled=True)

        shared = None
        if C > 0:
            shared = y[T * k:].view(C, T, self.hidden)
        elif self.shared_inter > 0:
            sact = torch.empty((T, self.shared_inter), dtype=rt.act_dtype, device=dev)
            if shared_dense:
                ws_gate = self.w_gate[E:].view(self.shared_inter, self.hidden) if self.gated else None
                ws_up = self.w_up[E:].view(self.shared_inter, self.hidden)
            else:
                ws_gate, ws_up = self.ws_gate, self.ws_up
            if self.gated:
                K.tag = "shared gate/up"
                project(rt, x, ws_gate, sact, w_up=ws_up, act_limit=self.shared_act_limit, act_alpha=self.shared_act_alpha)
            else:
                K.tag = "shared up"
                project(rt, x, ws_up, sact, act=self.activation)
            shared = torch.empty((T, self.hidden), dtype=torch.float32, device=dev)
            K.tag = "shared down"
            project(rt, sact, self.ws_down, shared)
        K.tag = "combine"
        K.moe_combine(residual, y, slot_of_pick, wts, k, shared, shared_scale)
        K.tag = None
