"""``gated_mlp``: the dense gated feed-forward: down(act(gate(x)) * up(x)), no biases; act is the
tanh-GELU or SiLU (``activation``: "gelu_pytorch_tanh", "silu").

Reference: src/model/layer.rs:696-710 (two products, the gated activation,
the down product), src/backend/cpu.rs:1190-1199 (tanh-GELU).  The gate and up
matrices are kept as ONE matrix so that one product makes both halves; when
the intermediate size allows it their rows are interleaved in groups of 8
(8 gate rows, then the 8 matching up rows), which puts a gate value and its
up value into the same thread of the weight-streaming kernel, whose epilogue
then writes act(gate) * up directly.

``mlp``: the feed-forward without a gate, down(act(up(x))), no biases; act is the square of
relu (``activation``: "relu_squared"), the tanh-GELU or SiLU.

``clipped_gated_mlp``: the dense form of the routed experts' clipped activation,
down(g * sigmoid(alpha g) * (u + 1)) with g = min(gate x, limit), u = clamp(up x, +-limit);
parameters ``intermediate_size``, ``limit``, ``alpha`` (default 1.702).

``routed_experts``: many small gated feed-forwards of which every row uses ``top``.  Parameters:
``experts``, ``top``, ``intermediate_size``, ``limit``, ``alpha`` (default 1.702), ``router_bias``,
``shared`` (None, or {"intermediate_size", "limit"}: one more expert that every row uses).
    expert(x) = down(g * sigmoid(alpha g) * (u + 1)),  g = min(gate x, limit),  u = clamp(up x, +-limit)
    z = router x + bias (32-bit);  the ``top`` largest z choose the experts (ties: the lower index),
    their weights are the softmax over the chosen z alone;  y = sum_k p_k expert_k(x) + shared(x)
``score`` "sigmoid" (default "softmax_top"): a chosen expert's weight is the sigmoid of its own
logit, not normalized over the chosen.  ``form`` "plain_gelu" (default "clipped_gated"): an
expert, and the shared one, is down(gelu(up x)) with the exact gelu and no gate matrix, and a
row's weight multiplies what ENTERS its expert, y = sum_k expert_k(p_k x) + shared(x); as the
experts have no biases, up(p x) = p up(x), so the weight is applied in 32-bit to the up
product's output in front of the gelu.
``form`` "gated_silu": an expert, and the shared one, is down(silu(gate x) * (up x)).  ``score``
"softmax_all": s = softmax(z) over all experts; the ``top`` largest s + ``correction`` (a stored
number per expert, with ``correction`` True) choose, and a chosen expert's weight is its s,
without the correction and not normalized, times ``router_scale`` (default 1).
``shared["gate"]`` True: the shared expert's output is multiplied by sigmoid(shared.gate.weight x),
one number per row (the gate's row lies behind the router's, so that one 32-bit product makes
both; the factor is applied in 32-bit where the experts' outputs are summed).
More than 128 bfloat16 rows of gated experts (recorded or not): the pairs are sorted by expert on the
device and all experts run as two grouped tcgen05 products over tiles of 256 sorted rows
(csrc/gemm_tcgen05.cu), the gated activation in the first one's epilogue; the host reads nothing,
and experts with many rows cost what their rows cost.
Few rows, and every recorded step: each (row, expert) pair streams its expert's matrices
(csrc/routed.cu routed_rows).  Many rows: the pairs are sorted by expert on the device into a
layout [experts, most rows of any expert, width] (that one number is read on the host; a recorded
step takes its number of rows instead and reads nothing) and all experts run as two batched library
products around one activation launch.
"""

from __future__ import annotations

import os
from typing import Dict, Mapping

import torch

from ..config.spec import ConfigError
from ..kernels import native
from ..weights.arena import Piece, Resident
from ..weights.loader import TensorDecl
from .registry import register_feed_forward

from typing import Optional

# activation of the gate -> (elementwise kernel's code, fused epilogue of the products or None)
_ACTIVATIONS = {"gelu_pytorch_tanh": (native.ACT_GELU_TANH, native.EPI_GEGLU),
                "silu": (native.ACT_SILU, native.EPI_SWIGLU)}
_GROUP = 8


class GatedMLP:
    chain_safe = True      # deferred results are read by this runtime's and native's launchers only
    captures_prompts = True   # row-wise: a recorded step of prompts may be replayed for others

    @staticmethod
    def tensors(params: Mapping, hidden: int) -> Dict[str, TensorDecl]:
        inter = params["intermediate_size"]
        return {
            "gate_proj.weight": TensorDecl((inter, hidden)),
            "up_proj.weight": TensorDecl((inter, hidden)),
            "down_proj.weight": TensorDecl((hidden, inter)),
        }

    @staticmethod
    def resident(params: Mapping, hidden: int) -> Dict[str, Resident]:
        """Gate and up as ONE matrix: runs of 8 gate rows followed by the 8 matching up
        rows when the intermediate size is a multiple of 8, else all gates, then all ups."""
        inter = int(params["intermediate_size"])
        if inter % _GROUP == 0:
            pieces = (Piece("gate_proj.weight", 0, _GROUP, 2 * _GROUP),
                      Piece("up_proj.weight", _GROUP, _GROUP, 2 * _GROUP))
        else:
            pieces = (Piece("gate_proj.weight", 0), Piece("up_proj.weight", inter))
        return {
            "gate_up_proj.weight": Resident((2 * inter, hidden), pieces=pieces),
            "down_proj.weight": Resident((hidden, inter), pieces=(Piece("down_proj.weight"),)),
        }

    def __init__(self, params: Mapping, hidden: int, weights: Mapping[str, torch.Tensor], rt):
        self.rt = rt
        self.inter = int(params["intermediate_size"])
        act = params.get("activation", "gelu_pytorch_tanh")
        if act not in _ACTIVATIONS:
            raise ConfigError(f"gated_mlp: activation {act!r} is not supported; "
                              f"known: {', '.join(_ACTIVATIONS)}")
        self.act, self.epilogue = _ACTIVATIONS[act]
        self.group = _GROUP if self.inter % _GROUP == 0 else 0
        self.w_gate_up = rt.cast_matrix(weights["gate_up_proj.weight"])
        self.w_down = rt.cast_matrix(weights["down_proj.weight"])

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        rt = self.rt
        R = x.shape[0]
        if (self.epilogue is not None and self.group == _GROUP and x.dtype == torch.bfloat16
                and x.shape[1] % 8 == 0
                and (R <= rt.skinny_max_rows or R > rt.gated_gemm_min_rows
                     or (rt.chain is not None and R <= rt.chain_max_rows
                         and self.epilogue == native.EPI_GEGLU))):
            t = rt.linear(x, self.w_gate_up, epilogue=self.epilogue)
        else:
            gate_up = rt.linear(x, self.w_gate_up)
            t = torch.empty((R, self.inter), dtype=x.dtype, device=x.device)
            native.gelu_mul(gate_up, t, self.group, self.act)
        return rt.linear(t, self.w_down)


_PLAIN_ACTIVATIONS = {"relu_squared": native.ACT_RELU_SQUARED, "gelu_pytorch_tanh": native.ACT_GELU_TANH,
                      "silu": native.ACT_SILU}


class PlainMLP:
    captures_prompts = True   # row-wise: a recorded step of prompts may be replayed for others

    @staticmethod
    def tensors(params: Mapping, hidden: int) -> Dict[str, TensorDecl]:
        inter = params["intermediate_size"]
        return {"up_proj.weight": TensorDecl((inter, hidden)),
                "down_proj.weight": TensorDecl((hidden, inter))}

    @staticmethod
    def resident(params: Mapping, hidden: int) -> Dict[str, Resident]:
        inter = int(params["intermediate_size"])
        return {"up_proj.weight": Resident((inter, hidden), pieces=(Piece("up_proj.weight"),)),
                "down_proj.weight": Resident((hidden, inter), pieces=(Piece("down_proj.weight"),))}

    def __init__(self, params: Mapping, hidden: int, weights: Mapping[str, torch.Tensor], rt):
        self.rt = rt
        self.inter = int(params["intermediate_size"])
        act = params.get("activation", "relu_squared")
        if act not in _PLAIN_ACTIVATIONS:
            raise ConfigError(f"mlp: activation {act!r} is not supported; "
                              f"known: {', '.join(_PLAIN_ACTIVATIONS)}")
        self.act = _PLAIN_ACTIVATIONS[act]
        self.w_up = rt.cast_matrix(weights["up_proj.weight"])
        self.w_down = rt.cast_matrix(weights["down_proj.weight"])

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        if self.act == native.ACT_RELU_SQUARED:
            # (the products have this activation as an epilogue; where a library product is
            # taken the runtime applies it behind)
            up = self.rt.linear(x, self.w_up, epilogue=native.EPI_RELU2)
        else:
            up = self.rt.linear(x, self.w_up)
            native.activate(up, up, self.act)
        return self.rt.linear(up, self.w_down)


class ClippedGatedMLP:
    captures_prompts = True   # row-wise: a recorded step of prompts may be replayed for others

    @staticmethod
    def tensors(params: Mapping, hidden: int) -> Dict[str, TensorDecl]:
        inter = params["intermediate_size"]
        return {"gate_proj.weight": TensorDecl((inter, hidden)),
                "up_proj.weight": TensorDecl((inter, hidden)),
                "down_proj.weight": TensorDecl((hidden, inter))}

    @staticmethod
    def resident(params: Mapping, hidden: int) -> Dict[str, Resident]:
        """Gate and up as ONE matrix, laid out as the gated feed-forward's: runs of 8 gate rows
        followed by the 8 matching up rows when the intermediate size is a multiple of 8 (the
        products' clipped epilogue then writes the activated middle itself), else all gates,
        then all ups."""
        inter = int(params["intermediate_size"])
        if inter % _GROUP == 0:
            pieces = (Piece("gate_proj.weight", 0, _GROUP, 2 * _GROUP),
                      Piece("up_proj.weight", _GROUP, _GROUP, 2 * _GROUP))
        else:
            pieces = (Piece("gate_proj.weight", 0), Piece("up_proj.weight", inter))
        return {"gate_up_proj.weight": Resident((2 * inter, hidden), pieces=pieces),
                "down_proj.weight": Resident((hidden, inter), pieces=(Piece("down_proj.weight"),))}

    def __init__(self, params: Mapping, hidden: int, weights: Mapping[str, torch.Tensor], rt):
        self.rt = rt
        self.inter = int(params["intermediate_size"])
        self.limit = float(params["limit"])
        self.alpha = float(params.get("alpha", 1.702))
        if self.inter <= 0 or self.limit <= 0:
            raise ConfigError(f"clipped_gated_mlp: intermediate_size {self.inter}, limit {self.limit}")
        self.w_gate_up = rt.cast_matrix(weights["gate_up_proj.weight"])
        self.w_down = rt.cast_matrix(weights["down_proj.weight"])

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        rt, R = self.rt, x.shape[0]
        group = _GROUP if self.inter % _GROUP == 0 else 0
        # (the products' epilogue has the design's constant 1.702 built in)
        if (group and self.alpha == 1.702 and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0
                and (R <= rt.skinny_max_rows or R > rt.gated_gemm_min_rows)):
            mid = rt.linear(x, self.w_gate_up, epilogue=native.EPI_CLIPPED, cap=self.limit)
        else:
            gu = rt.linear(x, self.w_gate_up)
            rt.flush()
            mid = torch.empty((R, self.inter), dtype=x.dtype, device=x.device)
            native.expert_activate(gu, mid, None, self.limit, self.alpha, native.FORM_CLIPPED_GATED, group)
        return rt.linear(mid, self.w_down)


_FORMS = {"clipped_gated": native.FORM_CLIPPED_GATED, "plain_gelu": native.FORM_PLAIN_GELU,
          "gated_silu": native.FORM_GATED_SILU}
_SCORES = {"softmax_top": native.SCORE_SOFTMAX_TOP, "sigmoid": native.SCORE_SIGMOID,
           "softmax_all": native.SCORE_SOFTMAX_ALL}


class RoutedExperts:
    captures_prompts = True   # a recorded step reads the choices on the device only

    def reads_sizes_on_host(self, rows: int) -> bool:
        """Whether a launched step of so many rows reads on the host how many rows chose each expert."""
        return rows > self.pair_rows and not self._grouped(rows)

    def _grouped(self, rows: int) -> bool:
        return (rows >= self.grouped_rows and self.rt.dtype == torch.bfloat16 and self.hidden % 8 == 0
                and self.ff % 8 == 0 and self.E <= 1024
                and (self.form == native.FORM_GATED_SILU or (self.clipped and self.alpha == 1.702)))

    @staticmethod
    def _sizes(params: Mapping):
        E, top, ff = int(params["experts"]), int(params["top"]), int(params["intermediate_size"])
        if E <= 0 or not 0 < top <= min(E, 32) or ff <= 0:
            raise ConfigError(f"routed_experts: {E} experts of {ff}, {top} a row (at most 32)")
        shared = params.get("shared") or None
        sff = int(shared["intermediate_size"]) if shared else 0
        if shared and sff <= 0:
            raise ConfigError("routed_experts: the shared expert's intermediate_size must be positive")
        return E, top, ff, sff

    @staticmethod
    def _form(params: Mapping) -> int:
        form, score = params.get("form", "clipped_gated"), params.get("score", "softmax_top")
        if form not in _FORMS or score not in _SCORES:
            raise ConfigError(f"routed_experts: form {form!r} and score {score!r}; known: "
                              f"{', '.join(_FORMS)}; {', '.join(_SCORES)}")
        if bool(params.get("correction")) and score != "softmax_all":
            raise ConfigError("routed_experts: a correction goes with the score 'softmax_all'")
        return _FORMS[form]

    @staticmethod
    def _shared_gate(params: Mapping) -> bool:
        return bool(params.get("shared") and params["shared"].get("gate"))

    @staticmethod
    def _shared_mlp(params: Mapping):
        """The shared expert of gated SiLU experts is the dense gated feed-forward, as it is."""
        return {"intermediate_size": int(params["shared"]["intermediate_size"]), "activation": "silu"}

    @classmethod
    def tensors(cls, params: Mapping, hidden: int) -> Dict[str, TensorDecl]:
        E, top, ff, sff = cls._sizes(params)
        out = {"router.weight": TensorDecl((E, hidden))}
        if params.get("router_bias", True):
            out["router.bias"] = TensorDecl((E,), init="norm")
        if params.get("correction"):
            out["correction"] = TensorDecl((E,), init="norm")
        if cls._shared_gate(params):
            out["shared.gate.weight"] = TensorDecl((1, hidden))
        gated = cls._form(params) != native.FORM_PLAIN_GELU
        for e in range(E):
            if gated:
                out[f"experts.{e}.gate_proj.weight"] = TensorDecl((ff, hidden))
            out[f"experts.{e}.up_proj.weight"] = TensorDecl((ff, hidden))
            out[f"experts.{e}.down_proj.weight"] = TensorDecl((hidden, ff))
        if sff:
            if gated:
                out["shared.gate_proj.weight"] = TensorDecl((sff, hidden))
            out["shared.up_proj.weight"] = TensorDecl((sff, hidden))
            out["shared.down_proj.weight"] = TensorDecl((hidden, sff))
        return out

    @classmethod
    def resident(cls, params: Mapping, hidden: int) -> Dict[str, Resident]:
        """All experts' gate and up matrices as one [experts, 2 ff, hidden] (an expert's gate
        rows, then its up rows; experts without a gate: [experts, ff, hidden], the up rows
        alone) and their down matrices as one [experts, hidden, ff]; the router's matrix 32-bit."""
        E, top, ff, sff = cls._sizes(params)
        form = cls._form(params)
        gated = form != native.FORM_PLAIN_GELU
        per = 2 if gated else 1
        gu, down = [], []
        for e in range(E):
            if gated:
                gu.append(Piece(f"experts.{e}.gate_proj.weight", e * 2 * ff))
            gu.append(Piece(f"experts.{e}.up_proj.weight", e * per * ff + (ff if gated else 0)))
            down.append(Piece(f"experts.{e}.down_proj.weight", e * hidden))
        router = (Piece("router.weight", 0),)
        if cls._shared_gate(params):
            router += (Piece("shared.gate.weight", E),)
        out = {"router.weight": Resident((E + len(router) - 1, hidden), torch.float32, router),
               "experts.gate_up.weight": Resident((E * per * ff, hidden), pieces=tuple(gu)),
               "experts.down.weight": Resident((E * hidden, ff), pieces=tuple(down))}
        if params.get("router_bias", True):
            out["router.bias"] = Resident((E,), torch.float32, (Piece("router.bias"),))
        if params.get("correction"):
            out["router.bias"] = Resident((E,), torch.float32, (Piece("correction"),))
        if sff and form == native.FORM_GATED_SILU:
            for name, res in GatedMLP.resident(cls._shared_mlp(params), hidden).items():
                out["shared." + name] = Resident(res.shape, res.dtype, tuple(
                    Piece("shared." + q.source, q.row_offset, q.group, q.group_stride) for q in res.pieces),
                    res.offset)
            return out
        if sff and not gated:
            out["shared.gate_up.weight"] = Resident((sff, hidden), pieces=(Piece("shared.up_proj.weight"),))
        elif sff:
            out["shared.gate_up.weight"] = Resident((2 * sff, hidden), pieces=(
                Piece("shared.gate_proj.weight", 0), Piece("shared.up_proj.weight", sff)))
        if sff:
            out["shared.down.weight"] = Resident((hidden, sff), pieces=(Piece("shared.down_proj.weight"),))
        return out

    def __init__(self, params: Mapping, hidden: int, weights: Mapping[str, torch.Tensor], rt):
        self.rt = rt
        self.hidden = hidden
        self.E, self.top, self.ff, self.sff = self._sizes(params)
        self.form = self._form(params)
        self.score = _SCORES[params.get("score", "softmax_top")]
        self.plain = self.form == native.FORM_PLAIN_GELU
        self.clipped = self.form == native.FORM_CLIPPED_GATED
        self.per = 1 if self.plain else 2          # matrix rows per middle column
        self.limit = float(params["limit"]) if self.clipped else 0.0
        self.router_scale = float(params.get("router_scale", 1.0))
        self.shared_gate = self._shared_gate(params)
        self.alpha = float(params.get("alpha", 1.702))
        self.w_router = weights["router.weight"]
        self.b_router = weights.get("router.bias")
        self.w_gu = rt.cast_matrix(weights["experts.gate_up.weight"]).view(self.E, self.per * self.ff, hidden)
        self.w_down = rt.cast_matrix(weights["experts.down.weight"]).view(self.E, hidden, self.ff)
        self.shared_limit = float(params["shared"]["limit"]) if self.sff and self.clipped else 0.0
        self.shared: Optional[GatedMLP] = None
        self.w_sgu = self.w_sdown = None
        if self.sff and self.form == native.FORM_GATED_SILU:
            self.shared = GatedMLP(self._shared_mlp(params), hidden, {
                k[len("shared."):]: v for k, v in weights.items() if k.startswith("shared.")}, rt)
        elif self.sff:
            self.w_sgu = rt.cast_matrix(weights["shared.gate_up.weight"])
            self.w_sdown = rt.cast_matrix(weights["shared.down.weight"])
        # up to this many rows every (row, expert) pair streams its own expert's matrices
        self.pair_rows = 32
        # from this many rows on gated experts run as grouped products (SIB_GROUPED_EXPERTS=0: never)
        self.grouped_rows = 129 if os.environ.get("SIB_GROUPED_EXPERTS", "1") != "0" else 1 << 40

    def choose(self, x: torch.Tensor):
        """(ids int32 [rows, top], weights 32-bit [rows, top]) of the rows' experts, and the
        shared expert's weight per row (32-bit [rows], None without such a gate)."""
        R = x.shape[0]
        gate = torch.empty(R, dtype=torch.float32, device=x.device) if self.shared_gate else None
        if R <= self.pair_rows and (self.hidden + self.E + 4) * 4 <= 48 * 1024:
            ids = torch.empty((R, self.top), dtype=torch.int32, device=x.device)
            p = torch.empty((R, self.top), dtype=torch.float32, device=x.device)
            native.router_rows(x, self.w_router, self.b_router, ids, p, self.score, self.router_scale, gate)
            return ids, p, gate
        x32 = x if x.dtype == torch.float32 else native.cast_rows(
            x, torch.empty(x.shape, dtype=torch.float32, device=x.device))
        with native.profile_region("library product (router, 32-bit)", (R + self.E) * self.hidden * 4,
                                   2.0 * R * self.E * self.hidden):
            z = torch.matmul(x32, self.w_router.t())
        ids = torch.empty((R, self.top), dtype=torch.int32, device=x.device)
        p = torch.empty((R, self.top), dtype=torch.float32, device=x.device)
        native.router_topk(z, self.b_router, ids, p, self.score, self.router_scale, gate)
        return ids, p, gate

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        rt, R = self.rt, x.shape[0]
        rt.flush()
        ids, p, base_weight = self.choose(x)
        base: Optional[torch.Tensor] = None
        if self.shared is not None:
            base = self.shared.forward(x, ctx)
        elif self.sff and self.plain:
            # (the gelu is an epilogue of the up product where a hand-written product runs)
            base = rt.linear(rt.linear(x, self.w_sgu, epilogue=native.EPI_GELU), self.w_sdown)
        elif self.sff:
            gu = rt.linear(x, self.w_sgu)
            mid = torch.empty((R, self.sff), dtype=x.dtype, device=x.device)
            native.expert_activate(gu, mid, None, self.shared_limit, self.alpha, self.form)
            base = rt.linear(mid, self.w_sdown)
        out = torch.empty((R, self.hidden), dtype=x.dtype, device=x.device)
        # (the streamed kernels keep a row and its `top` middles in shared memory)
        streams = self.hidden * 4 <= 48 * 1024 and self.top * self.ff * 4 <= 48 * 1024
        if R <= self.pair_rows and streams and R * self.top < 65536:
            return native.routed_rows(x, self.w_gu, self.w_down, ids, p, base, out, self.limit, self.alpha,
                                      self.form, base_weight)
        if self._grouped(R):
            where, tiles = native.expert_plan(ids, self.E)
            xs = native.spread_rows(x, where, torch.empty((R * self.top, self.hidden), dtype=x.dtype, device=x.device))
            mid = torch.empty((R * self.top, self.ff), dtype=x.dtype, device=x.device)
            native.gemm_tcgen05_grouped(xs, self.w_gu, tiles, mid, native.EPI_CLIPPED if self.clipped else
                                        native.EPI_SWIGLU, self.limit)
            # (the sorted rows have been read: their place takes the outputs)
            ys = native.gemm_tcgen05_grouped(mid, self.w_down, tiles, xs)
            return native.routed_combine(ys, where, p, base, out, base_weight)
        # The pairs sorted by expert and laid out [experts, most, width] with `most` the largest
        # number of rows any expert got (the one number read on the host; rows behind an
        # expert's own are zeros): all experts run as ONE batched library product for gate and
        # up, one activation launch and one batched product for down.  `where[r, k]`: the
        # place of row r's k-th pair in that layout.
        # A recorded step reads nothing on the host: every expert gets room for all the step's
        # rows (an expert is chosen at most once a row).  For the 33 to 64 rows of such a step
        # that is a few products' worth of zeros on the tensor cores, against the streamed
        # kernels' sums on the CUDA cores (64 rows of 4 experts each: 558 us a layer).
        E, top, W = self.E, self.top, self.hidden
        flat = ids.view(-1).to(torch.int64)
        order = torch.argsort(flat, stable=True)
        counts = torch.zeros(E, dtype=torch.int64, device=x.device).index_add_(
            0, flat, torch.ones_like(flat))
        most = R if ctx.graph_capture else int(counts.max().item())
        most = -(-most // 8) * 8
        by_expert = flat[order]
        place = by_expert * most + (torch.arange(order.numel(), device=x.device)
                                    - (torch.cumsum(counts, 0) - counts)[by_expert])
        xs = torch.zeros((E * most, W), dtype=x.dtype, device=x.device)
        xs.index_copy_(0, place, x.index_select(0, torch.div(order, top, rounding_mode="floor")))
        where = torch.empty(order.numel(), dtype=torch.int32, device=x.device)
        where[order] = place.to(torch.int32)
        esz = x.element_size()
        with native.profile_region(f"library product (experts, {E} x {most} rows, gate and up)",
                                   (E * most * (W + self.per * self.ff) + self.w_gu.numel()) * esz,
                                   2.0 * E * most * W * self.per * self.ff):
            gu = torch.bmm(xs.view(E, most, W), self.w_gu.transpose(1, 2))
        mid = torch.empty((E * most, self.ff), dtype=x.dtype, device=x.device)
        row_weight = None
        if self.plain:
            # a pair's weight enters its expert: on the sorted rows, in front of the gelu
            row_weight = torch.zeros(E * most, dtype=torch.float32, device=x.device)
            row_weight.index_copy_(0, place, p.view(-1).index_select(0, order))
        native.expert_activate(gu.view(E * most, self.per * self.ff), mid, row_weight, self.limit, self.alpha,
                               self.form)
        with native.profile_region(f"library product (experts, {E} x {most} rows, down)",
                                   (E * most * (W + self.ff) + self.w_down.numel()) * esz,
                                   2.0 * E * most * W * self.ff):
            ys = torch.bmm(mid.view(E, most, self.ff), self.w_down.transpose(1, 2))
        return native.routed_combine(ys.view(E * most, W), where.view(R, top), None if self.plain else p,
                                     base, out, base_weight)


register_feed_forward("gated_mlp", GatedMLP)
register_feed_forward("mlp", PlainMLP)
register_feed_forward("clipped_gated_mlp", ClippedGatedMLP)
register_feed_forward("routed_experts", RoutedExperts)
