"""Mixture-of-experts feed-forward with a softmax router.

    p = softmax(Wr x) over all experts; the top-k p, in descending order, are the
    weights (divided by their sum if ``norm_topk_prob``);
    y = sum_k w_k * down_e( silu(gate_e x) * (up_e x) ), summed in rank order;
    y += sigmoid(w_sg . x) * shared(x)   (the gate only if the checkpoint has it).

Variants the spec can ask for: ``scores="sigmoid"`` (the weights are sigmoid(logit) of the chosen experts; the
choice is the same, both scores rise with the logit); ``weight_on_input`` (y = sum_k expert_e(w_k x): the rows are
scaled while they are brought into expert order, and the combination adds the experts' outputs as they are);
``activation`` (what the gate passes through, e.g. the clamped unit with its limit; the shared expert may have its
own constants); ``plain_activation`` (experts without a gate, down(act(up x)), the shared expert likewise: the
products' epilogues apply act); ``choice_bias`` (a number per expert added to the sigmoid scores for the choice only;
the weights use the scores without it), ``weight_scale`` (a factor on the final weights) and ``renorm_eps`` (added to
the sum the kept scores are divided by).

``table``: no router at all.  An integer table names every token id's experts, each with weight 1/top_k; the choice
depends on the step's token ids alone, so the first such layer of a step sorts the tokens of all of them, in one launch.

Reference: router crates/ferrox-moe/src/lib.rs:333-355, expert :619-659, combine
:735-752, shared expert and its sigmoid gate crates/ferrox-models/src/decoder.rs:
2660-2681 and (batched) :1037-1093; tokens bucketed by expert :2792-2890.

Tokens are sorted by expert on the device (no host round trip between the router
and the experts); each expert's rows form one group of a grouped matrix product.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorDecl, WeightsError
from .base import FeedForward, register_part
from .mlp import pack_gate_up

# From this many tokens on the routed experts go through the tcgen05 kernel with swapped roles (measured).
SWAP_MIN_TOKENS = 8


def expert_tile_tokens(T: int, K: int, E: int):
    """Tokens per tile of the swapped-role kernel for the routed experts' products, by the mean number of rows
    an expert gets; None where the 128-row tiles of the plain tcgen05 kernel are as good.  Measured on a B200
    with 60 experts: decode batches of 8 to 64 tokens gain 5 to 25 %; with uniform routing the swapped kernel
    stays a few per cent ahead up to some 20 rows an expert, but routing is never uniform, an expert with more
    rows than a tile holds streams its matrix again for each further tile, and inside the model prompts of 512
    and 2048 tokens were faster with the 128-row tiles."""
    r = T * K / max(E, 1)
    if r <= 8:
        return 32, 32
    if r <= 16:
        return 64, 64
    return None




class SoftmaxTopkMoe(FeedForward):
    graph_safe = True
    fuses_norm = True
    fuses_post_norm = True
    gives_rows = True

    def __init__(self, spec):
        super().__init__(spec)
        s = spec
        self.table_name = getattr(s, "table", None)
        if self.table_name:
            if s.vocab < 1 or s.n_experts > ops.ROUTE_TABLE_MAX_EXPERTS:
                raise ValueError(f"an expert table of {s.vocab} token ids over {s.n_experts} experts (at most "
                                 f"{ops.ROUTE_TABLE_MAX_EXPERTS})")
            if s.shared_gate or getattr(s, "choice_bias", None) or getattr(s, "weight_on_input", False):
                raise ValueError("experts chosen by a table take no choice bias, no shared gate and their weight on the "
                                 "output")
        self.scores = getattr(s, "scores", "softmax")
        if self.scores not in ("softmax", "sigmoid"):
            raise ValueError(f"router scores {self.scores!r}: softmax or sigmoid")
        self.weight_on_input = bool(getattr(s, "weight_on_input", False))
        self.activation = getattr(s, "activation", "silu")
        self.shared_activation = getattr(s, "shared_activation", None) or self.activation
        self.plain = getattr(s, "plain_activation", None)
        if self.plain is not None:
            ops.unary_code(self.plain)                    # unknown activations fail here, by name
            if self.weight_on_input:
                raise ValueError("experts without a gate take their routing weight on the output")
            self._gated = False
        else:
            self._gated = ops.gated_arg(self.activation)
            ops.gated_arg(self.shared_activation)
        self._parts = ("up", "down") if self.plain else ("gate", "up", "down")
        self.choice_bias_name = getattr(s, "choice_bias", None)
        if self.choice_bias_name and self.scores != "sigmoid":
            raise ValueError("a choice bias goes with sigmoid scores")
        self._route_mode = int(bool(s.norm_topk_prob)) | (2 if self.scores == "sigmoid" else 0)
        router, expert, shared = getattr(s, "tensor_names", None) or (
            "gate.weight", "experts.{e}.{part}_proj.weight", "shared_expert.{part}_proj.weight")
        p = s.prefix
        self._router_name = p + router
        self._expert_name = lambda e, part: p + expert.format(e=e, part=part)
        self._shared_name = lambda part: p + shared.format(part=part)
        if not 1 <= s.top_k <= s.n_experts:
            raise ValueError(f"top_k={s.top_k} of {s.n_experts} experts")

    def tensor_decls(self):
        s, p = self.spec, self.spec.prefix
        if self.table_name:
            d = [TensorDecl(p + self.table_name, (s.vocab, s.top_k), integer=True, below=s.n_experts)]
        else:
            d = [TensorDecl(self._router_name, (s.n_experts, s.hidden))]
        shape = lambda part, inner: (s.hidden, inner) if part == "down" else (inner, s.hidden)
        for e in range(s.n_experts):
            d += [TensorDecl(self._expert_name(e, part), shape(part, s.expert_intermediate)) for part in self._parts]
        if self.choice_bias_name:
            d.append(TensorDecl(p + self.choice_bias_name, (s.n_experts,)))
        if s.shared_intermediate > 0:
            d += [TensorDecl(self._shared_name(part), shape(part, s.shared_intermediate)) for part in self._parts]
            if s.shared_gate:
                d.append(TensorDecl(self._shared_gate_name(), (1, s.hidden), optional=True))
        return d

    def _shared_gate_name(self):
        return self.spec.prefix + (getattr(self.spec, "shared_gate_name", None) or "shared_expert_gate.weight")

    def load(self, src, rt):
        super().load(src, rt)
        s, p = self.spec, self.spec.prefix
        if self.table_name:
            self._load_table(src, rt)
        else:
            self.w_router = src.get(self._router_name)
        E, I, H = s.n_experts, s.expert_intermediate, s.hidden
        # If any expert tensor is stored in 32 bits, the packed buffers are 32-bit.
        names = [self._expert_name(e, n) for e in range(E) for n in self._parts]
        dt = torch.float32 if any(src.dtype_of(n) == torch.float32 for n in names) else rt.dtype
        # (experts without a gate: w_gu holds the up rows alone)
        self.w_gu = torch.empty(E, I if self.plain else 2 * I, H, dtype=dt, device=rt.device)
        self.w_down = torch.empty(E, H, I, dtype=dt, device=rt.device)
        for e in range(E):
            if self.plain:
                self.w_gu[e].copy_(src.get(self._expert_name(e, "up")))
            else:
                self.w_gu[e, :I].copy_(src.get(self._expert_name(e, "gate")))
                self.w_gu[e, I:].copy_(src.get(self._expert_name(e, "up")))
            self.w_down[e].copy_(src.get(self._expert_name(e, "down")))
        self.w_shared_gu = self.w_shared_down = self.w_shared_gate = None
        if s.shared_intermediate > 0:
            if self.plain:
                self.w_shared_gu = src.get(self._shared_name("up"))
            else:
                self.w_shared_gu = pack_gate_up(src.get(self._shared_name("gate")), src.get(self._shared_name("up")))
            self.w_shared_down = src.get(self._shared_name("down"))
            if s.shared_gate and src.has(self._shared_gate_name()):
                self.w_shared_gate = src.get(self._shared_gate_name()).reshape(1, H).contiguous()
        # what the routing kernels take beside the mode: the choice bias (32-bit), a factor on the weights, the
        # number added to the sum the kept scores are divided by
        bias = src.get(p + self.choice_bias_name).to(torch.float32).contiguous() if self.choice_bias_name else None
        scale, eps = float(getattr(s, "weight_scale", 1.0)), float(getattr(s, "renorm_eps", 0.0))
        self._route_extra = (bias, scale, eps) if (bias is not None or scale != 1.0 or eps != 0.0) else None
        # router rows and the shared expert's gate row share one product: [E (+1), H]
        self.w_route = None if self.table_name else self.w_router
        if self.w_shared_gate is not None:
            dtr = torch.float32 if torch.float32 in (self.w_router.dtype, self.w_shared_gate.dtype) else self.w_router.dtype
            self.w_route = torch.cat([self.w_router.to(dtr), self.w_shared_gate.to(dtr)], dim=0).contiguous()
        self._scratch = torch.zeros(2 * E, dtype=torch.int32, device=rt.device)
        if self.w_shared_gu is not None and rt.device.type == "cuda":
            self._side = torch.cuda.Stream(device=rt.device)
            self._fork, self._join = torch.cuda.Event(), torch.cuda.Event()

    def _load_table(self, src, rt):
        s = self.spec
        name = s.prefix + self.table_name
        t = src.get(name).to(torch.int32).contiguous()
        row = torch.sort(t, dim=1).values
        if int(t.min()) < 0 or int(t.max()) >= s.n_experts or bool((row[:, 1:] == row[:, :-1]).any()):
            raise WeightsError(f"{name}: every row names {s.top_k} different experts of {s.n_experts}")
        # the tables of one model that one launch sorts tokens for: same sizes, in the order in which they were loaded
        self.table = t
        self._table_group = rt.groups.setdefault(("expert tables", s.vocab, s.top_k, s.n_experts), [])
        self._table_index = len(self._table_group)
        self._table_group.append(t)

    def _route_by_table(self, batch, T, small):
        """(weights, offsets, src_token, inv_perm, active) of this layer: the step's first layer of the group asks for
        all of them at once."""
        s, rt = self.spec, self.rt
        group = self._table_group
        key = ("expert tables", s.vocab, s.top_k, s.n_experts)
        routed = batch.shared.get(key)
        if routed is None:
            L, n, i32 = len(group), T * s.top_k, torch.int32
            ptrs = rt.groups.get(key + ("addresses",))
            if ptrs is None or ptrs.numel() != L:
                ptrs = torch.tensor([t.data_ptr() for t in group], dtype=torch.int64, device=rt.device)
                rt.groups[key + ("addresses",)] = ptrs
            # (a step's first layer asks for buffers of this order each time: they are kept from step to step)
            routed = (rt.empty(T, s.top_k, dtype=torch.float32), rt.empty(L, s.n_experts + 1, dtype=i32),
                      rt.empty(L, n, dtype=i32), rt.empty(L, n, dtype=i32), rt.empty(L, min(s.n_experts, n), dtype=i32))
            ops.route_table(batch.token_ids, ptrs, L, s.vocab, s.n_experts, s.top_k, *routed, stream=batch.stream)
            batch.shared[key] = routed
        w, offsets, src_token, inv_perm, active = routed
        l = self._table_index
        return w, offsets[l], src_token[l], inv_perm[l], active[l] if small else None

    def _shared_expert(self, x, batch, st):
        """silu(gate) * up, then down, of the expert that every token visits: [T, H]."""
        s, rt = self.spec, self.rt
        T, Is = x.shape[0], s.shared_intermediate
        sact = rt.empty(T, Is)
        if self.plain:
            ops.linear(x, self.w_shared_gu, sact, status=batch.status, stream=st, activation=self.plain)
        else:
            ops.gated_linear(x, self.w_shared_gu, sact, status=batch.status, stream=st, activation=self.shared_activation)
        shared = rt.empty(T, s.hidden)
        ops.linear(sact, self.w_shared_down, shared, status=batch.status, stream=st)
        return shared

    def _shared_on_side(self, x, batch):
        """The shared expert's two products on the second stream, from the point the fork event marks."""
        self._side.wait_event(self._fork)
        with torch.cuda.stream(self._side):
            out = self._shared_expert(x, batch, self._side.cuda_stream)
            self._join.record(self._side)
        return out

    def forward_add(self, x, h, batch, then_norm=None):
        st = batch.stream
        y, inv_perm, weights, shared, gate_logit = self.expert_rows(x, batch)
        K = self.spec.top_k
        # the combination applies the norm that follows it where that is an RMSNorm over rows it can hold
        rms = then_norm.as_rms() if then_norm is not None else None
        if rms is not None and ops.combine_norm_ok(h, y):
            out = self.rt.empty(h.shape[0], h.shape[1])
            return ops.moe_combine(h, y, inv_perm, weights, shared, gate_logit, stream=st, norm=(rms[0], rms[1], out),
                                   top_k=K)
        ops.moe_combine(h, y, inv_perm, weights, shared, gate_logit, stream=st, top_k=K)
        return None

    def forward_post(self, x, h, batch, post, then_norm=None):
        """h += post(ffn(x)): one kernel adds a token's expert rows up, norms the sum, adds it to the stream and applies
        the norm that follows to the new row."""
        y, inv_perm, weights, shared, gate_logit = self.expert_rows(x, batch)
        (w, eps), nxt = post.as_rms(), then_norm.as_rms() if then_norm is not None else None
        then = (nxt[0], nxt[1], self.rt.empty(h.shape[0], h.shape[1])) if nxt is not None else None
        return ops.rmsnorm_residual(h, y, w, eps, then=then, expert_rows=(inv_perm, weights, shared, gate_logit),
                                    stream=batch.stream)

    def expert_rows(self, x, batch):
        """The experts' results: (rows in expert order [T * K, H], each (token, rank) pair's row, the weights they are
        added up with (None: as they are), the shared expert's rows or None, its gate's logits or None)."""
        s, rt, st = self.spec, self.rt, batch.stream
        T, E, K, I, H = x.shape[0], s.n_experts, s.top_k, s.expert_intermediate, s.hidden
        i32 = torch.int32
        # A decode step of a few tokens: the router's product, the routing and the rows in expert order come from ONE
        # kernel (three dependent launches otherwise, each a few microseconds of waiting for the one before).
        table = self.table_name is not None
        fused = not table and ops.route_fused_ok(x, self.w_route, E, K)
        mode, gated, scaled = self._route_mode, self._gated, self.weight_on_input
        unary, extra = self.plain, self._route_extra
        tc = ops.tc_ok(x, self.w_gu) and I % 8 == 0 and E <= ops.TC_MAX_GROUPS
        tiles = expert_tile_tokens(T, K, E) if tc and T >= SWAP_MIN_TOKENS and E <= ops.TC_SWAP_MAX_GROUPS else None
        small = tiles is None and T <= ops.SKINNY_MAX_TOKENS and ops.skinny_ok(x, self.w_gu) and I % 32 == 0
        big = T > ops.SKINNY_MAX_TOKENS and tc
        # The shared expert's two products run on a second stream beside the routing and the routed experts; both
        # meet again at the combination.  In a decode step the routed experts' kernels leave most of the machine
        # idle; in a prompt the router's short kernels hide under the shared expert's products.  Measured on a
        # B200: 3 to 10 % of a decode step of 8 to 64 tokens, 14 % of a prompt portion of 256 tokens, 4 % at 2,048.
        shared = None
        overlap = self.w_shared_gu is not None

        if overlap:
            main = torch.cuda.current_stream()
            self._fork.record(main)          # the shared expert may start from here on
            if not fused:
                shared = self._shared_on_side(x, batch)
        if table:
            weights, offsets, src_token, inv_perm, active = self._route_by_table(batch, T, small)
        else:
            # E router logits, then the shared expert's gate logit if it has one
            logits = rt.empty(T, self.w_route.shape[0], dtype=torch.float32)
            ids = rt.empty(T, K, dtype=i32)
            weights = rt.empty(T, K, dtype=torch.float32)
            offsets = rt.empty(E + 1, dtype=i32)
            src_token = rt.empty(T * K, dtype=i32)
            inv_perm = rt.empty(T * K, dtype=i32)
            active = rt.empty(min(E, T * K), dtype=i32) if small else None
        xp = None
        if table:
            pass
        elif fused:
            # The cluster's kernel goes first: it needs eight free SMs of one GPC at once, which it finds now and would
            # not find once the shared expert's weight-streaming kernels (enqueued right after it, waiting only for what
            # was before it) fill every SM.
            xp = rt.empty(T * K, H) if tiles is not None or scaled else None
            ops.route_fused(x, self.w_route, logits, K, mode | (4 if scaled else 0), ids, weights, offsets, src_token, inv_perm, active,
                            n_experts=E, xp_out=xp, stream=st, extra=extra)
            if overlap:
                shared = self._shared_on_side(x, batch)
        elif T <= ops.ROUTE_SMALL_MAX_TOKENS and E <= ops.ROUTE_SMALL_MAX_EXPERTS:
            ops.linear(x, self.w_route, logits, status=batch.status, stream=st)
            ops.route_small(logits, K, mode, ids, weights, offsets, src_token, inv_perm, active,
                            n_experts=E, stream=st, extra=extra)
        else:
            ops.linear(x, self.w_route, logits, status=batch.status, stream=st)
            ops.route(logits, K, mode, ids, weights, self._scratch, offsets, src_token, inv_perm, active,
                      n_experts=E, stream=st, extra=extra)

        act = rt.empty(T * K, I)
        y = rt.empty(T * K, H)
        if scaled and xp is None:
            # the routing weight goes into the expert's input: rows scaled on their way into expert order (the
            # one-cluster routing kernel of a small step has done it already)
            xp = rt.empty(T * K, H)
            ops.gather_rows_scaled(x, src_token, inv_perm, weights, xp, stream=st)
        if tiles is not None:
            # a few rows for each expert: rows in expert order, then features in the lanes of the tensor-core tiles
            # and the expert's rows in their columns
            if xp is None:
                xp = rt.empty(T * K, H)
                ops.gather_rows(x, src_token, xp, stream=st)
            # (the offsets were written by the routing, before the gather: both products may fetch weights early;
            # when one kernel did both, the first product waits for it before it reads the offsets)
            ops.gemm_tc_swap(xp, self.w_gu, act, gated=gated, unary=unary, group_offsets=offsets, tokens_per_tile=tiles[0],
                             weights_first=not fused and not scaled, status=batch.status, stream=st)
            ops.gemm_tc_swap(act, self.w_down, y, group_offsets=offsets, tokens_per_tile=tiles[1],
                             weights_first=True, status=batch.status, stream=st)
        elif small:
            # very few tokens: every expert that was chosen is streamed once, gate/up fused with SiLU
            ops.gemm_skinny(xp if scaled else x, self.w_gu, act, gated=gated, unary=unary, x_rows=None if scaled else src_token,
                            group_offsets=offsets, active_groups=active, tokens_hint=T, stream=st)
            ops.gemm_skinny(act, self.w_down, y, group_offsets=offsets, active_groups=active, tokens_hint=T, stream=st)
        elif big:
            # many tokens: bring them into expert order once, then grouped tensor-core products
            if xp is None:
                xp = rt.empty(T * K, H)
                ops.gather_rows(x, src_token, xp, stream=st)
            ops.gemm_tc(xp, self.w_gu, act, gated=gated, unary=unary, group_offsets=offsets, status=batch.status, stream=st)
            ops.gemm_tc(act, self.w_down, y, group_offsets=offsets, status=batch.status, stream=st)
        else:
            gu = act if unary else rt.empty(T * K, 2 * I)
            ops.gemm(xp if scaled else x, self.w_gu, gu, a_rows=None if scaled else src_token, group_offsets=offsets,
                     stream=st)
            if unary:
                ops.relu_square_(act, stream=st)
            else:
                ops.silu_mul(gu, act, stream=st, activation=self.activation)
            ops.gemm(act, self.w_down, y, group_offsets=offsets, stream=st)

        gate_logit = None
        if self.w_shared_gu is not None:
            if overlap:
                main.wait_event(self._join)
            else:
                shared = self._shared_expert(x, batch, st)
            if self.w_shared_gate is not None:
                gate_logit = logits[:, E:]      # [T, 1] view with the logits' row stride
        return y, inv_perm, None if scaled else weights, shared, gate_logit


register_part("softmax_topk_moe", SoftmaxTopkMoe, replace=True)
