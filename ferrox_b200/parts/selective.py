"""The selective state space of a Mamba mixer.

    [x | z] = Win h;   x = silu(conv(x) + b)                      (causal, per channel; its last inputs are state)
    [low | B | C] = Wx x;   step = softplus(Wdt low + bdt)        (one step size a channel)
    a channel's state row s:   s = e^(-step e^A_log) * s + step x B;   y = s . C + D x
    out = Wo (y * silu(z))

The state [inner, n_state] lives in the cache manager's slots, 32-bit, and so do the convolution's last inputs.  The
projections run in the engine's dtype with 32-bit results where they feed the recurrence.  The inner width of dt is small
and its rows feed the step size: in the bfloat16 engine they are split into two bfloat16 halves that add up to sixteen
bits of mantissa, so that the product by Wdt stays on the tensor cores without rounding its input (``ops.split_rows``).
"""
from __future__ import annotations

import torch

from ..cache.specs import CacheSpec, StateSpec
from ..kernels import ops
from ..weights.loader import TensorDecl
from .base import Mixer, register_part


# A decode step of up to this many requests leaves the step sizes' small product to the recurrence's kernel.
STEP_IN_SCAN_MAX_TOKENS = 16


def _pad_rows(w: torch.Tensor, multiple: int) -> torch.Tensor:
    """Rows of zeros that bring a matrix's height to a multiple."""
    extra = -w.shape[0] % multiple
    return torch.cat([w, torch.zeros(extra, w.shape[1], dtype=w.dtype, device=w.device)]) if extra else w


class SelectiveScan(Mixer):
    graph_safe = True

    def __init__(self, spec):
        super().__init__(spec)
        s = spec
        if not 1 <= s.conv_taps <= 16:
            raise ValueError(f"conv_taps={s.conv_taps}: between 1 and 16")
        if not 1 <= s.n_state <= ops.SELECTIVE_SCAN_MAX_STATE:
            raise ValueError(f"n_state={s.n_state}: the recurrence kernel holds at most {ops.SELECTIVE_SCAN_MAX_STATE} states a channel")
        if s.dt_rank < 1:
            raise ValueError(f"dt_rank={s.dt_rank}: the inner width of the step size is positive")

    def cache_spec(self):
        s = self.spec
        return CacheSpec(state=StateSpec(parts=(
            ("matrix", (s.inner, s.n_state)),
            ("conv_tail", (max(1, s.conv_taps - 1), s.inner)),       # the convolution's last inputs, oldest first
        )))

    def tensor_decls(self):
        s, p = self.spec, self.spec.prefix
        return [
            TensorDecl(p + "in", (2 * s.inner, s.hidden)),
            TensorDecl(p + "conv", (s.inner, s.conv_taps)), TensorDecl(p + "conv.b", (s.inner,)),
            TensorDecl(p + "x", (s.dt_rank + 2 * s.n_state, s.inner)),
            TensorDecl(p + "dt", (s.inner, s.dt_rank)), TensorDecl(p + "dt.b", (s.inner,), mean=-3.0),
            TensorDecl(p + "A_log", (s.inner, s.n_state)), TensorDecl(p + "D", (s.inner,), mean=1.0),
            TensorDecl(p + "o", (s.hidden, s.inner)),
        ]

    def load(self, src, rt):
        super().load(src, rt)
        s, p = self.spec, self.spec.prefix
        f32 = torch.float32
        self.w_in = src.get(p + "in")
        self.conv_w, self.conv_b = src.get(p + "conv").to(f32).contiguous(), src.get(p + "conv.b").to(f32).contiguous()
        # rows of zeros keep the product's output rows a multiple of 32 bytes wide
        self.w_x = _pad_rows(src.get(p + "x"), 8).contiguous()
        w_dt = src.get(p + "dt")
        self.dt_pad = 0
        if rt.dtype == torch.bfloat16 and w_dt.dtype == torch.bfloat16:
            # the same matrix for both halves of the split rows, its columns padded to whole 16-byte pieces
            self.dt_pad = -(-s.dt_rank // 8) * 8
            half = torch.zeros(s.inner, self.dt_pad, dtype=w_dt.dtype, device=w_dt.device)
            half[:, :s.dt_rank] = w_dt
            w_dt = torch.cat([half, half], dim=1)
        self.w_dt = w_dt.contiguous()
        self.dt_b = src.get(p + "dt.b")
        self.a_log = src.get(p + "A_log").to(f32).contiguous()
        self.d_skip = src.get(p + "D").to(f32).contiguous()
        self.w_o = src.get(p + "o")

    def forward_add(self, x, h, batch, cache):
        self.forward_into(x, h, batch, cache, accumulate=True)

    def forward_into(self, x, out, batch, cache, accumulate=False):
        s, rt, st = self.spec, self.rt, batch.stream
        T, I, R = x.shape[0], s.inner, s.dt_rank
        f32 = torch.float32
        tail, state = cache.states["conv_tail"], cache.states["matrix"]
        xz = rt.empty(T, 2 * I)
        ops.linear(x, self.w_in, xz, status=batch.status, stream=st, after_short_kernel=True)
        single = batch.max_new == 1      # a decode step: the kernel that reads a channel's tail also moves it on
        xc = rt.empty(T, I)
        ops.input_conv(xz[:, :I], self.conv_w, s.conv_taps, tail, batch.token_seq, batch.seq_slot, xc, update_tail=single,
                       add_input=False, bias=self.conv_b, silu=True, stream=st)
        if not single and s.conv_taps > 1:
            ops.conv_tail_update(xz, I, s.conv_taps, tail, batch.token_seq, batch.seq_slot, batch.n_seqs, stream=st)
        low = rt.empty(T, self.w_x.shape[0], dtype=f32)              # [dt | B | C]
        ops.linear(xc, self.w_x, low, status=batch.status, stream=st)
        dt, dt_low, w_dt = None, low[:, :R], None
        if single and T <= STEP_IN_SCAN_MAX_TOKENS:
            dt, w_dt = dt_low, self.w_dt[:, :R]      # the recurrence's kernel works out its channels' step sizes itself
        else:
            dt = rt.empty(T, I, dtype=f32)
            if self.dt_pad:
                dt_low = ops.split_rows(dt_low, rt.empty(T, 2 * self.dt_pad, dtype=torch.bfloat16), stream=st)
            ops.linear(dt_low, self.w_dt, dt, status=batch.status, stream=st)
        y = rt.empty(T, I)
        ops.selective_scan(dt, self.dt_b, xc, xz[:, I:], low[:, R:R + 2 * s.n_state], self.a_log, self.d_skip, state, y,
                           batch.token_seq, batch.seq_slot, batch.n_seqs, stream=st, w_dt=w_dt)
        ops.linear(y, self.w_o, out, accumulate=accumulate, status=batch.status, stream=st)


register_part("selective_scan", SelectiveScan, replace=True)
