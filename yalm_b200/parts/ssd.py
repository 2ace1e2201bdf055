"""Mamba-2: a state-space recurrence with one decay per head, H heads of value size P, state size N, B and
C shared by the heads of each of G groups (inner = H P):

    [z | x | B | C | dt] = Win h                                 inner, inner, G N, G N, H rows
    [x | B | C] = silu(conv([x | B | C]) + b)                    a short causal convolution over time
    dt = softplus(dt + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T  [N, P];   y = S^T C + D x
    out = Wo (n(y silu(z)) * w)                                  n: each of `norm_groups` equal parts of the
                                                                 row over its own root mean square

Two fixed-size cache needs per sequence: the state (float32 [H, P, N], rows of a column neighbours) and
the convolution's last taps - 1 inputs (float32).  Convolution, steps, decays, state and output norm
are 32-bit; the products are in the compute type.
"""
from __future__ import annotations

import torch

from ..cache import CacheNeed
from ..csrc import ops
from ..weights import TensorNeed
from .base import register_mixer
from .linear import matmul_partials


@register_mixer("mamba2")
class Mamba2:
    def __init__(self, params: dict, rt):
        self.rt = rt
        self.D = int(params["hidden_size"])
        self.H = int(params["num_heads"])
        self.P = int(params["head_dim"])
        self.N = int(params["state"])
        self.G = int(params.get("groups") or 1)
        self.taps = int(params["conv"])
        self.norm_groups = int(params.get("norm_groups") or 1)
        self.eps = float(params["eps"])
        if min(self.H, self.P, self.N, self.G, self.norm_groups) <= 0 or self.H % self.G \
                or (self.H * self.P) % self.norm_groups or self.N > 256 or not 2 <= self.taps <= 8:
            raise ValueError(f"mamba2: {self.H} heads of {self.P} in {self.G} groups, state {self.N} (up to 256), "
                             f"{self.taps} taps (2 to 8), {self.norm_groups} norm groups")
        self.inner = self.H * self.P
        self.channels = self.inner + 2 * self.G * self.N            # convolved: x | B | C
        self.rows = self.inner + self.channels + self.H
        self.w_in = self.w_o = self.conv_w = self.conv_b = None
        self.dt_bias = self.a_log = self.d_skip = self.norm = None

    def tensor_needs(self):
        H, D = self.H, self.D
        return {"in": TensorNeed((self.rows, D)), "conv": TensorNeed((self.channels, self.taps)),
                "conv.b": TensorNeed((self.channels,), init="around_zero"),
                "dt_bias": TensorNeed((H,), init="around_zero"), "A_log": TensorNeed((H,), init="around_zero"),
                "D": TensorNeed((H,), init="ones"), "norm": TensorNeed((self.inner,), init="ones"),
                "o": TensorNeed((D, self.inner))}

    def bind(self, tensors) -> None:
        rt = self.rt
        w = tensors["in"]
        if self.rows % 4:                              # zero rows: the consumers' 16-byte loads
            w = torch.cat([w, torch.zeros((4 - self.rows % 4, self.D), dtype=w.dtype, device=w.device)], 0)
        self.w_in = rt.matrix(w)
        self.w_o = rt.matrix(tensors["o"])
        self.conv_w, self.conv_b = rt.vector(tensors["conv"]), rt.vector(tensors["conv.b"])
        self.dt_bias, self.a_log = rt.vector(tensors["dt_bias"]), rt.vector(tensors["A_log"])
        self.d_skip, self.norm = rt.vector(tensors["D"]), rt.vector(tensors["norm"])

    def cache_need(self):
        return {"state": CacheNeed("state", state_shape=(self.H, self.P, self.N), state_dtype=torch.float32),
                "conv": CacheNeed("state", state_shape=(self.taps - 1, self.channels), state_dtype=torch.float32)}

    def cache_read_bytes(self, contexts, element_size: int) -> int:
        return 2 * len(contexts) * (self.inner * self.N + (self.taps - 1) * self.channels) * 4

    def flops(self, q_lens, past) -> float:
        n = sum(q_lens)
        return 2.0 * n * (self.rows * self.D + self.D * self.inner + self.taps * self.channels) \
            + 4.0 * n * self.inner * self.N

    def forward(self, h, batch, stream, view, shared: bool = False):
        if shared:
            raise RuntimeError("a recurrent state cannot be read by another run entry")
        rt, n = self.rt, batch.n_tokens
        z, S = matmul_partials(rt, h, self.w_in, "ssd_in")
        act = rt.buffer("ssd_act", (n, self.channels), torch.float32)
        ops.short_conv(z, S, self.inner, self.channels, self.conv_w, view["conv"].state, batch, out32=act,
                       out_bias=self.conv_b, silu=True)
        y = rt.buffer("ssd_y", (n, self.inner), torch.float32)
        ops.ssd_scan(act, z, S, self.inner + self.channels, self.dt_bias, self.a_log, self.d_skip, batch,
                     view["state"].state, y, self.H, self.G, self.P, self.N)
        out = rt.buffer("ssd_normed", (n, self.inner), rt.dtype)
        ops.gated_group_norm(y, z, S, 0, self.norm, out, self.norm_groups, self.eps)
        stream.add_linear(out, self.w_o)
        return None
