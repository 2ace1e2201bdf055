"""Grouped-query causal attention with 32-bit scores, softmax weights and weighted sums, and keys and values
of sizes of their own (the cache keeps rows of either size):

    q = Wq h [H, dk];  k = Wk h [G, dk];  v = Wv h [G, dv]     one product over the stacked matrix
    o_h = sum_j softmax_j(scale q_h.k_j + bias) v_j over j <= i,  head h reading key head h // (H / G)
    out = Wo o

Options, each a parameter:

* ``values_from_keys``: there is no v projection; a position's value is its key as projected, before norm and
  rotation (then dv = dk);
* ``qk_head_norm`` = {"eps": e}: every head of q and k over its own root mean square, times a weight of size dk
  shared by the heads (``q.norm``, ``k.norm``), before the rotation;
* ``rotation`` = {"dims", "base"}: the first ``dims`` features of every head of q and k turn in pairs
  (i, i + dims/2) by pos * base^(-2i/dims);
* ``q_temperature`` = {"coef", "every"}: q at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1);
* ``distance_bias`` = {"rows": B, "largest": D}: a stored table ``rel`` [B, H]; a key n positions back adds
  row bucket(n) of it to the scaled score (see ``distance_buckets``);
* ``sink``: a stored number per head whose exponential joins the denominator alone.

Keys are cached as the scores read them (normed, rotated); the table is laid out by distance, in 32 bits, when
the weights are bound.
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from ..cache import CacheNeed
from ..csrc import ops
from ..weights import TensorNeed
from .base import register_mixer
from .linear import matmul_partials
from .position import yarn_frequencies


def distance_buckets(rows: int, largest: float) -> List[int]:
    """The table's row for every distance from 0 to the first one from which on it is the last row for good:
    half of the rows are distances of their own, the others logarithmically wider up to ``largest``,
    bucket(n) = min(rows - 1, half + floor(ln(n / half) / ln(largest / half) (rows - half))).  A value within
    1e-9 of a whole number counts as that number: an edge is where it is, however the logarithms round."""
    half = rows // 2
    if rows < 2 or not largest > half:
        raise ValueError(f"a distance table of {rows} rows (at least 2) up to distance {largest} (more than {half})")
    out, n = [], 0
    while not out or out[-1] < rows - 1:
        if n < half:
            out.append(n)
        else:
            x = math.log(n / half) / math.log(largest / half) * (rows - half)
            step = round(x) if abs(x - round(x)) < 1e-9 else math.floor(x)
            out.append(min(rows - 1, half + step))
        n += 1
    return out


@register_mixer("exact_attention")
class ExactAttention:
    prefers_longest_first = True           # long blocks that start last leave the SMs idle at the end

    def __init__(self, params: dict, rt):
        self.rt = rt
        self.D = int(params["hidden_size"])
        self.H = int(params["num_heads"])
        self.G = int(params["num_kv_heads"])
        self.dk_true = int(params["head_dim"])
        self.dv_true = int(params.get("value_dim") or self.dk_true)
        self.scale = float(params.get("scale") or self.dk_true ** -0.5)
        self.values_from_keys = bool(params.get("values_from_keys", False))
        self.head_norm = params.get("qk_head_norm") or None
        self.temperature = params.get("q_temperature") or None
        self.bias = params.get("distance_bias") or None
        self.sink = bool(params.get("sink", False))
        rot = params.get("rotation") or {}
        self.dims, self.base = int(rot.get("dims", 0)), float(rot.get("base", 1.0))
        if self.H % self.G or min(self.H, self.G, self.dk_true, self.dv_true) <= 0:
            raise ValueError(f"{self.H} heads over {self.G} kv heads of sizes {self.dk_true} and {self.dv_true}")
        if self.values_from_keys and self.dv_true != self.dk_true:
            raise ValueError(f"values that are the keys have the keys' size {self.dk_true}, not {self.dv_true}")
        if self.dims % 2 or not 0 <= self.dims <= self.dk_true:
            raise ValueError(f"{self.dims} rotated features of a head of {self.dk_true}")
        # rows as the kernels take them: multiples of 8 (zero rows of the weights, zero columns of Wo)
        self.dk, self.dv = -(-self.dk_true // 8) * 8, -(-self.dv_true // 8) * 8
        if max(self.dk, self.dv) > 256:
            raise ValueError(f"head sizes {self.dk_true} and {self.dv_true}: up to 256 are supported")
        self.freq: Optional[torch.Tensor] = None
        if self.dims:
            self.freq = yarn_frequencies(self.dims, self.base, None)[0].to(rt.device)
        self.w_qkv = self.w_o = self.norms = self.table = self.sinks = None

    def tensor_needs(self):
        H, G, dk, dv, D = self.H, self.G, self.dk_true, self.dv_true, self.D
        needs = {"q": TensorNeed((H * dk, D)), "k": TensorNeed((G * dk, D)), "o": TensorNeed((D, H * dv))}
        if not self.values_from_keys:
            needs["v"] = TensorNeed((G * dv, D))
        if self.head_norm:
            needs["q.norm"], needs["k.norm"] = TensorNeed((dk,), init="ones"), TensorNeed((dk,), init="ones")
        if self.bias:
            needs["rel"] = TensorNeed((int(self.bias["rows"]), H), init="around_zero")
        if self.sink:
            needs["sink"] = TensorNeed((H,), init="around_zero")
        return needs

    @staticmethod
    def _pad(w: torch.Tensor, heads: int, size: int, to: int) -> torch.Tensor:
        """[heads * size, ...] -> [heads * to, ...] with zeros after each head's own rows."""
        if size == to:
            return w
        out = torch.zeros((heads, to) + tuple(w.shape[1:]), dtype=w.dtype, device=w.device)
        out[:, :size] = w.view((heads, size) + tuple(w.shape[1:]))
        return out.view((heads * to,) + tuple(w.shape[1:]))

    def bind(self, tensors) -> None:
        rt, H, G = self.rt, self.H, self.G
        parts = [self._pad(tensors["q"], H, self.dk_true, self.dk), self._pad(tensors["k"], G, self.dk_true, self.dk)]
        if not self.values_from_keys:
            parts.append(self._pad(tensors["v"], G, self.dv_true, self.dv))
        if any(p.dtype == torch.float32 for p in parts):
            parts = [p.to(torch.float32) for p in parts]
        self.w_qkv = rt.matrix(torch.cat(parts, 0))
        self.w_o = rt.matrix(self._pad(tensors["o"].t().contiguous(), H, self.dv_true, self.dv).t().contiguous())
        if self.head_norm:
            q, k = (self._pad(rt.vector(tensors[x]), 1, self.dk_true, self.dk).contiguous() for x in ("q.norm", "k.norm"))
            self.norms = (q, k, float(self.head_norm["eps"]), self.dk_true)
        if self.bias:
            row = distance_buckets(int(self.bias["rows"]), float(self.bias["largest"]))
            rel = rt.vector(tensors["rel"])
            self.table = rel[torch.tensor(row, dtype=torch.long, device=rel.device)].t().contiguous()      # [H, distances]
        if self.sink:
            self.sinks = rt.vector(tensors["sink"])

    def cache_need(self) -> CacheNeed:
        return CacheNeed("kv", kv_heads=self.G, head_dim=self.dk, value_dim=self.dv)

    def cache_read_bytes(self, contexts, element_size: int) -> int:
        return sum(contexts) * self.G * (self.dk + self.dv) * element_size

    def flops(self, q_lens, past) -> float:
        n = sum(q_lens)
        rows = self.H * self.dk + self.G * self.dk + (0 if self.values_from_keys else self.G * self.dv)
        pairs = sum(q * p + q * (q + 1) / 2 for q, p in zip(q_lens, past))
        return 2.0 * n * (rows * self.D + self.D * self.H * self.dv) + 2.0 * self.H * (self.dk + self.dv) * pairs

    def _angles(self, batch, slot_pos):
        """(cos, sin) of every token's angles, made once per step for the layers with these constants."""
        if not self.dims:
            return None
        key = "rope_table_partial_%d_%r" % (self.dims, self.base)
        table = batch.notes.get(key)
        if table is None:
            table = self.rt.buffer(key, (batch.n_tokens, self.dims // 2, 2), torch.float32)
            ops.rope_table(self.freq, batch, slot_pos, table)
            batch.notes[key] = table
        return table

    def splits(self, batch) -> int:
        """Blocks that share one query's keys in a decode step: as many as fill the device twice, and no
        fewer than 64 keys each."""
        bound = max(1, batch.ctx_bound)
        blocks = batch.n_tokens * self.G * -(-(self.H // self.G) // 8)
        return max(1, min(-(-bound // 64), 2 * self.rt.sm_count // blocks, 64))

    def forward(self, h, batch, stream, view, shared: bool = False):
        if shared:
            raise RuntimeError("exact_attention does not read another run entry's cache")
        rt, H, G, dk, dv = self.rt, self.H, self.G, self.dk, self.dv
        n = batch.n_tokens
        z, S = matmul_partials(rt, h, self.w_qkv, "qkv")
        q = rt.buffer("q_rot", (n, H * dk), rt.dtype)
        kv_step = rt.buffer("kv_step", (n, G * (dk + dv)), rt.dtype)
        temp = (float(self.temperature["coef"]), float(self.temperature["every"])) if self.temperature else None
        ops.head_store(z, S, self.norms, self._angles(batch, view.slot_pos), self.dims, temp, batch, view.slot_pos, q,
                       kv_step, view.k, view.v, H, G, dk, dv, not self.values_from_keys, view.capacity, pages=view.pages)
        o = rt.buffer("attn_out", (n, H * dv), rt.dtype)
        mma = rt.attention != "simt" and rt.dtype in ops.HALF_TYPES
        ns = self.splits(batch) if batch.is_decode else 1
        scratch = {}
        if ns > 1:
            scratch = {"part_o": rt.buffer("attn_part_o", (n, H, ns, dv), torch.float32),
                       "part_ml": rt.buffer("attn_part_ml", (n, H, ns, 2), torch.float32),
                       "counters": rt.zeros("attn_counters", n * G * -(-(H // G) // 4))}
        ops.attention_kv(q, kv_step, view.k, view.v, batch, view.slot_pos, o, H, G, dk, dv, view.capacity, self.scale,
                         rt.status, bias=self.table, sink=self.sinks, mma=mma, nsplit=ns,
                         max_keys=max(1, batch.ctx_bound) if batch.is_decode else 1 << 30, pages=view.pages, **scratch)
        stream.add_linear(o, self.w_o)
        return None
