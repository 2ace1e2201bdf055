"""Attention over a cached latent (multi-head latent attention).  A token's keys and values of
all heads are functions of one small row, which is all the cache keeps:

    [c' | kr] = Wdkv h;   c = c' / sqrt(mean(c'^2) + eps) * w_c  [rank];   kr rotated  [rot_dim]
    head i:   key = [Wuk_i c | kr],   value = Wuv_i c,   query = [qa_i | rot(qr_i)] = Wq h
    score = scale (qa_i . Wuk_i c + qr_i . kr),  softmax,  o_i = sum_j p_j Wuv_i c_j

and Wo on the concatenated heads.  Options, each a parameter:

* ``rot_base``, ``rot_layout``, ``rot_scaling``: the rotation turns pairs (2i, 2i+1) ("neighbours") or
  (i, i + rot_dim/2) ("halves") by position * f_i, f_i = base^(-2i/rot_dim), with YaRN scaling (see
  ``position.yarn_frequencies``) where given;
* ``gate``: "element" multiplies the concatenated heads feature by feature by sigmoid(Wg h), "head" head
  i's output by sigmoid(Wg h)_i, None not at all;
* ``window``: a query sees the last ``window`` positions (itself included); the cache then keeps a ring of
  as many rows;
* ``sink``: the softmax's denominator also contains exp(sink_i), a stored number per head;
* ``owns_latent`` False: the layer has no Wdkv and reads the rows that another run entry cached (and that
  entry's rows of this step).

Two forms of the same sums (see csrc/latent.cu).  Absorbed, for decode steps, portions of prompts and the
32-bit path: queries are moved into the latent space, the attention runs over the cached rows
themselves -- keys and values of every head at once (a cache need with ``values=False``) -- and the mixed
latent is expanded by Wuv after.  Expanded, for whole prompts in 16 bits: keys and values of the step
are one product [Wuk; Wuv] c, and the attention runs per head.  Scores, softmax weights and the weighted sum
are 32-bit in both; the rows, queries, expanded keys and values and the mixed latent of one block
per query are in the compute type.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..cache import CacheNeed
from ..csrc import ops
from ..weights import TensorNeed
from .base import register_mixer
from .linear import matmul_partials, matmul_store
from .position import yarn_frequencies

GATES = {None: ops.GATE_NONE, "head": ops.GATE_HEAD, "element": ops.GATE_ELEMENT}


@register_mixer("latent_attention")
class LatentAttention:
    def __init__(self, params: dict, rt):
        self.rt = rt
        self.D = int(params["hidden_size"])
        self.H = int(params["num_heads"])
        self.dim = int(params["head_dim"])            # unrotated query/key features per head
        self.rd = int(params["rot_dim"])              # rotated features, shared by the heads' keys
        self.vdim = int(params["value_dim"])
        self.rank = int(params["kv_rank"])
        self.scale = float(params["scale"])
        self.eps = float(params["eps"])
        self.window: Optional[int] = params.get("window") or None
        self.has_sink = bool(params.get("sink", False))
        self.owns_latent = bool(params.get("owns_latent", True))
        if params.get("gate", "element") not in GATES or params.get("rot_layout", "neighbours") not in ("neighbours", "halves"):
            raise ValueError("latent_attention: gate is None, 'head' or 'element', rot_layout 'neighbours' or 'halves'")
        self.gate = GATES[params.get("gate", "element")]
        self.halves = params.get("rot_layout", "neighbours") == "halves"
        if min(self.H, self.dim, self.vdim, self.rank) <= 0 or self.rd < 0 or self.rd % 2:
            raise ValueError("latent_attention: heads, sizes and rank must be positive, rot_dim even")
        self.hd = -(-(self.rank + self.rd) // 16) * 16          # a cached row, padded
        if self.rank > 1024 or self.hd > 2048 or self.dim + self.rd > 4096:
            raise ValueError(f"latent_attention: kv_rank={self.rank} (up to 1,024), rot_dim={self.rd} and head_dim="
                             f"{self.dim} exceed the kernels' sizes")
        freq, self.mult = torch.zeros(1), 1.0
        if self.rd:
            freq, self.mult = yarn_frequencies(self.rd, float(params["rot_base"]), params.get("rot_scaling") or None)
        self.freq = freq.to(rt.device)
        self.w_in = self.w_kv = self.c_norm = self.w_uk = self.w_uv = self.w_o = self.sink = None
        # the columns of the stacked input product [Wq; Wdkv; Wg]
        self.col_dkv = self.H * (self.dim + self.rd)
        self.col_gate = self.col_dkv + (self.rank + self.rd if self.owns_latent else 0)

    def tensor_needs(self):
        H, D = self.H, self.D
        needs = {"q": TensorNeed((H * (self.dim + self.rd), D)), "uk": TensorNeed((H * self.dim, self.rank)),
                 "uv": TensorNeed((H * self.vdim, self.rank)), "o": TensorNeed((D, H * self.vdim))}
        if self.owns_latent:
            needs["dkv"] = TensorNeed((self.rank + self.rd, D))
            needs["dkv.norm"] = TensorNeed((self.rank,), init="ones")
        if self.gate:
            needs["g"] = TensorNeed((H if self.gate == ops.GATE_HEAD else H * self.vdim, D))
        if self.has_sink:
            needs["sink"] = TensorNeed((H,), init="around_zero")
        return needs

    def bind(self, tensors) -> None:
        rt = self.rt
        parts = [tensors[k] for k in ("q", "dkv", "g") if k in tensors]
        if any(p.dtype == torch.float32 for p in parts):
            parts = [p.to(torch.float32) for p in parts]
        rows = sum(p.shape[0] for p in parts)
        if rows % 4:                                   # zero rows: the consumers' 16-byte loads
            parts.append(torch.zeros((4 - rows % 4, self.D), dtype=parts[0].dtype, device=parts[0].device))
        self.w_in = rt.matrix(torch.cat(parts, 0))
        self.w_o = rt.matrix(tensors["o"])
        # [H, dim, rank] as stored; the value expansion transposed to [H, rank, vdim]
        uk, uv = tensors["uk"], tensors["uv"]
        self.w_uk = rt.matrix(uk)
        self.w_uv = rt.matrix(uv.view(self.H, self.vdim, self.rank).transpose(1, 2).contiguous())
        if self._expands():
            # both expansions of a head after one another, for the product over a prompt's rows
            self.w_kv = rt.matrix(torch.cat([uk.to(rt.dtype).view(self.H, self.dim, self.rank),
                                             uv.to(rt.dtype).view(self.H, self.vdim, self.rank)], 1)
                                  .reshape(self.H * (self.dim + self.vdim), self.rank).contiguous())
        if self.owns_latent:
            self.c_norm = rt.vector(tensors["dkv.norm"])
        if self.has_sink:
            self.sink = rt.vector(tensors["sink"])

    def _expands(self) -> bool:
        rt = self.rt
        return (rt.attention != "simt" and rt.gemm != "simt" and self.w_uk.dtype == rt.dtype
                and ops.latent_prefill_usable(rt.dtype, self.dim, self.rd, self.vdim, self.rank, self.hd))

    def cache_need(self):
        return CacheNeed("kv", kv_heads=1, head_dim=self.hd, window=self.window, values=False) if self.owns_latent else None

    prefers_longest_first = True

    def cache_read_bytes(self, contexts, element_size: int) -> int:
        return sum(min(c, self.window) if self.window else c for c in contexts) * self.hd * element_size

    def flops(self, q_lens, past) -> float:
        n = sum(q_lens)
        H, D = self.H, self.D
        gate = {ops.GATE_NONE: 0, ops.GATE_HEAD: H, ops.GATE_ELEMENT: H * self.vdim}[self.gate]
        lin = 2.0 * n * (H * (self.dim + self.rd) * D + gate * D + H * self.vdim * D
                         + ((self.rank + self.rd) * D if self.owns_latent else 0)
                         + H * self.dim * self.rank + H * self.vdim * self.rank)
        pairs = 0
        for q, p in zip(q_lens, past):
            full = q * p + q * (q + 1) // 2
            if self.window:
                full = sum(min(pos + 1, self.window) for pos in range(p, p + q))
            pairs += full
        # whole prompts run per head on keys of dim + rot_dim, everything else on the rows
        per_pair = self.dim + self.rd + self.vdim if all(p == 0 for p in past) else 2 * self.rank + self.rd
        return lin + 2.0 * H * per_pair * pairs

    def decode_splits(self, batch, mma: bool):
        """(runs of keys per query, keys per run): runs as long as let the runs of all queries fill the SMs'
        block slots (two each), two tiles of 32 keys at least.  Runs are of one size, so that a batch's
        long sequences get more blocks than its short ones; lengths are counted as they will be when the
        longest reaches the step's bound (a captured decode step keeps its plan)."""
        if batch.n_tokens > ops.LATENT_FEW_TOKENS or not (mma or batch.is_decode):
            return 1, 0
        bound = max(1, batch.ctx_bound)
        slack = max(0, bound - max(p + q for p, q in zip(batch.past, batch.q_lens)))
        seen = lambda n: -(-(min(n, self.window) if self.window else n) // 32)
        total = sum(q * seen(p + q + slack) for p, q in zip(batch.past, batch.q_lens))
        groups = -(-self.H // (16 if mma else 4))
        most = seen(bound)
        per = max(2, -(-total * groups // (2 * self.rt.sm_count)), -(-most // ops.LATENT_MAX_SPLIT))
        return -(-most // per), per * 32

    def forward(self, h, batch, stream, view, shared: bool = False):
        rt, H, hd, rank = self.rt, self.H, self.hd, self.rank
        n = batch.n_tokens
        if shared != (not self.owns_latent):
            raise RuntimeError("latent_attention: a layer without a down projection reads another run's cache")
        z, S = matmul_partials(rt, h, self.w_in, "latent_in")
        rot = {"halves": self.halves, "mult": self.mult}
        whole = self.w_kv is not None and all(p == 0 for p in batch.past) and not batch.is_decode
        kept = getattr(view, "kv_step", None) is not None
        kv_step = view.kv_step if kept else rt.buffer("latent_step", (n, 2, 1, hd), rt.dtype)
        # several tokens on top of a ring that wraps in this step: their rows would replace rows that the
        # first of them still has to see, so the ring is written after the attention
        late_write = not shared and any(p > 0 and ql > 1 and p + ql > view.capacity
                                        for p, ql in zip(batch.past, batch.q_lens))
        c_rows = rt.buffer("latent_c", (n, rank), rt.dtype) if whole else None
        if not shared:
            ops.latent_store(z, S, self.c_norm, self.eps, self.freq, batch, view.slot_pos, kv_step, view.k, rank,
                             self.rd, hd, view.capacity, write_cache=not late_write, pages=view.pages,
                             col0=self.col_dkv, c_rows=c_rows, **rot)
        elif whole:
            c_rows.copy_(kv_step[:, 0, 0, :rank])
        o = rt.buffer("attn_out", (n, H * self.vdim), rt.dtype)
        gate = {"gate_col0": self.col_gate, "gate_mode": self.gate}
        if whole:
            q = rt.buffer("latent_q", (n, H * (self.dim + self.rd)), rt.dtype)
            ops.latent_rotate_q(z, S, self.freq, batch, view.slot_pos, q, H, self.dim, self.rd, **rot)
            kv = rt.buffer("latent_kv", (n, H * (self.dim + self.vdim)), rt.dtype)
            matmul_store(rt, c_rows, self.w_kv, kv)
            ops.latent_prefill(q, kv, kv_step, batch, o, H, self.dim, self.rd, self.vdim, rank, hd, self.window,
                               self.scale, sink=self.sink, gate=z, gate_n=S, **gate)
        else:
            q = rt.buffer("latent_q_abs", (n, H * hd), rt.dtype)
            ops.latent_absorb_q(z, S, self.w_uk, self.freq, batch, view.slot_pos, q, H, self.dim, self.rd, rank, hd, **rot)
            mma = rt.attention != "simt" and ops.latent_attention_mma_usable(rt.dtype, rank, hd)
            nsplit, per = self.decode_splits(batch, mma)
            o_lat = parts = None
            if nsplit > 1:
                parts = (rt.buffer("latent_part_o", (n, H, nsplit, rank), torch.float32),
                         rt.buffer("latent_part_ml", (n, H, nsplit, 2), torch.float32), nsplit)
            else:
                o_lat = rt.buffer("latent_mixed", (n, H * hd), rt.dtype)
            ops.latent_attention(q, kv_step, view.k, batch, view.slot_pos, o_lat, H, rank, hd, view.capacity,
                                 self.window, self.scale, sink=self.sink, pages=view.pages, parts=parts,
                                 mma=mma, per_split=per)
            ops.latent_expand(o_lat, self.w_uv, z if self.gate else None, S, o, H, rank, self.vdim, hd, parts=parts, **gate)
        stream.add_linear(o, self.w_o)
        if late_write:
            def write_ring():
                ops.cache_write(kv_step, batch, view.k, view.k, view.slot_pos, 1, hd, view.capacity, pages=view.pages)
            if kept:
                return write_ring                      # other run entries still read the old rows
            write_ring()
        return None
