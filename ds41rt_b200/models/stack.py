"""Execution of layer-stack models (stack_config.StackConfig) with the hand-written sm_100a kernels.

`StackEngine` enqueues one pass over rows as a fixed sequence of launches: the residual step (csrc/kernels/stack_ops.cu)
closes a sublayer and opens the next one, the mixers (`MIXERS`) and the feed-forward part run between.  Everything that
depends on data stays on the device, so a decode pass is captured as a CUDA graph.  `dtype="bf16"` is the serving form
(matrix products and activations in bf16 with fp32 accumulation; streams, norms, gates, attention weights and recurrent
states in fp32); `dtype="f32"` keeps everything in true 32-bit.

`StackCache` holds what a request leaves behind: paged rows of the attention layers that produce them (a layer that reads
another layer's rows has none of its own) and one state per slot for recurrences and for the inputs of short convolutions.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from ..config import rope_inv_freq
from ..ops import lib
from ..ops import stack as S
from ..ops.stack import Matrix, Proj, ceil_to
from ..stack_config import GroupedAttentionSpec, LatentAttentionSpec, MLSTMSpec, MoESpec, StackConfig
from .base import RowsEngine
from .paged import PagedSlots

BF16, F32, I32 = torch.bfloat16, torch.float32, torch.int32
DTYPES = {"bf16": BF16, "f32": F32}


# ---------------------------------------------------------------------------------------------------- cache and states
@dataclass
class StackSnapshot:
    """State of one request after `n_tokens` positions.  Full pages are shared by reference (they are never written
    again); the rows of the partly filled last page and the recurrent states are copied."""
    n_tokens: int
    pages: List[int]
    partial: Dict[int, torch.Tensor]
    states: Dict[int, Tuple[torch.Tensor, ...]]

    def nbytes(self) -> int:
        ts = list(self.partial.values()) + [t for st in self.states.values() for t in st]
        return sum(t.numel() * t.element_size() for t in ts)


def latent_row_len(m: LatentAttentionSpec) -> Tuple[int, int]:
    """(padded latent width, cache row length): [latent | rotated key part], both padded to 16 values."""
    kv = ceil_to(m.kv_rank, 16)
    return kv, kv + ceil_to(m.rot_dim, 16)


def grouped_widths(m: GroupedAttentionSpec) -> Tuple[int, int, int]:
    """(query columns, key columns, value columns) of all heads, every head padded to 16 values."""
    d, v = ceil_to(m.dim, 16), ceil_to(m.vdim, 16)
    return m.heads * d, m.kv_heads * d, m.kv_heads * v


def cache_row_len(m) -> int:
    """Values of one token's cache row."""
    return latent_row_len(m)[1] if m.kind == "latent_attention" else sum(grouped_widths(m)[1:])


def state_shapes(m) -> Tuple[Tuple[int, ...], ...]:
    """fp32 state of one request: the recurrence's, or the convolution's last inputs (a ring over positions)."""
    if m.kind == "grouped_attention":
        return ((m.taps - 1, sum(grouped_widths(m))),)
    d, v = ceil_to(m.dim, 16), ceil_to(m.vdim, 16)
    nb = -(-v // S.STATE_COLS)
    return (m.heads, d, v), (m.heads, nb, d), (m.heads, nb)


class StackCache(PagedSlots):
    def __init__(self, cfg: StackConfig, slots: int, max_ctx: int, device, dtype=BF16, page_tokens: int = 64,
                 n_pages: Optional[int] = None):
        self.cfg, self.dtype = cfg, dtype
        self._init_pages(slots, max_ctx, device, page_tokens, n_pages)
        self.pools: Dict[int, torch.Tensor] = {}
        for l in cfg.cache_layers():
            row = cache_row_len(cfg.layers[l].mixer)
            self.pools[l] = torch.zeros(self.n_pages * page_tokens, row, dtype=dtype, device=device)
        self.states: Dict[int, Tuple[torch.Tensor, ...]] = {
            l: tuple(torch.zeros(slots, *shape, dtype=F32, device=device)
                     for shape in state_shapes(cfg.layers[l].mixer)) for l in cfg.state_layers()}

    def snapshot(self, slot: int, n_tokens: int) -> StackSnapshot:
        """Capture `slot`, whose last pass ended at position n_tokens - 1 (call it between passes, on the stream)."""
        P = self.page_tokens
        full, rem = n_tokens // P, n_tokens % P
        mine = self.alloc.pages(slot)
        pages = self.alloc.retain(slot, self._gen(slot), min(full, len(mine)))
        partial = {}
        if rem and full < len(mine):
            at = mine[full] * P
            partial = {l: t[at:at + rem].clone() for l, t in self.pools.items()}
        return StackSnapshot(n_tokens, pages, partial,
                             {l: tuple(t[slot].clone() for t in st) for l, st in self.states.items()})

    def restore(self, slot: int, snap: StackSnapshot) -> bool:
        """Continue a snapshot in an empty `slot`.  Returns False when no page is free for the partly filled page."""
        gen = self._gen(slot)
        assert self.alloc.page_count(slot) == 0, "restore needs an empty slot"
        if snap.partial and self.alloc.free_pages == 0:
            return False
        self.alloc.share(slot, gen, snap.pages)
        if snap.partial:
            self.alloc.ensure(slot, gen, (len(snap.pages) + 1) * self.page_tokens)
            at = self.alloc.pages(slot)[len(snap.pages)] * self.page_tokens
            for l, t in snap.partial.items():
                self.pools[l][at:at + t.shape[0]].copy_(t)
        self._publish(slot)
        for l, st in snap.states.items():
            for mine, kept in zip(self.states[l], st):
                mine[slot].copy_(kept)
        return True

    def restore_prefix(self, slot: int, snap: StackSnapshot, n_tokens: int) -> bool:
        """Only a snapshot's whole length can be continued where recurrent states belong to it."""
        return n_tokens == snap.n_tokens and self.restore(slot, snap)

    def nbytes(self) -> int:
        ts = list(self.pools.values()) + [t for st in self.states.values() for t in st]
        return sum(t.numel() * t.element_size() for t in ts)


# ---------------------------------------------------------------------------------------------------- mixers
class LatentAttention:
    """Weights of a latent-attention layer in kernel layout and its launch sequence.

    Head widths are padded to 16 values.  Two forms of the same attention: `absorbed` multiplies the queries by W_uk and
    attends over the latent rows themselves (decode, short portions, mixed passes); `expanded` makes keys and values of
    every visible position of one request first (long prompt passes)."""

    def __init__(self, spec: LatentAttentionSpec, cfg: StackConfig, t: Dict[str, torch.Tensor], gate: Dict[str, torch.Tensor],
                 device, dtype):
        self.spec, self.cfg = spec, cfg
        H, W = spec.heads, cfg.hidden
        self.dp, self.rp, self.vp = ceil_to(spec.dim, 16), ceil_to(spec.rot_dim, 16), ceil_to(spec.vdim, 16)
        self.kvp, self.row_len = latent_row_len(spec)
        self.hs = self.dp + self.rp
        own = spec.kv_from is None
        parts = [("dq", t["dq"])]
        if own:
            parts += [("kv", t["dkv"][:spec.kv_rank]), ("kr", t["dkv"][spec.kv_rank:])]
        parts += [("g", S.pad_heads(t["g"], H, spec.vdim, self.vp))]
        if gate:
            parts += [("gate", gate["w"])]
        self.w_in, self.at = S.stack_rows(parts, device, dtype)
        f32 = lambda x: x.to(device=device, dtype=F32).contiguous()
        self.dq_norm, self.sink = f32(t["dq.norm"]), f32(t["sink"])
        self.kv_norm = f32(t["dkv.norm"]) if own else None
        uq = t["uq"].view(H, spec.dim + spec.rot_dim, spec.q_rank)
        self.w_uq = Matrix(torch.cat([S.pad_heads(uq[:, :spec.dim].reshape(-1, spec.q_rank), H, spec.dim, self.dp)
                                      .view(H, self.dp, -1),
                                      S.pad_heads(uq[:, spec.dim:].reshape(-1, spec.q_rank), H, spec.rot_dim, self.rp)
                                      .view(H, self.rp, -1)], 1).reshape(H * self.hs, spec.q_rank), device, dtype)
        uk = S.pad_heads(t["uk"], H, spec.dim, self.dp)              # [H * dp, kv_rank]
        uv = S.pad_heads(t["uv"], H, spec.vdim, self.vp)
        z = lambda *shape: torch.zeros(*shape, dtype=dtype, device=device)
        self.w_ukt = z(H, self.kvp, self.dp)                         # per head: latent value <- query value
        self.w_ukt[:, :spec.kv_rank] = uk.view(H, self.dp, spec.kv_rank).transpose(1, 2).to(device=device, dtype=dtype)
        ukv = z(H * (self.dp + self.vp), self.kvp)                   # keys of all heads, then values of all heads
        ukv[:, :spec.kv_rank] = torch.cat([uk, uv], 0).to(device=device, dtype=dtype)
        self.w_ukv = Matrix(ukv, device, dtype)
        self.w_uv = self.w_ukv.w[H * self.dp:]
        self.w_o = Matrix(S.pad_heads(t["o"].t().contiguous(), H, spec.vdim, self.vp).t(), device, dtype)
        freq = rope_inv_freq(spec.rope, spec.rot_dim) if spec.rope is not None else [0.0] * (spec.rot_dim // 2)
        self.freq = torch.tensor(freq or [0.0], dtype=F32, device=device)

        # the expanded form keeps two query tiles, a key tile and a value tile of 128 rows in shared memory
        chunks = -(-self.dp // 64) + -(-self.rp // 64)
        self.expandable = dtype == BF16 and self.vp <= 128 and 3 * chunks + -(-self.vp // 64) <= 14

    def matrices(self):
        return {"a": [(self.w_in.n, self.w_in.k)], "b": [(self.w_uq.n, self.w_uq.k), (self.w_o.n, self.w_o.k)]}

    def run(self, e: "StackEngine", l: int, R: int, src: int) -> Tuple[Proj, Optional[Proj]]:
        sp, k, H = self.spec, e.k, self.spec.heads
        long = e.long_keys if self.expandable else 0
        pin = e.project_wide("gemm_mix_in", R, self.w_in) if long else \
            e.project("gemm_mix_in", e.h, e.ldh, R, self.w_in, e.planes_a)
        pool = e.cache.pools[src]
        a = S.LatentPostArgs()
        a.dq, a.dq_norm = pin.at(self.at["dq"]).args(), self.dq_norm.data_ptr()
        a.cq, a.ld_cq, a.q_rank = e.cq.data_ptr(), e.cq.shape[1], sp.q_rank
        if sp.kv_from is None:
            a.kv, a.kr, a.kv_norm = pin.at(self.at["kv"]).args(), pin.at(self.at["kr"]).args(), self.kv_norm.data_ptr()
            a.pool, a.freq, a.magnitude = pool.data_ptr(), self.freq.data_ptr(), sp.magnitude
        a.page_table, a.row_pos, a.row_slot = e.cache.page_table.data_ptr(), e.row_pos.data_ptr(), e.row_slot.data_ptr()
        a.eps, a.rows, a.kv_rank, a.kv_pad, a.rot_dim = self.cfg.norm_eps, R, sp.kv_rank, self.kvp, sp.rot_dim
        a.row_len, a.max_pages, a.page_tokens, a.f32 = self.row_len, e.cache.max_pages, e.cache.page_tokens, e.f32
        e._run("latent_post", k.ds41_latent_post, C.byref(a), lib.stream())
        ldq = H * self.hs
        if long:
            q = Proj(e.q, ldq)
            e._run("gemm_uq", S.project_bf16, e.cq, e.cq.shape[1], R, self.w_uq, e.q, ldq, e.status)
        else:
            q = e.project("gemm_uq", e.cq, e.cq.shape[1], R, self.w_uq, e.planes_b)
        e._run("latent_query", k.ds41_latent_query, C.byref(q.args()), lib.ptr(e.row_pos), lib.ptr(self.freq),
               C.c_float(sp.magnitude), R, H, self.dp, self.rp, sp.rot_dim, lib.ptr(e.q), ldq, e.f32, lib.stream())
        if long:
            self._expanded(e, R, ldq, pool, src, pin.at(self.at["g"]))
        else:
            self._absorbed(e, R, ldq, pool, pin.at(self.at["g"]))
        y = e.project("gemm_o", e.act, H * self.vp, R, self.w_o, e.planes_b)
        return y, (pin.at(self.at["gate"]) if "gate" in self.at else None)

    def _expanded(self, e: "StackEngine", R: int, ldq: int, pool, src: int, gate: Proj):
        sp, k, H, n = self.spec, e.k, self.spec.heads, e.long_keys
        lat, rot, kv = e.key_space(n, self.kvp, self.rp, self.w_ukv.n)
        if e.gathered != (src, n):           # a layer that reads the same rows finds them in place
            e._run("latent_gather", k.ds41_latent_gather, lib.ptr(pool), lib.ptr(e.cache.page_table), e.cache.max_pages,
                   e.cache.page_tokens, self.row_len, self.kvp, 0, lib.ptr(e.row_slot), n, lib.ptr(lat), lib.ptr(rot), 0,
                   lib.stream())
            e.gathered = (src, n)
        ldkv = self.w_ukv.n
        e._run("expand_kv", S.project_bf16, lat, self.kvp, n, self.w_ukv, kv, ldkv, e.status)
        a = S.LatentPrefillArgs()
        a.q, a.kv, a.rot, a.sink, a.out = (x.data_ptr() for x in (e.q, kv, rot, self.sink, e.act))
        a.status, a.gate, a.ld_q, a.ld_kv, a.scale = e.status.data_ptr(), gate.args(), ldq, ldkv, sp.scale
        a.rows, a.heads, a.dim_pad, a.rot_pad, a.vdim_pad = R, H, self.dp, self.rp, self.vp
        a.n_keys, a.pos0, a.ld_out = n, n - R, H * self.vp
        e._run("latent_prefill", k.ds41_latent_prefill, C.byref(a), lib.stream())

    def _absorbed(self, e: "StackEngine", R: int, ldq: int, pool, gate: Proj):
        sp, k, H = self.spec, e.k, self.spec.heads
        q = e.q.view(-1)
        for r0 in range(0, R, e.attn_rows):
            n = min(e.attn_rows, R - r0)
            qr = q[r0 * ldq:]
            e._run("absorb_q", S.per_head, qr, ldq, self.hs, n, H, self.w_ukt, self.kvp, self.dp, self.dp, e.q_abs,
                   H * self.kvp, e.status)
            splits = e.attn_splits(n, H)
            a = S.LatentAttendArgs()
            a.q_abs, a.ld_q_abs = e.q_abs.data_ptr(), H * self.kvp
            a.q_rot, a.ld_q_rot, a.q_rot_stride = qr[self.dp:].data_ptr(), ldq, self.hs
            a.pool, a.page_table = pool.data_ptr(), e.cache.page_table.data_ptr()
            a.row_pos, a.row_slot = e.row_pos[r0:].data_ptr(), e.row_slot[r0:].data_ptr()
            a.part_o, a.part_ml = e.part_o.data_ptr(), e.part_ml.data_ptr()
            a.scale, a.rows, a.heads, a.kv_pad, a.row_len, a.n_splits = sp.scale, n, H, self.kvp, self.row_len, splits
            a.max_pages, a.page_tokens, a.f32 = e.cache.max_pages, e.cache.page_tokens, e.f32
            e._run("latent_attend", k.ds41_latent_attend, C.byref(a), lib.stream())
            e._run("latent_merge", k.ds41_latent_merge, lib.ptr(e.part_o), lib.ptr(e.part_ml), lib.ptr(self.sink), splits, n,
                   H, self.kvp, lib.ptr(e.o_lat), H * self.kvp, e.f32, lib.stream())
            o = e.o_heads.view(-1)[r0 * H * self.vp:]
            e._run("values", S.per_head, e.o_lat, H * self.kvp, self.kvp, n, H, self.w_uv, self.vp, self.kvp, self.kvp, o,
                   H * self.vp, e.status)
        y = Proj(e.o_heads, H * self.vp)
        e._run("gate_mul", k.ds41_gate_mul, C.byref(y.args()), C.byref(gate.args()), R, H * self.vp, lib.ptr(e.act),
               H * self.vp, e.f32, lib.stream())


class MLSTM:
    def __init__(self, spec: MLSTMSpec, cfg: StackConfig, t: Dict[str, torch.Tensor], gate: Dict[str, torch.Tensor],
                 device, dtype):
        self.spec, self.cfg = spec, cfg
        H = spec.heads
        self.dp, self.vp = ceil_to(spec.dim, 16), ceil_to(spec.vdim, 16)
        parts = [("q", S.pad_heads(t["q"], H, spec.dim, self.dp)), ("k", S.pad_heads(t["k"], H, spec.dim, self.dp)),
                 ("v", S.pad_heads(t["v"], H, spec.vdim, self.vp)), ("g", S.pad_heads(t["g"], H, spec.vdim, self.vp))]
        if gate:
            parts += [("gate", gate["w"])]
        self.w_in, self.at = S.stack_rows(parts + [("i", t["i"]), ("f", t["f"])], device, dtype)
        # long passes take the log gates in fp32 from a product of their own and everything else in bf16
        self.w_main = self.w_in.rows(0, self.at["i"])
        self.w_gates = self.w_in.rows(self.at["i"], self.w_in.n)
        self.chunked = dtype == BF16 and self.dp <= 512
        f32 = lambda x: x.to(device=device, dtype=F32).contiguous()
        self.bias_i, self.bias_f = f32(t["i.b"]), f32(t["f.b"])
        self.norm = f32(S.pad_heads(t["norm"], H, spec.vdim, self.vp))
        self.w_o = Matrix(S.pad_heads(t["o"].t().contiguous(), H, spec.vdim, self.vp).t(), device, dtype)

    def matrices(self):
        return {"a": [(self.w_in.n, self.w_in.k)], "b": [(self.w_o.n, self.w_o.k)]}

    def run(self, e: "StackEngine", l: int, R: int, src: Optional[int]) -> Tuple[Proj, Optional[Proj]]:
        sp, k, H = self.spec, e.k, self.spec.heads
        long = e.long_keys > 0 and self.chunked
        if long:
            pin = e.project_wide("gemm_mix_in", R, self.w_main)
            log_gates: List[Proj] = []
            e._run("gemm_gates", lambda: log_gates.append(S.project_few(e.h, e.ldh, R, self.w_gates, e.planes_a, e.status)))
            gates = (log_gates[0] if log_gates else Proj(e.planes_a, self.w_gates.out_ld)).at(-self.at["i"])
        else:
            pin = gates = e.project("gemm_mix_in", e.h, e.ldh, R, self.w_in, e.planes_a)
        ld = H * self.vp
        s, n, m = e.cache.states[l]
        a = S.MlstmArgs()
        a.q, a.k, a.v = (pin.at(self.at[x]).args() for x in "qkv")
        a.gate_i, a.gate_f = gates.at(self.at["i"]).args(), gates.at(self.at["f"]).args()
        a.bias_i, a.bias_f = self.bias_i.data_ptr(), self.bias_f.data_ptr()
        a.row_pos, a.row_slot = e.row_pos.data_ptr(), e.row_slot.data_ptr()
        a.state_s, a.state_n, a.state_m, a.out = s.data_ptr(), n.data_ptr(), m.data_ptr(), e.o_heads.data_ptr()
        a.gate_cap, a.q_scale, a.den_eps = sp.gate_cap, sp.dim ** -0.5, sp.den_eps
        a.rows, a.heads, a.dim_pad, a.vdim_pad, a.slots, a.ld_out = R, H, self.dp, self.vp, e.cache.slots, ld
        a.work = e.recurrence_work.data_ptr()
        if long:
            e._run("mlstm_chunk", k.ds41_mlstm_chunk, C.byref(a), lib.stream())
        else:
            e._run("mlstm_step", k.ds41_mlstm_step, C.byref(a), lib.stream())
        e._run("head_norm_gate", k.ds41_head_norm_gate, lib.ptr(e.o_heads), ld, C.byref(pin.at(self.at["g"]).args()),
               lib.ptr(self.norm), R, H, sp.vdim, self.vp, C.c_float(self.cfg.norm_eps), lib.ptr(e.act), ld, e.f32,
               lib.stream())
        y = e.project("gemm_o", e.act, ld, R, self.w_o, e.planes_b)
        return y, (pin.at(self.at["gate"]) if "gate" in self.at else None)


class GroupedAttention:
    """Grouped-query attention over cached keys and values, head widths padded to 16 values: projection, then convolution,
    norm, rotation and cache rows in one launch, then attention with the head gates.  Long prompt passes of one request
    take the tcgen05 form, everything else a CTA (or a cluster of them) per row and key/value head."""

    def __init__(self, spec: GroupedAttentionSpec, cfg: StackConfig, t: Dict[str, torch.Tensor], gate: Dict[str, torch.Tensor],
                 device, dtype):
        self.spec, self.cfg = spec, cfg
        H, G = spec.heads, spec.kv_heads
        self.dp, self.vp = ceil_to(spec.dim, 16), ceil_to(spec.vdim, 16)
        self.cols = sum(grouped_widths(spec))

        def heads(name, suffix=""):
            n, w, p = {"q": (H, spec.dim, self.dp), "k": (G, spec.dim, self.dp), "v": (G, spec.vdim, self.vp)}[name]
            return S.pad_heads(t[name + suffix], n, w, p)

        f32 = lambda x: x.to(device=device, dtype=F32).contiguous()
        parts = [("u", torch.cat([heads(n) for n in "qkv"], 0))]
        if spec.head_gate:
            parts += [("g", t["g"])]
        if gate:
            parts += [("gate", gate["w"])]
        self.w_in, self.at = S.stack_rows(parts, device, dtype)
        self.conv = f32(torch.cat([heads(n, ".conv") for n in "qkv"], 0).t()) if spec.taps else None
        self.q_norm, self.k_norm = (f32(heads(n, ".norm")) if spec.qk_norm else None for n in "qk")
        self.freq = torch.tensor(rope_inv_freq(spec.rope, spec.rot_dim) or [0.0], dtype=F32, device=device) \
            if spec.rot_dim else None
        self.w_o = Matrix(S.pad_heads(t["o"].t().contiguous(), H, spec.vdim, self.vp).t(), device, dtype)
        # the tcgen05 form keeps two query tiles, a key tile and a value tile of 128 rows in shared memory
        self.tiled = dtype == BF16 and self.vp <= 128 and 3 * -(-self.dp // 64) + -(-self.vp // 64) <= 14

    def matrices(self):
        return {"a": [(self.w_in.n, self.w_in.k)], "b": [(self.w_o.n, self.w_o.k)]}

    def splits(self, e: "StackEngine", rows: int) -> int:
        """CTAs that share a row's keys: enough to fill the GPU, static per batch size (a captured pass replays while the
        context grows)."""
        sp = self.spec
        span = min(sp.chunk or e.cache.max_ctx, e.cache.max_ctx)
        blocks = rows * sp.kv_heads * -(-(sp.heads // sp.kv_heads) // 16)
        n = max(1, min(148 // blocks, 16, -(-span // 128)))
        return n if n <= 8 else (16 if n == 16 and blocks <= 4 else 8)        # larger clusters than 8 do not fill the GPU

    def run(self, e: "StackEngine", l: int, R: int, src: int) -> Tuple[Proj, Optional[Proj]]:
        sp, k, c = self.spec, e.k, e.cache
        long = e.long_keys if self.tiled and c.page_tokens in (32, 64, 128) else 0
        pin = e.project_wide("gemm_mix_in", R, self.w_in) if long else \
            e.project("gemm_mix_in", e.h, e.ldh, R, self.w_in, e.planes_a)
        u = pin.at(self.at["u"])
        state = c.states[l][0] if sp.taps > 1 else None
        ldq, ldo = sp.heads * self.dp, sp.heads * self.vp
        a = S.AttnPostArgs()
        a.u, a.conv, a.q_norm, a.k_norm, a.freq = u.args(), lib.ptr(self.conv), lib.ptr(self.q_norm), lib.ptr(self.k_norm), \
            lib.ptr(self.freq)
        a.state, a.q, a.pool, a.ld_q, a.eps = lib.ptr(state), lib.ptr(e.q), lib.ptr(c.pools[src]), ldq, self.cfg.norm_eps
        a.page_table, a.row_pos, a.row_slot = lib.ptr(c.page_table), lib.ptr(e.row_pos), lib.ptr(e.row_slot)
        a.rows, a.heads, a.kv_heads, a.dim, a.dim_pad, a.vdim_pad = R, sp.heads, sp.kv_heads, sp.dim, self.dp, self.vp
        a.rot_dim, a.taps, a.slots, a.max_pages, a.page_tokens, a.f32 = sp.rot_dim, max(sp.taps, 1), c.slots, c.max_pages, \
            c.page_tokens, e.f32
        e._run("attn_post", k.ds41_attn_post, C.byref(a), lib.stream())
        b = S.GroupAttendArgs()
        b.q, b.pool, b.out, b.status = lib.ptr(e.q), lib.ptr(c.pools[src]), lib.ptr(e.act), lib.ptr(e.status)
        b.page_table, b.row_pos, b.row_slot = a.page_table, a.row_pos, a.row_slot
        b.gate = pin.at(self.at["g"]).args() if sp.head_gate else S.NO_PROJ
        b.u, b.state, b.ld_q, b.scale = u.args(), lib.ptr(state), ldq, sp.scale
        b.rows, b.heads, b.kv_heads, b.dim_pad, b.vdim_pad, b.chunk = R, sp.heads, sp.kv_heads, self.dp, self.vp, sp.chunk
        b.taps, b.slots, b.ld_out, b.max_pages, b.page_tokens, b.f32 = a.taps, c.slots, ldo, c.max_pages, c.page_tokens, e.f32
        b.n_pages = c.n_pages
        if long:
            b.pos0, b.n_splits = long - R, 1
            e._run("group_prefill", k.ds41_group_prefill, C.byref(b), lib.stream())
        else:
            b.n_splits = self.splits(e, R)
            e._run("group_attend", k.ds41_group_attend, C.byref(b), lib.stream())
        y = e.project("gemm_o", e.act, ldo, R, self.w_o, e.planes_b)
        return y, (pin.at(self.at["gate"]) if "gate" in self.at else None)


MIXERS = {"latent_attention": LatentAttention, "grouped_attention": GroupedAttention, "mlstm": MLSTM}


class DenseMLP:
    def __init__(self, spec, cfg: StackConfig, t: Dict[str, torch.Tensor], gate: Dict[str, torch.Tensor], device, dtype):
        assert spec.activation == "polynorm"
        self.spec, self.cfg = spec, cfg
        self.ffp = ceil_to(spec.ff, 8)
        parts = [("up", t["up"])] + ([("gate", gate["w"])] if gate else [])
        self.w_up, self.at = S.stack_rows(parts, device, dtype)
        self.coef = t["act"].to(device=device, dtype=F32).contiguous()
        self.w_down = Matrix(t["down"], device, dtype)

    def matrices(self):
        return {"a": [(self.w_up.n, self.w_up.k)], "b": [(self.w_down.n, self.w_down.k)]}

    def run(self, e: "StackEngine", R: int) -> Tuple[Proj, Optional[Proj]]:
        pin = e.project_wide("gemm_up", R, self.w_up) if e.long_keys else \
            e.project("gemm_up", e.h, e.ldh, R, self.w_up, e.planes_a)
        e._run("polynorm", e.k.ds41_polynorm, C.byref(pin.at(self.at["up"]).args()), lib.ptr(self.coef), R, self.spec.ff,
               C.c_float(self.cfg.norm_eps), lib.ptr(e.act), self.ffp, e.f32, lib.stream())
        y = e.project("gemm_down", e.act, self.ffp, R, self.w_down, e.planes_b)
        return y, (pin.at(self.at["gate"]) if "gate" in self.at else None)


class RoutedExperts:
    """Mixture of experts.  Passes of up to `moe_rows` rows run every used expert over all rows, planned by the router's
    launch; longer ones sort the rows by expert (parallel/ep.py).  Either way the routes' results are summed by the residual
    step that follows.  32-bit passes always take the first form."""

    def __init__(self, spec: MoESpec, cfg: StackConfig, t: Dict[str, torch.Tensor], gate: Dict[str, torch.Tensor],
                 device, dtype):
        self.spec, self.cfg = spec, cfg
        E, W, ff = spec.experts, cfg.hidden, spec.ff
        self.ld, self.ffp = ceil_to(W, 8), ceil_to(ff, 8)
        self.w_router, self.at = S.stack_rows([("router", t["router"])] + ([("gate", gate["w"])] if gate else []), device, dtype)
        self.bias = t["router.b"].to(device=device, dtype=F32).contiguous() if "router.b" in t else None
        z = lambda *shape: torch.zeros(*shape, dtype=dtype, device=device)
        self.w13, self.w2 = z(E, 2 * self.ffp, self.ld), z(E, self.ld, self.ffp)
        for e in range(E):
            self.w13[e, :ff, :W] = t[f"e{e}.gate"].to(device=device, dtype=dtype)
            self.w13[e, self.ffp:self.ffp + ff, :W] = t[f"e{e}.up"].to(device=device, dtype=dtype)
            self.w2[e, :W, :ff] = t[f"e{e}.down"].to(device=device, dtype=dtype)

    def matrices(self):
        return {"a": [(self.w_router.n, self.w_router.k)]}

    def run(self, e: "StackEngine", R: int) -> Tuple[Proj, Optional[Proj]]:
        sp, k, E, top = self.spec, e.k, self.spec.experts, self.spec.top
        z = e.project("gemm_router", e.h, e.ldh, R, self.w_router, e.planes_a, few=True)
        planned = R <= e.moe_rows
        a = S.RouteArgs()
        a.z, a.bias, a.row_slot = z.at(self.at["router"]).args(), lib.ptr(self.bias), lib.ptr(e.row_slot)
        a.ids, a.weights, a.rows, a.experts, a.top = lib.ptr(e.ids), lib.ptr(e.route_w), R, E, top
        if planned:
            a.active, a.n_active, a.row_w, a.slot_of, a.ticket = (lib.ptr(x) for x in (e.active, e.n_active, e.row_w, e.slot_of,
                                                                                      e.ticket))
            a.max_active, a.row_w_ld = e.max_active(sp), e.moe_rows
        e._run("route", k.ds41_route_softmax, C.byref(a), lib.stream())
        gate = z.at(self.at["gate"]) if "gate" in self.at else None
        if not planned:
            ep = e.exchange(self)
            if e.only is None or "ep_moe" in e.only:
                e.launches += 4
            ids, wt = e.ids[:R * top].view(R, top), e.route_w[:R * top].view(R, top)
            e._run("ep_moe", ep.forward, e.h[:R], ids, wt, None)
            return S.RoutedProj(ep.comb, self.ld, route=e.ids, top=top), gate
        I, n = self.ffp, e.max_active(sp)
        if e.f32:
            some = dict(batch=n, batch_map=e.active, n_active=e.n_active)
            e._run("gemm_fc1", S.gemm_f32, e.h, self.w13, e.moe_up, R, 2 * I, self.ld, e.ldh, self.ld, 2 * I,
                   sb=2 * I * self.ld, so=R * 2 * I, **some)
            e._run("gated_act", k.ds41_gated_act, lib.ptr(e.moe_up), 2 * I, I, lib.ptr(e.row_w), e.moe_rows,
                   lib.ptr(e.n_active), n, R, I, C.c_float(sp.limit), C.c_float(sp.alpha), C.c_float(sp.shift),
                   lib.ptr(e.moe_act), I, lib.stream())
            e._run("gemm_fc2", S.gemm_f32, e.moe_act, self.w2, e.moe_out, R, self.ld, I, I, I, self.ld, sa=R * I,
                   sb=self.ld * I, so=R * self.ld, **some)
        else:
            act = dict(act_limit=sp.limit, act_alpha=sp.alpha, act_shift=sp.shift)
            many = dict(batch=n, a_batches=E, batch_map=e.active, n_active=e.n_active, row_w=e.row_w, row_w_ld=e.moe_rows,
                        bn=S.G.pick_bn(R), status=e.status)
            e._run("gemm_fc1", S.G.gemm_raw, self.w13, e.h, e.moe_act, I, R, self.ld, lda=self.ld, ldb=e.ldh, ldo=I, out_mode=4,
                   a_batch_stride=2 * I * self.ld, out_batch_stride=R * I, b_batch_kind=1, up_row_offset=I, **act, **many)
            e._run("gemm_fc2", S.G.gemm_raw, self.w2, e.moe_act, e.moe_out, self.ld, R, I, lda=I, ldb=I, ldo=self.ld, out_mode=5,
                   a_batch_stride=self.ld * I, b_batch_stride=R * I, out_batch_stride=R * self.ld, b_batch_kind=2, **many)
        return S.RoutedProj(e.moe_out, self.ld, route=e.slot_of, top=top, rows=R), gate


MLPS = {"dense": DenseMLP, "moe": RoutedExperts}


class TokenSide:
    """What a layer adds from its own part of the tokens' second embedding: norm(proj(gelu(gate x) * part))."""

    def __init__(self, layer: int, cfg: StackConfig, t: Dict[str, torch.Tensor], device, dtype):
        self.cfg, self.dim, self.col = cfg, cfg.token_side, layer * cfg.token_side
        self.w_gate, self.w_proj = Matrix(t["gate"], device, dtype), Matrix(t["proj"], device, dtype)
        self.norm = t["norm"].to(device=device, dtype=F32).contiguous()

    def matrices(self):
        return {"a": [(self.w_gate.n, self.w_gate.k)], "b": [(self.w_proj.n, self.w_proj.k)]}

    def run(self, e: "StackEngine", R: int) -> Tuple[Proj, Optional[Proj]]:
        z = e.project("gemm_side_gate", e.h, e.ldh, R, self.w_gate, e.planes_a, few=True)
        ld, table = self.w_proj.ld, e.w.side_embed
        e._run("side_act", e.k.ds41_side_act, C.byref(z.args()), lib.ptr(e.in_tokens), lib.ptr(table), C.c_longlong(table.shape[1]),
               self.col, self.cfg.vocab, R, self.dim, lib.ptr(e.act), ld, e.f32, lib.stream())
        return e.project("gemm_side_proj", e.act, ld, R, self.w_proj, e.planes_b), None


# ---------------------------------------------------------------------------------------------------- weights
@dataclass
class StackLayer:
    mixer: object
    norm1: torch.Tensor
    norm1b: Optional[torch.Tensor]
    bias1: Optional[torch.Tensor]
    mlp: object = None
    norm2: Optional[torch.Tensor] = None
    norm2b: Optional[torch.Tensor] = None
    bias2: Optional[torch.Tensor] = None
    mix: Optional[torch.Tensor] = None
    side: Optional[TokenSide] = None

    def parts(self):
        return [m for m in (self.mixer, self.mlp, self.side) if m is not None]


class StackWeights:
    """Kernel-layout weights built from a family's tensors: `get(l)` returns layer l's tensors under canonical names
    (mixer tensors "mix.*", feed-forward "mlp.*", "side.*", norms, "rg1" / "rg1.b" / "rg2" / "rg2.b", "dwa"); `top` has
    "embed", "final.norm", "head" (the same tensor as "embed" where they are tied) and "side.embed"."""

    def __init__(self, cfg: StackConfig, get, top: Dict[str, torch.Tensor], device, dtype: str = "bf16"):
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        dt = DTYPES[dtype]
        f32 = lambda x: x.to(device=device, dtype=F32).contiguous()
        self.embed = Matrix(top["embed"], device, BF16)
        self.final_norm = f32(top["final.norm"])
        self.head = self.embed if top["head"] is top["embed"] and dt == BF16 else Matrix(top["head"], device, dt)
        self.side_embed = top["side.embed"].to(device=device, dtype=BF16).contiguous() if cfg.token_side else None
        self.layers: List[StackLayer] = []
        for l, spec in enumerate(cfg.layers):
            t = get(l)
            part = lambda p: {n[len(p):]: x for n, x in t.items() if n.startswith(p)}
            gate = lambda n: {"w": t[n]} if cfg.residual_gate else {}
            bias = lambda n: f32(t[n]) if cfg.residual_gate else None
            post = lambda n: f32(t[n]) if cfg.post_norm else None
            lw = StackLayer(MIXERS[spec.mixer.kind](spec.mixer, cfg, part("mix."), gate("rg1"), device, dt),
                            f32(t["norm1"]), post("norm1b"), bias("rg1.b"))
            if spec.mlp is not None:
                lw.mlp = MLPS[spec.mlp.kind](spec.mlp, cfg, part("mlp."), gate("rg2"), device, dt)
                lw.norm2, lw.norm2b, lw.bias2 = f32(t["norm2"]), post("norm2b"), bias("rg2.b")
            if cfg.depth_average:
                lw.mix = f32(t["dwa"])
            if cfg.token_side:
                lw.side = TokenSide(l, cfg, part("side."), device, dt)
            self.layers.append(lw)

    def nbytes(self) -> int:
        seen, total, todo = set(), 0, [self]
        while todo:
            o = todo.pop()
            for v in (vars(o).values() if not isinstance(o, (list, tuple)) else o):
                if isinstance(v, torch.Tensor):
                    if v.untyped_storage().data_ptr() not in seen:
                        seen.add(v.untyped_storage().data_ptr())
                        total += v.untyped_storage().nbytes()
                elif isinstance(v, (list, Matrix, StackLayer, TokenSide) + tuple(MLPS.values()) + tuple(MIXERS.values())):
                    todo.append(v)
        return total


# ---------------------------------------------------------------------------------------------------- engine
class StackEngine(RowsEngine):
    partial_prefix = False        # recurrent states belong to a snapshot's whole length
    replay_window = 1 << 30       # the prefix banks then never prefer a truncated snapshot
    engram: dict = {}
    taps = None

    def __init__(self, cfg: StackConfig, weights: StackWeights, *, max_rows: int = 8, slots: int = 1, max_ctx: int = 4096,
                 page_tokens: int = 64, n_pages: Optional[int] = None, moe_rows: int = 32):
        self.cfg, self.w, self.device = cfg, weights, weights.device
        self.rank, self.world = 0, 1
        self.max_rows = R = max_rows
        self.n_layers = cfg.n_layers
        self.k = lib.kernels("stack")
        self.f32 = 1 if weights.dtype == "f32" else 0
        dev, dt = self.device, DTYPES[weights.dtype]
        self.cache = StackCache(cfg, slots, max_ctx, dev, dt, page_tokens, n_pages)
        z = lambda shape, d: torch.zeros(shape, dtype=d, device=dev)
        W = cfg.hidden
        # inputs
        self.in_tokens, self.row_pos = z((R,), I32), z((R,), I32)
        self.row_slot = torch.full((R,), -1, dtype=I32, device=dev)
        # residual streams: the kept result of every layer (depth average) and the working rows
        self.ldx = ceil_to(W, 4)
        self.kept = z((cfg.n_layers + 1 if cfg.depth_average else 1, R, self.ldx), F32)
        self.x_mid, self.x_avg = z((R, self.ldx), F32), z((R, self.ldx), F32)
        self.ldh = ceil_to(W, 8)
        self.h = z((R, self.ldh), dt)
        # projections
        need = {"a": 8, "b": 8}
        act = heads = q = 8
        q_rank = 8
        lat = 0
        self.attn_rows = min(R, 256)
        cells = 1
        for lw in weights.layers:
            for m in lw.parts():
                for b, ms in m.matrices().items():
                    for n, kk in ms:
                        need[b] = max(need[b], S.plane_floats(R, n, kk))
            mx = lw.mixer
            heads = max(heads, mx.spec.heads * mx.vp)
            if isinstance(lw.mlp, DenseMLP):
                act = max(act, lw.mlp.ffp)
            if lw.side is not None:
                act = max(act, lw.side.w_proj.ld)
            if isinstance(mx, GroupedAttention):
                q = max(q, mx.spec.heads * mx.dp)
            if isinstance(mx, LatentAttention):
                q = max(q, mx.spec.heads * mx.hs)
                q_rank = max(q_rank, mx.spec.q_rank)
                lat = max(lat, mx.spec.heads * mx.kvp)
                for n in range(1, self.attn_rows + 1):
                    cells = max(cells, n * self.attn_splits(n, mx.spec.heads) * mx.spec.heads * mx.kvp)
        self.planes_a, self.planes_b = z((need["a"],), F32), z((need["b"],), F32)
        # long passes: one request's rows with everything but the log gates and sublayer results in bf16
        self.long_rows = 64
        self.long_keys = 0            # > 0 during a long pass: positions its last row sees
        self.gathered = None
        wide = max(S.ceil_to(n, 8) for lw in weights.layers for m in lw.parts() for n, _ in m.matrices()["a"])
        self.wide = z((R * wide if R >= self.long_rows and not self.f32 else 8,), BF16)
        long_rec = [lw.mixer for lw in weights.layers if isinstance(lw.mixer, MLSTM) and lw.mixer.chunked] \
            if R >= self.long_rows else []
        self.recurrence_work = z((max([S.mlstm_chunk_work(R, m.spec.heads, m.dp, m.vp) for m in long_rec], default=0) // 4 + 4,),
                                 F32)
        self._keys = [z((8,), BF16) for _ in range(3)]
        self.act = z((R * max(act, heads),), dt)
        self.o_heads = z((R * heads,), F32)
        self.q = z((R * q,), dt)
        if lat:
            self.cq = z((R, ceil_to(q_rank, 8)), dt)
            self.q_abs, self.o_lat = z((self.attn_rows * lat,), dt), z((self.attn_rows * lat,), dt)
            self.part_o, self.part_ml = z((cells,), F32), z((cells // 8 + 2,), F32)
        self._init_experts(R, moe_rows, z, dt)
        # head
        self.head_cap = min(R, 64)
        self.last_head_row = 0
        self.logits = z((self.head_cap, cfg.vocab), F32)
        self.picked, self.pick_idx = z((self.head_cap, self.ldh), dt), z((self.head_cap,), I32)
        self.best_val, self.chosen = z((R,), F32), z((R,), I32)
        self.head_mask = None
        self._hint = None
        self.status = lib.new_status(dev)
        self._init_instruments()
        self.on_layer = None      # callable (layer, streams [rows, width]) after every layer of an eager pass

    def _init_experts(self, R: int, moe_rows: int, z, dt):
        """Routes, plans and buffers of the mixtures of experts: passes of at most `moe_rows` rows (32-bit passes: all) run
        every used expert over all rows, longer ones sort the rows by expert."""
        moes = [lw.mlp for lw in self.w.layers if isinstance(lw.mlp, RoutedExperts)]
        self.moe_rows = Rm = R if self.f32 else min(R, moe_rows)
        self._exchanges: Dict[tuple, object] = {}
        top = max([m.spec.top for m in moes], default=1)
        self.ids, self.route_w, self.slot_of = z((R * top,), I32), z((R * top,), F32), z((R * top,), I32)
        live = [(self.max_active(m.spec), m) for m in moes] or [(1, None)]
        most = max(n for n, _ in live)
        self.active, self.n_active, self.ticket = z((most,), I32), z((1,), I32), z((1,), I32)
        self.row_w = z((most * Rm,), F32)
        size = lambda f: max([n * Rm * f(m) for n, m in live if m is not None], default=8)
        self.moe_act, self.moe_out = z((size(lambda m: m.ffp),), dt), z((size(lambda m: m.ld),), F32)
        self.moe_up = z((size(lambda m: 2 * m.ffp) if self.f32 else 8,), F32)

    def max_active(self, m: MoESpec) -> int:
        """Most experts that a planned pass can use."""
        return min(m.experts, self.moe_rows * m.top)

    def exchange(self, m: RoutedExperts):
        """The sorted-rows form for experts of this shape, pointed at the layer's weights."""
        from ..parallel.ep import ExpertParallelMoE
        from ..parallel.fabric import Fabric
        sp = m.spec
        key = (sp.experts, sp.top, m.ffp, sp.limit, sp.alpha, sp.shift)
        if key not in self._exchanges:
            ep = ExpertParallelMoE(Fabric.single(self.device), m.w13, m.w2, topk=sp.top, max_tokens=self.max_rows,
                                   act_limit=sp.limit, act_alpha=sp.alpha, act_shift=sp.shift)
            ep.status = self.status
            self._exchanges[key] = ep
        self._exchanges[key].set_weights(m.w13, m.w2)
        return self._exchanges[key]

    # ------------------------------------------------------------------ helpers
    def attn_splits(self, rows: int, heads: int) -> int:
        """Key splits per row of the absorbed attention: enough blocks to fill the GPU about twice, static per batch
        size (a captured pass replays while the context grows)."""
        want = 2 * 148 // (rows * -(-heads // 32))
        return max(1, min(want, 32, -(-self.cache.max_ctx // 64)))

    def project(self, tag: str, x: torch.Tensor, ldx: int, rows: int, m: Matrix, buf: torch.Tensor, few: bool = False) -> Proj:
        """fp32 result of a projection; `few`: the matrix has few rows, which long passes take as the 128-row operand."""
        out: List[Proj] = []
        fn = S.project_few if few and rows > S.SWAP_ROWS and not self.f32 else S.project
        self._run(tag, lambda: out.append(fn(x, ldx, rows, m, buf, self.status)))
        return out[0] if out else S.Proj(buf, m.out_ld)

    def project_wide(self, tag: str, rows: int, m: Matrix) -> Proj:
        """bf16 result of a projection of self.h in a long pass."""
        self._run(tag, S.project_bf16, self.h, self.ldh, rows, m, self.wide, m.out_ld, self.status)
        return Proj(self.wide, m.out_ld)

    def key_space(self, n: int, kv_pad: int, rot_pad: int, width: int):
        """Buffers for one request's gathered latent rows, rotated key parts and expanded keys / values (they grow)."""
        for i, w in enumerate((kv_pad, rot_pad, width)):
            if self._keys[i].numel() < n * w:
                self.gathered = None
                self._keys[i] = torch.zeros(ceil_to(n, 1024) * w, dtype=BF16, device=self.device)
        return self._keys

    def _enter_rehearsal(self):
        self.row_slot.fill_(-1)       # no row owns a slot: caches and states keep what they hold

    def set_rows(self, tokens, positions, slots, row_hi=None, row_lo=None):
        """Host -> device copy of one pass's inputs.  Rows of one slot are adjacent, at consecutive positions."""
        assert row_lo is None and row_hi is None, "a layer stack has no window floor"
        n = len(positions)
        assert n <= self.max_rows
        slots, positions, seen = list(slots), list(positions), set()
        for i in range(n):
            if slots[i] < 0:
                continue
            if i and slots[i] == slots[i - 1]:
                assert positions[i] == positions[i - 1] + 1, "rows of a request must follow one another"
            else:
                assert slots[i] not in seen, "rows of a request must be adjacent"
                seen.add(slots[i])
        # what the host knows about the pass it just described: a long pass of one request
        one = n >= self.long_rows and len(seen) == 1 and min(slots) >= 0 and not self.f32
        self._hint = (n, positions[-1] + 1) if one else None
        pad = self.max_rows - n
        if tokens is not None:
            assert len(tokens) == n
            self.in_tokens.copy_(torch.tensor(list(tokens) + [0] * pad, dtype=I32), non_blocking=True)
        self.row_pos.copy_(torch.tensor(positions + [0] * pad, dtype=I32), non_blocking=True)
        self.row_slot.copy_(torch.tensor(slots + [-1] * pad, dtype=I32), non_blocking=True)

    def _resid(self, R: int, *, y: Optional[Proj] = None, gate: Optional[Proj] = None, bias=None, post=None, x_in=None,
               x_out=None, layer: Optional[int] = None, next_w=None, post_rms: bool = False):
        """`next_w`: weight of the norm that opens the next sublayer, None: that sublayer reads the stream itself."""
        a = S.ResidArgs()
        cfg = self.cfg
        a.y, a.gate = (y.args() if y is not None else S.NO_PROJ), (gate.args() if gate is not None else S.NO_PROJ)
        a.gate_bias, a.post_w, a.next_w = lib.ptr(bias), lib.ptr(post), lib.ptr(next_w)
        if x_in is None:
            a.tokens, a.embed, a.embed_ld = lib.ptr(self.in_tokens), lib.ptr(self.w.embed.w), self.w.embed.ld
        a.x_in, a.x_out = lib.ptr(x_in), lib.ptr(x_out)
        if layer is not None:
            a.mix, a.kept, a.kept_stride = lib.ptr(self.w.layers[layer].mix), lib.ptr(self.kept), self.kept.stride(0)
            a.n_mix, a.x_avg = layer + 2, lib.ptr(self.x_avg)
        a.h, a.ldh, a.ldx, a.vocab, a.rows, a.W = lib.ptr(self.h), self.ldh, self.ldx, cfg.vocab, R, cfg.hidden
        a.norm_kind, a.eps, a.f32 = cfg.norm_kind, cfg.norm_eps, self.f32
        a.raw_h, a.post_rms = int(next_w is None), int(post_rms)
        if isinstance(y, S.RoutedProj):
            a.y_route, a.y_top, a.y_rows = lib.ptr(y.route), y.top, y.rows
        self._run("resid_step", self.k.ds41_resid_step, C.byref(a), lib.stream())

    # ------------------------------------------------------------------ one pass
    def forward_rows(self, rows: int, *, head: bool = True, head_row: Optional[int] = None, sources: bool = True):
        """One pass over the `rows` rows described by set_rows()."""
        cfg, R, layers = self.cfg, rows, self.w.layers
        self.long_keys = self._hint[1] if self._hint is not None and self._hint[0] == R else 0
        self._hint = self.gathered = None
        if self.layer_timer is not None:
            self.layer_timer.begin()
        cur = self.kept[0]
        self._resid(R, x_out=cur, next_w=layers[0].norm1)
        for l, lw in enumerate(layers):
            after = layers[l + 1].norm1 if l + 1 < len(layers) else self.w.final_norm
            # (run, norm of its input, what follows its result) of the layer's sublayers
            subs = [(lambda: lw.mixer.run(self, l, R, cfg.source_of(l)), lw.norm1, dict(bias=lw.bias1, post=lw.norm1b))]
            if lw.mlp is not None:
                subs.append((lambda: lw.mlp.run(self, R), lw.norm2, dict(bias=lw.bias2, post=lw.norm2b)))
            if lw.side is not None:
                subs.append((lambda: lw.side.run(self, R), None, dict(post=lw.side.norm, post_rms=True)))
            for i, (run, _, closing) in enumerate(subs):
                y, gate = run()
                if i + 1 < len(subs):
                    self._resid(R, y=y, gate=gate, x_in=cur, x_out=self.x_mid, next_w=subs[i + 1][1], **closing)
                    cur = self.x_mid
                else:
                    self._resid(R, y=y, gate=gate, x_in=cur, x_out=self.kept[l + 1] if cfg.depth_average else self.kept[0],
                                layer=l if cfg.depth_average else None, next_w=after, **closing)
            cur = self.x_avg if cfg.depth_average else self.kept[0]
            if self.layer_timer is not None:
                self.layer_timer.mark()
            if self.activation_trace is not None:
                self.activation_trace.dump(l, cur[:, :cfg.hidden], self.row_pos, R)
            if self.on_layer is not None:
                self.on_layer(l, cur[:R, :cfg.hidden])
        if head:
            self.head_rows(R if head_row is None else head_row + 1)

    def _head_gemm(self, x: torch.Tensor, rows: int):
        m = self.w.head
        if self.f32:
            self._run("gemm_head", S.gemm_f32, x, m.w, self.logits, rows, m.n, m.k, self.ldh, m.ld, self.cfg.vocab)
            if self.cfg.logit_softcap:
                self._run("softcap_rows", self.k.ds41_softcap_rows, lib.ptr(self.logits), C.c_longlong(rows * self.cfg.vocab),
                          C.c_float(self.cfg.logit_softcap), lib.stream())
        else:
            from ..ops import gemm as G
            self._run("gemm_head", G.gemm_raw, m.w, x, self.logits, m.n, rows, m.k, lda=m.ld, ldb=self.ldh,
                      ldo=self.cfg.vocab, out_mode=3, status=self.status, static_operand=1, softcap=self.cfg.logit_softcap)

    def head_rows(self, rows: int, mask: Optional[torch.Tensor] = None):
        """Logits and greedy choice of the pass's rows; a long pass only needs its last row, whose logits land in row 0."""
        if mask is None:
            mask = self.head_mask
        x, self.last_head_row = self.h, rows - 1
        if rows > self.head_cap:
            x, rows, self.last_head_row = self.h[rows - 1:rows], 1, 0
        self._head_gemm(x, rows)
        V = self.cfg.vocab
        self._run("argmax_rows", self.k.ds41_argmax_rows, lib.ptr(self.logits), C.c_longlong(V), rows, V, 0, lib.ptr(mask),
                  0 if mask is None else mask.shape[-1], lib.ptr(self.best_val), lib.ptr(self.chosen), lib.ptr(None),
                  lib.stream())

    def logits_rows(self, rows: int) -> torch.Tensor:
        return self.logits[:rows].clone()

    def logits_at(self, rows: Sequence[int]) -> torch.Tensor:
        """fp32 logits of any rows of the last pass (run with head=False or True), [len(rows), vocab]."""
        out = []
        for i in range(0, len(rows), self.head_cap):
            part = list(rows[i:i + self.head_cap])
            n = len(part)
            self.pick_idx[:n].copy_(torch.tensor(part, dtype=I32))
            self._run("gather_rows", self.k.ds41_gather_rows, lib.ptr(self.h), self.ldh, lib.ptr(self.pick_idx),
                      self.max_rows, n, self.cfg.hidden, lib.ptr(self.picked), self.f32, lib.stream())
            self._head_gemm(self.picked, n)
            out.append(self.logits[:n].clone())
        return torch.cat(out) if out else torch.empty(0, self.cfg.vocab, device=self.device)
