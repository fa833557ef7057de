"""Front end of the layer-stack kernels (csrc/kernels/stack_ops.cu, latent_attn.cu, group_attn.cu, mlstm.cu, moe.cu, gemm_f32.cu)
and the projection helper that the stack engine's matrix products go through."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Dict, Optional, Sequence, Tuple

import torch

from . import gemm as G
from . import lib

BF16 = torch.bfloat16
F32 = torch.float32


def ceil_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class ProjArgs(C.Structure):
    _fields_ = [("data", C.c_void_p), ("plane", C.c_longlong), ("ld", C.c_int), ("splits", C.c_int), ("bf16", C.c_int),
                ("col", C.c_int)]


class ResidArgs(C.Structure):
    _fields_ = [("y", ProjArgs), ("gate", ProjArgs), ("gate_bias", C.c_void_p), ("post_w", C.c_void_p),
                ("tokens", C.c_void_p), ("embed", C.c_void_p), ("embed_ld", C.c_longlong), ("x_in", C.c_void_p),
                ("x_out", C.c_void_p), ("mix", C.c_void_p), ("kept", C.c_void_p), ("kept_stride", C.c_longlong),
                ("x_avg", C.c_void_p), ("next_w", C.c_void_p), ("h", C.c_void_p), ("ldx", C.c_longlong),
                ("ldh", C.c_int), ("n_mix", C.c_int), ("vocab", C.c_int), ("rows", C.c_int), ("W", C.c_int),
                ("norm_kind", C.c_int), ("eps", C.c_float), ("f32", C.c_int), ("y_route", C.c_void_p), ("y_top", C.c_int),
                ("y_rows", C.c_int), ("raw_h", C.c_int), ("post_rms", C.c_int)]


class LatentPostArgs(C.Structure):
    _fields_ = [("dq", ProjArgs), ("kv", ProjArgs), ("kr", ProjArgs), ("dq_norm", C.c_void_p), ("kv_norm", C.c_void_p),
                ("freq", C.c_void_p), ("cq", C.c_void_p), ("pool", C.c_void_p), ("page_table", C.c_void_p),
                ("row_pos", C.c_void_p), ("row_slot", C.c_void_p), ("magnitude", C.c_float), ("eps", C.c_float),
                ("rows", C.c_int), ("q_rank", C.c_int), ("ld_cq", C.c_int), ("kv_rank", C.c_int), ("kv_pad", C.c_int),
                ("rot_dim", C.c_int), ("row_len", C.c_int), ("max_pages", C.c_int), ("page_tokens", C.c_int),
                ("f32", C.c_int)]


class LatentAttendArgs(C.Structure):
    _fields_ = [("q_abs", C.c_void_p), ("q_rot", C.c_void_p), ("pool", C.c_void_p), ("page_table", C.c_void_p),
                ("row_pos", C.c_void_p), ("row_slot", C.c_void_p), ("part_o", C.c_void_p), ("part_ml", C.c_void_p),
                ("ld_q_abs", C.c_longlong), ("ld_q_rot", C.c_longlong), ("scale", C.c_float), ("rows", C.c_int),
                ("heads", C.c_int), ("kv_pad", C.c_int), ("row_len", C.c_int), ("q_rot_stride", C.c_int),
                ("n_splits", C.c_int), ("max_pages", C.c_int), ("page_tokens", C.c_int), ("f32", C.c_int)]


class LatentPrefillArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("kv", C.c_void_p), ("rot", C.c_void_p), ("sink", C.c_void_p), ("out", C.c_void_p),
                ("status", C.c_void_p), ("gate", ProjArgs), ("ld_q", C.c_longlong), ("ld_kv", C.c_longlong),
                ("scale", C.c_float), ("rows", C.c_int), ("heads", C.c_int), ("dim_pad", C.c_int), ("rot_pad", C.c_int),
                ("vdim_pad", C.c_int), ("n_keys", C.c_int), ("pos0", C.c_int), ("ld_out", C.c_int)]


class MlstmArgs(C.Structure):
    _fields_ = [("q", ProjArgs), ("k", ProjArgs), ("v", ProjArgs), ("gate_i", ProjArgs), ("gate_f", ProjArgs),
                ("bias_i", C.c_void_p), ("bias_f", C.c_void_p), ("row_pos", C.c_void_p), ("row_slot", C.c_void_p),
                ("state_s", C.c_void_p), ("state_n", C.c_void_p), ("state_m", C.c_void_p), ("out", C.c_void_p),
                ("work", C.c_void_p), ("gate_cap", C.c_float), ("q_scale", C.c_float), ("den_eps", C.c_float), ("rows", C.c_int),
                ("heads", C.c_int), ("dim_pad", C.c_int), ("vdim_pad", C.c_int), ("slots", C.c_int), ("ld_out", C.c_int)]


class AttnPostArgs(C.Structure):
    _fields_ = [("u", ProjArgs), ("conv", C.c_void_p), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("freq", C.c_void_p),
                ("state", C.c_void_p), ("q", C.c_void_p), ("pool", C.c_void_p), ("page_table", C.c_void_p),
                ("row_pos", C.c_void_p), ("row_slot", C.c_void_p), ("ld_q", C.c_longlong), ("eps", C.c_float),
                ("rows", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("dim_pad", C.c_int),
                ("vdim_pad", C.c_int), ("rot_dim", C.c_int), ("taps", C.c_int), ("slots", C.c_int), ("max_pages", C.c_int),
                ("page_tokens", C.c_int), ("f32", C.c_int)]


class GroupAttendArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("pool", C.c_void_p), ("page_table", C.c_void_p), ("row_pos", C.c_void_p),
                ("row_slot", C.c_void_p), ("out", C.c_void_p), ("status", C.c_void_p), ("gate", ProjArgs), ("u", ProjArgs),
                ("state", C.c_void_p), ("ld_q", C.c_longlong), ("scale", C.c_float), ("rows", C.c_int), ("heads", C.c_int),
                ("kv_heads", C.c_int), ("dim_pad", C.c_int), ("vdim_pad", C.c_int), ("chunk", C.c_int), ("taps", C.c_int),
                ("slots", C.c_int), ("n_splits", C.c_int), ("ld_out", C.c_int), ("max_pages", C.c_int),
                ("page_tokens", C.c_int), ("f32", C.c_int), ("n_pages", C.c_int), ("pos0", C.c_int)]


class RouteArgs(C.Structure):
    _fields_ = [("z", ProjArgs), ("bias", C.c_void_p), ("row_slot", C.c_void_p), ("ids", C.c_void_p), ("weights", C.c_void_p),
                ("active", C.c_void_p), ("n_active", C.c_void_p), ("row_w", C.c_void_p), ("slot_of", C.c_void_p),
                ("ticket", C.c_void_p), ("rows", C.c_int), ("experts", C.c_int), ("top", C.c_int), ("max_active", C.c_int),
                ("row_w_ld", C.c_int)]


def mlstm_chunk_work(rows: int, heads: int, dim_pad: int, vdim_pad: int) -> int:
    """Bytes of workspace of the chunked recurrence (mostly the state before every chunk)."""
    fn = lib.kernels("stack").ds41_mlstm_chunk_work
    fn.restype = C.c_longlong
    return fn(rows, heads, dim_pad, vdim_pad)


STATE_COLS = 32       # value columns per state block of the mLSTM kernels (kStateCols)


@dataclass
class Proj:
    """A projection's result as its consumer reads it (ds41_proj)."""
    data: torch.Tensor
    ld: int
    splits: int = 1
    plane: int = 0
    col: int = 0

    def at(self, col: int) -> "Proj":
        return Proj(self.data, self.ld, self.splits, self.plane, self.col + col)

    def args(self) -> ProjArgs:
        return ProjArgs(self.data.data_ptr(), self.plane, self.ld, self.splits, 1 if self.data.dtype == BF16 else 0, self.col)


@dataclass
class RoutedProj(Proj):
    """Rows of routed experts whose sum is a pass row's result: row route[r * top + k] * rows + r, or, with rows = 0, one row
    per route; negative routes count for nothing."""
    route: Optional[torch.Tensor] = None
    top: int = 1
    rows: int = 0


NO_PROJ = ProjArgs(None, 0, 0, 0, 0, 0)


class Matrix:
    """A weight matrix in kernel layout: `n` rows of `k` values, rows `ld` apart (16-byte aligned for the copy engine)."""

    def __init__(self, w: torch.Tensor, device, dtype):
        self.n, self.k = w.shape
        self.ld = ceil_to(self.k, 8)
        self.w = torch.zeros(self.n, self.ld, dtype=dtype, device=device)
        self.w[:, :self.k] = w.to(device=device, dtype=dtype)

    def rows(self, lo: int, hi: int) -> "Matrix":
        """Some of the rows, sharing the storage."""
        m = object.__new__(Matrix)
        m.n, m.k, m.ld, m.w = hi - lo, self.k, self.ld, self.w[lo:hi]
        return m

    @property
    def out_ld(self) -> int:
        return ceil_to(self.n, 8)


def stack_rows(parts: Sequence[Tuple[str, torch.Tensor]], device, dtype) -> Tuple[Matrix, Dict[str, int]]:
    """Weights that read the same input as one matrix; every part starts at a multiple of 8 columns of the result."""
    at, rows, cur = {}, [], 0
    for name, t in parts:
        at[name] = cur
        rows.append(t)
        pad = ceil_to(t.shape[0], 8) - t.shape[0]
        if pad:
            rows.append(t.new_zeros(pad, t.shape[1]))
        cur += t.shape[0] + pad
    return Matrix(torch.cat(rows, 0), device, dtype), at


def pad_heads(t: torch.Tensor, heads: int, width: int, padded: int) -> torch.Tensor:
    """[heads * width, ...] -> [heads * padded, ...] with zero rows at the end of every head."""
    if width == padded:
        return t
    out = t.new_zeros(heads, padded, *t.shape[1:])
    out[:, :width] = t.view(heads, width, *t.shape[1:])
    return out.view(heads * padded, *t.shape[1:])


SWAP_ROWS = 128      # up to this many rows the weights fill the 128-row operand of the tensor-core tile (swap-AB, split K)


def plane_floats(rows: int, n: int, k: int) -> int:
    """fp32 values that project() can need for passes of up to `rows` rows against an [n, k] matrix."""
    few = min(rows, SWAP_ROWS)
    return max(rows, few * _splits(n, k, few)) * ceil_to(n, 8)


def _splits(n: int, k: int, rows: int) -> int:
    return G.pick_splits(n, k, max_splits=16, n_tiles=-(-rows // G.pick_bn(rows)))


def project(x: torch.Tensor, ldx: int, rows: int, m: Matrix, buf: torch.Tensor, status) -> Proj:
    """x[rows, k] (leading dimension ldx) times the matrix -> fp32 planes in `buf`."""
    ldo = m.out_ld
    if x.dtype == F32:
        gemm_f32(x, m.w, buf, rows, m.n, m.k, ldx, m.ld, ldo)
        return Proj(buf, ldo)
    if rows <= SWAP_ROWS:
        s = _splits(m.n, m.k, rows)
        G.gemm_raw(m.w, x, buf if s == 1 else None, m.n, rows, m.k, lda=m.ld, ldb=ldx, ldo=ldo, out_mode=3, k_splits=s,
                   split_workspace=buf if s > 1 else None, status=status, static_operand=1)
        return Proj(buf, ldo, s, rows * ldo)
    G.gemm_raw(x, m.w, buf, rows, m.n, m.k, lda=ldx, ldb=m.ld, ldo=ldo, out_mode=1, bn=_wide_bn(m.n), status=status,
               static_operand=2)
    return Proj(buf, ldo)


def project_bf16(x: torch.Tensor, ldx: int, rows: int, m: Matrix, out: torch.Tensor, ldo: int, status) -> None:
    """The same with a bf16 result (long passes: half the bytes for the consumer)."""
    G.gemm_raw(x, m.w, out, rows, m.n, m.k, lda=ldx, ldb=m.ld, ldo=ldo,
               out_mode=6 if m.n >= 64 and ldo % 8 == 0 else 0, bn=_wide_bn(m.n), status=status, static_operand=2)


def project_few(x: torch.Tensor, ldx: int, rows: int, m: Matrix, buf: torch.Tensor, status) -> Proj:
    """fp32 result of a matrix with few rows, for any number of activation rows (weights as the 128-row operand)."""
    n_tiles = -(-rows // 128)
    s = G.pick_splits(m.n, m.k, max_splits=16, n_tiles=n_tiles)
    while s > 1 and s * rows * m.out_ld > buf.numel():
        s -= 1
    G.gemm_raw(m.w, x, buf if s == 1 else None, m.n, rows, m.k, lda=m.ld, ldb=ldx, ldo=m.out_ld, out_mode=3, k_splits=s,
               split_workspace=buf if s > 1 else None, bn=G.pick_bn(rows), status=status, static_operand=1)
    return Proj(buf, m.out_ld, s, rows * m.out_ld)


def _wide_bn(n: int) -> int:
    return 256 if n >= 256 else (128 if n >= 128 else 64)


def per_head(x: torch.Tensor, ldx: int, head_stride: int, rows: int, heads: int, w: torch.Tensor, n: int, k: int, ldw: int,
             out: torch.Tensor, ldo: int, status) -> None:
    """out[r, h * n + j] = sum_k w[h, j, k] * x[r, h * head_stride + k]: one small matrix per head."""
    if x.dtype == F32:
        gemm_f32(x, w, out, rows, n, k, ldx, ldw, ldo, batch=heads, sa=head_stride, sb=n * ldw, so=n)
        return
    G.gemm_raw(w, x, out, n, rows, k, lda=ldw, ldb=ldx, ldo=ldo, out_mode=2 if out.dtype == BF16 else 3, batch=heads,
               a_batch_stride=n * ldw, b_batch_stride=head_stride, out_batch_stride=n, status=status, static_operand=1)


def gemm_f32(a, b, out, M, N, K, lda, ldb, ldo, batch=1, sa=0, sb=0, so=0, batch_map=None, n_active=None):
    ll = C.c_longlong
    lib.check(lib.kernels("stack").ds41_gemm_f32(lib.ptr(a), lib.ptr(b), lib.ptr(out), M, N, K, ll(lda), ll(ldb), ll(ldo), batch,
                                          ll(sa), ll(sb), ll(so), lib.ptr(batch_map), lib.ptr(n_active),
                                                 lib.stream()), "ds41_gemm_f32")
