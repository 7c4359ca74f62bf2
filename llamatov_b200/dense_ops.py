"""Operators of the dense (bf16 / fp32) models as objects: packed matrices, norms, epilogues and prologues of their
launches (include/llamatov_b200_dense.h).

Matrices are packed with head sizes and row lengths padded to multiples of 8 with zeros, so kernels need no ragged edges.
"""
import ctypes

import torch

from . import _lib
from . import dev_residency as dr

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def pad8(n):
    return (n + 7) // 8 * 8


# --------------------------------------------------------------------------- packing helpers

def _head_rows(W, sizes, heads):
    """Rows of a projection laid out head by head, each head `sizes` = [(n, padded n), ...] consecutive pieces."""
    per = sum(n for n, _ in sizes)
    W = W.reshape(heads, per, *W.shape[1:])
    parts, r = [], 0
    for n, p in sizes:
        piece = W[:, r:r + n]
        r += n
        if p > n:
            piece = torch.cat([piece, piece.new_zeros((heads, p - n) + tuple(W.shape[2:]))], dim=1)
        parts.append(piece)
    out = torch.cat(parts, dim=1)
    return out.reshape(-1, *W.shape[2:])


def _head_cols(W, n, heads):
    """Columns of an output projection, each head's n padded to a multiple of 8."""
    return _head_rows(W.T.contiguous(), [(n, pad8(n))], heads).T.contiguous()


def _pad_cols(W, k):
    return W if W.shape[1] == k else torch.cat([W, W.new_zeros(W.shape[0], k - W.shape[1])], dim=1)


def _pad_rows(W, n):
    return W if W.shape[0] == n else torch.cat([W, W.new_zeros((n - W.shape[0],) + tuple(W.shape[1:]))], dim=0)


# --------------------------------------------------------------------------- launch helpers

class Linear:
    """A packed matrix on the device: rows() over token rows, row() for one token with the input made in the kernel."""

    def __init__(self, W, dtype):
        W = _pad_cols(W.to(dtype), pad8(W.shape[1])).contiguous()
        self.M, self.K = W.shape
        self.f32 = int(dtype == torch.float32)
        self.W = W.cuda()
        self.ptr = self.W.data_ptr()

    def rows(self, x, ldx, y, ldy, T, epi, M=None, first=0):
        """Outputs of the matrix rows from `first` on, M of them (gated: M gate rows, then M up rows)."""
        _lib.call("lt_dn_linear", self.ptr + first * self.K * self.W.element_size(), self.K, x, ldx, y, ldy, self.f32,
                  self.M - first if M is None else M, self.K, T, ctypes.byref(epi), 0, dr._stream())

    def row(self, pro, y, epi, M=None):
        _lib.call("lt_dn_gemv", self.ptr, self.K, y, self.f32, self.M if M is None else M, self.K, ctypes.byref(pro),
                  ctypes.byref(epi), dr._stream())


def epilogue(kind=_lib.DN_STORE, segs=(), bias=None, ls=None, out_f32=False, glu=None, tail_from=None):
    """segs: (end, activation name or None, scale) per output segment.  glu: (act, alpha, limit) of gated outputs.
    tail_from: outputs from there on go to an fp32 buffer (`with_tail`)."""
    e = _lib.DnEpilogue()
    e.kind, e.out_f32, e.nseg = kind, int(out_f32), len(segs)
    for i, (end, act, scale) in enumerate(segs):
        e.seg_end[i], e.seg_act[i], e.seg_scale[i] = end, _lib.DN_ACT[act], scale
    e.bias = None if bias is None else bias.data_ptr()
    e.ls = None if ls is None else ls.data_ptr()
    if glu is not None:
        e.glu_act, e.glu_alpha, e.glu_limit = glu
    if tail_from is not None:
        e.tail_from = tail_from
    return e


def with_tail(epi, tail, ld):
    """The epilogue with its fp32 tail at `tail`, row stride ld."""
    e = _lib.DnEpilogue.from_buffer_copy(epi)
    e.tail, e.ldtail = tail, ld
    return e


class Norm:
    """RMS norm over groups of `group` (padded) elements of which `count` are real; weight repeats every w_period.
    gate_first: a gate multiplies ahead of the norm.  seg = (n, padded n): groups of `count` real elements that do not
    follow the padded segments."""

    def __init__(self, w, count, group, eps, gate_first=False, seg=None):
        self.w = w.float().cuda().contiguous()
        self.count, self.group, self.eps = int(count), int(group), float(eps)
        self.gate_first = int(gate_first)
        self.seg, self.segp = seg or (0, 0)

    def prologue(self, x, gate=None):
        return _lib.DnPrologue(_lib.DN_IN_NORM, 0, self.group, self.count, self.eps, x, None, self.w.data_ptr(),
                               self.w.numel(), gate, self.gate_first, self.seg, self.segp)

    def rows(self, x, ldx, y, ldy, f32, T, N, gate=None, ldg=0, index=None):
        _lib.call("lt_dn_norm_rows", x, ldx, index, self.w.data_ptr(), self.w.numel(), gate, ldg, y, ldy, f32, T, N,
                  self.group, self.count, self.eps, self.gate_first, self.seg, self.segp, dr._stream())


def typed_input(x):
    return _lib.DnPrologue(_lib.DN_IN_TYPED, 0, 0, 0, 0.0, x, None, None, 0, None, 0, 0, 0)


def cast_input(x, n1, x2=None):
    return _lib.DnPrologue(_lib.DN_IN_CAST, n1, 0, 0, 0.0, x, x2, None, 0, None, 0, 0, 0)
